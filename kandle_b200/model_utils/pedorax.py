"""Configuration of the Pedorax design: a decoder whose layers are a free list of mixers (latent
attention, channel-wise gated delta rule), each beside an optional expert feed-forward that reads the same
Dynamic Tanh norm.  Parsed from the design's config.json; nothing here touches the device."""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass(frozen=True)
class LatentAttentionSpec:
    heads: int
    dim: int                  # unrotated query/key dimensions per head
    rotDim: int               # rotated ones (shared key part)
    vdim: int
    kvRank: int
    scale: float
    rotBase: float
    kvFrom: int | None = None  # layer whose cached rows this layer reads instead of its own


@dataclass(frozen=True)
class ChannelDeltaSpec:
    heads: int
    kvHeads: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self) -> int:      # channels that pass the short convolution: q, k, v side by side
        return 2 * self.kvHeads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    groups: int
    keep: int
    ff: int
    limit: float


@dataclass(frozen=True)
class HybridLayerSpec:
    mixer: LatentAttentionSpec | ChannelDeltaSpec
    experts: ExpertsSpec | None


@dataclass
class PedoraxConfig:
    vocabSize: int
    hiddenSize: int
    layers: list = field(default_factory=list)
    embeddingScale: float = 1.0
    logitScale: float = 1.0
    normEps: float = 1e-6
    dtype: str = "bfloat16"

    @classmethod
    def fromDict(cls, c: dict, dtype: str = "bfloat16") -> "PedoraxConfig":
        layers = [HybridLayerSpec(_mixer(e["type"], e["mixer"]), _experts(e.get("mlp"))) for e in c["layers"]]
        cfg = cls(int(c["vocab"]), int(c["width"]), layers, float(c["embedding"]["scale"]), float(c["logit_scale"]),
                  float(c["norm"]["eps"]), dtype)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("the model has no layers")
        for i, layer in enumerate(self.layers):
            m, e = layer.mixer, layer.experts
            if isinstance(m, LatentAttentionSpec):
                if m.rotDim % 2:
                    raise ValueError(f"layer {i}: rot_dim {m.rotDim} is odd")
                if m.kvFrom is not None:
                    src = self.layers[m.kvFrom].mixer if 0 <= m.kvFrom < i else None
                    if not isinstance(src, LatentAttentionSpec) or src.kvFrom is not None:
                        raise ValueError(f"layer {i}: kv_from {m.kvFrom} is not an earlier latent-attention layer with rows of its own")
                    if (src.kvRank, src.rotDim, src.rotBase) != (m.kvRank, m.rotDim, m.rotBase):
                        raise ValueError(f"layer {i}: latent sizes or rotation differ from layer {m.kvFrom}, whose rows it reads")
            elif m.heads % m.kvHeads:
                raise ValueError(f"layer {i}: {m.heads} heads over {m.kvHeads} key heads")
            if e is not None and (e.experts % e.groups or not 1 <= e.keep <= e.groups or not 1 <= e.top <= e.keep * (e.experts // e.groups)):
                raise ValueError(f"layer {i}: {e.experts} experts in {e.groups} groups, {e.keep} kept, top {e.top}")


def _mixer(kind: str, m: dict):
    if kind == "latent_attention":
        rot = m["rot"]
        if int(rot["dims"]) != int(m["rot_dim"]):
            raise ValueError(f"rot.dims {rot['dims']} must equal rot_dim {m['rot_dim']}")
        src = m.get("kv_from")
        return LatentAttentionSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                   float(m["scale"]), float(rot["base"]), None if src is None else int(src))
    if kind == "channel_delta":
        return ChannelDeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
    raise ValueError(f"unknown mixer {kind!r}")


def _experts(m: dict | None):
    if m is None:
        return None
    if m.get("kind", "moe") != "moe":
        raise ValueError(f"unknown feed-forward {m['kind']!r}")
    r, x = m["router"], m["expert"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    return ExpertsSpec(int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]), int(x["ff"]), float(x["limit"]))
