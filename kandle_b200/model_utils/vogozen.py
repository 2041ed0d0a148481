"""Configuration of the Vogozen design: a decoder whose layers are a free list of mixers (sliding-window
attention, WKV time mixing, gated delta rule with one decay per head), each followed by an optional dense
feed-forward, with the norms on the sublayers' outputs.  Parsed from the design's config.json; nothing here
touches the device."""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass(frozen=True)
class WindowAttentionSpec:
    heads: int
    kvHeads: int
    dim: int                  # query/key size of a head
    vdim: int
    scale: float
    rotBase: float
    rotDims: int              # rotated dimensions at the front of a head
    window: int               # keys a query sees, itself included
    kvFrom: int | None = None  # layer whose cached keys and values this layer reads instead of its own


@dataclass(frozen=True)
class WkvSpec:
    heads: int
    dim: int


@dataclass(frozen=True)
class HeadDeltaSpec:
    heads: int
    kvHeads: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self) -> int:      # channels that pass the short convolution: q, k, v side by side
        return 2 * self.kvHeads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class SequentialLayerSpec:
    mixer: WindowAttentionSpec | WkvSpec | HeadDeltaSpec
    dense: DenseSpec | None


@dataclass
class VogozenConfig:
    vocabSize: int
    hiddenSize: int
    layers: list = field(default_factory=list)
    normEps: float = 1e-6
    dtype: str = "bfloat16"

    @classmethod
    def fromDict(cls, c: dict, dtype: str = "bfloat16") -> "VogozenConfig":
        layers = [SequentialLayerSpec(_mixer(e["type"], e["mixer"]), _dense(e.get("mlp"))) for e in c["layers"]]
        cfg = cls(int(c["vocab"]), int(c["width"]), layers, float(c["norm"]["eps"]), dtype)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("the model has no layers")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, WkvSpec):
                continue
            if m.heads % m.kvHeads:
                raise ValueError(f"layer {i}: {m.heads} heads over {m.kvHeads} key heads")
            if isinstance(m, HeadDeltaSpec):
                continue
            if m.rotDims % 2 or not 0 <= m.rotDims <= m.dim:
                raise ValueError(f"layer {i}: {m.rotDims} rotated of {m.dim} dimensions")
            if m.window < 1:
                raise ValueError(f"layer {i}: a window of {m.window}")
            if m.kvFrom is not None:
                src = self.layers[m.kvFrom].mixer if 0 <= m.kvFrom < i else None
                if not isinstance(src, WindowAttentionSpec) or src.kvFrom is not None:
                    raise ValueError(f"layer {i}: kv_from {m.kvFrom} is not an earlier attention layer with keys and values of its own")
                if (src.kvHeads, src.dim, src.vdim) != (m.kvHeads, m.dim, m.vdim):
                    raise ValueError(f"layer {i}: head counts or sizes differ from layer {m.kvFrom}, whose keys and values it reads")


def _mixer(kind: str, m: dict):
    if kind == "attention":
        rot, src = m["rot"], m.get("kv_from")
        return WindowAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), float(rot["base"]),
                                   int(rot["dims"]), int(m["mask"]["size"]), None if src is None else int(src))
    if kind == "wkv":
        return WkvSpec(int(m["heads"]), int(m["dim"]))
    if kind == "delta":
        return HeadDeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
    raise ValueError(f"unknown mixer {kind!r}")


def _dense(m: dict | None):
    if m is None:
        return None
    if m.get("kind", "dense") != "dense":
        raise ValueError(f"unknown feed-forward {m['kind']!r}")
    return DenseSpec(int(m["ff"]))
