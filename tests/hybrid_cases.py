"""Small random models of the hybrid designs (Pedorax here, Vogozen in vogozen_cases.py) for the tests:
configurations, weights (rounded to bf16, so that both sides see the same numbers) and comparisons with the plain
implementations in oracle/hybrid.py and oracle/vogozen.py."""
from __future__ import annotations

import numpy as np

from kandle_b200 import lib, registry
from oracle import hybrid, vogozen

ORACLES = {"Pedorax": hybrid, "Vogozen": vogozen}


def latent(heads=3, dim=24, rot=16, vdim=40, rank=48, scale=0.2, base=5000.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def delta(heads=4, kv_heads=2, dim=40, vdim=24, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(experts=12, top=3, groups=4, keep=2, ff=40, limit=1.2):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


def config(layers, vocab=150, width=72, embed=2.5, logit=0.7, eps=1e-5):
    return {"architecture": "Pedorax", "vocab": vocab, "width": width, "embedding": {"scale": embed}, "logit_scale": logit,
            "norm": {"eps": eps}, "layers": [dict(layer, mlp=mlp) for layer, mlp in layers]}


def mixed_config(**kw):
    """Every branch: an own latent, a delta layer whose key heads are shared, a layer that reads the first one's rows with
    other head counts, a layer without feed-forward, routers of different sizes."""
    return config([(latent(), moe()),
                   (delta(), moe(experts=8, top=2, groups=8, keep=3)),
                   (latent(heads=2, dim=16, vdim=56, scale=0.3, kv_from=0), None),
                   (delta(heads=3, kv_heads=3, dim=20, vdim=36, conv=3), moe(experts=6, top=1, groups=1, keep=1, ff=33)),
                   (latent(heads=5, dim=20, rot=8, vdim=12, rank=40, base=700.0), moe())], **kw)


def weights(cfg, seed=0, sharp=1.0):
    """name -> float32 (bf16-representable).  sharp scales the queries of the latent-attention layers."""
    rng = np.random.default_rng(seed)
    w, W = {}, cfg["width"]

    def n(name, *shape, sd=1.0, mean=0.0):
        w[name] = lib.round_to_bf16((rng.standard_normal(shape) * sd + mean).astype(np.float32)).reshape(shape)

    def norm(name):
        n(name, W, sd=0.3, mean=1.2)
        n(name + ".b", W, sd=0.1)
        w[name + ".alpha"] = lib.round_to_bf16(np.float32(rng.uniform(0.4, 0.8))).reshape(())
    n("embed", cfg["vocab"], W, sd=0.5)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H = m["heads"]
        norm(p + "norm1")
        if layer["type"] == "latent_attention":
            d, r, dv, rank = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            n(p + "mix.q", H * (d + r), W, sd=sharp * W ** -0.5)
            if "kv_from" not in m:
                n(p + "mix.dkv", rank + r, W, sd=W ** -0.5)
                n(p + "mix.dkv.norm", rank, sd=0.2, mean=1.0)
            n(p + "mix.uk", H * d, rank, sd=rank ** -0.5)
            n(p + "mix.uv", H * dv, rank, sd=rank ** -0.5)
            n(p + "mix.sink", H, sd=1.0, mean=1.0)
            n(p + "mix.o", W, H * dv, sd=(H * dv) ** -0.5)
        else:
            d, dv, Hk, taps = m["dim"], m["vdim"], m["kv_heads"], m["conv"]
            for name, rows in (("q", Hk * d), ("k", Hk * d), ("v", H * dv)):
                n(p + "mix." + name, rows, W, sd=W ** -0.5)
                n(p + f"mix.{name}.conv", rows, taps, sd=0.6, mean=0.2)
            n(p + "mix.b", H, W, sd=W ** -0.5)
            n(p + "mix.A_log", H, sd=1.5, mean=-1.0)
            n(p + "mix.dt_bias", H * d, sd=1.0, mean=-2.0)
            n(p + "mix.norm", dv, sd=0.2, mean=1.0)
            n(p + "mix.a1", 12, W, sd=W ** -0.5)
            n(p + "mix.a2", H * d, 12, sd=0.3)
            n(p + "mix.g1", 10, W, sd=W ** -0.5)
            n(p + "mix.g2", H * dv, 10, sd=0.4)
            n(p + "mix.o", W, H * dv, sd=(H * dv) ** -0.5)
        if layer["mlp"] is not None:
            e, ff = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            n(p + "mlp.router", e, W, sd=2.0 * W ** -0.5)
            for x in range(e):
                n(f"{p}mlp.e{x}.gate", ff, W, sd=1.5 * W ** -0.5)
                n(f"{p}mlp.e{x}.up", ff, W, sd=1.5 * W ** -0.5)
                n(f"{p}mlp.e{x}.down", W, ff, sd=ff ** -0.5)
    norm("final.norm")
    return w


def engine(cfg, w, batch=1, max_s=256, dtype="float32"):
    entry = registry.lookup(cfg)
    return entry.engine(entry.config(cfg, dtype), w, batch, max_s)


def tokens(cfg, *shape, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], shape).astype(np.int32)


def run_cut(eng, ids, cuts):
    """Logits [B, S, V] of ids [B, S] run in portions of the given sizes (the last size repeats)."""
    eng.reset()
    B, S = ids.shape
    out, at, k = [], 0, 0
    while at < S:
        n = min(cuts[min(k, len(cuts) - 1)], S - at)
        out.append(eng.extend(ids[:, at:at + n], range(n)).dataAsync().reshape(B, n, -1))
        at, k = at + n, k + 1
    return np.concatenate(out, axis=1)


def reference(cfg, w, ids):
    return np.stack([ORACLES[cfg["architecture"]].forward(cfg, w, row) for row in ids])


def row_errors(got, ref):
    """Per position: rms difference over the vocabulary over the rms of all reference logits."""
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())
