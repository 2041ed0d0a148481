"""Small random models of the Vogozen design for the tests; engine, tokens and comparisons as in hybrid_cases.py."""
from __future__ import annotations

import numpy as np

from kandle_b200 import lib


def attention(heads=4, kv_heads=2, dim=20, vdim=28, rot=12, base=3000.0, scale=0.25, window=11, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def wkv(heads=3, dim=24):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}}


def delta(heads=4, kv_heads=2, dim=40, vdim=24, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def config(layers, vocab=150, width=72, eps=1e-5):
    return {"architecture": "Vogozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [dict(layer, mlp=mlp) for layer, mlp in layers]}


def mixed_config(**kw):
    """Every branch: own keys under a short window, both recurrences, a layer that reads the first one's rows through a
    longer window, layers without feed-forward, the last of them at the end."""
    return config([(attention(), dense()),
                   (wkv(), dense(40)),
                   (delta(), dense(33)),
                   (attention(window=40, scale=0.4, kv_from=0), None),
                   (wkv(heads=2, dim=40), dense()),
                   (attention(heads=3, kv_heads=3, dim=16, vdim=16, rot=16, base=500.0, window=25), dense()),
                   (delta(heads=3, kv_heads=1, dim=20, vdim=36, conv=3), None)], **kw)


def weights(cfg, seed=0, sharp=1.0):
    """name -> float32 (bf16-representable).  sharp scales the queries of the attention layers."""
    rng = np.random.default_rng(seed)
    w, W = {}, cfg["width"]

    def n(name, *shape, sd=1.0, mean=0.0):
        w[name] = lib.round_to_bf16((rng.standard_normal(shape) * sd + mean).astype(np.float32)).reshape(shape)

    n("embed", cfg["vocab"], W)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H = m["heads"]
        n(p + "norm1", W, sd=0.3)
        if layer["type"] == "attention":
            G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
            n(p + "mix.q", H * d, W, sd=W ** -0.5)
            n(p + "mix.q.norm", H * d, sd=0.3 * sharp, mean=sharp)
            if "kv_from" not in m:
                n(p + "mix.k", G * d, W, sd=W ** -0.5)
                n(p + "mix.k.norm", G * d, sd=0.3, mean=1.0)
                n(p + "mix.v", G * dv, W, sd=W ** -0.5)
            n(p + "mix.o", W, H * dv, sd=(H * dv) ** -0.5)
        elif layer["type"] == "wkv":
            N = H * m["dim"]
            for x in "rkvgw":
                w[f"{p}mix.mu.{x}"] = lib.round_to_bf16(rng.uniform(0, 1, W).astype(np.float32))
            for x in "rkvg":
                n(f"{p}mix.{x}", N, W, sd=W ** -0.5)
            n(p + "mix.w1", 13, W, sd=2 * W ** -0.5)
            n(p + "mix.w2", N, 13, sd=0.4)
            n(p + "mix.w0", N, sd=2.0, mean=-1.5)
            n(p + "mix.u", H, m["dim"], sd=0.7, mean=0.5)
            n(p + "mix.norm", N, sd=0.2, mean=1.0)
            n(p + "mix.o", W, N, sd=N ** -0.5)
        else:
            d, dv, Hk, taps = m["dim"], m["vdim"], m["kv_heads"], m["conv"]
            for name, rows in (("q", Hk * d), ("k", Hk * d), ("v", H * dv)):
                n(p + "mix." + name, rows, W, sd=W ** -0.5)
                n(p + f"mix.{name}.conv", rows, taps, sd=0.6, mean=0.2)
            n(p + "mix.b", H, W, sd=W ** -0.5)
            n(p + "mix.a", H, W, sd=W ** -0.5)
            n(p + "mix.A_log", H, sd=1.5, mean=-1.0)
            n(p + "mix.dt_bias", H, sd=1.0, mean=-2.0)
            n(p + "mix.g", H * dv, W, sd=W ** -0.5)
            n(p + "mix.norm", dv, sd=0.2, mean=1.0)
            n(p + "mix.o", W, H * dv, sd=(H * dv) ** -0.5)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            n(p + "norm2", W, sd=0.3)
            n(p + "mlp.gate", ff, W, sd=1.5 * W ** -0.5)
            n(p + "mlp.up", ff, W, sd=W ** -0.5)
            n(p + "mlp.down", W, ff, sd=ff ** -0.5)
    n("final.norm", W, sd=0.3)
    n("head", cfg["vocab"], W, sd=W ** -0.5)
    return w
