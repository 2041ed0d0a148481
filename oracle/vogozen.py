"""Plain, slow CPU implementation of the Vogozen decoder design for the tests: one function per mechanism,
straight from its equations, in float64 by default.  It shares no code with `kandle_b200`.

Conventions as in oracle/hybrid.py: a model is a dict `cfg` (the parsed config.json) and a dict `w` of float
arrays by tensor name; every function takes whole sequences h [T, width] of one request, position 0 first.
"""
from __future__ import annotations

import numpy as np

from .hybrid import causal_conv_silu, delta_rule, rms_norm, sigmoid, softplus, unit


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


# ----------------------------------------------------------------------------- attention
def rotate_half(x, positions, base, dims):
    """Rotary positions on the first `dims` entries of the last axis, entry i paired with i + dims/2.  x [T, heads, d]."""
    n = dims // 2
    a = np.asarray(positions, np.float64)[:, None] * float(base) ** (-2.0 * np.arange(n, dtype=np.float64) / max(dims, 1))[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :n], x[..., n:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def normed_heads(h, w, p, name, heads, m, eps):
    """Queries or keys [T, heads, dim]: one RMS norm over all heads together, then the rotation."""
    x = rms_norm(h @ w[f"{p}mix.{name}"].T, w[f"{p}mix.{name}.norm"], eps).reshape(len(h), heads, m["dim"])
    return rotate_half(x, np.arange(len(h)), m["rot"]["base"], m["rot"]["dims"])


def keys_values(h, w, p, m, eps):
    """What an attention layer keeps: keys [T, kv_heads, dim] after norm and rotation, values [T, kv_heads, vdim]."""
    return normed_heads(h, w, p, "k", m["kv_heads"], m, eps), (h @ w[p + "mix.v"].T).reshape(len(h), m["kv_heads"], m["vdim"])


def quiet_softmax(scores):
    """exp(s) / (1 + sum exp(s)) along the last axis; -inf marks masked scores."""
    top = np.maximum(scores.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(scores - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(-top))


def window_attention(q, k, v, scale, size):
    """Query i of q [T, H, d] sees keys j with 0 <= i - j < size; G key heads serve H / G query heads each."""
    T, H, _ = q.shape
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    hidden = (j > i) | (i - j >= size)
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for head in range(H):
        g = head // (H // k.shape[1])
        s = q[:, head] @ k[:, g].T * scale
        s[hidden] = -np.inf
        out[:, head] = quiet_softmax(s) @ v[:, g]
    return out


def attention(h, w, p, m, eps, kept):
    """kept: keys and values of the layer that owns them (this one, or the one kv_from names)."""
    q = normed_heads(h, w, p, "q", m["heads"], m, eps)
    o = window_attention(q, *kept, m["scale"], m["mask"]["size"])
    return o.reshape(len(h), -1) @ w[p + "mix.o"].T


# ----------------------------------------------------------------------------- recurrences
def wkv(r, k, v, decay, u):
    """Token by token, S [H, d, d] from zero: o = (S + diag(u) k v^T)^T r, then S = diag(decay) S + k v^T."""
    T, H, d = r.shape
    S, o = np.zeros((H, d, v.shape[2]), r.dtype), np.empty(v.shape, r.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return o, S


def shifted(h):
    """The previous token's row, zeros for the first."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def wkv_inputs(h, w, p, m):
    T, H, d = len(h), m["heads"], m["dim"]
    before = shifted(h)
    mix = {n: h + (before - h) * w[f"{p}mix.mu.{n}"] for n in "rkvgw"}
    r, k, v = ((mix[n] @ w[f"{p}mix.{n}"].T).reshape(T, H, d) for n in "rkv")
    gate = silu(mix["g"] @ w[p + "mix.g"].T)
    logit = np.tanh(mix["w"] @ w[p + "mix.w1"].T) @ w[p + "mix.w2"].T + w[p + "mix.w0"]
    return r, k, v, gate, np.exp(-np.exp(logit)).reshape(T, H, d)


def wkv_mixer(h, w, p, m, eps):
    r, k, v, gate, decay = wkv_inputs(h, w, p, m)
    o, _ = wkv(r, k, v, decay, w[p + "mix.u"])
    return (rms_norm(o, 1.0, eps).reshape(len(h), -1) * w[p + "mix.norm"] * gate) @ w[p + "mix.o"].T


def delta_inputs(h, w, p, m):
    T, H, Hk, d, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv_silu(h @ w[p + "mix." + n].T, w[p + "mix." + n + ".conv"]) for n in "qkv")
    q = np.repeat(unit(q.reshape(T, Hk, d)) * d ** -0.5, H // Hk, axis=1)
    k = np.repeat(unit(k.reshape(T, Hk, d)), H // Hk, axis=1)
    beta = sigmoid(h @ w[p + "mix.b"].T)
    g = np.exp(-np.exp(w[p + "mix.A_log"]) * softplus(h @ w[p + "mix.a"].T + w[p + "mix.dt_bias"]))
    return q, k, v.reshape(T, H, dv), np.repeat(g[:, :, None], d, axis=2), beta


def delta_mixer(h, w, p, m, eps):
    T, H, dv = len(h), m["heads"], m["vdim"]
    o, _ = delta_rule(*delta_inputs(h, w, p, m))
    gate = silu(h @ w[p + "mix.g"].T).reshape(T, H, dv)
    return (rms_norm(o, w[p + "mix.norm"], eps) * gate).reshape(T, H * dv) @ w[p + "mix.o"].T


# ----------------------------------------------------------------------------- the rest
def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "mlp.gate"].T) * (h @ w[p + "mlp.up"].T)) @ w[p + "mlp.down"].T


def forward(cfg, w, ids, dtype=np.float64, layers=None):
    """Logits [T, vocab] of one request; `layers` (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(ids)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = keys_values(x, w, p, m, eps)
            y = attention(x, w, p, m, eps, kept[i if src is None else src])
        else:
            y = {"wkv": wkv_mixer, "delta": delta_mixer}[layer["type"]](x, w, p, m, eps)
        x = x + rms_norm(y, 1.0 + w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(dense(x, w, p), 1.0 + w[p + "norm2"], eps)
        if layers is not None:
            layers.append(x.copy())
    return rms_norm(x, 1.0 + w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, ids, steps, dtype=np.float64):
    ids = list(ids)
    for _ in range(steps):
        ids.append(int(forward(cfg, w, ids, dtype)[-1].argmax()))
    return ids[-steps:]
