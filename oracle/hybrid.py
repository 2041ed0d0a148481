"""Plain, slow CPU implementation of the hybrid decoder designs (Pedorax) for the tests: one function per
mechanism, straight from its equations, in float64 by default.  It shares no code with `kandle_b200`.

A model is a dict `cfg` (the parsed config.json) and a dict `w` of float arrays by tensor name.  Every
function takes whole sequences: x [T, width] of one request, position 0 first; there is no cache, so what a
cached, cut or batched run of the product must reproduce is simply this function on the whole prefix.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def dynamic_tanh(x, alpha, weight, bias):
    """tanh(alpha x) weight + bias; no statistics of x."""
    return np.tanh(alpha * x) * weight + bias


def rotate_interleaved(x, positions, base, dims):
    """Rotary positions on the first `dims` entries of the last axis, pairs (2i, 2i+1)."""
    f = float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    a = np.asarray(positions, np.float64)[:, None] * f[None, :]
    a = a.reshape((len(positions),) + (1,) * (x.ndim - 2) + (dims // 2,))
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.copy()
    out[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return out


def latent_rows(h, w, p, m, eps):
    """What a latent-attention layer keeps per token: (normed latent [T, kv_rank], rotated shared key [T, rot_dim])."""
    r = m["kv_rank"]
    both = h @ w[p + "mix.dkv"].T
    c = rms_norm(both[:, :r], w[p + "mix.dkv.norm"], eps)
    return c, rotate_interleaved(both[:, r:], np.arange(len(h)), m["rot"]["base"], m["rot"]["dims"])


def sink_softmax(scores, sink):
    """Row softmax whose denominator also holds exp(sink); -inf marks masked scores."""
    mx = np.maximum(scores.max(axis=-1, keepdims=True), sink)
    e = np.exp(scores - mx)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - mx))


def latent_attention(h, w, p, m, eps, kept):
    """kept: (c, k_rot) of the layer that owns the latent (this one, or the one kv_from names)."""
    T, H, d, r, dv = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = kept
    q = (h @ w[p + "mix.q"].T).reshape(T, H, d + r)
    q_rot = rotate_interleaved(q[:, :, d:], np.arange(T), m["rot"]["base"], m["rot"]["dims"])
    k = (c @ w[p + "mix.uk"].T).reshape(T, H, d)
    v = (c @ w[p + "mix.uv"].T).reshape(T, H, dv)
    future = np.triu(np.ones((T, T), bool), 1)
    out = np.empty((T, H, dv), h.dtype)
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        s[future] = -np.inf
        out[:, i] = sink_softmax(s, w[p + "mix.sink"][i]) @ v[:, i]
    return out.reshape(T, H * dv) @ w[p + "mix.o"].T


def causal_conv_silu(x, taps):
    """Depthwise causal convolution over time (taps [channels, n], last column = current token), then silu."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1]), x.dtype), x])
    y = sum(padded[j:j + len(x)] * taps[:, j] for j in range(n))
    return y * sigmoid(y)


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """Gated delta rule with one decay per key channel, token by token.
    q, k, g [T, H, d]; v [T, H, dv]; beta [T, H].  Returns o [T, H, dv] and the final state [H, d, dv]."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), q.dtype) if state is None else state.copy()
    o = np.empty(v.shape, q.dtype)
    for t in range(T):
        S *= g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S += k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def delta_inputs(h, w, p, m):
    """Projections, short convolutions, unit norms, decays and step sizes of a channel_delta layer."""
    T, H, Hk, d, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv_silu(h @ w[p + "mix." + n].T, w[p + "mix." + n + ".conv"]) for n in "qkv")
    rep = H // Hk
    q = np.repeat(unit(q.reshape(T, Hk, d)) * d ** -0.5, rep, axis=1)
    k = np.repeat(unit(k.reshape(T, Hk, d)), rep, axis=1)
    beta = sigmoid(h @ w[p + "mix.b"].T)
    a = (h @ w[p + "mix.a1"].T) @ w[p + "mix.a2"].T + w[p + "mix.dt_bias"]
    g = np.exp(-np.exp(w[p + "mix.A_log"])[None, :, None] * softplus(a).reshape(T, H, d))
    return q, k, v.reshape(T, H, dv), g, beta


def channel_delta(h, w, p, m, eps):
    T, H, dv = len(h), m["heads"], m["vdim"]
    o, _ = delta_rule(*delta_inputs(h, w, p, m))
    gate = sigmoid((h @ w[p + "mix.g1"].T) @ w[p + "mix.g2"].T).reshape(T, H, dv)
    return (rms_norm(o, w[p + "mix.norm"], eps) * gate).reshape(T, H * dv) @ w[p + "mix.o"].T


def clamped_glu_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, router, r):
    """Group-limited sigmoid routing: chosen experts [T, top] and their weights [T, top]."""
    s = sigmoid(h @ router.T)
    T, E = s.shape
    gc, keep = r["groups"]["count"], r["groups"]["keep"]
    grouped = s.reshape(T, gc, E // gc)
    group_score = np.sort(grouped, axis=-1)[:, :, -2:].sum(-1)
    best = np.argsort(-group_score, axis=-1, kind="stable")[:, :keep]
    allowed = np.zeros((T, gc), bool)
    np.put_along_axis(allowed, best, True, axis=1)
    masked = np.where(np.repeat(allowed, E // gc, axis=1), s, -np.inf)
    chosen = np.argsort(-masked, axis=-1, kind="stable")[:, :r["top"]]
    ws = np.take_along_axis(s, chosen, axis=1)
    return chosen, ws / (ws.sum(-1, keepdims=True) + 1e-20)


def mixture_of_experts(h, w, p, mlp):
    chosen, ws = route(h, w[p + "mlp.router"], mlp["router"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, slot = np.nonzero(chosen == e)
        if len(t):
            y = clamped_glu_expert(h[t], *(w[f"{p}mlp.e{e}.{n}"] for n in ("gate", "up", "down")), mlp["expert"]["limit"])
            out[t] += ws[t, slot][:, None] * y
    return out


def forward(cfg, w, ids, dtype=np.float64, layers=None):
    """Logits [T, vocab] of one request; `layers` (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])

    x = w["embed"][np.asarray(ids)] * dtype(cfg["embedding"]["scale"])
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm(x, p + "norm1")
        if layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = latent_rows(h, w, p, m, eps)
            y = latent_attention(h, w, p, m, eps, kept[i if src is None else src])
        else:
            y = channel_delta(h, w, p, m, eps)
        if layer["mlp"] is not None:
            y = y + mixture_of_experts(h, w, p, layer["mlp"])
        x = x + y
        if layers is not None:
            layers.append(x.copy())
    return norm(x, "final.norm") @ w["embed"].T * cfg["logit_scale"]


def greedy(cfg, w, ids, steps, dtype=np.float64):
    ids = list(ids)
    for _ in range(steps):
        ids.append(int(forward(cfg, w, ids, dtype)[-1].argmax()))
    return ids[-steps:]
