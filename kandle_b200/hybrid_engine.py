"""Engine for decoders that mix layer types, in bf16 or in fp32 throughout:

  Pedorax   latent attention and gated delta rule (a decay per key channel), each beside an expert feed-forward,
            behind one Dynamic Tanh norm
  Vogozen   sliding-window attention, WKV time mixing and gated delta rule (a decay per head), each followed by a
            dense feed-forward, RMS norms on the sublayers' outputs

One step function, `_run`, serves whole prompts, portions of prompts and decode steps: it takes S new
tokens of B sequences at the cache's position and leaves their rows and states in the cache.  A design is a
frame (what surrounds the sublayers: embedding, norms, residual, feed-forward, head) and a list of mixers:

  frames   _ParallelFrame      h = norm(x);  x += mixer(h) + experts(h): residual and the NEXT layer's norm in one kernel
           _SequentialFrame    x += norm(mixer(x));  x += norm(ff(x)): each residual and norm in one kernel
  mixers   one GEMM for everything that reads the sublayer's input (small fp32 outputs such as router or decay logits
           ride along as its tail), then
           latent attention    norm + rotation + cache row -> attention over the cache rows (W_uk absorbed into the
                               queries, W_uv applied to the combined latents), or, for long bf16 prompts, keys and
                               values expanded once and the tcgen05 prefill kernel -> W_o
           window attention    norm + rotation + cache rows -> tcgen05 prefill or split-KV decode kernel -> W_o
           gated delta rule    convolution + unit norms + decays + recurrence in one kernel -> output norm and gate -> W_o
           WKV                 token shift -> r, k, v, gate as one grouped GEMM, decay logits -> recurrence -> output norm
                               and gate -> W_o
  experts  route -> rows in expert order -> gate/up with the clamped GLU in the epilogue -> down

A decode step is captured once as a CUDA graph with the position in device memory (DecoderEngine).

Numerics in bf16 mode: weights, GEMM and attention operands bf16 with fp32 accumulation; residual stream,
norms, angles, scores, softmax, router, decays, step sizes, recurrent state and logits fp32.
"""
from __future__ import annotations

import ctypes
import math

import numpy as np

from . import core, lib
from .cache import SequenceCache
from .core import Tensor
from .engine import DecoderEngine, RandomInit, _r, interleave_gate_up
from .model_utils.pedorax import ChannelDeltaSpec, ExpertsSpec, LatentAttentionSpec, PedoraxConfig
from .model_utils.vogozen import DenseSpec, HeadDeltaSpec, VogozenConfig, WindowAttentionSpec, WkvSpec

KD_EPI_NONE, KD_EPI_CLAMPED_GLU, KD_EPI_GEGLU = 0, 4, 5
KD_GATE_SIGMOID, KD_GATE_SILU = 0, 1


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class _Buffers:
    """Named device buffers that grow on demand; views by shape are kept, so a repeated step allocates nothing."""

    def __init__(self):
        self._flat, self._views = {}, {}

    def __call__(self, name: str, shape, dtype: str) -> Tensor:
        key = (name, tuple(shape), dtype)
        if key not in self._views:
            n = math.prod(shape)
            flat = self._flat.get(name)
            if flat is None or flat.dtype != dtype or flat.numel < n:
                self._views = {k: v for k, v in self._views.items() if k[0] != name}
                flat = self._flat[name] = core.empty((max(n, 1),), dtype)
            if len(self._views) > 4096:
                self._views = {}
            st, strides = 1, []
            for s in reversed(shape):
                strides.append(st)
                st *= s
            self._views[key] = flat._view(tuple(shape), tuple(reversed(strides)), 0)
        return self._views[key]


def _cols(t: Tensor, a: int, b: int) -> Tensor:
    return t.slice([slice(None)] * (t.ndim - 1) + [slice(a, b)])


def _rows(t: Tensor, a: int, b: int) -> Tensor:
    return t.slice([slice(a, b)] + [slice(None)] * (t.ndim - 1))


class _Weights:
    """Turns named matrices (or random numbers) into device tensors of the engine's layout."""

    def __init__(self, source, dtype: str):
        self.src, self.dtype, self.random = source, dtype, isinstance(source, RandomInit)
        self._offset = 0
        self._rng = np.random.Generator(np.random.PCG64(source.seed)) if self.random else None

    def _draw(self, shape, std=None) -> Tensor:
        t = core.empty(shape, self.dtype)
        lib.call("kd_randn", _r(t), ctypes.c_uint64(self.src.seed), ctypes.c_uint32(self._offset & 0xFFFFFFFF), ctypes.c_float(0.0),
                 ctypes.c_float(self.src.std if std is None else std), 0, 0, 0)
        self._offset += (math.prod(shape) + 1) // 2
        return t

    def matrix(self, name: str, shape) -> Tensor:
        return self._draw(shape) if self.random else self._put(self._get(name, shape))

    def _get(self, name: str, shape) -> np.ndarray:
        a = np.asarray(self.src[name], np.float32)
        if shape == () and a.size == 1:      # a scalar may be stored as a vector of one
            a = a.reshape(())
        if tuple(a.shape) != tuple(shape):
            raise ValueError(f"{name} has shape {tuple(a.shape)}, the configuration says {tuple(shape)}")
        return a

    def _put(self, a: np.ndarray) -> Tensor:
        return Tensor(np.ascontiguousarray(a, np.float32), dtype=self.dtype)

    def vector(self, name: str, shape, random=None) -> np.ndarray:
        """Small fp32 parameters, on the host.  random: value (or function of the shape) when weights are drawn."""
        if self.random:
            return np.asarray(random(shape) if callable(random) else np.full(shape, random), np.float32)
        return self._get(name, shape)

    def stacked_rows(self, parts, cols: int) -> Tensor:
        """[rows, cols] from (name or None, rows, padded rows) parts; missing and padding rows are zero."""
        total = sum(p for _, _, p in parts)
        if self.random:
            return self._draw((total, cols))
        a = np.zeros((total, cols), np.float32)
        at = 0
        for name, rows, padded in parts:
            if name is not None:
                a[at:at + rows] = self._get(name, (rows, cols))
            at += padded
        return self._put(a)

    def rank_of(self, name: str, default: int) -> int:
        """Rows of a low-rank factor: a size that only the tensor itself states."""
        if self.random:
            return default
        return int(np.asarray(self.src[name]).shape[0])

    def host(self, name: str, shape) -> np.ndarray:
        return self._get(name, shape)

    def padded(self, name: str, rows: int, cols: int, to_rows: int, to_cols: int) -> Tensor:
        """A matrix with zero rows and columns behind its own."""
        if self.random:
            return self._draw((to_rows, to_cols))
        a = np.zeros((to_rows, to_cols), np.float32)
        a[:rows, :cols] = self._get(name, (rows, cols))
        return self._put(a)

    def vector_t(self, name: str, shape, random=None, plus: float = 0.0) -> Tensor:
        return Tensor(self.vector(name, shape, random) + np.float32(plus), dtype="float32")


class _Norm:
    def __init__(self, w: _Weights, name: str, width: int):
        self.alpha = float(w.vector(name + ".alpha", (), 0.5))
        self.w = Tensor(w.vector(name, (width,), 1.0), dtype="float32")
        self.b = Tensor(w.vector(name + ".b", (width,), 0.0), dtype="float32")

    def args(self):
        return ctypes.c_float(self.alpha), _r(self.w), _r(self.b)


class _Projection:
    """The GEMM over a sublayer's input: columns in the engine's type, `tail` rows in fp32 behind them.
    parts, tail: (tensor name behind the layer's prefix, rows, padded to a multiple of)."""

    def __init__(self, w: _Weights, parts, width: int, prefix: str, tail=()):
        self.cols, at = {}, 0
        for key, rows, pad in parts:
            self.cols[key] = at
            at += _up(rows, pad)
        self.n = _up(at, 32)
        rows = [(prefix + "mix." + key, r, _up(r, pad)) for key, r, pad in parts]
        rows.append((None, 0, self.n - at))
        rows += [(prefix + key, r, _up(r, pad)) for key, r, pad in tail]
        self.tail = sum(_up(r, pad) for _, r, pad in tail)
        self.weight = w.stacked_rows(rows, width)

    def __call__(self, eng: "HybridEngine", ws: _Buffers, h: Tensor, B: int, S: int):
        """[B, S, n] in the engine's type and the tail [B*S, tail] in fp32 (or None)."""
        T = B * S
        out = ws("proj", (B, S, self.n), eng.dtype)
        tail = ws("tail", (T, self.tail), "float32") if self.tail else None
        eng.linear(h, self.weight, out.view(T, self.n), tail=tail)
        return out, tail


def _first(t: Tensor, B: int) -> Tensor:
    """The first B sequences of something kept per sequence."""
    return t if t.shape[0] == B else t.slice([slice(0, B)] + [slice(None)] * (t.ndim - 1))


class _LatentAttention:
    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m: LatentAttentionSpec, tail=()):
        self.m, self.i, p = m, i, f"l{i}."
        self.own = m.kvFrom is None
        parts = [("q", m.heads * (m.dim + m.rotDim), 8)]
        if self.own:
            parts.append(("dkv", m.kvRank + m.rotDim, 8))
        self.proj = _Projection(w, parts, eng.W, p, tail)
        self.norm = Tensor(w.vector(p + "mix.dkv.norm", (m.kvRank,), 1.0), dtype="float32") if self.own else None
        self.sink = Tensor(w.vector(p + "mix.sink", (m.heads,), 0.0), dtype="float32")
        self.wo = w.matrix(p + "mix.o", (eng.W, m.heads * m.vdim))
        self.wukv = None          # [W_uk; W_uv] as stored, for prompts whose keys and values are expanded
        expandable = eng.dtype == "bfloat16" and m.dim in (64, 128) and m.vdim == m.dim and m.rotDim == 64 and m.kvRank % 8 == 0
        if w.random:
            self.wuk, self.wuk_t = w.matrix("", (m.heads, m.dim, m.kvRank)), w.matrix("", (m.heads, m.kvRank, m.dim))
            self.wuv_t, self.wuv = w.matrix("", (m.heads, m.kvRank, m.vdim)), w.matrix("", (m.heads, m.vdim, m.kvRank))
            if expandable:
                self.wukv = w.matrix("", (m.heads * (m.dim + m.vdim), m.kvRank))
        else:
            uk, uv = w.host(p + "mix.uk", (m.heads * m.dim, m.kvRank)), w.host(p + "mix.uv", (m.heads * m.vdim, m.kvRank))
            self.wuk = w._put(uk.reshape(m.heads, m.dim, m.kvRank))
            self.wuv_t = w._put(uv.reshape(m.heads, m.vdim, m.kvRank).transpose(0, 2, 1))
            self.wuk_t = self.wuv = None      # the layouts of the tensor-core forms
            if eng.dtype == "bfloat16":
                self.wuk_t = w._put(uk.reshape(m.heads, m.dim, m.kvRank).transpose(0, 2, 1))
                self.wuv = w._put(uv.reshape(m.heads, m.vdim, m.kvRank))
            if expandable:
                self.wukv = w._put(np.concatenate([uk, uv], axis=0))
        self.cos, self.sin = eng.rotation(m.rotBase, m.rotDim)

    def __call__(self, eng: "HybridEngine", ws: _Buffers, h: Tensor, B: int, S: int, pos) -> Tensor:
        m, T, dt = self.m, B * S, eng.dtype
        pos_dev, pos_host = pos
        proj3, _ = self.proj(eng, ws, h, B, S)
        cache = _first(eng.cache.of(self.i).rows, B)
        expand = self.wukv is not None and pos_dev is None and S >= eng.expand_from
        # (the layers that read another layer's rows expand the same dense copy)
        owner = self if self.own else eng.mixers[m.kvFrom]
        dense = ws(f"latent{owner.i}", (T, m.kvRank), dt) if expand and owner.wukv is not None and B > 1 and pos_host == 0 else None
        lib.call("kd_latent_prep", _r(proj3), self.proj.cols["q"], m.heads, m.dim, m.rotDim, self.proj.cols.get("dkv", -1), m.kvRank,
                 _r(self.norm), ctypes.c_float(eng.cfg.normEps), _r(self.cos), _r(self.sin), _r(cache), _r(pos_dev), pos_host, _r(dense) if self.own else None)
        out = ws("mixed", (T, m.heads * m.vdim), dt)
        if expand:
            self._expanded(eng, ws, proj3, cache, dense, B, S, pos_host, out)
            return out
        width = cache.shape[2]
        splits = ctypes.c_int(0)
        lib.call("kd_latent_attention_splits", B, S, m.heads, eng.max_seq_len if pos_dev is not None else pos_host + S, ctypes.byref(splits))
        ns = splits.value
        q_abs = ws("q_abs", (B, S, m.heads, width), dt)
        part_o = ws("part_o", (T * m.heads, ns, m.kvRank), "float32")
        part_ml = ws("part_ml", (T * m.heads, ns, 2), "float32")
        lib.call("kd_latent_absorb", _r(proj3), self.proj.cols["q"], m.rotDim, _r(self.wuk), _r(self.wuk_t), _r(q_abs))
        lib.call("kd_latent_attention", _r(q_abs), _r(cache), m.kvRank, ctypes.c_float(m.scale), _r(pos_dev), pos_host, _r(part_o), _r(part_ml))
        latents = ws("latents", (T * m.heads, m.kvRank), dt) if self.wuv is not None else None
        lib.call("kd_latent_values", _r(part_o), _r(part_ml), _r(self.sink), _r(self.wuv_t), _r(self.wuv), _r(latents), _r(out))
        return out


    def _expanded(self, eng: "HybridEngine", ws: _Buffers, proj3: Tensor, cache: Tensor, dense, B: int, S: int, pos: int, out: Tensor) -> None:
        """Keys and values of the whole context from its latents, then the tcgen05 prefill kernel."""
        m, ctx = self.m, pos + S
        n = m.heads * (m.dim + m.vdim)
        kv = ws("kv", (B, ctx, n), eng.dtype)
        if dense is not None:
            eng.linear(dense, self.wukv, kv.view(B * ctx, n))
        else:
            for b in range(B):
                eng.linear(cache.slice([b, slice(0, ctx), slice(0, m.kvRank)]), self.wukv, kv.slice([b, slice(None), slice(None)]))
        lib.call("kd_latent_prefill", _r(proj3), self.proj.cols["q"], m.heads, m.dim, m.rotDim, _r(kv), m.vdim, _r(cache), m.kvRank,
                 _r(self.sink), ctypes.c_float(m.scale), pos, _r(out))


class _DeltaRule:
    """Gated delta rule: the parts that its forms share.  A form provides the projections, the decay logits and the gate."""

    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m, decays: int, gate_act: int):
        self.m, self.i, self.gate_act, p = m, i, gate_act, f"l{i}."
        qk, vv = m.kvHeads * m.dim, m.heads * m.vdim
        # q, k, v side by side without padding: their channels are the convolution's
        self.parts = [("q", qk, 1), ("k", qk, 1), ("v", vv, 8)]
        self.conv = tuple(w.vector_t(p + f"mix.{n}.conv", (rows, m.taps), lambda s: w._rng.standard_normal(s) * 0.5) for n, rows in (("q", qk), ("k", qk), ("v", vv)))
        self.neg_rate = Tensor(-np.exp(w.vector(p + "mix.A_log", (m.heads,), -1.0)), dtype="float32")
        self.dt_bias = w.vector_t(p + "mix.dt_bias", (decays,), -3.0)
        self.norm = w.vector_t(p + "mix.norm", (m.vdim,), 1.0)
        self.wo = w.matrix(p + "mix.o", (eng.W, vv))

    def __call__(self, eng: "HybridEngine", ws: _Buffers, h: Tensor, B: int, S: int, pos) -> Tensor:
        m, T, c = self.m, B * S, self.proj.cols
        kept = eng.cache.of(self.i)
        state, history = _first(kept.state, B), _first(kept.history, B)
        proj3, tail = self.proj(eng, ws, h, B, S)
        decay, gate = self.decay_and_gate(eng, ws, proj3.view(T, self.proj.n), tail)
        o, out = ws("delta_o", (T, m.heads * m.vdim), "float32"), ws("mixed", (T, m.heads * m.vdim), eng.dtype)
        lib.call("kd_delta_rule", _r(proj3), c["q"], c["k"], c["v"], c["b"], _r(decay), m.heads, m.kvHeads, m.dim, m.vdim,
                 *(_r(t) for t in self.conv), _r(self.neg_rate), _r(self.dt_bias), _r(history), _r(state), _r(o))
        lib.call("kd_delta_out", _r(o), _r(gate), _r(self.norm), ctypes.c_float(eng.cfg.normEps), self.gate_act, _r(proj3), c["q"], m.taps, _r(history), _r(out))
        return out


class _ChannelDelta(_DeltaRule):
    """A decay per key channel; decay and gate through low-rank factors."""

    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m: ChannelDeltaSpec, tail=()):
        super().__init__(eng, w, i, m, m.heads * m.dim, KD_GATE_SIGMOID)
        p, vv = f"l{i}.", m.heads * m.vdim
        ra, rg = w.rank_of(p + "mix.a1", m.dim), w.rank_of(p + "mix.g1", m.vdim)
        self.ra, self.rg = _up(ra, 8), _up(rg, 8)
        self.proj = _Projection(w, self.parts + [("a1", ra, 8), ("g1", rg, 8), ("b", m.heads, 8)], eng.W, p, tail)
        self.wa2 = w.padded(p + "mix.a2", m.heads * m.dim, ra, m.heads * m.dim, self.ra)
        self.wg2 = w.padded(p + "mix.g2", vv, rg, vv, self.rg)

    def decay_and_gate(self, eng, ws, proj2: Tensor, tail):
        m, T, c = self.m, proj2.shape[0], self.proj.cols
        decay, gate = ws("decay", (T, m.heads * m.dim), "float32"), ws("gate", (T, m.heads * m.vdim), eng.dtype)
        eng.linear(_cols(proj2, c["a1"], c["a1"] + self.ra), self.wa2, decay)
        eng.linear(_cols(proj2, c["g1"], c["g1"] + self.rg), self.wg2, gate)
        return decay, gate


class _HeadDelta(_DeltaRule):
    """One decay per head, whose logits leave the first GEMM in fp32; a full-rank gate through silu."""

    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m: HeadDeltaSpec, tail=()):
        super().__init__(eng, w, i, m, m.heads, KD_GATE_SILU)
        self.proj = _Projection(w, self.parts + [("g", m.heads * m.vdim, 8), ("b", m.heads, 8)], eng.W, f"l{i}.", [("mix.a", m.heads, 8), *tail])

    def decay_and_gate(self, eng, ws, proj2: Tensor, tail):
        g, vv = self.proj.cols["g"], self.m.heads * self.m.vdim
        return _cols(tail, 0, self.m.heads), _cols(proj2, g, g + vv)


class _WindowAttention:
    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m: WindowAttentionSpec, tail=()):
        self.m, self.i, p = m, i, f"l{i}."
        self.own = m.kvFrom is None
        qd, vd = ctypes.c_int(0), ctypes.c_int(0)
        lib.call("kd_attention_head_sizes", lib.DTYPES[eng.dtype][0], m.dim, m.vdim, ctypes.byref(qd), ctypes.byref(vd))
        self.q_size, self.v_size = qd.value, vd.value
        parts = [("q", m.heads * m.dim, 8)]
        if self.own:
            parts += [("k", m.kvHeads * m.dim, 8), ("v", m.kvHeads * m.vdim, 8)]
        self.proj = _Projection(w, parts, eng.W, p, tail)
        self.q_norm = w.vector_t(p + "mix.q.norm", (m.heads * m.dim,), 1.0)
        self.k_norm = w.vector_t(p + "mix.k.norm", (m.kvHeads * m.dim,), 1.0) if self.own else None
        self.sink = core.zeros((m.heads,), "float32")     # the one in the softmax denominator: a score of 0
        self.cos, self.sin = eng.rotation(m.rotBase, m.rotDims)
        if w.random or self.v_size == m.vdim:
            self.wo = w.matrix(p + "mix.o", (eng.W, m.heads * self.v_size))
        else:                                             # the padding columns of a head's output meet zeros
            wo = np.zeros((eng.W, m.heads, self.v_size), np.float32)
            wo[:, :, :m.vdim] = w.host(p + "mix.o", (eng.W, m.heads * m.vdim)).reshape(eng.W, m.heads, m.vdim)
            self.wo = w._put(wo.reshape(eng.W, m.heads * self.v_size))

    def __call__(self, eng: "HybridEngine", ws: _Buffers, h: Tensor, B: int, S: int, pos) -> Tensor:
        m, c = self.m, self.proj.cols
        pos_dev, pos_host = pos
        proj3, _ = self.proj(eng, ws, h, B, S)
        kept = eng.cache.of(self.i)
        keys, values = _first(kept.keys, B), _first(kept.values, B)
        q = ws("q", (B, S, m.heads, self.q_size), eng.dtype)
        out = ws("mixed", (B * S, m.heads * self.v_size), eng.dtype)
        lib.call("kd_qk_norm_rope_cache", _r(proj3), c["q"], c.get("k", -1), c.get("v", -1), m.dim, m.vdim, m.rotDims, _r(self.q_norm), _r(self.k_norm),
                 ctypes.c_float(eng.cfg.normEps), _r(self.cos), _r(self.sin), _r(keys), _r(values), _r(pos_dev), pos_host, _r(q))
        lib.call("kd_window_attention", _r(q), _r(keys), _r(values), _r(self.sink), ctypes.c_float(m.scale), m.window, _r(pos_dev), pos_host, _r(out))
        return out


class _Wkv:
    MIXES = "rkvgw"          # order of the shifted inputs: the first four meet one matrix each in one grouped GEMM

    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m: WkvSpec, tail=()):
        if tail:
            raise ValueError("a WKV layer has no common projection for other rows to join")
        self.m, self.i, p = m, i, f"l{i}."
        n, W = m.heads * m.dim, eng.W
        self.mu = Tensor(np.stack([w.vector(f"{p}mix.mu.{x}", (W,), 0.5) for x in self.MIXES]), dtype="float32")
        if w.random:
            self.w4 = w.matrix("", (4, n, W))
        else:
            self.w4 = w._put(np.stack([w.host(f"{p}mix.{x}", (n, W)) for x in self.MIXES[:4]]))
        rank = w.rank_of(p + "mix.w1", 64)
        self.rank = _up(rank, 8)
        self.w1 = w.padded(p + "mix.w1", rank, W, self.rank, W)
        self.w2 = w.padded(p + "mix.w2", n, rank, n, self.rank)
        self.w0 = w.vector_t(p + "mix.w0", (n,), -1.0)
        self.u = w.vector_t(p + "mix.u", (m.heads, m.dim), 0.5).view(n)
        self.norm = w.vector_t(p + "mix.norm", (n,), 1.0)
        self.wo = w.matrix(p + "mix.o", (W, n))

    def __call__(self, eng: "HybridEngine", ws: _Buffers, h: Tensor, B: int, S: int, pos) -> Tensor:
        m, T, dt, W = self.m, B * S, eng.dtype, eng.W
        n = m.heads * m.dim
        kept = eng.cache.of(self.i)
        state, last = _first(kept.state, B), _first(kept.last, B)
        mixes, rkvg = ws("mixes", (5 * T, W), dt), ws("rkvg", (4 * T, n), dt)
        lib.call("kd_token_shift", _r(h.view(B, S, W)), _r(self.mu), _r(last), _r(mixes))
        lib.call("kd_moe_linear", _r(_rows(mixes, 0, 4 * T)), _r(self.w4), None, KD_EPI_NONE, ctypes.c_float(0.0), _r(rkvg))
        low, logits = ws("wkv_low", (T, self.rank), dt), ws("decay", (T, n), "float32")
        lib.call("kd_linear_tanh", _r(_rows(mixes, 4 * T, 5 * T)), _r(self.w1), _r(low))
        eng.linear(low, self.w2, logits)
        r, k, v = (_rows(rkvg, x * T, (x + 1) * T).view(B, S, n) for x in range(3))
        o, out = ws("delta_o", (T, n), "float32"), ws("mixed", (T, n), dt)
        lib.call("kd_wkv", _r(r), _r(k), _r(v), _r(logits), _r(self.w0), _r(self.u), _r(state), _r(o))
        lib.call("kd_gated_head_norm", _r(o), _r(_rows(rkvg, 3 * T, 4 * T)), _r(self.norm), m.heads, ctypes.c_float(eng.cfg.normEps), KD_GATE_SILU, _r(out))
        return out


_MIXERS = {LatentAttentionSpec: _LatentAttention, ChannelDeltaSpec: _ChannelDelta, HeadDeltaSpec: _HeadDelta, WindowAttentionSpec: _WindowAttention, WkvSpec: _Wkv}


class _Experts:
    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, e: ExpertsSpec):
        self.e, p = e, f"l{i}.mlp."
        self.ff = _up(e.ff, 16)        # gate and up rows interleave in blocks of 16; padding rows and columns are zero
        if w.random:
            self.wgu = w.matrix("", (e.experts, 2 * self.ff, eng.W))
            self.wdown = w.matrix("", (e.experts, eng.W, self.ff))
            return
        gu = np.zeros((e.experts, 2 * self.ff, eng.W), np.float32)
        down = np.zeros((e.experts, eng.W, self.ff), np.float32)
        grow = lambda a: np.concatenate([a, np.zeros((self.ff - e.ff, eng.W), np.float32)]) if self.ff > e.ff else a  # noqa: E731
        for x in range(e.experts):
            gu[x] = interleave_gate_up(grow(w.host(f"{p}e{x}.gate", (e.ff, eng.W))), grow(w.host(f"{p}e{x}.up", (e.ff, eng.W))))
            down[x, :, :e.ff] = w.host(f"{p}e{x}.down", (eng.W, e.ff))
        self.wgu, self.wdown = w._put(gu), w._put(down)

    def __call__(self, eng: "HybridEngine", ws: _Buffers, h: Tensor, logits: Tensor, counts: Tensor):
        """Expert rows [T*top, W], their slots and weights [T, top]."""
        e, T, dt = self.e, h.shape[0], eng.dtype
        R = T * e.top
        ids, ranks, slots = (ws(n, (T, e.top), "int32") for n in ("moe_ids", "moe_ranks", "moe_slots"))
        weights, offsets = ws("moe_w", (T, e.top), "float32"), ws("moe_off", (e.experts + 1,), "int32")
        xs, act, y = ws("moe_x", (R, eng.W), dt), ws("moe_act", (R, self.ff), dt), ws("moe_y", (R, eng.W), dt)
        lib.call("kd_moe_route", _r(_cols(logits, 0, e.experts)), e.top, e.groups, e.keep, _r(ids), _r(weights), _r(ranks), _r(counts))
        lib.call("kd_moe_gather", _r(h), _r(ids), _r(ranks), _r(counts), e.experts, _r(slots), _r(offsets), _r(xs))
        lib.call("kd_moe_linear", _r(xs), _r(self.wgu), _r(offsets), KD_EPI_CLAMPED_GLU, ctypes.c_float(e.limit), _r(act))
        lib.call("kd_moe_linear", _r(act), _r(self.wdown), _r(offsets), KD_EPI_NONE, ctypes.c_float(0.0), _r(y))
        return y, slots, weights


class _GatedDense:
    """Dense feed-forward, GELU(gate) * up in the GEMM's epilogue."""

    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, d: DenseSpec):
        p, self.ff = f"l{i}.mlp.", _up(d.ff, 16)      # gate and up rows interleave in blocks of 16; padding is zero
        if w.random:
            self.wgu = w.matrix("", (2 * self.ff, eng.W))
        else:
            grown = lambda n: np.concatenate([w.host(p + n, (d.ff, eng.W)), np.zeros((self.ff - d.ff, eng.W), np.float32)])  # noqa: E731
            self.wgu = w._put(interleave_gate_up(grown("gate"), grown("up")))
        self.wdown = w.padded(p + "down", eng.W, d.ff, eng.W, self.ff)

    def __call__(self, eng: "HybridEngine", ws: _Buffers, h: Tensor) -> Tensor:
        act = ws("act", (h.shape[0], self.ff), eng.dtype)
        lib.call("kd_linear_glu", _r(h), _r(self.wgu), KD_EPI_GEGLU, _r(act))
        return act


class _ParallelFrame:
    """Pedorax: one Dynamic Tanh norm per layer feeds the mixer and, beside it, the experts."""

    def __init__(self, eng: "HybridEngine", w: _Weights, cfg: PedoraxConfig):
        self.embed = w.matrix("embed", (eng.V, eng.W))
        self.norms, self.mixers, self.experts = [], [], []
        for i, layer in enumerate(cfg.layers):
            self.norms.append(_Norm(w, f"l{i}.norm1", eng.W))
            tail = [("mlp.router", layer.experts.experts, 8)] if layer.experts is not None else []
            self.mixers.append(_MIXERS[type(layer.mixer)](eng, w, i, layer.mixer, tail))
            self.experts.append(_Experts(eng, w, i, layer.experts) if layer.experts is not None else None)
        self.norms.append(_Norm(w, "final.norm", eng.W))
        self.max_experts = max([e.e.experts for e in self.experts if e is not None], default=1)
        self.head, self.embed_scale, self.logit_scale = self.embed, cfg.embeddingScale, cfg.logitScale

    def run(self, eng: "HybridEngine", ws: _Buffers, ids: Tensor, B: int, S: int, pos) -> Tensor:
        T, dt = B * S, eng.dtype
        x, h = ws("x", (T, eng.W), "float32"), ws("h", (T, eng.W), dt)
        counts = ws("moe_counts", (len(self.experts), self.max_experts), "int32")
        lib.call("kd_fill", _r(counts), ctypes.c_double(0.0))
        lib.call("kd_embed_dynamic_tanh", _r(self.embed), _r(ids), ctypes.c_float(self.embed_scale), *self.norms[0].args(), _r(x), _r(h))
        for i, (mixer, experts) in enumerate(zip(self.mixers, self.experts)):
            mixed = mixer(eng, ws, h, B, S, pos)
            mix = self._out_projection(eng, ws, mixed, mixer.wo, x, T)
            y = slots = weights = None
            if experts is not None:
                y, slots, weights = experts(eng, ws, h, ws("tail", (T, mixer.proj.tail), "float32"),
                                            counts.slice([slice(i, i + 1), slice(0, experts.e.experts)]))
            lib.call("kd_residual_dynamic_tanh", _r(x), _r(mix), _r(y), _r(slots), _r(weights), *self.norms[i + 1].args(), _r(x), _r(h))
            eng.traced(x)
        return h

    @staticmethod
    def _out_projection(eng: "HybridEngine", ws: _Buffers, mixed: Tensor, wo: Tensor, x: Tensor, T: int):
        """x += mixed W_o^T in the GEMM's epilogue for many rows (returns None); for a few rows fp32 partial sums that
        the residual kernel adds."""
        if eng.dtype == "bfloat16" and T > 64 and mixed.shape[1] % 8 == 0 and eng.W % 8 == 0:
            eng.linear(mixed, wo, x, residual=x)
            return None
        return eng.partial_sums(ws, mixed, wo, "float32")


class _SequentialFrame:
    """Vogozen: mixer, then feed-forward; each reads the residual itself and is normed before it is added."""

    def __init__(self, eng: "HybridEngine", w: _Weights, cfg: VogozenConfig):
        self.embed = w.matrix("embed", (eng.V, eng.W))
        self.mixers, self.dense, self.norms = [], [], []
        for i, layer in enumerate(cfg.layers):
            self.mixers.append(_MIXERS[type(layer.mixer)](eng, w, i, layer.mixer))
            self.dense.append(_GatedDense(eng, w, i, layer.dense) if layer.dense is not None else None)
            # norm weights are stored around zero
            norm = lambda n: w.vector_t(f"l{i}.{n}", (eng.W,), 0.0, plus=1.0)  # noqa: E731
            self.norms.append((norm("norm1"), norm("norm2") if layer.dense is not None else None))
        self.final = w.vector_t("final.norm", (eng.W,), 0.0, plus=1.0)
        self.head, self.logit_scale = w.matrix("head", (eng.V, eng.W)), 1.0

    def run(self, eng: "HybridEngine", ws: _Buffers, ids: Tensor, B: int, S: int, pos) -> Tensor:
        T, eps, n = B * S, ctypes.c_float(eng.cfg.normEps), len(self.mixers)
        x, h = ws("x", (T, eng.W), "float32"), ws("h", (T, eng.W), eng.dtype)
        lib.call("kd_embed_rows", _r(self.embed), _r(ids), _r(x), _r(h))
        for i, (mixer, dense, (norm1, norm2)) in enumerate(zip(self.mixers, self.dense, self.norms)):
            last = i + 1 == n
            y = eng.partial_sums(ws, mixer(eng, ws, h, B, S, pos), mixer.wo, eng.dtype)
            lib.call("kd_residual_post_norm", _r(x), _r(y), _r(norm1), eps, _r(self.final) if last and dense is None else None, _r(x), _r(h))
            if dense is not None:
                y = eng.partial_sums(ws, dense(eng, ws, h), dense.wdown, eng.dtype)
                lib.call("kd_residual_post_norm", _r(x), _r(y), _r(norm2), eps, _r(self.final) if last else None, _r(x), _r(h))
            eng.traced(x)
        return h


_FRAMES = {PedoraxConfig: _ParallelFrame, VogozenConfig: _SequentialFrame}


class HybridEngine(DecoderEngine):
    def __init__(self, cfg: PedoraxConfig | VogozenConfig, weights, max_batch: int, max_seq_len: int):
        """weights: a mapping of the checkpoint's tensor names to float32 arrays (io.SafetensorStateDict, a
        dict), or a RandomInit.  cfg.dtype is "bfloat16" or "float32"."""
        cfg.validate()
        if cfg.dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {cfg.dtype!r}: the hybrid engine runs in bfloat16 or float32")
        self._init_decoding(max_batch, max_seq_len)
        self.cfg, self.dtype, self.W, self.V = cfg, cfg.dtype, cfg.hiddenSize, cfg.vocabSize
        self._tables = {}
        self.frame = _FRAMES[type(cfg)](self, _Weights(weights, self.dtype), cfg)
        self.mixers = self.frame.mixers
        self.cache = SequenceCache(cfg.layers, max_batch, max_seq_len, self.dtype, self.W)
        self.expand_from = 64      # portions of at least this many tokens expand keys and values (latent attention)
        self._prompt = _Buffers()
        self.cur_B = 0
        self.trace = None          # a list: receives the residual stream [T, W] after every layer (tests)

    # ------------------------------------------------------------------ helpers
    def rotation(self, base: float, dims: int):
        """cos / sin [maxS, dims/2] of position x base^(-2i/dims), from angles in float64."""
        key = (base, dims)
        if key not in self._tables:
            f = base ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims) if dims else np.zeros(1)
            a = np.arange(self.max_seq_len, dtype=np.float64)[:, None] * f[None, :]
            self._tables[key] = Tensor(np.cos(a).astype(np.float32)), Tensor(np.sin(a).astype(np.float32))
        return self._tables[key]

    def linear(self, x: Tensor, w: Tensor, out: Tensor, residual: Tensor | None = None, alpha: float = 1.0, tail: Tensor | None = None) -> None:
        lib.call("kd_linear_ex", _r(x), _r(w), _r(residual), ctypes.c_float(alpha), _r(out), _r(tail))

    def partial_sums(self, ws: _Buffers, x: Tensor, w: Tensor, dtype: str) -> Tensor:
        """x w^T for a kernel that adds up split-K partial sums: fp32 [splits, T, W] for a few bf16 rows, else [1, T, W]
        in `dtype`."""
        T, k = x.shape
        if self.dtype == "bfloat16" and T <= 64 and k % 8 == 0:
            s = ctypes.c_int(0)
            lib.call("kd_linear_bf16_skinny_splits", ctypes.c_int64(self.W), ctypes.c_int64(k), ctypes.byref(s))
            y = ws("mix", (s.value, T, self.W), "float32")
            lib.call("kd_linear_bf16_skinny", _r(x), _r(w), 0, _r(y))
            return y
        y = ws("mix" if dtype == "float32" else "mix16", (1, T, self.W), dtype)
        self.linear(x, w, y.view(T, self.W))
        return y

    def traced(self, x: Tensor) -> None:
        if self.trace is not None:
            self.trace.append(x.dataAsync().copy())

    # ------------------------------------------------------------------ one step over S tokens of B sequences
    def _run(self, ws: _Buffers, ids: Tensor, B: int, S: int, pos_dev: Tensor | None, pos_host: int) -> Tensor:
        """ids: device int32/int64 [B*S].  Runs them at the given position; returns the final norm's output [B*S, W]."""
        return self.frame.run(self, ws, ids, B, S, (pos_dev, pos_host))

    def _logits(self, ws: _Buffers, rows: Tensor, out: Tensor) -> None:
        """out [n, V] fp32 = logit_scale * rows [n, W] head^T (64 rows a call: the vocabulary matrix streams once each)."""
        n = rows.shape[0]
        for a in range(0, n, 64):
            b = min(n, a + 64)
            r, o = (t.slice([slice(a, b), slice(None)]) for t in (rows, out))
            self.linear(r, self.frame.head, o, alpha=self.frame.logit_scale)

    # ------------------------------------------------------------------ prompts and portions
    def reset(self) -> None:
        """Ends the current sequences; the next portion starts new ones at position 0."""
        self.cache.reset()
        self.pos = 0

    def extend(self, ids, want=None) -> Tensor:
        """Runs the next tokens ids [B, S] (host int array, or a device int32 Tensor) of the current sequences.  Returns fp32 logits
        [B * len(want), V] at the places `want` of the portion, sequence by sequence (default: the last)."""
        if not isinstance(ids, Tensor):
            ids = np.ascontiguousarray(ids, dtype=np.int32)
        B, S = ids.shape
        if B > self.B:
            raise ValueError(f"{B} sequences exceed the engine's {self.B}")
        if self.pos and B != self.cur_B:
            raise ValueError(f"{B} token rows for {self.cur_B} running sequences")
        self.cache.room(S)
        want = [S - 1] if want is None else [int(p) for p in want]
        if any(p < 0 or p >= S for p in want):
            raise ValueError(f"places {want} outside a portion of {S} tokens")
        self.cur_B = B
        if S == 1 and self.pos:
            logits = self._decode_given(ids.dataAsync() if isinstance(ids, Tensor) else ids)
            return logits if want == [0] else self._take(logits, [b for b in range(B) for _ in want])
        if isinstance(ids, Tensor):
            t = ids.view(B * S)
        else:
            t = self._prompt("ids", (B * S,), "int32")
            core._backend().upload(t._handle, ids.reshape(-1))
        h = self._run(self._prompt, t, B, S, None, self.pos)
        self.pos += S
        self.cache.pos = self.pos
        out = core.empty((B * len(want), self.V), "float32")
        if want:
            rows = self._take(h, [b * S + p for b in range(B) for p in want])
            self._logits(self._prompt, rows, out)
        return out

    def _take(self, t: Tensor, rows) -> Tensor:
        out = core.empty((len(rows), t.shape[1]), t.dtype)
        if rows:
            core._kernel("index_select")(t._handle, Tensor(np.asarray(rows, np.int32))._handle, {"dim": 0}, out._handle)
        return out

    def prefill(self, ids, all_logits: bool = False, portion: int | None = None):
        """New sequences with prompts ids [B, S] (host array or device int32 Tensor), in portions of `portion` tokens (default: whole).
        Returns the next token per sequence, device int64 [B] (and fp32 logits [B, S, V] with all_logits)."""
        if isinstance(ids, Tensor) and portion:
            ids = ids.dataAsync()
        if not isinstance(ids, Tensor):
            ids = np.ascontiguousarray(ids, dtype=np.int32)
        B, S = ids.shape
        self.reset()
        self.cache.room(S)
        parts, step = [], portion or S
        for a in range(0, S, step):
            n = min(step, S - a)
            last = a + n == S
            lg = self.extend(ids if n == S else ids[:, a:a + n], list(range(n)) if all_logits else ([n - 1] if last else []))
            if all_logits:
                parts.append(lg.dataAsync().reshape(B, n, self.V))
        if all_logits:
            full = np.concatenate(parts, axis=1)
            lg = Tensor(np.ascontiguousarray(full[:, -1]))
        tok, uniforms = core.empty((B,), "int64"), core.zeros((B,), "float32")
        if self.sampler is not None:
            self._fresh_uniforms(uniforms)
        self._next_tokens(lg, uniforms, tok)
        return (tok, Tensor(full)) if all_logits else tok

    # ------------------------------------------------------------------ decode
    def _decode_state(self, B: int) -> dict:
        if self._decode is not None and self._decode["B"] == B:
            return self._decode
        self.dispose()
        d = {"B": B, "graph": None, "scalars": core.zeros((2,), "int32"), "ids": core.zeros((B,), "int64"), "ws": _Buffers(),
             "logits": core.empty((B, self.V), "float32"), "uniforms": core.zeros((B,), "float32"), "at": -1}
        d["pos"] = d["scalars"].slice([slice(0, 1)])
        self._decode = d
        return d

    def _enqueue_decode_step(self, d: dict) -> None:
        lib.call("kd_set_pdl", 1 if self.use_pdl else 0)
        try:
            h = self._run(d["ws"], d["ids"], d["B"], 1, d["pos"], 0)
            self._logits(d["ws"], h, d["logits"])
            self._next_tokens(d["logits"], d["uniforms"], d["ids"])
            lib.call("kd_increment_i32", _r(d["pos"]), 1)
        finally:
            lib.call("kd_set_pdl", 0)

    def _warm_decode_step(self, d: dict) -> None:
        saved = self.cache.snapshot()       # the step advances the recurrent states
        self._enqueue_decode_step(d)
        self.cache.restore(saved)

    def start_decode(self, first_tokens: Tensor, use_graph: bool = True) -> dict:
        d = super().start_decode(first_tokens, use_graph)
        d["at"] = self.pos
        return d

    def decode_step(self) -> Tensor:
        self.cache.room(1)
        out = super().decode_step()
        self.cache.pos = self._decode["at"] = self.pos
        return out

    def _decode_given(self, ids: np.ndarray) -> Tensor:
        """One decode step on given tokens [B, 1]; returns the step's logits [B, V] (a copy)."""
        toks = Tensor(ids.reshape(-1).astype(np.int64))
        d = self._decode
        if d is None or d["B"] != ids.shape[0] or d["graph"] is None or d["at"] != self.pos:
            d = self.start_decode(toks)
        else:
            core.copy_(d["ids"], toks)
        self.decode_step()
        return d["logits"].clone()
