"""Engine for decoders that mix layer types: latent attention, gated delta rule, expert feed-forward,
Dynamic Tanh norms (the Pedorax design), in bf16 or in fp32 throughout.

One step function, `_run`, serves whole prompts, portions of prompts and decode steps: it takes S new
tokens of B sequences at the cache's position and leaves their rows and states in the cache.  Per layer:

  one GEMM for everything that reads the norm's output (queries, latent or q/k/v, decay and gate inputs,
  step sizes; the router's rows ride along and leave in fp32)
  latent attention    norm + rotation + cache row -> attention over the cache rows (W_uk absorbed into the
                      queries, W_uv applied to the combined latents), or, for long bf16 prompts, keys and
                      values expanded once and the tcgen05 prefill kernel -> W_o
  gated delta rule    decay / gate projections -> convolution + unit norms + recurrence in one kernel ->
                      output norm and gate -> W_o
  experts             route -> rows in expert order -> gate/up with the clamped GLU in the epilogue -> down
  residual            x += mixer + weighted expert rows, and the NEXT layer's norm, in one kernel

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

KD_EPI_NONE, KD_EPI_CLAMPED_GLU = 0, 4


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


class _Norm:
    def __init__(self, w: _Weights, name: str, width: int):
        self.alpha = float(w.vector(name + ".alpha", (), 0.5))
        self.w = Tensor(w.vector(name, (width,), 1.0), dtype="float32")
        self.b = Tensor(w.vector(name + ".b", (width,), 0.0), dtype="float32")

    def args(self):
        return ctypes.c_float(self.alpha), _r(self.w), _r(self.b)


class _Projection:
    """The GEMM over the norm's output: mixer columns in the engine's type, router rows in fp32 behind them."""

    def __init__(self, w: _Weights, parts, width: int, prefix: str, experts: ExpertsSpec | None):
        self.cols, at = {}, 0
        for key, rows, pad in parts:
            self.cols[key] = at
            at += _up(rows, pad)
        self.n = _up(at, 32)
        rows = [(prefix + "mix." + key, r, _up(r, pad)) for key, r, pad in parts]
        rows.append((None, 0, self.n - at))
        self.tail = 0
        if experts is not None:
            self.tail = _up(experts.experts, 8)
            rows.append((prefix + "mlp.router", experts.experts, self.tail))
        self.weight = w.stacked_rows(rows, width)


class _LatentAttention:
    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m: LatentAttentionSpec, experts):
        self.m, self.i, p = m, i, f"l{i}."
        self.own = m.kvFrom is None
        parts = [("q", m.heads * (m.dim + m.rotDim), 8)]
        if self.own:
            parts.append(("dkv", m.kvRank + m.rotDim, 8))
        self.proj = _Projection(w, parts, eng.W, p, experts)
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

    def __call__(self, eng: "HybridEngine", ws: _Buffers, proj3: Tensor, B: int, S: int, pos) -> Tensor:
        m, T, dt = self.m, B * S, eng.dtype
        pos_dev, pos_host = pos
        cache = eng.cache.of(self.i).rows
        cache = cache if cache.shape[0] == B else cache.slice([slice(0, B), slice(None), slice(None)])
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


class _ChannelDelta:
    def __init__(self, eng: "HybridEngine", w: _Weights, i: int, m: ChannelDeltaSpec, experts):
        self.m, self.i, p = m, i, f"l{i}."
        qk, vv = m.kvHeads * m.dim, m.heads * m.vdim
        ra, rg = w.rank_of(p + "mix.a1", m.dim), w.rank_of(p + "mix.g1", m.vdim)
        self.ra, self.rg = _up(ra, 8), _up(rg, 8)
        # q, k, v side by side without padding: their channels are the convolution's
        self.proj = _Projection(w, [("q", qk, 1), ("k", qk, 1), ("v", vv, 8), ("a1", ra, 8), ("g1", rg, 8), ("b", m.heads, 8)], eng.W, p, experts)

        def low_rank(name, rows, rank, padded):
            if w.random:
                return w.matrix("", (rows, padded))
            a = np.zeros((rows, padded), np.float32)
            a[:, :rank] = w.host(p + name, (rows, rank))
            return w._put(a)
        self.wa2 = low_rank("mix.a2", m.heads * m.dim, ra, self.ra)
        self.wg2 = low_rank("mix.g2", vv, rg, self.rg)
        taps = lambda n, rows: Tensor(w.vector(p + f"mix.{n}.conv", (rows, m.taps), lambda s: w._rng.standard_normal(s) * 0.5), dtype="float32")  # noqa: E731
        self.conv = taps("q", qk), taps("k", qk), taps("v", vv)
        self.neg_rate = Tensor(-np.exp(w.vector(p + "mix.A_log", (m.heads,), -1.0)), dtype="float32")
        self.dt_bias = Tensor(w.vector(p + "mix.dt_bias", (m.heads * m.dim,), -3.0), dtype="float32")
        self.norm = Tensor(w.vector(p + "mix.norm", (m.vdim,), 1.0), dtype="float32")
        self.wo = w.matrix(p + "mix.o", (eng.W, vv))

    def __call__(self, eng: "HybridEngine", ws: _Buffers, proj3: Tensor, B: int, S: int, pos) -> Tensor:
        m, T, dt, c = self.m, B * S, eng.dtype, self.proj.cols
        kept = eng.cache.of(self.i)
        part = lambda t: t if t.shape[0] == B else t.slice([slice(0, B)] + [slice(None)] * (t.ndim - 1))  # noqa: E731
        state, history = part(kept.state), part(kept.history)
        proj2 = proj3.view(T, self.proj.n)
        decay, gate = ws("decay", (T, m.heads * m.dim), "float32"), ws("gate", (T, m.heads * m.vdim), dt)
        eng.linear(_cols(proj2, c["a1"], c["a1"] + self.ra), self.wa2, decay)
        eng.linear(_cols(proj2, c["g1"], c["g1"] + self.rg), self.wg2, gate)
        o, out = ws("delta_o", (T, m.heads * m.vdim), "float32"), ws("mixed", (T, m.heads * m.vdim), dt)
        lib.call("kd_delta_rule", _r(proj3), c["q"], c["k"], c["v"], c["b"], _r(decay), m.heads, m.kvHeads, m.dim, m.vdim,
                 *(_r(t) for t in self.conv), _r(self.neg_rate), _r(self.dt_bias), _r(history), _r(state), _r(o))
        lib.call("kd_delta_out", _r(o), _r(gate), _r(self.norm), ctypes.c_float(eng.cfg.normEps), _r(proj3), c["q"], m.taps, _r(history), _r(out))
        return out


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


class HybridEngine(DecoderEngine):
    def __init__(self, cfg: PedoraxConfig, weights, max_batch: int, max_seq_len: int):
        """weights: a mapping of the checkpoint's tensor names to float32 arrays (io.SafetensorStateDict, a
        dict), or a RandomInit.  cfg.dtype is "bfloat16" or "float32"."""
        cfg.validate()
        if cfg.dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {cfg.dtype!r}: the hybrid engine runs in bfloat16 or float32")
        self._init_decoding(max_batch, max_seq_len)
        self.cfg, self.dtype, self.W, self.V = cfg, cfg.dtype, cfg.hiddenSize, cfg.vocabSize
        self._tables = {}
        w = _Weights(weights, self.dtype)
        self.embed = w.matrix("embed", (self.V, self.W))
        self.norms, self.mixers, self.experts = [], [], []
        for i, layer in enumerate(cfg.layers):
            self.norms.append(_Norm(w, f"l{i}.norm1", self.W))
            kind = _LatentAttention if isinstance(layer.mixer, LatentAttentionSpec) else _ChannelDelta
            self.mixers.append(kind(self, w, i, layer.mixer, layer.experts))
            self.experts.append(_Experts(self, w, i, layer.experts) if layer.experts is not None else None)
        self.norms.append(_Norm(w, "final.norm", self.W))
        self.max_experts = max([e.e.experts for e in self.experts if e is not None], default=1)
        self.cache = SequenceCache(cfg.layers, max_batch, max_seq_len, self.dtype)
        self.expand_from = 64      # portions of at least this many tokens expand keys and values
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

    # ------------------------------------------------------------------ one step over S tokens of B sequences
    def _run(self, ws: _Buffers, ids: Tensor, B: int, S: int, pos_dev: Tensor | None, pos_host: int) -> Tensor:
        """ids: device int32/int64 [B*S].  Runs them at the given position; returns the final norm's output [B*S, W]."""
        T, dt, c = B * S, self.dtype, self.cfg
        x, h = ws("x", (T, self.W), "float32"), ws("h", (T, self.W), dt)
        counts = ws("moe_counts", (len(self.experts), self.max_experts), "int32")
        lib.call("kd_fill", _r(counts), ctypes.c_double(0.0))
        lib.call("kd_embed_dynamic_tanh", _r(self.embed), _r(ids), ctypes.c_float(c.embeddingScale), *self.norms[0].args(), _r(x), _r(h))
        for i, (mixer, experts) in enumerate(zip(self.mixers, self.experts)):
            p = mixer.proj
            proj3 = ws("proj", (B, S, p.n), dt)
            tail = ws("tail", (T, p.tail), "float32") if p.tail else None
            self.linear(h, p.weight, proj3.view(T, p.n), tail=tail)
            mixed = mixer(self, ws, proj3, B, S, (pos_dev, pos_host))
            mix = self._out_projection(ws, mixed, mixer.wo, x, T)
            y = slots = weights = None
            if experts is not None:
                y, slots, weights = experts(self, ws, h, tail, counts.slice([slice(i, i + 1), slice(0, experts.e.experts)]))
            lib.call("kd_residual_dynamic_tanh", _r(x), _r(mix), _r(y), _r(slots), _r(weights), *self.norms[i + 1].args(), _r(x), _r(h))
            if self.trace is not None:
                self.trace.append(x.dataAsync().copy())
        return h

    def _out_projection(self, ws: _Buffers, mixed: Tensor, wo: Tensor, x: Tensor, T: int):
        """x += mixed W_o^T in the GEMM's epilogue for many rows (returns None); for a few rows fp32 partial sums that
        the residual kernel adds."""
        if self.dtype == "bfloat16" and T > 64 and mixed.shape[1] % 8 == 0 and self.W % 8 == 0:
            self.linear(mixed, wo, x, residual=x)
            return None
        if self.dtype == "bfloat16" and T <= 64 and mixed.shape[1] % 8 == 0:
            s = ctypes.c_int(0)
            lib.call("kd_linear_bf16_skinny_splits", ctypes.c_int64(self.W), ctypes.c_int64(mixed.shape[1]), ctypes.byref(s))
            mix = ws("mix", (s.value, T, self.W), "float32")
            lib.call("kd_linear_bf16_skinny", _r(mixed), _r(wo), 0, _r(mix))
            return mix
        mix = ws("mix", (1, T, self.W), "float32")
        self.linear(mixed, wo, mix.view(T, self.W))
        return mix

    def _logits(self, ws: _Buffers, rows: Tensor, out: Tensor) -> None:
        """out [n, V] fp32 = logit_scale * rows [n, W] embed^T (64 rows a call: the vocabulary matrix streams once each)."""
        n = rows.shape[0]
        for a in range(0, n, 64):
            b = min(n, a + 64)
            r, o = (t.slice([slice(a, b), slice(None)]) for t in (rows, out))
            self.linear(r, self.embed, o, alpha=self.cfg.logitScale)

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
