"""The kernels behind the hybrid engine, one by one, against plain formulations in float64.  Where random numbers
would hide a fault, the inputs are made so that it shows: one key among hundreds takes all the weight, a sink
takes most of it, decays span the whole range of fp32."""
import collections
import ctypes

import numpy as np
import pytest

from kandle_b200 import core, lib
from kandle_b200.core import Tensor
from oracle import hybrid

pytestmark = pytest.mark.gpu
F = ctypes.c_float


_alive = collections.deque(maxlen=64)      # operands of recent calls (a dropped tensor frees its storage at once)


def _r(t):
    _alive.append(t)
    return ctypes.byref(t._handle.c()) if t is not None else None


def _put(a, dtype="float32"):
    return Tensor(np.ascontiguousarray(a, np.float32), dtype=dtype)


def _get(t):
    return np.asarray(t.dataAsync(), np.float64)


def _bf(a):
    return lib.round_to_bf16(np.asarray(a, np.float32))


def _rng(*seed):
    return np.random.default_rng(list(seed))


# ----------------------------------------------------------------------------- Dynamic Tanh and the residual
@pytest.mark.parametrize("width", [64, 50, 1032])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_embedding_and_residual_norms(backend, width, dtype):
    rng = _rng(width)
    T, V, top, R = 5, 11, 3, 20
    table, ids = _bf(rng.standard_normal((V, width))), rng.integers(0, V, T)
    w, b = rng.standard_normal(width), rng.standard_normal(width)
    tol = 2e-6 if dtype == "float32" else 1e-2
    x, h = core.empty((T, width)), core.empty((T, width), dtype)
    lib.call("kd_embed_dynamic_tanh", _r(_put(table, dtype)), _r(Tensor(ids.astype(np.int64))), F(1.7), F(0.6), _r(_put(w)), _r(_put(b)), _r(x), _r(h))
    want = table[ids] * 1.7
    assert np.abs(_get(x) - want).max() <= 1e-6 * np.abs(want).max()
    assert np.abs(_get(h) - hybrid.dynamic_tanh(want, 0.6, w, b)).max() <= tol * 3
    x0, mix, y = rng.standard_normal((T, width)), rng.standard_normal((2, T, width)), _bf(rng.standard_normal((R, width)))
    slots, ws = rng.integers(0, R, (T, top)).astype(np.int32), rng.uniform(size=(T, top))
    for use_mix, use_y in ((1, 1), (1, 0), (0, 1), (0, 0)):
        want = x0 + (mix.sum(0) if use_mix else 0) + (np.einsum("tk,tkw->tw", ws, y[slots]) if use_y else 0)
        lib.call("kd_residual_dynamic_tanh", _r(_put(x0)), _r(_put(mix)) if use_mix else None, _r(_put(y, dtype)) if use_y else None,
                 _r(Tensor(slots)) if use_y else None, _r(_put(ws)) if use_y else None, F(-0.4), _r(_put(w)), _r(_put(b)), _r(x), _r(h))
        assert np.abs(_get(x) - want).max() <= 3e-6 * np.abs(want).max()
        assert np.abs(_get(h) - hybrid.dynamic_tanh(want, -0.4, w, b)).max() <= tol * 3


# ----------------------------------------------------------------------------- linears
@pytest.mark.parametrize("M, N, K, tail", [(3, 96, 64, 16), (64, 160, 72, 8), (65, 160, 72, 8), (300, 512, 256, 64), (5, 50, 33, 7), (200, 40, 24, 0), (1, 64, 64, 0)])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_linear_with_strided_rows_and_fp32_tail(backend, M, N, K, tail, dtype):
    rng = _rng(M, N, K)
    x, w = _bf(rng.standard_normal((M, K + 16))), _bf(rng.standard_normal((N, K)))
    xd, want = _put(x, dtype), x[:, 8:8 + K].astype(np.float64) @ w.T
    xs = xd.slice([slice(None), slice(8, 8 + K)])
    n = N - tail
    out, t = core.empty((M, n), dtype), core.empty((M, tail), "float32") if tail else None
    lib.call("kd_linear_ex", _r(xs), _r(_put(w, dtype)), None, F(1.0), _r(out), _r(t))
    scale = np.abs(want).max()
    assert np.abs(_get(out) - want[:, :n]).max() <= (1e-5 if dtype == "float32" else 6e-3) * scale
    if tail:
        assert np.abs(_get(t) - want[:, n:]).max() <= 1e-5 * scale      # never rounded to bf16
    o32, res = core.empty((M, N)), rng.standard_normal((M, N))
    lib.call("kd_linear_ex", _r(xs), _r(_put(w, dtype)), _r(_put(res)), F(1.0), _r(o32), None)
    assert np.abs(_get(o32) - want - res).max() <= 1e-5 * scale
    lib.call("kd_linear_ex", _r(xs), _r(_put(w, dtype)), None, F(0.3), _r(o32), None)
    assert np.abs(_get(o32) - 0.3 * want).max() <= 1e-5 * scale


# ----------------------------------------------------------------------------- experts
def _route(logits, top, groups, keep, h):
    T, E = logits.shape
    ids, ranks, slots = (core.empty((T, top), "int32") for _ in range(3))
    ws, counts, off = core.empty((T, top)), core.zeros((E,), "int32"), core.empty((E + 1,), "int32")
    lib.call("kd_moe_route", _r(_put(logits)), top, groups, keep, _r(ids), _r(ws), _r(ranks), _r(counts))
    xs = core.empty((T * top, h.shape[1]), h.dtype)
    lib.call("kd_moe_gather", _r(h), _r(ids), _r(ranks), _r(counts), E, _r(slots), _r(off), _r(xs))
    return ids.dataAsync(), _get(ws), slots.dataAsync(), off.dataAsync(), xs


@pytest.mark.parametrize("E, top, groups, keep", [(8, 3, 4, 2), (64, 6, 8, 4), (12, 1, 1, 1), (6, 4, 6, 4), (300, 8, 10, 5), (64, 8, 32, 32), (4, 4, 2, 2)])
@pytest.mark.parametrize("T", [1, 37, 700])
def test_routing_and_expert_order(backend, E, top, groups, keep, T):
    rng = _rng(E, T)
    logits = rng.standard_normal((T, E)) * (3 if E < 100 else 1)
    h = rng.standard_normal((T, 24)).astype(np.float32)
    ids, ws, slots, off, xs = _route(logits, top, groups, keep, _put(h))
    want_ids, want_w = hybrid.route(logits.astype(np.float32).astype(np.float64), np.eye(E), {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}})
    same = (ids == want_ids).all(1)
    assert same.all() if E < 100 else same.mean() >= 0.99      # (hundreds of sigmoids a row: some are equal in fp32)
    assert np.abs(ws - want_w)[same].max() <= 1e-5
    counts = np.bincount(ids.ravel(), minlength=E)
    assert np.array_equal(off, np.concatenate([[0], np.cumsum(counts)]))
    assert np.array_equal(np.sort(slots.ravel()), np.arange(T * top))        # a permutation ...
    assert ((slots >= off[ids]) & (slots < off[ids + 1])).all()               # ... by expert
    assert np.array_equal(np.asarray(xs.dataAsync())[slots], np.repeat(h[:, None], top, 1))


@pytest.mark.parametrize("E, N, K, counts", [(3, 64, 64, [1, 0, 5]), (5, 96, 72, [130, 0, 7, 256, 1]), (64, 512, 128, None), (4, 48, 40, [0, 0, 0, 9]), (2, 32, 18, [3, 4]), (8, 256, 512, None)])
@pytest.mark.parametrize("glu", [False, True])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_grouped_linear(backend, E, N, K, counts, glu, dtype):
    rng = _rng(E, N, K)
    counts = rng.integers(0, 9, E) if counts is None else np.array(counts)
    if glu and N % 32:
        N = (N + 31) // 32 * 32
    off = np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)
    R = int(off[-1])
    x, w, limit = _bf(rng.standard_normal((R, K))), _bf(rng.standard_normal((E, N, K)) * 2 * K ** -0.5), 1.3
    out = core.empty((R, N // 2 if glu else N), dtype)
    lib.call("kd_moe_linear", _r(_put(x, dtype)), _r(_put(w, dtype)), _r(Tensor(off)), 4 if glu else 0, F(limit), _r(out))
    want = np.concatenate([x[off[e]:off[e + 1]].astype(np.float64) @ w[e].T.astype(np.float64) for e in range(E)])
    if glu:
        both = want.reshape(R, N // 32, 2, 16)
        g, u = np.minimum(both[:, :, 0], limit).reshape(R, -1), np.clip(both[:, :, 1], -limit, limit).reshape(R, -1)
        assert (g == limit).any() and (np.abs(u) == limit).any()             # the clamps are in play
        want = g * hybrid.sigmoid(1.702 * g) * (u + 1)
    assert np.abs(_get(out) - want).max() <= (1e-5 if dtype == "float32" else 6e-3) * max(1.0, np.abs(want).max())


# ----------------------------------------------------------------------------- latent attention
def _attend(q, cache, rank, scale, sink, pos):
    """q [B,S,H,width], cache [B,ctx,width] (float64): [B,S,H,rank] of latents."""
    B, S, H, _ = q.shape
    out = np.empty((B, S, H, rank))
    for b in range(B):
        for s in range(S):
            rows = cache[b, :pos + s + 1]
            p = hybrid.sink_softmax(q[b, s] @ rows.T * scale, sink[:, None])
            out[b, s] = p @ rows[:, :rank]
    return out


def _latent_case(B, S, H, rank, rot, vdim, pos, max_s, dtype, splits=None, edit=None, seed=0):
    """Runs attention + values over a cache; rows past the context are NaN.  edit(q, cache, sink) plants what shows."""
    rng = _rng(B, S, H, rank, rot, pos, seed)
    width = (rank + rot + 15) // 16 * 16
    q, cache = np.zeros((B, S, H, width)), np.zeros((B, max_s, width))
    q[..., :rank + rot], cache[..., :rank + rot] = rng.standard_normal((B, S, H, rank + rot)), rng.standard_normal((B, max_s, rank + rot))
    sink, wuv = rng.standard_normal(H), _bf(rng.standard_normal((H, vdim, rank)) * rank ** -0.5)
    if edit:
        edit(q, cache, sink)
    q, cache = _bf(q), _bf(cache)
    scale = (rank + rot) ** -0.5
    ref = np.einsum("hvr,bshr->bshv", wuv.astype(np.float64), _attend(q.astype(np.float64), cache.astype(np.float64), rank, scale, sink, pos))
    cache[:, pos + S:] = np.nan
    if splits is None:
        n = ctypes.c_int(0)
        lib.call("kd_latent_attention_splits", B, S, H, max_s, ctypes.byref(n))
        splits = n.value
    T = B * S
    po, pm = core.full((T * H, splits, rank), float("nan")), core.full((T * H, splits, 2), float("nan"))
    qd, cd, pd = _put(q, dtype), _put(cache, dtype), Tensor(np.array([pos], np.int32))
    for dev in (None, pd):
        lib.call("kd_latent_attention", _r(qd), _r(cd), rank, F(scale), _r(dev), 0 if dev is not None else pos, _r(po), _r(pm))
        got = []
        for tensor_cores in (False, True):
            out = core.full((T, H * vdim), float("nan"), dtype)
            a, c = (_put(wuv, dtype), core.empty((T * H, rank), dtype)) if tensor_cores else (None, None)
            lib.call("kd_latent_values", _r(po), _r(pm), _r(_put(sink)), _r(_put(wuv.transpose(0, 2, 1), dtype)), _r(a), _r(c), _r(out))
            got.append(_get(out).reshape(ref.shape))
        tol = (2e-6 if dtype == "float32" else 1.2e-2) * max(1.0, np.abs(ref).max())
        for g in got:
            assert np.abs(g - ref).max() <= tol, (np.abs(g - ref).max(), tol)
    return ref


SHAPES = [(1, 1, 7, 160, 16, 40), (2, 1, 16, 512, 64, 128), (1, 1, 40, 64, 16, 24), (2, 3, 5, 40, 8, 12), (1, 7, 20, 256, 64, 64), (1, 2, 3, 600, 64, 16), (1, 1, 33, 9, 2, 5)]


@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("pos", [0, 1, 30, 31, 62, 63, 64, 127, 128, 300])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_latent_attention_at_tile_edges(backend, shape, pos, dtype):
    _latent_case(*shape, pos, 320, dtype)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("key", [0, 1, 63, 64, 200, 698, 699])
@pytest.mark.parametrize("splits", [1, 5, 11, 40])
def test_one_key_among_hundreds(backend, dtype, key, splits):
    """Head 0's query is that one key times a factor: its output is that key's value alone."""
    def edit(q, cache, sink):
        q[:, :, 0] = cache[:, None, key] * 8.0
    ref = _latent_case(1, 1, 4, 48, 16, 48, 699, 704, dtype, splits, edit)
    plain = _latent_case(1, 1, 4, 48, 16, 48, 699, 704, dtype, splits)
    assert np.abs(ref[0, 0, 0]).max() > 3 * np.abs(plain[0, 0, 0]).max()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_a_key_just_past_a_query_stays_unseen(backend, dtype):
    """Portion of three queries: the row behind the first query would take all the weight if it were seen too early."""
    def edit(q, cache, sink):
        q[:, :, 1] = cache[:, None, 65] * 8.0
    ref = _latent_case(1, 3, 4, 48, 16, 48, 64, 80, dtype, None, edit)
    assert np.abs(ref[0, 1, 1] - ref[0, 0, 1]).max() > 0.3


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("value", [-60.0, 0.0, 12.0, 95.0])
def test_sink_from_nothing_to_everything(backend, dtype, value):
    def edit(q, cache, sink):
        sink[:] = value
    _latent_case(2, 1, 4, 48, 16, 48, 130, 256, dtype, 3, edit)


@pytest.mark.parametrize("dim, rot, rank, H", [(128, 64, 512, 16), (32, 16, 160, 7), (24, 16, 48, 3), (7, 2, 9, 2), (64, 0, 40, 3), (96, 32, 64, 5)])
@pytest.mark.parametrize("T", [1, 5, 40])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_absorbed_queries(backend, dim, rot, rank, H, T, dtype):
    rng = _rng(dim, rank, T)
    width, n = (rank + rot + 15) // 16 * 16, 8 + H * (dim + rot) + 8
    n = (n + 7) // 8 * 8
    proj, wuk = _bf(rng.standard_normal((1, T, n))), _bf(rng.standard_normal((H, dim, rank)) * max(dim, 1) ** -0.5)
    q = proj[0, :, 8:8 + H * (dim + rot)].reshape(T, H, dim + rot).astype(np.float64)
    want = np.zeros((T, H, width))
    want[..., :rank] = np.einsum("thd,hdr->thr", q[..., :dim], wuk)
    want[..., rank:rank + rot] = q[..., dim:]
    for given in (False, True):
        out = core.full((T, H, width), float("nan"), dtype)
        lib.call("kd_latent_absorb", _r(_put(proj, dtype)), 8, rot, _r(_put(wuk, dtype)), _r(_put(wuk.transpose(0, 2, 1), dtype)) if given else None, _r(out))
        assert np.abs(_get(out) - want).max() <= (1e-5 if dtype == "float32" else 6e-3) * np.abs(want).max()


# ----------------------------------------------------------------------------- gated delta rule
def _delta_case(B, S, H, Hk, dim, vdim, taps, dtype, cuts, a_mean=-2.0, a_sd=1.0, rate_sd=1.0, seed=0):
    rng = _rng(B, S, H, dim, vdim, taps, seed)
    qk, vv = Hk * dim, H * vdim
    n = ((2 * qk + vv + H) + 15) // 8 * 8
    proj = _bf(rng.standard_normal((B, S, n)))
    a = rng.standard_normal((B, S, H * dim)).astype(np.float32) * a_sd
    conv = [_bf(rng.standard_normal((r, taps)) * 0.6 + 0.2) for r in (qk, qk, vv)]
    rate, bias = np.exp(rng.standard_normal(H) * rate_sd).astype(np.float32), (rng.standard_normal(H * dim) + a_mean).astype(np.float32)
    r, c = ctypes.c_int(0), ctypes.c_int(0)
    lib.call("kd_delta_state_shape", dim, vdim, ctypes.byref(r), ctypes.byref(c))
    state, hist = core.zeros((B, H, r.value, c.value)), core.zeros((B, max(taps - 1, 1), 2 * qk + vv), dtype)
    ws = [_put(x) for x in conv]
    norm_w, gate = rng.standard_normal(vdim).astype(np.float32), _bf(rng.standard_normal((B, S, vv)))
    outs, finals, at = [], [], 0
    for n_tok in cuts:
        pd = _put(proj[:, at:at + n_tok], dtype)
        o, y = core.full((B * n_tok, vv), float("nan")), core.full((B * n_tok, vv), float("nan"), dtype)
        lib.call("kd_delta_rule", _r(pd), 0, qk, 2 * qk, 2 * qk + vv, _r(_put(a[:, at:at + n_tok].reshape(B * n_tok, -1))), H, Hk, dim, vdim, *(_r(x) for x in ws),
                 _r(_put(-rate)), _r(_put(bias)), _r(hist), _r(state), _r(o))
        lib.call("kd_delta_out", _r(o), _r(_put(gate[:, at:at + n_tok].reshape(B * n_tok, -1), dtype)), _r(_put(norm_w)), F(1e-5), 0, _r(pd), 0, taps, _r(hist), _r(y))
        outs.append(_get(o).reshape(B, n_tok, H, vdim))
        finals.append(_get(y).reshape(B, n_tok, H, vdim))
        at += n_tok
    assert at == S
    got, fin = np.concatenate(outs, 1), np.concatenate(finals, 1)
    for b in range(B):
        p = proj[b].astype(np.float64)
        q, k, v = (hybrid.causal_conv_silu(p[:, i:i + len(w)], w.astype(np.float64)) for i, w in zip((0, qk, 2 * qk), conv))
        rep = H // Hk
        q = np.repeat(hybrid.unit(q.reshape(S, Hk, dim)) * dim ** -0.5, rep, 1)
        k = np.repeat(hybrid.unit(k.reshape(S, Hk, dim)), rep, 1)
        g = np.exp(-rate[None, :, None].astype(np.float64) * hybrid.softplus(a[b].astype(np.float64) + bias).reshape(S, H, dim))
        o, s = hybrid.delta_rule(q, k, v.reshape(S, H, vdim), g, hybrid.sigmoid(p[:, 2 * qk + vv:2 * qk + vv + H]))
        scale = np.sqrt((o ** 2).mean())
        assert np.abs(got[b] - o).max() <= 3e-5 * max(scale, np.abs(o).max()), (np.abs(got[b] - o).max(), scale)
        kept = _get(state)[b]
        assert np.abs(kept[:, :dim, :vdim] - s).max() <= 3e-5 * np.abs(s).max()
        assert (kept[:, dim:] == 0).all() and (kept[:, :, vdim:] == 0).all()
        want = hybrid.rms_norm(o, norm_w, 1e-5) * hybrid.sigmoid(gate[b].astype(np.float64)).reshape(S, H, vdim)
        assert np.abs(fin[b] - want).max() <= (1e-4 if dtype == "float32" else 1e-2) * np.abs(want).max()


SIZES = [(2, 1, 16, 8, 4), (3, 3, 64, 64, 4), (3, 3, 20, 36, 3), (4, 2, 128, 128, 4), (2, 2, 130, 40, 4), (1, 1, 256, 128, 2), (2, 1, 33, 65, 1), (2, 2, 32, 300, 4), (6, 2, 48, 24, 8), (1, 1, 9, 7, 5)]


@pytest.mark.parametrize("size", SIZES, ids=str)
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_delta_rule_sizes_and_portions(backend, size, dtype):
    for cuts in ([37], [1, 2, 3, 16, 15], [1] * 5 + [32]):
        _delta_case(2, 37, *size, dtype, cuts)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_delta_rule_long_sequences(backend, dtype):
    _delta_case(1, 700, 2, 2, 64, 32, 4, dtype, [400, 2, 298], a_mean=-4.0)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("a_mean, a_sd, rate_sd", [(-12.0, 3.0, 0.5), (3.0, 4.0, 1.5), (8.0, 12.0, 2.0), (60.0, 30.0, 1.0)])
def test_delta_rule_decays_from_one_to_zero(backend, dtype, a_mean, a_sd, rate_sd):
    """Decays that keep the state, that wipe single channels, and that underflow to zero outright."""
    for cuts in ([50], [3, 4, 5, 38]):
        _delta_case(1, 50, 3, 3, 40, 24, 4, dtype, cuts, a_mean, a_sd, rate_sd)


def test_delta_rule_many_heads_share_a_block(backend):
    """Enough heads for several per block, in a batch: bf16 and fp32 agree with the plain form for every one."""
    _delta_case(20, 19, 16, 8, 64, 64, 4, "bfloat16", [18, 1])
    _delta_case(12, 19, 32, 16, 32, 32, 4, "float32", [2, 17])
