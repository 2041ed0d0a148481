"""The kernels behind the Vogozen layers, one by one, against the plain formulations in float64.  Where random numbers
would hide a fault, the inputs are made so that it shows: one key takes all the weight just inside or just outside a
window, scores stay far below the sink, decays span the whole range of fp32."""
import collections
import ctypes

import numpy as np
import pytest

from kandle_b200 import core, lib
from kandle_b200.core import Tensor
from oracle import hybrid, vogozen

pytestmark = pytest.mark.gpu
F = ctypes.c_float
DTYPES = ["bfloat16", "float32"]

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


def _close(got, want, tol, what=""):
    err = np.abs(got - want).max() / max(1e-30, np.abs(want).max())
    assert err <= tol, f"{what}: {err:.2e} > {tol:.0e}"


# ----------------------------------------------------------------------------- embedding, residual and output norm
@pytest.mark.parametrize("width", [64, 50, 516, 1032, 4096, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_and_output_norm(backend, width, dtype):
    rng = _rng(width)
    T, V = 5, 11
    table, ids = _bf(rng.standard_normal((V, width))), rng.integers(0, V, T)
    x, h = core.empty((T, width)), core.empty((T, width), dtype)
    lib.call("kd_embed_rows", _r(_put(table, dtype)), _r(Tensor(ids.astype(np.int64))), _r(x), _r(h))
    assert np.array_equal(_get(x), table[ids]) and np.array_equal(_get(h), table[ids])
    w, fw = 1 + 0.3 * rng.standard_normal(width), 1 + 0.3 * rng.standard_normal(width)
    for splits, ydt, scale in ((1, dtype, 1.0), (3, "float32", 30.0), (2, "float32", 1e-4)):
        y = _bf(rng.standard_normal((splits, T, width)) * scale)
        before = _get(x)
        want = before + hybrid.rms_norm(y.astype(np.float64).sum(0), w, 1e-3)
        lib.call("kd_residual_post_norm", _r(x), _r(_put(y, ydt)), _r(_put(w)), F(1e-3), None, _r(x), _r(h))
        _close(_get(x), want, 2e-6, "residual")
        _close(_get(h), want, 1e-6 if dtype == "float32" else 5e-3, "copy")
        out = core.full((T, width), float("nan"))
        lib.call("kd_residual_post_norm", _r(_put(before)), _r(_put(y, ydt)), _r(_put(w)), F(1e-3), _r(_put(fw)), _r(out), _r(h))
        _close(_get(out), want, 2e-6, "residual beside the final norm")
        _close(_get(h), hybrid.rms_norm(want, fw, 1e-3), 2e-6 if dtype == "float32" else 5e-3, "final norm")


def test_embedding_reports_a_bad_id(backend):
    x, h = core.empty((1, 8)), core.empty((1, 8))
    lib.call("kd_embed_rows", _r(_put(np.ones((3, 8)))), _r(Tensor(np.array([3], np.int32))), _r(x), _r(h))
    with pytest.raises(lib.KandleCudaError, match="101"):
        backend.synchronize()


# ----------------------------------------------------------------------------- projections
@pytest.mark.parametrize("M, K, ff", [(1, 64, 32), (7, 72, 48), (40, 256, 9600), (5, 50, 16), (200, 128, 80), (300, 64, 512), (129, 136, 2048)])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("epilogue", [2, 5])
def test_gated_projection(backend, M, K, ff, dtype, epilogue):
    rng = _rng(M, K, ff)
    x, g, u = _bf(rng.standard_normal((M, K))), _bf(rng.standard_normal((ff, K)) * 2 * K ** -0.5), _bf(rng.standard_normal((ff, K)) * K ** -0.5)
    from kandle_b200.engine import interleave_gate_up
    out = core.full((M, ff), float("nan"), dtype)
    lib.call("kd_linear_glu", _r(_put(x, dtype)), _r(_put(interleave_gate_up(g, u), dtype)), epilogue, _r(out))
    xd = x.astype(np.float64)
    act = vogozen.silu if epilogue == 2 else vogozen.gelu_tanh
    _close(_get(out), act(xd @ g.T) * (xd @ u.T), 2e-6 if dtype == "float32" else 6e-3)


@pytest.mark.parametrize("M, K, N", [(1, 64, 8), (9, 72, 16), (33, 50, 13), (300, 128, 64)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_tanh_projection(backend, M, K, N, dtype):
    rng = _rng(M, K, N)
    x, w = _bf(rng.standard_normal((M, K))), _bf(rng.standard_normal((N, K)) * 3 * K ** -0.5)
    out = core.full((M, N), float("nan"), dtype)
    lib.call("kd_linear_tanh", _r(_put(x, dtype)), _r(_put(w, dtype)), _r(out))
    _close(_get(out), np.tanh(x.astype(np.float64) @ w.T), 2e-6 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("M, K, N, E", [(1, 64, 40, 4), (5, 72, 72, 4), (130, 64, 264, 4), (33, 50, 20, 3), (400, 256, 512, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_stacked_projections_over_inputs_of_their_own(backend, M, K, N, E, dtype):
    rng = _rng(M, K, N, E)
    x, w = _bf(rng.standard_normal((E, M, K))), _bf(rng.standard_normal((E, N, K)) * K ** -0.5)
    out = core.full((E * M, N), float("nan"), dtype)
    lib.call("kd_moe_linear", _r(_put(x.reshape(E * M, K), dtype)), _r(_put(w, dtype)), None, 0, F(0), _r(out))
    _close(_get(out).reshape(E, M, N), np.einsum("emk,enk->emn", x.astype(np.float64), w), 2e-6 if dtype == "float32" else 5e-3)


# ----------------------------------------------------------------------------- norm, rotation, cache rows
def _head_sizes(dtype, dim, vdim):
    a, b = ctypes.c_int(0), ctypes.c_int(0)
    lib.call("kd_attention_head_sizes", lib.DTYPES[dtype][0], dim, vdim, ctypes.byref(a), ctypes.byref(b))
    return a.value, b.value


@pytest.mark.parametrize("H, G, dim, vdim, rot", [(4, 2, 64, 64, 64), (6, 3, 128, 128, 32), (3, 1, 20, 28, 12), (2, 2, 48, 80, 48), (5, 5, 7, 9, 0), (4, 1, 96, 64, 96), (2, 1, 160, 40, 16),
                                                  (4, 4, 64, 64, 8)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_query_key_norm_rotation_and_cache_rows(backend, H, G, dim, vdim, rot, dtype):
    rng = _rng(H, G, dim, vdim, rot)
    B, S, pos, max_s, eps, base = 2, 3, 37, 45, 1e-4, 1000.0
    up = lambda n: (n + 7) // 8 * 8  # noqa: E731
    qc, kc, vc = 8, 8 + up(H * dim), 8 + up(H * dim) + up(G * dim)
    proj = _bf(rng.standard_normal((B, S, up(vc + G * vdim))) * 3)
    qw, kw = 1 + 0.4 * rng.standard_normal(H * dim), 1 + 0.4 * rng.standard_normal(G * dim)
    n2 = rot // 2
    a = np.arange(max_s)[:, None] * base ** (-2.0 * np.arange(n2) / max(rot, 1))[None, :]
    cos, sin = (_put(f(a)) if n2 else core.zeros((1,)) for f in (np.cos, np.sin))
    dq, dv = _head_sizes(dtype, dim, vdim)
    assert dq >= dim and dv >= vdim
    pd = proj.astype(np.float64)
    tol = 3e-6 if dtype == "float32" else 5e-3
    for dev in (False, True):
        for own in (True, False):
            keys, values = core.full((B + 1, G, max_s, dq), 7.0, dtype), core.full((B + 1, G, max_s, dv), 7.0, dtype)
            q = core.full((B, S, H, dq), float("nan"), dtype)
            where = Tensor(np.array([pos], np.int32)) if dev else None
            lib.call("kd_qk_norm_rope_cache", _r(_put(proj, dtype)), qc, kc if own else -1, vc if own else -1, dim, vdim, rot, _r(_put(qw)), _r(_put(kw)) if own else None,
                     F(eps), _r(cos), _r(sin), _r(keys), _r(values), _r(where), 0 if dev else pos, _r(q))
            q, keys, values = _get(q), _get(keys), _get(values)
            at = np.arange(pos, pos + S)
            for b in range(B):
                want = vogozen.rotate_half(hybrid.rms_norm(pd[b, :, qc:qc + H * dim], qw, eps).reshape(S, H, dim), at, base, rot)
                _close(q[b, :, :, :dim], want, tol, "queries")
                assert (q[b, :, :, dim:] == 0).all()
                if own:
                    want = vogozen.rotate_half(hybrid.rms_norm(pd[b, :, kc:kc + G * dim], kw, eps).reshape(S, G, dim), at, base, rot)
                    _close(keys[b, :, at, :dim], want, tol, "keys")
                    assert np.array_equal(values[b, :, at, :vdim], pd[b, :, vc:vc + G * vdim].reshape(S, G, vdim))
                    assert (keys[b, :, at, dim:] == 0).all() and (values[b, :, at, vdim:] == 0).all()
            rest = np.ones(max_s, bool)
            if own:
                rest[at] = False
            assert (keys[:B, :, rest] == 7).all() and (values[:B, :, rest] == 7).all() and (keys[B] == 7).all() and (values[B] == 7).all()


# ----------------------------------------------------------------------------- window attention
def _attend(q, k, v, scale, window, sink, pos):
    """Queries q [S, H, d] at positions pos .. over keys [pos + S, G, d]: exp(sink) joins every head's denominator."""
    S, H, _ = q.shape
    out = np.empty((S, H, v.shape[2]))
    for h in range(H):
        g = h // (H // k.shape[1])
        s = q[:, h] @ k[:, g].T * scale
        i, j = pos + np.arange(S)[:, None], np.arange(len(k))[None, :]
        s[(j > i) | (i - j >= window)] = -np.inf
        if sink is None:
            e = np.exp(s - s.max(1, keepdims=True))
            out[:, h] = e / e.sum(1, keepdims=True) @ v[:, g]
        else:
            out[:, h] = hybrid.sink_softmax(s, sink[h]) @ v[:, g]
    return out


def _window_case(B, S, H, G, d, pos, window, dtype, dv=None, scale=None, sink=0.0, edit=None, seed=0, extra=9):
    """Rows past the context hold large finite numbers, as memory of an earlier request may.  edit(q, k, v) plants what shows."""
    rng = _rng(B, S, H, G, d, pos, window, seed)
    dv = dv or d
    ctx = pos + S
    q, k, v = rng.standard_normal((B, S, H, d)), rng.standard_normal((B, ctx, G, d)), rng.standard_normal((B, ctx, G, dv))
    if edit:
        edit(q, k, v)
    q, k, v = _bf(q), _bf(k), _bf(v)
    scale = scale or d ** -0.5
    sinks = None if sink is None else np.full(H, sink) if np.isscalar(sink) else np.asarray(sink)
    ref = np.stack([_attend(q[b].astype(np.float64), k[b].astype(np.float64), v[b].astype(np.float64), scale, window or 1 << 30, sinks, pos) for b in range(B)])
    max_s = ctx + extra
    keys, values = np.full((B, G, max_s, d), 300.0, np.float32), np.full((B, G, max_s, dv), 300.0, np.float32)
    keys[:, :, :ctx], values[:, :, :ctx] = k.transpose(0, 2, 1, 3), v.transpose(0, 2, 1, 3)
    qd, kd, vd = _put(q, dtype), _put(keys, dtype), _put(values, dtype)
    for dev in ([False, True] if S == 1 else [False]):
        out = core.full((B * S, H * dv), float("nan"), dtype)
        lib.call("kd_window_attention", _r(qd), _r(kd), _r(vd), _r(_put(sinks)) if sinks is not None else None, F(scale), window,
                 _r(Tensor(np.array([pos], np.int32))) if dev else None, 0 if dev else pos, _r(out))
        err = np.abs(_get(out).reshape(ref.shape) - ref).max()
        assert err <= (1e-5 if dtype == "float32" else 1.2e-2) * max(1.0, np.abs(ref).max()), (dev, err)
    return ref


@pytest.mark.parametrize("H, G, d", [(4, 2, 64), (6, 2, 128), (2, 2, 64), (3, 3, 128), (20, 1, 64), (12, 1, 128)], ids=str)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 128, 136, 200, 0])
@pytest.mark.parametrize("dtype", DTYPES)
def test_one_token_at_tile_and_window_edges(backend, H, G, d, window, dtype):
    for pos in (0, 1, 62, 63, 64, 127, 128, 135, 199, 200, 263, 455):
        _window_case(2, 1, H, G, d, pos, window, dtype)


@pytest.mark.parametrize("H, G, d", [(4, 2, 64), (6, 2, 128), (2, 2, 64), (3, 3, 128)], ids=str)
@pytest.mark.parametrize("window", [1, 2, 17, 100, 127, 128, 129, 300, 0])
@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_at_tile_and_window_edges(backend, H, G, d, window, dtype):
    for pos, S in ((0, 2), (0, 130), (0, 400), (1, 127), (126, 3), (127, 2), (128, 257), (255, 128), (301, 64), (640, 5)):
        _window_case(1, S, H, G, d, pos, window, dtype)


@pytest.mark.parametrize("H, G, d, dv", [(2, 1, 160, 40), (3, 3, 24, 200), (4, 2, 256, 256), (6, 3, 48, 300)], ids=str)
@pytest.mark.parametrize("dtype", DTYPES)
def test_heads_that_only_the_cuda_cores_take(backend, H, G, d, dv, dtype):
    for pos, S, window in ((0, 1, 5), (50, 1, 20), (0, 45, 20), (33, 37, 64), (70, 3, 0)):
        _window_case(2, S, H, G, d, pos, window, dtype, dv=dv)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [64, 128])
@pytest.mark.parametrize("S", [1, 5, 140])
@pytest.mark.parametrize("window", [48, 129, 257, 500])
@pytest.mark.parametrize("behind", [-1, 0, 1])
def test_one_key_just_inside_and_just_outside_the_window(backend, dtype, d, S, window, behind):
    """For the last query of a portion the key window - 1 + behind tokens back would take all the weight."""
    pos = 700
    i = S - 1
    j = pos + i - (window - 1) - behind

    def edit(q, k, v):
        k[:, j, 0] = q[:, i, 0] * 6.0
        v[:, j, 0] = 5.0
    ref = _window_case(1, S, 2, 2, d, pos, window, dtype, edit=edit)
    assert (np.abs(ref[0, i, 0] - 5.0).max() < 0.1) == (behind <= 0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("far", [0, 1, 63, 64, 127, 128, 511, 899])
def test_one_far_key_among_hundreds(backend, dtype, far):
    def edit(q, k, v):
        k[:, far, 1] = q[:, -1, 2] * 6.0
        v[:, far, 1] = -4.0
    for S, pos in ((1, 900), (70, 831)):
        ref = _window_case(1, S, 4, 2, 64, pos, 901 - far, dtype, edit=edit)
        assert np.abs(ref[0, -1, 2] + 4.0).max() < 0.1


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_just_past_a_query_stays_unseen(backend, dtype):
    def edit(q, k, v):
        k[:, 65, 0] = q[:, 0, 0] * 6.0
        v[:, 65, 0] = 5.0
    ref = _window_case(1, 3, 2, 2, 64, 64, 30, dtype, edit=edit)
    assert np.abs(ref[0, 0, 0]).max() < 3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", [None, -50.0, 0.0, 12.0, 60.0, [0.0, 3.0, -2.0, 8.0]])
def test_sink_from_nothing_to_everything(backend, dtype, sink):
    for S, pos in ((1, 0), (1, 130), (1, 700), (2, 0), (150, 90)):
        _window_case(2, S, 4, 2, 64, pos, 100, dtype, sink=sink)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S, pos", [(1, 300), (140, 160)])
def test_scores_far_below_the_sink_give_almost_nothing(backend, dtype, S, pos):
    """Every score is about -30: without the sink the weights would sum to one."""
    def edit(q, k, v):
        q[..., 0], k[..., 0] = 16.0, -15.0
    ref = _window_case(1, S, 2, 1, 64, pos, 90, dtype, edit=edit)
    assert np.abs(ref).max() < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence(backend, dtype):
    """The first token sees itself and the sink, nothing of what the memory held before."""
    for S in (1, 2, 3, 129):
        ref = _window_case(3, S, 4, 2, 64, 0, 2, dtype)
        assert np.abs(ref[:, 0]).max() < 5


def test_window_attention_with_many_splits(backend):
    """One sequence, one key head: the window's tiles are spread over the whole GPU."""
    for pos in (4000, 4095, 4096):
        _window_case(1, 1, 8, 1, 128, pos, 3000, "bfloat16")


# ----------------------------------------------------------------------------- token shift
@pytest.mark.parametrize("width", [64, 50, 516])
@pytest.mark.parametrize("dtype", DTYPES)
def test_token_shift_over_portions(backend, width, dtype):
    rng = _rng(width)
    B, mixes = 3, 5
    mu = rng.uniform(-0.2, 1.2, (mixes, width)).astype(np.float32)
    for cuts in ([23], [1, 2, 3, 4, 5, 8], [1] * 5 + [18], [4, 4, 15]):
        h = _bf(rng.standard_normal((B, 23, width)))
        before = np.concatenate([np.zeros((B, 1, width)), h[:, :-1]], axis=1)
        want = h + (before - h) * mu[:, None, None].astype(np.float64)
        last, at = core.zeros((B + 1, width), dtype), 0
        for n in cuts:
            out = core.full((mixes, B * n, width), float("nan"), dtype)
            lib.call("kd_token_shift", _r(_put(h[:, at:at + n], dtype)), _r(_put(mu)), _r(last), _r(out))
            _close(_get(out).reshape(mixes, B, n, width), want[:, :, at:at + n], 1e-6 if dtype == "float32" else 5e-3, (cuts, at))
            at += n
        assert np.array_equal(_get(last)[:B], h[:, -1]) and (_get(last)[B] == 0).all()


# ----------------------------------------------------------------------------- WKV
def _wkv_case(B, S, H, dim, dtype, cuts, w_mean=-1.0, w_sd=1.0, seed=0):
    rng = _rng(B, S, H, dim, seed)
    n = H * dim
    r, k, v = (_bf(rng.standard_normal((B, S, n))) for _ in range(3))
    logits, w0 = (rng.standard_normal((B, S, n)) * w_sd).astype(np.float32), (rng.standard_normal(n) + w_mean).astype(np.float32)
    u, norm_w, gate = rng.standard_normal(n).astype(np.float32), rng.standard_normal(n).astype(np.float32), _bf(rng.standard_normal((B, S, n)))
    a, b = ctypes.c_int(0), ctypes.c_int(0)
    lib.call("kd_delta_state_shape", dim, dim, ctypes.byref(a), ctypes.byref(b))
    state = core.zeros((B, H, a.value, b.value))
    outs, fins, at = [], [], 0
    for m in cuts:
        part = lambda x: np.ascontiguousarray(x[:, at:at + m])  # noqa: E731
        o, y = core.full((B * m, n), float("nan")), core.full((B * m, n), float("nan"), dtype)
        lib.call("kd_wkv", _r(_put(part(r), dtype)), _r(_put(part(k), dtype)), _r(_put(part(v), dtype)), _r(_put(part(logits).reshape(B * m, n))), _r(_put(w0)), _r(_put(u)),
                 _r(state), _r(o))
        lib.call("kd_gated_head_norm", _r(o), _r(_put(part(gate).reshape(B * m, n), dtype)), _r(_put(norm_w)), H, F(1e-4), 1, _r(y))
        outs.append(_get(o).reshape(B, m, H, dim))
        fins.append(_get(y).reshape(B, m, n))
        at += m
    assert at == S
    got, fin, kept = np.concatenate(outs, 1), np.concatenate(fins, 1), _get(state)
    for i in range(B):
        heads = lambda x: x[i].astype(np.float64).reshape(S, H, dim)  # noqa: E731
        decay = np.exp(-np.exp((logits[i] + w0).astype(np.float64))).reshape(S, H, dim)
        o, s = vogozen.wkv(heads(r), heads(k), heads(v), decay, u.reshape(H, dim).astype(np.float64))
        _close(got[i], o, 3e-5, "outputs")
        _close(kept[i, :, :dim, :dim], s, 3e-5, "state")
        assert (kept[i, :, dim:] == 0).all() and (kept[i, :, :, dim:] == 0).all()
        want = hybrid.rms_norm(o, 1.0, 1e-4).reshape(S, n) * norm_w * vogozen.silu(gate[i].astype(np.float64))
        _close(fin[i], want, 1e-4 if dtype == "float32" else 1e-2, "norm and gate")


@pytest.mark.parametrize("H, dim", [(2, 16), (3, 64), (3, 20), (4, 128), (2, 130), (1, 256), (2, 33), (5, 48), (1, 7), (2, 96)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_wkv_sizes_and_portions(backend, H, dim, dtype):
    for cuts in ([37], [1, 2, 3, 16, 15], [1] * 5 + [32], [7, 9, 8, 13]):
        _wkv_case(2, 37, H, dim, dtype, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_wkv_long_sequences(backend, dtype):
    _wkv_case(1, 700, 2, 64, dtype, [400, 2, 298], w_mean=-6.0)
    _wkv_case(1, 300, 2, 48, dtype, [3] + [1] * 297, w_mean=-4.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("w_mean, w_sd", [(-12.0, 3.0), (1.0, 1.5), (3.0, 3.0), (30.0, 20.0)])
def test_wkv_decays_from_one_to_zero(backend, dtype, w_mean, w_sd):
    """Decays that keep the state, that wipe single channels, and that underflow to zero outright."""
    for cuts in ([50], [3, 4, 5, 38], [1] * 9 + [41]):
        _wkv_case(1, 50, 3, 40, dtype, cuts, w_mean, w_sd)


def test_wkv_many_heads_share_a_block(backend):
    _wkv_case(20, 19, 16, 64, "bfloat16", [18, 1])
    _wkv_case(12, 19, 32, 32, "float32", [2, 17])
    _wkv_case(10, 21, 32, 128, "bfloat16", [21])


def test_wkv_bonus_is_for_the_current_token_alone(backend):
    """One token writes, all read: the bonus shows in its own output and nowhere else."""
    S, dim = 6, 32
    r, k, v = np.ones((1, S, dim)), np.zeros((1, S, dim)), np.ones((1, S, dim))
    k[0, 2, 0] = 1.0
    state = core.zeros((1, 1, 32, 32))
    o = core.empty((S, dim))
    lib.call("kd_wkv", _r(_put(r)), _r(_put(k)), _r(_put(v)), _r(core.full((S, dim), -60.0)), _r(core.zeros((dim,))), _r(core.full((dim,), 7.0)), _r(state), _r(o))
    assert np.allclose(_get(o)[:, 0], [0, 0, 7, 1, 1, 1])


# ----------------------------------------------------------------------------- delta rule with a decay per head
def _head_delta_case(B, S, H, Hk, dim, vdim, taps, dtype, cuts, a_mean=-2.0, a_sd=1.0, rate_sd=1.0, seed=0):
    rng = _rng(B, S, H, dim, vdim, taps, seed)
    qk, vv = Hk * dim, H * vdim
    n = ((2 * qk + 2 * vv + H) + 23) // 8 * 8
    gc = (2 * qk + vv + 7) // 8 * 8
    bc = gc + vv
    proj = _bf(rng.standard_normal((B, S, n)))
    ld = (H + 7) // 8 * 8                                       # decay logits are columns of a wider matrix
    a = (rng.standard_normal((B, S, ld)) * a_sd).astype(np.float32)
    conv = [_bf(rng.standard_normal((rows, taps)) * 0.6 + 0.2) for rows in (qk, qk, vv)]
    rate, bias = np.exp(rng.standard_normal(H) * rate_sd).astype(np.float32), (rng.standard_normal(H) + a_mean).astype(np.float32)
    rows, cols = ctypes.c_int(0), ctypes.c_int(0)
    lib.call("kd_delta_state_shape", dim, vdim, ctypes.byref(rows), ctypes.byref(cols))
    state, hist = core.zeros((B, H, rows.value, cols.value)), core.zeros((B, max(taps - 1, 1), 2 * qk + vv), dtype)
    norm_w = rng.standard_normal(vdim).astype(np.float32)
    outs, fins, at = [], [], 0
    for m in cuts:
        pd = _put(proj[:, at:at + m], dtype)
        ad = _put(a[:, at:at + m].reshape(B * m, ld)).slice([slice(None), slice(0, H)])
        o, y = core.full((B * m, vv), float("nan")), core.full((B * m, vv), float("nan"), dtype)
        lib.call("kd_delta_rule", _r(pd), 0, qk, 2 * qk, bc, _r(ad), H, Hk, dim, vdim, *(_r(_put(x)) for x in conv), _r(_put(-rate)), _r(_put(bias)), _r(hist), _r(state), _r(o))
        gate = pd.view(B * m, n).slice([slice(None), slice(gc, gc + vv)])
        lib.call("kd_delta_out", _r(o), _r(gate), _r(_put(norm_w)), F(1e-5), 1, _r(pd), 0, taps, _r(hist), _r(y))
        outs.append(_get(o).reshape(B, m, H, vdim))
        fins.append(_get(y).reshape(B, m, H, vdim))
        at += m
    assert at == S
    got, fin, kept = np.concatenate(outs, 1), np.concatenate(fins, 1), _get(state)
    for b in range(B):
        p = proj[b].astype(np.float64)
        q, k, v = (hybrid.causal_conv_silu(p[:, i:i + len(w)], w.astype(np.float64)) for i, w in zip((0, qk, 2 * qk), conv))
        rep = H // Hk
        q = np.repeat(hybrid.unit(q.reshape(S, Hk, dim)) * dim ** -0.5, rep, 1)
        k = np.repeat(hybrid.unit(k.reshape(S, Hk, dim)), rep, 1)
        g = np.exp(-rate.astype(np.float64) * hybrid.softplus((a[b, :, :H] + bias).astype(np.float64)))
        o, s = hybrid.delta_rule(q, k, v.reshape(S, H, vdim), np.repeat(g[:, :, None], dim, 2), hybrid.sigmoid(p[:, bc:bc + H]))
        _close(got[b], o, 3e-5, "outputs")
        _close(kept[b, :, :dim, :vdim], s, 3e-5, "state")
        want = hybrid.rms_norm(o, norm_w, 1e-5) * vogozen.silu(p[:, gc:gc + vv]).reshape(S, H, vdim)
        _close(fin[b], want, 1e-4 if dtype == "float32" else 1e-2, "norm and gate")


@pytest.mark.parametrize("size", [(2, 1, 16, 8, 4), (3, 3, 64, 64, 4), (3, 3, 20, 36, 3), (4, 2, 128, 128, 4), (2, 2, 130, 40, 4), (1, 1, 256, 128, 2), (2, 1, 33, 65, 1), (2, 2, 32, 300, 4),
                                  (6, 2, 48, 24, 8), (1, 1, 9, 7, 5), (2, 1, 1, 8, 2)], ids=str)
@pytest.mark.parametrize("dtype", DTYPES)
def test_head_decay_delta_rule_sizes_and_portions(backend, size, dtype):
    for cuts in ([37], [1, 2, 3, 16, 15], [1] * 5 + [32]):
        _head_delta_case(2, 37, *size, dtype, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("a_mean, a_sd, rate_sd", [(-12.0, 3.0, 0.5), (3.0, 4.0, 1.5), (8.0, 12.0, 2.0), (60.0, 30.0, 1.0)])
def test_head_decays_from_one_to_zero(backend, dtype, a_mean, a_sd, rate_sd):
    for cuts in ([50], [3, 4, 5, 38]):
        _head_delta_case(1, 50, 3, 3, 40, 24, 4, dtype, cuts, a_mean, a_sd, rate_sd)


def test_head_decay_delta_rule_long_and_wide(backend):
    _head_delta_case(1, 700, 2, 2, 64, 32, 4, "bfloat16", [400, 2, 298], a_mean=-5.0)
    _head_delta_case(20, 19, 16, 8, 64, 64, 4, "bfloat16", [18, 1])
    _head_delta_case(12, 19, 32, 16, 32, 32, 4, "float32", [2, 17])
