"""CPU tests of the Vogozen design: configuration and registry, and the plain implementation itself against
independent formulations."""
import numpy as np
import pytest

from oracle import vogozen
from tests import vogozen_cases as vc


def _parse(cfg):
    from kandle_b200.model_utils.vogozen import VogozenConfig
    return VogozenConfig.fromDict(cfg)


def test_config_reads_every_size():
    c = _parse(vc.mixed_config(eps=3e-6, vocab=99, width=56))
    assert (c.vocabSize, c.hiddenSize, c.normEps, len(c.layers)) == (99, 56, 3e-6, 7)
    m = c.layers[3].mixer
    assert (m.heads, m.kvHeads, m.dim, m.vdim, m.scale, m.rotBase, m.rotDims, m.window, m.kvFrom) == (4, 2, 20, 28, 0.4, 3000.0, 12, 40, 0)
    assert c.layers[3].dense is None and c.layers[2].dense.ff == 33
    d = c.layers[6].mixer
    assert (d.heads, d.kvHeads, d.dim, d.vdim, d.taps, d.channels) == (3, 1, 20, 36, 3, 2 * 20 + 108)
    assert (c.layers[4].mixer.heads, c.layers[4].mixer.dim) == (2, 40)


@pytest.mark.parametrize("layers, text", [
    ([(vc.attention(kv_from=0), None)], "kv_from"),
    ([(vc.wkv(), None), (vc.attention(kv_from=0), None)], "kv_from"),
    ([(vc.attention(), None), (vc.attention(kv_from=0), None), (vc.attention(kv_from=1), None)], "kv_from"),
    ([(vc.attention(), None), (vc.attention(dim=24, kv_from=0), None)], "differ"),
    ([(vc.attention(), None), (vc.attention(heads=4, kv_heads=4, kv_from=0), None)], "differ"),
    ([(vc.attention(heads=3, kv_heads=2), None)], "key heads"),
    ([(vc.delta(heads=3, kv_heads=2), None)], "key heads"),
    ([(vc.attention(rot=13), None)], "rotated"),
    ([(vc.attention(rot=22), None)], "rotated"),
    ([(vc.attention(window=0), None)], "window"),
    ([], "no layers"),
])
def test_config_rejects_what_cannot_run(layers, text):
    with pytest.raises(ValueError, match=text):
        _parse(vc.config(layers))


def test_config_rejects_unknown_kinds():
    cfg = vc.config([(vc.wkv(), None)])
    cfg["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        _parse(cfg)
    with pytest.raises(ValueError, match="unknown feed-forward"):
        _parse(vc.config([(vc.wkv(), {"kind": "moe"})]))


def test_registry_chooses_by_config():
    from kandle_b200 import registry
    entry = registry.lookup({"architecture": "Vogozen"})
    assert entry.dtypes == ("bfloat16", "float32")
    c = entry.config(vc.mixed_config(), "float32")
    assert type(c).__name__ == "VogozenConfig" and c.dtype == "float32"


# ----------------------------------------------------------------------------- the plain implementation
def test_quiet_softmax_has_a_silent_extra_score():
    s = np.random.default_rng(0).standard_normal((4, 6))
    e = np.exp(np.concatenate([s, np.zeros((4, 1))], axis=1))
    assert np.allclose(vogozen.quiet_softmax(s), (e / e.sum(1, keepdims=True))[:, :6])
    assert np.allclose(vogozen.quiet_softmax(s - 1000.0), 0.0) and np.allclose(vogozen.quiet_softmax(s + 1000.0).sum(1), 1.0)


def test_window_holds_exactly_its_keys():
    """Zero queries weigh every visible key alike, so the outputs count them."""
    T, size = 9, 4
    q, k, v = np.zeros((T, 2, 3)), np.ones((T, 1, 3)), np.ones((T, 1, 1))
    o = vogozen.window_attention(q, k, v, 1.0, size)
    n = np.minimum(np.arange(T) + 1, size)
    assert np.allclose(o[:, :, 0], (n / (n + 1.0))[:, None])


def test_query_heads_share_key_heads_in_order():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((5, 4, 3)), rng.standard_normal((5, 2, 3)), rng.standard_normal((5, 2, 3))
    o = vogozen.window_attention(q, k, v, 0.7, 5)
    for h, g in ((0, 0), (1, 0), (2, 1), (3, 1)):
        assert np.allclose(o[:, h], vogozen.window_attention(q[:, h:h + 1], k[:, g:g + 1], v[:, g:g + 1], 0.7, 5)[:, 0])


def test_rotation_is_relative_and_pairs_halves():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    dot = lambda a, b: float(vogozen.rotate_half(q, [a], 50.0, 8)[0, 0] @ vogozen.rotate_half(k, [b], 50.0, 8)[0, 0])  # noqa: E731
    assert np.isclose(dot(5, 2), dot(13, 10)) and not np.isclose(dot(5, 2), dot(5, 3))
    y = vogozen.rotate_half(q, [3], 50.0, 8)[0, 0]
    assert np.allclose(y[8:], q[0, 0, 8:])
    for i in range(4):
        z = (q[0, 0, i] + 1j * q[0, 0, i + 4]) * np.exp(3j * 50.0 ** (-2 * i / 8))
        assert np.allclose([y[i], y[i + 4]], [z.real, z.imag])


def test_wkv_equals_its_explicit_sum():
    """o_t = sum over s < t of (r_t . (decays between s and t) k_s) v_s + (r_t . u k_t) v_t."""
    rng = np.random.default_rng(0)
    T, H, d = 7, 2, 5
    r, k, v = rng.standard_normal((3, T, H, d))
    decay, u = rng.uniform(0.1, 1.0, (T, H, d)), rng.standard_normal((H, d))
    o, state = vogozen.wkv(r, k, v, decay, u)
    for t in range(T):
        want = (r[t] * u * k[t]).sum(-1, keepdims=True) * v[t]
        for s in range(t):
            want = want + (r[t] * decay[s + 1:t].prod(0) * k[s]).sum(-1, keepdims=True) * v[s]
        assert np.allclose(o[t], want)
    want = sum(decay[s + 1:].prod(0)[:, :, None] * k[s][:, :, None] * v[s][:, None] for s in range(T))
    assert np.allclose(state, want)


def test_shift_brings_the_previous_token():
    h = np.arange(6.0).reshape(3, 2)
    assert np.array_equal(vogozen.shifted(h), [[0, 0], [0, 1], [2, 3]])


def test_first_tokens_do_not_depend_on_later_ones():
    cfg = vc.mixed_config()
    w = vc.weights(cfg)
    ids = np.random.default_rng(3).integers(0, cfg["vocab"], 30)
    whole, part = vogozen.forward(cfg, w, ids), vogozen.forward(cfg, w, ids[:17])
    assert np.allclose(whole[:17], part)
