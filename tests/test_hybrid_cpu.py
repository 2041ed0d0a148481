"""CPU tests of the Pedorax design: configuration and registry, and the plain implementation itself against
independent formulations."""
import json

import numpy as np
import pytest

from oracle import hybrid
from tests import hybrid_cases as hc


def _parse(cfg):
    from kandle_b200.model_utils.pedorax import PedoraxConfig
    return PedoraxConfig.fromDict(cfg)


def test_config_reads_every_size():
    c = _parse(hc.mixed_config(embed=1.5, logit=0.25, eps=3e-6))
    assert (c.vocabSize, c.hiddenSize, c.embeddingScale, c.logitScale, c.normEps) == (150, 72, 1.5, 0.25, 3e-6)
    m = c.layers[2].mixer
    assert (m.heads, m.dim, m.rotDim, m.vdim, m.kvRank, m.scale, m.rotBase, m.kvFrom) == (2, 16, 16, 56, 48, 0.3, 5000.0, 0)
    assert c.layers[2].experts is None
    e = c.layers[1].experts
    assert (e.experts, e.top, e.groups, e.keep, e.ff, e.limit) == (8, 2, 8, 3, 40, 1.2)
    d = c.layers[3].mixer
    assert (d.heads, d.kvHeads, d.dim, d.vdim, d.taps, d.channels) == (3, 3, 20, 36, 3, 2 * 60 + 108)


@pytest.mark.parametrize("layers, text", [
    ([(hc.latent(kv_from=0), None)], "kv_from"),
    ([(hc.delta(), None), (hc.latent(kv_from=0), None)], "kv_from"),
    ([(hc.latent(), None), (hc.latent(rank=32, kv_from=0), None)], "differ"),
    ([(hc.latent(), None), (hc.latent(kv_from=0), None), (hc.latent(kv_from=1), None)], "kv_from"),
    ([(hc.delta(heads=3, kv_heads=2), None)], "key heads"),
    ([(hc.delta(), hc.moe(experts=10, groups=4))], "experts"),
    ([(hc.delta(), hc.moe(top=7, keep=2))], "top 7"),
])
def test_config_rejects_what_cannot_run(layers, text):
    with pytest.raises(ValueError, match=text):
        _parse(hc.config(layers))


def test_config_rejects_unknown_kinds():
    cfg = hc.config([(hc.latent(), None)])
    cfg["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        _parse(cfg)
    cfg = hc.config([(hc.latent(), {"kind": "dense"})])
    with pytest.raises(ValueError, match="unknown feed-forward"):
        _parse(cfg)


def test_registry_chooses_by_config():
    from kandle_b200 import registry
    assert {"Pedorax", "Qwen3ForCausalLM"} <= set(registry.architectures())
    assert registry.lookup({"architecture": "Pedorax"}).dtypes == ("bfloat16", "float32")
    q = registry.lookup({"architectures": ["Qwen3ForCausalLM"]})
    assert q.dtypes == ("bfloat16",)
    c = q.config({"vocab_size": 10, "hidden_size": 64, "intermediate_size": 96, "num_hidden_layers": 2, "num_attention_heads": 4,
                  "num_key_value_heads": 2, "head_dim": 32}, "bfloat16")
    assert (c.vocabSize, c.headDim, c.numKeyValueHeads) == (10, 32, 2)
    with pytest.raises(ValueError, match="known"):
        registry.lookup({"architecture": "Nothing"})
    with pytest.raises(ValueError, match="no architecture"):
        registry.lookup({})


def test_replay_takes_one_request_after_the_other(tmp_path):
    from kandle_b200 import trace

    class Fake:
        def __init__(self):
            self.log = []

        def reset(self):
            self.log.append("reset")

        def extend(self, ids, want):
            self.log.append((ids.tolist(), list(want)))

            class T:
                def dataAsync(self):
                    return np.arange(len(want) * 3, dtype=np.float32).reshape(-1, 3)
            return T()
    e, said = Fake(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [3], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [4], "want": [0]}], "end": ["b"]}]
    trace.replay(e, [json.dumps(s) for s in steps] + ["\n"], str(tmp_path), said.append)
    assert e.log == ["reset", ([[1, 2]], [1]), ([[3]], []), "reset", ([[4]], [0])]
    assert said == ["done 0", "done 1", "done 2"]
    assert sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "2.f32"]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [0.0, 1.0, 2.0]
    with pytest.raises(ValueError, match="before"):
        trace.replay(Fake(), [json.dumps(steps[0]), json.dumps(steps[2])], str(tmp_path), said.append)


# ----------------------------------------------------------------------------- the plain implementation
def test_sink_counts_once_in_the_denominator():
    s, sink = np.random.default_rng(0).standard_normal((4, 6)), 0.7
    padded = np.concatenate([s, np.full((4, 1), sink)], axis=1)
    want = np.exp(padded) / np.exp(padded).sum(1, keepdims=True)
    assert np.allclose(hybrid.sink_softmax(s, sink), want[:, :6])


def test_rotation_is_relative():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    dot = lambda a, b: float(hybrid.rotate_interleaved(q, [a], 100.0, 8)[0] @ hybrid.rotate_interleaved(k, [b], 100.0, 8)[0])  # noqa: E731
    assert np.isclose(dot(5, 2), dot(13, 10)) and not np.isclose(dot(5, 2), dot(5, 3))
    assert np.allclose(hybrid.rotate_interleaved(q, [3], 100.0, 4)[0, 4:], q[0, 4:])


def test_delta_rule_without_decay_solves_exact_recall():
    """beta 1, no decay, orthonormal keys: the state stores every value; reading with a key returns its value."""
    k = np.eye(4)[:, None, :]
    v = np.random.default_rng(0).standard_normal((4, 1, 3))
    one = np.ones((4, 1, 4))
    _, s = hybrid.delta_rule(k, k, v, one, np.ones((4, 1)))
    assert np.allclose(s[0], v[:, 0])
    # a second write under the same key replaces the value
    o, _ = hybrid.delta_rule(k[:1], k[:1], 2 * v[:1], one[:1], np.ones((1, 1)), s)
    assert np.allclose(o[0, 0], 2 * v[0, 0])


def test_delta_rule_carries_state():
    rng = np.random.default_rng(0)
    q, k, g = rng.standard_normal((3, 9, 2, 5))
    g, v, b = np.exp(-np.abs(g)), rng.standard_normal((9, 2, 4)), rng.uniform(size=(9, 2))
    whole, s = hybrid.delta_rule(q, k, v, g, b)
    a, s1 = hybrid.delta_rule(q[:4], k[:4], v[:4], g[:4], b[:4])
    c, s2 = hybrid.delta_rule(q[4:], k[4:], v[4:], g[4:], b[4:], s1)
    assert np.allclose(np.concatenate([a, c]), whole) and np.allclose(s, s2)


def test_routing_against_enumeration():
    rng = np.random.default_rng(0)
    r = {"experts": 12, "top": 3, "groups": {"count": 4, "keep": 2}}
    h, router = rng.standard_normal((50, 8)), rng.standard_normal((12, 8))
    chosen, w = hybrid.route(h, router, r)
    s = hybrid.sigmoid(h @ router.T)
    for t in range(50):
        score = [sum(sorted(s[t, g * 3:g * 3 + 3])[-2:]) for g in range(4)]
        best = sorted(range(4), key=lambda g: -score[g])[:2]
        allowed = [e for e in range(12) if e // 3 in best]
        want = sorted(allowed, key=lambda e: -s[t, e])[:3]
        assert chosen[t].tolist() == want
        assert np.allclose(w[t], s[t, want] / s[t, want].sum())


def test_convolution_sees_only_the_past():
    x = np.zeros((6, 1))
    x[2] = 1.0
    y = hybrid.causal_conv_silu(x, np.array([[1.0, 2.0, 3.0]]))
    z = np.array([0, 0, 3.0, 2.0, 1.0, 0])[:, None]
    assert np.allclose(y, z * hybrid.sigmoid(z))
