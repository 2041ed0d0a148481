"""The hybrid engine on the Vogozen design against the plain implementation: whole prompts, portions, decoding, batches,
reused sequences, generation, checkpoints.  fp32 runs are compared at every position; they are what shows a wrong key,
state or schedule.  bf16 runs exercise the tensor-core kernels (tests/test_vogozen_kernels_gpu.py compares those one by
one)."""
import ctypes
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from kandle_b200 import io, lib
from oracle import vogozen
from tests import hybrid_cases as hc
from tests import vogozen_cases as vc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _assert_close(got, ref, dtype, what="", f32=1e-4):
    """The norms on small sublayer outputs (a first token's recurrence, say) enlarge rounding, in bf16 the operands', so single
    positions may be off by more; a wrong key or state shows at most positions that see it, by far more."""
    e = hc.row_errors(got, ref)
    worst = f"{what}: worst position {np.unravel_index(e.argmax(), e.shape)} error {e.max():.2e}, median {np.median(e):.2e}"
    if dtype == "float32":
        assert e.max() <= f32 and np.median(e) <= 5e-6, worst
    else:
        assert np.median(e) <= 2.5e-2 and (e > 8e-2).mean() <= 0.05 and e.max() <= 0.5, worst


@pytest.fixture(scope="module")
def mixed():
    cfg = vc.mixed_config()
    w = vc.weights(cfg, sharp=1.2)
    ids = hc.tokens(cfg, 2, 150)
    return cfg, w, ids, hc.reference(cfg, w, ids)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cuts", [[150], [118, 1], [64, 64], [2], [3, 37, 2, 5, 40, 63], [10, 1, 1, 11, 1, 12, 2, 1], [1]], ids=str)
def test_prompts_portions_and_decoding(backend, mixed, dtype, cuts):
    cfg, w, ids, ref = mixed
    eng = hc.engine(cfg, w, 1, 150, dtype)
    _assert_close(hc.run_cut(eng, ids[:1], cuts), ref[:1], dtype, f"cuts {cuts}")
    eng.dispose()


def test_residual_stream_layer_by_layer(backend, mixed):
    cfg, w, ids, _ = mixed
    eng = hc.engine(cfg, w, 1, 64)
    eng.trace, layers = [], []
    eng.extend(ids[:1, :43], [])
    vogozen.forward(cfg, w, ids[0, :43], layers=layers)
    assert len(eng.trace) == len(layers) == 7
    for i, (a, b) in enumerate(zip(eng.trace, layers)):
        assert np.abs(a.reshape(b.shape) - b).max() <= 2e-5 * np.abs(b).max(), f"layer {i}"
    eng.dispose()


def test_sequences_of_a_batch_do_not_meet(backend, mixed):
    cfg, w, ids, ref = mixed
    for dtype in ("float32", "bfloat16"):
        eng = hc.engine(cfg, w, 3, 150, dtype)
        _assert_close(hc.run_cut(eng, ids, [40, 7, 60, 1]), ref, dtype, "batch of two in an engine for three")
        _assert_close(hc.run_cut(eng, ids[1:], [150]), ref[1:], dtype, "then one alone")
        eng.dispose()


def _poison(eng):
    """States become NaN; cache rows, whose stale contents must be finite, something large."""
    for kept in eng.cache._own:
        for t, value in [(t, float("nan")) for t in kept.carried()] + ([(kept.keys, 200.0), (kept.values, -200.0)] if hasattr(kept, "keys") else []):
            lib.call("kd_fill", ctypes.byref(t._handle.c()), ctypes.c_double(value))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_freed_memory_is_used_again(backend, mixed, dtype):
    """Everything the caches hold is overwritten between two requests: the reset must clear the recurrent state and the
    second request must weigh no row it has not written.  A used engine computes what a fresh one does."""
    cfg, w, ids, ref = mixed
    used, fresh = hc.engine(cfg, w, 1, 150, dtype), hc.engine(cfg, w, 1, 150, dtype)
    hc.run_cut(used, ids[:1], [149, 1])
    for row, want, cuts in ((ids[1:, :67], ref[1:, :67], [30, 5, 1]), (ids[:1, :1], ref[:1, :1], [1]), (ids[:1, :90], ref[:1, :90], [64, 2, 24])):
        _poison(used)
        got = hc.run_cut(used, row, cuts)
        assert np.array_equal(got, hc.run_cut(fresh, row, cuts)), cuts
        _assert_close(got, want, dtype, cuts)
        fresh.dispose()
        fresh = hc.engine(cfg, w, 1, 150, dtype)
    used.dispose()
    fresh.dispose()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(backend, mixed, dtype):
    """A short prompt, then every token alone: windows pass over decoded tokens, states are carried over hundreds of steps."""
    cfg, w, _, _ = mixed
    ids = hc.tokens(cfg, 1, 400, seed=9)
    eng = hc.engine(cfg, w, 1, 400, dtype)
    _assert_close(hc.run_cut(eng, ids, [5, 1]), hc.reference(cfg, w, ids), dtype)
    eng.dispose()


OTHER = [
    ("wide odd", [(vc.attention(heads=1, kv_heads=1, dim=7, vdim=5, rot=2, window=3), vc.dense(17)), (vc.wkv(heads=1, dim=9), None),
                  (vc.delta(heads=1, kv_heads=1, dim=9, vdim=7, conv=2), vc.dense(5))], dict(width=50, vocab=33)),
    ("single tap, unrotated", [(vc.delta(heads=2, kv_heads=1, dim=33, vdim=65, conv=1), None), (vc.attention(rot=0), vc.dense())], {}),
    ("six taps, wide heads", [(vc.delta(heads=6, kv_heads=2, dim=130, vdim=40, conv=6), vc.dense()), (vc.wkv(heads=1, dim=200), None),
                              (vc.attention(heads=2, kv_heads=1, dim=160, vdim=136, rot=160, window=20), vc.dense())], {}),
    ("aligned", [(vc.attention(heads=8, kv_heads=2, dim=64, vdim=64, rot=64, window=33), vc.dense(256)), (vc.wkv(heads=2, dim=64), vc.dense(128)),
                 (vc.delta(heads=6, kv_heads=3, dim=64, vdim=64), vc.dense(64)), (vc.attention(heads=3, kv_heads=3, dim=128, vdim=96, rot=32, window=64), vc.dense(256))],
     dict(width=128, vocab=256)),
    ("only windows of one", [(vc.attention(window=1), vc.dense()), (vc.attention(window=1, kv_from=0), None)], {}),
    ("window past the end", [(vc.attention(window=5000), vc.dense()), (vc.attention(window=2, kv_from=0), None)], {}),
    ("rows of others", [(vc.attention(), None), (vc.attention(window=30), None), (vc.attention(window=19, scale=1.1, kv_from=0), vc.dense()),
                        (vc.attention(window=8, kv_from=1), None), (vc.attention(window=75, kv_from=0), None)], {}),
    ("many query heads a key head", [(vc.attention(heads=20, kv_heads=1, dim=32, vdim=32, rot=32), vc.dense())], {}),
    ("only recurrences", [(vc.wkv(heads=4, dim=32), vc.dense()), (vc.wkv(heads=1, dim=24), vc.dense()), (vc.delta(), vc.dense())], dict(eps=1e-2)),
]


@pytest.mark.parametrize("name, layers, kw", OTHER, ids=[o[0] for o in OTHER])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(backend, name, layers, kw, dtype):
    cfg = vc.config(layers, **kw)
    w = vc.weights(cfg, seed=3, sharp=1.5)
    ids = hc.tokens(cfg, 1, 75, seed=4)
    eng = hc.engine(cfg, w, 1, 80, dtype)
    ref = hc.reference(cfg, w, ids)
    for cuts in ([75], [2, 31, 1]):
        # (tiny heads: norms of a few small numbers, where fp32's own rounding is enlarged too)
        _assert_close(hc.run_cut(eng, ids, cuts), ref, dtype, f"{name} {cuts}", f32=3e-4 if name == "wide odd" else 1e-4)
    eng.dispose()


@pytest.mark.parametrize("dim", [64, 128])
@pytest.mark.parametrize("window", [100, 128, 200])
def test_long_prompts_through_the_tensor_core_kernels(backend, dim, window):
    cfg = vc.config([(vc.attention(heads=4, kv_heads=2, dim=dim, vdim=dim, rot=dim, window=window), vc.dense()),
                     (vc.attention(heads=4, kv_heads=2, dim=dim, vdim=dim, rot=dim, window=window // 2 + 1, kv_from=0), None)], width=128)
    w = vc.weights(cfg, seed=5, sharp=1.5)
    ids = hc.tokens(cfg, 2, 390)
    ref = hc.reference(cfg, w, ids)
    eng = hc.engine(cfg, w, 2, 400, "bfloat16")
    for cuts in ([390], [130, 128, 70, 62], [64, 1, 100, 225], [7, 2, 300, 1]):
        _assert_close(hc.run_cut(eng, ids, cuts), ref, "bfloat16", cuts)
    eng.dispose()


@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation(backend, mixed, graph):
    cfg, w, ids, _ = mixed
    eng = hc.engine(cfg, w, 2, 64)
    got = eng.generate(ids[:, :20], 12, use_graph=graph)
    want = np.array([vogozen.greedy(cfg, w, row, 12) for row in ids[:, :20]])
    assert np.array_equal(got, want)
    # again in the same engine (captured step kept), and in portions
    assert np.array_equal(eng.generate(ids[:, :20], 12, use_graph=graph), want)
    tok = eng.prefill(ids[:, :20], portion=7)
    assert np.array_equal(tok.dataAsync(), want[:, 0])
    eng.dispose()


def test_sampled_generation_at_low_temperature_is_greedy(backend, mixed):
    cfg, w, ids, _ = mixed
    eng = hc.engine(cfg, w, 1, 64)
    want = eng.generate(ids[:1, :20], 8)
    eng.set_sampler(temperature=1e-4, top_k=5, seed=3)
    assert np.array_equal(eng.generate(ids[:1, :20], 8), want)
    eng.set_sampler(temperature=5.0, seed=3)
    assert not np.array_equal(eng.generate(ids[:1, :20], 8), want)
    eng.dispose()


def test_engine_reports_misuse(backend, mixed):
    cfg, w, ids, _ = mixed
    eng = hc.engine(cfg, w, 1, 16)
    with pytest.raises(ValueError, match="overflow"):
        eng.extend(ids[:1, :17])
    eng.extend(ids[:1, :16])
    with pytest.raises(ValueError, match="overflow"):
        eng.extend(ids[:1, :1])
    eng.reset()
    eng.extend(np.array([[cfg["vocab"]]], np.int32))
    with pytest.raises(lib.KandleCudaError, match="101"):
        backend.synchronize()
    eng.dispose()
    short = dict(w)
    short["l1.mix.w0"] = w["l1.mix.w0"][:-1]
    with pytest.raises(ValueError, match="l1.mix.w0"):
        hc.engine(cfg, short, 1, 16)


def _checkpoint(folder, cfg, w):
    (folder / "config.json").write_text(json.dumps(cfg))
    io.save_file({k: (lib.f32_to_bf16_bits(v).reshape(np.shape(v)), "BF16") for k, v in w.items()}, str(folder / "model.safetensors"))


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_program_on_a_checkpoint(backend, mixed, tmp_path, dtype):
    cfg, w, ids, ref = mixed
    model, out = tmp_path / "m", tmp_path / "o"
    model.mkdir()
    out.mkdir()
    _checkpoint(model, cfg, w)
    steps, at = [], {"a": 0, "b": 0}
    for name, n, last in (("a", 31, 0), ("a", 2, 0), ("a", 1, 1), ("b", 40, 0), ("b", 1, 1)):
        row = ids[0] if name == "a" else ids[1]
        steps.append({"step": len(steps), "entries": [{"id": name, "tokens": row[at[name]:at[name] + n].tolist(), "want": [0, n - 1]}], "end": [name] if last else []})
        at[name] += n
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out), "--max-tokens", "41"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(5)]
    at = {"a": 0, "b": 0}
    for s in steps:
        e = s["entries"][0]
        got = np.fromfile(out / f"{s['step']}.f32", "<f4").reshape(2, cfg["vocab"])
        want = ref[0 if e["id"] == "a" else 1][[at[e["id"]] + p for p in e["want"]]]
        _assert_close(got, want, dtype, s["step"])
        at[e["id"]] += len(e["tokens"])


def test_command_line_generates(backend, mixed, tmp_path):
    cfg, w, ids, _ = mixed
    _checkpoint(tmp_path, cfg, w)
    r = subprocess.run([sys.executable, "-m", "kandle_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--steps", "6",
                        "--prompt", " ".join(map(str, ids[0, :20]))], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(x) for x in r.stdout.split()] == vogozen.greedy(cfg, w, ids[0, :20], 6)
