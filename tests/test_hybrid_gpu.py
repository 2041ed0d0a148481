"""The hybrid engine (Pedorax) against the plain implementation: whole prompts, portions, decoding, batches,
reused sequences, generation, checkpoints.  fp32 runs are compared at every position; they are what shows a
wrong key, state or schedule.  bf16 runs exercise the tensor-core kernels (tests/test_hybrid_kernels_gpu.py
compares those one by one); a close routing call may flip there, so a few positions may differ."""
import ctypes
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from kandle_b200 import io, lib
from oracle import hybrid
from tests import hybrid_cases as hc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = 2e-5


def _assert_f32(got, ref, what=""):
    e = hc.row_errors(got, ref)
    assert e.max() <= F32, f"{what}: worst position {np.unravel_index(e.argmax(), e.shape)} error {e.max():.2e}"


def _assert_bf16(got, ref, what=""):
    e = hc.row_errors(got, ref)
    assert np.median(e) <= 1.5e-2 and (e > 4e-2).mean() <= 0.05, f"{what}: median {np.median(e):.2e}, {(e > 4e-2).mean():.1%} of positions off, worst {e.max():.2e}"


@pytest.fixture(scope="module")
def mixed():
    cfg = hc.mixed_config()
    w = hc.weights(cfg, sharp=3.0)
    ids = hc.tokens(cfg, 2, 150)
    return cfg, w, ids, hc.reference(cfg, w, ids)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cuts", [[150], [118, 1], [64, 64], [2], [3, 37, 2, 5, 40, 63], [1]], ids=str)
def test_prompts_portions_and_decoding(backend, mixed, dtype, cuts):
    cfg, w, ids, ref = mixed
    eng = hc.engine(cfg, w, 1, 150, dtype)
    got = hc.run_cut(eng, ids[:1], cuts)
    (_assert_f32 if dtype == "float32" else _assert_bf16)(got, ref[:1], f"cuts {cuts}")
    eng.dispose()


def test_residual_stream_layer_by_layer(backend, mixed):
    cfg, w, ids, _ = mixed
    eng = hc.engine(cfg, w, 1, 64)
    eng.trace, layers = [], []
    eng.extend(ids[:1, :23], [])
    hybrid.forward(cfg, w, ids[0, :23], layers=layers)
    assert len(eng.trace) == len(layers) == 5
    for i, (a, b) in enumerate(zip(eng.trace, layers)):
        assert np.abs(a.reshape(b.shape) - b).max() <= 2e-5 * np.abs(b).max(), f"layer {i}"
    eng.dispose()


def test_sequences_of_a_batch_do_not_meet(backend, mixed):
    cfg, w, ids, ref = mixed
    eng = hc.engine(cfg, w, 3, 150)
    _assert_f32(hc.run_cut(eng, ids, [40, 7, 60, 1]), ref, "batch of two in an engine for three")
    _assert_f32(hc.run_cut(eng, ids[1:], [150]), ref[1:], "then one alone")
    eng.dispose()


def _poison(eng):
    for kept in eng.cache._own:
        for t in ([kept.rows] if hasattr(kept, "rows") else kept.carried()):
            lib.call("kd_fill", ctypes.byref(t._handle.c()), ctypes.c_double(float("nan")))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_freed_memory_is_used_again(backend, mixed, dtype):
    """Everything the caches hold is overwritten with NaN between two requests: the reset must clear the recurrent state
    and the second request must read no row it has not written.  A used engine computes what a fresh one does."""
    cfg, w, ids, ref = mixed
    used, fresh = hc.engine(cfg, w, 1, 150, dtype), hc.engine(cfg, w, 1, 150, dtype)
    hc.run_cut(used, ids[:1], [149, 1])
    for row, cuts in ((ids[1:, :67], [30, 5, 1]), (ids[:1, :1], [1]), (ids[:1, :90], [64, 2, 24])):
        _poison(used)
        got = hc.run_cut(used, row, cuts)
        _poison(fresh)
        assert np.array_equal(got, hc.run_cut(fresh, row, cuts)), cuts
        if dtype == "float32":
            _assert_f32(got, ref[1:, :67] if len(row[0]) == 67 else ref[:1, :row.shape[1]])
        fresh.dispose()
        fresh = hc.engine(cfg, w, 1, 150, dtype)
    used.dispose()
    fresh.dispose()


def test_long_decoding(backend, mixed):
    """A short prompt, then every token alone: states and rows carried over hundreds of steps."""
    cfg, w, _, _ = mixed
    ids = hc.tokens(cfg, 1, 400, seed=9)
    eng = hc.engine(cfg, w, 1, 400)
    _assert_f32(hc.run_cut(eng, ids, [5, 1]), hc.reference(cfg, w, ids))
    eng.dispose()


@pytest.mark.parametrize("name, layers, kw", [
    ("one expert per group", [(hc.delta(), hc.moe(experts=6, groups=6, keep=4, top=4))], {}),
    ("wide odd", [(hc.latent(heads=1, dim=7, rot=2, vdim=5, rank=9), hc.moe(ff=17)), (hc.delta(heads=1, kv_heads=1, dim=9, vdim=7, conv=2), None)], dict(width=50, vocab=33)),
    ("single tap", [(hc.delta(heads=2, kv_heads=1, dim=33, vdim=65, conv=1), None)], {}),
    ("six taps", [(hc.delta(heads=6, kv_heads=2, dim=130, vdim=40, conv=6), None)], {}),
    ("all experts", [(hc.latent(), hc.moe(experts=4, groups=2, keep=2, top=4))], {}),
    ("aligned", [(hc.latent(heads=4, dim=64, rot=32, vdim=64, rank=96), hc.moe(experts=16, top=4, groups=4, ff=64)),
                 (hc.delta(heads=6, kv_heads=3, dim=64, vdim=64), hc.moe(experts=16, top=2, groups=2, keep=1, ff=32))], dict(width=128, vocab=256)),
    ("rows of others", [(hc.latent(), None), (hc.latent(), None), (hc.latent(heads=7, kv_from=0), None), (hc.latent(heads=1, kv_from=1), None),
                        (hc.latent(kv_from=0), None)], {}),
])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(backend, name, layers, kw, dtype):
    cfg = hc.config(layers, **kw)
    w = hc.weights(cfg, seed=3, sharp=2.0)
    ids = hc.tokens(cfg, 1, 75, seed=4)
    eng = hc.engine(cfg, w, 1, 80, dtype)
    ref = hc.reference(cfg, w, ids)
    for cuts in ([75], [2, 31, 1]):
        (_assert_f32 if dtype == "float32" else _assert_bf16)(hc.run_cut(eng, ids, cuts), ref, f"{name} {cuts}")
    eng.dispose()


@pytest.mark.parametrize("dim", [64, 128])
def test_expanded_prompts_agree_with_absorbed_ones(backend, dim):
    """Head sizes with a tcgen05 prefill kernel: whole prompts, portions behind cached rows, batches, shared rows."""
    mk = lambda heads, **k: hc.latent(heads=heads, dim=dim, rot=64, vdim=dim, rank=96, scale=0.11, **k)  # noqa: E731
    cfg = hc.config([(mk(3), None), (mk(2, kv_from=0), None)], width=128)
    w = hc.weights(cfg, seed=5)
    ids = hc.tokens(cfg, 2, 390)
    ref = hc.reference(cfg, w, ids)
    eng = hc.engine(cfg, w, 2, 400, "bfloat16")
    assert all(m.wukv is not None for m in eng.mixers)
    for expand_from in (64, 1 << 30):
        eng.expand_from = expand_from
        for cuts in ([390], [130, 128, 70, 62], [64, 1, 100, 225]):
            e = hc.row_errors(hc.run_cut(eng, ids, cuts), ref)
            assert e.max() <= 1.5e-2, (expand_from, cuts, e.max())
    eng.dispose()


def test_expanded_reader_of_rows_that_their_owner_does_not_expand(backend):
    """The owner's head sizes have no prefill kernel, the reader's do: a batch must expand the cache rows themselves."""
    cfg = hc.config([(hc.latent(heads=2, dim=32, rot=64, vdim=48, rank=96, scale=0.11), None),
                     (hc.latent(heads=3, dim=64, rot=64, vdim=64, rank=96, scale=0.11, kv_from=0), None)], width=128)
    w = hc.weights(cfg, seed=6)
    ids = hc.tokens(cfg, 2, 200)
    eng = hc.engine(cfg, w, 2, 200, "bfloat16")
    assert [m.wukv is not None for m in eng.mixers] == [False, True]
    e = hc.row_errors(hc.run_cut(eng, ids, [200]), hc.reference(cfg, w, ids))
    assert e.max() <= 1.5e-2, e.max()
    eng.dispose()


@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation(backend, mixed, graph):
    cfg, w, ids, _ = mixed
    eng = hc.engine(cfg, w, 2, 64)
    got = eng.generate(ids[:, :20], 12, use_graph=graph)
    want = np.array([hybrid.greedy(cfg, w, row, 12) for row in ids[:, :20]])
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
    eng.extend(ids[:1, :15])
    with pytest.raises(ValueError, match="running sequences|exceed"):
        eng.extend(ids[:2, :1])
    eng.extend(ids[:1, :1])
    with pytest.raises(ValueError, match="overflow"):
        eng.extend(ids[:1, :1])
    eng.reset()
    with pytest.raises(ValueError, match="outside"):
        eng.extend(ids[:1, :3], [3])
    eng.extend(np.array([[cfg["vocab"]]], np.int32))
    with pytest.raises(lib.KandleCudaError, match="101"):
        backend.synchronize()
    eng.dispose()


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
        k = 0 if e["id"] == "a" else 1
        got = np.fromfile(out / f"{s['step']}.f32", "<f4").reshape(2, cfg["vocab"])
        want = ref[k][[at[e["id"]] + p for p in e["want"]]]
        # (bf16: a first-token routing call of the second request is close)
        assert hc.row_errors(got, want).max() <= (F32 if dtype == "float32" else 6e-2 if k == 0 else 0.25), s["step"]
        at[e["id"]] += len(e["tokens"])


def test_command_line_generates(backend, mixed, tmp_path):
    cfg, w, ids, _ = mixed
    _checkpoint(tmp_path, cfg, w)
    r = subprocess.run([sys.executable, "-m", "kandle_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--steps", "6",
                        "--prompt", " ".join(map(str, ids[0, :20]))], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(x) for x in r.stdout.split()] == hybrid.greedy(cfg, w, ids[0, :20], 6)
