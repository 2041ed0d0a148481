"""Throughput of the Pedorax design beside Qwen3 at equal size (`bench.py --hybrid`): random weights, a few
layers of sizes that resemble real models, prefill and decode of a batch of equal-length prompts, and the
device time of every kernel call of a prefill against its roofline.

Equal size: the same width, heads, layers and vocabulary, and a dense MLP as wide as the experts that a
token passes (top x ff).
"""
from __future__ import annotations

import ctypes
import json
import time
from collections import OrderedDict

import numpy as np

from . import core, lib, synth
from .backend import CudaEvent
from .core import Tensor
from .engine import Qwen3Engine, RandomInit, _r
from .hybrid_engine import HybridEngine
from .model_utils.pedorax import PedoraxConfig
from .model_utils.qwen3 import Qwen3Config

VOCAB = 32768
SIZES = {
    "1k": dict(width=1024, heads=8, rank=256, experts=32, top=4, ff=512, groups=4, keep=2, qheads=8, kv_heads=4),
    "2k": dict(width=2048, heads=16, rank=512, experts=64, top=6, ff=1024, groups=8, keep=4, qheads=16, kv_heads=8),
    "4k": dict(width=4096, heads=32, rank=512, experts=64, top=8, ff=1536, groups=8, keep=4, qheads=32, kv_heads=8),
}


def pedorax_config(s: dict, layers: int, dtype: str = "bfloat16") -> PedoraxConfig:
    mlp = {"kind": "moe", "expert": {"ff": s["ff"], "limit": 7.0},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": s["groups"], "keep": s["keep"]}}}
    latent = {"heads": s["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": s["rank"], "scale": 192 ** -0.5,
              "rot": {"base": 10000.0, "dims": 64}}
    delta = {"heads": s["heads"], "kv_heads": s["heads"], "dim": 128, "vdim": 128, "conv": 4}
    entries = [{"type": "channel_delta", "mixer": delta, "mlp": mlp} if i % 2 == 0 else {"type": "latent_attention", "mixer": latent, "mlp": mlp}
               for i in range(layers)]
    return PedoraxConfig.fromDict({"vocab": VOCAB, "width": s["width"], "layers": entries, "embedding": {"scale": 1.0}, "logit_scale": 1.0,
                                   "norm": {"eps": 1e-6}}, dtype)


def engines(size: str, layers: int, batch: int, max_s: int):
    s = SIZES[size]
    yield "pedorax", lambda: HybridEngine(pedorax_config(s, layers), RandomInit(seed=1234, std=0.02), batch, max_s)
    q = Qwen3Config(vocabSize=VOCAB, hiddenSize=s["width"], intermediateSize=s["top"] * s["ff"], numHiddenLayers=layers, numAttentionHeads=s["qheads"],
                    numKeyValueHeads=s["kv_heads"], headDim=128, dtype="bfloat16")
    yield "qwen3", lambda: Qwen3Engine(q, RandomInit(seed=1234, std=0.02), batch, max_s)


class CallTimer:
    """Wraps the library's call function for the duration of a block: device time per entry point."""

    def __init__(self):
        self.marks, self.order = [], OrderedDict()

    def __enter__(self):
        self._call = lib.call

        def timed(name, *args):
            if name.startswith(("kd_event", "kd_set_pdl", "kd_upload", "kd_download", "kd_storage", "kd_synchronize", "kd_latent_attention_splits",
                                "kd_linear_bf16_skinny_splits", "kd_graph")):
                return self._call(name, *args)
            a, b = CudaEvent(), CudaEvent()
            self._call("kd_event_record", ctypes.c_uint64(a.handle))
            self._call(name, *args)
            self._call("kd_event_record", ctypes.c_uint64(b.handle))
            label = name
            if name in ("kd_linear_ex", "kd_linear_bf16", "kd_moe_linear"):
                w = args[1]._obj
                label = f"{name} [{w.shape[w.ndim - 2]},{w.shape[w.ndim - 1]}]"
            self.marks.append((label, a, b))
        lib.call = timed
        return self

    def __exit__(self, *exc):
        lib.call = self._call
        return False

    def totals(self) -> dict:
        out = OrderedDict()
        for name, a, b in self.marks:
            n, ms = out.get(name, (0, 0.0))
            out[name] = (n + 1, ms + a.elapsed_ms(b))
        return {k: {"calls": n, "ms": round(ms, 4)} for k, (n, ms) in out.items()}


def _timed(fn, reps: int) -> float:
    fn()
    best = []
    for _ in range(reps):
        a, b = CudaEvent(), CudaEvent()
        a.record()
        fn()
        b.record()
        best.append(a.elapsed_ms(b))
    return float(np.median(best))


def decode_rooflines(size: str, batch: int, ctx: int, hbm_gbs: float) -> dict:
    """The HBM-bound kernels of a decode step alone, each over enough operand sets that every launch streams from HBM
    (one captured graph of 8 launches, replayed), and Qwen3's decode attention beside them."""
    s = SIZES[size]
    H, rank, W, E, ff = s["heads"], s["rank"], s["width"], s["experts"], s["ff"]
    width = (rank + 64 + 15) // 16 * 16
    out = {}

    def rand(shape, dtype="bfloat16"):
        t = core.empty(shape, dtype)
        lib.call("kd_randn", _r(t), ctypes.c_uint64(1), ctypes.c_uint32(0), ctypes.c_float(0.0), ctypes.c_float(0.05), 0, 0, 0)
        return t

    def measure(name, nbytes, launches):
        for fn in launches:
            fn()
        lib.call("kd_graph_begin")
        for i in range(8):
            launches[i % len(launches)]()
        g = ctypes.c_uint64(0)
        lib.call("kd_graph_end", ctypes.byref(g))
        ms = _timed(lambda: lib.call("kd_graph_launch", g), 5) / 8
        lib.call("kd_graph_destroy", g)
        out[name] = {"us": round(ms * 1e3, 2), "bytes": int(nbytes), "gbs": round(nbytes / ms / 1e6), "of_measured_hbm": round(nbytes / ms / 1e6 / hbm_gbs, 3)}

    sets = 4
    caches = [rand((batch, ctx + 64, width)) for _ in range(sets)]
    q = rand((batch, 1, H, width))
    n = ctypes.c_int(0)
    lib.call("kd_latent_attention_splits", batch, 1, H, ctx + 64, ctypes.byref(n))
    po, pm = core.empty((batch * H, n.value, rank)), core.empty((batch * H, n.value, 2))
    measure("latent_attention", batch * ctx * (rank + 64) * 2, [
        (lambda c: lambda: lib.call("kd_latent_attention", _r(q), _r(c), rank, ctypes.c_float(0.07), None, ctx - 1, _r(po), _r(pm)))(c) for c in caches])
    del caches
    N = 3 * H * 128 + H + 64 - H % 8
    proj, dec = rand((batch, 1, N)), rand((batch, H * 128), "float32")
    conv, vec, big = rand((H * 128, 4), "float32"), rand((H,), "float32"), rand((H * 128,), "float32")
    states = [core.zeros((batch, H, 128, 128), "float32") for _ in range(sets)]
    hist, o = core.zeros((batch, 3, 3 * H * 128), "bfloat16"), core.empty((batch, H * 128), "float32")
    measure("delta_step", 2 * batch * H * 128 * 128 * 4, [
        (lambda st: lambda: lib.call("kd_delta_rule", _r(proj), 0, H * 128, 2 * H * 128, 3 * H * 128, _r(dec), H, H, 128, 128, _r(conv), _r(conv), _r(conv),
                                     _r(vec), _r(big), _r(hist), _r(st), _r(o)))(st) for st in states])
    del states
    R = batch * s["top"]
    off = Tensor((np.arange(E + 1) * R // E).astype(np.int32))
    used = len({int(e) for e in np.arange(R) * E // R}) if R < E else E
    x, act, y = rand((R, W)), core.empty((R, ff), "bfloat16"), core.empty((R, W), "bfloat16")
    gus, downs = [rand((E, 2 * ff, W)) for _ in range(2)], [rand((E, W, ff)) for _ in range(2)]
    measure("expert_gate_up", used * 2 * ff * W * 2, [(lambda w: lambda: lib.call("kd_moe_linear", _r(x), _r(w), _r(off), 4, ctypes.c_float(7.0), _r(act)))(w) for w in gus])
    measure("expert_down", used * ff * W * 2, [(lambda w: lambda: lib.call("kd_moe_linear", _r(act), _r(w), _r(off), 0, ctypes.c_float(0.0), _r(y)))(w) for w in downs])
    del gus, downs
    Hq, Hk = s["qheads"], s["kv_heads"]
    kv = [(rand((batch, Hk, ctx + 64, 128)), rand((batch, Hk, ctx + 64, 128))) for _ in range(sets)]
    qq, oo = rand((batch, Hq, 1, 128)), core.empty((batch, Hq, 1, 128), "bfloat16")
    measure("qwen3_decode_attention", 2 * batch * Hk * ctx * 128 * 2, [
        (lambda k, v: lambda: lib.call("kd_attention_decode", _r(qq), _r(k), _r(v), None, ctx, ctypes.c_float(0.088), 0, _r(oo)))(k, v) for k, v in kv])
    return out


def run_size(size: str, layers: int, batch: int, prompt: int, steps: int, profile: bool, hbm_gbs: float) -> dict:
    rec = {"size": size, "layers": layers, "batch": batch, "prompt": prompt, "decode_steps": steps}
    ids = Tensor(synth.token_ids(f"hybrid.{size}", (batch, prompt), VOCAB))
    for name, make in engines(size, layers, batch, prompt + 5 * steps + 8):
        eng = make()
        r = {}
        prefill_ms = _timed(lambda: eng.prefill(ids), 3)
        r["prefill_ms"], r["prefill_tokens_per_s"] = round(prefill_ms, 3), round(batch * prompt / prefill_ms * 1e3)
        tok = eng.prefill(ids)
        eng.start_decode(tok)

        def decode():
            for _ in range(steps):
                eng.decode_step()
        ms = _timed(decode, 3) / steps
        r["decode_ms_per_step"], r["decode_tokens_per_s"] = round(ms, 4), round(batch / ms * 1e3)
        if profile:
            with CallTimer() as t:
                eng.prefill(ids)
            r["prefill_calls"] = t.totals()
        rec[name] = r
        eng.dispose()
        del eng
        import gc
        gc.collect()
        lib.call("kd_empty_cache")
    if profile:
        rec["decode_kernels"] = decode_rooflines(size, batch, prompt, hbm_gbs)
    rec["prefill_ratio"] = round(rec["pedorax"]["prefill_tokens_per_s"] / rec["qwen3"]["prefill_tokens_per_s"], 3)
    rec["decode_ratio"] = round(rec["pedorax"]["decode_tokens_per_s"] / rec["qwen3"]["decode_tokens_per_s"], 3)
    return rec


def main(sizes, layers: int, batch: int, prompt: int, steps: int, hbm_gbs: float, profile: bool = True) -> None:
    t0 = time.time()
    for size in sizes:
        print(json.dumps(run_size(size, layers, batch, prompt, steps, profile, hbm_gbs)), flush=True)
    print(json.dumps({"hybrid_bench_seconds": round(time.time() - t0, 1)}), flush=True)
