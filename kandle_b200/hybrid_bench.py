"""Throughput of the hybrid designs beside Qwen3 at equal size (`bench.py --hybrid [--hybrid-design vogozen]`):
random weights, a few layers of sizes that resemble real models, prefill and decode of a batch of equal-length
prompts, the device time of every kernel call of a prefill, and the design's kernels alone against their rooflines
beside the like kernels of the other models.

Equal size: the same width, heads, layers and vocabulary, and a dense MLP of the same width (Pedorax: as wide as the
experts that a token passes, top x ff).
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
from .model_utils.vogozen import VogozenConfig

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


WINDOW = 1024


def vogozen_config(s: dict, layers: int, dtype: str = "bfloat16") -> VogozenConfig:
    attention = {"heads": s["qheads"], "kv_heads": s["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOW},
                 "rot": {"base": 1e6, "dims": 128}}
    wkv = {"heads": s["width"] // 64, "dim": 64}
    delta = {"heads": s["heads"], "kv_heads": s["heads"], "dim": 128, "vdim": 128, "conv": 4}
    kinds = [("attention", attention), ("wkv", wkv), ("delta", delta)]
    entries = [{"type": kinds[i % 3][0], "mixer": kinds[i % 3][1], "mlp": {"kind": "dense", "ff": s["top"] * s["ff"]}} for i in range(layers)]
    return VogozenConfig.fromDict({"vocab": VOCAB, "width": s["width"], "layers": entries, "norm": {"eps": 1e-6}}, dtype)


def engines(design: str, size: str, layers: int, batch: int, max_s: int):
    s = SIZES[size]
    config = {"pedorax": pedorax_config, "vogozen": vogozen_config}[design]
    yield design, lambda: HybridEngine(config(s, layers), RandomInit(seed=1234, std=0.02), batch, max_s)
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
                                "kd_linear_bf16_skinny_splits", "kd_graph", "kd_attention_head_sizes")):
                return self._call(name, *args)
            a, b = CudaEvent(), CudaEvent()
            self._call("kd_event_record", ctypes.c_uint64(a.handle))
            self._call(name, *args)
            self._call("kd_event_record", ctypes.c_uint64(b.handle))
            label = name
            if name in ("kd_linear_ex", "kd_linear_bf16", "kd_moe_linear", "kd_linear_glu", "kd_linear_tanh", "kd_linear_bf16_skinny"):
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


def _rand(shape, dtype="bfloat16", std=0.05):
    t = core.empty(shape, dtype)
    lib.call("kd_randn", _r(t), ctypes.c_uint64(1), ctypes.c_uint32(0), ctypes.c_float(0.0), ctypes.c_float(std), 0, 0, 0)
    return t


class _Rooflines:
    """Kernels alone, each over enough operand sets that every launch streams from HBM (one captured graph of 8 launches,
    replayed), as fractions of the bound that is named."""

    def __init__(self, hbm_gbs: float, tflops: float):
        self.hbm, self.tflops, self.out = hbm_gbs, tflops, {}

    def __call__(self, name, launches, nbytes=None, flops=None, fp32_pairs=None):
        for fn in launches:
            fn()
        lib.call("kd_graph_begin")
        for i in range(8):
            launches[i % len(launches)]()
        g = ctypes.c_uint64(0)
        lib.call("kd_graph_end", ctypes.byref(g))
        ms = _timed(lambda: lib.call("kd_graph_launch", g), 5) / 8
        lib.call("kd_graph_destroy", g)
        r = self.out[name] = {"us": round(ms * 1e3, 2)}
        if nbytes is not None:
            r.update(bytes=int(nbytes), gbs=round(nbytes / ms / 1e6), of_measured_hbm=round(nbytes / ms / 1e6 / self.hbm, 3))
        if flops is not None:
            r.update(tflops=round(flops / ms / 1e9, 1), of_measured_bf16=round(flops / ms / 1e9 / self.tflops, 3))
        if fp32_pairs is not None:      # multiply-adds against 128 a clock and SM at the maximum clock (1965 MHz)
            r.update(of_fp32_rate=round(fp32_pairs / ms / 1e9 / (128 * 148 * 1.965e-3), 3))


def vogozen_rooflines(size: str, batch: int, ctx: int, hbm_gbs: float, tflops: float) -> dict:
    """The design's kernels in a decode step (suffix _step) and in a prefill of batch x ctx tokens, and the like kernels of
    Qwen3 and Pedorax: add + RMS norm, q/k norm + rotation + cache row, full and decode attention, the delta rule with a
    decay per channel."""
    s = SIZES[size]
    W, H, G, HD, D, HW = s["width"], s["qheads"], s["kv_heads"], s["heads"], 128, s["width"] // 64
    m = _Rooflines(hbm_gbs, tflops)
    f32 = ctypes.c_float
    C = lib.call
    for tag, S, sets in (("", ctx, 1), ("_step", 1, 4)):
        T, max_s, pos = batch * S, ctx + 64, 0 if S > 1 else ctx - 1
        # residual and norms
        x, y, h = _rand((T, W), "float32"), _rand((1, T, W), "bfloat16" if S > 1 else "float32"), core.empty((T, W), "bfloat16")
        w32, w16 = _rand((W,), "float32"), _rand((W,))
        yb = T * W * (2 if S > 1 else 4)
        m("residual_post_norm" + tag, [lambda: C("kd_residual_post_norm", _r(x), _r(y), _r(w32), f32(1e-6), None, _r(x), _r(h))], nbytes=T * W * 10 + yb)
        m("qwen3_add_rmsnorm" + tag, [lambda: C("kd_add_rmsnorm", _r(y), _r(x), _r(w16), f32(1e-6), _r(x), _r(h))], nbytes=T * W * 10 + yb)
        del x, y, h
        # attention
        N = (H + 2 * G) * D
        proj, q, out = _rand((batch, S, N), std=1.0), core.empty((batch, S, H, D), "bfloat16"), core.empty((T, H * D), "bfloat16")
        qn, kn, cos, sin = _rand((H * D,), "float32", 1.0), _rand((G * D,), "float32", 1.0), _rand((max_s, D // 2), "float32"), _rand((max_s, D // 2), "float32")
        kv = [(_rand((batch, G, max_s, D), std=1.0), _rand((batch, G, max_s, D), std=1.0)) for _ in range(sets)]
        sink, qn16 = core.zeros((H,), "float32"), _rand((D,))
        prep = 2 * T * N * 2
        m("qk_norm_rope" + tag, [lambda: C("kd_qk_norm_rope_cache", _r(proj), 0, H * D, (H + G) * D, D, D, D, _r(qn), _r(kn), f32(1e-6), _r(cos), _r(sin),
                                           _r(kv[0][0]), _r(kv[0][1]), None, pos, _r(q))], nbytes=prep)
        cs, sn = (t.slice([slice(pos, pos + S), slice(None)]) for t in (cos, sin))
        p2, q4 = proj.view(T, N), q.view(batch, S, H, D)
        m("qwen3_qk_norm_rope" + tag, [lambda: C("kd_qkv_norm_rope_cachewrite", _r(p2), _r(qn16), _r(qn16), f32(1e-6), _r(cs), _r(sn),
                                                 _r(kv[0][0]), _r(kv[0][1]), None, pos, _r(q4))], nbytes=prep)
        bound = {}
        if S > 1:
            seen = sum(min(i + 1, WINDOW) for i in range(S))
            bound = {"window": dict(flops=4.0 * batch * H * D * seen), "full": dict(flops=4.0 * batch * H * D * S * (S + 1) / 2)}
        else:
            row = 2 * batch * G * D * 2
            bound = {"window": dict(nbytes=row * min(WINDOW, ctx)), "full": dict(nbytes=row * ctx)}
        m("window_attention" + tag, [(lambda k, v: lambda: C("kd_window_attention", _r(q), _r(k), _r(v), _r(sink), f32(D ** -0.5), WINDOW, None, pos, _r(out)))(k, v) for k, v in kv],
          **bound["window"])
        m("all_keys_attention" + tag, [(lambda k, v: lambda: C("kd_window_attention", _r(q), _r(k), _r(v), _r(sink), f32(D ** -0.5), 0, None, pos, _r(out)))(k, v) for k, v in kv],
          **bound["full"])
        if S > 1:
            qv, ov = q.permute([0, 2, 1, 3]), out.view(batch, S, H, D).permute([0, 2, 1, 3])
            kvs = [tuple(t.slice([slice(None), slice(None), slice(0, S), slice(None)]) for t in p) for p in kv]
            m("qwen3_attention", [lambda: C("kd_flash_attention", _r(qv), _r(kvs[0][0]), _r(kvs[0][1]), _r(ov), f32(D ** -0.5), 1)], **bound["full"])
        else:
            qv, ov = q.view(batch, H, 1, D), out.view(batch, H, 1, D)
            m("qwen3_attention_step", [(lambda k, v: lambda: C("kd_attention_decode", _r(qv), _r(k), _r(v), None, ctx, f32(D ** -0.5), 0, _r(ov)))(k, v) for k, v in kv], **bound["full"])
            mid = (WINDOW + 63) // 64 * 64
            ks = [tuple(t.slice([slice(None), slice(None), slice(0, mid), slice(None)]) for t in p) for p in kv]
            m("qwen3_attention_step_window_keys", [(lambda k, v: lambda: C("kd_attention_decode", _r(qv), _r(k), _r(v), None, min(WINDOW, ctx), f32(D ** -0.5), 0, _r(ov)))(k, v) for k, v in ks],
              **bound["window"])
        del kv, proj, q, out
        # recurrences
        n = HW * 64
        hh, mixes = _rand((batch, S, W)), core.empty((5 * T, W), "bfloat16")
        last, mu = core.zeros((batch, W), "bfloat16"), _rand((5, W), "float32")
        m("token_shift" + tag, [lambda: C("kd_token_shift", _r(hh), _r(mu), _r(last), _r(mixes))], nbytes=T * W * 2 * 6)
        w4, rkvg = _rand((4, n, W)), core.empty((4 * T, n), "bfloat16")
        x4 = mixes.slice([slice(0, 4 * T), slice(None)])
        m("wkv_projections" + tag, [lambda: C("kd_moe_linear", _r(x4), _r(w4), None, 0, f32(0), _r(rkvg))],
          **(dict(flops=2.0 * 4 * T * n * W) if S > 1 else dict(nbytes=4 * n * W * 2)))
        del hh, mixes
        r, k, v = (rkvg.slice([slice(i * T, (i + 1) * T), slice(None)]).view(batch, S, n) for i in range(3))
        logits, o, w0 = _rand((T, n), "float32"), core.empty((T, n), "float32"), core.full((n,), -3.0)
        states = [core.zeros((batch, HW, 64, 64), "float32") for _ in range(sets * 2)]
        m("wkv" + tag, [(lambda st: lambda: C("kd_wkv", _r(r), _r(k), _r(v), _r(logits), _r(w0), _r(w0), _r(st), _r(o)))(st) for st in states],
          **(dict(fp32_pairs=2.25 * T * HW * 64 * 64) if S > 1 else dict(nbytes=2 * batch * HW * 64 * 64 * 4)))
        gate, y = rkvg.slice([slice(3 * T, 4 * T), slice(None)]), core.empty((T, n), "bfloat16")
        m("gated_head_norm" + tag, [lambda: C("kd_gated_head_norm", _r(o), _r(gate), _r(w0), HW, f32(1e-6), 1, _r(y))], nbytes=T * n * 8)
        del states, rkvg, logits, o, y
        vv = HD * 128
        N = 3 * vv + HD + 64 - HD % 8
        proj, conv, rate, o = _rand((batch, S, N)), _rand((vv, 4), "float32"), _rand((HD,), "float32"), core.empty((T, vv), "float32")
        hist, states = core.zeros((batch, 3, 3 * vv), "bfloat16"), [core.zeros((batch, HD, 128, 128), "float32") for _ in range(sets)]
        for name, width, bias in (("delta_head_decay", HD, rate), ("pedorax_delta_channel_decay", vv, _rand((vv,), "float32"))):
            dec = _rand((T, width), "float32")
            m(name + tag, [(lambda st: lambda: C("kd_delta_rule", _r(proj), 0, vv, 2 * vv, 3 * vv, _r(dec), HD, HD, 128, 128, _r(conv), _r(conv), _r(conv),
                                                 _r(rate), _r(bias), _r(hist), _r(st), _r(o)))(st) for st in states],
              **(dict(fp32_pairs=3.25 * T * HD * 128 * 128) if S > 1 else dict(nbytes=2 * batch * HD * 128 * 128 * 4)))
        del proj, o, states
        # feed-forward
        ff = s["top"] * s["ff"]
        hx, act = _rand((T, W)), core.empty((T, ff), "bfloat16")
        gus = [_rand((2 * ff, W)) for _ in range(1 if S > 1 else 4)]
        cost = dict(flops=4.0 * T * ff * W) if S > 1 else dict(nbytes=2 * ff * W * 2)
        m("geglu" + tag, [(lambda w: lambda: C("kd_linear_glu", _r(hx), _r(w), 5, _r(act)))(w) for w in gus], **cost)
        if S > 1:
            m("qwen3_swiglu", [lambda: C("kd_linear_bf16", _r(hx), _r(gus[0]), None, 2, _r(act))], **cost)
        else:
            m("qwen3_swiglu_step", [(lambda w: lambda: C("kd_linear_bf16_skinny", _r(hx), _r(w), 2, _r(act)))(w) for w in gus], **cost)
        del hx, act, gus
        import gc
        gc.collect()
        lib.call("kd_empty_cache")
    return m.out


def decode_rooflines(size: str, batch: int, ctx: int, hbm_gbs: float) -> dict:
    """The HBM-bound kernels of a Pedorax decode step alone, and Qwen3's decode attention beside them."""
    s = SIZES[size]
    H, rank, W, E, ff = s["heads"], s["rank"], s["width"], s["experts"], s["ff"]
    width = (rank + 64 + 15) // 16 * 16
    roofs, rand = _Rooflines(hbm_gbs, 1.0), _rand

    def measure(name, nbytes, launches):
        roofs(name, launches, nbytes=nbytes)

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
    return roofs.out


def run_size(design: str, size: str, layers: int, batch: int, prompt: int, steps: int, profile: bool, hbm_gbs: float, tflops: float) -> dict:
    rec = {"design": design, "size": size, "layers": layers, "batch": batch, "prompt": prompt, "decode_steps": steps}
    ids = Tensor(synth.token_ids(f"hybrid.{size}", (batch, prompt), VOCAB))
    for name, make in engines(design, size, layers, batch, prompt + 5 * steps + 8):
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
        if design == "vogozen":
            rec["kernels"] = vogozen_rooflines(size, batch, prompt, hbm_gbs, tflops)
        else:
            rec["decode_kernels"] = decode_rooflines(size, batch, prompt, hbm_gbs)
    rec["prefill_ratio"] = round(rec[design]["prefill_tokens_per_s"] / rec["qwen3"]["prefill_tokens_per_s"], 3)
    rec["decode_ratio"] = round(rec[design]["decode_tokens_per_s"] / rec["qwen3"]["decode_tokens_per_s"], 3)
    return rec


def main(design: str, sizes, layers: int, batch: int, prompt: int, steps: int, hbm_gbs: float, tflops: float, profile: bool = True) -> None:
    t0 = time.time()
    for size in sizes:
        print(json.dumps(run_size(design, size, layers, batch, prompt, steps, profile, hbm_gbs, tflops)), flush=True)
    print(json.dumps({"hybrid_bench_seconds": round(time.time() - t0, 1)}), flush=True)
