"""Trace replay: given tokens through an engine's own portion and decode steps (see bin/trace_run)."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def replay(engine, lines, out_dir: str, emit) -> None:
    """lines: JSON texts, one step each.  emit("done <step>") after every step."""
    running = None
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        if len(step["entries"]) > 1:
            raise ValueError(f"step {step['step']}: one entry a step, got {len(step['entries'])}")
        for entry in step["entries"]:
            if running != entry["id"]:
                if running is not None:
                    raise ValueError(f"request {entry['id']} begins before {running} has ended")
                engine.reset()
                running = entry["id"]
            logits = engine.extend(np.asarray([entry["tokens"]], np.int32), entry["want"])
            if entry["want"]:
                logits.dataAsync().astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        if running in step["end"]:
            running = None
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays tokens from standard input through a model and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits, one <step>.f32 a step")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that the running request holds")
    a = ap.parse_args(argv)
    import kandle_b200
    from . import registry
    if a.dtype not in registry.lookup(registry.load_config(a.model)).dtypes:
        print(f"{a.dtype} is not available for this model", file=sys.stderr)
        return 3
    kandle_b200.init(0)
    engine = registry.load_engine(a.model, 1, max(a.max_tokens, 1), a.dtype)
    replay(engine, iter(sys.stdin.readline, ""), a.out, lambda text: print(text, flush=True))
    return 0
