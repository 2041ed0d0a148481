"""Generation from a checkpoint folder:

    python -m kandle_b200.generate --model DIR --prompt "5 17 3" [--steps 32] [--dtype bfloat16|float32]
                                   [--temperature T --top-k K --top-p P --seed S]

The model class follows from config.json (kandle_b200.registry).  Prompts are token ids (this package has no
tokenizer); several --prompt of one length run as a batch.  Prints the generated ids, one line a prompt.
"""
from __future__ import annotations

import argparse

import numpy as np


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m kandle_b200.generate", description="Generates tokens from a checkpoint folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", required=True, action="append", help="token ids; repeat for a batch of equal lengths")
    ap.add_argument("--steps", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--temperature", type=float, default=None, help="sample instead of the greedy choice")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    a = ap.parse_args(argv)
    rows = [[int(x) for x in p.split()] for p in a.prompt]
    if len({len(r) for r in rows}) != 1 or not rows[0]:
        ap.error("prompts must have one length, at least one token")
    import kandle_b200
    from . import registry
    kandle_b200.init(0)
    engine = registry.load_engine(a.model, len(rows), len(rows[0]) + a.steps, a.dtype)
    if a.temperature is not None:
        engine.set_sampler(a.temperature, a.top_k, a.top_p, a.seed)
    for row in engine.generate(np.asarray(rows, np.int32), a.steps):
        print(" ".join(str(t) for t in row))
    engine.dispose()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
