"""Replays given token ids through a model, step by step, and writes logits: no sampling, no batching of its own,
only the runtime's caches, prompt passes and decode steps (lbk_model_forward_rows).

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input, one JSON object a line: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}],
"end": []}. Every entry's tokens continue its request; the logits at the wanted places go to DIR/<step>.f32 (f32,
little-endian, [wanted, vocab], in the order of the entries), then `done <step>` is printed. Requests listed in
"end" give their cache back, and the next request takes it over as it is.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

import numpy as np


def replay(net, lines, out_dir, max_tokens: int, emit) -> None:
    """`lines`: the steps as JSON text; `emit(step)` is called after each."""
    live, free = {}, []
    out_dir = Path(out_dir)
    for line in lines:
        line = line.strip()
        if not line:
            continue
        step = json.loads(line)
        rows = []
        for entry in step["entries"]:
            rid = entry["id"]
            if rid not in live:
                live[rid] = free.pop() if free else net.new_cache(1, max_tokens)
            want = entry.get("want", [])
            if len(entry["tokens"]):
                rows.append(net.forward_rows(entry["tokens"], live[rid], want))
        net.ctx.check_device_error()
        if any(len(r) for r in rows):
            np.concatenate(rows).astype("<f4").tofile(out_dir / f"{step['step']}.f32")
        for rid in step.get("end", []):
            if rid in live:
                cache = live.pop(rid)
                net.reset_cache(cache)
                free.append(cache)
        emit(step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="the most tokens live requests hold at any time")
    a = ap.parse_args(argv)
    from . import _lib, build, runtime
    _lib.use(build.library_for(runtime.architecture_of(a.model)))
    net = runtime.load_model(a.model, dtype=a.dtype)

    def emit(step):
        sys.stdout.write(f"done {step}\n")
        sys.stdout.flush()

    replay(net, sys.stdin, a.out, max(1, a.max_tokens), emit)
    net.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
