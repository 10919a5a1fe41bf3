"""Greedy generation from token ids through the batcher, for any model family:

    python -m lemonade_burn_b200.generate --model DIR --prompt 5,17,3 [--prompt 9,2] --max-new 32

prints one line of generated ids per prompt. There is no tokenizer here (the reference's lb-run has one,
crates/lb-model/src/bin/lb-run.rs).
"""
from __future__ import annotations

import argparse
import sys


def generate(net, prompts, max_new: int, slots: int = 4, capacity: int = 0, eos: int = -1):
    """Lists of generated token ids, one per prompt; the prompts share decode steps."""
    capacity = capacity or max(len(p) for p in prompts) + max_new
    bt = net.batcher(max(1, min(slots, len(prompts), 16)), capacity)
    ids = [bt.submit(p, max_new, eos) for p in prompts]
    bt.run()
    out = [bt.poll(i)[0] for i in ids]
    bt.close()
    return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description="greedy generation from token ids")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--prompt", required=True, action="append", help="token ids with commas between them; may be given several times")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--slots", type=int, default=4)
    ap.add_argument("--eos", type=int, default=-1)
    a = ap.parse_args(argv)
    from . import _lib, build, runtime
    _lib.use(build.library_for(runtime.architecture_of(a.model)))
    net = runtime.load_model(a.model, dtype=a.dtype)
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    for toks in generate(net, prompts, a.max_new, a.slots, eos=a.eos):
        print(",".join(str(t) for t in toks))
    net.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
