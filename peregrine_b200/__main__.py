"""Command line.

    python -m peregrine_b200 generate --model PATH --prompt 1,2,3 [--prompt 4,5] --max-new 16
    python -m peregrine_b200 trace    --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N   < steps.jsonl

--model: a folder with config.json and model.safetensors, or a GGUF file.  Prompts and output are token ids.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="peregrine_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy continuation of prompts of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--dtype", choices=["bfloat16", "float32", "int8"], help="default: bfloat16 for a folder, int8 for a GGUF file")
    g.add_argument("--prompt", action="append", required=True, help="token ids with commas between them; one option per prompt")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--stop", default="", help="token ids that end a continuation")
    g.add_argument("--slots", type=int, default=0, help="sequences decoded together (default: one per prompt, at most 16)")
    g.add_argument("--capacity", type=int, default=0, help="positions per sequence (default: the model's)")
    g.add_argument("--portion", type=int, default=0, help="most prompt tokens of one step")
    t = sub.add_parser("trace", help="replay steps of given token ids and write logits")
    t.add_argument("--model", required=True)
    t.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    t.add_argument("--out", required=True)
    t.add_argument("--max-tokens", type=int, default=0)
    a = ap.parse_args(argv)
    if a.command == "trace":
        from . import trace

        return trace.run(a.model, a.dtype, a.out, a.max_tokens)
    from .registry import load_engine

    ids = lambda text: [int(x) for x in text.split(",") if x.strip()]
    prompts = [ids(p) for p in a.prompt]
    options = {"slots": a.slots or min(16, len(prompts)), "capacity": a.capacity}
    if a.dtype:
        options["dtype"] = a.dtype
    if a.portion:
        options["portion"] = a.portion
    for out in load_engine(a.model, **options).generate(prompts, a.max_new, ids(a.stop)):
        print(",".join(map(str, out)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
