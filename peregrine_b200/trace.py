"""Replays a trace: steps of given token ids, read as JSON lines, through a model's engine, writing logits.

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

A step in which logits are wanted writes <out>/<step>.f32: little-endian f32 [wanted, vocab], in the order of the entries
and of their `want`.  After every step a line `done <step>` is printed.  Requests in `end` give their slots back after the
step.
"""
from __future__ import annotations

import json
import os
import sys

import numpy as np

from .registry import load_engine


def run(model: str, dtype: str, out: str, max_tokens: int, lines=sys.stdin, log=sys.stdout, slots: int = 8) -> int:
    engine = load_engine(model, dtype=dtype, slots=slots, capacity=max_tokens)
    if not hasattr(engine, "step"):
        print(f"{model}: this model's engine takes no single steps", file=sys.stderr)
        return 3
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = engine.step([(e["id"], e["tokens"], e.get("want", [])) for e in s["entries"]])
        if len(logits):
            path = os.path.join(out, f"{s['step']}.f32")
            with open(path + ".tmp", "wb") as f:
                f.write(np.ascontiguousarray(logits, "<f4").tobytes())
            os.replace(path + ".tmp", path)
        for key in s.get("end", []):
            engine.end(key)
        print(f"done {s['step']}", file=log, flush=True)
    return 0
