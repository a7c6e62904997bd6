"""Trace replay: ``bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N`` feeds given token ids through a
model step by step and writes the logits that are asked for; nothing is sampled.

Steps come on standard input, one JSON object a line: ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [id, ...]}``.
``want`` lists places among the entry's tokens; their logits go to ``DIR/<step>.f32`` (little-endian fp32, entries in order).
``done <step>`` is printed after every step.  The model runs through the engine its configuration selects, with its own
sequences and caches.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from .checkpoint import load_engine


class TraceRunner:
    def __init__(self, engine, out_dir: str):
        self.engine, self.out_dir, self.live = engine, out_dir, {}

    def step(self, doc: dict) -> int:
        parts = []
        for e in doc["entries"]:
            if e["id"] not in self.live:
                self.live[e["id"]] = self.engine.open_sequence()
            logits = self.live[e["id"]].append(e["tokens"], e.get("want", []))
            if len(logits):
                parts.append(logits)
        for rid in doc.get("end", []):
            if rid in self.live:
                self.live.pop(rid).close()
        if parts:
            np.concatenate(parts).astype("<f4").tofile(os.path.join(self.out_dir, f"{doc['step']}.f32"))
        return doc["step"]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed token ids through a model step by step and write logits.")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors files")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory of the logit files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    engine, ck = load_engine(args.model, max(args.max_tokens, 1), dtype=args.dtype)
    try:
        if not hasattr(engine, "open_sequence"):
            raise ValueError(f"trace replay runs layered decoders; {args.model} holds a {ck.spec.arch} model")
        runner = TraceRunner(engine, args.out)
        for line in sys.stdin:
            if line.strip():
                print(f"done {runner.step(json.loads(line))}", flush=True)
    finally:
        engine.close()
        ck.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
