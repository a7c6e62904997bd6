"""Generate token ids from a prompt of token ids: ``python -m fusekit_b200.generate --model DIR --prompt 5,17,3 --max-tokens 20``.

Any model the registry or a checkpoint directory names runs (``--config NAME`` takes a registered shape with synthetic
weights); greedy by default, sampled with ``--temperature``.  One line of comma-separated token ids comes out.
"""
from __future__ import annotations

import argparse
import sys

from .checkpoint import load_engine
from .model_spec import CONFIGS, LAYERED_CONFIGS, LayeredSpec, config
from .runtime import attach


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m fusekit_b200.generate", description="Generate token ids after a prompt of token ids.")
    src = ap.add_mutually_exclusive_group(required=True)
    src.add_argument("--model", help="directory with config.json and safetensors files")
    src.add_argument("--config", choices=sorted(CONFIGS) + sorted(LAYERED_CONFIGS), help="registered shape with synthetic weights")
    ap.add_argument("--prompt", required=True, help="comma-separated token ids")
    ap.add_argument("--max-tokens", type=int, default=32)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default=None, help="number format of a layered decoder (default bfloat16)")
    args = ap.parse_args(argv)
    prompt = [int(t) for t in args.prompt.split(",")]
    kw = {"want_logits": args.temperature > 0.0}
    if args.dtype is not None:
        kw["dtype"] = args.dtype
    capacity = len(prompt) + args.max_tokens
    if args.model:
        engine, _ = load_engine(args.model, capacity, **kw)
    else:
        spec = config(args.config)
        if args.dtype is not None and not isinstance(spec, LayeredSpec):
            ap.error("--dtype applies to layered decoders")
        engine = attach(spec, capacity, **kw)
        engine.load_synthetic()
    try:
        toks = engine.complete(prompt, args.max_tokens, args.temperature, args.top_k, args.top_p, args.seed)
        print(",".join(str(int(t)) for t in toks))
    finally:
        engine.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
