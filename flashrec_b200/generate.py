"""Command line of the step engine: tokens generated after prompts of token ids.

    bin/generate --model DIR [--dtype bfloat16|float32] --max-new-tokens N --prompt "1 2 3" [--prompt ...]

Prints one JSON object per prompt: {"prompt": i, "tokens": [...]}. The model class comes from ``config.json``."""

from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--prompt", action="append", required=True, help="token ids separated by blanks; may be repeated")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--max-tokens", type=int, default=8192, help="tokens the live requests may hold in the cache")
    ap.add_argument("--max-requests", type=int, default=32)
    ap.add_argument("--step-tokens", type=int, default=2048, help="tokens per step (prompts are fed in portions)")
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)

    import torch

    from flashrec_b200 import _lib, build, registry
    from flashrec_b200.engine import LMEngine, generate
    from flashrec_b200.sampling import SamplingParams

    if "FLASHREC_B200_LIB" not in os.environ:
        _lib.use_library(build.build())
    prompts = [[int(t) for t in p.split()] for p in args.prompt]
    model = registry.load_model(args.model, getattr(torch, args.dtype), "cuda:0")
    longest = max(len(p) for p in prompts) + args.max_new_tokens
    engine = LMEngine(model, max(args.max_tokens, longest), args.max_requests, longest)
    out = generate(engine, prompts, args.max_new_tokens, SamplingParams(args.temperature, args.top_k, args.seed),
                   args.step_tokens)
    for i, toks in enumerate(out):
        print(json.dumps({"prompt": i, "tokens": toks}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
