"""Replays a trace of token ids through a model, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Reads one JSON object a line from standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

For a step that wants something it writes OUT/<step>.f32, the logits in the order of entries and ``want`` as
little-endian 32-bit floats; after every step it prints ``done <step>``. Requests in ``end`` give back what they hold.
The first call in a checkout compiles the part of the kernel library that the model needs."""

from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path

EXIT_NO_SUCH_DTYPE = 3


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096)
    ap.add_argument("--max-requests", type=int, default=32)
    args = ap.parse_args(argv)

    import torch

    from flashrec_b200 import _lib, build, registry
    from flashrec_b200.engine import LMEngine, StepEntry

    family = registry.lookup(registry.read_config(args.model))
    dtype = getattr(torch, args.dtype)
    if dtype not in family.dtypes:
        print(f"{family.name} does not run in {args.dtype}", file=sys.stderr)
        return EXIT_NO_SUCH_DTYPE
    if "FLASHREC_B200_LIB" not in os.environ:
        _lib.use_library(build.build() if family.sources is None else build.build_subset(family.name, family.sources))
    out = Path(args.out)
    model = registry.load_model(args.model, dtype, "cuda:0")
    engine = LMEngine(model, args.max_tokens, max_requests=args.max_requests)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = engine.step([StepEntry(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]])
        if logits.shape[0]:
            data = logits.float().cpu().numpy().astype("<f4", copy=False)
            (out / f"{step['step']}.f32").write_bytes(data.tobytes())
        for req in step.get("end", []):
            engine.finish(req)
        torch.cuda.synchronize()
        print(f"done {step['step']}", flush=True)
    if _lib.device_status() != (0, 0):
        print("a kernel reported a timeout", file=sys.stderr)
        return 1
    return 0


if __name__ == "__main__":
    sys.exit(main())
