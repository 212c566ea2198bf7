"""Replay given token ids through a model, step by step, and write logits (nothing is sampled).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Every line of standard input is a step, a JSON object: ``entries``, each a request ``id`` with its next
``tokens`` and the places ``want`` among them whose logits are asked for, and ``end``, the ids of
requests that are over after it.  A step with wanted logits writes ``OUT/<step>.f32``: little-endian
fp32 [wanted, vocab] in the order asked for.  ``done <step>`` is printed after each.  Requests come one
after the other, each through the engine that generates.  Exit code 3: the design has no fp32 form.

The kernels the design needs are compiled when they are missing or older than their sources.
"""

from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


def main() -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, default=32768, help="most tokens a request holds at any time")
    args = ap.parse_args()
    import torch
    from . import build
    from .engine import Engine
    from .registry import design_of_directory
    design, dtype = design_of_directory(args.model), getattr(torch, args.dtype)
    if dtype not in design.dtypes:
        print(f"{design.name} does not run in {args.dtype}", file=sys.stderr)
        return 3
    build.build(targets=design.libraries)
    out = Path(args.out)
    engine = Engine.from_pretrained(args.model, max_context=max(1, args.max_tokens), device="cuda", dtype=dtype)
    live = None
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for entry in step["entries"]:
            if not entry["tokens"]:
                continue
            if live is None:
                engine.reset()
                live = entry["id"]
            if entry["id"] != live:
                raise RuntimeError(f"request {entry['id']} while {live} is not over: one request at a time")
            rows.append(engine.extend(entry["tokens"], entry["want"]))
        if any(r.shape[0] for r in rows):
            (out / f"{step['step']}.f32").write_bytes(torch.cat(rows).cpu().numpy().astype("<f4").tobytes())
        if live in step["end"]:
            live = None
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
