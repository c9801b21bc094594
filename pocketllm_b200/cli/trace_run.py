"""Replay a trace of token ids through a model, step by step, and write the logits that the trace asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is a step: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}. The
entries of a step run as one batch through the same step function, cache manager and kernels that generation uses; nothing
is sampled. Wanted logits go to OUT/<step>.f32 (little-endian fp32, [wanted, vocab]), `done <step>` is printed after every
step, and requests named in `end` give back their slot and pages.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

MAX_REQUESTS = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", required=True, type=int, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    import torch
    from ..models import registry
    from ..ops import lib
    from ..runtime.mixer_runtime import StepEntry
    lib.use_kernel_set("mixer")
    rt = registry.build_runtime(args.model, dtype=getattr(torch, args.dtype), max_requests=MAX_REQUESTS, max_tokens=args.max_tokens)
    out = Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [StepEntry(e["id"], e["tokens"], e["want"]) for e in step["entries"]]
        logits = rt.step(entries)
        if any(len(e.want) for e in entries):
            (out / f"{step['step']}.f32").write_bytes(logits.float().cpu().numpy().astype("<f4").tobytes())
        rt.check_status()
        for rid in step["end"]:
            rt.release(rid)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
