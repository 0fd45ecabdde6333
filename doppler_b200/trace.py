"""Replays a trace of token ids through a model and writes logits; nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

An entry runs a request's next tokens; ``want`` lists places among them whose logits are written to OUT/<step>.f32
(little-endian f32, [wanted, vocab], in the order of entries and places).  Requests in ``end`` are finished after the
step.  Every step is answered with a line ``done <step>``.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def run_step(scheduler, step: dict, out_dir: str):
    rows = []
    for e in step.get("entries", []):
        want = e.get("want") or []
        got = scheduler.step(e["id"], e["tokens"], want)
        if want:
            rows.append(got)
    if rows:
        path = os.path.join(out_dir, f"{step['step']}.f32")
        with open(path + ".part", "wb") as f:
            f.write(np.concatenate(rows).astype("<f4").tobytes())
        os.replace(path + ".part", path)
    for request in step.get("end", []):
        scheduler.finish(request)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="model folder")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens live requests hold at any time")
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)

    from . import build

    build.build()  # compiles what is missing or out of date
    from .ops import Device
    from .registry import load_model
    from .scheduler import Scheduler

    device = Device(args.device)
    model = load_model(device, args.model, max_seq=max(args.max_tokens, 1), dtype=args.dtype)
    scheduler = Scheduler(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        run_step(scheduler, step, args.out)
        print(f"done {step['step']}", flush=True)
    model.destroy()
    device.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
