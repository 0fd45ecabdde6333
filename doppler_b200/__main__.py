"""Command line.

    python -m doppler_b200 generate --model DIR --prompt 5,17,3 [--prompt ...] --max-new 32 [--dtype float32]
    python -m doppler_b200 trace --model DIR --dtype bfloat16 --out DIR --max-tokens N < steps
    python -m doppler_b200 info --model DIR

Prompts are token ids (the package has no tokenizer); generation is greedy.
"""
from __future__ import annotations

import argparse
import json
import sys

from . import trace


def _ids(text: str):
    return [int(t) for t in text.replace(",", " ").split()]


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="doppler_b200 generate")
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", required=True, action="append", type=_ids, help="token ids, comma separated; may be given several times")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--stop", type=_ids, default=[], help="token ids that end a sequence")
    ap.add_argument("--batch", type=int, default=0, help="sequences decoded together (default: all prompts, at most 256)")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)
    from . import build

    build.build()
    from .ops import Device
    from .registry import load_model
    from .scheduler import Scheduler

    device = Device(args.device)
    batch = args.batch or min(len(args.prompt), 256)
    model = load_model(device, args.model, max(len(p) for p in args.prompt) + args.max_new, batch, args.dtype)
    for prompt, new in zip(args.prompt, Scheduler(model).generate(args.prompt, args.max_new, args.stop)):
        print(json.dumps({"prompt": prompt, "tokens": new}), flush=True)
    model.destroy()
    device.close()
    return 0


def info(argv) -> int:
    ap = argparse.ArgumentParser(prog="doppler_b200 info")
    ap.add_argument("--model", required=True)
    args = ap.parse_args(argv)
    from . import registry

    d = registry.describe(args.model)
    if d["kind"] in registry.ARCHITECTURES:
        stack, layers = registry.ARCHITECTURES[d["kind"]].describe(args.model, d["config"])
        print(json.dumps({"kind": d["kind"], "stack": stack, "layers": layers}))
    else:
        print(json.dumps(d))
    return 0


COMMANDS = {"generate": generate, "trace": trace.main, "info": info}


def main() -> int:
    if len(sys.argv) < 2 or sys.argv[1] not in COMMANDS:
        print(__doc__.strip(), file=sys.stderr)
        return 2
    return COMMANDS[sys.argv[1]](sys.argv[2:])


if __name__ == "__main__":
    sys.exit(main())
