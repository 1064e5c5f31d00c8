"""Replays a trace of token ids through a model and writes logits.

Steps come from standard input, one JSON object a line:

    {"step": 7, "entries": [{"id": "q1", "tokens": [101, 9], "want": [1]}], "end": ["q1"]}

An entry appends ``tokens`` to request ``id`` (what it fed before sits in the cache) and asks for the
logits behind the tokens numbered in ``want``; ``end`` lists requests whose cache slot is free again
after the step.  OUT/<step>.f32 receives the step's logits, f32 little-endian [wanted, vocab], and
``done <step>`` is printed when the step is complete.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

REFUSED = 3  # exit code: the model's class does not run in the type asked for


def _arguments(argv):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="cache positions to set aside")
    ap.add_argument("--max-requests", type=int, default=1, help="cache slots")
    ap.add_argument("--device", type=int, default=0)
    return ap.parse_args(argv)


def replay(runner, lines, out_dir: str, say=print) -> None:
    """Feeds the steps of ``lines`` to ``runner``."""
    live: dict[str, int] = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for entry in step["entries"]:
            name = entry["id"]
            if name not in live:
                live[name] = runner.open()
            logits = runner.feed(live[name], entry["tokens"], entry["want"])
            if len(entry["want"]):
                parts.append(logits)
        if parts:
            data = np.ascontiguousarray(np.concatenate(parts), dtype="<f4")
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(data.tobytes())
        for name in step.get("end", []):
            if name in live:
                runner.close(live.pop(name))
        say(f"done {step['step']}")


def main(argv=None) -> int:
    args = _arguments(argv)
    from . import _lib, build, registry
    from .api import Device
    name, _ = registry.identify(args.model)
    if args.dtype not in registry.ARCHITECTURES[name].dtypes:
        print(f"{name} models do not run in {args.dtype}", file=sys.stderr)
        return REFUSED
    _lib.use(build.ensure(registry.ARCHITECTURES[name].part))  # compiles in a fresh checkout
    runner = registry.load(Device(args.device), args.model, args.dtype, max_seq=args.max_tokens, max_batch=args.max_requests,
                           max_prefill=min(args.max_tokens, 2048))
    replay(runner, sys.stdin, args.out, lambda s: print(s, flush=True))
    return 0
