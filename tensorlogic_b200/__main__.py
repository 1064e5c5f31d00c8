"""Command line.

    python -m tensorlogic_b200 generate --model PATH --prompt 1,15,7 [--new 32] [--dtype D]
                                        [--temperature T --seed S] [--max-seq N]
    python -m tensorlogic_b200 info --model PATH

PATH is a GGUF file or a folder with config.json and model.safetensors; prompts and output are token ids.
"""
from __future__ import annotations

import argparse
import sys

from . import registry
from .api import Device, TensorError


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="tensorlogic_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="continue a prompt of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt", required=True, help="token ids, separated by commas")
    g.add_argument("--new", type=int, default=32, help="tokens to generate")
    g.add_argument("--dtype", default=None)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--max-seq", type=int, default=None, help="cache positions (default: what the call needs)")
    g.add_argument("--device", type=int, default=0)
    i = sub.add_parser("info", help="which model class serves the files")
    i.add_argument("--model", required=True)
    args = ap.parse_args(argv)
    try:
        if args.command == "info":
            name, _ = registry.identify(args.model)
            print(f"{name}: runs in {', '.join(registry.ARCHITECTURES[name].dtypes)}")
            return 0
        prompt = [int(t) for t in args.prompt.split(",") if t.strip()]
        need = len(prompt) + args.new
        runner = registry.load(Device(args.device), args.model, args.dtype, max_seq=args.max_seq or need,
                               max_prefill=min(len(prompt), 4096))
        if args.temperature > 0:
            runner.set_sampling(args.temperature, args.seed)
        for token in registry.generate(runner, prompt, args.new):
            print(token, flush=True)
        return 0
    except TensorError as e:
        print(e, file=sys.stderr)
        return 1


if __name__ == "__main__":
    sys.exit(main())
