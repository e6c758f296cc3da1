"""Command line: ``python -m tensorwarp_b200 generate|trace|models``."""
from __future__ import annotations

import argparse
import json
import sys


def _generate(args) -> int:
    import torch

    from . import registry
    from .scheduler import Scheduler
    options = {"max_live": args.max_live}
    if args.max_tokens:
        options["max_tokens"] = args.max_tokens
    engine = registry.load(args.model, dtype={"bfloat16": torch.bfloat16, "float32": torch.float32}[args.dtype], **options)
    scheduler = Scheduler(engine, portion=args.portion)
    index = {}
    for i, text in enumerate(args.tokens):
        request = scheduler.submit([int(t) for t in text.split(",")], args.max_new_tokens, args.stop_token)
        index[id(request)] = i
    for request in scheduler.run():
        print(json.dumps({"request": index[id(request)], "generated": request.generated}), flush=True)
    return 0


def _models(args) -> int:
    from . import registry
    print("\n".join(registry.architectures()))
    return 0


def _trace(args) -> int:
    from . import trace
    return trace.main(args)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="tensorwarp_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy generation from token ids")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--tokens", required=True, action="append", help="a prompt as comma-separated token ids (repeat for more)")
    g.add_argument("--max-new-tokens", type=int, default=16)
    g.add_argument("--stop-token", type=int, default=None)
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--max-tokens", type=int, default=None, help="longest sequence to make room for")
    g.add_argument("--max-live", type=int, default=4, help="sequences in flight at once")
    g.add_argument("--portion", type=int, default=2048, help="most prompt tokens per step")
    g.set_defaults(run=_generate)
    t = sub.add_parser("trace", help="replay a trace of steps from standard input and write the logits it asks for")
    t.add_argument("--model", required=True)
    t.add_argument("--dtype", choices=["bfloat16", "float32"], required=True)
    t.add_argument("--out", required=True, help="folder for <step>.f32")
    t.add_argument("--max-tokens", type=int, required=True, help="room for this many tokens per sequence")
    t.set_defaults(run=_trace)
    m = sub.add_parser("models", help="list the architectures")
    m.set_defaults(run=_models)
    args = ap.parse_args(argv)
    return args.run(args)


if __name__ == "__main__":
    sys.exit(main())
