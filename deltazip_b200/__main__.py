"""Command line of the framework.

    python -m deltazip_b200 models
    python -m deltazip_b200 generate --model DIR --prompt "1 2 3" [--prompt ...] --max-new 16
    python -m deltazip_b200 replay   --model DIR --out DIR < steps

Prompts and results are token ids (there is no tokenizer here)."""
from __future__ import annotations

import argparse
import json
import sys


def cmd_models(args) -> int:
    from . import registry
    for name in registry.names():
        print(name)
    return 0


def cmd_generate(args) -> int:
    import torch

    from . import build
    build.build_library()
    from . import registry
    from .engine import DecodeEngine
    dtype = getattr(torch, args.dtype) if args.dtype else None
    cfg, model = registry.load_model(args.model, dtype=dtype)
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in args.prompt]
    longest = max(len(p) for p in prompts) + args.max_new
    block = 16
    eng = DecodeEngine(cfg, None, args.max_seqs, args.max_seqs * -(-longest // block), block, model=model)
    for ids in eng.generate(prompts, args.max_new, stop_id=args.stop_id):
        print(json.dumps(ids))
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv[:1] == ["replay"]:
        from .replay import main as replay
        return replay(argv[1:])
    ap = argparse.ArgumentParser(prog="deltazip_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    sub.add_parser("models", help="list the architectures the registry knows").set_defaults(fn=cmd_models)
    g = sub.add_parser("generate", help="greedy generation from a checkpoint folder")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt", action="append", required=True, help="token ids; repeat for a batch")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--max-seqs", type=int, default=16)
    g.add_argument("--stop-id", type=int, default=None)
    g.add_argument("--dtype", choices=["bfloat16", "float16", "float32"], default=None)
    g.set_defaults(fn=cmd_generate)
    sub.add_parser("replay", help="replay given tokens, write logits (see replay --help)")
    args = ap.parse_args(argv)
    return args.fn(args)


if __name__ == "__main__":
    sys.exit(main())
