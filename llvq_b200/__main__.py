"""Command line: `python -m llvq_b200 generate|models|build ...` (trace replay is bin/trace_run)."""
from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m llvq_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="greedy continuation of token ids")
    g.add_argument("--model", required=True, help="sealed archive file, or folder with config.json and model.safetensors")
    g.add_argument("--tokens", required=True, help="prompt token ids, separated by commas")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--dtype", default="", help="element type (default: the architecture's own)")
    g.add_argument("--capacity", type=int, default=0, help="tokens the cache holds (default: prompt and new tokens)")
    g.add_argument("--prefill-chunk", type=int, default=2048, help="most tokens of a prompt portion")
    g.add_argument("--eager", action="store_true", help="launch every token step instead of replaying its CUDA graph")
    sub.add_parser("models", help="list the known architectures")
    sub.add_parser("build", help="compile the CUDA libraries")
    args = ap.parse_args(argv)
    if args.cmd == "models":
        from .registry import architectures
        for a in {id(a): a for a in architectures().values()}.values():
            print(f"{a.name}: {a.container}, {', '.join(a.dtypes)}")
        return 0
    if args.cmd == "build":
        from . import _build
        for lib in _build.SOURCES:
            print(_build.build(lib=lib))
        return 0
    from .registry import load_model
    prompt = [int(t) for t in args.tokens.split(",")]
    model = load_model(args.model, args.capacity or len(prompt) + args.max_new, args.dtype, prefill_chunk=args.prefill_chunk)
    print(json.dumps({"tokens": model.generate(prompt, args.max_new, use_graph=not args.eager)}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
