"""Replay a trace of given tokens and write logits: `bin/trace_run`.

One JSON object a line on standard input, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: the next
tokens of a request and the places among them whose logits are asked for, then the requests that are finished. A
step that asks for something writes <out>/<step>.f32 ([wanted, vocab] little-endian 32-bit floats); every step prints
"done <step>". The tokens go through `TokenLoop.feed`: the prompt path and the token step (replayed from its CUDA
graph) that generation uses. A model holds one live sequence; requests follow one another.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def run(model, lines, out_dir: str, out=sys.stdout) -> None:
    import numpy as np
    live = None
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            if live is not None and live != e["id"]:
                raise ValueError(f"step {step['step']}: request {e['id']} while {live} holds the cache")
            live = e["id"]
            y = model.feed(e["tokens"], e.get("want", ()))
            if y is not None:
                rows.append(y.float().cpu().numpy())
        for name in step.get("end", ()):
            if name == live:
                model.release()
                live = None
        if rows:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            np.concatenate(rows).astype("<f4").tofile(path + ".part")
            os.replace(path + ".part", path)
        print(f"done {step['step']}", file=out, flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed given tokens through a model, step by step, and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a sealed archive")
    ap.add_argument("--dtype", default="", help="element type (default: the architecture's own); exit code 3 where the model does not run in it")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens the live request holds: sizes the cache")
    args = ap.parse_args(argv)
    from .registry import UnsupportedDtype, load_model
    try:
        model = load_model(args.model, max(1, args.max_tokens), args.dtype)
    except UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    run(model, sys.stdin, args.out)
    return 0
