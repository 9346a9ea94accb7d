"""Replays a trace of token ids through a model and writes the logits asked for.

Standard input has one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
Each entry's tokens continue the sequence of that id; `want` names places among them.  <out>/<step>.f32 receives the wanted rows,
in order, as little-endian f32 [wanted, vocab]; then `done <step>` is printed.  The sequences in `end` give their pages back.
Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and .safetensors weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits, one file per step that asks for some")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live sequences hold at any time")
    args = ap.parse_args(argv)
    import torch

    from . import registry
    from .engine import Engine

    dtype = getattr(torch, args.dtype)
    arch = registry.ARCHITECTURES[registry.architecture_of(registry.read_config(args.model))]
    if dtype not in arch.dtypes:
        print(f"this model does not run in {args.dtype}", file=sys.stderr)
        return 3
    tokens = max(args.max_tokens, 1)
    engine = Engine(registry.load(args.model, dtype=dtype, max_len=tokens, cache_tokens=tokens, max_tokens=min(2048, tokens)))
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = engine.feed([(e["id"], e["tokens"], e["want"]) for e in step["entries"]])
        if any(len(e["want"]) for e in step["entries"]):
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                for r in rows:
                    f.write(r.numpy().astype("<f4").tobytes())
        for key in step["end"]:
            engine.close(key)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
