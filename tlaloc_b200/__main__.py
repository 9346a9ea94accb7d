"""The command line: python -m tlaloc_b200 generate | trace | models ...

    python -m tlaloc_b200 models
    python -m tlaloc_b200 generate --model DIR --max-new 32 --prompt 5,17,3 --prompt 9,9,1
    python -m tlaloc_b200 trace --model DIR --dtype float32 --out DIR --max-tokens 4096 < steps
"""
from __future__ import annotations

import argparse
import json
import sys


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="tlaloc_b200 generate", description="greedy continuations of token-id prompts")
    ap.add_argument("--model", required=True, help="folder with config.json and .safetensors weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--prompt", action="append", default=[], help="token ids with commas between them; may be repeated")
    ap.add_argument("--prompts", help="file with one JSON list of token ids a line")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--stop", type=int, action="append", default=[], help="a token id that ends a continuation")
    ap.add_argument("--max-len", type=int, default=4096, help="longest sequence, prompt and continuation")
    ap.add_argument("--cache-tokens", type=int, help="tokens the cache holds (default: four sequences of --max-len)")
    args = ap.parse_args(argv)
    import torch

    from . import registry
    from .engine import Engine

    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    if args.prompts:
        with open(args.prompts) as f:
            prompts += [json.loads(line) for line in f if line.strip()]
    if not prompts:
        ap.error("no prompt")
    engine = Engine(registry.load(args.model, dtype=getattr(torch, args.dtype), max_len=args.max_len, cache_tokens=args.cache_tokens))
    for out in engine.generate(prompts, args.max_new, args.stop):
        print(json.dumps(out))
    return 0


def models(argv) -> int:
    from . import registry

    for name, arch in sorted(registry.ARCHITECTURES.items()):
        print(name, *(str(d).replace("torch.", "") for d in arch.dtypes))
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    from . import trace

    commands = {"generate": generate, "trace": trace.main, "models": models}
    if not argv or argv[0] not in commands:
        print(__doc__, file=sys.stderr)
        return 2
    return commands[argv[0]](argv[1:])


if __name__ == "__main__":
    sys.exit(main())
