"""Command line over the serving loop.

    python -m wayruntime_b200.cli models
    python -m wayruntime_b200.cli generate --model DIR --prompt 1,2,3 [--prompt 7,8] --max-new 16

A model folder has no tokenizer: prompts and results are token ids.
"""
from __future__ import annotations

import argparse
import json
import sys


def generate(a) -> int:
    from . import models
    from .binding import Context
    from .engine import Engine, Request, Sampling
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    longest = max(len(p) for p in prompts) + a.max_new
    ctx = Context(a.device, attn_max_seq=max(longest, 64))
    model = models.load(ctx, a.model, a.dtype, a.max_rows)
    reqs = [Request(p, a.max_new, Sampling(a.temperature, a.top_k, a.top_p, a.seed + i), frozenset(a.stop))
            for i, p in enumerate(prompts)]
    try:
        for r in Engine(model).run(reqs):
            print(json.dumps({"prompt": r.prompt, "output": r.output}))
    finally:
        model.close()
        ctx.close()
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="wayruntime_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    sub.add_parser("models", help="list the architectures the registry knows")
    g = sub.add_parser("generate", help="generate from prompts of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--prompt", action="append", required=True, help="comma-separated ids; may be given several times")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--max-rows", type=int, default=2048, help="tokens of a prompt per pass")
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--stop", type=int, action="append", default=[])
    g.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    if a.command == "models":
        from . import models
        print("\n".join(models.architectures()))
        return 0
    return generate(a)


if __name__ == "__main__":
    sys.exit(main())
