"""Command line:

    python -m inference_engine_b200 models
    python -m inference_engine_b200 build [--force]
    python -m inference_engine_b200 generate --model DIR --prompt "5 17 3" [--prompt ...] [--max-new-tokens N] [--tau T]

Prompts are token ids (there is no tokenizer); a prompt that starts with @ names a file of them, one prompt a line.
"""
from __future__ import annotations

import argparse
import json
import sys


def read_prompts(args: list[str]) -> list[list[int]]:
    lines = []
    for p in args:
        if p.startswith("@"):
            with open(p[1:]) as f:
                lines += [x for x in f if x.strip()]
        else:
            lines.append(p)
    return [[int(t) for t in x.replace(",", " ").split()] for x in lines]


def generate(a) -> int:
    import torch

    from .engine import Engine
    from .models import load_model

    prompts = read_prompts(a.prompt)
    model = load_model(a.model, "cuda", getattr(torch, a.dtype), a.random_weights)
    if any(not p or any(not 0 <= t < model.vocab for t in p) for p in prompts):
        raise SystemExit(f"a prompt is empty or has ids outside 0 .. {model.vocab - 1}")
    longest = max(len(p) for p in prompts) + a.max_new_tokens
    engine = Engine(model, max_batch_size=a.max_batch, max_len=a.max_len or max(longest, model.page_size), stop_token_id=a.stop_token,
                    max_tokens_per_step=max(a.max_tokens_per_step, a.max_batch + 64), tau=a.tau, seed=a.seed)
    for r in engine.generate(prompts, a.max_new_tokens):
        print(json.dumps({"id": r.id, "prompt_tokens": len(r.prompt_ids), "output": r.output,
                          "seconds": round(r.t_finish - r.t_submit, 4)}), flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="inference_engine_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    sub.add_parser("models", help="list the architectures of the registry")
    b = sub.add_parser("build", help="compile the CUDA libraries")
    b.add_argument("--force", action="store_true")
    g = sub.add_parser("generate", help="continue prompts of token ids with a model folder")
    g.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    g.add_argument("--prompt", action="append", required=True, help="token ids, or @file with one prompt a line; may repeat")
    g.add_argument("--max-new-tokens", type=int, default=16)
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--tau", type=float, default=0.0, help="sampling temperature, 0 = greedy")
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--stop-token", type=int, default=-1)
    g.add_argument("--max-batch", type=int, default=16)
    g.add_argument("--max-len", type=int, default=0, help="longest request; default: what the prompts need")
    g.add_argument("--max-tokens-per-step", type=int, default=1024)
    g.add_argument("--random-weights", action="store_true", help="random weights of the configuration's sizes")
    a = ap.parse_args(argv)
    if a.command == "models":
        from .models import load_all

        print("\n".join(sorted(load_all())))
        return 0
    if a.command == "build":
        from . import build

        build.build(force=a.force)
        return 0
    return generate(a)


if __name__ == "__main__":
    sys.exit(main())
