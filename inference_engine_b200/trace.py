"""Replay of recorded token streams: feeds given token ids through a model step by step and writes logits.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

One JSON object a line on standard input:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
entries: each request's next tokens and the places among them whose logits are wanted; end: requests that are finished
after the step.  A step with wanted places writes OUT/<step>.f32 (little-endian fp32 [wanted, vocab], in the order of the
entries and of `want`); after every step 'done <step>' is printed.  The engine's own step, cache, page pool and graphs
do the work (Engine.replay).
"""
from __future__ import annotations

import argparse
import json
import math
import os
import sys


def make_engine(model, max_tokens: int, max_batch: int):
    from .engine import Engine

    page = model.page_size
    max_len = max(page, math.ceil((max_tokens + 1) / page) * page)
    return Engine(model, max_batch_size=max_batch, max_len=max_len, stop_token_id=-1, page_size=page,
                  num_pages=math.ceil(min(512, max_len) / page) + math.ceil(max_tokens / page) + 2 * max_batch,
                  max_tokens_per_step=max_len + max_batch, min_first_chunk=1)


def run(engine, lines, out_dir: str, done) -> None:
    live = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_replay()
            entries.append((live[e["id"]], e["tokens"], e["want"]))
        logits = engine.replay(entries)
        if logits.shape[0]:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4", copy=False).tobytes())
            os.replace(path + ".part", path)
        for name in step["end"]:
            engine.close_replay(live.pop(name))
        bits = engine.K.check_status(engine.device)
        if bits:
            raise RuntimeError(f"device status word {bits:#x} after step {step['step']}")
        done(step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="feed recorded token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-batch", type=int, default=4, help="most entries of a step")
    a = ap.parse_args(argv)

    import torch

    from .models import load_model

    model = load_model(a.model, "cuda", getattr(torch, a.dtype))
    engine = make_engine(model, a.max_tokens, a.max_batch)
    run(engine, sys.stdin, a.out, lambda n: print(f"done {n}", flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
