"""Replays a trace of given tokens through the engine, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come as JSON lines on standard input::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` are one batch: each request's next tokens, and the places among them whose logits are wanted; ``end`` lists
requests whose memory is given back after the step.  A step in which something is wanted writes ``OUT/<step>.f32`` (fp32,
little-endian, [wanted, vocab], in the order of the entries and places); every step is acknowledged with ``done <step>``.

The pool holds N tokens in requests' counts of 64 (each request rounded up to the engine's own block size), and there are
four state slots: requests that do not fit are an error, so blocks and slots must have been given back in time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

LIVE_REQUESTS = 4
BLOCK = 128                 # the smallest block the prefill kernel takes
COUNT = 64                  # granularity of --max-tokens


def pool_blocks(max_tokens: int) -> int:
    """Blocks for requests of ``max_tokens`` tokens in all, counted in 64s, when each is rounded up to a block instead."""
    return max(1, (max_tokens + LIVE_REQUESTS * (BLOCK - COUNT)) // BLOCK)


def make_engine(model: str, dtype: str, max_tokens: int):
    import torch
    from .config import Config
    from .engine.engine import Engine
    torch.set_float32_matmul_precision("highest")
    return Engine(Config(model=model, dtype=getattr(torch, dtype), kv_cache_num_blocks=pool_blocks(max_tokens),
                         kv_cache_block_size=BLOCK, max_model_len=-(-max_tokens // COUNT) * COUNT,
                         max_num_batched_seqs=LIVE_REQUESTS, num_state_slots=LIVE_REQUESTS, gpu_memory_utilization=0.8))


def replay(engine, lines, out_dir: str, acknowledge) -> None:
    from .engine.request import Request
    live: dict[str, Request] = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            entries.append((live.setdefault(e["id"], Request([])), e["tokens"], e.get("want", [])))
        logits = engine.replay_step(entries) if entries else None
        if logits is not None:
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(logits.cpu().numpy().astype("<f4").tobytes())
        for name in step.get("end", []):
            engine.release(live.pop(name))
        engine.executor.check_device_status()
        acknowledge(step["step"])


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of given tokens and write logits")
    ap.add_argument("--model", required=True, help="checkpoint directory")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold, in 64s")
    args = ap.parse_args(argv)
    from .csrc.build import build
    build()
    engine = make_engine(args.model, args.dtype, args.max_tokens)
    replay(engine, sys.stdin, args.out, lambda n: print(f"done {n}", flush=True))
    return 0
