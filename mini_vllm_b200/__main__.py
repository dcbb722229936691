"""Offline generation from a checkpoint directory.

    python -m mini_vllm_b200 --model DIR --prompt "1 5 9" [--prompt ...] [--max-tokens N] [--temperature T --top-k K --top-p P]

Prompts are token ids, or text where the checkpoint comes with a tokenizer.  One JSON line per prompt.
"""
from __future__ import annotations

import argparse
import json
import sys


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="mini_vllm_b200", description="generate from a checkpoint directory")
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="token ids (or text, with a tokenizer); repeatable")
    ap.add_argument("--dtype", default=None, choices=["bfloat16", "float32"])
    ap.add_argument("--max-tokens", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--ignore-eos", action="store_true")
    ap.add_argument("--max-model-len", type=int, default=4096)
    ap.add_argument("--chunked-prefill", action="store_true", help="prompts enter in portions of the token budget")
    ap.add_argument("--max-batched-tokens", type=int, default=16384)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    import torch
    from .config import Config, SamplingParams
    from .engine.engine import Engine
    engine = Engine(Config(model=args.model, dtype=getattr(torch, args.dtype) if args.dtype else None,
                           max_model_len=args.max_model_len, max_num_batched_tokens=args.max_batched_tokens,
                           max_num_batched_seqs=max(8, len(args.prompt)), enable_chunked_prefill=args.chunked_prefill, seed=args.seed))
    encode = (lambda p: [int(t) for t in p.split()]) if engine.tokenizer is None else engine.tokenizer.encode
    params = SamplingParams(temperature=args.temperature, max_tokens=args.max_tokens, top_k=args.top_k, top_p=args.top_p,
                            ignore_eos=args.ignore_eos)
    for prompt, out in zip(args.prompt, engine.generate([encode(p) for p in args.prompt], params, use_tqdm=False)):
        print(json.dumps({"prompt": prompt, **{k: v for k, v in out.items() if k != "prompt"}}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
