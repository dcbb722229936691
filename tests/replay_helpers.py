"""Driving the engine over given tokens, and comparing what comes out: shared by the tests of the assembled decoders."""
from __future__ import annotations

import json

import torch

from mini_vllm_b200.config import Config


def write_checkpoint(path, cfg: dict, weights: dict) -> str:
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(weights, str(path / "model.safetensors"))
    return str(path)


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per row: RMS difference with the mean taken off, relative to the RMS of all wanted logits."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()


def make_engine(path, dtype, blocks=12, slots=4, seqs=4, **extra):
    from mini_vllm_b200.engine.engine import Engine
    return Engine(Config(model=path, dtype=dtype, kv_cache_num_blocks=blocks, kv_cache_block_size=128, max_model_len=1024,
                         max_num_batched_seqs=seqs, num_state_slots=slots, gpu_memory_utilization=0.5, **extra))


def feed(eng, prompts, plan):
    """Runs a plan - steps of (prompt index, number of tokens) - and returns each prompt's logits; a prompt fed to its end
    gives its memory back at once."""
    from mini_vllm_b200.engine.request import Request
    live, at, got = {}, {}, {}
    for step in plan:
        entries = []
        for i, n in step:
            lo = at.get(i, 0)
            at[i] = lo + n
            entries.append((live.setdefault(i, Request([])), prompts[i][lo:lo + n], list(range(n))))
        out, row = eng.replay_step(entries).cpu(), 0
        for i, n in step:
            got.setdefault(i, []).append(out[row:row + n])
            row += n
            if at[i] == len(prompts[i]):
                eng.release(live.pop(i))
                at.pop(i)
    eng.executor.check_device_status()
    bm = eng.scheduler.block_manager
    if not live:                                                     # everything was given back
        assert bm.num_free_blocks == bm.capacity
        assert bm.state_slots is None or bm.state_slots.num_free == bm.state_slots.capacity
    return {i: torch.cat(v) for i, v in got.items()}


def portions(n, sizes):
    out = []
    while sum(out) < n:
        out.append(min(sizes[len(out) % len(sizes)], n - sum(out)))
    return out


def assert_tokens(got, want, margin):
    """Equal until the oracle's own two best logits come closer than rounding can keep apart."""
    compared = 0
    for toks, (ref, margins) in zip(got, want):
        for t, r, m in zip(toks, ref, margins):
            if m < margin:
                break
            assert t == r
            compared += 1
    return compared
