#!/usr/bin/env python
"""Benchmark of the ragged continuous-batching attention path on B200.

    python bench.py --gpus N --steps K --warmup W [--impl reference]

Workload (``config.workload``): Qwen3-0.6B-shape random-init model, greedy decoding, continuous batching.
Default: the per-GPU share of the box-scale offline-serving job the headline metric is quoted on
(4096 requests over 8 GPUs = 512 requests per GPU, prompt lengths log-uniform [32,4096], output lengths
U[64,1024], random token ids); ``--workload config2`` selects the 64-request job (prompt U[100,1024],
prompt+output <= 1024).  One "step" is one complete generation job over the rank's request set.  At
N > 1 each rank is an independent engine replica (no collective on the data path); the global list of
512*N requests is partitioned by the host dispatcher by token count, so per-GPU work is fixed (weak
scaling) and N = 8 is exactly the 4096-request job.

Metric: prompt+generated tokens per second, whole job, all GPUs.
* ``value``: the job's device time, CUDA events around its first and last kernel (the engine's step loop
  is pipelined: sampled ids stay in HBM and feed the next step's packing kernel).
* ``e2e``: the same job through ``Engine.generate`` with host token lists in and out (wall clock:
  request submission, every step's metadata upload, every step's token read-back and the final list
  assembly are inside the timed region).
* ``roofline``: decode attention kernel, the largest kernel of the step: K/V bytes of the contexts
  it read / CUDA-event time, replayed on contexts recorded during the job, against the measured
  HBM copy bandwidth.  ``kernels`` adds the same figure on the fixed 240-sequence decode batch
  (contexts U[128,4096]) and the prefill kernel's TFLOP/s.
* ``cpu_baseline`` / ``--impl reference``: the oracle restatement of the reference's PyTorch path
  timed on the host cores on a bounded sample of the same workload (per-token extrapolation).
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import time
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

from mini_vllm_b200.config import Config, SamplingParams, qwen3_shape  # noqa: E402
from mini_vllm_b200.dispatcher import partition_by_tokens, request_cost  # noqa: E402
from mini_vllm_b200.workloads import (GEMMA3_1B, QWEN3_0P6B, config2_requests, config3, config4,  # noqa: E402
                                       decode_kv_bytes, prefill_flops)

METRIC = "ragged prefill+decode tokens/s (Qwen3-0.6B shapes, continuous batching, greedy)"
WORKLOADS = {
    "config5": "config5 share: Qwen3-0.6B random-init, 512 req/GPU (one of the 8 shares of 4096 requests per GPU), "
               "prompt log-U[32,4096], output U[64,1024], continuous batching",
    "config2": "config2: Qwen3-0.6B random-init, 64 req/GPU, prompt U[100,1024], total<=1024, continuous batching",
}


def workload_requests(workload: str, world: int = 1, rank: int = 0):
    """The requests of one replica.

    Requests are split by token count - the K/V tokens a request will have read by its end, one context per
    generated token: out * (prompt + out / 2).  (The plain prompt + output sum balances the token totals to
    0.01 % but leaves the replicas' attention work 3 % apart, and a job is bound by its slowest replica.)
    Config 5 is 4096 requests over 8 GPUs: it is cut into its 8 shares once, and a run on N GPUs takes the
    first N of them, so every replica's job is the same at every N."""
    kv_tokens = lambda r: request_cost(len(r.prompt), r.max_tokens)
    if workload == "config5" and world <= 8:
        from mini_vllm_b200.workloads import config5_requests
        all_reqs, parts = config5_requests(seed=0, n=4096), 8
    elif workload == "config5":
        from mini_vllm_b200.workloads import config5_requests
        all_reqs, parts = config5_requests(seed=0, n=512 * world), world
    else:
        all_reqs, parts = config2_requests(seed=0, n=64 * world), world
    return [all_reqs[i] for i in partition_by_tokens([kv_tokens(r) for r in all_reqs], parts)[rank]]


def measured_peaks() -> tuple[dict, str]:
    p = ROOT / "MEASURED_PEAKS.json"
    if p.exists():
        return json.loads(p.read_text()), "measured"
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}, "fallback"


class ClockSampler:
    QUERY = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.gpu, self.proc = gpu_index, None
        self.file = tempfile.NamedTemporaryFile("w+", suffix=".csv", delete=False)

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                          "-lms", "200", "-i", str(self.gpu)], stdout=self.file, stderr=subprocess.DEVNULL)
        except OSError:
            self.proc = None

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        self.file.flush()
        rows = [r.split(", ") for r in Path(self.file.name).read_text().strip().splitlines() if r.count(",") >= 8]
        os.unlink(self.file.name)
        if not rows:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["no samples"]}
        sm = [float(r[1]) for r in rows]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = sorted({n for r in rows for n, v in zip(names, r[5:9]) if v.strip().lower().startswith("active")})
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": float(rows[0][2]), "samples": len(rows),
                "power_w_max": max(float(r[3]) for r in rows), "reasons": reasons}


# ---------------------------------------------------------------------------------------------------
def build_config(workload: str = "config5") -> Config:
    if workload == "config5":        # long prompts, hundreds of live sequences: a large pool, preemption allowed
        # up to 512 live sequences (the reference's default max_num_batched_seqs), all decode batches from graphs
        return Config(hf_config=qwen3_shape(), kv_cache_num_blocks=4096,
                      max_num_batched_seqs=512, max_graph_batch_size=512,
                      max_num_batched_tokens=16384, gpu_memory_utilization=0.85, use_cuda_graph=True, seed=0)
    return Config(hf_config=qwen3_shape(), kv_cache_num_blocks=512, max_num_batched_seqs=64,
                  max_num_batched_tokens=16384, gpu_memory_utilization=0.5, use_cuda_graph=True, seed=0)


def build_engine(local_rank: int, workload: str = "config5", mixed_steps: bool = False, fused_head: bool = True):
    import dataclasses
    from mini_vllm_b200.engine.engine import Engine
    torch.cuda.set_device(local_rank)
    return Engine(dataclasses.replace(build_config(workload), enable_mixed_steps=mixed_steps, fused_greedy_head=fused_head))


class ContextSpy:
    """Records the contexts of every 40th decode step of a job (for the in-situ roofline replay)."""

    def __init__(self, executor, sink):
        self.ex, self.sink, self.count, self.orig = executor, sink, 0, executor.launch

    def __enter__(self):
        if self.sink is not None:
            def spy(batch, slots):
                if batch.type == 1:
                    if self.count % 40 == 20:
                        self.sink.append(([len(r.tokens) for r in batch.requests], [list(r.blocks) for r in batch.requests]))
                    self.count += 1
                return self.orig(batch, slots)
            self.ex.launch = spy
        return self

    def __exit__(self, *exc):
        self.ex.launch = self.orig
        return False


def run_job(engine, reqs, record_contexts=None, group=None):
    """One generation job through the public API; returns (tokens processed, wall seconds, this rank's cuda ms).

    ``group is None``: this process's ``Engine.generate`` on ``reqs``.  Otherwise a collective over the ranks of
    ``group``: rank 0 holds ``reqs`` (ALL requests of the job), the host dispatcher scatters the shares, every rank
    generates, rank 0 gathers and merges; the wall time on rank 0 covers all of it and the token count is taken from
    the merged results (other ranks return 0 tokens).
    """
    prompts = params = None
    if reqs is not None:
        prompts = [r.prompt for r in reqs]
        params = [SamplingParams(max_tokens=r.max_tokens, ignore_eos=True) for r in reqs]
    torch.cuda.synchronize()
    with ContextSpy(engine.executor, record_contexts):
        t0 = time.perf_counter()
        if group is None:
            out = engine.generate(prompts, params, use_tqdm=False)
        else:
            from mini_vllm_b200.dispatcher import generate_over_ranks
            out = generate_over_ranks(engine, prompts, params, group=group)
        torch.cuda.synchronize()
        wall = time.perf_counter() - t0
    n_tok = 0
    if out is not None:
        n_tok = sum(len(p) for p in prompts) + sum(len(o["tokens"]) for o in out)
        assert all(len(o["tokens"]) == r.max_tokens for o, r in zip(out, reqs))
    return n_tok, wall, engine.last_job_device_ms


def decode_roofline(engine, contexts, peaks):
    """Replay the decode-attention kernel on recorded step contexts over the engine's own KV pool."""
    from mini_vllm_b200 import ops
    from mini_vllm_b200.workloads import table_tensor
    ex = engine.executor
    dev, hf = ex.device, engine.config.hf_config
    hq, hkv, d, layers = hf.num_attention_heads, hf.num_key_value_heads, hf.head_dim, hf.num_hidden_layers
    total_bytes = total_ms = 0.0
    launches = 0
    for lens, blocks in contexts:
        b = len(lens)
        q = torch.randn(b, hq, d, device=dev, dtype=torch.bfloat16)
        seqlens = torch.tensor(lens, dtype=torch.int32, device=dev)
        bt = table_tensor(blocks).to(dev)
        ws = ops.decode_workspace(b, hq, d, dev)
        out = torch.empty_like(q)
        ops.decode_plan(seqlens, -1, hq, hkv, d, ws, block_table=bt, block_size=256)
        def all_layers():                                        # distinct layer pools: no L2 reuse between launches
            for layer in range(layers):
                ops.decode_attn(q, ex.kv_cache[0, layer], ex.kv_cache[1, layer], seqlens, bt, d ** -0.5, -1, ws, out=out)
        all_layers()                                             # warm-up, also outside any capture
        torch.cuda.synchronize()
        # launch the 28 layers back to back from a CUDA graph, as the engine does, so that the
        # event-to-event time is device time and not the host's launch rate
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            all_layers()
        graph.replay()
        reps = 3
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(reps):
            graph.replay()
        e1.record()
        torch.cuda.synchronize()
        total_ms += e0.elapsed_time(e1) / reps
        total_bytes += layers * decode_kv_bytes(QWEN3_0P6B, lens)
        launches += layers
    achieved = total_bytes / (total_ms * 1e-3) / 1e9 if total_ms else 0.0
    return {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
            "frac": round(achieved / peaks["hbm_gbs"], 4),
            # ncu on the 2.063 GB config-3 launch read 2.0733 GB and wrote 5.8 MB (profiles/): traffic is
            # 1.008 x the algorithmic bytes and grows in proportion, so it is scaled to this launch size
            "traffic": int(1.008 * total_bytes / max(launches, 1)), "kernel": "decode_attn_kernel<128,8>",
            "launches_timed": launches, "avg_launch_us": round(total_ms * 1e3 / max(launches, 1), 2),
            "avg_bytes_per_launch": int(total_bytes / max(launches, 1)),
            "note": "algorithmic K+V bytes of recorded decode steps, 28 layer launches replayed from a CUDA graph; peak = STREAM copy"}


LEGS = ("attn3", "prefill", "attn4", "sampler", "rope", "pack", "head", "glue")


def graph_time_ms(sweep, launches_per_sweep: int, reps: int = 5) -> float:
    """Device time per launch of ``sweep`` (a function that enqueues ``launches_per_sweep`` kernels over
    distinct buffers), replayed from a CUDA graph so that short kernels are not timed at the host's launch rate."""
    sweep()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        sweep()
    graph.replay()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        graph.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / (reps * launches_per_sweep)


def rope_and_pack_legs(dev, peaks, legs) -> dict:
    """The elementwise and integer kernels of the path on config-3 / config-5 sized steps."""
    from mini_vllm_b200 import ops
    from mini_vllm_b200.models.layers.rotary import build_cos_sin_cache
    import numpy as np
    out = {}
    hq, hkv, d = 16, 8, 128
    case, g = config3()
    q_lens = [n - c for n, c in zip(case.prefill_lens, case.prefill_cached)]
    if "rope" in legs:
        table = build_cos_sin_cache(d, 8192, 1e6).to(dev)
        wq = torch.ones(d, device=dev, dtype=torch.bfloat16)
        for name, tokens in (("prefill12784", sum(q_lens)), ("decode512", 512)):
            nbuf = max(2, min(8, int(400e6 / (tokens * (hq + 2 * hkv) * d * 2))))
            qkvs = [torch.randn(tokens, (hq + 2 * hkv) * d, device=dev).to(torch.bfloat16) for _ in range(nbuf)]
            pools = [torch.zeros(2, tokens // 256 + 2, 256, hkv, d, device=dev, dtype=torch.bfloat16) for _ in range(nbuf)]
            pos = torch.arange(tokens, device=dev, dtype=torch.int64) % 4096
            slots = torch.randperm(tokens, device=dev).to(torch.int32)          # every token its own slot, scattered
            views = [tuple(t.view(tokens, -1, d) for t in x.split([hq * d, hkv * d, hkv * d], dim=-1)) for x in qkvs]
            # q, k, v read where the projection left them; q written back in place, k and v to their cache slots
            byts = tokens * (hq + 2 * hkv) * d * 2 * 2
            for kern, call in (("rope_kv_write", lambda v3, p: ops.rope_kv_write(v3[0], v3[1], v3[2], pos, table, slots, p[0], p[1], k_in_place=False)),
                               ("qk_norm_rope_kv_write", lambda v3, p: ops.qk_norm_rope_kv_write(v3[0], v3[1], v3[2], wq, wq, 1e-6, False, pos, table, slots, p[0], p[1], k_in_place=False))):
                ms = graph_time_ms(lambda: [call(v3, p) for v3, p in zip(views, pools)], nbuf)
                out[f"{kern}_{name}"] = {"GB/s": round(byts / ms / 1e6, 1), "us": round(ms * 1e3, 2), "bytes": byts,
                                         "frac_of_measured_hbm": round(byts / ms / 1e6 / peaks["hbm_gbs"], 4)}
            del qkvs, pools, views
    if "glue" in legs:
        # the decoder glue between the GEMMs on config 3's prefill rows (Qwen3-0.6B: hidden 1024, intermediate 3072)
        hidden, inter = 1024, 3072
        for name, tokens in (("prefill12784", sum(q_lens)), ("decode512", 512)):
            nbuf = max(2, min(8, int(400e6 / (tokens * inter * 6))))
            gus = [torch.randn(tokens, 2 * inter, device=dev).to(torch.bfloat16) for _ in range(nbuf)]
            outs = [torch.empty(tokens, inter, device=dev, dtype=torch.bfloat16) for _ in range(nbuf)]
            byts = tokens * inter * 2 * 3
            ms = graph_time_ms(lambda: [ops.act_mul(gu, inter, False, out=o) for gu, o in zip(gus, outs)], nbuf)
            out[f"act_mul_{name}"] = {"GB/s": round(byts / ms / 1e6, 1), "us": round(ms * 1e3, 2), "bytes": byts,
                                      "frac_of_measured_hbm": round(byts / ms / 1e6 / peaks["hbm_gbs"], 4)}
            del gus, outs
            nbuf = 8
            xs = [torch.randn(tokens, hidden, device=dev).to(torch.bfloat16) for _ in range(nbuf)]
            ys = [torch.randn(tokens, hidden, device=dev).to(torch.bfloat16) for _ in range(nbuf)]
            os_ = [torch.empty(tokens, hidden, device=dev, dtype=torch.bfloat16) for _ in range(nbuf)]
            w = torch.ones(hidden, device=dev, dtype=torch.bfloat16)
            byts = tokens * hidden * 2 * 4                     # x and y read, x and the normed row written
            ms = graph_time_ms(lambda: [ops.add_rmsnorm(x, y, w, 1e-6, False, out=o) for x, y, o in zip(xs, ys, os_)], nbuf)
            out[f"add_rmsnorm_{name}"] = {"GB/s": round(byts / ms / 1e6, 1), "us": round(ms * 1e3, 2), "bytes": byts,
                                          "frac_of_measured_hbm": round(byts / ms / 1e6 / peaks["hbm_gbs"], 4)}
            del xs, ys, os_
    if "pack" in legs:
        # prefill packing of config 3's 16 prompts (12 784 new tokens, cached prefixes) and decode packing of 512 rows
        seq_len = np.asarray(case.prefill_lens, np.int32)
        cached = np.asarray(case.prefill_cached, np.int32)
        nblk = np.asarray([len(b) for b in case.prefill_blocks], np.int32)
        blk_off = np.concatenate([[0], np.cumsum(nblk)]).astype(np.int32)
        blocks = np.concatenate([np.asarray(b, np.int32) for b in case.prefill_blocks])
        t = int((seq_len - cached).sum())
        toks = torch.randint(0, 151936, (t,), generator=g).numpy().astype(np.int32)
        meta = torch.from_numpy(np.concatenate([seq_len, cached, blk_off, blocks, toks])).to(dev)
        ms = graph_time_ms(lambda: [ops.pack_prefill(meta, 16, t, int(blk_off[-1]), int(nblk.max()), 256, True) for _ in range(8)], 8)
        out["pack_prefill_config3"] = {"us": round(ms * 1e3, 2), "tokens": t, "out_bytes": t * 20 + 16 * int(nblk.max()) * 4}
        b = 512
        ctx = torch.randint(32, 5120, (b,), generator=g).numpy().astype(np.int32)
        nb = (ctx + 255) // 256
        off = np.concatenate([[0], np.cumsum(nb)]).astype(np.int32)
        flat = np.arange(int(off[-1]), dtype=np.int32)
        meta = torch.from_numpy(np.concatenate([ctx, off, flat, np.zeros(b, np.int32), np.full(b, -1, np.int32)])).to(dev)
        ids, pos = torch.empty(b, dtype=torch.int64, device=dev), torch.empty(b, dtype=torch.int64, device=dev)
        slot, lens = torch.empty(b, dtype=torch.int32, device=dev), torch.empty(b, dtype=torch.int32, device=dev)
        table = torch.empty(b, 4096, dtype=torch.int32, device=dev)[:, :int(nb.max())]   # row stride of a graph runner's table
        ms = graph_time_ms(lambda: [ops.pack_decode(meta, b, int(off[-1]), int(nb.max()), 256, ids, pos, slot, lens, table)
                                    for _ in range(8)], 8)
        out["pack_decode_512"] = {"us": round(ms * 1e3, 2), "rows": b, "out_bytes": b * (8 + 8 + 4 + 4 + int(nb.max()) * 4)}
    return out


def head_legs(dev, peaks) -> dict:
    """lm_head + greedy sampling on Qwen3's head (hidden 1024, vocabulary 151 936): the fused kernel against the
    cuBLAS GEMM followed by the greedy sampler.  The floor of either is reading the 311 MB weight matrix once."""
    from mini_vllm_b200 import ops
    out = {}
    hidden, vocab = 1024, 151936
    ws = [(torch.randn(vocab, hidden, device=dev) * 0.02).to(torch.bfloat16) for _ in range(2)]   # 2 x 311 MB > L2
    for rows in (512, 256, 128, 64):
        xs = [torch.randn(rows, hidden, device=dev).to(torch.bfloat16) for _ in range(2)]
        scratch = ops.lm_head_argmax_scratch(rows, dev)
        tok = torch.empty(rows, dtype=torch.int64, device=dev)
        logits = torch.empty(rows, vocab, dtype=torch.bfloat16, device=dev)
        flops, w_bytes = 2 * rows * hidden * vocab, vocab * hidden * 2

        def unfused():
            for x, w in zip(xs, ws):
                torch.matmul(x, w.t(), out=logits)
                ops.sample(logits, out=tok)
        ms_fused = graph_time_ms(lambda: [ops.lm_head_argmax(x, w, scratch, out=tok) for x, w in zip(xs, ws)], 2)
        ms_unfused = graph_time_ms(unfused, 2)
        out[f"lm_head_argmax_{rows}"] = {"us": round(ms_fused * 1e3, 1), "unfused_us": round(ms_unfused * 1e3, 1),
                                         "TFLOP/s": round(flops / ms_fused / 1e9, 1),
                                         "weight_GB/s": round(w_bytes / ms_fused / 1e6, 1),
                                         "frac_of_measured_bf16": round(flops / ms_fused / 1e9 / peaks["bf16_tflops"], 4),
                                         "frac_of_measured_hbm": round(w_bytes / ms_fused / 1e6 / peaks["hbm_gbs"], 4)}
    return out


def kernel_extras(dev, peaks, nl=4, legs=LEGS):
    """Fixed single-layer cases: the 240-sequence decode batch and the 16-sequence prefill batch.

    ``nl`` distinct KV pools (2.3 GB each) are rotated so that consecutive launches share nothing in L2.
    """
    out = {}
    if "attn3" in legs or "prefill" in legs:
        out.update(attention_legs_qwen3(dev, peaks, nl, legs))
    if "attn4" in legs:
        out.update(decode_legs_gemma3(dev, peaks, nl))
    if "sampler" in legs:
        out.update(sampler_legs(dev, peaks))
    out.update(rope_and_pack_legs(dev, peaks, legs))
    if "head" in legs:
        out.update(head_legs(dev, peaks))
    return out


def decode_leg_config3(dev, peaks, nl, case, pools, out):
    from mini_vllm_b200 import ops
    from mini_vllm_b200.workloads import table_tensor
    hq, hkv, d = 16, 8, 128
    # decode part
    b = len(case.decode_ctx)
    q = torch.randn(b, hq, d, device=dev, dtype=torch.bfloat16)
    lens = torch.tensor(case.decode_ctx, dtype=torch.int32, device=dev)
    bt = table_tensor(case.decode_blocks).to(dev)
    ws = ops.decode_workspace(b, hq, d, dev)
    o = torch.empty_like(q)
    ops.decode_plan(lens, -1, hq, hkv, d, ws, block_table=bt, block_size=256)
    ms = event_time_ms(lambda i: ops.decode_attn(q, pools[i % nl][0], pools[i % nl][1], lens, bt, d ** -0.5, -1, ws, out=o),
                       24, warm=8)
    byts = decode_kv_bytes(QWEN3_0P6B, case.decode_ctx)
    gbs = byts / ms / 1e6
    out["decode_attn_config3"] = {"GB/s": round(gbs, 1), "us": round(ms * 1e3, 1), "bytes": byts,
                                  "frac_of_measured_hbm": round(gbs / peaks["hbm_gbs"], 4),
                                  "frac_of_8TBs_nominal": round(gbs / 8000.0, 4)}
    return out


def event_time_ms(call, iters: int, warm: int = 3) -> float:
    """Median device time of ``call(i)`` over ``iters`` launches, CUDA events on the launching stream."""
    for i in range(warm):
        call(i)
    evs = [torch.cuda.Event(enable_timing=True) for _ in range(iters + 1)]
    evs[0].record()
    for i in range(iters):
        call(i)
        evs[i + 1].record()
    torch.cuda.synchronize()
    return statistics.median(evs[i].elapsed_time(evs[i + 1]) for i in range(iters))


def attention_legs_qwen3(dev, peaks, nl, legs):
    from mini_vllm_b200 import ops
    from mini_vllm_b200.workloads import table_tensor
    case, _ = config3()
    hq, hkv, d = 16, 8, 128
    pools = [torch.randn(2, case.pool_blocks, 256, hkv, d, device=dev, dtype=torch.bfloat16) for _ in range(nl)]
    out = {}
    if "attn3" in legs:
        decode_leg_config3(dev, peaks, nl, case, pools, out)
    if "prefill" not in legs:
        return out
    cu = lambda xs: torch.tensor([0] + list(torch.tensor(xs).cumsum(0)), dtype=torch.int32, device=dev)
    # prefill part (paged, half the sequences with a cached 512-token prefix)
    q_lens = [n - c for n, c in zip(case.prefill_lens, case.prefill_cached)]
    qp = torch.randn(sum(q_lens), hq, d, device=dev, dtype=torch.bfloat16)
    btp = table_tensor(case.prefill_blocks).to(dev)
    cq, ck = cu(q_lens), cu(case.prefill_lens)
    # the launch's work list, built on the host from the lengths as the executor does while packing the step
    rows = ops.prefill_item_rows(hq, hkv, d)
    work = lambda ql, kl: torch.from_numpy(ops.build_prefill_items(ql, kl, rows)).to(dev)
    items = work(q_lens, case.prefill_lens)
    fl = prefill_flops(QWEN3_0P6B, case.prefill_lens, case.prefill_cached)
    for name, it in (("prefill_attn_config3", items), ("prefill_attn_config3_no_list", None)):
        ms = event_time_ms(lambda i: ops.prefill_attn(qp, pools[i % nl][0], pools[i % nl][1], cq, ck, max(q_lens), d ** -0.5,
                                                      -1, block_table=btp, items=it), 10)
        tf = fl / ms / 1e9
        out[name] = {"TFLOP/s": round(tf, 1), "us": round(ms * 1e3, 1), "flops": fl,
                     "frac_of_measured_bf16": round(tf / peaks["bf16_tflops"], 4)}
    del pools
    # the same kernel on long and on short prompts (dense K/V): 4 x 8192 and 32 x 1024 tokens
    for name, (nseq, slen) in (("prefill_attn_4x8192", (4, 8192)), ("prefill_attn_32x1024", (32, 1024))):
        lens_p = [slen] * nseq
        qd = torch.randn(nseq * slen, hq, d, device=dev, dtype=torch.bfloat16)
        kd = torch.randn(nseq * slen, hkv, d, device=dev, dtype=torch.bfloat16)
        vd = torch.randn(nseq * slen, hkv, d, device=dev, dtype=torch.bfloat16)
        cd = cu(lens_p)
        fl = prefill_flops(QWEN3_0P6B, lens_p, [0] * nseq)
        for key, it in ((name, work(lens_p, lens_p)), (name + "_no_list", None)):
            ms = event_time_ms(lambda i: ops.prefill_attn(qd, kd, vd, cd, cd, slen, d ** -0.5, -1, items=it), 10)
            out[key] = {"TFLOP/s": round(fl / ms / 1e9, 1), "us": round(ms * 1e3, 1), "flops": fl,
                        "frac_of_measured_bf16": round(fl / ms / 1e9 / peaks["bf16_tflops"], 4)}
        del qd, kd, vd
    return out


def decode_legs_gemma3(dev, peaks, nl):
    """Gemma3-1B shapes (4 q heads, 1 kv head, head_dim 256), 128 sequences, contexts U[512,4096]: a global layer
    and a sliding-window-512 layer (window layers count only the visible keys)."""
    from mini_vllm_b200 import ops
    from mini_vllm_b200.workloads import table_tensor
    out = {}
    g4, _ = config4()
    hq, hkv, d = 4, 1, 256
    gpools = [torch.randn(2, g4.pool_blocks, 256, hkv, d, device=dev, dtype=torch.bfloat16) for _ in range(max(nl, 2) * 2)]
    b = len(g4.decode_ctx)
    q = torch.randn(b, hq, d, device=dev, dtype=torch.bfloat16)
    lens = torch.tensor(g4.decode_ctx, dtype=torch.int32, device=dev)
    bt = table_tensor(g4.decode_blocks).to(dev)
    o = torch.empty_like(q)
    for name, window in (("decode_attn_config4_global", -1), ("decode_attn_config4_window512", 512)):
        ws = ops.decode_workspace(b, hq, d, dev)
        ops.decode_plan(lens, window, hq, hkv, d, ws, block_table=bt, block_size=256)
        ms = graph_time_ms(lambda: [ops.decode_attn(q, gp[0], gp[1], lens, bt, d ** -0.5, window, ws, out=o) for gp in gpools],
                           len(gpools))
        byts = decode_kv_bytes(GEMMA3_1B, g4.decode_ctx, window)
        gbs = byts / ms / 1e6
        out[name] = {"GB/s": round(gbs, 1), "us": round(ms * 1e3, 1), "bytes": byts,
                     "frac_of_measured_hbm": round(gbs / peaks["hbm_gbs"], 4)}
    return out


def sampler_legs(dev, peaks):
    """The sampler over Qwen3's vocabulary: the 512-row and the 64-row decode batch, greedy and top-k/top-p."""
    from mini_vllm_b200 import ops
    out = {}
    vocab = 151936
    for rows in (512, 64):
        bufs = [torch.randn(rows, vocab, device=dev).to(torch.bfloat16) for _ in range(max(2, min(16, int(600e6 / (rows * vocab * 2)))))]
        temps = torch.full((rows,), 0.8, device=dev)
        topk = torch.full((rows,), 50, dtype=torch.int32, device=dev)
        topp = torch.full((rows,), 0.9, device=dev)
        for name, call in ((f"sample_greedy_{rows}", lambda x: ops.sample(x)),
                           (f"sample_top50_p0.9_{rows}", lambda x: ops.sample(x, temps, topk, 1, 0, top_p=topp))):
            ms = graph_time_ms(lambda: [call(x) for x in bufs], len(bufs))       # distinct buffers: nothing comes from L2
            byts = rows * vocab * 2
            out[name] = {"GB/s": round(byts / ms / 1e6, 1), "us": round(ms * 1e3, 1), "bytes": byts,
                         "frac_of_measured_hbm": round(byts / ms / 1e6 / peaks["hbm_gbs"], 4)}
    return out


def config3_engine_step(mixed: bool) -> dict:
    """Config 3 through the engine (28 layers): 240 requests decoding at contexts U[128,4096] when 16 prompts
    arrive, 8 of them sharing a resident 512-token prefix (prefix cache on).  With mixed steps that is ONE
    forward pass; the reference's scheduler makes it a prefill step followed by a decode step."""
    import dataclasses
    from mini_vllm_b200.engine.engine import Engine
    case, g = config3()
    cfg = Config(hf_config=qwen3_shape(), kv_cache_num_blocks=2400, max_num_batched_seqs=512, max_graph_batch_size=256,
                 max_num_batched_tokens=20480, enable_prefix_cache=True, enable_mixed_steps=mixed,
                 gpu_memory_utilization=0.85, use_cuda_graph=True, seed=0)
    eng = Engine(cfg)
    vocab = cfg.hf_config.vocab_size
    tok = lambda n: torch.randint(0, vocab, (int(n),), generator=g).tolist()
    long_run = SamplingParams(max_tokens=4096, ignore_eos=True)
    shared = tok(512)
    warm = eng.submit(shared + tok(8), SamplingParams(max_tokens=1, ignore_eos=True))   # leaves the prefix resident
    while not eng.finished:
        eng.step()
    for c in case.decode_ctx:                      # the decoding population: prompts one token short of the context
        eng.submit(tok(c - 1), long_run)
    while eng.scheduler.waiting:
        eng.step()
    for _ in range(3):                             # settle: a few decode steps (graphs warm)
        eng.step()
    for i, (n, c) in enumerate(zip(case.prefill_lens, case.prefill_cached)):
        eng.submit((shared if c else []) + tok(n - c), long_run)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    steps, new_tokens, kinds = 0, 0, []
    while eng.scheduler.waiting or (not mixed and kinds[-1] != 1):   # the plain scheduler needs a decode step after
        b = eng.step()
        kinds.append(b.type)
        bp = len(b.requests) - b.num_decode
        new_tokens += sum(len(r.tokens) - 1 - r.num_cached_tokens for r in b.requests[:bp]) + b.num_decode
        steps += 1
    e1.record()
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1)
    eng.executor.check_device_status()
    return {"mixed_steps": mixed, "steps": steps, "step_types": kinds, "ms": round(ms, 3), "tokens": new_tokens,
            "tokens_per_s": round(new_tokens / ms * 1e3, 1)}


def config4_engine_step() -> dict:
    """Config 4 through the engine: Gemma3-1B shapes (26 layers, 4 global / 22 window-512), 128 requests
    decoding at contexts U[512,4096].  Device time of a decode step = (job with 65 generated tokens - job with
    1) / 64, both through the pipelined loop with CUDA graphs."""
    from mini_vllm_b200.config import gemma3_shape
    from mini_vllm_b200.engine.engine import Engine
    case, g = config4()
    cfg = Config(hf_config=gemma3_shape(), kv_cache_num_blocks=1400, max_num_batched_seqs=128, max_graph_batch_size=128,
                 max_num_batched_tokens=16384, gpu_memory_utilization=0.85, use_cuda_graph=True, seed=0)
    eng = Engine(cfg)
    vocab = cfg.hf_config.vocab_size
    prompts = [torch.randint(0, vocab, (int(c) - 1,), generator=g).tolist() for c in case.decode_ctx]
    times = {}
    for n in (1, 65, 1, 65):
        eng.generate(prompts, SamplingParams(max_tokens=n, ignore_eos=True), use_tqdm=False)
        times[n] = eng.last_job_device_ms
    step_ms = (times[65] - times[1]) / 64
    ctx_mid = [c + 32 for c in case.decode_ctx]
    byts = 4 * decode_kv_bytes(GEMMA3_1B, ctx_mid, -1) + 22 * decode_kv_bytes(GEMMA3_1B, ctx_mid, 512)
    return {"decode_step_ms": round(step_ms, 4), "sequences": len(prompts), "kv_bytes_per_step": byts,
            "kv_GB/s_over_whole_step": round(byts / step_ms / 1e6, 1), "tokens_per_s": round(len(prompts) / step_ms * 1e3, 1),
            "prefill_job_ms": round(times[1], 2)}


def config2_parity() -> dict:
    """First-32-token greedy identity on the real config-2 shape against the committed reference tokens
    (tests/golden/config2_tokens.npz: the reference's own engine loop on a B200, prompts screened for a top-1/top-2
    margin of more than one bf16 step at every step of the reference)."""
    import numpy as np
    from mini_vllm_b200.engine.engine import Engine
    z = np.load(ROOT / "tests" / "golden" / "config2_tokens.npz")
    cuts = np.concatenate([[0], np.cumsum(z["prompt_lens"])])
    prompts = [z["prompts_flat"][a:b].tolist() for a, b in zip(cuts[:-1], cuts[1:])]
    eng = Engine(build_config("config2"))
    out = eng.generate(prompts, SamplingParams(max_tokens=32, ignore_eos=True), use_tqdm=False)
    got = np.asarray([o["tokens"] for o in out], dtype=np.int32)
    same = (got == z["ref_tokens"]).all(axis=1)
    return {"prompts": len(prompts), "tokens_per_prompt": 32, "identical_prompts": int(same.sum()),
            "identical_tokens": int((got == z["ref_tokens"]).sum()), "reference": str(z["reference_kind"]),
            "min_reference_margin_bf16_steps": float(z["ref_margin_ulps"].min()),
            "screen": {"candidates": int(z["candidates"]), "pass_product_margin": int(z["pass_product_margin"]),
                       "pass_both_margins": int(z["pass_both_margins"]),
                       "differ_after_screen": int(z["mismatches_after_screen"])},
            "unscreened_identical_of_64": int(z["unscreened_identical"])}


# ---- Fupupel: prefill and decode beside the closest existing model, and the kernels of its own ----------------
FUPUPEL_SIZES = {      # width, heads / KV heads (128 wide), feed-forward, layers (half of them selective scans)
    "w1024": (1024, 16, 8, 3072, 12), "w2048": (2048, 16, 8, 6144, 12), "w4096": (4096, 32, 8, 12288, 8)}


def fupupel_bench_shape(size: str, window: int = 1024):
    from mini_vllm_b200.config import fupupel_shape
    width, heads, kv, ff, layers = FUPUPEL_SIZES[size]
    scan = {"type": "mamba1", "mixer": {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}, "mlp": None}
    both = {"type": "parallel", "mlp": {"kind": "dense", "ff": ff, "limit": 7.0},
            "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "mask": {"size": window},
                               "rot": {"base": 1e6, "dims": 128}, "scale": 128 ** -0.5, "softcap": 30.0},
                      "right": {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4, "decay_rank": 128,
                                "gate_rank": 128}, "left_scale": 0.5, "right_scale": 0.5}}
    return fupupel_shape([scan if i % 2 == 0 else both for i in range(layers)], width, 32768)


def engine_throughput(models) -> dict:
    """Prefill (8 prompts of 2048 tokens) and decode (32 and 256 sequences) through ``Engine.generate`` with random weights, for each
    (name, model description)."""
    from mini_vllm_b200.engine.engine import Engine
    out = {}
    for name, hf in models:
        eng = Engine(Config(hf_config=hf, kv_cache_num_blocks=1024, max_num_batched_seqs=256, max_graph_batch_size=256,
                            max_num_batched_tokens=16384, gpu_memory_utilization=0.85, seed=0))
        params = sum(p.numel() for p in eng.executor.model.parameters())
        job = lambda n, length, new: (eng.generate([[(7 * i + j) % 32768 for j in range(length)] for i in range(n)],
                                                   SamplingParams(max_tokens=new, ignore_eos=True), use_tqdm=False),
                                      eng.last_job_device_ms)[1]
        med = lambda *a: statistics.median(job(*a) for _ in range(3))
        job(8, 2048, 1)
        row = {"parameters": params, "prefill_tok_s": round(8 * 2048 / med(8, 2048, 1) * 1e3)}
        for n in (32, 256):
            job(n, 512, 2)
            row[f"decode{n}_step_ms"] = round((med(n, 512, 65) - med(n, 512, 1)) / 64, 4)
            row[f"decode{n}_tok_s"] = round(n / row[f"decode{n}_step_ms"] * 1e3)
        out[name] = row
        del eng
        torch.cuda.empty_cache()
    return out


def qwen3_twin(size: str):
    width, heads, kv, ff, layers = FUPUPEL_SIZES[size]
    return qwen3_shape(num_hidden_layers=layers, hidden_size=width, intermediate_size=ff, num_attention_heads=heads,
                       num_key_value_heads=kv, vocab_size=32768)


def fupupel_throughput(sizes=tuple(FUPUPEL_SIZES)) -> dict:
    """Beside Qwen3 layers of the same width, heads, feed-forward and count."""
    return engine_throughput((f"{size}_{name}", hf) for size in sizes
                             for name, hf in (("fupupel", fupupel_bench_shape(size)), ("qwen3", qwen3_twin(size))))


class Legs:
    """Kernels against their rooflines: each leg is timed from a CUDA graph over ``nbuf`` launches on buffers of their own."""

    def __init__(self, dev, peaks):
        self.peaks, self.rows = peaks, {}
        self.sms, self.ghz = torch.cuda.get_device_properties(dev).multi_processor_count, 1.9

    def __call__(self, name, call, nbuf, byts=None, flops=None, mufu=None, fp32=None):
        ms = graph_time_ms(lambda: [call(i) for i in range(nbuf)], nbuf)
        row = {"us": round(ms * 1e3, 2)}
        if byts:
            row.update({"GB/s": round(byts / ms / 1e6, 1), "frac_of_measured_hbm": round(byts / ms / 1e6 / self.peaks["hbm_gbs"], 4)})
        if flops:
            row.update({"TFLOP/s": round(flops / ms / 1e9, 1), "frac_of_measured_bf16": round(flops / ms / 1e9 / self.peaks["bf16_tflops"], 4)})
        if mufu:
            row["frac_of_special_function_rate"] = round(mufu / (self.sms * 16 * self.ghz * 1e9) / (ms * 1e-3), 4)
        if fp32:
            row["frac_of_fp32_fma_rate"] = round(fp32 / (self.sms * 128 * self.ghz * 1e9) / (ms * 1e-3), 4)
        self.rows[name] = row


def fupupel_kernel_legs(dev, peaks) -> dict:
    """Each kernel of the design against its roofline, next to the like kernel of the existing models where there is one.
    16 heads of 128 (8 KV heads), width 2048, scan of 4096 channels x 16 states, 8192 prefill tokens, 256 decode rows."""
    from mini_vllm_b200 import ops
    bf, leg = torch.bfloat16, Legs(dev, peaks)
    rnd = lambda *shape, scale=1.0: (torch.randn(*shape, device=dev) * scale).to(bf)
    heads, kv, d, width, ff, window = 16, 8, 128, 2048, 6144, 1024
    for tag, lens in (("4x2048", [2048] * 4), ("1x8192", [8192])):
        tokens = sum(lens)
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        pos = torch.cat([torch.arange(n, device=dev) for n in lens])
        q, k, v = rnd(tokens, heads, d), rnd(tokens, kv, d), rnd(tokens, kv, d)
        pairs = sum(sum(min(i + 1, window) for i in range(n)) for n in lens)
        for name, cap in (("prefill_attn_window1024", 0.0), ("prefill_attn_window1024_capped", 30.0)):
            leg(f"{name}_{tag}", lambda i: ops.prefill_attn(q, k, v, cu, cu, max(lens), d ** -0.5, window - 1, softcap=cap), 4,
                flops=4 * heads * d * pairs)
        full = sum(n * (n + 1) // 2 for n in lens)
        for name, cap in (("prefill_attn_full", 0.0), ("prefill_attn_full_capped", 30.0)):
            leg(f"{name}_{tag}", lambda i: ops.prefill_attn(q, k, v, cu, cu, max(lens), d ** -0.5, -1, softcap=cap), 4,
                flops=4 * heads * d * full)
        inner, n = 4096, 16
        state = torch.zeros(len(lens), inner, n, device=dev)
        slots = torch.arange(len(lens), dtype=torch.int32, device=dev)
        u, dt, z, y = (rnd(tokens, inner) for _ in range(4))
        bc = rnd(tokens, 2 * n)
        a = -torch.arange(1, n + 1, device=dev).float().expand(inner, n).contiguous() * 1.44
        bias, skip = torch.full((inner,), -4.0, device=dev), torch.ones(inner, device=dev)
        leg(f"selective_scan_{tag}", lambda i: ops.selective_scan(u, dt, z, bc[:, :n], bc[:, n:], bias, a, skip, y, state, slots,
                                                                  cu, pos), 2,
            byts=tokens * (inner * 4 + 2 * n) * 2, mufu=tokens * inner * n)
        w4, cstate = rnd(4, inner), torch.zeros(len(lens), 3, inner, device=dev, dtype=bf)
        leg(f"short_conv_{tag}", lambda i: ops.short_conv_silu(u, w4, None, cstate, slots, cu, pos), 4, byts=tokens * inner * 4)
        qd, kd, vd, gate, od = (rnd(tokens, heads, d) for _ in range(5))
        raw_a, raw_b = rnd(tokens, heads * d), rnd(tokens, heads)
        ea, db, nw = torch.rand(heads, device=dev) * 8 + 1, torch.full((heads * d,), -4.0, device=dev), torch.ones(d, device=dev)
        dstate = torch.zeros(len(lens), heads, d, d, device=dev)
        leg(f"gated_delta_{tag}", lambda i: ops.gated_delta(qd, kd, vd, raw_a, raw_b, gate.flatten(1), ea, db, nw, od, dstate,
                                                            slots, cu, pos, d ** -0.5, 1e-6), 1,
            byts=tokens * heads * d * 6 * 2, fp32=tokens * heads * d * d * 4)
    tokens = 8192
    gu = [rnd(tokens, 2 * ff) for _ in range(2)]
    leg("act_mul_8192", lambda i: ops.act_mul(gu[i], ff, False), 2, byts=tokens * ff * 6)
    leg("clamped_glu_8192", lambda i: ops.clamped_glu(gu[i], ff, 7.0, 1.702), 2, byts=tokens * ff * 6)
    del gu
    w, ys = torch.ones(width, device=dev, dtype=bf), [rnd(tokens, width) for _ in range(4)]
    xs16, xs32 = [rnd(tokens, width) for _ in range(4)], [torch.randn(tokens, width, device=dev) for _ in range(4)]
    leg("add_rmsnorm_branch_norm_8192", lambda i: ops.add_rmsnorm(xs16[i], ys[i], w, 1e-6, True, y_weight=w), 4, byts=tokens * width * 8)
    leg("residual_norm_f32_8192", lambda i: ops.residual_norm(xs32[i], ys[i], w, 1e-6, y_weight=w), 4, byts=tokens * width * 12)
    # decode: 256 sequences, contexts of 1024 and more (a window layer reads 1024 keys of each)
    b, blocks = 256, 256 * 5
    pools = [torch.randn(2, blocks, 256, kv, d, device=dev, dtype=bf) for _ in range(2)]
    lens = torch.full((b,), 1200, dtype=torch.int32, device=dev)
    bt = torch.arange(blocks, dtype=torch.int32, device=dev).view(b, 5)
    q, o = rnd(b, heads, d), rnd(b, heads, d)
    ws = ops.decode_workspace(b, heads, d, dev)
    ops.decode_plan(lens, window - 1, heads, kv, d, ws, block_table=bt, block_size=256)
    for name, cap in (("decode_attn_window1024", 0.0), ("decode_attn_window1024_capped", 30.0)):
        leg(f"{name}_256", lambda i: ops.decode_attn(q, pools[i][0], pools[i][1], lens, bt, d ** -0.5, window - 1, ws, out=o,
                                                     softcap=cap), 2, byts=b * window * 2 * kv * d * 2)
    del pools
    pos, slots = torch.full((b,), 1199, device=dev), torch.arange(b, dtype=torch.int32, device=dev)
    inner, n = 4096, 16
    states = [torch.randn(b, inner, n, device=dev) for _ in range(4)]
    u, dt, z, y, bc = rnd(b, inner), rnd(b, inner), rnd(b, inner), rnd(b, inner), rnd(b, 2 * n)
    a = -torch.arange(1, n + 1, device=dev).float().expand(inner, n).contiguous() * 1.44
    bias, skip = torch.full((inner,), -4.0, device=dev), torch.ones(inner, device=dev)
    leg("selective_scan_decode256", lambda i: ops.selective_scan(u, dt, z, bc[:, :n], bc[:, n:], bias, a, skip, y, states[i], slots,
                                                                 None, pos), 4, byts=b * inner * n * 8)
    del states
    dstates = [torch.randn(b, heads, d, d, device=dev) * 0.01 for _ in range(2)]
    qd, kd, vd, gate, od = (rnd(b, heads, d) for _ in range(5))
    raw_a, raw_b = rnd(b, heads * d), rnd(b, heads)
    ea, db, nw = torch.rand(heads, device=dev) * 8 + 1, torch.full((heads * d,), -4.0, device=dev), torch.ones(d, device=dev)
    leg("gated_delta_decode256", lambda i: ops.gated_delta(qd, kd, vd, raw_a, raw_b, gate.flatten(1), ea, db, nw, od, dstates[i],
                                                           slots, None, pos, d ** -0.5, 1e-6), 2, byts=b * heads * d * d * 8)
    w4, cstate, uc = rnd(4, 6144), torch.zeros(b, 3, 6144, device=dev, dtype=bf), rnd(b, 6144)
    leg("short_conv_decode256", lambda i: ops.short_conv_silu(uc, w4, None, cstate, slots, None, pos), 4, byts=b * 6144 * 2 * 8)
    x32, y16, w = torch.randn(b, width, device=dev), rnd(b, width), torch.ones(width, device=dev, dtype=bf)
    x16 = rnd(b, width)
    leg("add_rmsnorm_branch_norm_256", lambda i: ops.add_rmsnorm(x16, y16, w, 1e-6, True, y_weight=w), 8, byts=b * width * 8)
    leg("residual_norm_f32_256", lambda i: ops.residual_norm(x32, y16, w, 1e-6, y_weight=w), 8, byts=b * width * 12)
    return leg.rows


# ---- Vebonex: beside the models above, and the kernels of its own ---------------------------------------------
def vebonex_bench_shape(size: str):
    """Layers in turn: matrix LSTM, gated linear attention, latent attention, latent attention on the latents of the one before; heads of
    128 everywhere; a feed-forward of as many weights as the gated one of the other models."""
    from mini_vllm_b200.config import vebonex_shape
    width, heads, _, ff, layers = FUPUPEL_SIZES[size]
    mlp = {"kind": "dense", "ff": ff * 3 // 2}
    head = {"heads": heads, "dim": 128, "vdim": 128}
    latent = {**head, "kv_rank": 512, "q_rank": width * 3 // 4, "scale": 128 ** -0.5}
    turn = lambda i: [("mlstm", {**head, "gate_cap": 15.0}), ("gla", {**head, "tau": 16.0, "decay_rank": 16}), ("latent_attention", latent),
                      ("latent_attention", {**latent, "kv_from": i - 1})][i % 4]
    return vebonex_shape([{"type": turn(i)[0], "mixer": turn(i)[1], "mlp": mlp} for i in range(layers)], width, 32768, streams=4, groups=8)


def vebonex_throughput(sizes=tuple(FUPUPEL_SIZES)) -> dict:
    """Beside Fupupel, the closest design there is, and Qwen3 layers of the same width, heads, feed-forward and count."""
    return engine_throughput((f"{size}_{name}", hf) for size in sizes
                             for name, hf in (("vebonex", vebonex_bench_shape(size)), ("fupupel", fupupel_bench_shape(size)), ("qwen3", qwen3_twin(size))))


def vebonex_kernel_legs(dev, peaks) -> dict:
    """Each kernel of the design against its roofline, next to the like kernel of the other models.  16 heads of 128, width 2048, latent
    of 512, 4 streams, 8192 prefill tokens, 256 decode rows."""
    from mini_vllm_b200 import ops
    bf, leg = torch.bfloat16, Legs(dev, peaks)
    rnd = lambda *shape, scale=1.0: (torch.randn(*shape, device=dev) * scale).to(bf)
    heads, d, width, ff, latent, streams, tokens = 16, 128, 2048, 9216, 512, 4, 8192
    hd, scale, eps = heads * d, d ** -0.5, 1e-6
    ones = torch.ones(hd, device=dev)
    qd, kd, vd, gate, od = (rnd(tokens, heads, d) for _ in range(5))
    raw_a, raw_b, raw_c = rnd(tokens, hd), rnd(tokens, heads), rnd(tokens, heads)
    ea, db, hb = torch.rand(heads, device=dev) * 8 + 1, torch.full((hd,), -4.0, device=dev), torch.full((heads,), 4.0, device=dev)

    def recurrent(tag, rows, cu, pos, slots, nbuf):
        states = [(torch.randn(slots.numel(), heads, d, d, device=dev) * 0.01, torch.zeros(slots.numel(), heads, d, device=dev),
                   torch.zeros(slots.numel(), heads, device=dev)) for _ in range(nbuf)]
        q, k, v, o, g, a, b, c = qd[:rows], kd[:rows], vd[:rows], od[:rows], gate[:rows].flatten(1), raw_a[:rows], raw_b[:rows], raw_c[:rows]
        work = {"byts": rows * heads * d * d * 8} if cu is None else {"byts": rows * hd * 6 * 2, "fp32": rows * heads * d * d * 2}
        leg(f"gated_delta_{tag}", lambda i: ops.gated_delta(q, k, v, a, b, g, ea, db, ones[:d], o, states[i][0], slots, cu, pos, scale, eps), nbuf, **work)
        leg(f"gated_linear_{tag}", lambda i: ops.gated_linear(q, k, v, a, db, 16.0, g, ones[:d], o, states[i][0], slots, cu, pos, scale, eps), nbuf, **work)
        if cu is not None:
            work["byts"] = rows * hd * 5 * 2
        leg(f"mlstm_{tag}", lambda i: ops.mlstm(q, k, v, b, hb, c, hb, 15.0, g, ones, o, states[i], slots, cu, pos, scale, eps), nbuf, **work)

    w16 = torch.ones(width, device=dev, dtype=bf)
    for tag, lens in (("4x2048", [2048] * 4), ("1x8192", [8192])):
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        pos = torch.cat([torch.arange(n, device=dev) for n in lens])
        recurrent(tag, tokens, cu, pos, torch.arange(len(lens), dtype=torch.int32, device=dev), 1)
        k8, v8, kv = rnd(tokens, heads // 2, d), rnd(tokens, heads // 2, d), rnd(tokens, 2 * heads, d)
        pairs = sum(n * (n + 1) // 2 for n in lens)
        leg(f"prefill_attn_{tag}", lambda i: ops.prefill_attn(qd, k8, v8, cu, cu, max(lens), scale), 2, flops=4 * hd * pairs)
        leg(f"prefill_attn_of_latents_{tag}", lambda i: ops.prefill_attn(qd, kv[:, :heads], kv[:, heads:], cu, cu, max(lens), scale), 2, flops=4 * hd * pairs)
    xs32, ys = [torch.randn(tokens, width, device=dev) for _ in range(3)], [rnd(tokens, width) for _ in range(3)]
    leg("residual_norm_8192", lambda i: ops.residual_norm(xs32[i], ys[i], w16, eps, y_weight=w16), 3, byts=tokens * width * 12)
    x4 = [torch.randn(tokens, streams, width, device=dev) for _ in range(2)]
    mix, sw = torch.eye(streams, device=dev), torch.full((streams,), 0.25, device=dev)
    leg("hyper_norm_8192", lambda i: ops.hyper_norm(x4[i], ys[i], mix, sw, sw, w16, eps, 8), 2, byts=tokens * width * (8 * streams + 4))
    del x4, xs32
    z, act = [rnd(tokens, ff) for _ in range(2)], torch.tensor([0.5, 0.4, 0.3, 0.1], device=dev)
    leg("act_mul_8192", lambda i: ops.act_mul(z[i], ff // 2, False), 2, byts=tokens * ff * 3)
    leg("poly_norm_8192", lambda i: ops.poly_norm(z[i], ff, act, eps), 2, byts=tokens * ff * 4)
    del z
    proj = [rnd(tokens, 1536 + latent + hd) for _ in range(3)]
    pool, slots = torch.zeros(tokens // 256, 256, latent, device=dev, dtype=bf), torch.arange(tokens, dtype=torch.int32, device=dev)
    lw = torch.ones(1536, device=dev, dtype=bf)
    leg("latent_norm_8192", lambda i: ops.latent_norm(proj[i][:, :1536], lw, 1536, proj[i][:, 1536:2048], lw[:latent], latent, eps, pool, slots), 3,
        byts=tokens * (1536 * 2 + latent * 3) * 2)
    leg("gate_mul_8192", lambda i: ops.gate_mul(od.flatten(1), proj[i][:, 2048:], ys[i]), 3, byts=tokens * hd * 6)
    # decode: 256 sequences
    b = 256
    pos, slots = torch.full((b,), 1199, device=dev), torch.arange(b, dtype=torch.int32, device=dev)
    recurrent(f"decode{b}", b, None, pos, slots, 2)
    x4 = [torch.randn(b, streams, width, device=dev) for _ in range(24)]
    xs32 = [torch.randn(b, width, device=dev) for _ in range(64)]
    leg(f"residual_norm_{b}", lambda i: ops.residual_norm(xs32[i], ys[0][:b], w16, eps, y_weight=w16), 64, byts=b * width * 12)
    leg(f"hyper_norm_{b}", lambda i: ops.hyper_norm(x4[i], ys[0][:b], mix, sw, sw, w16, eps, 8), 24, byts=b * width * (8 * streams + 4))
    zs = [rnd(b, ff) for _ in range(32)]
    leg(f"act_mul_{b}", lambda i: ops.act_mul(zs[i], ff // 2, False), 32, byts=b * ff * 3)
    leg(f"poly_norm_{b}", lambda i: ops.poly_norm(zs[i], ff, act, eps), 32, byts=b * ff * 4)
    del x4, xs32, zs
    for n in (1200, 4096):
        per = -(-n // 256)
        lens = torch.full((b,), n, dtype=torch.int32, device=dev)
        bt = torch.arange(b * per, dtype=torch.int32, device=dev).view(b, per)
        pools = torch.randn(2, b * per, 256, heads // 2, d, device=dev, dtype=bf)
        ws = ops.decode_workspace(b, heads, d, dev)
        ops.decode_plan(lens, -1, heads, heads // 2, d, ws, block_table=bt, block_size=256)
        leg(f"decode_attn_{b}x{n}", lambda i: ops.decode_attn(qd[:b], pools[0], pools[1], lens, bt, scale, -1, ws), 1, byts=b * n * hd * 2)
        del pools
        for h in (16, 32):
            ws = ops.decode_workspace(b, h, latent, dev)
            ops.latent_decode_plan(lens, bt, 256, h, latent, ws)
            lat, ql = rnd(b * per, 256, latent), rnd(h, b, latent)
            leg(f"latent_decode_{h}heads_{b}x{n}", lambda i: ops.latent_decode(ql, lat, lens, bt, scale, ws), 1, byts=b * n * latent * 2)
            del lat
    # the projections around it, as the batched products they are
    up, qh = rnd(heads, d, latent), rnd(b, heads, d)
    leg(f"absorb_queries_{b}", lambda i: torch.bmm(qh.transpose(0, 1), up), 8, byts=(heads * d * latent + b * heads * (d + latent)) * 2)
    return leg.rows


# ---- Sunulorn: beside Qwen3 layers of as many active weights, and the kernels of its own ------------------------
SUNULORN_EXPERTS, SUNULORN_TOP = 16, 2


def sunulorn_bench_shape(size: str, window: int = 1024, keep: int = 64):
    """Layers in turn: convolved keys + dense, window + experts, distance bias + dense, the same on borrowed keys + experts.  A token meets
    as many feed-forward weights in every layer: two experts of a quarter and a shared one of half the dense size."""
    from mini_vllm_b200.config import sunulorn_shape
    width, heads, kv, ff, layers = FUPUPEL_SIZES[size]
    head = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "expert": {"ff": ff // 4, "limit": 7.0}, "router": {"experts": SUNULORN_EXPERTS, "top": SUNULORN_TOP},
           "shared": {"ff": ff // 2, "limit": 7.0}}
    turn = lambda i: [("attention", {**head, "conv": 4, "rot": {"dims": 64, "base": 1e6}}, dense),
                      ("attention_2", {**head, "rot": {"dims": 128, "base": 1e6}, "mask": {"size": window, "keep_first": keep}}, moe),
                      ("attention_3", head, dense), ("attention_3", {**head, "kv_from": i - 1}, moe)][i % 4]
    return sunulorn_shape([dict(zip(("type", "mixer", "mlp"), turn(i))) for i in range(layers)], width, 32768)


def sunulorn_throughput(sizes=tuple(FUPUPEL_SIZES)) -> dict:
    return engine_throughput((f"{size}_{name}", hf) for size in sizes
                             for name, hf in (("sunulorn", sunulorn_bench_shape(size)), ("qwen3", qwen3_twin(size))))


def sunulorn_kernel_legs(dev, peaks) -> dict:
    """Each kernel of the design against its roofline, next to the like kernel of the other models.  16 heads of 128 (8 KV heads), width
    2048, 16 experts of 1536 with 2 per token, 8192 prefill tokens, 32 and 256 decode rows."""
    from mini_vllm_b200 import ops
    from mini_vllm_b200.models.layers.branches import alibi_slopes
    from mini_vllm_b200.models.layers.rotary import build_cos_sin_cache
    bf, leg = torch.bfloat16, Legs(dev, peaks)
    rnd = lambda *shape, scale=1.0: (torch.randn(*shape, device=dev) * scale).to(bf)
    heads, kv, d, width, ff, tokens, window, keep, eps = 16, 8, 128, 2048, 6144, 8192, 1024, 64, 1e-6
    sinks, slopes, scale = torch.zeros(heads, device=dev), alibi_slopes(heads).to(dev), d ** -0.5
    gate = rnd(tokens, heads)
    forms = {"plain": (-1, None), "sink": (-1, ops.AttnExtras(sinks=sinks)),
             "distance_sink_gate": (-1, ops.AttnExtras(sinks=sinks, slopes=slopes, head_gate=gate)),
             "window": (window - 1, None), "window_kept": (window - 1, ops.AttnExtras(keep_first=keep))}
    q, k, v = rnd(tokens, heads, d), rnd(tokens, kv, d), rnd(tokens, kv, d)
    for tag, lens in (("4x2048", [2048] * 4), ("1x8192", [8192])):
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        for name, (wl, ex) in forms.items():
            kept = keep if ex is not None and ex.keep_first else 0
            seen = lambda i: i + 1 if wl < 0 else min(i + 1, wl + 1) + min(kept, max(i - wl, 0))
            leg(f"prefill_attn_{name}_{tag}", lambda i: ops.prefill_attn(q, k, v, cu, cu, max(lens), scale, wl, extras=ex), 4,
                flops=4 * heads * d * sum(sum(seen(i) for i in range(n)) for n in lens))
    # between projection and attention
    proj = [rnd(tokens, (heads + 2 * kv) * d) for _ in range(4)]
    cut = lambda x: tuple(t.unflatten(1, (-1, d)) for t in x.split([heads * d, kv * d, kv * d], dim=1))
    pools = [torch.zeros(2, tokens // 256 + 2, 256, kv, d, device=dev, dtype=bf) for _ in range(4)]
    table, ones = build_cos_sin_cache(128, 8192, 1e6, head_dim=128).to(dev), torch.ones(d, device=dev, dtype=bf)
    for rows in (tokens, 256):
        pos, slots = torch.arange(rows, device=dev), torch.randperm(rows, device=dev).to(torch.int32)
        byts = rows * (heads + 2 * kv) * d * 2 * 2
        part = lambda i: cut(proj[i][:rows])
        leg(f"rope_kv_write_{rows}", lambda i: ops.rope_kv_write(*part(i), pos, table, slots, *pools[i], k_in_place=False), 4, byts=byts)
        leg(f"qk_norm_rope_kv_write_{rows}", lambda i: ops.qk_norm_rope_kv_write(*part(i), ones, ones, eps, False, pos, table, slots, *pools[i],
                                                                               k_in_place=False), 4, byts=byts)
        leg(f"rope_norm_kv_write_{rows}", lambda i: ops.rope_norm_kv_write(*part(i), pos, table, slots, *pools[i], k_in_place=False, norm_dim=d,
                                                                         eps=eps), 4, byts=byts)
        qk = (heads + kv) * d
        cu = None if rows == 256 else torch.tensor([0, rows], dtype=torch.int32, device=dev)
        w4, state = rnd(4, qk), torch.zeros(256, 3, qk, device=dev, dtype=bf)
        sl = torch.arange(256 if cu is None else 1, dtype=torch.int32, device=dev)
        more = rows * qk * 2 * 6 if cu is None else 0
        leg(f"short_conv_silu_{rows}", lambda i: ops.short_conv_silu(proj[i][:rows, :qk], w4, None, state, sl, cu, pos), 4, byts=rows * qk * 4 + more)
        leg(f"short_conv_copied_keys_{rows}", lambda i: ops.short_conv(proj[i][:rows, :qk], w4, None, state, sl, cu, pos, copies=kv * d), 4,
            byts=rows * (2 * qk + kv * d) * 2 + more)
    del pools
    o2 = [rnd(tokens, heads * d) for _ in range(3)]
    leg("gate_mul_8192", lambda i: ops.gate_mul(q.flatten(1), proj[i][:, :heads * d], o2[i]), 3, byts=tokens * heads * d * 6)
    del proj, o2
    # norms and gated units
    for rows, n in ((tokens, 3), (256, 48)):
        xs, ys, w = [torch.randn(rows, width, device=dev) for _ in range(n)], [rnd(rows, width) for _ in range(n)], torch.ones(width, device=dev, dtype=bf)
        extra, index = rnd(rows * 2, width), torch.randperm(rows * 2, device=dev).view(rows, 2).to(torch.int32)
        leg(f"residual_norm_{rows}", lambda i: ops.residual_norm(xs[i], ys[i], w, eps, y_weight=w), n, byts=rows * width * 12)
        leg(f"residual_norm_pair_{rows}", lambda i: ops.residual_norm_pair(xs[i], ys[i], w, w, eps), n, byts=rows * width * 14)
        leg(f"residual_norm_pair_experts_{rows}", lambda i: ops.residual_norm_pair(xs[i], ys[i], w, w, eps, extra, index), n, byts=rows * width * 18)
        del xs, ys
        m = 2 if rows == tokens else 32
        gu = [rnd(rows, 2 * ff) for _ in range(m)]
        leg(f"act_mul_{rows}", lambda i: ops.act_mul(gu[i], ff, False), m, byts=rows * ff * 6)
        leg(f"glu_{rows}", lambda i: ops.glu(gu[i], ff), m, byts=rows * ff * 6)
        leg(f"glu_clamped_row_gate_{rows}", lambda i: ops.glu(gu[i], ff, 7.0, 1.702, 1.0, row_gate=gu[i][:, 0]), m, byts=rows * ff * 6)
        del gu
    # experts beside a dense product of as many operations
    E, top, inter = SUNULORN_EXPERTS, SUNULORN_TOP, ff // 4
    for rows in (tokens, 256, 32):
        nbuf = 2 if rows == tokens else 4
        up, down = [rnd(E, 2, inter, width, scale=width ** -0.5) for _ in range(nbuf)], [rnd(E, width, inter, scale=inter ** -0.5) for _ in range(nbuf)]
        h, counters = rnd(rows, width), torch.zeros(E + 1, dtype=torch.int32, device=dev)
        logits = torch.randn(rows, E, device=dev)
        leg(f"moe_route_and_gather_{rows}", lambda i: ops.moe_sort(h, logits, top, counters), 4, byts=rows * (1 + top) * width * 2)
        x, er = ops.moe_sort(h, logits, top, counters)
        y = ops.moe_gemm(x, up[0], er, width, gated=(7.0, 1.702, 1.0))
        used = len(set(torch.topk(logits, top).indices.flatten().tolist()))
        work = lambda m, k: ({"flops": 2 * rows * top * m * k} if rows == tokens else {"byts": (used * m * k + rows * top * (m + k)) * 2})
        leg(f"moe_gemm_gated_{rows}", lambda i: ops.moe_gemm(x, up[i], er, width, gated=(7.0, 1.702, 1.0)), nbuf, **work(2 * inter, width))
        leg(f"moe_gemm_down_{rows}", lambda i: ops.moe_gemm(y, down[i], er, inter), nbuf, **work(width, inter))
        # dense: as many operations for a prompt, as many weights for decoding
        xr, wide = (rows * top, 2 * inter) if rows == tokens else (rows * top // E if rows > E else 1, used * 2 * inter)
        wd, xd = [rnd(wide, width, scale=width ** -0.5) for _ in range(nbuf)], rnd(xr, width)
        leg(f"dense_gemm_up_{rows}", lambda i: torch.nn.functional.linear(xd, wd[i]), nbuf,
            **({"flops": 2 * xr * wide * width} if rows == tokens else {"byts": (wide * width + xr * (wide + width)) * 2}))
        del up, down, wd
    # decode attention
    b = 256
    for n in (1200, 4096):
        per = -(-n // 256)
        lens, bt = torch.full((b,), n, dtype=torch.int32, device=dev), torch.arange(b * per, dtype=torch.int32, device=dev).view(b, per)
        pool = torch.randn(2, b * per, 256, kv, d, device=dev, dtype=bf)
        ws = ops.decode_workspace(b, heads, d, dev)
        for name, (wl, ex) in forms.items():
            ex = None if ex is None else ex.rows(0, b)
            kept = 0 if ex is None else ex.keep_first
            ops.decode_plan(lens, wl, heads, kv, d, ws, block_table=bt, block_size=256, keep_first=kept)
            seen = n if wl < 0 else min(n, wl + 1) + min(kept, max(n - wl - 1, 0))
            leg(f"decode_attn_{name}_{b}x{n}", lambda i: ops.decode_attn(q[:b], pool[0], pool[1], lens, bt, scale, wl, ws, extras=ex), 1,
                byts=b * seen * kv * d * 4)
        del pool
    return leg.rows


# ---- Rasezen: beside Sunulorn, Fupupel and Qwen3 layers of about as many active weights, and the kernels of its own ----------------
def rasezen_bench_shape(size: str, window: int = 1024):
    """Layers in turn: state space + dense, window + experts, state space + experts, window + dense.  State-space layers have twice the width
    in heads of 64, 128 states and 8 groups; the dense feed-forward has as many weights as a gated one of ``ff``, the experts as in
    ``sunulorn_bench_shape`` with two identity experts more."""
    from mini_vllm_b200.config import rasezen_shape
    width, heads, kv, ff, layers = FUPUPEL_SIZES[size]
    space = {"heads": 2 * width // 64, "groups": 8, "state": 128, "vdim": 64, "conv": 4, "norm_groups": 8}
    attn = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": window}, "rot": {"base": 1e6, "dims": 128}}
    dense = {"kind": "dense", "ff": ff * 3 // 2}
    moe = {"kind": "moe", "expert": {"ff": ff // 4}, "router": {"experts": SUNULORN_EXPERTS, "top": SUNULORN_TOP, "identity": 2, "scale": 2.0},
           "shared": {"ff": ff // 2}}
    turn = [("mamba2", space, dense), ("attention", attn, moe), ("mamba2", space, moe), ("attention", attn, dense)]
    return rasezen_shape([dict(zip(("type", "mixer", "mlp"), turn[i % 4])) for i in range(layers)], width, 32768)


def rasezen_throughput(sizes=tuple(FUPUPEL_SIZES)) -> dict:
    return engine_throughput((f"{size}_{name}", hf) for size in sizes
                             for name, hf in (("rasezen", rasezen_bench_shape(size)), ("sunulorn", sunulorn_bench_shape(size)),
                                              ("fupupel", fupupel_bench_shape(size)), ("qwen3", qwen3_twin(size))))


def rasezen_kernel_legs(dev, peaks) -> dict:
    """Each kernel of the design against its roofline, next to the like kernel of the other models.  Width 2048, state-space layers of 64
    heads of 64 (and, for the comparison, 16 of 128) with 128 states, 16 attention heads of 128 (8 KV heads), 16 experts of 1536 with
    2 per token and 2 identity experts, 8192 prefill tokens, 256 decode rows."""
    from mini_vllm_b200 import ops
    from mini_vllm_b200.models.layers.rotary import build_cos_sin_cache
    bf, leg = torch.bfloat16, Legs(dev, peaks)
    rnd = lambda *shape, scale=1.0: (torch.randn(*shape, device=dev) * scale).to(bf)
    width, tokens, n, eps, inner = 2048, 8192, 128, 1e-6, 4096

    def recurrences(tag, rows, cu, pos, slots, nbuf, longest=0):
        for heads, vdim, groups in ((64, 64, 8), (16, 128, 16)):
            cols, keys = heads * vdim, groups * n
            xbc, dt = [rnd(rows, cols + 2 * keys) for _ in range(nbuf)], rnd(rows, heads)
            bias, a, d = torch.full((heads,), -4.0, device=dev), -torch.rand(heads, device=dev) * 8 - 1, torch.ones(heads, device=dev)
            states, y = [torch.randn(slots.numel(), heads, n, vdim, device=dev) * 0.01 for _ in range(nbuf)], torch.empty(rows, heads, vdim, device=dev, dtype=bf)

            def run(i):
                x, b, c = xbc[i].split([cols, keys, keys], dim=1)
                ops.state_space(x.unflatten(1, (heads, vdim)), b.unflatten(1, (groups, n)), c.unflatten(1, (groups, n)), dt, bias, a, d, y, states[i],
                                slots, cu, pos, longest)
            work = {"byts": rows * heads * n * vdim * 8} if cu is None else {"byts": rows * (2 * cols + 2 * keys) * 2, "fp32": rows * heads * n * vdim * 2}
            leg(f"state_space_{heads}x{vdim}_{tag}", run, nbuf, **work)
            del xbc, states
        heads, d = 16, 128
        q, k, v, o, gate = (rnd(rows, heads, d) for _ in range(5))
        bc, hb, w = rnd(rows, heads), torch.full((heads,), 4.0, device=dev), torch.ones(heads * d, device=dev)
        states = [(torch.randn(slots.numel(), heads, d, d, device=dev) * 0.01, torch.zeros(slots.numel(), heads, d, device=dev),
                   torch.zeros(slots.numel(), heads, device=dev)) for _ in range(nbuf)]
        work = {"byts": rows * heads * d * d * 8} if cu is None else {"byts": rows * heads * d * 10, "fp32": rows * heads * d * d * 2}
        leg(f"mlstm_16x128_{tag}", lambda i: ops.mlstm(q, k, v, bc, hb, bc, hb, 15.0, gate.flatten(1), w, o, states[i], slots, cu, pos, d ** -0.5, eps),
            nbuf, **work)
        del states
        u, dt, z, y = (rnd(rows, inner) for _ in range(4))
        b, c = rnd(rows, 32).split([16, 16], dim=1)
        bias, a, skip = torch.full((inner,), -4.0, device=dev), -torch.rand(inner, 16, device=dev) * 8 - 1, torch.ones(inner, device=dev)
        states = [torch.zeros(slots.numel(), inner, 16, device=dev) for _ in range(nbuf)]
        work = {"byts": rows * inner * 16 * 8} if cu is None else {"byts": rows * inner * 8, "mufu": rows * inner * 16}
        leg(f"selective_scan_{inner}x16_{tag}", lambda i: ops.selective_scan(u, dt, z, b, c, bias, a, skip, y, states[i], slots, cu, pos), nbuf, **work)

    for tag, lens in (("4x2048", [2048] * 4), ("1x8192", [8192])):
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        recurrences(tag, tokens, cu, torch.cat([torch.arange(m, device=dev) for m in lens]), torch.arange(len(lens), dtype=torch.int32, device=dev), 2,
                    max(lens))
    recurrences("decode256", 256, None, torch.full((256,), 1199, device=dev), torch.arange(256, dtype=torch.int32, device=dev), 2)

    heads, kv, d, ff = 16, 8, 128, 9216
    proj = [rnd(tokens, (heads + 2 * kv) * d) for _ in range(4)]
    cut = lambda x: tuple(t.unflatten(1, (-1, d)) for t in x.split([heads * d, kv * d, kv * d], dim=1))
    pools = [torch.zeros(2, tokens // 256 + 2, 256, kv, d, device=dev, dtype=bf) for _ in range(4)]
    table, ones = build_cos_sin_cache(128, 8192, 1e6, head_dim=128).to(dev), torch.ones(d, device=dev, dtype=bf)
    norm = ops.RowNorm(torch.ones(heads * d, device=dev, dtype=bf), torch.ones(kv * d, device=dev, dtype=bf), heads * d, kv * d, d, eps)
    for rows in (tokens, 256):
        pos, slots = torch.arange(rows, device=dev), torch.randperm(rows, device=dev).to(torch.int32)
        byts = rows * (heads + 2 * kv) * d * 2 * 2
        part = lambda i: cut(proj[i][:rows])
        leg(f"qk_norm_rope_kv_write_{rows}", lambda i: ops.qk_norm_rope_kv_write(*part(i), ones, ones, eps, False, pos, table, slots, *pools[i],
                                                                               k_in_place=False), 4, byts=byts)
        leg(f"row_norm_rope_kv_write_{rows}", lambda i: ops.row_norm_rope_kv_write(*part(i), norm, pos, table, slots, *pools[i], kv_in_place=False), 4,
            byts=byts)
    del pools, proj
    for rows, m in ((tokens, 3), (256, 48)):
        # the state-space layer's convolution and norm
        chan = inner + 2 * 8 * n
        us, cu = [rnd(rows, chan) for _ in range(min(m, 8))], None if rows == 256 else torch.tensor([0, rows], dtype=torch.int32, device=dev)
        w4, bias, state = rnd(4, chan), rnd(chan), torch.zeros(256, 3, chan, device=dev, dtype=bf)
        pos, sl = torch.arange(rows, device=dev), torch.arange(256 if cu is None else 1, dtype=torch.int32, device=dev)
        leg(f"short_conv_silu_{rows}", lambda i: ops.short_conv_silu(us[i], w4, bias, state, sl, cu, pos), len(us),
            byts=rows * chan * 4 + (rows * chan * 12 if cu is None else 0))
        del us
        ys, zs, os = ([rnd(rows, inner) for _ in range(m)] for _ in range(3))
        w = torch.ones(inner, device=dev)
        leg(f"gated_group_norm_8_{rows}", lambda i: ops.gated_group_norm(ys[i], zs[i], w, os[i], 8, eps), m, byts=rows * inner * 6)
        leg(f"gated_group_norm_1_{rows}", lambda i: ops.gated_group_norm(ys[i], zs[i], w, os[i], 1, eps), m, byts=rows * inner * 6)
        leg(f"gate_mul_{rows}", lambda i: ops.gate_mul(ys[i], zs[i], os[i]), m, byts=rows * inner * 6)
        del ys, zs, os
        zs, os, act = [rnd(rows, ff) for _ in range(m)], [rnd(rows, ff) for _ in range(m)], torch.ones(2, device=dev)
        leg(f"act_mul_{rows}", lambda i: ops.act_mul(zs[i], ff // 2, False, out=os[i][:, :ff // 2]), m, byts=rows * ff * 3)
        leg(f"xielu_{rows}", lambda i: ops.xielu(zs[i], act, out=os[i]), m, byts=rows * ff * 4)
        del zs, os
        xs, ys, hs, w = [torch.randn(rows, width, device=dev) for _ in range(m)], [rnd(rows, width) for _ in range(m)], [rnd(rows, width) for _ in range(m)], ones.new_ones(width)
        extra, index, own = rnd(rows * 2, width), torch.randperm(rows * 2, device=dev).view(rows, 2).to(torch.int32), torch.rand(rows, device=dev)
        own[torch.rand(rows, device=dev) > 0.25] = 0                 # one token in four has an identity expert, and one expert's row less
        index2 = torch.where((own != 0)[:, None] & (torch.arange(2, device=dev) == 0), -1, index)
        leg(f"residual_norm_experts_{rows}", lambda i: ops.residual_norm_pair(xs[i], ys[i], w, None, eps, extra, index), m, byts=rows * width * 16)
        leg(f"residual_norm_experts_identity_{rows}", lambda i: ops.residual_norm_pair(xs[i], ys[i], w, None, eps, extra, index2, own=hs[i],
                                                                                     own_weights=own), m, byts=rows * width * 16)
        del xs, ys, hs, extra
        E, top = SUNULORN_EXPERTS, SUNULORN_TOP
        h, counters, logits = rnd(rows, width), torch.zeros(E + 1, dtype=torch.int32, device=dev), torch.randn(rows, E + 2, device=dev)
        routing = ops.Routing(True, torch.zeros(E + 2, device=dev), 2.0, 2)
        taken = rows * top * E / (E + 2)
        leg(f"moe_route_and_gather_{rows}", lambda i: ops.moe_sort(h, logits[:, :E], top, counters), 4,
            byts=rows * (1 + top) * width * 2)
        leg(f"moe_route_and_gather_identity_{rows}", lambda i: ops.moe_sort(h, logits, top, counters, routing), 4, byts=(rows + taken) * width * 2)
    return leg.rows


# ---- CPU leg: the oracle restatement of the reference path on the host cores ------------------------
class CpuReference:
    """The oracle model (restatement of the reference's PyTorch path, pinned to the reference's own engine loop by
    tests/test_reference_engine.py) on the host cores.  Built once; ``sample()`` runs one bounded sample of the
    workload: the first requests of the share until ``prompt_tokens`` prompt tokens are reached (at least two
    requests), full prompts, ``n_dec`` generated tokens each, through the scheduler like any job."""

    def __init__(self, workload: str, prompt_tokens: int = 1200, n_dec: int = 16, seed: int = 0):
        from mini_vllm_b200.models.loader import load_model
        from oracle.model import OracleExecutor, OracleModel, reference_names
        self.threads = os.cpu_count() or 1
        torch.set_num_threads(self.threads)
        hf = qwen3_shape()
        self.cfg = Config(hf_config=hf, kv_cache_num_blocks=160, max_num_batched_seqs=8, use_cuda_graph=False, seed=seed)
        model = load_model(self.cfg, device="cpu")
        weights = reference_names(dict(model.state_dict()), "qwen3", hf)
        del model
        self.executor = OracleExecutor(OracleModel(weights, hf, "qwen3", 160, 256, device="cpu"), 256)
        reqs, total = [], 0
        for r in workload_requests(workload):
            if len(reqs) >= 2 and total >= prompt_tokens:
                break
            if len(r.prompt) > 2048:                 # keep one sample to seconds: the longest prompts are skipped
                continue
            reqs.append(r)
            total += len(r.prompt)
        self.reqs, self.n_dec = reqs, n_dec
        self.describe = (f"{len(reqs)} requests of the workload ({total} prompt tokens, prompts over 2048 skipped), "
                         f"{n_dec} generated tokens each, bf16 weights, prefill+decode tokens / wall time "
                         "(per-token extrapolation; prefill-heavy, which favours the CPU)")

    def sample(self) -> tuple[int, float]:
        from mini_vllm_b200.engine.request import Request
        from mini_vllm_b200.scheduler.scheduler import Scheduler
        sch = Scheduler(self.cfg)
        for r in self.reqs:
            sch.submit(Request(r.prompt, SamplingParams(max_tokens=self.n_dec, ignore_eos=True)))
        t0 = time.perf_counter()
        tokens = 0
        while not sch.finished:
            batch = sch.schedule()
            out = self.executor.execute(batch)
            tokens += sum(len(r.tokens) - r.num_cached_tokens for r in batch.requests) if batch.type == 0 else len(out)
            sch.update(batch, out)
        return tokens, time.perf_counter() - t0


def workload_config(workload: str, world: int, requests_per_gpu: int, tokens_per_step: int, mixed: bool = False) -> dict:
    """The ``config`` object of the bench line: both arms print the same keys and values for the same run."""
    return {"workload": WORKLOADS[workload] + (", mixed steps" if mixed else ""), "requests_per_gpu": requests_per_gpu,
            "parallelism": f"replicas x{world}",
            "l2": "KV pool (28 layers, >126 MB per step) exceeds L2; kernel legs rotate distinct pools",
            "tokens_per_step_all_gpus": tokens_per_step}


def reference_arm(args):
    """The reference's path on the host cores (rank 0 only): ``--warmup`` untimed and exactly ``--steps`` timed
    bounded samples; ``ms_per_step`` x ``steps`` is the time really spent in the timed region."""
    rank = int(os.environ.get("RANK", "0"))
    if rank != 0:
        return
    world = int(os.environ.get("WORLD_SIZE", "1"))
    cpu = CpuReference(args.workload)
    for _ in range(args.warmup):
        cpu.sample()
    tokens, secs = 0, 0.0
    for _ in range(args.steps):
        n, dt = cpu.sample()
        tokens += n
        secs += dt
    value = tokens / secs
    mine = workload_requests(args.workload, world, 0)
    per_step_all = sum(len(r.prompt) + r.max_tokens for k in range(world) for r in workload_requests(args.workload, world, k))
    config = workload_config(args.workload, world, len(mine), per_step_all)
    config["sample"] = cpu.describe
    line = {"impl": "reference", "metric": METRIC, "value": round(value, 2), "unit": "tokens/s", "n_gpus": args.gpus,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(1e3 * secs / args.steps, 1),
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
            "config": config,
            "cpu_baseline": {"value": round(value, 2), "unit": "tokens/s", "cores": cpu.threads, "kind": "port",
                             "sample": cpu.describe, "tokens_per_sample": tokens // args.steps},
            "e2e": {"value": round(value, 2), "unit": "tokens/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0}}
    print(json.dumps(line))


# ---------------------------------------------------------------------------------------------------
def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=3)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--no-strong-scaling", action="store_true",
                    help="skip the extra N=1 job over all 4096 config-5 requests (about a minute)")
    ap.add_argument("--workload", default="config5", choices=["config5", "config2"],
                    help="config5 (default): 512 requests per GPU, prompts log-uniform [32,4096], outputs "
                         "U[64,1024]; config2: 64 requests per GPU, prompt U[100,1024], total <= 1024")
    ap.add_argument("--kernel-legs", nargs="?", const="all", default=None, metavar="LEGS",
                    help="only the fixed single-kernel cases (one 2.3 GB pool), then exit; optionally a comma list out "
                         "of " + ",".join(LEGS) + " to keep a profiler capture small")
    ap.add_argument("--no-fused-head", action="store_true",
                    help="variant: lm_head and the sampler as two kernels on every step (Config.fused_greedy_head=False)")
    ap.add_argument("--mixed-steps", action="store_true",
                    help="variant: prompts join steps of running decodes (Config.enable_mixed_steps)")
    ap.add_argument("--config3-step", action="store_true",
                    help="engine-level config 3: 16 prefix-cached prompts arriving among 240 decodes, as one mixed "
                         "step and as the reference's two steps")
    ap.add_argument("--config2-parity", action="store_true",
                    help="first-32-token greedy identity with the reference engine's committed tokens on the 28-layer "
                         "config-2 model (64 screened prompts)")
    ap.add_argument("--config4-step", action="store_true",
                    help="engine-level config 4: a decode step of 128 sequences on Gemma3-1B shapes")
    ap.add_argument("--fupupel", nargs="?", const="all", default=None, choices=["all", "engine", "kernels"],
                    help="the Fupupel design with random weights: prefill and decode throughput beside Qwen3 layers of equal "
                         "size, and its kernels against their rooflines beside the like kernels")
    ap.add_argument("--vebonex", nargs="?", const="all", default=None, choices=["all", "engine", "kernels"],
                    help="the same for the Vebonex design, beside Fupupel and Qwen3")
    ap.add_argument("--sunulorn", nargs="?", const="all", default=None, choices=["all", "engine", "kernels"],
                    help="the same for the Sunulorn design, beside Qwen3")
    ap.add_argument("--rasezen", nargs="?", const="all", default=None, choices=["all", "engine", "kernels"],
                    help="the same for the Rasezen design, beside Sunulorn, Fupupel and Qwen3")
    ap.add_argument("--engine-steps", type=int, default=0,
                    help="profiling aid: prefill + N decode steps of the workload without CUDA graphs, then exit")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm(args)
    if args.config3_step:
        torch.cuda.set_device(0)
        out = []
        for mixed in (True, False):
            out.append(config3_engine_step(mixed))
            torch.cuda.empty_cache()
        print(json.dumps({"config3_engine_step": out}))
        return
    if args.config2_parity:
        torch.cuda.set_device(0)
        print(json.dumps({"config2_parity": config2_parity()}))
        return
    if args.config4_step:
        torch.cuda.set_device(0)
        print(json.dumps({"config4_engine_step": config4_engine_step()}))
        return
    if args.fupupel:
        torch.cuda.set_device(0)
        line = {}
        if args.fupupel in ("all", "kernels"):
            line["kernels"] = fupupel_kernel_legs(torch.device("cuda", 0), measured_peaks()[0])
        if args.fupupel in ("all", "engine"):
            line["engine"] = fupupel_throughput()
        print(json.dumps({"fupupel": line}))
        return
    if args.vebonex:
        torch.cuda.set_device(0)
        line = {}
        if args.vebonex in ("all", "kernels"):
            line["kernels"] = vebonex_kernel_legs(torch.device("cuda", 0), measured_peaks()[0])
        if args.vebonex in ("all", "engine"):
            line["engine"] = vebonex_throughput()
        print(json.dumps({"vebonex": line}))
        return
    if args.sunulorn:
        torch.cuda.set_device(0)
        line = {}
        if args.sunulorn in ("all", "kernels"):
            line["kernels"] = sunulorn_kernel_legs(torch.device("cuda", 0), measured_peaks()[0])
        if args.sunulorn in ("all", "engine"):
            line["engine"] = sunulorn_throughput()
        print(json.dumps({"sunulorn": line}))
        return
    if args.rasezen:
        torch.cuda.set_device(0)
        line = {}
        if args.rasezen in ("all", "kernels"):
            line["kernels"] = rasezen_kernel_legs(torch.device("cuda", 0), measured_peaks()[0])
        if args.rasezen in ("all", "engine"):
            line["engine"] = rasezen_throughput()
        print(json.dumps({"rasezen": line}))
        return
    if args.kernel_legs:
        peaks, _ = measured_peaks()
        legs = LEGS if args.kernel_legs == "all" else tuple(args.kernel_legs.split(","))
        unknown = [x for x in legs if x not in LEGS]
        if unknown:
            ap.error(f"unknown kernel legs {unknown}; choose from {LEGS}")
        print(json.dumps(kernel_extras(torch.device("cuda", 0), peaks, nl=1, legs=legs)))
        return
    if args.engine_steps:
        import dataclasses
        from mini_vllm_b200.engine.engine import Engine
        torch.cuda.set_device(0)
        eng = Engine(dataclasses.replace(build_config(args.workload), use_cuda_graph=False))   # every kernel its own launch
        for r in workload_requests(args.workload):
            eng.submit(r.prompt, SamplingParams(max_tokens=r.max_tokens, ignore_eos=True))
        done = 0
        while done < args.engine_steps:
            done += eng.step().type == 1
        torch.cuda.synchronize()
        print(json.dumps({"prefill_steps": eng.metrics.prefill_steps, "decode_steps": eng.metrics.decode_steps}))
        return

    from mini_vllm_b200 import ops
    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    dist = None
    if world > 1:
        import torch.distributed as dist
        torch.cuda.set_device(local_rank)
        dist.init_process_group("nccl", device_id=torch.device("cuda", local_rank))
    peaks, peak_kind = measured_peaks()

    mine = workload_requests(args.workload, world, rank)
    engine = build_engine(local_rank, args.workload, mixed_steps=args.mixed_steps, fused_head=not args.no_fused_head)
    dev = engine.executor.device
    # At N > 1 the job goes through the host dispatcher: rank 0 holds every request of the job (the shares of all
    # ranks), scatters them by token cost over a gloo group, and gets the completions back.
    group, job = None, mine
    if dist is not None:
        group = dist.new_group(backend="gloo")
        job = None
        if rank == 0:
            job = [r for k in range(world) for r in workload_requests(args.workload, world, k)]

    def sync_all():
        torch.cuda.synchronize()
        if dist is not None:
            dist.barrier()
            torch.cuda.synchronize()

    for _ in range(args.warmup):
        run_job(engine, job, group=group)
    sampler = ClockSampler(local_rank)
    contexts = []
    ex = engine.executor
    sync_all()
    if rank == 0:
        sampler.start()
    launches0, h2d0, d2h0 = ops.LaunchCounter.total, ex.h2d_bytes, ex.d2h_bytes
    steps0 = engine.metrics.prefill_steps + engine.metrics.decode_steps
    t0 = time.perf_counter()
    tok = 0
    cuda_ms = 0.0
    for i in range(args.steps):
        n, wall, ms = run_job(engine, job, contexts if (rank == 0 and i == args.steps - 1) else None, group=group)
        tok += n
        cuda_ms += ms
    sync_all()
    wall_total = time.perf_counter() - t0
    clocks = sampler.stop() if rank == 0 else None
    launches = ops.LaunchCounter.total - launches0
    engine_steps = engine.metrics.prefill_steps + engine.metrics.decode_steps - steps0
    h2d, d2h = ex.h2d_bytes - h2d0, ex.d2h_bytes - d2h0

    stats = torch.tensor([cuda_ms, wall_total * 1e3, float(tok), float(launches)], dtype=torch.float64, device=dev)
    if dist is not None:
        mx = stats.clone()
        dist.all_reduce(mx, op=dist.ReduceOp.MAX)
        sm = stats.clone()
        dist.all_reduce(sm, op=dist.ReduceOp.SUM)
        cuda_ms_max, wall_ms_max, tok_all, launches_all = mx[0].item(), mx[1].item(), sm[2].item(), sm[3].item()
    else:
        cuda_ms_max, wall_ms_max, tok_all, launches_all = cuda_ms, wall_total * 1e3, float(tok), float(launches)

    # Strong-scaling reference point, N = 1 only: the whole 4096-request job of config 5 on this one GPU, once.
    strong = None
    if world == 1 and args.workload == "config5" and not args.no_strong_scaling:
        from mini_vllm_b200.workloads import config5_requests
        n, wall, ms = run_job(engine, config5_requests(seed=0, n=4096))
        strong = {"requests": 4096, "tokens": n, "device_ms": round(ms, 1), "tokens_per_s": round(n / ms * 1e3, 1),
                  "e2e_tokens_per_s": round(n / wall, 1),
                  "note": "all of config 5 on one GPU, one job; the 8-GPU run of the same 4096 requests is the N=8 line"}

    if rank == 0:
        roof = decode_roofline(engine, contexts, peaks)
        roof["peak_kind"] = f"of {peak_kind}"
        extras = kernel_extras(dev, peaks)
        cpu = None
        if world == 1 and not args.no_cpu_baseline:
            ref = CpuReference(args.workload)
            ref.sample()                                                # warm-up (allocator, thread pool)
            n1, dt1 = ref.sample()
            n2, dt2 = ref.sample()
            cpu = {"value": round((n1 + n2) / (dt1 + dt2), 2), "unit": "tokens/s", "cores": ref.threads, "kind": "port",
                   "sample": ref.describe, "seconds": round(dt1 + dt2, 1)}
        line = {
            "metric": METRIC, "value": round(tok_all / (cuda_ms_max * 1e-3), 1), "unit": "tokens/s",
            "n_gpus": world, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": round(cuda_ms_max / args.steps, 2), "higher_is_better": True, "scaling": "weak",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
            "config": workload_config(args.workload, world, len(mine), int(tok_all / args.steps), args.mixed_steps),
            "e2e": {"value": round(tok_all / (wall_ms_max * 1e-3), 1), "unit": "tokens/s",
                    "h2d_bytes_per_step": int(h2d / max(engine_steps, 1)),
                    "d2h_bytes_per_step": int(d2h / max(engine_steps, 1)),
                    "engine_steps_per_job": engine_steps // args.steps},
            "gpu_launches": int(launches_all),
            "clocks": clocks, "roofline": roof, "kernels": extras, "cpu_baseline": cpu,
        }
        if strong is not None:
            line["strong_scaling_n1_tok_s"] = strong["tokens_per_s"]
            line["strong_scaling_n1"] = strong
        if world > 1:
            line["e2e"]["path"] = ("rank 0 holds all requests: host dispatcher scatter (gloo) -> Engine.generate on every "
                                   "rank -> gather and merge on rank 0; wall clock on rank 0")
        print(json.dumps(line))
    if dist is not None:
        dist.barrier()
        dist.destroy_process_group()


if __name__ == "__main__":
    main()
