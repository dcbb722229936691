"""Tensor-level wrappers over the C ABI: pointers, strides and the current CUDA stream.

Each function validates shapes/dtypes, passes raw device pointers to the library and
raises on a non-zero status.  Nothing here computes on the host.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, replace

import torch

from . import _cabi

_DEV_ERRORS = {1: "slot outside the KV pool", 2: "block id outside the KV pool",
               3: "position outside the cos/sin table", 4: "a bounded device wait ran out",
               5: "sequence length does not fit its block list"}
_DTYPE = {torch.bfloat16: 0, torch.float32: 1}      # the dtype argument of the entry points that take either


class LaunchCounter:
    """Counts kernels of this library enqueued through the wrappers below (graph replays add theirs)."""
    total = 0

    @classmethod
    def add(cls, n: int) -> None:
        cls.total += n


def _ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _need(t: torch.Tensor, dtype, name: str) -> None:
    if not t.is_cuda:
        raise ValueError(f"{name} must be a CUDA tensor (the kernels have no CPU path)")
    if t.dtype != dtype:
        raise TypeError(f"{name} must be {dtype}, got {t.dtype}")


def _heads_contiguous(t: torch.Tensor, name: str) -> None:
    if t.dim() != 3 or t.stride(2) != 1 or (t.shape[1] != 1 and t.stride(1) != t.shape[2]):
        raise ValueError(f"{name} must be [tokens, heads, head_dim] with contiguous heads")


@dataclass(frozen=True)
class AttnExtras:
    """What attention may have beyond a window and a cap: ``sinks`` (fp32 [heads], a score that takes its part of the softmax and brings
    no value), ``slopes`` (fp32 [heads], taken off a score per token of distance), ``head_gate`` ([tokens, heads], a head's output is
    multiplied by the sigmoid), ``keep_first`` (with a window: these first tokens stay visible)."""
    sinks: torch.Tensor | None = None
    slopes: torch.Tensor | None = None
    head_gate: torch.Tensor | None = None
    keep_first: int = 0

    def rows(self, start: int, end: int) -> "AttnExtras":
        """The same for a part of the step's tokens."""
        return self if self.head_gate is None else replace(self, head_gate=self.head_gate[start:end])

    def struct(self, q: torch.Tensor):
        """The C argument for queries ``q`` [tokens, heads, size]."""
        for t, name in ((self.sinks, "sinks"), (self.slopes, "slopes")):
            if t is not None:
                _need(t, torch.float32, name)
                assert t.numel() == q.shape[1] and t.is_contiguous()
        gate = self.head_gate
        if gate is not None:
            _need(gate, q.dtype, "head_gate")
            assert gate.shape == q.shape[:2] and gate.stride(1) == 1
        return ctypes.byref(_cabi.AttnExtras(_ptr(self.sinks), _ptr(self.slopes), _ptr(gate), 0 if gate is None else gate.stride(0),
                                             int(self.keep_first)))


def new_status(device) -> torch.Tensor:
    """A zeroed device int32[4] for kernels to record device-detected errors in."""
    return torch.zeros(4, dtype=torch.int32, device=device)


def check_status(status: torch.Tensor) -> None:
    """Synchronising read of a status word; raises if a kernel recorded an error."""
    code, detail, block, thread = status.tolist()
    if code:
        raise _cabi.KernelError(f"device error {code} ({_DEV_ERRORS.get(code, '?')}), detail {detail}, "
                                f"block {block}, thread {thread}")


def selftest_wait_timeout(status: torch.Tensor, limit: int = 1024) -> None:
    """Run the kernels' bounded mbarrier wait on a barrier nobody arrives at; ``status`` then reads
    ``[4, limit, 0, 0]`` (a wait timeout), and the stream carries on."""
    _need(status, torch.int32, "status")
    _cabi.check(_cabi.load().mvb_selftest_wait_timeout(_ptr(status), int(limit), _stream()), "mvb_selftest_wait_timeout")
    LaunchCounter.add(1)


def pack_prefill(meta: torch.Tensor, num_seqs: int, num_tokens: int, num_blocks_total: int, table_width: int,
                 block_size: int, want_table: bool, status: torch.Tensor | None = None) -> dict:
    """meta: device int32 = [seq_len(B) | cached_len(B) | blk_off(B+1) | blocks_flat | new_tokens(T)]."""
    _need(meta, torch.int32, "meta")
    dev = meta.device
    B, T = num_seqs, num_tokens
    base, es = meta.data_ptr(), 4
    o_seq, o_cached, o_off = 0, B, 2 * B
    o_blocks = o_off + B + 1
    o_tok = o_blocks + num_blocks_total
    assert meta.numel() >= o_tok + T
    out = {
        "input_ids": torch.empty(T, dtype=torch.int64, device=dev),
        "positions": torch.empty(T, dtype=torch.int64, device=dev),
        "slot_mapping": torch.empty(T, dtype=torch.int32, device=dev),
        "cu_seqlens_q": torch.empty(B + 1, dtype=torch.int32, device=dev),
        "cu_seqlens_k": torch.empty(B + 1, dtype=torch.int32, device=dev),
        "block_table": torch.empty(B, table_width, dtype=torch.int32, device=dev) if want_table else None,
    }
    rc = _cabi.load().mvb_pack_prefill(
        base + es * o_seq, base + es * o_cached, base + es * o_off, base + es * o_blocks, base + es * o_tok,
        B, T, table_width, block_size, _ptr(out["input_ids"]), _ptr(out["positions"]), _ptr(out["slot_mapping"]),
        _ptr(out["cu_seqlens_q"]), _ptr(out["cu_seqlens_k"]), _ptr(out["block_table"]), _ptr(status), _stream())
    _cabi.check(rc, "mvb_pack_prefill")
    LaunchCounter.add(1)
    return out


def pack_decode(meta: torch.Tensor, num_seqs: int, num_blocks_total: int, table_width: int, block_size: int,
                input_ids: torch.Tensor, positions: torch.Tensor, slot_mapping: torch.Tensor,
                cache_seqlens: torch.Tensor, block_table: torch.Tensor, padded_seqs: int | None = None,
                prev_sampled: torch.Tensor | None = None, status: torch.Tensor | None = None) -> None:
    """meta: device int32 = [seq_len(B) | blk_off(B+1) | blocks_flat | host_tokens(B) | src_index(B)].

    Outputs are written into the given (possibly static, graph-owned) buffers; rows
    ``num_seqs..padded_seqs-1`` become padding rows.
    """
    _need(meta, torch.int32, "meta")
    B = num_seqs
    padded = B if padded_seqs is None else padded_seqs
    base, es = meta.data_ptr(), 4
    o_off = B
    o_blocks = o_off + B + 1
    o_tok = o_blocks + num_blocks_total
    o_src = o_tok + B
    assert meta.numel() >= o_src + B
    assert block_table.dim() == 2 and block_table.stride(1) == 1 and block_table.shape[1] >= table_width
    for t, n in ((input_ids, "input_ids"), (positions, "positions")):
        _need(t, torch.int64, n)
        assert t.numel() >= padded and t.is_contiguous()
    for t, n in ((slot_mapping, "slot_mapping"), (cache_seqlens, "cache_seqlens"), (block_table, "block_table")):
        _need(t, torch.int32, n)
    assert block_table.shape[0] >= padded
    rc = _cabi.load().mvb_pack_decode(
        base, base + es * o_off, base + es * o_blocks, base + es * o_tok, _ptr(prev_sampled),
        base + es * o_src if prev_sampled is not None else None, B, padded, table_width, block_table.stride(0),
        block_size, _ptr(input_ids), _ptr(positions), _ptr(slot_mapping), _ptr(cache_seqlens), _ptr(block_table),
        _ptr(status), _stream())
    _cabi.check(rc, "mvb_pack_decode")
    LaunchCounter.add(1)


def rope_kv_write(q: torch.Tensor | None, k: torch.Tensor, v: torch.Tensor, positions: torch.Tensor | None,
                  cos_sin: torch.Tensor | None, slot_mapping: torch.Tensor | None,
                  k_cache: torch.Tensor | None, v_cache: torch.Tensor | None, k_in_place: bool = True,
                  status: torch.Tensor | None = None) -> None:
    """Rotate q (in place) and k, write k/v to their cache slots.  cos_sin=None: no rotation."""
    _need(k, torch.bfloat16, "k"); _need(v, torch.bfloat16, "v")
    _heads_contiguous(k, "k"); _heads_contiguous(v, "v")
    T, hkv, d = k.shape
    hq = 0
    if q is not None:
        _need(q, torch.bfloat16, "q"); _heads_contiguous(q, "q")
        assert q.shape[0] == T and q.shape[2] == d
        hq = q.shape[1]
    max_pos = 0
    if cos_sin is not None:
        _need(cos_sin, torch.float32, "cos_sin"); _need(positions, torch.int64, "positions")
        assert cos_sin.is_contiguous() and cos_sin.shape[1] == d and positions.numel() == T
        max_pos = cos_sin.shape[0]
    num_slots = 0
    if slot_mapping is not None:
        _need(slot_mapping, torch.int32, "slot_mapping")
        assert slot_mapping.numel() == T
        assert k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.shape[-2:] == (hkv, d)
        num_slots = k_cache.shape[0] * k_cache.shape[1]
    rc = _cabi.load().mvb_rope_kv_write(
        _ptr(q), q.stride(0) if q is not None else 0, _ptr(k), k.stride(0), _ptr(v), v.stride(0),
        _ptr(positions) if cos_sin is not None else None, _ptr(cos_sin), max_pos, _ptr(slot_mapping),
        _ptr(k_cache) if slot_mapping is not None else None, _ptr(v_cache) if slot_mapping is not None else None,
        num_slots, T, hq, hkv, d, 1 if k_in_place else 0, _ptr(status), _stream())
    _cabi.check(rc, "mvb_rope_kv_write")
    LaunchCounter.add(1)


def qk_norm_rope_kv_write(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, q_weight: torch.Tensor,
                          k_weight: torch.Tensor, eps: float, unit_offset: bool, positions: torch.Tensor,
                          cos_sin: torch.Tensor, slot_mapping: torch.Tensor | None, k_cache: torch.Tensor | None,
                          v_cache: torch.Tensor | None, k_in_place: bool = True,
                          status: torch.Tensor | None = None) -> None:
    """Per-head RMSNorm of q and k, RoPE and the cache write in one kernel; q (and k) updated in place."""
    for t, n in ((q, "q"), (k, "k"), (v, "v")):
        _need(t, torch.bfloat16, n); _heads_contiguous(t, n)
    _need(q_weight, torch.bfloat16, "q_weight"); _need(k_weight, torch.bfloat16, "k_weight")
    _need(cos_sin, torch.float32, "cos_sin"); _need(positions, torch.int64, "positions")
    T, hkv, d = k.shape
    hq = q.shape[1]
    assert q.shape[0] == T and q.shape[2] == d and cos_sin.is_contiguous() and cos_sin.shape[1] == d
    assert q_weight.numel() == d and k_weight.numel() == d and q_weight.is_contiguous() and k_weight.is_contiguous()
    num_slots = 0
    if slot_mapping is not None:
        _need(slot_mapping, torch.int32, "slot_mapping")
        assert slot_mapping.numel() == T and k_cache.is_contiguous() and v_cache.is_contiguous()
        num_slots = k_cache.shape[0] * k_cache.shape[1]
    rc = _cabi.load().mvb_qk_norm_rope_kv_write(
        _ptr(q), q.stride(0), _ptr(k), k.stride(0), _ptr(v), v.stride(0), _ptr(q_weight), _ptr(k_weight), float(eps),
        1 if unit_offset else 0, _ptr(positions), _ptr(cos_sin), cos_sin.shape[0], _ptr(slot_mapping),
        _ptr(k_cache) if slot_mapping is not None else None, _ptr(v_cache) if slot_mapping is not None else None,
        num_slots, T, hq, hkv, d, 1 if k_in_place else 0, _ptr(status), _stream())
    _cabi.check(rc, "mvb_qk_norm_rope_kv_write")
    LaunchCounter.add(1)


def decode_workspace(max_seqs: int, num_q_heads: int, head_dim: int, device) -> torch.Tensor:
    n = _cabi.load().mvb_decode_workspace_bytes(max_seqs, num_q_heads, head_dim)
    if n == 0:
        raise ValueError("bad decode workspace shape")
    return torch.empty(n, dtype=torch.uint8, device=device)


def decode_plan(cache_seqlens: torch.Tensor, window_left: int, num_q_heads: int, num_kv_heads: int,
                head_dim: int, workspace: torch.Tensor, block_table: torch.Tensor | None = None,
                block_size: int = 0, keep_first: int = 0) -> None:
    """Plan the split of one decode step.  With ``block_table`` (the one the attention calls will get)
    the plan also records each CTA's first block id, sparing every layer a dependent load.  ``keep_first`` (needs the table): as
    in the attention's ``AttnExtras``."""
    _need(cache_seqlens, torch.int32, "cache_seqlens")
    if block_table is not None:
        _need(block_table, torch.int32, "block_table")
        assert block_table.stride(1) == 1 and block_table.shape[0] >= cache_seqlens.numel() and block_size > 0
        rc = _cabi.load().mvb_decode_plan_ext(
            _ptr(cache_seqlens), _ptr(block_table), block_table.stride(0), block_size, cache_seqlens.numel(),
            window_left, int(keep_first), num_q_heads, num_kv_heads, head_dim, _ptr(workspace), workspace.numel(), _stream())
    else:
        assert keep_first == 0
        rc = _cabi.load().mvb_decode_plan(_ptr(cache_seqlens), cache_seqlens.numel(), window_left, num_q_heads,
                                          num_kv_heads, head_dim, _ptr(workspace), workspace.numel(), _stream())
    _cabi.check(rc, "mvb_decode_plan")
    LaunchCounter.add(1)


def decode_attn(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, cache_seqlens: torch.Tensor,
                block_table: torch.Tensor, scale: float, window_left: int, workspace: torch.Tensor,
                out: torch.Tensor | None = None, status: torch.Tensor | None = None, softcap: float = 0.0,
                out_scale: float = 1.0, extras: AttnExtras | None = None) -> torch.Tensor:
    """q [B,Hq,D]; the plan for (cache_seqlens, window_left) must already be in ``workspace``.  ``softcap`` > 0: scores
    pass ``softcap * tanh(score / softcap)``; ``out_scale`` multiplies the output."""
    _need(q, torch.bfloat16, "q"); _heads_contiguous(q, "q")
    _need(cache_seqlens, torch.int32, "cache_seqlens"); _need(block_table, torch.int32, "block_table")
    B, hq, d = q.shape
    nblk, bs, hkv, d2 = k_cache.shape
    assert d2 == d and k_cache.is_contiguous() and v_cache.is_contiguous() and v_cache.shape == k_cache.shape
    assert block_table.dim() == 2 and block_table.stride(1) == 1 and block_table.shape[0] >= B
    assert cache_seqlens.numel() >= B
    if out is None:
        out = torch.empty(B, hq, d, dtype=torch.bfloat16, device=q.device)
    args = (_ptr(q), q.stride(0), _ptr(k_cache), _ptr(v_cache), nblk, bs, _ptr(cache_seqlens), _ptr(block_table),
            block_table.stride(0), block_table.shape[1], B, hq, hkv, d, float(scale), window_left, _ptr(out),
            out.stride(0), _ptr(workspace), workspace.numel())
    if extras is None:
        rc = _cabi.load().mvb_decode_attn_capped(*args, float(softcap), float(out_scale), _ptr(status), _stream())
    else:
        assert softcap == 0
        rc = _cabi.load().mvb_decode_attn_ext(*args, float(out_scale), extras.struct(q), _ptr(status), _stream())
    _cabi.check(rc, "mvb_decode_attn_capped")
    LaunchCounter.add(1)
    return out


def decode_attn_static(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, cache_seqlens: torch.Tensor,
                       block_table: torch.Tensor, scale: float, window_left: int, out: torch.Tensor,
                       status: torch.Tensor | None = None) -> torch.Tensor:
    """Decode attention that brings its own scratch (``mvb_decode_attn_static``).

    For callers that have no way to allocate a workspace next to this call: the plan and the partial
    results live in an 8 MiB array inside the library, so the only buffers involved are the ones passed
    here, ``out`` included.  Calls on one device share that array and must not overlap on the GPU;
    the first call on a device should happen outside stream capture.  Raises ``KernelError`` when the
    request is too large for the built-in array.
    """
    _need(q, torch.bfloat16, "q"); _heads_contiguous(q, "q")
    _need(cache_seqlens, torch.int32, "cache_seqlens"); _need(block_table, torch.int32, "block_table")
    _need(out, torch.bfloat16, "out")
    B, hq, d = q.shape
    nblk, bs, hkv, _ = k_cache.shape
    assert k_cache.is_contiguous() and v_cache.is_contiguous() and block_table.stride(1) == 1
    rc = _cabi.load().mvb_decode_attn_static(
        _ptr(q), q.stride(0), _ptr(k_cache), _ptr(v_cache), nblk, bs, _ptr(cache_seqlens), _ptr(block_table),
        block_table.stride(0), block_table.shape[1], B, hq, hkv, d, float(scale), window_left, _ptr(out),
        out.stride(0), _ptr(status), _stream())
    _cabi.check(rc, "mvb_decode_attn_static")
    LaunchCounter.add(2)
    return out


def prefill_item_rows(num_q_heads: int, num_kv_heads: int, head_dim: int) -> int:
    """Rows of q that one work item of the prefill kernel covers (128 or 256; a property of the head layout)."""
    rows = _cabi.load().mvb_prefill_item_rows(num_q_heads, num_kv_heads, head_dim)
    _cabi.check(min(rows, 0), "mvb_prefill_item_rows")
    return rows


def build_prefill_items(q_lens, k_lens, item_rows: int):
    """The work list of a prefill launch: int32 [n, 2] of (sequence, query block), every query block of every
    sequence once, the blocks that see the most keys first (the order in which the GPU takes them).  Pure host
    arithmetic on the per-sequence lengths the packing step already has; numpy in, numpy out."""
    import numpy as np
    q_lens = np.asarray(q_lens, np.int64)
    k_lens = np.asarray(k_lens, np.int64)
    n_qb = (q_lens + item_rows - 1) // item_rows
    seq = np.repeat(np.arange(q_lens.size, dtype=np.int64), n_qb)
    first = np.cumsum(n_qb) - n_qb
    qb = np.arange(int(n_qb.sum()), dtype=np.int64) - np.repeat(first, n_qb)
    # keys visible to the block's last row: its position + 1
    visible = k_lens[seq] - q_lens[seq] + np.minimum((qb + 1) * item_rows, q_lens[seq])
    order = np.argsort(-visible, kind="stable")
    return np.stack([seq[order], qb[order]], axis=1).astype(np.int32)


def prefill_attn(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_seqlens_q: torch.Tensor,
                 cu_seqlens_k: torch.Tensor, max_seqlen_q: int, scale: float, window_left: int = -1,
                 block_table: torch.Tensor | None = None, out: torch.Tensor | None = None,
                 status: torch.Tensor | None = None, items: torch.Tensor | None = None, softcap: float = 0.0,
                 out_scale: float = 1.0, extras: AttnExtras | None = None) -> torch.Tensor:
    """q [Tq,Hq,D]; k/v dense [Tk,Hkv,D] (block_table None) or the paged pool [blocks,bs,Hkv,D].

    ``items`` (int32 [n, 2] on the device, from ``build_prefill_items``) gives the launch its work as a list of
    (sequence, query block) pairs instead of a grid over the longest sequence's block count: same result, no
    empty block indices, the longest blocks first."""
    _need(q, torch.bfloat16, "q"); _heads_contiguous(q, "q")
    _need(cu_seqlens_q, torch.int32, "cu_seqlens_q"); _need(cu_seqlens_k, torch.int32, "cu_seqlens_k")
    Tq, hq, d = q.shape
    if block_table is None:
        _heads_contiguous(k, "k"); _heads_contiguous(v, "v")
        kv_rows, hkv, k_stride, v_stride, bs, tstride = k.shape[0], k.shape[1], k.stride(0), v.stride(0), 0, 0
    else:
        _need(block_table, torch.int32, "block_table")
        assert k.dim() == 4 and k.is_contiguous() and v.is_contiguous()
        nblk, bs, hkv, _ = k.shape
        kv_rows, k_stride, v_stride, tstride = nblk * bs, hkv * d, hkv * d, block_table.stride(0)
    if out is None:
        out = torch.empty(Tq, hq, d, dtype=torch.bfloat16, device=q.device)
    use = items is not None and 0 < items.shape[0] <= 65535
    if use:
        _need(items, torch.int32, "items")
        assert items.dim() == 2 and items.shape[1] == 2 and items.is_contiguous()
    args = (_ptr(q), q.stride(0), _ptr(k), k_stride, _ptr(v), v_stride, kv_rows, _ptr(cu_seqlens_q), _ptr(cu_seqlens_k),
            _ptr(block_table), tstride, bs, cu_seqlens_q.numel() - 1, Tq, int(max_seqlen_q), hq, hkv, d, float(scale),
            window_left, _ptr(out), out.stride(0), _ptr(items) if use else None, items.shape[0] if use else 0)
    if extras is None:
        rc = _cabi.load().mvb_prefill_attn_capped(*args, float(softcap), float(out_scale), _ptr(status), _stream())
    else:
        assert softcap == 0
        rc = _cabi.load().mvb_prefill_attn_ext(*args, float(out_scale), extras.struct(q), _ptr(status), _stream())
    _cabi.check(rc, "mvb_prefill_attn_capped")
    LaunchCounter.add(1)
    return out


def sample(logits: torch.Tensor, temperatures: torch.Tensor | None = None, top_k: torch.Tensor | None = None,
           seed: int = 0, offset: int = 0, out: torch.Tensor | None = None, top_p: torch.Tensor | None = None,
           scatter_table: torch.Tensor | None = None, scatter_index: torch.Tensor | None = None) -> torch.Tensor:
    """logits bf16 [B,V] -> int64 [B].  top_k and top_p None: greedy; else temperature/top-k/top-p/Gumbel-max.

    With ``scatter_table`` (int64) and ``scatter_index`` (int32 [B]) the tokens are also written to
    ``scatter_table[scatter_index]`` on the device."""
    _need(logits, torch.bfloat16, "logits")
    assert logits.dim() == 2 and logits.stride(1) == 1
    B, V = logits.shape
    if temperatures is not None:
        _need(temperatures, torch.float32, "temperatures")
    if top_k is not None:
        _need(top_k, torch.int32, "top_k")
    if out is None:
        out = torch.empty(B, dtype=torch.int64, device=logits.device)
    if scatter_table is not None:
        _need(scatter_table, torch.int64, "scatter_table"); _need(scatter_index, torch.int32, "scatter_index")
        assert scatter_index.numel() >= B
    if top_p is not None:
        _need(top_p, torch.float32, "top_p")
    rc = _cabi.load().mvb_sample(_ptr(logits), logits.stride(0), B, V, _ptr(temperatures), _ptr(top_k), _ptr(top_p),
                                 seed & (2**64 - 1), offset & (2**64 - 1), _ptr(out), _ptr(scatter_table),
                                 _ptr(scatter_index), None, _stream())
    _cabi.check(rc, "mvb_sample")
    LaunchCounter.add(1)
    return out


def act_mul(gate_up: torch.Tensor, intermediate: int, gelu_tanh: bool, out: torch.Tensor | None = None) -> torch.Tensor:
    """``act(gate) * up`` on a packed ``[rows, 2 * intermediate]`` projection (SiLU, or tanh-GELU)."""
    _need(gate_up, torch.bfloat16, "gate_up")
    assert gate_up.dim() == 2 and gate_up.stride(1) == 1 and gate_up.shape[1] == 2 * intermediate
    rows = gate_up.shape[0]
    if out is None:
        out = torch.empty(rows, intermediate, dtype=torch.bfloat16, device=gate_up.device)
    rc = _cabi.load().mvb_act_mul(_ptr(gate_up), gate_up.stride(0), _ptr(out), out.stride(0), rows, intermediate,
                                  1 if gelu_tanh else 0, _stream())
    _cabi.check(rc, "mvb_act_mul")
    LaunchCounter.add(1)
    return out


def add_rmsnorm(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float, unit_offset: bool,
                y_weight: torch.Tensor | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """``x += y`` (or ``x += rmsnorm(y, y_weight)``) in place, returns ``rmsnorm(x, weight)``."""
    _need(x, torch.bfloat16, "x"); _need(y, torch.bfloat16, "y"); _need(weight, torch.bfloat16, "weight")
    assert x.dim() == 2 and x.is_contiguous() and y.shape == x.shape and y.stride(1) == 1
    rows, hidden = x.shape
    if out is None:
        out = torch.empty_like(x)
    rc = _cabi.load().mvb_add_rmsnorm(_ptr(x), _ptr(y), y.stride(0), _ptr(y_weight), _ptr(weight), _ptr(out), rows,
                                      hidden, float(eps), 1 if unit_offset else 0, _stream())
    _cabi.check(rc, "mvb_add_rmsnorm")
    LaunchCounter.add(1)
    return out


def add_rmsnorm_last_tokens(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float, unit_offset: bool,
                            cu_seqlens_q: torch.Tensor, y_weight: torch.Tensor | None = None) -> torch.Tensor:
    """``rmsnorm(x + y)`` (or ``x + rmsnorm(y, y_weight)``) for the last token of every sequence only:
    ``[num_seqs, hidden]``, row r from source row ``cu_seqlens_q[r + 1] - 1``.  ``x`` is left untouched."""
    _need(x, torch.bfloat16, "x"); _need(y, torch.bfloat16, "y"); _need(weight, torch.bfloat16, "weight")
    _need(cu_seqlens_q, torch.int32, "cu_seqlens_q")
    assert x.dim() == 2 and x.is_contiguous() and y.shape == x.shape and y.stride(1) == 1
    num_seqs, hidden = cu_seqlens_q.numel() - 1, x.shape[1]
    out = torch.empty(num_seqs, hidden, dtype=torch.bfloat16, device=x.device)
    rc = _cabi.load().mvb_add_rmsnorm_last_tokens(_ptr(x), _ptr(y), y.stride(0), _ptr(y_weight), _ptr(weight), _ptr(out),
                                                  _ptr(cu_seqlens_q), num_seqs, hidden, float(eps),
                                                  1 if unit_offset else 0, _stream())
    _cabi.check(rc, "mvb_add_rmsnorm_last_tokens")
    LaunchCounter.add(1)
    return out


def lm_head_argmax_scratch(max_rows: int, device) -> torch.Tensor:
    """Zeroed scratch for ``lm_head_argmax`` (every call leaves it zeroed again)."""
    n = _cabi.load().mvb_lm_head_argmax_scratch_bytes(max_rows)
    return torch.zeros(n, dtype=torch.uint8, device=device)


def lm_head_argmax(hidden_states: torch.Tensor, weight: torch.Tensor, scratch: torch.Tensor,
                   out: torch.Tensor | None = None, scatter_table: torch.Tensor | None = None,
                   scatter_index: torch.Tensor | None = None, status: torch.Tensor | None = None) -> torch.Tensor:
    """``argmax(hidden_states @ weight.T)`` per row over bf16-rounded logits, without materialising them."""
    _need(hidden_states, torch.bfloat16, "hidden_states"); _need(weight, torch.bfloat16, "weight")
    assert hidden_states.dim() == 2 and weight.dim() == 2 and hidden_states.stride(1) == 1 and weight.stride(1) == 1
    rows, hidden = hidden_states.shape
    vocab = weight.shape[0]
    assert weight.shape[1] == hidden
    if out is None:
        out = torch.empty(rows, dtype=torch.int64, device=hidden_states.device)
    if scatter_table is not None:
        _need(scatter_table, torch.int64, "scatter_table"); _need(scatter_index, torch.int32, "scatter_index")
        assert scatter_index.numel() >= rows
    rc = _cabi.load().mvb_lm_head_argmax(_ptr(hidden_states), hidden_states.stride(0), _ptr(weight), weight.stride(0), rows,
                                         hidden, vocab, _ptr(out), _ptr(scatter_table), _ptr(scatter_index), _ptr(scratch),
                                         scratch.numel(), _ptr(status), _stream())
    _cabi.check(rc, "mvb_lm_head_argmax")
    LaunchCounter.add(1)
    return out


# ---- kernels that run in bf16 or fp32 -----------------------------------------------------------------------
def _dtype_of(t: torch.Tensor, name: str) -> int:
    if not t.is_cuda:
        raise ValueError(f"{name} must be a CUDA tensor (the kernels have no CPU path)")
    if t.dtype not in _DTYPE:
        raise TypeError(f"{name} must be bfloat16 or float32, got {t.dtype}")
    return _DTYPE[t.dtype]


def _same(dtype, **tensors) -> None:
    for name, t in tensors.items():
        if t is not None:
            _need(t, dtype, name)


def any_attn(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, positions: torch.Tensor, scale: float,
             window_left: int = -1, cu_seqlens_q: torch.Tensor | None = None, cu_seqlens_k: torch.Tensor | None = None,
             block_table: torch.Tensor | None = None, cache_seqlens: torch.Tensor | None = None, softcap: float = 0.0,
             out_scale: float = 1.0, out: torch.Tensor | None = None, status: torch.Tensor | None = None,
             extras: AttnExtras | None = None) -> torch.Tensor:
    """Attention of any head size, group size and dtype (one warp per token and head).  k/v are the paged pool with a
    ``block_table``, else dense rows; without ``cu_seqlens_q`` every row is a sequence of its own."""
    code = _dtype_of(q, "q")
    _same(q.dtype, k=k, v=v)
    _heads_contiguous(q, "q")
    _need(positions, torch.int64, "positions")
    tokens, hq, d = q.shape
    if block_table is not None:
        _need(block_table, torch.int32, "block_table")
        assert k.dim() == 4 and k.is_contiguous() and v.is_contiguous() and v.shape == k.shape and block_table.stride(1) == 1
        nblk, bs, hkv, _ = k.shape
        kv_rows, ks, vs, tstride, width = nblk * bs, hkv * d, hkv * d, block_table.stride(0), block_table.shape[1]
    else:
        _heads_contiguous(k, "k"); _heads_contiguous(v, "v")
        _need(cu_seqlens_k, torch.int32, "cu_seqlens_k")
        kv_rows, hkv, ks, vs, bs, tstride, width = k.shape[0], k.shape[1], k.stride(0), v.stride(0), 0, 0, 0
    num_seqs = tokens if cu_seqlens_q is None else cu_seqlens_q.numel() - 1
    if out is None:
        out = torch.empty(tokens, hq, d, dtype=q.dtype, device=q.device)
    rc = _cabi.load().mvb_any_attn_ext(
        code, _ptr(q), q.stride(0), _ptr(k), ks, _ptr(v), vs, kv_rows, _ptr(block_table), tstride, width, bs,
        _ptr(cu_seqlens_q), _ptr(cu_seqlens_k), _ptr(positions), _ptr(cache_seqlens), num_seqs, tokens, hq, hkv, d,
        float(scale), window_left, float(softcap), float(out_scale), None if extras is None else extras.struct(q), _ptr(out),
        out.stride(0), _ptr(status), _stream())
    _cabi.check(rc, "mvb_any_attn_ext")
    LaunchCounter.add(1)
    return out


def rope_kv_write_f32(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, positions: torch.Tensor, cos_sin: torch.Tensor,
                      slot_mapping: torch.Tensor | None, k_cache: torch.Tensor | None, v_cache: torch.Tensor | None,
                      k_in_place: bool = True, status: torch.Tensor | None = None) -> None:
    """``rope_kv_write`` for fp32 activations and pools."""
    _same(torch.float32, q=q, k=k, v=v, cos_sin=cos_sin)
    for t, n in ((q, "q"), (k, "k"), (v, "v")):
        _heads_contiguous(t, n)
    _need(positions, torch.int64, "positions")
    tokens, hkv, d = k.shape
    assert cos_sin.is_contiguous() and cos_sin.shape[1] == d and q.shape[2] == d
    num_slots = 0
    if slot_mapping is not None:
        _need(slot_mapping, torch.int32, "slot_mapping")
        _same(torch.float32, k_cache=k_cache, v_cache=v_cache)
        assert k_cache.is_contiguous() and v_cache.is_contiguous()
        num_slots = k_cache.shape[0] * k_cache.shape[1]
    rc = _cabi.load().mvb_rope_kv_write_f32(
        _ptr(q), q.stride(0), _ptr(k), k.stride(0), _ptr(v), v.stride(0), _ptr(positions), _ptr(cos_sin), cos_sin.shape[0],
        _ptr(slot_mapping), _ptr(k_cache) if slot_mapping is not None else None,
        _ptr(v_cache) if slot_mapping is not None else None, num_slots, tokens, q.shape[1], hkv, d, 1 if k_in_place else 0,
        _ptr(status), _stream())
    _cabi.check(rc, "mvb_rope_kv_write_f32")
    LaunchCounter.add(1)


def rope_norm_kv_write(q: torch.Tensor, k: torch.Tensor | None, v: torch.Tensor | None, positions: torch.Tensor,
                       cos_sin: torch.Tensor | None, slot_mapping: torch.Tensor | None, k_cache: torch.Tensor | None,
                       v_cache: torch.Tensor | None, k_in_place: bool = True, norm_dim: int = 0, eps: float = 0.0,
                       status: torch.Tensor | None = None) -> None:
    """Rotates q (in place) and k, divides every head by the root mean square of its ``norm_dim`` used coordinates (0: no norm), and
    writes k and v to their cache slots.  ``cos_sin`` None: no rotation; ``k`` None: q alone.  Either dtype, any even head size."""
    code = _dtype_of(q, "q")
    _same(q.dtype, k=k, v=v)
    _same(torch.float32, cos_sin=cos_sin)
    _need(positions, torch.int64, "positions")
    for t, n in ((q, "q"), (k, "k"), (v, "v")):
        if t is not None:
            _heads_contiguous(t, n)
    tokens, hq, d = q.shape
    hkv, num_slots = 0 if k is None else k.shape[1], 0
    assert k is None or (v is not None and k.shape == v.shape == (tokens, hkv, d))
    assert cos_sin is None or (cos_sin.is_contiguous() and cos_sin.shape[1] == d)
    if k is None:
        slot_mapping = None
    if slot_mapping is not None:
        _need(slot_mapping, torch.int32, "slot_mapping")
        _same(q.dtype, k_cache=k_cache, v_cache=v_cache)
        assert k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.shape[-2:] == (hkv, d)
        num_slots = k_cache.shape[0] * k_cache.shape[1]
    cached = slot_mapping is not None
    rc = _cabi.load().mvb_rope_norm_kv_write(
        code, _ptr(q), q.stride(0), _ptr(k), 0 if k is None else k.stride(0), _ptr(v), 0 if v is None else v.stride(0), _ptr(positions),
        _ptr(cos_sin), 0 if cos_sin is None else cos_sin.shape[0], _ptr(slot_mapping), _ptr(k_cache) if cached else None,
        _ptr(v_cache) if cached else None, num_slots, tokens, hq, hkv, d, 1 if k_in_place else 0, int(norm_dim), float(eps), _ptr(status),
        _stream())
    _cabi.check(rc, "mvb_rope_norm_kv_write")
    LaunchCounter.add(1)


@dataclass(frozen=True)
class RowNorm:
    """Norms in front of the rotation: q and k over the root mean square of their whole row (``q_dim``, ``k_dim`` used coordinates) times
    weights [heads * head_dim] (None: neither), values over that of their head's ``v_dim`` used coordinates (0: not)."""
    q_weight: torch.Tensor | None
    k_weight: torch.Tensor | None
    q_dim: int
    k_dim: int
    v_dim: int
    eps: float


def row_norm_rope_kv_write(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, norm: RowNorm, positions: torch.Tensor,
                           cos_sin: torch.Tensor | None, slot_mapping: torch.Tensor | None, k_cache: torch.Tensor | None,
                           v_cache: torch.Tensor | None, kv_in_place: bool = True, status: torch.Tensor | None = None) -> None:
    """``norm``, then the rotation (``cos_sin`` None: none), then the cache write; q in place, k and v too if asked.  Either dtype, any even
    head size."""
    code = _dtype_of(q, "q")
    _same(q.dtype, k=k, v=v, q_weight=norm.q_weight, k_weight=norm.k_weight)
    _same(torch.float32, cos_sin=cos_sin)
    _need(positions, torch.int64, "positions")
    for t, n in ((q, "q"), (k, "k"), (v, "v")):
        _heads_contiguous(t, n)
    (tokens, hq, d), hkv, num_slots = q.shape, k.shape[1], 0
    assert k.shape == v.shape == (tokens, hkv, d) and (cos_sin is None or (cos_sin.is_contiguous() and cos_sin.shape[1] == d))
    for w, heads in ((norm.q_weight, hq), (norm.k_weight, hkv)):
        assert w is None or (w.is_contiguous() and w.numel() == heads * d)
    if slot_mapping is not None:
        _need(slot_mapping, torch.int32, "slot_mapping")
        _same(q.dtype, k_cache=k_cache, v_cache=v_cache)
        assert k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.shape[-2:] == (hkv, d)
        num_slots = k_cache.shape[0] * k_cache.shape[1]
    cached = slot_mapping is not None
    rc = _cabi.load().mvb_row_norm_rope_kv_write(
        code, _ptr(q), q.stride(0), _ptr(k), k.stride(0), _ptr(v), v.stride(0), _ptr(norm.q_weight), _ptr(norm.k_weight), norm.q_dim,
        norm.k_dim, norm.v_dim, float(norm.eps), _ptr(positions), _ptr(cos_sin), 0 if cos_sin is None else cos_sin.shape[0],
        _ptr(slot_mapping), _ptr(k_cache) if cached else None, _ptr(v_cache) if cached else None, num_slots, tokens, hq, hkv, d,
        1 if kv_in_place else 0, _ptr(status), _stream())
    _cabi.check(rc, "mvb_row_norm_rope_kv_write")
    LaunchCounter.add(1)


def residual_norm(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float, y_weight: torch.Tensor | None = None,
                  row_ends: torch.Tensor | None = None) -> torch.Tensor:
    """fp32 residual stream: ``x += y`` (or ``x += rmsnorm(y, y_weight)``) in place, returns ``rmsnorm(x, weight)`` in y's
    dtype.  With ``row_ends`` (int32 [n + 1]) only rows ``row_ends[1:] - 1`` are produced and ``x`` is left as it is."""
    code = _dtype_of(y, "y")
    _need(x, torch.float32, "x"); _same(y.dtype, weight=weight, y_weight=y_weight)
    assert x.dim() == 2 and x.is_contiguous() and y.shape == x.shape and y.stride(1) == 1
    rows = x.shape[0]
    if row_ends is not None:
        _need(row_ends, torch.int32, "row_ends")
        rows = row_ends.numel() - 1
    out = torch.empty(rows, x.shape[1], dtype=y.dtype, device=x.device)
    if rows == 0:
        return out
    rc = _cabi.load().mvb_residual_norm(code, _ptr(x), _ptr(y), y.stride(0), _ptr(y_weight), _ptr(weight), _ptr(out),
                                        _ptr(row_ends), rows, x.shape[1], float(eps), _stream())
    _cabi.check(rc, "mvb_residual_norm")
    LaunchCounter.add(1)
    return out


def embed_norm(ids: torch.Tensor, table: torch.Tensor, weight: torch.Tensor, eps: float,
               status: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """(fp32 residual stream ``table[ids]``, ``rmsnorm`` of it in the table's dtype)."""
    code = _dtype_of(table, "table")
    _need(ids, torch.int64, "ids"); _same(table.dtype, weight=weight)
    assert table.is_contiguous() and ids.dim() == 1 and ids.is_contiguous()
    rows, width = ids.numel(), table.shape[1]
    x = torch.empty(rows, width, dtype=torch.float32, device=table.device)
    out = torch.empty(rows, width, dtype=table.dtype, device=table.device)
    rc = _cabi.load().mvb_embed_norm(code, _ptr(ids), _ptr(table), table.shape[0], _ptr(x), _ptr(weight), _ptr(out), rows,
                                     width, float(eps), _ptr(status), _stream())
    _cabi.check(rc, "mvb_embed_norm")
    LaunchCounter.add(1)
    return x, out


def residual_norm_pair(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, weight2: torch.Tensor | None, eps: float,
                       extra: torch.Tensor | None = None, extra_index: torch.Tensor | None = None,
                       row_ends: torch.Tensor | None = None, own: torch.Tensor | None = None, own_weights: torch.Tensor | None = None,
                       status: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor | None]:
    """``x += y`` in place, and ``extra[extra_index[row, j]]`` for every j (an index of -1: nothing), and ``own_weights[row] own[row]``;
    returns the norms of x with ``weight`` and ``weight2`` (None: None) in y's dtype.  ``row_ends`` as in ``residual_norm``."""
    code = _dtype_of(y, "y")
    _need(x, torch.float32, "x"); _same(y.dtype, weight=weight, weight2=weight2, extra=extra, own=own)
    assert x.dim() == 2 and x.is_contiguous() and y.shape == x.shape and y.stride(1) == 1
    rows, width = x.shape
    if row_ends is not None:
        _need(row_ends, torch.int32, "row_ends")
        rows = row_ends.numel() - 1
    count = 0
    if extra is not None:
        _need(extra_index, torch.int32, "extra_index")
        count = extra_index.shape[1]
        assert extra_index.shape[0] == x.shape[0] and extra_index.is_contiguous() and extra.shape[1] >= width and extra.stride(1) == 1
    if own_weights is not None:
        _need(own_weights, torch.float32, "own_weights")
        assert own.shape == x.shape and own.stride(1) == 1 and own_weights.is_contiguous() and own_weights.numel() == x.shape[0]
    out = torch.empty(rows, width, dtype=y.dtype, device=x.device)
    out2 = None if weight2 is None else torch.empty_like(out)
    if rows == 0:
        return out, out2
    rc = _cabi.load().mvb_residual_norm_pair_ext(
        code, _ptr(x), _ptr(y), y.stride(0), _ptr(extra), 0 if extra is None else extra.stride(0), 0 if extra is None else extra.shape[0],
        _ptr(extra_index), count, _ptr(own) if own_weights is not None else None, 0 if own is None else own.stride(0), _ptr(own_weights),
        _ptr(weight), _ptr(out), _ptr(weight2), _ptr(out2), _ptr(row_ends), rows, width, float(eps), _ptr(status), _stream())
    _cabi.check(rc, "mvb_residual_norm_pair_ext")
    LaunchCounter.add(1)
    return out, out2


def embed_norm_pair(ids: torch.Tensor, table: torch.Tensor, scale: float, weight: torch.Tensor, weight2: torch.Tensor | None, eps: float,
                    status: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor, torch.Tensor | None]:
    """(fp32 residual stream ``scale * table[ids]``, its norms with ``weight`` and ``weight2`` in the table's dtype)."""
    code = _dtype_of(table, "table")
    _need(ids, torch.int64, "ids"); _same(table.dtype, weight=weight, weight2=weight2)
    assert table.is_contiguous() and ids.dim() == 1 and ids.is_contiguous()
    rows, width = ids.numel(), table.shape[1]
    x = torch.empty(rows, width, dtype=torch.float32, device=table.device)
    out = torch.empty(rows, width, dtype=table.dtype, device=table.device)
    out2 = None if weight2 is None else torch.empty_like(out)
    rc = _cabi.load().mvb_embed_norm_pair(code, _ptr(ids), _ptr(table), table.shape[0], float(scale), _ptr(x), _ptr(weight), _ptr(out),
                                          _ptr(weight2), _ptr(out2), rows, width, float(eps), _ptr(status), _stream())
    _cabi.check(rc, "mvb_embed_norm_pair")
    LaunchCounter.add(1)
    return x, out, out2


def glu(gate_up: torch.Tensor, intermediate: int, limit: float = float("inf"), alpha: float = 1.0, offset: float = 0.0,
        row_gate: torch.Tensor | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """``g sigmoid(alpha g) (u + offset)``, ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``, packed ``[gate | up]``; times
    ``sigmoid(row_gate)`` ([rows], any stride) of the row.  The defaults are the SiLU-gated unit."""
    code = _dtype_of(gate_up, "gate_up")
    assert gate_up.dim() == 2 and gate_up.stride(1) == 1 and gate_up.shape[1] == 2 * intermediate
    rows = gate_up.shape[0]
    _same(gate_up.dtype, row_gate=row_gate, out=out)
    assert row_gate is None or row_gate.shape == (rows,)
    if out is None:
        out = torch.empty(rows, intermediate, dtype=gate_up.dtype, device=gate_up.device)
    assert out.shape == (rows, intermediate) and out.stride(1) == 1
    rc = _cabi.load().mvb_glu(code, _ptr(gate_up), gate_up.stride(0), _ptr(out), out.stride(0), rows, intermediate, float(limit),
                              float(alpha), float(offset), _ptr(row_gate), 0 if row_gate is None else row_gate.stride(0), _stream())
    _cabi.check(rc, "mvb_glu")
    LaunchCounter.add(1)
    return out


def clamped_glu(gate_up: torch.Tensor, intermediate: int, limit: float, alpha: float) -> torch.Tensor:
    """``glu`` with one added to the clamped up projection."""
    return glu(gate_up, intermediate, limit, alpha, 1.0)


def xielu(z: torch.Tensor, act: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``act[0] z^2 + z / 2`` for z > 0, ``act[1] (e^z - 1 - z) + z / 2`` for z <= 0 (``act``: fp32 [2])."""
    code = _dtype_of(z, "z")
    _need(act, torch.float32, "act")
    if out is None:
        out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    _same(z.dtype, out=out)
    assert z.dim() == 2 and z.stride(1) == 1 and out.shape == z.shape and out.stride(1) == 1 and act.numel() == 2
    rc = _cabi.load().mvb_xielu(code, _ptr(z), z.stride(0), _ptr(out), out.stride(0), z.shape[0], z.shape[1], _ptr(act), _stream())
    _cabi.check(rc, "mvb_xielu")
    LaunchCounter.add(1)
    return out


def cap_logits(logits: torch.Tensor, cap: float, out_dtype: torch.dtype) -> torch.Tensor:
    """``cap * tanh(logits / cap)`` (``cap`` 0: the logits as they are) in ``out_dtype``."""
    code = _dtype_of(logits, "logits")
    assert logits.dim() == 2 and logits.stride(1) == 1
    out = torch.empty(logits.shape, dtype=out_dtype, device=logits.device)
    rc = _cabi.load().mvb_cap_logits(code, _DTYPE[out_dtype], _ptr(logits), logits.stride(0), _ptr(out), out.stride(0),
                                     logits.shape[0], logits.shape[1], float(cap), _stream())
    _cabi.check(rc, "mvb_cap_logits")
    LaunchCounter.add(1)
    return out


def argmax_f32(logits: torch.Tensor, scatter_table: torch.Tensor | None = None,
               scatter_index: torch.Tensor | None = None) -> torch.Tensor:
    """Greedy tokens of fp32 logits (the lowest column wins ties)."""
    _need(logits, torch.float32, "logits")
    assert logits.dim() == 2 and logits.stride(1) == 1
    out = torch.empty(logits.shape[0], dtype=torch.int64, device=logits.device)
    if scatter_table is not None:
        _need(scatter_table, torch.int64, "scatter_table"); _need(scatter_index, torch.int32, "scatter_index")
    rc = _cabi.load().mvb_argmax_f32(_ptr(logits), logits.stride(0), logits.shape[0], logits.shape[1], _ptr(out),
                                     _ptr(scatter_table), _ptr(scatter_index), _stream())
    _cabi.check(rc, "mvb_argmax_f32")
    LaunchCounter.add(1)
    return out


def _state_args(state: torch.Tensor | None, slots: torch.Tensor | None):
    """(state pointer, slot-index pointer, number of slots); a step without slots keeps no state."""
    if state is None or slots is None:
        return None, None, 0
    _need(slots, torch.int32, "state_slots")
    assert state.is_contiguous()
    return _ptr(state), _ptr(slots), state.shape[0]


def short_conv_silu(u: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor | None, state: torch.Tensor | None,
                    state_slots: torch.Tensor | None, cu_seqlens_q: torch.Tensor | None, positions: torch.Tensor,
                    status: torch.Tensor | None = None) -> torch.Tensor:
    """``short_conv`` with SiLU behind it."""
    return short_conv(u, weight, bias, state, state_slots, cu_seqlens_q, positions, silu=True, status=status)


def short_conv(u: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor | None, state: torch.Tensor | None,
               state_slots: torch.Tensor | None, cu_seqlens_q: torch.Tensor | None, positions: torch.Tensor, silu: bool = False,
               copies: int = 0, status: torch.Tensor | None = None) -> torch.Tensor:
    """Causal depthwise convolution, optionally with SiLU.  ``u`` [T, C] (free row stride), ``weight`` [taps, C] (row j weighs the
    input j tokens back), ``state`` [slots, taps - 1, C].  [T, C + copies]: the last ``copies`` channels come a second time."""
    code = _dtype_of(u, "u")
    _same(u.dtype, weight=weight, bias=bias, state=state)
    _need(positions, torch.int64, "positions")
    tokens, channels = u.shape
    taps = weight.shape[0]
    assert u.stride(1) == 1 and weight.is_contiguous() and weight.shape[1] == channels
    assert state is None or state.shape[1:] == (taps - 1, channels)
    out = torch.empty(tokens, channels + copies, dtype=u.dtype, device=u.device)
    st, sl, n = _state_args(state, state_slots)
    num_seqs = tokens if cu_seqlens_q is None else cu_seqlens_q.numel() - 1
    rc = _cabi.load().mvb_short_conv(code, _ptr(u), u.stride(0), _ptr(weight), _ptr(bias), _ptr(out), out.stride(0), st, sl,
                                     n, _ptr(cu_seqlens_q), _ptr(positions), num_seqs, tokens, channels, taps, 1 if silu else 0,
                                     int(copies), _ptr(status), _stream())
    _cabi.check(rc, "mvb_short_conv")
    LaunchCounter.add(2 if cu_seqlens_q is not None and st is not None and taps > 1 else 1)
    return out


def selective_scan(u: torch.Tensor, dt: torch.Tensor, z: torch.Tensor, b: torch.Tensor, c: torch.Tensor,
                   dt_bias: torch.Tensor, a_log2e: torch.Tensor, d: torch.Tensor, out: torch.Tensor,
                   state: torch.Tensor | None, state_slots: torch.Tensor | None, cu_seqlens_q: torch.Tensor | None,
                   positions: torch.Tensor, status: torch.Tensor | None = None) -> torch.Tensor:
    """Selective scan with its gate: u, dt (raw), z, out [T, channels]; b, c [T, N] with one row stride; fp32 ``dt_bias``,
    ``d`` [channels] and ``a_log2e`` [channels, N padded to 4]; ``state`` fp32 [slots, channels, N padded]."""
    code = _dtype_of(u, "u")
    _same(u.dtype, dt=dt, z=z, b=b, c=c, out=out)
    _same(torch.float32, dt_bias=dt_bias, a_log2e=a_log2e, d=d, state=state)
    _need(positions, torch.int64, "positions")
    tokens, channels = u.shape
    assert b.stride(0) == c.stride(0) or tokens <= 1
    assert a_log2e.is_contiguous() and a_log2e.shape[0] == channels
    st, sl, n = _state_args(state, state_slots)
    num_seqs = tokens if cu_seqlens_q is None else cu_seqlens_q.numel() - 1
    rc = _cabi.load().mvb_selective_scan(
        code, _ptr(u), u.stride(0), _ptr(dt), dt.stride(0), _ptr(z), z.stride(0), _ptr(b), _ptr(c), b.stride(0),
        _ptr(dt_bias), _ptr(a_log2e), _ptr(d), _ptr(out), out.stride(0), st, sl, n, _ptr(cu_seqlens_q), _ptr(positions),
        num_seqs, tokens, channels, b.shape[1], a_log2e.shape[1], _ptr(status), _stream())
    _cabi.check(rc, "mvb_selective_scan")
    LaunchCounter.add(1)
    return out


def state_space(x: torch.Tensor, b: torch.Tensor, c: torch.Tensor, dt: torch.Tensor, dt_bias: torch.Tensor, a_log2e: torch.Tensor,
                d: torch.Tensor, out: torch.Tensor, state: torch.Tensor | None, state_slots: torch.Tensor | None,
                cu_seqlens_q: torch.Tensor | None, positions: torch.Tensor, longest: int = 0,
                status: torch.Tensor | None = None) -> torch.Tensor:
    """``S <- e^(a dt) S + dt b x^T``, ``out = S^T c + d x`` per head, dt = softplus(raw + bias): x and out [T, heads, vdim], b and c
    [T, groups, N], raw ``dt`` [T, heads]; fp32 ``dt_bias``, ``a_log2e`` (a times log2(e)) and ``d`` [heads]; ``state`` fp32
    [slots, heads, N, vdim padded to 4].  ``longest``: tokens of the step's longest sequence; few long ones are cut into segments."""
    code = _dtype_of(x, "x")
    _same(x.dtype, b=b, c=c, dt=dt, out=out)
    _same(torch.float32, dt_bias=dt_bias, a_log2e=a_log2e, d=d, state=state)
    _need(positions, torch.int64, "positions")
    for t, name in ((x, "x"), (b, "b"), (c, "c"), (out, "out")):
        _heads_contiguous(t, name)
    (tokens, heads, vdim), (groups, n) = x.shape, b.shape[1:]
    assert x.stride(0) == b.stride(0) == c.stride(0) or tokens <= 1
    assert b.shape == c.shape == (tokens, groups, n) and out.shape == x.shape and dt.shape == (tokens, heads) and dt.stride(1) == 1
    assert state is None or state.shape[1:] == (heads, n, -(-vdim // 4) * 4)
    st, sl, slots = _state_args(state, state_slots)
    num_seqs = tokens if cu_seqlens_q is None else cu_seqlens_q.numel() - 1
    lib, ragged = _cabi.load(), cu_seqlens_q is not None
    need = lib.mvb_state_space_scratch_bytes(code, tokens, num_seqs, longest, heads, n, vdim, int(ragged))
    scratch = torch.empty(need, dtype=torch.uint8, device=x.device) if need else None
    rc = lib.mvb_state_space(
        code, _ptr(x), _ptr(b), _ptr(c), x.stride(0), _ptr(dt), dt.stride(0), _ptr(dt_bias), _ptr(a_log2e), _ptr(d), _ptr(out),
        out.stride(0), st, sl, slots, _ptr(cu_seqlens_q), _ptr(positions), num_seqs, tokens, longest, heads, groups, n, vdim, _ptr(scratch), need,
        _ptr(status), _stream())
    _cabi.check(rc, "mvb_state_space")
    LaunchCounter.add(3 if need else 1)
    return out


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """``u / rms(u) * weight`` with ``u = y silu(z)``, the root mean square over each of ``groups`` equal parts of the row (fp32 weight)."""
    code = _dtype_of(y, "y")
    _same(y.dtype, z=z, out=out); _need(weight, torch.float32, "weight")
    rows, width = y.shape
    assert z.shape == out.shape == y.shape and y.stride(1) == z.stride(1) == out.stride(1) == 1 and weight.numel() == width
    rc = _cabi.load().mvb_gated_group_norm(code, _ptr(y), y.stride(0), _ptr(z), z.stride(0), _ptr(weight), _ptr(out), out.stride(0), rows,
                                           width, groups, float(eps), _stream())
    _cabi.check(rc, "mvb_gated_group_norm")
    LaunchCounter.add(1)
    return out


def gated_delta(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, a: torch.Tensor, b: torch.Tensor, gate: torch.Tensor,
                exp_a: torch.Tensor, dt_bias: torch.Tensor, norm_weight: torch.Tensor, out: torch.Tensor,
                state: torch.Tensor | None, state_slots: torch.Tensor | None, cu_seqlens_q: torch.Tensor | None,
                positions: torch.Tensor, q_scale: float, eps: float, out_scale: float = 1.0,
                status: torch.Tensor | None = None) -> torch.Tensor:
    """Gated delta rule with its gated output norm: q, k [T, kv_heads, dim], v and out [T, heads, vdim], raw decay ``a``
    [T, heads * dim], raw ``b`` [T, heads], raw ``gate`` [T, heads * vdim]; ``state`` fp32 [slots, heads, dim, vdim padded to 4]."""
    code = _dtype_of(q, "q")
    _same(q.dtype, k=k, v=v, a=a, b=b, gate=gate, out=out)
    _same(torch.float32, exp_a=exp_a, dt_bias=dt_bias, norm_weight=norm_weight, state=state)
    _need(positions, torch.int64, "positions")
    for t, name in ((q, "q"), (k, "k"), (v, "v"), (out, "out")):
        _heads_contiguous(t, name)
    tokens, kv_heads, dim = q.shape
    heads, vdim = v.shape[1:]
    assert q.stride(0) == k.stride(0) == v.stride(0) or tokens <= 1
    st, sl, n = _state_args(state, state_slots)
    ragged = cu_seqlens_q is not None
    num_seqs = cu_seqlens_q.numel() - 1 if ragged else tokens
    lib = _cabi.load()
    scratch = torch.empty(lib.mvb_gated_delta_scratch_bytes(code, tokens, num_seqs, heads, kv_heads, dim, vdim, int(ragged)), dtype=torch.uint8,
                          device=q.device)
    rc = lib.mvb_gated_delta(
        code, _ptr(q), _ptr(k), _ptr(v), q.stride(0), _ptr(a), a.stride(0), _ptr(b), b.stride(0), _ptr(gate), gate.stride(0),
        _ptr(exp_a), _ptr(dt_bias), _ptr(norm_weight), _ptr(out), out.stride(0), st, sl, n, _ptr(cu_seqlens_q),
        _ptr(positions), num_seqs, tokens, heads, kv_heads, dim, vdim, float(q_scale), float(eps), float(out_scale),
        _ptr(scratch), scratch.numel(), _ptr(status), _stream())
    _cabi.check(rc, "mvb_gated_delta")
    LaunchCounter.add(3 if ragged else (2 if vdim > 128 else 1))
    return out


def _linear_scratch(code: int, tokens: int, num_seqs: int, heads: int, dim: int, vdim: int, exp_gates: bool, ragged: bool, device):
    n = _cabi.load().mvb_linear_attn_scratch_bytes(code, tokens, num_seqs, heads, dim, vdim, int(exp_gates), int(ragged))
    return torch.empty(n, dtype=torch.uint8, device=device)


def _linear_shapes(q, k, v, out):
    for t, name in ((q, "q"), (k, "k"), (v, "v"), (out, "out")):
        _heads_contiguous(t, name)
    assert q.shape == k.shape and out.shape == v.shape and v.shape[:2] == q.shape[:2]
    assert q.stride(0) == k.stride(0) == v.stride(0) or q.shape[0] <= 1
    return (*q.shape, v.shape[2])


def gated_linear(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, decay_bias: torch.Tensor, tau: float,
                 gate: torch.Tensor, norm_weight: torch.Tensor, out: torch.Tensor, state: torch.Tensor | None,
                 state_slots: torch.Tensor | None, cu_seqlens_q: torch.Tensor | None, positions: torch.Tensor, q_scale: float,
                 eps: float, status: torch.Tensor | None = None) -> torch.Tensor:
    """Linear attention with a decay per key channel, ``sigmoid(decay + bias)^(1/tau)``, and its SiLU-gated output norm: q, k
    [T, heads, dim], v and out [T, heads, vdim], raw ``decay`` [T, heads * dim], raw ``gate`` [T, heads * vdim]; ``state`` fp32
    [slots, heads, dim, vdim padded to 4]."""
    code = _dtype_of(q, "q")
    _same(q.dtype, k=k, v=v, decay=decay, gate=gate, out=out)
    _same(torch.float32, decay_bias=decay_bias, norm_weight=norm_weight, state=state)
    _need(positions, torch.int64, "positions")
    tokens, heads, dim, vdim = _linear_shapes(q, k, v, out)
    st, sl, n = _state_args(state, state_slots)
    ragged = cu_seqlens_q is not None
    num_seqs = cu_seqlens_q.numel() - 1 if ragged else tokens
    scratch = _linear_scratch(code, tokens, num_seqs, heads, dim, vdim, False, ragged, q.device)
    rc = _cabi.load().mvb_gated_linear(
        code, _ptr(q), _ptr(k), _ptr(v), q.stride(0), _ptr(decay), decay.stride(0), _ptr(decay_bias), 1.0 / tau, _ptr(gate),
        gate.stride(0), _ptr(norm_weight), _ptr(out), out.stride(0), st, sl, n, _ptr(cu_seqlens_q), _ptr(positions), num_seqs,
        tokens, heads, dim, vdim, float(q_scale), float(eps), _ptr(scratch), scratch.numel(), _ptr(status), _stream())
    _cabi.check(rc, "mvb_gated_linear")
    LaunchCounter.add(3 if ragged else 1)
    return out


def mlstm(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, forget: torch.Tensor, forget_bias: torch.Tensor, inp: torch.Tensor,
          inp_bias: torch.Tensor, cap: float, gate: torch.Tensor, norm_weight: torch.Tensor, out: torch.Tensor,
          states: tuple | None, state_slots: torch.Tensor | None, cu_seqlens_q: torch.Tensor | None, positions: torch.Tensor,
          q_scale: float, eps: float, status: torch.Tensor | None = None) -> torch.Tensor:
    """Matrix memory with capped exponential gates, a normaliser and a running maximum, and its sigmoid-gated output norm: raw
    ``forget`` and ``inp`` [T, heads], ``norm_weight`` [heads * vdim]; ``states`` = fp32 (memory [slots, heads, dim, vdim padded to 4],
    normaliser [slots, heads, dim], maximum [slots, heads])."""
    code = _dtype_of(q, "q")
    _same(q.dtype, k=k, v=v, forget=forget, inp=inp, gate=gate, out=out)
    memory, normaliser, maximum = states or (None, None, None)
    _same(torch.float32, forget_bias=forget_bias, inp_bias=inp_bias, norm_weight=norm_weight, memory=memory, normaliser=normaliser,
          maximum=maximum)
    _need(positions, torch.int64, "positions")
    tokens, heads, dim, vdim = _linear_shapes(q, k, v, out)
    st, sl, n = _state_args(memory, state_slots)
    ragged = cu_seqlens_q is not None
    num_seqs = cu_seqlens_q.numel() - 1 if ragged else tokens
    scratch = _linear_scratch(code, tokens, num_seqs, heads, dim, vdim, True, ragged, q.device)
    rc = _cabi.load().mvb_mlstm(
        code, _ptr(q), _ptr(k), _ptr(v), q.stride(0), _ptr(forget), forget.stride(0), _ptr(forget_bias), _ptr(inp), inp.stride(0),
        _ptr(inp_bias), float(cap), _ptr(gate), gate.stride(0), _ptr(norm_weight), _ptr(out), out.stride(0), st,
        _ptr(normaliser) if st else None, _ptr(maximum) if st else None, sl, n, _ptr(cu_seqlens_q), _ptr(positions), num_seqs, tokens,
        heads, dim, vdim, float(q_scale), float(eps), _ptr(scratch), scratch.numel(), _ptr(status), _stream())
    _cabi.check(rc, "mvb_mlstm")
    LaunchCounter.add(3 if ragged else 1)
    return out


def hyper_embed_norm(ids: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, pos_table: torch.Tensor, streams: int,
                     in_weights: torch.Tensor, weight: torch.Tensor, eps: float, groups: int,
                     status: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """(fp32 streams [T, streams, width], all ``table[ids] + pos_table[positions]``; the normalised input of the first sublayer)."""
    code = _dtype_of(table, "table")
    _need(ids, torch.int64, "ids"); _need(positions, torch.int64, "positions")
    _same(table.dtype, weight=weight, pos_table=pos_table); _need(in_weights, torch.float32, "in_weights")
    assert table.is_contiguous() and pos_table.is_contiguous() and pos_table.shape[1] == table.shape[1]
    rows, width = ids.numel(), table.shape[1]
    x = torch.empty(rows, streams, width, dtype=torch.float32, device=table.device)
    h = torch.empty(rows, width, dtype=table.dtype, device=table.device)
    rc = _cabi.load().mvb_hyper_embed_norm(
        code, _ptr(ids), _ptr(positions), _ptr(table), table.shape[0], _ptr(pos_table), pos_table.shape[0], _ptr(x), _ptr(in_weights),
        _ptr(weight), _ptr(h), rows, width, streams, groups, float(eps), _ptr(status), _stream())
    _cabi.check(rc, "mvb_hyper_embed_norm")
    LaunchCounter.add(1)
    return x, h


def hyper_norm(x: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, out_weights: torch.Tensor, in_weights: torch.Tensor | None,
               weight: torch.Tensor, eps: float, groups: int, row_ends: torch.Tensor | None = None) -> torch.Tensor:
    """Streams ``x`` [T, streams, width] in place: ``x_t <- sum_s mix[s, t] x_s + out[t] y``; returns the grouped norm of
    ``sum_s in[s] x_s`` (``in_weights`` None: of the plain sum) in y's dtype.  With ``row_ends`` only rows ``row_ends[1:] - 1`` are
    produced and ``x`` is left as it is."""
    code = _dtype_of(y, "y")
    _need(x, torch.float32, "x"); _same(y.dtype, weight=weight); _same(torch.float32, mix=mix, out_weights=out_weights, in_weights=in_weights)
    rows, streams, width = x.shape
    assert x.is_contiguous() and y.shape == (rows, width) and y.stride(1) == 1 and mix.shape == (streams, streams) and mix.is_contiguous()
    if row_ends is not None:
        _need(row_ends, torch.int32, "row_ends")
        rows = row_ends.numel() - 1
    h = torch.empty(rows, width, dtype=y.dtype, device=x.device)
    if rows == 0:
        return h
    rc = _cabi.load().mvb_hyper_norm(code, _ptr(x), _ptr(y), y.stride(0), _ptr(mix), _ptr(out_weights), _ptr(in_weights), _ptr(weight),
                                     _ptr(h), _ptr(row_ends), rows, width, streams, groups, float(eps), _stream())
    _cabi.check(rc, "mvb_hyper_norm")
    LaunchCounter.add(1)
    return h


def poly_norm(z: torch.Tensor, cols: int, act: torch.Tensor, eps: float) -> torch.Tensor:
    """``a N(z) + b N(z^2) + c N(z^3) + e`` over the first ``cols`` columns (N: over the row's root mean square, act = fp32 {a, b, c, e});
    the columns behind them become 0."""
    code = _dtype_of(z, "z")
    _need(act, torch.float32, "act")
    assert z.dim() == 2 and z.stride(1) == 1 and z.shape[1] >= cols and act.numel() == 4
    out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    rc = _cabi.load().mvb_poly_norm(code, _ptr(z), z.stride(0), _ptr(out), out.stride(0), z.shape[0], cols, z.shape[1], _ptr(act),
                                    float(eps), _stream())
    _cabi.check(rc, "mvb_poly_norm")
    LaunchCounter.add(1)
    return out


LATENT_WIDTHS = (64, 128, 192, 256, 384, 512)      # cached row sizes of latent_decode


def latent_norm(q: torch.Tensor, q_weight: torch.Tensor, q_pad: int, c: torch.Tensor | None, c_weight: torch.Tensor | None, c_pad: int,
                eps: float, cache: torch.Tensor | None = None, slot_mapping: torch.Tensor | None = None,
                status: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor | None]:
    """RMS norms of the query latent ``q`` and, unless None, of the key/value latent ``c``, each zero-padded to a width; ``c`` also goes
    to its slots of ``cache`` [blocks, block_size, c_pad]."""
    code = _dtype_of(q, "q")
    _same(q.dtype, q_weight=q_weight, c=c, c_weight=c_weight, cache=cache)
    tokens = q.shape[0]
    assert q.stride(1) == 1 and q_weight.numel() == q.shape[1]
    q_out = torch.empty(tokens, q_pad, dtype=q.dtype, device=q.device)
    c_out, slots = None, 0
    if c is not None:
        assert c.stride(1) == 1 and c.shape[0] == tokens and c_weight.numel() == c.shape[1]
        c_out = torch.empty(tokens, c_pad, dtype=q.dtype, device=q.device)
        if cache is not None:
            _need(slot_mapping, torch.int32, "slot_mapping")
            assert cache.is_contiguous() and cache.shape[-1] == c_pad and slot_mapping.numel() == tokens
            slots = cache.shape[0] * cache.shape[1]
    rc = _cabi.load().mvb_latent_norm(
        code, _ptr(q), q.stride(0), _ptr(q_weight), _ptr(q_out), q.shape[1], q_pad, _ptr(c), c.stride(0) if c is not None else 0,
        _ptr(c_weight), _ptr(c_out), c.shape[1] if c is not None else 0, c_pad, _ptr(cache) if slots else None,
        _ptr(slot_mapping) if slots else None, slots, tokens, float(eps), _ptr(status), _stream())
    _cabi.check(rc, "mvb_latent_norm")
    LaunchCounter.add(1)
    return q_out, c_out


def gather_latents(cache: torch.Tensor, block_table: torch.Tensor, cu_seqlens_k: torch.Tensor, rows: int,
                   status: torch.Tensor | None = None) -> torch.Tensor:
    """The contexts of a ragged step ([blocks, block_size, width] pool, lengths in ``cu_seqlens_k``, ``rows`` in all) as dense rows."""
    _need(block_table, torch.int32, "block_table"); _need(cu_seqlens_k, torch.int32, "cu_seqlens_k")
    assert cache.is_cuda and cache.is_contiguous() and block_table.stride(1) == 1
    out = torch.empty(rows, cache.shape[-1], dtype=cache.dtype, device=cache.device)
    rc = _cabi.load().mvb_gather_latents(
        _ptr(cache), cache.shape[0] * cache.shape[1], cache.shape[-1] * cache.element_size(), _ptr(block_table), block_table.stride(0),
        block_table.shape[1], cache.shape[1], _ptr(cu_seqlens_k), cu_seqlens_k.numel() - 1, rows, _ptr(out), _ptr(status), _stream())
    _cabi.check(rc, "mvb_gather_latents")
    LaunchCounter.add(1)
    return out


def gate_mul(o: torch.Tensor, gate: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``out = o * sigmoid(gate)``; 2-D, free row strides."""
    code = _dtype_of(o, "o")
    _same(o.dtype, gate=gate, out=out)
    assert o.shape == gate.shape == out.shape and o.stride(1) == gate.stride(1) == out.stride(1) == 1
    rc = _cabi.load().mvb_gate_mul(code, _ptr(o), o.stride(0), _ptr(gate), gate.stride(0), _ptr(out), out.stride(0), o.shape[0], o.shape[1],
                                   _stream())
    _cabi.check(rc, "mvb_gate_mul")
    LaunchCounter.add(1)
    return out


def latent_decode_plan(cache_seqlens: torch.Tensor, block_table: torch.Tensor, block_size: int, heads: int, width: int,
                       workspace: torch.Tensor) -> None:
    _need(cache_seqlens, torch.int32, "cache_seqlens"); _need(block_table, torch.int32, "block_table")
    assert block_table.stride(1) == 1 and block_table.shape[0] >= cache_seqlens.numel()
    rc = _cabi.load().mvb_latent_decode_plan(_ptr(cache_seqlens), _ptr(block_table), block_table.stride(0), block_size,
                                             cache_seqlens.numel(), heads, width, _ptr(workspace), workspace.numel(), _stream())
    _cabi.check(rc, "mvb_latent_decode_plan")
    LaunchCounter.add(1)


def latent_decode(q: torch.Tensor, cache: torch.Tensor, cache_seqlens: torch.Tensor, block_table: torch.Tensor, scale: float,
                  workspace: torch.Tensor, status: torch.Tensor | None = None) -> torch.Tensor:
    """Absorbed decode attention: q [heads, B, width] (queries already in the latent's space) over ``cache`` [blocks, block_size, width];
    returns [heads, B, width].  The plan for ``cache_seqlens`` must already be in ``workspace``."""
    _need(q, torch.bfloat16, "q"); _need(cache, torch.bfloat16, "cache")
    _need(cache_seqlens, torch.int32, "cache_seqlens"); _need(block_table, torch.int32, "block_table")
    heads, b, width = q.shape
    nblk, bs, w2 = cache.shape
    assert w2 == width and cache.is_contiguous() and q.stride(2) == 1 and block_table.stride(1) == 1 and cache_seqlens.numel() >= b
    out = torch.empty(heads, b, width, dtype=q.dtype, device=q.device)
    rc = _cabi.load().mvb_latent_decode(
        _ptr(q), q.stride(1), q.stride(0), _ptr(cache), nblk, bs, _ptr(cache_seqlens), _ptr(block_table), block_table.stride(0),
        block_table.shape[1], b, heads, width, float(scale), _ptr(out), out.stride(1), out.stride(0), _ptr(workspace), workspace.numel(),
        _ptr(status), _stream())
    _cabi.check(rc, "mvb_latent_decode")
    LaunchCounter.add(1)
    return out


# ---- mixture of experts -----------------------------------------------------------------------------------------
@dataclass(frozen=True)
class ExpertRows:
    """A step's tokens sorted by expert, as the grouped products need them; every number stays on the device."""
    slots: torch.Tensor           # int32 [T, top]: the sorted row of a token's j-th expert
    weights: torch.Tensor         # fp32 [T * top], in sorted order
    tiles: torch.Tensor           # int32 [max tiles, 4]
    num_tiles: torch.Tensor       # int32 [1]
    block_rows: int
    experts: int
    identity: torch.Tensor | None = None      # fp32 [T]: what a token's identity experts weigh together


@dataclass(frozen=True)
class Routing:
    """How router logits become choices and weights: scores are sigmoids or the ``softmax`` over all outputs; the choice is by score plus
    ``correction`` (fp32 [outputs]; None: by score); the weight is the score times ``scale``.  The last ``identity`` outputs are experts
    that return a token's own row."""
    softmax: bool = False
    correction: torch.Tensor | None = None
    scale: float = 1.0
    identity: int = 0


def moe_block_rows(rows: int, experts: int, dtype: torch.dtype) -> int:
    """Rows of a tile of the grouped products, by how many an expert gets on average."""
    if dtype == torch.float32:
        return 64
    return 128 if rows >= 40 * experts else 64 if rows >= 16 * experts else 32


def moe_sort(h: torch.Tensor, logits: torch.Tensor, top: int, counters: torch.Tensor,
             routing: Routing = Routing()) -> tuple[torch.Tensor, ExpertRows]:
    """Picks each token's ``top`` experts by the fp32 ``logits`` [T, E + identity] and gathers the rows of ``h`` expert by expert.
    ``counters``: int32 [E + 1], zero, left zero."""
    code = _dtype_of(h, "h")
    _need(logits, torch.float32, "logits"); _need(counters, torch.int32, "counters"); _same(torch.float32, correction=routing.correction)
    (tokens, width), experts, dev, lib = h.shape, logits.shape[1] - routing.identity, h.device, _cabi.load()
    assert routing.correction is None or routing.correction.numel() == logits.shape[1]
    assert h.stride(1) == 1 and logits.shape[0] == tokens and logits.stride(1) == 1 and counters.numel() > experts
    rows = tokens * top
    block_rows = moe_block_rows(rows, experts, h.dtype)
    max_tiles = rows // block_rows + min(rows, experts)
    ints = torch.empty(3, rows, dtype=torch.int32, device=dev)           # expert, rank, slot
    picked = torch.empty(2, rows, dtype=torch.float32, device=dev)       # weights by token, by sorted row
    offsets = torch.empty(2, experts + 1, dtype=torch.int32, device=dev)
    tiles = torch.empty(max_tiles, 4, dtype=torch.int32, device=dev)
    identity = torch.empty(tokens, dtype=torch.float32, device=dev) if routing.identity else None
    rc = lib.mvb_moe_route_ext(_ptr(logits), logits.stride(0), tokens, experts, routing.identity, top, int(routing.softmax),
                               _ptr(routing.correction), float(routing.scale), block_rows, max_tiles, _ptr(counters), _ptr(ints[0]),
                               _ptr(picked[0]), _ptr(ints[1]), _ptr(offsets[0]), _ptr(offsets[1]), _ptr(tiles), _ptr(identity), _stream())
    _cabi.check(rc, "mvb_moe_route_ext")
    x = torch.empty(rows, -(-width // 8) * 8, dtype=h.dtype, device=dev)[:, :width]
    rc = lib.mvb_moe_gather(code, _ptr(h), h.stride(0), _ptr(ints[0]), _ptr(picked[0]), _ptr(ints[1]), _ptr(offsets[0]), _ptr(x),
                            x.stride(0), _ptr(ints[2]), _ptr(picked[1]), tokens, top, width, _stream())
    _cabi.check(rc, "mvb_moe_gather")
    LaunchCounter.add(2)
    return x, ExpertRows(ints[2].view(tokens, top), picked[1], tiles, offsets[1, experts:], block_rows, experts, identity)


def moe_gemm(x: torch.Tensor, weight: torch.Tensor, rows: ExpertRows, k: int,
             gated: tuple[float, float, float] | None = None, weigh_output: bool = False, status: torch.Tensor | None = None) -> torch.Tensor:
    """Each expert's product over its sorted rows: ``weight`` [E, m, K] or, ``gated`` = (limit, alpha, offset), [E, 2, m, K] with the
    gated unit behind it and the token's weight on the expert's input, or on the unit's output (``weigh_output``).  K >= k is what a weight row is padded to."""
    code = _dtype_of(x, "x")
    _same(x.dtype, weight=weight)
    m = weight.shape[-2]
    assert weight.is_contiguous() and weight.shape[0] == rows.experts and weight.dim() == (3 if gated is None else 4)
    assert x.stride(1) == 1 and x.shape[1] >= k and weight.shape[-1] >= k
    out = torch.empty(x.shape[0], -(-m // 8) * 8, dtype=x.dtype, device=x.device)[:, :m]
    limit, alpha, offset = gated or (0.0, 0.0, 0.0)
    rc = _cabi.load().mvb_moe_gemm(
        code, _ptr(x), x.stride(0), x.shape[0], _ptr(weight), weight.shape[-1], rows.experts, m, k, 0 if gated is None else 2 if weigh_output else 1, float(limit),
        float(alpha), float(offset), None if gated is None else _ptr(rows.weights), _ptr(rows.num_tiles), _ptr(rows.tiles),
        rows.tiles.shape[0], rows.block_rows, _ptr(out), out.stride(0), _ptr(status), _stream())
    _cabi.check(rc, "mvb_moe_gemm")
    LaunchCounter.add(1)
    return out
