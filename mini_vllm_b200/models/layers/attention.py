"""Attention layer: drop-in for ``FlashAttention`` of ``minivllm/models/layers/attention.py:46-92``.

Same constructor, same ``forward(ctx, q, k, v)`` contract (q/k already rotated; k/v are written
to the paged cache at ``ctx.slot_mapping`` first; prefill attends causally over ``cu_seqlens``,
decode attends one token per sequence over ``cache_seqlens`` through ``block_table``), same
``k_cache``/``v_cache`` attributes that the executor rebinds to views of its KV pool.
``forward_fused`` additionally takes ``positions`` and the cos/sin table and applies the rotary
embedding inside the KV-write kernel, saving one round trip of q and k through HBM.

Unlike the reference, ``scaling`` and ``sliding_window`` are honoured (the reference stores both
and passes neither to its attention calls, ``attention.py:84-91``).

Beyond the reference: ``softcap`` (scores pass ``c tanh(s / c)``), ``out_scale`` (a constant factor of the output), kept first
tokens, sinks, a bias by distance and head gates (``ops.AttnExtras``), a norm behind the rotation, a layer that reads an earlier layer's
keys and values (``source``) and, for activations or head layouts the tensor-core kernels do not take (fp32, head sizes other than 128 / 256, more than
eight query heads per KV head in a decode step), the general attention kernel over the same cache.
"""
from __future__ import annotations

import torch
from torch import nn

from ... import ops
from ...executor.context import Context

_workspaces: dict = {}
_superseded: list = []      # outgrown buffers stay allocated: captured CUDA graphs keep writing through their pointers


def decode_workspace_for(device, max_seqs: int, num_heads: int, num_kv_heads: int, head_dim: int, window_left) -> torch.Tensor:
    """One scratch buffer per (device, head shape, window or kind of attention); a larger one takes its place when a larger batch
    arrives.  The smaller buffer is never freed: a graph captured while it was current has its address
    baked in, and a replay after the memory went back to the allocator would scribble over someone else."""
    key = (device, num_heads, num_kv_heads, head_dim, window_left)
    ws = _workspaces.get(key)
    need = ops._cabi.load().mvb_decode_workspace_bytes(max_seqs, num_heads, head_dim)
    if ws is None or ws.numel() < need:
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("decode workspace must be allocated before CUDA graph capture "
                               "(run one eager decode step of the largest batch first)")
        if ws is not None:
            _superseded.append(ws)
        ws = ops.decode_workspace(max(max_seqs, 512), num_heads, head_dim, device)
        _workspaces[key] = ws
    return ws


def prefill_items_for(ctx: Context, layer):
    """The step's prefill work list, if the packing step built one for the layer's query-block size."""
    if ctx.prefill_items is None:
        return None
    if layer._item_rows is None:
        layer._item_rows = ops.prefill_item_rows(layer.num_heads, layer.num_kv_heads, layer.head_dim)
    return ctx.prefill_items if ctx.prefill_item_rows == layer._item_rows else None


class FlashAttention(nn.Module):
    def __init__(self, num_heads: int, head_dim: int, scaling: float, num_kv_heads: int,
                 sliding_window=(-1, -1), softcap: float = 0.0, out_scale: float = 1.0, keep_first: int = 0,
                 source: "FlashAttention | None" = None):
        super().__init__()
        self.num_heads = num_heads
        self.head_dim = head_dim
        self.scaling = scaling
        self.num_kv_heads = num_kv_heads
        self.sliding_window = tuple(sliding_window)
        self.softcap, self.out_scale = float(softcap), float(out_scale)
        self.keep_first = int(keep_first) if self.window_left >= 0 else 0
        self.sinks = self.slopes = None   # fp32 [num_heads] each, set by whoever owns them
        self.__dict__["source"] = source  # (not a submodule of this one)
        self.lends = False                # some later layer reads this one's keys and values
        if source is None:
            # placeholders the executor replaces with views of its KV pool (found by hasattr)
            self.k_cache = self.v_cache = torch.tensor([])
        else:
            source.lends = True
        self._item_rows = None            # query-block size of the prefill kernel's work items for this head layout

    @property
    def window_left(self) -> int:
        left = self.sliding_window[0]
        return int(left) if left is not None and left >= 0 else -1

    def _has_cache(self) -> bool:
        return self.k_cache.numel() > 0 and self.v_cache.numel() > 0

    def _caches(self) -> tuple[torch.Tensor, torch.Tensor]:
        owner = self if self.source is None else self.source
        return owner.k_cache, owner.v_cache

    def _extras(self, head_gate: torch.Tensor | None) -> ops.AttnExtras | None:
        if self.sinks is None and self.slopes is None and head_gate is None and self.keep_first == 0:
            return None
        return ops.AttnExtras(self.sinks, self.slopes, head_gate, self.keep_first)

    def forward(self, ctx: Context, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
        if self._has_cache():
            ops.rope_kv_write(None, k, v, None, None, ctx.slot_mapping, self.k_cache, self.v_cache,
                              k_in_place=False, status=ctx.status)
        return self._attend(ctx, q, k, v)

    def forward_fused(self, ctx: Context, q: torch.Tensor, k: torch.Tensor | None, v: torch.Tensor | None, positions: torch.Tensor,
                      cos_sin_cache: torch.Tensor | None, out: torch.Tensor | None = None, head_gate: torch.Tensor | None = None,
                      norm: tuple[int, float] | None = None, row_norm: ops.RowNorm | None = None) -> torch.Tensor:
        """q, k NOT yet rotated: RoPE (in place on q and k) + cache write in one kernel, then attention.  ``cos_sin_cache`` None: no
        rotation; ``norm`` (size, eps): q and k are divided by their root mean square behind it; ``row_norm``: norms in front of it, in
        the same kernel.  With a ``source`` k and v are None."""
        if self.source is not None:
            k, v = ctx.shared.get(self.source, (None, None))          # this step's own, for prompts without earlier tokens
            if cos_sin_cache is not None or norm is not None:
                ops.rope_norm_kv_write(q, None, None, positions, cos_sin_cache, None, None, None, norm_dim=norm[0] if norm else 0,
                                       eps=norm[1] if norm else 0.0, status=ctx.status)
        else:
            cached = (ctx.slot_mapping, self.k_cache, self.v_cache) if self._has_cache() else (None, None, None)
            in_place = ctx.prefill and ctx.block_table is None
            if row_norm is not None:
                ops.row_norm_rope_kv_write(q, k, v, row_norm, positions, cos_sin_cache, *cached, kv_in_place=in_place, status=ctx.status)
            elif norm is not None or (cos_sin_cache is None and q.dtype != torch.bfloat16):
                ops.rope_norm_kv_write(q, k, v, positions, cos_sin_cache, *cached, k_in_place=in_place, norm_dim=norm[0] if norm else 0,
                                       eps=norm[1] if norm else 0.0, status=ctx.status)
            else:
                write = ops.rope_kv_write if q.dtype == torch.bfloat16 else ops.rope_kv_write_f32
                write(q, k, v, positions, cos_sin_cache, *cached, k_in_place=in_place, status=ctx.status)
            if self.lends:
                ctx.shared[self] = (k, v)
        extras = self._extras(head_gate)
        if not self.tensor_cores(q.dtype, decode=not ctx.prefill or ctx.num_decode > 0):
            return self._attend_any(ctx, q, k, v, positions, out, extras)
        return self._attend(ctx, q, k, v, out, extras)

    def tensor_cores(self, dtype: torch.dtype, decode: bool) -> bool:
        """Whether the tensor-core kernels take this layer's activations and head layout."""
        return (dtype == torch.bfloat16 and self.head_dim in (128, 256) and
                (not decode or self.num_heads <= 8 * self.num_kv_heads))

    def _attend_any(self, ctx: Context, q, k, v, positions, out, extras) -> torch.Tensor:
        if ctx.block_table is not None:
            k, v = self._caches()
        return ops.any_attn(q, k, v, positions, self.scaling,
                            self.window_left, cu_seqlens_q=ctx.cu_seqlens_q if ctx.prefill else None,
                            cu_seqlens_k=ctx.cu_seqlens_k, block_table=ctx.block_table,
                            cache_seqlens=None if ctx.prefill else ctx.cache_seqlens, softcap=self.softcap,
                            out_scale=self.out_scale, out=out, status=ctx.status, extras=extras)

    def forward_fused_norm(self, ctx: Context, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor,
                           positions: torch.Tensor, cos_sin_cache: torch.Tensor, q_weight: torch.Tensor,
                           k_weight: torch.Tensor, eps: float, unit_offset: bool) -> torch.Tensor:
        """q, k straight from the projection (views of the packed qkv output): per-head RMSNorm, RoPE
        and the cache write in one kernel (q and k updated in place), then attention."""
        has_cache = self._has_cache()
        ops.qk_norm_rope_kv_write(q, k, v, q_weight, k_weight, eps, unit_offset, positions, cos_sin_cache,
                                  ctx.slot_mapping if has_cache else None, self.k_cache if has_cache else None,
                                  self.v_cache if has_cache else None,
                                  k_in_place=ctx.prefill and ctx.block_table is None, status=ctx.status)
        return self._attend(ctx, q, k, v)

    def _decode(self, ctx: Context, q: torch.Tensor, table: torch.Tensor, out: torch.Tensor | None = None,
                extras: ops.AttnExtras | None = None) -> torch.Tensor:
        (k_cache, v_cache), wl = self._caches(), self.window_left
        kind = (wl, self.keep_first) if self.keep_first else wl
        key = (kind, self.num_heads, self.num_kv_heads, self.head_dim)
        ws = ctx.decode_plans.get(key)
        if ws is None:
            ws = decode_workspace_for(q.device, ctx.cache_seqlens.numel(), self.num_heads, self.num_kv_heads, self.head_dim, kind)
            ops.decode_plan(ctx.cache_seqlens, wl, self.num_heads, self.num_kv_heads, self.head_dim, ws,
                            block_table=table, block_size=k_cache.shape[1], keep_first=self.keep_first)
            ctx.decode_plans[key] = ws
        return ops.decode_attn(q, k_cache, v_cache, ctx.cache_seqlens, table, self.scaling, wl, ws, out=out,
                               status=ctx.status, softcap=self.softcap, out_scale=self.out_scale, extras=extras)

    def _prefill(self, ctx: Context, q, k, v, cu_q, cu_k, table, out=None, extras=None) -> torch.Tensor:
        return ops.prefill_attn(q, k, v, cu_q, cu_k, ctx.max_seqlen_q, self.scaling, self.window_left, block_table=table,
                                out=out, status=ctx.status, items=prefill_items_for(ctx, self), softcap=self.softcap,
                                out_scale=self.out_scale, extras=extras)

    def _attend_mixed(self, ctx: Context, q: torch.Tensor, out: torch.Tensor | None = None,
                      extras: ops.AttnExtras | None = None) -> torch.Tensor:
        """A step holding both kinds of sequence (an extension; the reference's Context is one or the
        other): the prompts go through the prefill kernel, the single-token sequences at the end through
        the decode kernel, both over the paged pool the write kernel has just filled."""
        nd = ctx.num_decode
        bp, tp = ctx.cu_seqlens_q.numel() - 1 - nd, q.shape[0] - nd
        if out is None:
            out = torch.empty(q.shape, dtype=q.dtype, device=q.device)
        part = (lambda a, b: None) if extras is None else extras.rows
        self._prefill(ctx, q[:tp], *self._caches(), ctx.cu_seqlens_q[:bp + 1], ctx.cu_seqlens_k[:bp + 1],
                      ctx.block_table[:bp], out[:tp], part(0, tp))
        self._decode(ctx, q[tp:], ctx.block_table[bp:], out[tp:], part(tp, q.shape[0]))
        return out

    def _attend(self, ctx: Context, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor,
                out: torch.Tensor | None = None, extras: ops.AttnExtras | None = None) -> torch.Tensor:
        if ctx.prefill and ctx.num_decode:
            return self._attend_mixed(ctx, q, out, extras)
        if ctx.prefill:
            if ctx.block_table is not None:        # prefix cache in play: keys come from the pool
                k, v = self._caches()
            return self._prefill(ctx, q, k, v, ctx.cu_seqlens_q, ctx.cu_seqlens_k, ctx.block_table, out, extras)
        # decode: q [B,Hq,D] -> [B,1,Hq,D] like flash_attn_with_kvcache on q.unsqueeze(1)
        return self._decode(ctx, q, ctx.block_table, out, extras).unsqueeze(1)
