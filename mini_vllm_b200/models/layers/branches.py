"""Mixer branches for decoders whose layers are assembled from parts.

A branch is one token mixer (attention, latent attention, selective scan, state space, gated delta rule, gated linear attention,
matrix-memory LSTM) without its outer projections: it declares how
many rows it needs in the layer's packed input projection and how many columns it brings to the packed output
projection, and works between the two.  ``PackedMixer`` puts any number of branches side by side on the same input: ONE
input GEMM over the concatenated rows, the branches, ONE output GEMM over the concatenated columns, which also adds the
branches up.  A branch's constant factor is applied where it writes its columns (in fp32, before rounding).

Layout rules: every block a branch takes from the packed projection starts at a multiple of 8 rows, so that its view is
16-byte aligned; padding rows have zero weights.  Recurrent branches name their per-sequence state in ``state_specs``;
the executor owns the buffers (one row per state slot) and binds them to the attributes of the same names.
"""
from __future__ import annotations

import math
from typing import Callable

import torch
import torch.nn.functional as F
from torch import nn

from ... import ops
from ...executor.context import Context
from .attention import FlashAttention, decode_workspace_for, prefill_items_for
from .rotary import RotaryEmbedding

LOG2E = 1.0 / math.log(2.0)
Weights = Callable[[str], torch.Tensor]        # tensor of this branch by its name


def pad8(n: int) -> int:
    return -(-n // 8) * 8


def pad_rows(w: torch.Tensor, rows: int) -> torch.Tensor:
    return w if w.shape[0] == rows else F.pad(w, (0, 0, 0, rows - w.shape[0]))


def pad_cols(w: torch.Tensor, cols: int) -> torch.Tensor:
    return w if w.shape[1] == cols else F.pad(w, (0, cols - w.shape[1]))


def weight(*shape: int) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape), requires_grad=False)


def weight_f32(*shape: int) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape, dtype=torch.float32), requires_grad=False)


def ragged(ctx: Context) -> torch.Tensor | None:
    """Row boundaries of the step's sequences; None when every sequence brings one token."""
    return ctx.cu_seqlens_q if ctx.prefill else None


class Branch(nn.Module):
    in_rows: int        # rows of the packed input projection, a multiple of 8
    out_cols: int       # columns of the packed output projection, a multiple of 8
    out_used: int       # of these, the ones the branch writes (the rest stay zero)
    in_bias = out_bias = False          # whether the branch's projections have biases

    def state_specs(self, dtype: torch.dtype) -> dict[str, tuple[tuple[int, ...], torch.dtype]]:
        return {}

    def load(self, w: Weights) -> tuple[torch.Tensor, torch.Tensor]:
        """Load the branch's own parameters; returns its input rows [in_rows, width] and output columns [width, out_cols]."""
        raise NotImplementedError

    def load_biases(self, w: Weights) -> tuple[torch.Tensor | None, torch.Tensor | None]:
        """Bias of the input rows [in_rows] and of the output [width]; None where the branch has none."""
        return None, None

    def forward(self, ctx: Context, proj: torch.Tensor, out: torch.Tensor, positions: torch.Tensor) -> None:
        raise NotImplementedError


def alibi_slopes(heads: int) -> torch.Tensor:
    """2^(-8 (h + 1) / heads): what a distance bias takes off a score per token, head by head."""
    return torch.exp2(-8.0 * torch.arange(1, heads + 1, dtype=torch.float64, device="cpu") / heads).float()


class AttentionBranch(Branch):
    """Grouped-query attention with rotation, optional window and score cap, and a value size of its own.

    Options, each independent of the others:

    * ``interleaved``: the rotated pairs are (2i, 2i + 1) instead of (i, i + dims/2); ``rotary`` None: no rotation
    * ``taps``: a causal convolution over time on the channels of q and k, in front of the rotation (its inputs are per-sequence state)
    * ``keys_are_values``: v is k in front of the rotation (``vdim`` = ``dim``)
    * ``norm_eps``: q and k are divided by their root mean square behind the rotation
    * ``row_norm_eps``: the rows of q and of k, all heads together, are normalised in front of the rotation, with weights
    * ``value_norm_eps``: every value head is divided by its root mean square
    * ``in_bias``, ``out_bias``: the projections have biases (the gate's has none)
    * ``keep_first``: first tokens that the window never drops
    * ``sink``: "zero" or "learned" - a score per head in the softmax's denominator; ``slopes``: a bias by distance, per head
    * ``gate``: "value" or "head" - the sigmoid of a projection multiplies every value of the output, or a head's
    * ``source``: an earlier layer's branch whose keys and values this one reads instead of making its own

    The kernels know one head size, so q/k heads (``dim``) and v heads (``vdim``) are both padded to it inside the packed
    projections: zero rows cost nothing but projection width, leave every score unchanged and give zero output columns
    that meet zero columns of the output projection.  The rotated pairs (i, i + dims/2) are laid out at (i, i + D/2) - a
    permutation common to q and k, which no score sees - so the kernel that pairs the halves of a head serves any
    ``rot_dims``; the coordinates that are not rotated fill the other pairs and get angle 0."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, rotary: RotaryEmbedding | None, rot_dims: int,
                 padded: int, window: int | None = None, softcap: float | None = None, factor: float = 1.0, interleaved: bool = False,
                 taps: int = 0, keys_are_values: bool = False, norm_eps: float | None = None, in_bias: bool = False,
                 out_bias: bool = False, keep_first: int = 0, sink: str | None = None, slopes: torch.Tensor | None = None,
                 gate: str | None = None, source: "AttentionBranch | None" = None, row_norm_eps: float | None = None,
                 value_norm_eps: float | None = None):
        super().__init__()
        row_eps = row_norm_eps if row_norm_eps is not None else value_norm_eps
        if row_eps is not None and (norm_eps is not None or source is not None or value_norm_eps not in (None, row_eps)):
            raise ValueError("norms in front of the rotation have one epsilon, no norm behind it, and keys of their own")
        if keys_are_values and vdim != dim:
            raise ValueError(f"values that are the keys have their size, not {vdim} beside {dim}")
        if source is not None and (source.kv_heads, source.dim, source.vdim, source.d) != (kv_heads, dim, vdim, padded):
            raise ValueError(f"keys and values of {source.kv_heads} heads of {source.dim} and {source.vdim} cannot serve a layer with "
                             f"{kv_heads} of {dim} and {vdim}")
        if source is not None and taps:
            raise ValueError("a layer that borrows its keys has no convolution")
        self.heads, self.kv_heads, self.dim, self.vdim, self.d, self.rot_dims = heads, kv_heads, dim, vdim, padded, rot_dims
        self.rotary, self.interleaved, self.keys_are_values, self.gate, self.sink = rotary, interleaved, keys_are_values, gate, sink
        self.norm = None if norm_eps is None else (dim, norm_eps)
        self.in_bias, self.out_bias, self.borrows = in_bias, out_bias, source is not None
        self.attn = FlashAttention(heads, padded, scale, kv_heads, (-1 if window is None else window - 1, -1),
                                   softcap=softcap or 0.0, out_scale=factor, keep_first=keep_first,
                                   source=None if source is None else source.attn)
        if sink is not None:
            self.attn.sinks = weight_f32(heads)
        if slopes is not None:
            self.attn.slopes = nn.Parameter(slopes.to(torch.empty(0).device), requires_grad=False)
        self.made = [] if self.borrows else ["k"] if keys_are_values else ["k", "v"]
        self.qk = (heads + (0 if self.borrows else kv_heads)) * padded
        self.gate_rows = {None: 0, "value": heads * padded, "head": pad8(heads)}[gate]
        self.in_sizes = [heads * padded] + [kv_heads * padded] * len(self.made) + [self.gate_rows]
        self.in_rows = sum(self.in_sizes)
        self.out_cols = self.out_used = heads * padded
        self.row_norm, self.normed_rows = row_eps, row_norm_eps is not None
        self.value_dim = 0 if value_norm_eps is None else vdim
        if self.normed_rows:
            self.q_norm, self.k_norm = weight(heads * padded), weight(kv_heads * padded)
        self.taps = taps
        if taps:
            self.conv_weight = weight(taps, self.qk)
            self.conv_state = None

    def state_specs(self, dtype):
        return {"conv_state": ((self.taps - 1, self.qk), dtype)} if self.taps > 1 else {}

    @staticmethod
    def padded_size(dim: int, vdim: int, dtype: torch.dtype) -> int:
        d = max(dim, vdim)
        if dtype == torch.bfloat16 and d <= 256:
            return 128 if d <= 128 else 256
        return -(-d // 16) * 16

    def _layout(self) -> torch.Tensor:
        """Where coordinate i of a q/k head goes inside the padded head."""
        half, r = self.d // 2, self.rot_dims // 2
        free = [j for j in range(self.d) if not (j < r or half <= j < half + r)]
        low, high = list(range(r)), [half + i for i in range(r)]
        turned = [j for pair in zip(low, high) for j in pair] if self.interleaved else low + high
        return torch.tensor(turned + free[:self.dim - 2 * r], dtype=torch.long)

    def _place(self, name: str) -> torch.Tensor:
        """Where coordinate i of a head of ``name`` goes; values keep their order unless they are the keys."""
        return torch.arange(self.vdim) if name == "v" and not self.keys_are_values else self._layout()

    def _heads(self, src: torch.Tensor, name: str, n: int) -> torch.Tensor:
        """``src`` [n * size, ...] with every head laid out in ``d`` rows."""
        place = self._place(name).to(src.device)
        dst = src.new_zeros(n, self.d, *src.shape[1:])
        dst[:, place] = src.view(n, place.numel(), *src.shape[1:])
        return dst.flatten(0, 1)

    def load(self, w: Weights):
        rows = [self._heads(w("q"), "q", self.heads)] + [self._heads(w(n), n, self.kv_heads) for n in self.made]
        if self.taps:
            conv = [self._heads(w(n + ".conv"), n, c) for n, c in (("q", self.heads), ("k", self.kv_heads))]
            self.conv_weight.copy_(torch.cat(conv).flip(1).T)
        if self.normed_rows:
            self.q_norm.copy_(self._heads(w("q.norm"), "q", self.heads))
            self.k_norm.copy_(self._heads(w("k.norm"), "k", self.kv_heads))
        if self.gate == "value":
            rows.append(self._heads(w("g"), "v", self.heads))
        elif self.gate == "head":
            rows.append(pad_rows(w("g"), self.gate_rows))
        if self.sink == "learned":
            self.attn.sinks.copy_(w("sink").float().reshape(-1))
        o = w("o")
        place = self._place("v").to(o.device)
        cols = o.new_zeros(o.shape[0], self.heads, self.d)
        cols[:, :, place] = o.view(o.shape[0], self.heads, self.vdim)
        return torch.cat(rows), cols.view(o.shape[0], -1)

    def load_biases(self, w: Weights):
        rows = None
        if self.in_bias:
            parts = [self._heads(w("q.b"), "q", self.heads)] + [self._heads(w(n + ".b"), n, self.kv_heads) for n in self.made]
            rows = F.pad(torch.cat(parts), (0, self.gate_rows))
        return rows, w("o.b") if self.out_bias else None

    def forward(self, ctx, proj, out, positions):
        h, g, d = self.heads, self.kv_heads, self.d
        q, *made, gate = proj.split(self.in_sizes, dim=1)
        if self.taps:
            turned = ops.short_conv(proj[:, :self.qk], self.conv_weight, None, self.conv_state, ctx.state_slots, ragged(ctx), positions,
                                    copies=g * d if self.keys_are_values else 0, status=ctx.status)
            q, *rest = turned.split([h * d] + [g * d] * (2 if self.keys_are_values else 1), dim=1)
            made = rest if self.keys_are_values else [rest[0], made[1]]
        elif self.keys_are_values:
            made = [made[0], made[0].clone()]                                 # (the rotation works in place)
        q, *kv = (t.unflatten(1, (-1, d)) for t in (q, *made))
        k, v = kv or (None, None)
        o = out.unflatten(1, (h, d))
        mixed = torch.empty(o.shape, dtype=o.dtype, device=o.device) if self.gate == "value" else o
        row_norm = None
        if self.row_norm is not None:
            weights = (self.q_norm, self.k_norm) if self.normed_rows else (None, None)
            row_norm = ops.RowNorm(*weights, h * self.dim, g * self.dim, self.value_dim, self.row_norm)
        self.attn.forward_fused(ctx, q, k, v, positions, None if self.rotary is None else self.rotary.cos_sin_cache, out=mixed,
                                head_gate=gate[:, :h] if self.gate == "head" else None, norm=self.norm, row_norm=row_norm)
        if self.gate == "value":
            ops.gate_mul(mixed.flatten(1), gate, out)


class SelectiveScanBranch(Branch):
    """Mamba's selective scan: short convolution, input-dependent step and B / C, diagonal recurrence, gate."""

    def __init__(self, inner: int, states: int, dt_rank: int, taps: int):
        super().__init__()
        self.inner, self.states, self.rank, self.taps = inner, states, dt_rank, taps
        self.ip, self.rp, self.sp = pad8(inner), pad8(dt_rank), pad8(states)
        self.np = -(-states // 4) * 4
        self.in_rows, self.out_cols, self.out_used = 2 * self.ip, self.ip, inner
        self.conv_weight, self.conv_bias = weight(taps, self.ip), weight(self.ip)
        self.x_proj, self.dt_proj = weight(self.rp + 2 * self.sp, self.ip), weight(inner, self.rp)
        self.dt_bias, self.a_log2e, self.skip = weight_f32(inner), weight_f32(inner, self.np), weight_f32(inner)
        self.conv_state = self.scan_state = None

    def state_specs(self, dtype):
        return {"conv_state": ((self.taps - 1, self.ip), dtype), "scan_state": ((self.inner, self.np), torch.float32)}

    def load(self, w: Weights):
        x, z = w("in").split([self.inner, self.inner])
        self.conv_weight.copy_(pad_cols(w("conv").flip(1).T, self.ip))
        self.conv_bias.copy_(F.pad(w("conv.b"), (0, self.ip - self.inner)))
        dt, b, c = (pad_cols(t, self.ip) for t in w("x").split([self.rank, self.states, self.states]))
        self.x_proj.copy_(torch.cat([pad_rows(dt, self.rp), pad_rows(b, self.sp), pad_rows(c, self.sp)]))
        self.dt_proj.copy_(pad_cols(w("dt"), self.rp))
        self.dt_bias.copy_(w("dt.b").float())
        self.a_log2e.copy_(pad_cols(-torch.exp(w("A_log").float()) * LOG2E, self.np))
        self.skip.copy_(w("D").float())
        return torch.cat([pad_rows(x, self.ip), pad_rows(z, self.ip)]), pad_cols(w("o"), self.out_cols)

    def forward(self, ctx, proj, out, positions):
        cu = ragged(ctx)
        u = ops.short_conv_silu(proj[:, :self.ip], self.conv_weight, self.conv_bias, self.conv_state, ctx.state_slots, cu,
                                positions, status=ctx.status)
        x = F.linear(u, self.x_proj)
        dt = F.linear(x[:, :self.rp], self.dt_proj)
        ops.selective_scan(u[:, :self.inner], dt, proj[:, self.ip:self.ip + self.inner], x[:, self.rp:self.rp + self.states],
                           x[:, self.rp + self.sp:self.rp + self.sp + self.states], self.dt_bias, self.a_log2e, self.skip,
                           out[:, :self.inner], self.scan_state, ctx.state_slots, cu, positions, status=ctx.status)


class StateSpaceBranch(Branch):
    """Mamba-2: a short convolution on values, keys and queries, one decay and step per head, keys and queries shared by groups of heads,
    and a norm behind the output gate over equal parts of the row."""

    def __init__(self, heads: int, groups: int, states: int, vdim: int, taps: int, norm_groups: int, eps: float):
        super().__init__()
        if heads % groups or heads * vdim % norm_groups:
            raise ValueError(f"{heads} heads of {vdim} values do not split into {groups} groups and {norm_groups} norm groups")
        self.heads, self.groups, self.states, self.vdim, self.taps = heads, groups, states, vdim, taps
        self.norm_groups, self.eps, self.inner = norm_groups, eps, heads * vdim
        self.ip, self.gp, self.hp = pad8(self.inner), pad8(groups * states), pad8(heads)
        self.channels = self.ip + 2 * self.gp                                 # conv channels: x | B | C
        self.in_sizes = [self.ip, self.channels, self.hp]                     # z | x B C | dt
        self.in_rows, self.out_cols, self.out_used = sum(self.in_sizes), self.ip, self.inner
        self.conv_weight, self.conv_bias = weight(taps, self.channels), weight(self.channels)
        self.dt_bias, self.a_log2e, self.skip = weight_f32(heads), weight_f32(heads), weight_f32(heads)
        self.norm_weight = weight_f32(self.inner)
        self.conv_state = self.memory = None

    def state_specs(self, dtype):
        return {"conv_state": ((self.taps - 1, self.channels), dtype),
                "memory": ((self.heads, self.states, -(-self.vdim // 4) * 4), torch.float32)}

    def _channels(self, t: torch.Tensor) -> torch.Tensor:
        """Rows of x, B and C, each padded to its place."""
        gn = self.groups * self.states
        return torch.cat([pad_rows(p, n) for p, n in zip(t.split([self.inner, gn, gn]), (self.ip, self.gp, self.gp))])

    def load(self, w: Weights):
        z, xbc, dt = w("in").split([self.inner, self.inner + 2 * self.groups * self.states, self.heads])
        self.conv_weight.copy_(self._channels(w("conv")).flip(1).T)
        self.conv_bias.copy_(self._channels(w("conv.b").unsqueeze(1)).squeeze(1))
        self.dt_bias.copy_(w("dt_bias").float())
        self.a_log2e.copy_(-torch.exp(w("A_log").float()) * LOG2E)
        self.skip.copy_(w("D").float())
        self.norm_weight.copy_(w("norm").float())
        return torch.cat([pad_rows(z, self.ip), self._channels(xbc), pad_rows(dt, self.hp)]), pad_cols(w("o"), self.out_cols)

    def forward(self, ctx, proj, out, positions):
        cu, gn = ragged(ctx), self.groups * self.states
        z, xbc, dt = proj.split(self.in_sizes, dim=1)
        u = ops.short_conv_silu(xbc, self.conv_weight, self.conv_bias, self.conv_state, ctx.state_slots, cu, positions, status=ctx.status)
        x, b, c = u.split([self.ip, self.gp, self.gp], dim=1)
        b, c = (t[:, :gn].unflatten(1, (self.groups, self.states)) for t in (b, c))
        y = torch.empty(u.shape[0], self.ip, dtype=u.dtype, device=u.device)
        x, o = (t[:, :self.inner].unflatten(1, (self.heads, self.vdim)) for t in (x, y))
        ops.state_space(x, b, c, dt[:, :self.heads], self.dt_bias, self.a_log2e, self.skip, o, self.memory, ctx.state_slots, cu, positions,
                        longest=ctx.max_seqlen_q if ctx.prefill else 0, status=ctx.status)
        ops.gated_group_norm(y[:, :self.inner], z[:, :self.inner], self.norm_weight, out[:, :self.inner], self.norm_groups, self.eps)


class GatedDeltaBranch(Branch):
    """Gated delta rule with a decay per head and key channel, short convolutions on q, k, v and a gated output norm.

    The two low-rank pairs (decay, output gate) share one second GEMM with a block-diagonal weight."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, decay_rank: int, gate_rank: int, eps: float,
                 factor: float = 1.0):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps = heads, kv_heads, dim, vdim, taps
        self.eps, self.factor = eps, factor
        self.decay_rank, self.gate_rank = decay_rank, gate_rank
        self.kp, self.vp = pad8(kv_heads * dim), pad8(heads * vdim)            # conv channels: q | k | v
        self.channels = 2 * self.kp + self.vp
        self.bp, self.ap, self.gp = pad8(heads), pad8(decay_rank), pad8(gate_rank)
        self.hp = pad8(heads * dim)
        self.in_rows = self.channels + self.bp + self.ap + self.gp
        self.out_cols, self.out_used = self.vp, heads * vdim
        self.conv_weight = weight(taps, self.channels)
        self.low_rank = weight(self.hp + self.vp, self.ap + self.gp)
        self.exp_a, self.dt_bias, self.norm_weight = weight_f32(heads), weight_f32(heads * dim), weight_f32(vdim)
        self.conv_state = self.delta_state = None

    def state_specs(self, dtype):
        return {"conv_state": ((self.taps - 1, self.channels), dtype),
                "delta_state": ((self.heads, self.dim, -(-self.vdim // 4) * 4), torch.float32)}

    def load(self, w: Weights):
        sizes = {"q": self.kp, "k": self.kp, "v": self.vp}
        self.conv_weight.copy_(torch.cat([pad_cols(w(n + ".conv").flip(1).T, c) for n, c in sizes.items()], dim=1))
        self.low_rank.zero_()
        a2, g2 = w("a2"), w("g2")
        self.low_rank[:a2.shape[0], :self.decay_rank].copy_(a2)
        self.low_rank[self.hp:self.hp + g2.shape[0], self.ap:self.ap + self.gate_rank].copy_(g2)
        self.exp_a.copy_(torch.exp(w("A_log").float()).reshape(-1))
        self.dt_bias.copy_(w("dt_bias").float().reshape(-1))
        self.norm_weight.copy_(w("norm").float())
        rows = [pad_rows(w(n), c) for n, c in sizes.items()]
        rows += [pad_rows(w(n), c) for n, c in (("b", self.bp), ("a1", self.ap), ("g1", self.gp))]
        return torch.cat(rows), pad_cols(w("o"), self.out_cols)

    def forward(self, ctx, proj, out, positions):
        cu, c, kv, h = ragged(ctx), self.channels, self.kv_heads * self.dim, self.heads
        low = F.linear(proj[:, c + self.bp:], self.low_rank)
        qkv = ops.short_conv_silu(proj[:, :c], self.conv_weight, None, self.conv_state, ctx.state_slots, cu, positions,
                                  status=ctx.status)
        q, k = (qkv[:, i * self.kp:i * self.kp + kv].unflatten(1, (self.kv_heads, self.dim)) for i in (0, 1))
        v = qkv[:, 2 * self.kp:2 * self.kp + h * self.vdim].unflatten(1, (h, self.vdim))
        ops.gated_delta(q, k, v, low[:, :h * self.dim], proj[:, c:c + h], low[:, self.hp:self.hp + h * self.vdim], self.exp_a,
                        self.dt_bias, self.norm_weight, out[:, :h * self.vdim].unflatten(1, (h, self.vdim)), self.delta_state,
                        ctx.state_slots, cu, positions, self.dim ** -0.5, self.eps, self.factor, status=ctx.status)


class GatedLinearBranch(Branch):
    """Linear attention with a decay per head and key channel, ``sigmoid(z)^(1/tau)`` with z from a low-rank pair, and a SiLU-gated
    output norm."""

    def __init__(self, heads: int, dim: int, vdim: int, tau: float, decay_rank: int, eps: float):
        super().__init__()
        self.heads, self.dim, self.vdim, self.tau, self.eps, self.decay_rank = heads, dim, vdim, tau, eps, decay_rank
        self.kp, self.vp, self.ap = pad8(heads * dim), pad8(heads * vdim), pad8(decay_rank)
        self.in_rows = 2 * self.kp + 2 * self.vp + self.ap                    # q | k | v | gate | decay
        self.out_cols, self.out_used = self.vp, heads * vdim
        self.decay_up = weight(self.kp, self.ap)
        self.decay_bias, self.norm_weight = weight_f32(heads * dim), weight_f32(vdim)
        self.memory = None

    def state_specs(self, dtype):
        return {"memory": ((self.heads, self.dim, -(-self.vdim // 4) * 4), torch.float32)}

    def load(self, w: Weights):
        self.decay_up.copy_(pad_cols(pad_rows(w("a2"), self.kp), self.ap))
        self.decay_bias.copy_(w("a2.b").float().reshape(-1))
        self.norm_weight.copy_(w("norm").float())
        rows = [pad_rows(w(n), c) for n, c in (("q", self.kp), ("k", self.kp), ("v", self.vp), ("g", self.vp), ("a1", self.ap))]
        return torch.cat(rows), pad_cols(w("o"), self.out_cols)

    def forward(self, ctx, proj, out, positions):
        q, k, v, gate, a = proj.split([self.kp, self.kp, self.vp, self.vp, self.ap], dim=1)
        nk, nv = self.heads * self.dim, self.heads * self.vdim
        decay = F.linear(a, self.decay_up)
        q, k = (t[:, :nk].unflatten(1, (self.heads, self.dim)) for t in (q, k))
        v, o = (t[:, :nv].unflatten(1, (self.heads, self.vdim)) for t in (v, out))
        ops.gated_linear(q, k, v, decay[:, :nk], self.decay_bias, self.tau, gate[:, :nv], self.norm_weight, o, self.memory,
                         ctx.state_slots, ragged(ctx), positions, self.dim ** -0.5, self.eps, status=ctx.status)


class MatrixLSTMBranch(Branch):
    """Matrix memory with exponential gates per head, a normaliser and a running maximum of the exponents, and a sigmoid-gated output
    norm with a weight per head."""

    def __init__(self, heads: int, dim: int, vdim: int, gate_cap: float, eps: float):
        super().__init__()
        self.heads, self.dim, self.vdim, self.cap, self.eps = heads, dim, vdim, gate_cap, eps
        self.kp, self.vp, self.hp = pad8(heads * dim), pad8(heads * vdim), pad8(heads)
        self.in_rows = 2 * self.kp + 2 * self.vp + 2 * self.hp                # q | k | v | output gate | input gate | forget gate
        self.out_cols, self.out_used = self.vp, heads * vdim
        self.input_bias, self.forget_bias, self.norm_weight = weight_f32(heads), weight_f32(heads), weight_f32(heads * vdim)
        self.memory = self.normaliser = self.maximum = None

    def state_specs(self, dtype):
        return {"memory": ((self.heads, self.dim, -(-self.vdim // 4) * 4), torch.float32),
                "normaliser": ((self.heads, self.dim), torch.float32), "maximum": ((self.heads,), torch.float32)}

    def load(self, w: Weights):
        self.input_bias.copy_(w("i.b").float())
        self.forget_bias.copy_(w("f.b").float())
        self.norm_weight.copy_(w("norm").float())
        rows = [pad_rows(w(n), c) for n, c in (("q", self.kp), ("k", self.kp), ("v", self.vp), ("g", self.vp), ("i", self.hp), ("f", self.hp))]
        return torch.cat(rows), pad_cols(w("o"), self.out_cols)

    def forward(self, ctx, proj, out, positions):
        q, k, v, gate, i, f = proj.split([self.kp, self.kp, self.vp, self.vp, self.hp, self.hp], dim=1)
        nk, nv = self.heads * self.dim, self.heads * self.vdim
        q, k = (t[:, :nk].unflatten(1, (self.heads, self.dim)) for t in (q, k))
        v, o = (t[:, :nv].unflatten(1, (self.heads, self.vdim)) for t in (v, out))
        states = None if self.memory is None else (self.memory, self.normaliser, self.maximum)
        ops.mlstm(q, k, v, f[:, :self.heads], self.forget_bias, i[:, :self.heads], self.input_bias, self.cap, gate[:, :nv],
                  self.norm_weight, o, states, ctx.state_slots, ragged(ctx), positions, self.dim ** -0.5, self.eps, status=ctx.status)


class LatentAttentionBranch(Branch):
    """Causal attention whose keys and values are projections of one cached latent per token, with a query latent and an output gate.

    Two forms of the same product.  Prompts: keys and values of the whole context are computed from the latents (one GEMM) and go to
    the prefill attention kernel, key and value sizes padded to a size it knows.  Decoding, and whatever that kernel does not take (fp32,
    head sizes above 256): the key projection is applied to the query and the value projection to the attention's output, so that
    attention itself runs over the latents, which all heads share.

    ``source``: another latent branch, of an earlier layer, whose latents this one reads instead of making its own."""

    def __init__(self, heads: int, dim: int, vdim: int, q_rank: int, kv_rank: int, scale: float, eps: float, dtype: torch.dtype,
                 source: "LatentAttentionBranch | None" = None):
        super().__init__()
        self.num_heads = self.num_kv_heads = heads
        self.scale, self.eps, self.q_rank, self.kv_rank = scale, eps, q_rank, kv_rank
        self.__dict__["source"] = source                                      # (not a submodule of this one)
        self.expands = dtype == torch.bfloat16 and max(dim, vdim) <= 256
        self.head_dim = AttentionBranch.padded_size(dim, vdim, dtype) if self.expands else 0
        self.dim, self.vdim = dim, vdim
        self.dk, self.dv = (self.head_dim, self.head_dim) if self.expands else (pad8(dim), pad8(vdim))
        self.qp = pad8(q_rank)
        self.latent_width = pad8(kv_rank)
        if dtype == torch.bfloat16:
            self.latent_width = next((n for n in ops.LATENT_WIDTHS if n >= kv_rank), self.latent_width)
        self.tensor_core_decode = dtype == torch.bfloat16 and self.latent_width in ops.LATENT_WIDTHS
        if source is not None and source.kv_rank != kv_rank:
            raise ValueError(f"latents of {source.kv_rank} values cannot serve a layer of kv_rank {kv_rank}")
        own = self.latent_width if source is None else 0
        self.in_sizes = [self.qp, own, heads * self.dv]                       # query latent | latent | gate
        self.in_rows = sum(self.in_sizes)
        self.out_cols = self.out_used = heads * self.dv
        self.q_norm, self.q_up = weight(q_rank), weight(heads * self.dk, self.qp)
        self.kv_up = weight(heads * (self.dk + self.dv), self.latent_width)   # keys of all heads, then values
        if source is None:
            self.kv_norm = weight(kv_rank)
            self.latent_cache = torch.tensor([])                              # the executor's pool [blocks, block_size, latent_width]
        self._item_rows = None

    def load(self, w: Weights):
        def heads_of(name: str, n: int, padded: int, cols: int) -> torch.Tensor:
            src = w(name)
            dst = src.new_zeros(self.num_heads, padded, cols)
            dst[:, :n, :src.shape[1]] = src.view(self.num_heads, n, -1)
            return dst.view(self.num_heads * padded, cols)
        self.q_norm.copy_(w("dq.norm"))
        self.q_up.copy_(heads_of("uq", self.dim, self.dk, self.qp))
        self.kv_up.copy_(torch.cat([heads_of("uk", self.dim, self.dk, self.latent_width), heads_of("uv", self.vdim, self.dv, self.latent_width)]))
        rows = [pad_rows(w("dq"), self.qp)]
        if self.source is None:
            self.kv_norm.copy_(w("dkv.norm"))
            rows.append(pad_rows(w("dkv"), self.latent_width))
        rows.append(heads_of("g", self.vdim, self.dv, w("g").shape[1]))
        o = w("o")
        cols = o.new_zeros(o.shape[0], self.num_heads, self.dv)
        cols[:, :, :self.vdim] = o.view(o.shape[0], self.num_heads, self.vdim)
        return torch.cat(rows), cols.view(o.shape[0], -1)

    def forward(self, ctx, proj, out, positions):
        dq, c, gate = proj.split(self.in_sizes, dim=1)
        owner = self if self.source is None else self.source
        cache = owner.latent_cache if owner.latent_cache.numel() else None
        if self.source is None:
            cq, c = ops.latent_norm(dq[:, :self.q_rank], self.q_norm, self.qp, c[:, :self.kv_rank], self.kv_norm, self.latent_width,
                                    self.eps, cache, ctx.slot_mapping, status=ctx.status)
            ctx.shared[owner] = c                                            # this step's rows, for layers that share them
        else:
            cq, _ = ops.latent_norm(dq[:, :self.q_rank], self.q_norm, self.qp, None, None, 0, self.eps, status=ctx.status)
            c = ctx.shared[owner]
        q = F.linear(cq, self.q_up).unflatten(1, (self.num_heads, self.dk))
        o = torch.empty(q.shape[0], self.num_heads, self.dv, dtype=q.dtype, device=q.device)
        if not self.expands or (not self.tensor_core_decode and (not ctx.prefill or ctx.num_decode)):
            self._absorbed(ctx, q, c, cache, positions, o)
        elif not ctx.prefill:
            self._decode(ctx, q, cache, ctx.block_table, o)
        else:
            nd = ctx.num_decode
            bp, tp = ctx.cu_seqlens_q.numel() - 1 - nd, q.shape[0] - nd
            self._prompts(ctx, q[:tp], c, cache, ctx.cu_seqlens_q[:bp + 1], ctx.cu_seqlens_k[:bp + 1],
                          None if ctx.block_table is None else ctx.block_table[:bp], o[:tp])
            if nd:
                self._decode(ctx, q[tp:], cache, ctx.block_table[bp:], o[tp:])
        ops.gate_mul(o.flatten(1), gate, out)

    def _prompts(self, ctx, q, c, cache, cu_q, cu_k, table, o) -> None:
        if table is not None:                                                 # earlier tokens are in the cache
            c = ops.gather_latents(cache, table, cu_k, ctx.prompt_keys, status=ctx.status)
        kv = F.linear(c, self.kv_up).unflatten(1, (2 * self.num_heads, self.head_dim))
        k, v = kv.split([self.num_heads, self.num_heads], dim=1)
        ops.prefill_attn(q, k, v, cu_q, cu_k, ctx.max_seqlen_q, self.scale, -1, out=o, status=ctx.status, items=prefill_items_for(ctx, self))

    def _up(self) -> tuple[torch.Tensor, torch.Tensor]:
        """Key projection [heads, dk, latent] and value projection [heads, latent, dv] as views."""
        k, v = self.kv_up.split([self.num_heads * self.dk, self.num_heads * self.dv])
        return k.unflatten(0, (self.num_heads, self.dk)), v.unflatten(0, (self.num_heads, self.dv)).transpose(1, 2)

    def _decode(self, ctx, q, cache, table, o) -> None:
        uk, uv = self._up()
        key = ("latent", self.num_heads, self.latent_width)
        ws = ctx.decode_plans.get(key)
        if ws is None:
            ws = decode_workspace_for(q.device, ctx.cache_seqlens.numel(), self.num_heads, 1, self.latent_width, key)
            ops.latent_decode_plan(ctx.cache_seqlens, table, cache.shape[1], self.num_heads, self.latent_width, ws)
            ctx.decode_plans[key] = ws
        mixed = ops.latent_decode(torch.bmm(q.transpose(0, 1), uk), cache, ctx.cache_seqlens, table, self.scale, ws, status=ctx.status)
        torch.bmm(mixed, uv, out=o.transpose(0, 1))

    def _absorbed(self, ctx, q, c, cache, positions, o) -> None:
        uk, uv = self._up()
        paged = ctx.block_table is not None
        keys = cache.unsqueeze(2) if paged else c.unsqueeze(1)
        mixed = ops.any_attn(torch.bmm(q.transpose(0, 1), uk).transpose(0, 1).contiguous(), keys, keys, positions, self.scale,
                             cu_seqlens_q=ctx.cu_seqlens_q if ctx.prefill else None, cu_seqlens_k=ctx.cu_seqlens_k,
                             block_table=ctx.block_table, cache_seqlens=None if ctx.prefill else ctx.cache_seqlens, status=ctx.status)
        torch.bmm(mixed.transpose(0, 1), uv, out=o.transpose(0, 1))


class PackedMixer(nn.Module):
    """Branches side by side on one input; their outputs meet in one output projection.

    ``feed``: a feed-forward (``feedforward.py``) beside the branches, on an input of its own, whose down projection is part of the
    same output projection."""

    def __init__(self, width: int, branches: dict[str, Branch], feed: nn.Module | None = None):
        super().__init__()
        self.branches, self.feed = nn.ModuleDict(branches), feed
        self.in_sizes = [b.in_rows for b in branches.values()]
        self.out_sizes = [b.out_cols for b in branches.values()] + ([] if feed is None else [feed.out_cols])
        self.in_proj, self.out_proj = weight(sum(self.in_sizes), width), weight(width, sum(self.out_sizes))
        self.in_bias = weight(sum(self.in_sizes)) if any(b.in_bias for b in branches.values()) else None
        self.out_bias = weight(width) if any(b.out_bias for b in branches.values()) else None
        self.dense_out = all(b.out_used == b.out_cols for b in branches.values())

    @torch.no_grad()
    def load(self, prefixes: dict[str, str], w: Weights, feed_prefix: str = "") -> None:
        named = [(b, lambda n, p=prefixes[key]: w(p + n)) for key, b in self.branches.items()]
        parts = [b.load(of) for b, of in named]
        cols = [p[1] for p in parts]
        if self.feed is not None:
            down = self.feed.load(lambda n: w(feed_prefix + n))
            cols += [] if down is None else [down]
        self.in_proj.copy_(torch.cat([p[0] for p in parts]))
        self.out_proj.copy_(torch.cat(cols, dim=1))
        biases = [b.load_biases(of) for b, of in named]
        if self.in_bias is not None:
            self.in_bias.copy_(torch.cat([self.in_bias.new_zeros(n) if b[0] is None else b[0] for n, b in zip(self.in_sizes, biases)]))
        if self.out_bias is not None:
            self.out_bias.copy_(sum(b[1].float() for b in biases if b[1] is not None))

    def forward(self, ctx: Context, h: torch.Tensor, positions: torch.Tensor, h_feed: torch.Tensor | None = None) -> torch.Tensor:
        proj = F.linear(h, self.in_proj, self.in_bias)
        make = torch.empty if self.dense_out else torch.zeros     # columns nobody writes meet zero weights and must be finite
        y = make(h.shape[0], self.out_proj.shape[1], dtype=h.dtype, device=h.device)
        cols = y.split(self.out_sizes, dim=1)
        for b, pi, yi in zip(self.branches.values(), proj.split(self.in_sizes, dim=1), cols):
            b(ctx, pi, yi, positions)
        if self.feed is not None:
            self.feed.write(h_feed, cols[-1])
        return F.linear(y, self.out_proj, self.out_bias)
