"""Residual streams: what lies between the sublayers of an assembled decoder.

A stream object starts the residual from the token ids and, after each sublayer, takes the sublayer's output in and hands out the
normalised input of the next one - one kernel each time.  Its per-sublayer parameters are a connection module, so a layer holds one
per sublayer:

* ``SandwichStream``: one fp32 stream, a norm in front of and behind every sublayer;
* ``HyperStream``: several fp32 streams.  A sublayer reads a weighted sum of them; afterwards every stream becomes a weighted sum of all
  old ones plus its own multiple of the output.  Norms in equal consecutive groups, learned positions added to the embedding;
* ``ParallelStream``: one fp32 stream, from which a mixer and a feed-forward side by side read through norms of their own or through one
  they share.
"""
from __future__ import annotations

import torch
from torch import nn

from ... import ops
from .branches import Weights, weight, weight_f32


def gain(width: int) -> nn.Parameter:
    return nn.Parameter(torch.ones(width), requires_grad=False)


class SandwichConnection(nn.Module):
    def __init__(self, width: int):
        super().__init__()
        self.norm, self.out_norm = gain(width), gain(width)

    @torch.no_grad()
    def load(self, prefix: str, index: int, w: Weights) -> None:
        self.norm.copy_(w(f"{prefix}norm{index}"))
        self.out_norm.copy_(w(f"{prefix}norm{index}b"))


class SandwichStream(nn.Module):
    def __init__(self, width: int, eps: float):
        super().__init__()
        self.width, self.eps = width, eps

    def connection(self) -> nn.Module:
        return SandwichConnection(self.width)

    def load(self, w: Weights) -> None:
        pass

    def start(self, ctx, ids: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, first: SandwichConnection):
        return ops.embed_norm(ids, table, first.norm, self.eps, status=ctx.status)

    def advance(self, x: torch.Tensor, y: torch.Tensor, done: SandwichConnection, following: SandwichConnection | None,
                final_norm: torch.Tensor, rows: torch.Tensor | None = None) -> torch.Tensor:
        return ops.residual_norm(x, y, final_norm if following is None else following.norm, self.eps, y_weight=done.out_norm, row_ends=rows)

    @staticmethod
    def total(x: torch.Tensor) -> torch.Tensor:
        return x


class HyperConnection(nn.Module):
    def __init__(self, width: int, streams: int):
        super().__init__()
        self.norm = gain(width)
        self.in_weights, self.out_weights, self.mix = weight_f32(streams), weight_f32(streams), weight_f32(streams, streams)

    @torch.no_grad()
    def load(self, prefix: str, index: int, w: Weights) -> None:
        self.norm.copy_(w(f"{prefix}norm{index}"))
        self.in_weights.copy_(w(f"{prefix}hc{index}.in"))
        self.out_weights.copy_(w(f"{prefix}hc{index}.out"))
        self.mix.copy_(w(f"{prefix}hc{index}.mix"))                   # [from, to]


class HyperStream(nn.Module):
    def __init__(self, width: int, eps: float, streams: int, groups: int, positions: int):
        super().__init__()
        if width % groups:
            raise ValueError(f"a width of {width} does not split into {groups} norm groups")
        self.width, self.eps, self.streams, self.groups = width, eps, streams, groups
        self.positions = weight(positions, width)

    def connection(self) -> nn.Module:
        return HyperConnection(self.width, self.streams)

    @torch.no_grad()
    def load(self, w: Weights) -> None:
        self.positions.copy_(w("pos"))

    def start(self, ctx, ids: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, first: HyperConnection):
        return ops.hyper_embed_norm(ids, positions, table, self.positions, self.streams, first.in_weights, first.norm, self.eps,
                                    self.groups, status=ctx.status)

    def advance(self, x: torch.Tensor, y: torch.Tensor, done: HyperConnection, following: HyperConnection | None,
                final_norm: torch.Tensor, rows: torch.Tensor | None = None) -> torch.Tensor:
        in_weights, norm = (None, final_norm) if following is None else (following.in_weights, following.norm)
        return ops.hyper_norm(x, y, done.mix, done.out_weights, in_weights, norm, self.eps, self.groups, row_ends=rows)

    @staticmethod
    def total(x: torch.Tensor) -> torch.Tensor:
        return x.sum(1)


class ParallelConnection(nn.Module):
    def __init__(self, width: int, norms: int):
        super().__init__()
        self.norm, self.feed_norm = gain(width), gain(width) if norms > 1 else None

    @torch.no_grad()
    def load(self, prefix: str, index: int, w: Weights) -> None:
        self.norm.copy_(w(f"{prefix}norm{index}"))                    # (a single number is every coordinate's)
        if self.feed_norm is not None:
            self.feed_norm.copy_(w(f"{prefix}norm{index + 1}"))


class ParallelStream(nn.Module):
    """A sublayer's input is a pair of normalised rows (the second None without a feed-forward, the same as the first with
    ``shared_norm``); its output what one GEMM adds up, with what routed experts add beside it, if there are any."""

    def __init__(self, width: int, eps: float, embedding_scale: float = 1.0, shared_norm: bool = False):
        super().__init__()
        self.width, self.eps, self.embedding_scale, self.shared_norm = width, eps, embedding_scale, shared_norm

    def connection(self, norms: int = 2) -> nn.Module:
        return ParallelConnection(self.width, 1 if self.shared_norm else norms)

    def load(self, w: Weights) -> None:
        pass

    def start(self, ctx, ids: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, first: ParallelConnection):
        x, h, h_feed = ops.embed_norm_pair(ids, table, self.embedding_scale, first.norm, first.feed_norm, self.eps, status=ctx.status)
        return x, (h, h if self.shared_norm else h_feed)

    def advance(self, x: torch.Tensor, y, done: ParallelConnection, following: ParallelConnection | None, final_norm: torch.Tensor,
                rows: torch.Tensor | None = None):
        summed, routed = y
        norm, feed_norm = (final_norm, None) if following is None else (following.norm, following.feed_norm)
        more = {} if routed is None else {"extra": routed.rows, "extra_index": routed.slots, "own": routed.own, "own_weights": routed.own_weights}
        h, h_feed = ops.residual_norm_pair(x, summed, norm, feed_norm, self.eps, row_ends=rows, **more)
        return h if following is None else (h, h if self.shared_norm else h_feed)

    @staticmethod
    def total(x: torch.Tensor) -> torch.Tensor:
        return x
