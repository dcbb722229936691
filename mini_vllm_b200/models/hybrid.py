"""Decoder assembled layer by layer from mixer branches (attention, latent attention, selective scan, state space, gated delta rule,
gated linear attention, matrix-memory LSTM), a feed-forward of its own kind, and an fp32 residual of its own kind
(``layers/residual.py``), with optional tanh caps on the logits.

The step contract is ``DecoderLM``'s (``models/decoder.py``): ``forward(ctx, input_ids, positions, head)``, one row per
sequence - or per entry of ``ctx.logit_rows`` - and the same loader, executor, KV pool, CUDA graphs and sampler.  Recurrent
branches keep a row of state per sequence in slots that the scheduler hands out with the KV blocks; a sequence whose
first token of a step has position 0 starts from zero, so a reused slot needs no clearing.

Per sublayer the kernels are: input GEMM, branch kernels, output GEMM, and one kernel for everything between the sublayer's output
and the normalised input of the next one.  A layer has its mixer and its feed-forward one after the other (``HybridLayer``) or side by
side as one sublayer (``ParallelLayer``).
"""
from __future__ import annotations

from typing import Iterable

import torch
import torch.nn.functional as F
from torch import nn

from .. import ops
from ..executor.context import Context
from .layers.branches import PackedMixer, Weights, pad8, pad_cols, pad_rows, weight, weight_f32


class ClampedGLU(nn.Module):
    """``down(g sigmoid(alpha g) (u + 1))`` with ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``."""

    def __init__(self, width: int, inter: int, limit: float, alpha: float):
        super().__init__()
        self.ip, self.limit, self.alpha = pad8(inter), limit, alpha        # padding: gate 0 gives 0
        self.gate_up, self.down = weight(2 * self.ip, width), weight(width, self.ip)

    @torch.no_grad()
    def load(self, w: Weights) -> None:
        self.gate_up.copy_(torch.cat([pad_rows(w("gate"), self.ip), pad_rows(w("up"), self.ip)]))
        self.down.copy_(pad_cols(w("down"), self.ip))

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return F.linear(ops.clamped_glu(F.linear(h, self.gate_up), self.ip, self.limit, self.alpha), self.down)


class PolyNormMLP(nn.Module):
    """``down(a N(z) + b N(z^2) + c N(z^3) + e)`` with ``z = up(h)``, N over the row's root mean square, and four learned numbers."""

    def __init__(self, width: int, inter: int, eps: float):
        super().__init__()
        self.inter, self.ip, self.eps = inter, pad8(inter), eps
        self.up, self.down, self.act = weight(self.ip, width), weight(width, self.ip), weight_f32(4)

    @torch.no_grad()
    def load(self, w: Weights) -> None:
        self.up.copy_(pad_rows(w("up"), self.ip))
        self.down.copy_(pad_cols(w("down"), self.ip))
        self.act.copy_(w("act"))

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return F.linear(ops.poly_norm(F.linear(h, self.up), self.inter, self.act, self.eps), self.down)


class HybridLayer(nn.Module):
    """A mixer and, optionally, a feed-forward, each with its connection to the residual stream."""

    def __init__(self, stream: nn.Module, mixer: PackedMixer, mlp: nn.Module | None):
        super().__init__()
        self.mixer, self.mlp = mixer, mlp
        self.connections = nn.ModuleList([stream.connection() for _ in range(1 if mlp is None else 2)])

    def sublayers(self):
        """(connection, callable(ctx, h, positions)) in order."""
        yield self.connections[0], self.mixer
        if self.mlp is not None:
            yield self.connections[1], lambda ctx, h, positions: self.mlp(h)


    @torch.no_grad()
    def load(self, prefix: str, mixer_prefixes: dict[str, str], w: Weights) -> None:
        self.mixer.load(mixer_prefixes, w)
        for q, connection in enumerate(self.connections, 1):
            connection.load(prefix, q, w)
        if self.mlp is not None:
            self.mlp.load(lambda n: w(prefix + "mlp." + n))


class ParallelLayer(nn.Module):
    """A mixer and, optionally, a feed-forward beside it: one sublayer over two norms of the same stream (``ParallelStream``).  The
    feed-forward is part of the mixer's packed output projection; routed experts' rows are added where the stream is brought up to date."""

    def __init__(self, stream: nn.Module, mixer: PackedMixer):
        super().__init__()
        self.mixer = mixer
        self.connections = nn.ModuleList([stream.connection(1 if mixer.feed is None else 2)])

    def run(self, ctx: Context, h: tuple, positions: torch.Tensor):
        h_mix, h_feed = h
        y = self.mixer(ctx, h_mix, positions, h_feed)
        return y, None if self.mixer.feed is None else self.mixer.feed.routed(h_feed, ctx.status)

    def sublayers(self):
        yield self.connections[0], self.run

    @torch.no_grad()
    def load(self, prefix: str, mixer_prefixes: dict[str, str], w: Weights) -> None:
        self.mixer.load(mixer_prefixes, w, prefix + "mlp.")
        self.connections[0].load(prefix, 1, w)


class HybridDecoder(nn.Module):
    def __init__(self, cfg, layers: list[HybridLayer | ParallelLayer], stream: nn.Module):
        super().__init__()
        self.config, self.eps = cfg, cfg.rms_norm_eps
        self.logit_cap = float(getattr(cfg, "logit_softcap", None) or 0.0)
        self.embed_tokens = weight(cfg.vocab_size, cfg.hidden_size)
        self.stream = stream
        self.layers = nn.ModuleList(layers)
        self.norm = nn.Parameter(torch.ones(cfg.hidden_size), requires_grad=False)
        self.lm_head_weight = weight(cfg.vocab_size, cfg.hidden_size)
        # with recurrent branches the scheduler hands out state slots
        self.recurrent = any(b.state_specs(torch.float32) for layer in layers for b in layer.mixer.branches.values())
        self.residual_tap = None          # debugging aid: called with (layer index, residual stream) after each layer

    # ---- step ----------------------------------------------------------------------------------
    def forward(self, ctx: Context, input_ids: torch.Tensor, positions: torch.Tensor, head: bool = True) -> torch.Tensor:
        flags = torch.backends.cuda.matmul
        reduced = flags.allow_bf16_reduced_precision_reduction
        flags.allow_bf16_reduced_precision_reduction = False       # split-K partial sums stay fp32
        try:
            h = self._hidden_rows(ctx, input_ids, positions)
            return self.logits(h) if head else h
        finally:
            flags.allow_bf16_reduced_precision_reduction = reduced

    def _hidden_rows(self, ctx: Context, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        steps = [(i, *sub) for i, layer in enumerate(self.layers) for sub in layer.sublayers()]
        x, h = self.stream.start(ctx, input_ids, positions, self.embed_tokens, steps[0][1])
        rows = None
        if ctx.prefill:
            rows = ctx.logit_rows if ctx.logit_rows is not None else ctx.cu_seqlens_q
        for n, (i, connection, run) in enumerate(steps):
            y = run(ctx, h, positions)
            last = n == len(steps) - 1
            following = None if last else steps[n + 1][1]
            if last and self.residual_tap is None:
                # the head reads a few rows: the closing add + final norm gather those themselves
                return self.stream.advance(x, y, connection, None, self.norm, rows)
            h = self.stream.advance(x, y, connection, following, self.norm)
            if self.residual_tap is not None and (last or steps[n + 1][0] != i):
                self.residual_tap(i, self.stream.total(x))
        return h if rows is None else h[(rows[1:] - 1).long()]

    def logits(self, hidden_rows: torch.Tensor, out_dtype: torch.dtype | None = None) -> torch.Tensor:
        """Capped logits of final-norm rows, in the model's dtype unless told otherwise."""
        if hidden_rows.dtype == torch.float32:
            raw = F.linear(hidden_rows, self.lm_head_weight)
        else:
            raw = torch.mm(hidden_rows, self.lm_head_weight.T, out_dtype=torch.float32)
        return ops.cap_logits(raw, self.logit_cap, out_dtype or hidden_rows.dtype)

    @property
    def fuses_greedy_head(self) -> bool:
        return self.lm_head_weight.dtype == torch.bfloat16 and self.config.hidden_size % 64 == 0

    def greedy_tokens(self, hidden_rows: torch.Tensor, scratch: torch.Tensor, out: torch.Tensor | None = None,
                      scatter_table: torch.Tensor | None = None, scatter_index: torch.Tensor | None = None,
                      status: torch.Tensor | None = None) -> torch.Tensor:
        """argmax of the head in one kernel; the cap is monotonic, so the uncapped logits decide."""
        return ops.lm_head_argmax(hidden_rows, self.lm_head_weight, scratch, out=out, scatter_table=scatter_table,
                                  scatter_index=scatter_index, status=status)

    # ---- weights ---------------------------------------------------------------------------------
    def mixer_prefixes(self, index: int) -> dict[str, str]:
        """Checkpoint prefix of each branch of layer ``index``."""
        raise NotImplementedError

    def random_tensors(self, seed: int):
        """(name, tensor) pairs in checkpoint form for a random-init model."""
        raise NotImplementedError

    def init_random(self, seed: int) -> None:
        self.load_weights(self.random_tensors(seed))

    @torch.no_grad()
    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> None:
        tensors, used = dict(weights), set()
        dev = self.embed_tokens.device

        def w(name: str) -> torch.Tensor:
            if name not in tensors:
                raise KeyError(f"the checkpoint has no tensor {name}")
            used.add(name)
            return tensors[name].to(dev)

        self.embed_tokens.copy_(w("embed"))
        self.norm.copy_(w("final.norm"))
        self.lm_head_weight.copy_(w("head"))
        self.stream.load(w)
        for i, layer in enumerate(self.layers):
            layer.load(f"l{i}.", self.mixer_prefixes(i), w)
        unknown = set(tensors) - used
        if unknown:
            raise KeyError(f"unrecognised parameter {sorted(unknown)[0]}")
