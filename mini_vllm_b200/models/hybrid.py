"""Decoder assembled layer by layer from mixer branches (attention, selective scan, gated delta rule), with norms before
and after each sublayer, an fp32 residual stream, and optional tanh caps on the logits.

The step contract is ``DecoderLM``'s (``models/decoder.py``): ``forward(ctx, input_ids, positions, head)``, one row per
sequence - or per entry of ``ctx.logit_rows`` - and the same loader, executor, KV pool, CUDA graphs and sampler.  Recurrent
branches keep a row of state per sequence in slots that the scheduler hands out with the KV blocks; a sequence whose
first token of a step has position 0 starts from zero, so a reused slot needs no clearing.

Per sublayer the kernels are: input GEMM, branch kernels, output GEMM, and one kernel for [norm of the branch output +
residual add + norm for the next sublayer].
"""
from __future__ import annotations

from typing import Iterable

import torch
import torch.nn.functional as F
from torch import nn

from .. import ops
from ..executor.context import Context
from .layers.branches import PackedMixer, pad8, pad_cols, pad_rows, weight


class ClampedGLU(nn.Module):
    """``down(g sigmoid(alpha g) (u + 1))`` with ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``."""

    def __init__(self, width: int, inter: int, limit: float, alpha: float):
        super().__init__()
        self.ip, self.limit, self.alpha = pad8(inter), limit, alpha        # padding: gate 0 gives 0
        self.gate_up, self.down = weight(2 * self.ip, width), weight(width, self.ip)

    @torch.no_grad()
    def load(self, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> None:
        self.gate_up.copy_(torch.cat([pad_rows(gate, self.ip), pad_rows(up, self.ip)]))
        self.down.copy_(pad_cols(down, self.ip))

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return F.linear(ops.clamped_glu(F.linear(h, self.gate_up), self.ip, self.limit, self.alpha), self.down)


class HybridLayer(nn.Module):
    """A mixer and, optionally, a feed-forward; each between a norm of its input and a norm of its output."""

    def __init__(self, width: int, mixer: PackedMixer, mlp: nn.Module | None):
        super().__init__()
        self.mixer, self.mlp = mixer, mlp
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp is not None else ()):
            self.register_parameter(name, nn.Parameter(torch.ones(width), requires_grad=False))

    def sublayers(self):
        """(input norm, callable(ctx, h, positions), output norm) in order."""
        yield self.norm1, self.mixer, self.norm1b
        if self.mlp is not None:
            yield self.norm2, (lambda ctx, h, positions: self.mlp(h)), self.norm2b


class HybridDecoder(nn.Module):
    recurrent = False          # set by subclasses with recurrent branches: the scheduler hands out state slots

    def __init__(self, cfg, layers: list[HybridLayer]):
        super().__init__()
        self.config, self.eps = cfg, cfg.rms_norm_eps
        self.logit_cap = float(getattr(cfg, "logit_softcap", None) or 0.0)
        self.embed_tokens = weight(cfg.vocab_size, cfg.hidden_size)
        self.layers = nn.ModuleList(layers)
        self.norm = nn.Parameter(torch.ones(cfg.hidden_size), requires_grad=False)
        self.lm_head_weight = weight(cfg.vocab_size, cfg.hidden_size)
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
        x, h = ops.embed_norm(input_ids, self.embed_tokens, steps[0][1], self.eps, status=ctx.status)
        rows = None
        if ctx.prefill:
            rows = ctx.logit_rows if ctx.logit_rows is not None else ctx.cu_seqlens_q
        for n, (i, _, run, out_norm) in enumerate(steps):
            last = n == len(steps) - 1
            y = run(ctx, h, positions)
            if last and self.residual_tap is None:
                # the head reads a few rows: the closing add + final norm gather those themselves
                return ops.residual_norm(x, y, self.norm, self.eps, y_weight=out_norm, row_ends=rows)
            h = ops.residual_norm(x, y, self.norm if last else steps[n + 1][1], self.eps, y_weight=out_norm)
            if self.residual_tap is not None and (last or steps[n + 1][0] != i):
                self.residual_tap(i, x)
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
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            layer.mixer.load(self.mixer_prefixes(i), w)
            layer.norm1.copy_(w(p + "norm1")); layer.norm1b.copy_(w(p + "norm1b"))
            if layer.mlp is not None:
                layer.norm2.copy_(w(p + "norm2")); layer.norm2b.copy_(w(p + "norm2b"))
                layer.mlp.load(w(p + "mlp.gate"), w(p + "mlp.up"), w(p + "mlp.down"))
        unknown = set(tensors) - used
        if unknown:
            raise KeyError(f"unrecognised parameter {sorted(unknown)[0]}")
