"""Feed-forwards that sit beside a mixer on the same packed output projection.

One declares how many columns it brings (``out_cols``), writes its activations into them, and its down projection becomes part of the
layer's one output GEMM - which thereby adds mixer and feed-forward up.  What cannot go that way (experts: every token has its own
weights) comes back as rows to be added to the residual stream (``routed``).
"""
from __future__ import annotations

from dataclasses import dataclass, replace

import torch
import torch.nn.functional as F
from torch import nn

from ... import ops
from .branches import Weights, pad8, pad_cols, pad_rows, weight, weight_f32


@dataclass(frozen=True)
class Routed:
    """What routed experts add to the residual stream: token t gets ``rows[slots[t, j]]`` for every j (a slot of -1: nothing) and, with
    identity experts, ``own_weights[t]`` times its own input row."""
    rows: torch.Tensor
    slots: torch.Tensor
    own: torch.Tensor | None = None
    own_weights: torch.Tensor | None = None


class GatedFeed(nn.Module):
    """``g sigmoid(alpha g) (u + offset)`` with ``g = min(gate h, limit)``, ``u = clamp(up h, -limit, limit)``; the defaults are the
    SiLU-gated unit.  ``token_gate``: the whole is multiplied by the sigmoid of a number per token (the row ``sg``)."""

    def __init__(self, width: int, inter: int, limit: float = float("inf"), alpha: float = 1.0, offset: float = 0.0, token_gate: bool = False):
        super().__init__()
        self.ip, self.unit, self.token_gate = pad8(inter), (limit, alpha, offset), token_gate    # padding: gate 0 gives 0
        self.out_cols = self.ip
        self.gate_up = weight(2 * self.ip + (8 if token_gate else 0), width)

    @torch.no_grad()
    def load(self, w: Weights) -> torch.Tensor:
        rows = [pad_rows(w("gate"), self.ip), pad_rows(w("up"), self.ip)]
        if self.token_gate:
            rows.append(pad_rows(w("sg"), 8))
        self.gate_up.copy_(torch.cat(rows))
        return pad_cols(w("down"), self.ip)

    def write(self, h: torch.Tensor, out: torch.Tensor) -> None:
        z = F.linear(h, self.gate_up)
        ops.glu(z[:, :2 * self.ip], self.ip, *self.unit, row_gate=z[:, 2 * self.ip] if self.token_gate else None, out=out)

    def routed(self, h: torch.Tensor, status: torch.Tensor | None) -> None:
        return None


class XieluFeed(nn.Module):
    """``p z^2 + z / 2`` for z = up h > 0, ``(1/2 + q) (e^z - 1 - z) + z / 2`` below, p and q the softplus of two learned numbers."""

    def __init__(self, width: int, inter: int):
        super().__init__()
        self.ip = self.out_cols = pad8(inter)                                     # padding: 0 gives 0
        self.up, self.act = weight(self.ip, width), weight_f32(2)

    @torch.no_grad()
    def load(self, w: Weights) -> torch.Tensor:
        self.up.copy_(pad_rows(w("up"), self.ip))
        self.act.copy_(F.softplus(w("act").float()) + torch.tensor([0.0, 0.5], device=self.act.device))
        return pad_cols(w("down"), self.ip)

    def write(self, h: torch.Tensor, out: torch.Tensor) -> None:
        ops.xielu(F.linear(h, self.up), self.act, out=out)

    def routed(self, h: torch.Tensor, status: torch.Tensor | None) -> None:
        return None


class ExpertFeed(nn.Module):
    """Each token through the ``top`` of ``experts`` gated units that score highest.  ``shared`` (a ``GatedFeed``) runs for every token
    beside them.

    Options: ``softmax`` - scores are the softmax over all router outputs instead of sigmoids; ``corrected`` - a number per output is
    added for the choice alone; ``scale`` - a factor of the scores as weights; ``weigh_output`` - the weight multiplies the expert's output
    instead of its input; ``identity`` - so many further router outputs return the token's own row."""

    def __init__(self, width: int, inter: int, experts: int, top: int, limit: float = float("inf"), alpha: float = 1.0, offset: float = 0.0,
                 shared: GatedFeed | None = None, softmax: bool = False, corrected: bool = False, scale: float = 1.0,
                 weigh_output: bool = False, identity: int = 0):
        super().__init__()
        if not 0 < top <= experts + identity:
            raise ValueError(f"{top} of {experts + identity} experts cannot be chosen")
        self.width, self.inter, self.ip, self.top, self.unit, self.shared = width, inter, pad8(inter), top, (limit, alpha, offset), shared
        self.experts, self.weigh_output = experts, weigh_output
        self.correction = weight_f32(experts + identity) if corrected else None
        self.routing = ops.Routing(softmax, None, scale, identity)
        self.out_cols = 0 if shared is None else shared.out_cols
        kp = width if torch.get_default_dtype() == torch.float32 else pad8(width)      # (TMA rows start at 16-byte boundaries)
        self.router = weight(experts + identity, width)
        self.gate_up, self.down = weight(experts, 2, self.ip, kp), weight(experts, width, self.ip)
        self.register_buffer("counters", torch.zeros(experts + 1, dtype=torch.int32), persistent=False)

    @torch.no_grad()
    def load(self, w: Weights) -> torch.Tensor | None:
        self.router.copy_(w("router"))
        if self.correction is not None:
            self.correction.copy_(w("correction").float())
        for e in range(self.experts):
            for i, name in enumerate(("gate", "up")):
                self.gate_up[e, i].copy_(pad_cols(pad_rows(w(f"e{e}.{name}"), self.ip), self.gate_up.shape[3]))
            self.down[e].copy_(pad_cols(w(f"e{e}.down"), self.ip))
        return None if self.shared is None else self.shared.load(lambda n: w("shared." + n))

    def write(self, h: torch.Tensor, out: torch.Tensor) -> None:
        if self.shared is not None:
            self.shared.write(h, out)

    def routed(self, h: torch.Tensor, status: torch.Tensor | None) -> Routed:
        if h.dtype == torch.float32:
            logits = F.linear(h, self.router)
        else:
            logits = torch.mm(h, self.router.T, out_dtype=torch.float32)
        x, rows = ops.moe_sort(h, logits, self.top, self.counters, replace(self.routing, correction=self.correction))
        y = ops.moe_gemm(x, self.gate_up, rows, self.width, gated=self.unit, weigh_output=self.weigh_output, status=status)
        return Routed(ops.moe_gemm(y, self.down, rows, self.ip, status=status), rows.slots, h, rows.identity)
