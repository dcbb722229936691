"""The Sunulorn decoder restated plainly: one whole sequence at a time, one function per mechanism.  TEST INFRASTRUCTURE.

Everything runs on the CPU in the dtype of ``OracleSunulorn`` (float64 unless a caller asks for float32), from the checkpoint's own
tensor names and the parsed ``config.json``.  Nothing here is shared with the product package: no paging, no padding, no packing, no
permuted coordinates, no sorting of tokens by expert.

Symbols: ``x`` is the residual stream [T, width], ``h`` a normalised input, ``q``, ``k``, ``v`` are [T, heads, size].
"""
from __future__ import annotations

import math

import torch


# ---- elementary mechanisms -------------------------------------------------------------------------------
def rms_norm(x: torch.Tensor, w: torch.Tensor | None, eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, channels], w [channels, taps]; the last tap weighs the token itself, zeros before the start."""
    taps, y = w.shape[1], torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y[t] = y[t] + w[:, j] * u[src]
    return y


def rotate(z: torch.Tensor, dims: int, base: float, interleaved: bool) -> torch.Tensor:
    """z [T, heads, d]: the first ``dims`` coordinates in pairs, turned by position times base^(-2i/dims)."""
    out = z.clone()
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        angle = torch.arange(z.shape[0], dtype=z.dtype)[:, None] * base ** (-2.0 * i / dims)
        u, v = z[..., a], z[..., b]
        out[..., a] = u * angle.cos() - v * angle.sin()
        out[..., b] = v * angle.cos() + u * angle.sin()
    return out


def visible(t: int, size: int | None, keep_first: int) -> torch.Tensor:
    """[T, T] of booleans: which keys (columns) a query (row) sees."""
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    near = (j >= 0) if size is None else ((i - j < size) | (j < keep_first))
    return (j <= i) & near


def alibi_slope(h: int, heads: int) -> float:
    return 2.0 ** (-8.0 * (h + 1) / heads)


def attention(q, k, v, scale: float, seen: torch.Tensor, sinks: torch.Tensor | None = None, slopes=None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv].  ``sinks`` [H]: a score that takes its part of the softmax and gives
    nothing; ``slopes`` [H]: taken off a score per token of distance."""
    t, heads, group = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    out = torch.empty(t, heads, v.shape[2], dtype=q.dtype)
    distance = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).to(q.dtype)
    for h in range(heads):
        s = q[:, h] @ k[:, h // group].T * scale
        if slopes is not None:
            s = s - slopes[h] * distance
        s = s.masked_fill(~seen, -math.inf)
        top = s.max(-1, keepdim=True).values
        if sinks is not None:
            top = torch.maximum(top, sinks[h])
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True)
        if sinks is not None:
            total = total + torch.exp(sinks[h] - top)
        out[:, h] = (e / total) @ v[:, h // group]
    return out


# ---- the mixers ------------------------------------------------------------------------------------------
def heads_of(z: torch.Tensor, heads: int) -> torch.Tensor:
    return z.view(z.shape[0], heads, -1)


def conv_attention(h, w, p, m, eps):
    """Convolved queries and keys, interleaved rotation, the unrotated keys as values, a sink of score 0."""
    q = heads_of(causal_conv(h @ w[p + "q"].T, w[p + "q.conv"]), m["heads"])
    k = heads_of(causal_conv(h @ w[p + "k"].T, w[p + "k.conv"]), m["kv_heads"])
    turn = lambda z: rotate(z, m["rot"]["dims"], m["rot"]["base"], True)
    o = attention(turn(q), turn(k), k, m["scale"], visible(h.shape[0], None, 0), torch.zeros(m["heads"], dtype=h.dtype))
    return o.flatten(1) @ w[p + "o"].T


def window_attention(h, w, p, m, eps):
    """Rotation, then a norm; a window beside kept first tokens; biases; a gate per value."""
    lin = lambda n: h @ w[p + n].T + w[p + n + ".b"]
    turn = lambda z: rms_norm(rotate(z, m["rot"]["dims"], m["rot"]["base"], False), None, eps)
    q, k, v = turn(heads_of(lin("q"), m["heads"])), turn(heads_of(lin("k"), m["kv_heads"])), heads_of(lin("v"), m["kv_heads"])
    o = attention(q, k, v, m["scale"], visible(h.shape[0], m["mask"]["size"], m["mask"]["keep_first"])).flatten(1)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T + w[p + "o.b"]


def distance_attention(h, w, p, m, eps, kv: dict, index: int):
    """No rotation; a bias by distance, a learned sink, a gate per head; perhaps with an earlier layer's keys and values."""
    lin = lambda n: h @ w[p + n].T + w[p + n + ".b"]
    if m.get("kv_from") is None:
        kv[index] = heads_of(lin("k"), m["kv_heads"]), heads_of(lin("v"), m["kv_heads"])
    k, v = kv[index if m.get("kv_from") is None else m["kv_from"]]
    slopes = [alibi_slope(j, m["heads"]) for j in range(m["heads"])]
    o = attention(heads_of(lin("q"), m["heads"]), k, v, m["scale"], visible(h.shape[0], None, 0), w[p + "sink"], slopes)
    return (o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]).flatten(1) @ w[p + "o"].T


# ---- the feed-forwards -------------------------------------------------------------------------------------
def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped(h, w, p, limit: float):
    g, u = torch.clamp(h @ w[p + "gate"].T, max=limit), torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def experts(h, w, p, m):
    """Each token's best experts by sigmoid score, the score on their input; a gated shared expert beside them."""
    scores, out = torch.sigmoid(h @ w[p + "router"].T), torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(scores[t], m["router"]["top"]).indices.tolist():
            out[t] += clamped(scores[t, e] * h[t:t + 1], w, f"{p}e{e}.", m["expert"]["limit"])[0]
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * clamped(h, w, p + "shared.", m["shared"]["limit"])
    return out


# ---- the model -------------------------------------------------------------------------------------------
class OracleSunulorn:
    def __init__(self, tensors: dict, config: dict, dtype=torch.float64):
        self.cfg = config
        self.w = {k: t.to(dtype) for k, t in tensors.items()}

    def mixer(self, i: int, h: torch.Tensor, kv: dict) -> torch.Tensor:
        spec, args = self.cfg["layers"][i], (h, self.w, f"l{i}.mix.", self.cfg["layers"][i]["mixer"], self.cfg["norm"]["eps"])
        if spec["type"] == "attention":
            return conv_attention(*args)
        if spec["type"] == "attention_2":
            return window_attention(*args)
        assert spec["type"] == "attention_3"
        return distance_attention(*args, kv, i)

    @torch.inference_mode()
    def forward(self, tokens: list[int], streams: list | None = None) -> torch.Tensor:
        """Logits of every position [T, vocab]; ``streams`` receives the residual stream after each layer."""
        cfg, w, eps, kv = self.cfg, self.w, self.cfg["norm"]["eps"], {}
        x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            y = self.mixer(i, rms_norm(x, w[p + "norm1"], eps), kv)
            if layer["mlp"] is not None:
                h = rms_norm(x, w[p + "norm2"], eps)
                y = y + (dense(h, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else experts(h, w, p + "mlp.", layer["mlp"]))
            x = x + y
            if streams is not None:
                streams.append(x)
        return rms_norm(x, w["final.norm"], eps) @ w["head"].T

    def greedy(self, prompt: list[int], n: int) -> tuple[list[int], list[float]]:
        """``n`` greedy tokens and, for each, the margin between the best and the second-best logit."""
        toks, out, margins = list(prompt), [], []
        for _ in range(n):
            top = torch.topk(self.forward(toks)[-1], 2)
            out.append(int(top.indices[0]))
            margins.append(float(top.values[0] - top.values[1]))
            toks.append(out[-1])
        return out, margins
