"""The Rasezen decoder restated plainly: one whole sequence at a time, one function per mechanism.  TEST INFRASTRUCTURE.

Everything runs on the CPU in the dtype of ``OracleRasezen`` (float64 unless a caller asks for float32), from the checkpoint's own
tensor names and the parsed ``config.json``.  Nothing here is shared with the product package: no paging, no padding, no packing, no
chunks, no sorting of tokens by expert.

Symbols: ``x`` is the residual stream [T, width], ``h`` a normalised input, ``q``, ``k``, ``v`` are [T, heads, size], ``S`` a head's state
[N, vdim].
"""
from __future__ import annotations

import math

import torch


# ---- elementary mechanisms -------------------------------------------------------------------------------
def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over the root mean square of its last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x: torch.Tensor, g: torch.Tensor, eps: float) -> torch.Tensor:
    """One number scales every coordinate."""
    assert g.numel() == 1
    return over_rms(x, eps) * g


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def xielu(z: torch.Tensor, p: torch.Tensor, q: torch.Tensor) -> torch.Tensor:
    below = torch.clamp(z, max=0)
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(below) - below)) + z / 2


def causal_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, channels], w [channels, taps]; the last tap weighs the token itself, zeros before the start."""
    taps, rows = w.shape[1], []
    for t in range(u.shape[0]):
        y = b
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y = y + w[:, j] * u[src]
        rows.append(y)
    return torch.stack(rows)


def rotate_half(z: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """z [T, heads, d]: coordinates i and i + dims/2 of the first ``dims`` turn by position times base^(-2i/dims)."""
    out = z.clone()
    for i in range(dims // 2):
        angle = torch.arange(z.shape[0], dtype=z.dtype)[:, None] * base ** (-2.0 * i / dims)
        u, v = z[..., i], z[..., i + dims // 2]
        out[..., i] = u * angle.cos() - v * angle.sin()
        out[..., i + dims // 2] = v * angle.cos() + u * angle.sin()
    return out


def in_window(t: int, size: int) -> torch.Tensor:
    """[T, T] of booleans: a query (row) sees itself and the ``size - 1`` keys (columns) before it."""
    back = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return (back >= 0) & (back < size)


def attention(q, k, v, scale: float, seen: torch.Tensor) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]"""
    heads, group = q.shape[1], q.shape[1] // k.shape[1]
    out = torch.empty(q.shape[0], heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        s = (q[:, h] @ k[:, h // group].T * scale).masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, h // group]
    return out


def state_space(x, b, c, dt, a, d) -> torch.Tensor:
    """x [T, heads, vdim], b and c [T, groups, N], dt [T, heads] (positive), a and d [heads] (a negative) -> [T, heads, vdim]:
    S <- e^{a dt} S + dt b x^T, y = S^T c + d x, token by token."""
    group_of = torch.arange(x.shape[1]) // (x.shape[1] // b.shape[1])
    S, y = torch.zeros(x.shape[1], b.shape[2], x.shape[2], dtype=x.dtype), torch.empty_like(x)
    for t in range(x.shape[0]):
        key, query = b[t, group_of], c[t, group_of]                  # [heads, N]
        S = torch.exp(a * dt[t])[:, None, None] * S + dt[t, :, None, None] * key[:, :, None] * x[t, :, None, :]
        y[t] = (query[:, :, None] * S).sum(1) + d[:, None] * x[t]
    return y


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """The gate first, then a norm over each of ``groups`` equal parts of the row, then a weight per coordinate."""
    y = y * silu(z)
    return over_rms(y.view(y.shape[0], groups, -1), eps).flatten(1) * w


# ---- the mixers ------------------------------------------------------------------------------------------
def mamba2(h, w, p, m, eps):
    heads, vdim, n, groups = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = heads * vdim
    z, xbc, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * groups * n, heads], dim=1)
    x, b, c = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])).split([inner, groups * n, groups * n], dim=1)
    t = h.shape[0]
    y = state_space(x.reshape(t, heads, vdim), b.reshape(t, groups, n), c.reshape(t, groups, n), softplus(dt + w[p + "dt_bias"]),
                    -torch.exp(w[p + "A_log"]), w[p + "D"])
    return gated_group_norm(y.flatten(1), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


def window_attention(h, w, p, m, eps):
    """Biases; q and k normalised as whole rows, then rotated; values over their root mean square; a window."""
    lin = lambda n: h @ w[p + n].T + w[p + n + ".b"]
    t, rot = h.shape[0], m["rot"]
    q = (over_rms(lin("q"), eps) * w[p + "q.norm"]).view(t, m["heads"], m["dim"])
    k = (over_rms(lin("k"), eps) * w[p + "k.norm"]).view(t, m["kv_heads"], m["dim"])
    v = over_rms(lin("v").view(t, m["kv_heads"], m["vdim"]), eps)
    turn = lambda u: rotate_half(u, rot["dims"], rot["base"])
    return attention(turn(q), turn(k), v, m["scale"], in_window(t, m["mask"]["size"])).flatten(1) @ w[p + "o"].T


# ---- the feed-forwards -------------------------------------------------------------------------------------
def dense(h, w, p):
    return xielu(h @ w[p + "up"].T, w[p + "act"][0], w[p + "act"][1]) @ w[p + "down"].T


def gated(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(z: torch.Tensor, correction: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Of logits [E]: the chosen outputs by corrected score, and their uncorrected softmax scores."""
    s = torch.softmax(z, -1)
    ids = torch.topk(s + correction, top).indices
    return ids, s[ids]


def experts(h, w, p, m):
    r, out = m["router"], torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, s = choose(w[p + "router"] @ h[t], w[p + "correction"], r["top"])
        for e, weight in zip(ids.tolist(), s):
            y = gated(h[t:t + 1], w, f"{p}e{e}.")[0] if e < r["experts"] else h[t]
            out[t] += weight * r["scale"] * y
    return out + gated(h, w, p + "shared.") if m.get("shared") else out


# ---- the model -------------------------------------------------------------------------------------------
class OracleRasezen:
    def __init__(self, tensors: dict, config: dict, dtype=torch.float64):
        self.cfg = config
        self.w = {k: t.to(dtype) for k, t in tensors.items()}

    @torch.inference_mode()
    def forward(self, tokens: list[int], streams: list | None = None) -> torch.Tensor:
        """Logits of every position [T, vocab]; ``streams`` receives the residual stream after each layer."""
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = w["embed"][torch.tensor(tokens)]
        for i, layer in enumerate(cfg["layers"]):
            p, ff = f"l{i}.", layer["mlp"]
            h = scalar_norm(x, w[p + "norm1"], eps)
            y = {"mamba2": mamba2, "attention": window_attention}[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
            if ff is not None:
                y = y + (dense(h, w, p + "mlp.") if ff["kind"] == "dense" else experts(h, w, p + "mlp.", ff))
            x = x + y
            if streams is not None:
                streams.append(x)
        return scalar_norm(x, w["final.norm"], eps) @ w["head"].T

    def greedy(self, prompt: list[int], n: int) -> tuple[list[int], list[float]]:
        """``n`` greedy tokens and, for each, the margin between the best and the second-best logit."""
        toks, out, margins = list(prompt), [], []
        for _ in range(n):
            top = torch.topk(self.forward(toks)[-1], 2)
            out.append(int(top.indices[0]))
            margins.append(float(top.values[0] - top.values[1]))
            toks.append(out[-1])
        return out, margins
