"""The Fupupel decoder restated plainly: one whole sequence at a time, one function per mechanism, token loops where
the mathematics is a recurrence.  TEST INFRASTRUCTURE.

Everything runs on the CPU in the dtype of ``f`` (float64 unless a caller asks for float32), from the checkpoint's own
tensor names and the parsed ``config.json``.  Nothing here is shared with the product package: no paging, no padding,
no packing, no chunking.

Symbols: ``x`` is the residual stream [tokens, width], ``h`` a normalised sublayer input, ``S`` a recurrent state.
"""
from __future__ import annotations

import math

import torch


# ---- elementary mechanisms -------------------------------------------------------------------------------
def rms_norm(x: torch.Tensor, w: torch.Tensor | None, eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def soft_cap(z: torch.Tensor, cap: float | None) -> torch.Tensor:
    return z if not cap else cap * torch.tanh(z / cap)


def causal_conv(u: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None) -> torch.Tensor:
    """u [T, C], w [C, taps]: out[t, c] = bias[c] + sum_j w[c, taps-1-j] u[t-j, c], zeros before the start."""
    taps, out = w.shape[1], torch.zeros_like(u)
    for j in range(min(taps, u.shape[0])):
        out[j:] += w[:, taps - 1 - j] * u[:u.shape[0] - j]
    return out if bias is None else out + bias


def rotate(u: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """u [T, heads, d]: coordinates i and i + dims/2 of the token at position p turn by p * base^(-2i/dims)."""
    half = dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    a = (torch.arange(u.shape[0], dtype=torch.float64)[:, None] * f)[:, None, :]
    c, s = a.cos().to(u.dtype), a.sin().to(u.dtype)
    lo, hi = u[..., :half], u[..., half:dims]
    return torch.cat([lo * c - hi * s, hi * c + lo * s, u[..., dims:]], dim=-1)


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: float | None,
              window: int | None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; a query sees itself and the window - 1 tokens before it."""
    t, heads = q.shape[:2]
    per = heads // k.shape[1]
    i = torch.arange(t)
    dist = i[:, None] - i[None, :]
    seen = dist >= 0
    if window is not None:
        seen &= dist < window
    out = torch.empty(t, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        s = soft_cap(q[:, h] @ k[:, h // per].T * scale, cap).masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, h // per]
    return out


def selective_scan(u: torch.Tensor, dt: torch.Tensor, a: torch.Tensor, b: torch.Tensor, c: torch.Tensor, d: torch.Tensor,
                   s: torch.Tensor | None = None):
    """u, dt [T, inner]; a [inner, N] (negative); b, c [T, N]; d [inner] -> (y [T, inner], final state [inner, N])."""
    s = torch.zeros_like(a) if s is None else s.clone()
    y = torch.empty_like(u)
    for t in range(u.shape[0]):
        s = torch.exp(dt[t][:, None] * a) * s + (dt[t] * u[t])[:, None] * b[t][None, :]
        y[t] = s @ c[t] + d * u[t]
    return y, s


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
               s: torch.Tensor | None = None):
    """One head: q, k, g [T, d] (g is the decay factor of a key channel), v [T, dv], beta [T] -> (o [T, dv], S [d, dv])."""
    s = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if s is None else s.clone()
    o = torch.empty_like(v)
    for t in range(q.shape[0]):
        s = g[t][:, None] * s
        u = beta[t] * (v[t] - s.T @ k[t])
        s = s + k[t][:, None] * u[None, :]
        o[t] = s.T @ q[t]
    return o, s


def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


# ---- the mixers ------------------------------------------------------------------------------------------
def mamba_mixer(h, w, p, m):
    inner, rank, n = m["inner"], m["dt_rank"], m["state"]
    u, z = (h @ w[p + "in"].T).split([inner, inner], dim=-1)
    u = silu(causal_conv(u, w[p + "conv"], w[p + "conv.b"]))
    dt, b, c = (u @ w[p + "x"].T).split([rank, n, n], dim=-1)
    dt = softplus(dt @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_scan(u, dt, -torch.exp(w[p + "A_log"]), b, c, w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


def attention_mixer(h, w, p, m):
    t = h.shape[0]
    q = (h @ w[p + "q"].T).view(t, m["heads"], m["dim"])
    k = (h @ w[p + "k"].T).view(t, m["kv_heads"], m["dim"])
    v = (h @ w[p + "v"].T).view(t, m["kv_heads"], m["vdim"])
    if m.get("rot"):
        q, k = (rotate(a, m["rot"]["dims"], m["rot"]["base"]) for a in (q, k))
    mask = m.get("mask") or {}
    return attention(q, k, v, m["scale"], m.get("softcap"), mask.get("size")).reshape(t, -1) @ w[p + "o"].T


def delta_mixer(h, w, p, m, eps):
    t, heads, kv, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"], None)) for n in "qkv")
    q, k, v = q.view(t, kv, d), k.view(t, kv, d), v.view(t, heads, dv)
    unit = lambda a: a / torch.sqrt((a * a).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    pre = (h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "dt_bias"].reshape(-1)).view(t, heads, d)
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * softplus(pre))
    o = torch.stack([delta_rule(q[:, i // (heads // kv)], k[:, i // (heads // kv)], v[:, i], g[:, i], beta[:, i])[0]
                     for i in range(heads)], dim=1)
    gate = torch.sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T).view(t, heads, dv)
    return (rms_norm(o, w[p + "norm"], eps) * gate).reshape(t, -1) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    return (m["left_scale"] * attention_mixer(h, w, p + "left.", m["left"]) +
            m["right_scale"] * delta_mixer(h, w, p + "right.", m["right"], eps))


# ---- the model -------------------------------------------------------------------------------------------
class OracleFupupel:
    def __init__(self, tensors: dict, config: dict, dtype=torch.float64):
        self.cfg = config
        self.w = {k: t.to(dtype) for k, t in tensors.items()}

    @torch.inference_mode()
    def forward(self, tokens: list[int], streams: list | None = None) -> torch.Tensor:
        """Logits of every position [T, vocab]; ``streams`` receives the residual stream after each layer."""
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = w["embed"][torch.tensor(tokens)]
        for i, layer in enumerate(cfg["layers"]):
            p, m = f"l{i}.", layer["mixer"]
            h = rms_norm(x, w[p + "norm1"], eps)
            y = mamba_mixer(h, w, p + "mix.", m) if layer["type"] == "mamba1" else parallel_mixer(h, w, p + "mix.", m, eps)
            x = x + rms_norm(y, w[p + "norm1b"], eps)
            if layer["mlp"] is not None:
                h = rms_norm(x, w[p + "norm2"], eps)
                y = clamped_glu(h @ w[p + "mlp.gate"].T, h @ w[p + "mlp.up"].T, layer["mlp"]["limit"]) @ w[p + "mlp.down"].T
                x = x + rms_norm(y, w[p + "norm2b"], eps)
            if streams is not None:
                streams.append(x)
        return soft_cap(rms_norm(x, w["final.norm"], eps) @ w["head"].T, cfg.get("logit_softcap"))

    def greedy(self, prompt: list[int], n: int) -> tuple[list[int], list[float]]:
        """``n`` greedy tokens and, for each, the margin between the best and the second-best logit."""
        toks, out, margins = list(prompt), [], []
        for _ in range(n):
            top = torch.topk(self.forward(toks)[-1], 2)
            out.append(int(top.indices[0]))
            margins.append(float(top.values[0] - top.values[1]))
            toks.append(out[-1])
        return out, margins
