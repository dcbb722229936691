"""The Vebonex decoder restated plainly: one whole sequence at a time, one function per mechanism, token loops where the
mathematics is a recurrence.  TEST INFRASTRUCTURE.

Everything runs on the CPU in the dtype of ``OracleVebonex`` (float64 unless a caller asks for float32), from the checkpoint's own
tensor names and the parsed ``config.json``.  Nothing here is shared with the product package: no paging, no padding, no packing,
no chunking, no absorbed projections.

Symbols: ``X`` are the residual streams [streams, tokens, width], ``h`` a normalised sublayer input, ``S`` a recurrent state.
"""
from __future__ import annotations

import math

import torch


# ---- elementary mechanisms -------------------------------------------------------------------------------
def rms_norm(x: torch.Tensor, w: torch.Tensor | None, eps: float, groups: int = 1) -> torch.Tensor:
    """Each of ``groups`` equal consecutive parts of the last axis over its own root mean square."""
    parts = x.unflatten(-1, (groups, -1))
    y = (parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)).flatten(-2)
    return y if w is None else y * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def poly_norm(z: torch.Tensor, act: torch.Tensor, eps: float) -> torch.Tensor:
    """act = (a, b, c, e): a N(z) + b N(z^2) + c N(z^3) + e, N over the last axis."""
    return sum(act[i] * rms_norm(z ** (i + 1), None, eps) for i in range(3)) + act[3]


def connect_in(X: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """The sublayer's input: a weighted sum of the streams."""
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + w_in[s] * X[s]
    return u


def connect_out(X: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, w_out: torch.Tensor) -> torch.Tensor:
    """Stream t becomes a sum of the old streams weighted by mix[from, t], plus out[t] times the sublayer's output."""
    new = []
    for t in range(X.shape[0]):
        x = w_out[t] * y
        for s in range(X.shape[0]):
            x = x + mix[s, t] * X[s]
        new.append(x)
    return torch.stack(new)


def gated_linear(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, alpha: torch.Tensor, s: torch.Tensor | None = None):
    """One head: q, k, alpha [T, d] (alpha: decay factor of a key channel), v [T, dv] -> (o [T, dv], S [d, dv])."""
    s = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if s is None else s.clone()
    o = torch.empty_like(v)
    for t in range(q.shape[0]):
        s = alpha[t][:, None] * s + k[t][:, None] * v[t][None, :]
        o[t] = s.T @ q[t]
    return o, s


def mlstm_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor, state=None):
    """One head: q, k [T, d], v [T, dv], log gates i, f [T] -> (o [T, dv], (S, n, m)); m is the running maximum of the exponents."""
    if state is None:
        state = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype), torch.zeros(q.shape[1], dtype=q.dtype), torch.zeros((), dtype=q.dtype)
    s, n, m = (x.clone() for x in state)
    o = torch.empty_like(v)
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        s, n, m = keep * s + take * k[t][:, None] * v[t][None, :], keep * n + take * k[t], new
        o[t] = s.T @ q[t] / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return o, (s, n, m)


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv] -> [T, H, dv]; causal, ordinary softmax."""
    t = q.shape[0]
    seen = torch.arange(t)[:, None] >= torch.arange(t)[None, :]
    out = torch.empty(t, q.shape[1], v.shape[2], dtype=q.dtype)
    for h in range(q.shape[1]):
        s = (q[:, h] @ k[:, h].T * scale).masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, h]
    return out


# ---- the mixers ------------------------------------------------------------------------------------------
def gla_mixer(h, w, p, m, eps):
    t, heads, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(t, heads, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).view(t, heads, d), (h @ w[p + "v"].T).view(t, heads, dv)
    z = (h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "a2.b"].reshape(-1)).view(t, heads, d)
    alpha = torch.exp(log_sigmoid(z) / m["tau"])
    o = torch.stack([gated_linear(q[:, j], k[:, j], v[:, j], alpha[:, j])[0] for j in range(heads)], dim=1)
    return (rms_norm(o, w[p + "norm"], eps).reshape(t, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mlstm_mixer(h, w, p, m, eps):
    t, heads, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(t, heads, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).view(t, heads, d), (h @ w[p + "v"].T).view(t, heads, dv)
    i = soft_cap(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w[p + "f"].T + w[p + "f.b"], cap))
    o = torch.stack([mlstm_memory(q[:, j], k[:, j], v[:, j], i[:, j], f[:, j])[0] for j in range(heads)], dim=1)
    return (rms_norm(o, None, eps).reshape(t, -1) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def latent_mixer(h, w, p, m, eps, latent):
    """``latent`` [T, kv_rank]: the mixer's own, or that of the layer it borrows from."""
    t, heads = h.shape[0], m["heads"]
    cq = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).view(t, heads, m["dim"])
    k, v = (latent @ w[p + "uk"].T).view(t, heads, m["dim"]), (latent @ w[p + "uv"].T).view(t, heads, m["vdim"])
    o = attention(q, k, v, m["scale"]).reshape(t, -1)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- the model -------------------------------------------------------------------------------------------
class OracleVebonex:
    def __init__(self, tensors: dict, config: dict, dtype=torch.float64):
        self.cfg = config
        self.w = {k: t.to(dtype) for k, t in tensors.items()}

    def mixer(self, i: int, h: torch.Tensor, latents: dict) -> torch.Tensor:
        spec, w, eps, p = self.cfg["layers"][i], self.w, self.cfg["norm"]["eps"], f"l{i}.mix."
        m = spec["mixer"]
        if spec["type"] == "gla":
            return gla_mixer(h, w, p, m, eps)
        if spec["type"] == "mlstm":
            return mlstm_mixer(h, w, p, m, eps)
        src = m.get("kv_from")
        if src is None:
            src, latents[i] = i, rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
        return latent_mixer(h, w, p, m, eps, latents[src])

    @torch.inference_mode()
    def forward(self, tokens: list[int], streams: list | None = None) -> torch.Tensor:
        """Logits of every position [T, vocab]; ``streams`` receives the sum of the residual streams after each layer."""
        cfg, w, latents = self.cfg, self.w, {}
        eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
        x = w["embed"][torch.tensor(tokens)] + w["pos"][:len(tokens)]
        X = torch.stack([x] * cfg["streams"])
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            y = self.mixer(i, rms_norm(connect_in(X, w[p + "hc1.in"]), w[p + "norm1"], eps, groups), latents)
            X = connect_out(X, y, w[p + "hc1.mix"], w[p + "hc1.out"])
            if layer["mlp"] is not None:
                h = rms_norm(connect_in(X, w[p + "hc2.in"]), w[p + "norm2"], eps, groups)
                y = poly_norm(h @ w[p + "mlp.up"].T, w[p + "mlp.act"], eps) @ w[p + "mlp.down"].T
                X = connect_out(X, y, w[p + "hc2.mix"], w[p + "hc2.out"])
            if streams is not None:
                streams.append(X.sum(0))
        return rms_norm(X.sum(0), w["final.norm"], eps, groups) @ w["head"].T

    def greedy(self, prompt: list[int], n: int) -> tuple[list[int], list[float]]:
        """``n`` greedy tokens and, for each, the margin between the best and the second-best logit."""
        toks, out, margins = list(prompt), [], []
        for _ in range(n):
            top = torch.topk(self.forward(toks)[-1], 2)
            out.append(int(top.indices[0]))
            margins.append(float(top.values[0] - top.values[1]))
            toks.append(out[-1])
        return out, margins
