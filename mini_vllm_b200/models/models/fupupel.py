"""Fupupel: layers of Mamba selective scan, and layers with windowed, score-capped attention beside a gated delta rule;
a clamped gated feed-forward on some layers, norms around every sublayer, capped logits."""
from __future__ import annotations

import torch

from ..hybrid import ClampedGLU, HybridDecoder, HybridLayer
from ..layers.branches import AttentionBranch, GatedDeltaBranch, PackedMixer, SelectiveScanBranch
from ..layers.residual import SandwichStream
from ..layers.rotary import RotaryEmbedding

GLU_ALPHA = 1.702


class FupupelForCausalLM(HybridDecoder):
    def __init__(self, cfg):
        width, tables, layers = cfg.hidden_size, {}, []
        stream = SandwichStream(width, cfg.rms_norm_eps)

        def rotary(dims: int, base: float, padded: int) -> RotaryEmbedding:
            key = (dims, float(base), padded)
            if key not in tables:
                tables[key] = RotaryEmbedding(dims, cfg.max_position_embeddings, float(base), head_dim=padded)
            return tables[key]

        def attention(m: dict, factor: float) -> AttentionBranch:
            d = AttentionBranch.padded_size(m["dim"], m["vdim"], cfg.dtype)
            rot, mask = m.get("rot") or {"dims": 0, "base": 1.0}, m.get("mask") or {}
            return AttentionBranch(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"],
                                   rotary(rot["dims"], rot["base"], d), rot["dims"], d, window=mask.get("size"),
                                   softcap=m.get("softcap"), factor=factor)

        for spec in cfg.layers:
            m = spec["mixer"]
            if spec["type"] == "mamba1":
                branches = {"scan": SelectiveScanBranch(m["inner"], m["state"], m["dt_rank"], m["conv"])}
            elif spec["type"] == "parallel":
                r = m["right"]
                branches = {"left": attention(m["left"], m["left_scale"]),
                            "right": GatedDeltaBranch(r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"],
                                                      r["decay_rank"], r["gate_rank"], cfg.rms_norm_eps, m["right_scale"])}
            else:
                raise ValueError(f"unknown layer type {spec['type']!r}")
            ff = spec.get("mlp")
            if ff is not None and ff.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {ff['kind']!r}")
            mlp = None if ff is None else ClampedGLU(width, ff["ff"], ff["limit"], GLU_ALPHA)
            layers.append(HybridLayer(stream, PackedMixer(width, branches), mlp))
        super().__init__(cfg, layers, stream)

    def mixer_prefixes(self, index: int) -> dict[str, str]:
        p = f"l{index}.mix."
        return {"scan": p} if self.config.layers[index]["type"] == "mamba1" else {"left": p + "left.", "right": p + "right."}

    def random_tensors(self, seed: int):
        cfg, dev = self.config, self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(seed)
        width = cfg.hidden_size
        randn = lambda *s, std=None: torch.randn(*s, generator=g, device=dev, dtype=torch.float32) * (s[-1] ** -0.5 if std is None else std)
        uniform = lambda lo, hi, *s: torch.rand(*s, generator=g, device=dev, dtype=torch.float32) * (hi - lo) + lo
        inv_softplus = lambda y: torch.log(torch.expm1(y))
        yield "embed", randn(cfg.vocab_size, width, std=1.0)
        yield "head", randn(cfg.vocab_size, width)
        yield "final.norm", torch.ones(width, device=dev)
        for i, spec in enumerate(cfg.layers):
            p, m = f"l{i}.", spec["mixer"]
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if spec.get("mlp") else ()):
                yield p + n, torch.ones(width, device=dev)
            if spec.get("mlp"):
                ff = spec["mlp"]["ff"]
                yield p + "mlp.gate", randn(ff, width)
                yield p + "mlp.up", randn(ff, width)
                yield p + "mlp.down", randn(width, ff)
            p += "mix."
            if spec["type"] == "mamba1":
                inner, n, rank = m["inner"], m["state"], m["dt_rank"]
                yield p + "in", randn(2 * inner, width)
                yield p + "conv", randn(inner, m["conv"])
                yield p + "conv.b", randn(inner, std=0.1)
                yield p + "x", randn(rank + 2 * n, inner)
                yield p + "dt", randn(inner, rank)
                yield p + "dt.b", inv_softplus(uniform(0.001, 0.1, inner))
                yield p + "A_log", torch.log(torch.arange(1, n + 1, device=dev, dtype=torch.float32)).expand(inner, n)
                yield p + "D", torch.ones(inner, device=dev)
                yield p + "o", randn(width, inner)
                continue
            a, r = m["left"], m["right"]
            yield p + "left.q", randn(a["heads"] * a["dim"], width)
            yield p + "left.k", randn(a["kv_heads"] * a["dim"], width)
            yield p + "left.v", randn(a["kv_heads"] * a["vdim"], width)
            yield p + "left.o", randn(width, a["heads"] * a["vdim"])
            p += "right."
            for n, c in (("q", r["kv_heads"] * r["dim"]), ("k", r["kv_heads"] * r["dim"]), ("v", r["heads"] * r["vdim"])):
                yield p + n, randn(c, width)
                yield p + n + ".conv", randn(c, r["conv"])
            yield p + "b", randn(r["heads"], width)
            yield p + "A_log", torch.log(uniform(1.0, 16.0, r["heads"]))
            yield p + "dt_bias", inv_softplus(uniform(0.001, 0.1, r["heads"] * r["dim"]))
            yield p + "norm", torch.ones(r["vdim"], device=dev)
            yield p + "a1", randn(r["decay_rank"], width)
            yield p + "a2", randn(r["heads"] * r["dim"], r["decay_rank"])
            yield p + "g1", randn(r["gate_rank"], width)
            yield p + "g2", randn(r["heads"] * r["vdim"], r["gate_rank"])
            yield p + "o", randn(width, r["heads"] * r["vdim"])
