"""Rasezen: Mamba-2 state-space layers and windowed attention with whole-row query and key norms and normalised values, each beside an
xIELU feed-forward or a mixture of experts with identity experts, on one norm of a single number."""
from __future__ import annotations

import torch

from ..hybrid import HybridDecoder, ParallelLayer
from ..layers.branches import AttentionBranch, Branch, PackedMixer, StateSpaceBranch
from ..layers.feedforward import ExpertFeed, GatedFeed, XieluFeed
from ..layers.residual import ParallelStream
from ..layers.rotary import RotaryEmbedding


class RasezenForCausalLM(HybridDecoder):
    def __init__(self, cfg):
        width, eps, tables, layers = cfg.hidden_size, cfg.rms_norm_eps, {}, []
        stream = ParallelStream(width, eps, shared_norm=True)

        def rotary(rot: dict, padded: int) -> RotaryEmbedding:
            key = (rot["dims"], float(rot["base"]), padded)
            if key not in tables:
                tables[key] = RotaryEmbedding(rot["dims"], cfg.max_position_embeddings, float(rot["base"]), head_dim=padded)
            return tables[key]

        def branch(kind: str, m: dict) -> Branch:
            if kind == "mamba2":
                return StateSpaceBranch(m["heads"], m["groups"], m["state"], m["vdim"], m["conv"], m["norm_groups"], eps)
            if kind != "attention":
                raise ValueError(f"unknown layer type {kind!r}")
            d = AttentionBranch.padded_size(m["dim"], m["vdim"], cfg.dtype)
            return AttentionBranch(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], rotary(m["rot"], d), m["rot"]["dims"], d,
                                   window=m["mask"]["size"], in_bias=True, row_norm_eps=eps, value_norm_eps=eps)

        def feed(ff: dict | None):
            if ff is None:
                return None
            if ff.get("kind", "dense") == "dense":
                return XieluFeed(width, ff["ff"])
            if ff["kind"] != "moe":
                raise ValueError(f"unknown feed-forward kind {ff['kind']!r}")
            r, s = ff["router"], ff.get("shared")
            return ExpertFeed(width, ff["expert"]["ff"], r["experts"], r["top"], shared=None if s is None else GatedFeed(width, s["ff"]),
                              softmax=True, corrected=True, scale=r["scale"], weigh_output=True, identity=r.get("identity", 0))

        for spec in cfg.layers:
            mixer = PackedMixer(width, {"mixer": branch(spec["type"], spec["mixer"])}, feed(spec.get("mlp")))
            layers.append(ParallelLayer(stream, mixer))
        super().__init__(cfg, layers, stream)

    def mixer_prefixes(self, index: int) -> dict[str, str]:
        return {"mixer": f"l{index}.mix."}

    def random_tensors(self, seed: int):
        cfg, dev = self.config, self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(seed)
        width = cfg.hidden_size
        randn = lambda *s, std=None: torch.randn(*s, generator=g, device=dev, dtype=torch.float32) * (s[-1] ** -0.5 if std is None else std)
        uniform = lambda lo, hi, *s: torch.rand(*s, generator=g, device=dev, dtype=torch.float32) * (hi - lo) + lo
        one = torch.ones((), device=dev)
        yield "embed", randn(cfg.vocab_size, width, std=1.0)
        yield "head", randn(cfg.vocab_size, width)
        yield "final.norm", one

        def unit(p: str, ff: int):
            yield p + "gate", randn(ff, width)
            yield p + "up", randn(ff, width)
            yield p + "down", randn(width, ff)

        for i, spec in enumerate(cfg.layers):
            p, m, ff = f"l{i}.", spec["mixer"], spec.get("mlp")
            yield p + "norm1", one
            if ff and ff.get("kind", "dense") == "dense":
                yield p + "mlp.up", randn(ff["ff"], width)
                yield p + "mlp.down", randn(width, ff["ff"])
                yield p + "mlp.act", torch.zeros(2, device=dev)
            elif ff:
                outputs = ff["router"]["experts"] + ff["router"].get("identity", 0)
                yield p + "mlp.router", randn(outputs, width)
                yield p + "mlp.correction", torch.zeros(outputs, device=dev)
                for e in range(ff["router"]["experts"]):
                    yield from unit(f"{p}mlp.e{e}.", ff["expert"]["ff"])
                if ff.get("shared"):
                    yield from unit(p + "mlp.shared.", ff["shared"]["ff"])
            p += "mix."
            heads, vdim = m["heads"], m["vdim"]
            yield p + "o", randn(width, heads * vdim)
            if spec["type"] == "mamba2":
                channels = heads * vdim + 2 * m["groups"] * m["state"]
                yield p + "in", randn(heads * vdim + channels + heads, width)
                yield p + "conv", randn(channels, m["conv"])
                yield p + "conv.b", randn(channels, std=0.1)
                yield p + "dt_bias", torch.log(torch.expm1(uniform(0.001, 0.1, heads)))
                yield p + "A_log", torch.log(uniform(1.0, 16.0, heads))
                yield p + "D", torch.ones(heads, device=dev)
                yield p + "norm", torch.ones(heads * vdim, device=dev)
                continue
            for n, c in (("q", heads * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * vdim)):
                yield p + n, randn(c, width)
                yield f"{p}{n}.b", randn(c, std=0.1)
                if n != "v":
                    yield f"{p}{n}.norm", torch.ones(c, device=dev)
