"""Sunulorn: three kinds of attention - over convolved keys that are their own values, in a window with kept first tokens, and with a bias
by distance (perhaps over an earlier layer's keys and values) - each beside a dense feed-forward or a mixture of experts."""
from __future__ import annotations

import torch

from ..hybrid import HybridDecoder, ParallelLayer
from ..layers.branches import AttentionBranch, PackedMixer, alibi_slopes
from ..layers.feedforward import ExpertFeed, GatedFeed
from ..layers.residual import ParallelStream
from ..layers.rotary import RotaryEmbedding

GLU_ALPHA, GLU_OFFSET = 1.702, 1.0          # the experts' unit: g sigmoid(alpha g) (u + offset)


class SunulornForCausalLM(HybridDecoder):
    def __init__(self, cfg):
        width, eps, tables, layers = cfg.hidden_size, cfg.rms_norm_eps, {}, []
        stream = ParallelStream(width, eps, cfg.embedding_scale)
        by_distance: dict[int, AttentionBranch] = {}

        def rotary(rot: dict, padded: int) -> RotaryEmbedding:
            key = (rot["dims"], float(rot["base"]), padded)
            if key not in tables:
                tables[key] = RotaryEmbedding(rot["dims"], cfg.max_position_embeddings, float(rot["base"]), head_dim=padded)
            return tables[key]

        def branch(i: int, kind: str, m: dict) -> AttentionBranch:
            d = AttentionBranch.padded_size(m["dim"], m["vdim"], cfg.dtype)
            sizes = (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"])
            if kind == "attention":
                return AttentionBranch(*sizes, rotary(m["rot"], d), m["rot"]["dims"], d, interleaved=True, taps=m["conv"],
                                       keys_are_values=True, sink="zero")
            if kind == "attention_2":
                return AttentionBranch(*sizes, rotary(m["rot"], d), m["rot"]["dims"], d, window=m["mask"]["size"],
                                       keep_first=m["mask"]["keep_first"], norm_eps=eps, in_bias=True, out_bias=True, gate="value")
            if kind != "attention_3":
                raise ValueError(f"unknown layer type {kind!r}")
            src = m.get("kv_from")
            if src is not None and (src not in by_distance or by_distance[src].borrows):
                raise ValueError(f"layer {i} takes its keys from layer {src}, which is no earlier layer of its kind with keys of its own")
            by_distance[i] = AttentionBranch(*sizes, None, 0, d, in_bias=True, sink="learned", slopes=alibi_slopes(m["heads"]),
                                             gate="head", source=None if src is None else by_distance[src])
            return by_distance[i]

        def feed(ff: dict | None):
            if ff is None:
                return None
            if ff.get("kind", "dense") == "dense":
                return GatedFeed(width, ff["ff"])
            if ff["kind"] != "moe":
                raise ValueError(f"unknown feed-forward kind {ff['kind']!r}")
            e, s = ff["expert"], ff.get("shared")
            shared = None if s is None else GatedFeed(width, s["ff"], s["limit"], GLU_ALPHA, GLU_OFFSET, token_gate=True)
            return ExpertFeed(width, e["ff"], ff["router"]["experts"], ff["router"]["top"], e["limit"], GLU_ALPHA, GLU_OFFSET, shared)

        for i, spec in enumerate(cfg.layers):
            layers.append(ParallelLayer(stream, PackedMixer(width, {"mixer": branch(i, spec["type"], spec["mixer"])}, feed(spec.get("mlp")))))
        super().__init__(cfg, layers, stream)

    def mixer_prefixes(self, index: int) -> dict[str, str]:
        return {"mixer": f"l{index}.mix."}

    def random_tensors(self, seed: int):
        cfg, dev = self.config, self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(seed)
        width = cfg.hidden_size
        randn = lambda *s, std=None: torch.randn(*s, generator=g, device=dev, dtype=torch.float32) * (s[-1] ** -0.5 if std is None else std)
        yield "embed", randn(cfg.vocab_size, width, std=1.0 / cfg.embedding_scale)
        yield "head", randn(cfg.vocab_size, width)
        yield "final.norm", torch.ones(width, device=dev)

        def unit(p: str, ff: int):
            yield p + "gate", randn(ff, width)
            yield p + "up", randn(ff, width)
            yield p + "down", randn(width, ff)

        for i, spec in enumerate(cfg.layers):
            p, m, ff, kind = f"l{i}.", spec["mixer"], spec.get("mlp"), spec["type"]
            yield p + "norm1", torch.ones(width, device=dev)
            if ff:
                yield p + "norm2", torch.ones(width, device=dev)
            if ff and ff.get("kind", "dense") == "dense":
                yield from unit(p + "mlp.", ff["ff"])
            elif ff:
                yield p + "mlp.router", randn(ff["router"]["experts"], width)
                for e in range(ff["router"]["experts"]):
                    yield from unit(f"{p}mlp.e{e}.", ff["expert"]["ff"])
                if ff.get("shared"):
                    yield from unit(p + "mlp.shared.", ff["shared"]["ff"])
                    yield p + "mlp.shared.sg", randn(1, width)
            p += "mix."
            heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            rows = {"q": heads * dim, "k": kv * dim, "v": kv * vdim}
            if kind == "attention":
                del rows["v"]
            elif m.get("kv_from") is not None:
                rows = {"q": heads * dim}
            for n, c in rows.items():
                yield p + n, randn(c, width)
                if kind == "attention":
                    yield f"{p}{n}.conv", randn(c, m["conv"])
                else:
                    yield f"{p}{n}.b", randn(c, std=0.1)
            yield p + "o", randn(width, heads * vdim)
            if kind == "attention_2":
                yield p + "o.b", randn(width, std=0.1)
                yield p + "g", randn(heads * vdim, width)
            elif kind == "attention_3":
                yield p + "g", randn(heads, width)
                yield p + "sink", randn(heads, std=1.0)
