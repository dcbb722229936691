"""Vebonex: layers of matrix-memory LSTM, gated linear attention and latent attention (which may share an earlier layer's latents), a
polynomial-norm feed-forward, several hyper-connected residual streams, learned positions."""
from __future__ import annotations

import torch

from ..hybrid import HybridDecoder, HybridLayer, PolyNormMLP
from ..layers.branches import GatedLinearBranch, LatentAttentionBranch, MatrixLSTMBranch, PackedMixer
from ..layers.residual import HyperStream


class VebonexForCausalLM(HybridDecoder):
    def __init__(self, cfg):
        width, eps, layers = cfg.hidden_size, cfg.rms_norm_eps, []
        stream = HyperStream(width, eps, cfg.streams, cfg.norm_groups, cfg.max_position_embeddings)
        latent: dict[int, LatentAttentionBranch] = {}

        def branch(i: int, kind: str, m: dict):
            if kind == "mlstm":
                return MatrixLSTMBranch(m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps)
            if kind == "gla":
                return GatedLinearBranch(m["heads"], m["dim"], m["vdim"], m["tau"], m["decay_rank"], eps)
            if kind != "latent_attention":
                raise ValueError(f"unknown layer type {kind!r}")
            src = m.get("kv_from")
            if src is not None and (src not in latent or latent[src].source is not None):
                raise ValueError(f"layer {i} takes its latents from layer {src}, which is no earlier layer with latents of its own")
            latent[i] = LatentAttentionBranch(m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], eps, cfg.dtype,
                                              None if src is None else latent[src])
            return latent[i]

        for i, spec in enumerate(cfg.layers):
            ff = spec.get("mlp")
            if ff is not None and ff.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {ff['kind']!r}")
            mixer = PackedMixer(width, {"mixer": branch(i, spec["type"], spec["mixer"])})
            layers.append(HybridLayer(stream, mixer, None if ff is None else PolyNormMLP(width, ff["ff"], eps)))
        super().__init__(cfg, layers, stream)

    def mixer_prefixes(self, index: int) -> dict[str, str]:
        return {"mixer": f"l{index}.mix."}

    def random_tensors(self, seed: int):
        cfg, dev = self.config, self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(seed)
        width, streams = cfg.hidden_size, cfg.streams
        randn = lambda *s, std=None: torch.randn(*s, generator=g, device=dev, dtype=torch.float32) * (s[-1] ** -0.5 if std is None else std)
        ones = lambda *s: torch.ones(*s, device=dev)
        yield "embed", randn(cfg.vocab_size, width, std=1.0)
        yield "pos", randn(cfg.max_position_embeddings, width, std=0.3)
        yield "head", randn(cfg.vocab_size, width)
        yield "final.norm", ones(width)
        for i, spec in enumerate(cfg.layers):
            p, m = f"l{i}.", spec["mixer"]
            for q in (1, 2) if spec.get("mlp") else (1,):
                yield f"{p}norm{q}", ones(width)
                yield f"{p}hc{q}.in", ones(streams) / streams + randn(streams, std=0.1)
                yield f"{p}hc{q}.out", ones(streams) + randn(streams, std=0.1)
                yield f"{p}hc{q}.mix", torch.eye(streams, device=dev) + randn(streams, streams, std=0.1)
            if spec.get("mlp"):
                ff = spec["mlp"]["ff"]
                yield p + "mlp.up", randn(ff, width)
                yield p + "mlp.down", randn(width, ff)
                yield p + "mlp.act", torch.tensor([0.5, 0.4, 0.3, 0.0], device=dev)
            p += "mix."
            heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
            yield p + "g", randn(heads * vdim, width)
            yield p + "o", randn(width, heads * vdim)
            if spec["type"] == "latent_attention":
                yield p + "dq", randn(m["q_rank"], width)
                yield p + "dq.norm", ones(m["q_rank"])
                yield p + "uq", randn(heads * dim, m["q_rank"])
                if m.get("kv_from") is None:
                    yield p + "dkv", randn(m["kv_rank"], width)
                    yield p + "dkv.norm", ones(m["kv_rank"])
                yield p + "uk", randn(heads * dim, m["kv_rank"])
                yield p + "uv", randn(heads * vdim, m["kv_rank"])
                continue
            yield p + "q", randn(heads * dim, width)
            yield p + "k", randn(heads * dim, width)
            yield p + "v", randn(heads * vdim, width)
            if spec["type"] == "mlstm":
                yield p + "norm", ones(heads * vdim)
                for n, bias in (("i", 0.0), ("f", 4.0)):
                    yield p + n, randn(heads, width)
                    yield f"{p}{n}.b", ones(heads) * bias
            else:
                yield p + "norm", ones(vdim)
                yield p + "a1", randn(m["decay_rank"], width)
                yield p + "a2", randn(heads * dim, m["decay_rank"])
                yield p + "a2.b", ones(heads * dim) * 2.0
