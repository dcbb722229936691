"""Small Vebonex models with weights of the tests' own making (nothing here comes from the package's initialiser)."""
from __future__ import annotations

import copy

import torch


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def lstm_layer(heads=3, dim=24, vdim=40, cap=7.0, ff=56):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": dense(ff)}


def gla_layer(heads=3, dim=20, vdim=28, tau=8.0, ff=56):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": dense(ff)}


def latent_layer(heads=3, dim=24, vdim=40, q_rank=36, kv_rank=50, scale=0.3, kv_from=None, ff=56):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": dense(ff)}


def config(layers, width=72, vocab=96, streams=3, groups=3, eps=1e-5, max_positions=600):
    return {"architecture": "Vebonex", "layers": copy.deepcopy(layers), "width": width, "vocab": vocab, "streams": streams,
            "norm": {"eps": eps, "groups": groups}, "max_positions": max_positions}


CONFIGS = {
    # sizes off every multiple, a layer without feed-forward, latents shared across other layers and heads of other sizes
    "shared": config([latent_layer(), gla_layer(), latent_layer(heads=5, dim=16, vdim=8, q_rank=20, kv_from=0), lstm_layer(ff=None),
                      latent_layer(heads=2, q_rank=12, kv_rank=20, scale=0.7), latent_layer(heads=2, vdim=12, kv_rank=20, kv_from=4)]),
    # everything one: one stream, one group, single heads, unit constants, a width that is no multiple of 8
    "ones": config([lstm_layer(heads=1, dim=8, vdim=8, cap=1.0, ff=30), latent_layer(heads=1, dim=8, vdim=8, q_rank=5, kv_rank=4, scale=1.0, ff=None),
                    gla_layer(heads=1, dim=8, vdim=8, tau=1.0, ff=30)], width=30, vocab=50, streams=1, groups=1),
    # more heads than a tile of the decode kernel holds, head sizes above 128, values wider than a column tile, five streams
    "wide": config([gla_layer(heads=2, dim=136, vdim=72, tau=30.0, ff=96), latent_layer(heads=17, dim=136, vdim=24, q_rank=64, kv_rank=200, scale=0.1),
                    lstm_layer(heads=2, dim=40, vdim=136, cap=20.0)], width=160, vocab=130, streams=5, groups=5),
    # what the tensor-core attention kernels do not take: value heads above 256, a latent above 512
    "large": config([latent_layer(heads=2, dim=16, vdim=264, q_rank=24, kv_rank=40, ff=None), latent_layer(heads=2, kv_rank=520, ff=40)],
                    width=64, vocab=60, streams=2, groups=2),
}


def tensors(cfg: dict, seed: int = 0, decay_rank: int = 6) -> dict[str, torch.Tensor]:
    """bf16 checkpoint tensors: decays from fast to very slow, every constant away from its neutral value."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s, std=None, mean=0.0: torch.randn(*s, generator=g) * (s[-1] ** -0.5 if std is None else std) + mean
    un = lambda lo, hi, *s: torch.rand(*s, generator=g) * (hi - lo) + lo
    width, streams, out = cfg["width"], cfg["streams"], {}
    out["embed"], out["head"] = rn(cfg["vocab"], width, std=1.0), rn(cfg["vocab"], width, std=2.0 * width ** -0.5)
    out["pos"], out["final.norm"] = rn(cfg["max_positions"], width, std=0.4), rn(width, std=0.2, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer["mlp"] else (1,):
            out.update({f"{p}norm{q}": rn(width, std=0.2, mean=1.0), f"{p}hc{q}.in": rn(streams, std=0.15, mean=1.0 / streams),
                        f"{p}hc{q}.out": rn(streams, std=0.3, mean=1.0),
                        f"{p}hc{q}.mix": torch.eye(streams) * 0.8 + rn(streams, streams, std=0.2)})
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({p + "mlp.up": rn(ff, width, std=1.3 * width ** -0.5), p + "mlp.down": rn(width, ff),
                        p + "mlp.act": torch.tensor([0.5, 0.35, 0.25, 0.4]) + rn(4, std=0.1)})
        p += "mix."
        h, d, dv = m["heads"], m["dim"], m["vdim"]
        out.update({p + "g": rn(h * dv, width, std=1.5 * width ** -0.5), p + "o": rn(width, h * dv)})
        if layer["type"] == "latent_attention":
            out.update({p + "dq": rn(m["q_rank"], width), p + "dq.norm": rn(m["q_rank"], std=0.2, mean=1.0),
                        p + "uq": rn(h * d, m["q_rank"], std=1.5 * m["q_rank"] ** -0.5), p + "uk": rn(h * d, m["kv_rank"], std=1.5 * m["kv_rank"] ** -0.5),
                        p + "uv": rn(h * dv, m["kv_rank"])})
            if "kv_from" not in m:
                out.update({p + "dkv": rn(m["kv_rank"], width), p + "dkv.norm": rn(m["kv_rank"], std=0.2, mean=1.0)})
            continue
        out.update({p + "q": rn(h * d, width), p + "k": rn(h * d, width), p + "v": rn(h * dv, width)})
        if layer["type"] == "mlstm":
            out.update({p + "norm": rn(h * dv, std=0.2, mean=1.0), p + "i": rn(h, width), p + "i.b": un(-1.0, 1.0, h), p + "f": rn(h, width),
                        p + "f.b": un(0.5, 6.0, h)})
        else:
            out.update({p + "norm": rn(dv, std=0.2, mean=1.0), p + "a1": rn(decay_rank, width), p + "a2": rn(h * d, decay_rank, std=1.0),
                        p + "a2.b": un(-3.0, 6.0, h * d)})
    return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}
