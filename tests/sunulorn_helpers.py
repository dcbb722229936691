"""Small Sunulorn models with weights of the tests' own making (nothing here comes from the package's initialiser)."""
from __future__ import annotations

import copy

import torch


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24, limit=0.8, shared=40, shared_limit=1.3):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top},
            "shared": None if shared is None else {"ff": shared, "limit": shared_limit}}


def conv_layer(heads=6, kv=2, dim=28, taps=3, rot=10, base=500.0, scale=0.3, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "conv": taps, "scale": scale,
                                                       "rot": {"base": base, "dims": rot}}}


def window_layer(heads=4, kv=2, dim=20, vdim=36, size=37, keep=9, rot=20, base=3000.0, scale=0.25, mlp=None):
    return {"type": "attention_2", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                                                         "mask": {"size": size, "keep_first": keep}, "rot": {"base": base, "dims": rot}}}


def distance_layer(heads=6, kv=3, dim=24, vdim=40, scale=0.35, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention_3", "mlp": mlp, "mixer": m}


def config(layers, width=72, vocab=96, eps=1e-5, scale=3.3):
    return {"architecture": "Sunulorn", "layers": copy.deepcopy(layers), "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"scale": scale}}


CONFIGS = {
    # sizes off every multiple, a layer without feed-forward, borrowed keys across other layers, experts with and without a shared one
    "several": config([distance_layer(mlp=moe()), conv_layer(mlp=dense()), distance_layer(kv_from=0, mlp=dense(33)),
                       window_layer(mlp=moe(7, 3, 13, 0.5, None)), conv_layer(heads=3, kv=3, dim=20, taps=5, rot=20, mlp=None),
                       distance_layer(heads=5, kv=5, dim=17, vdim=9), distance_layer(heads=5, kv=5, dim=17, vdim=9, kv_from=5, mlp=moe(2, 2))]),
    # everything one: single heads and experts, one tap, a window that sees the token itself alone, a width that is no multiple of 8
    "ones": config([conv_layer(heads=1, kv=1, dim=8, taps=1, rot=2, scale=1.0, mlp=moe(1, 1, 30, 1.0, 1, 1.0)),
                    window_layer(heads=1, kv=1, dim=8, vdim=8, size=1, keep=0, rot=8, scale=1.0, mlp=None),
                    distance_layer(heads=1, kv=1, dim=8, vdim=8, scale=1.0, mlp=dense(1))], width=30, vocab=50, scale=1.0),
    # windows and kept tokens wider than a page, heads above 128, more experts than lanes
    "wide": config([window_layer(heads=6, kv=2, dim=136, vdim=72, size=150, keep=131, rot=64, mlp=moe(37, 4, 40, 2.0, 64)),
                    conv_layer(heads=4, kv=1, dim=160, taps=4, rot=96, mlp=dense(96)),
                    distance_layer(heads=2, kv=1, dim=64, vdim=128, mlp=moe(33, 1, 72, 0.4, 16))], width=160, vocab=130),
    # what the tensor-core attention does not take: more than eight heads per KV head, heads above 256
    "large": config([distance_layer(heads=18, kv=2, dim=16, vdim=24, mlp=dense(40)), window_layer(heads=9, kv=1, dim=16, vdim=16, rot=4),
                     conv_layer(heads=2, kv=1, dim=264, taps=2, rot=264, mlp=None), distance_layer(heads=18, kv=2, dim=16, vdim=24, kv_from=0)],
                    width=64, vocab=60),
}


def tensors(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    """bf16 checkpoint tensors, every constant away from its neutral value."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s, std=None, mean=0.0: torch.randn(*s, generator=g) * (s[-1] ** -0.5 if std is None else std) + mean
    width, out = cfg["width"], {}
    out["embed"], out["head"] = rn(cfg["vocab"], width, std=1.0 / cfg["embedding"]["scale"]), rn(cfg["vocab"], width, std=2.0 * width ** -0.5)
    out["final.norm"] = rn(width, std=0.2, mean=1.0)

    def unit(p, ff):
        out.update({p + "gate": rn(ff, width, std=1.5 * width ** -0.5), p + "up": rn(ff, width, std=1.5 * width ** -0.5), p + "down": rn(width, ff)})

    for i, layer in enumerate(cfg["layers"]):
        p, m, ff, kind = f"l{i}.", layer["mixer"], layer["mlp"], layer["type"]
        out[p + "norm1"] = rn(width, std=0.2, mean=1.0)
        if ff:
            out[p + "norm2"] = rn(width, std=0.2, mean=1.0)
        if ff and ff["kind"] == "dense":
            unit(p + "mlp.", ff["ff"])
        elif ff:
            out[p + "mlp.router"] = rn(ff["router"]["experts"], width, std=4.0 * width ** -0.5)
            for e in range(ff["router"]["experts"]):
                unit(f"{p}mlp.e{e}.", ff["expert"]["ff"])
            if ff["shared"]:
                unit(p + "mlp.shared.", ff["shared"]["ff"])
                out[p + "mlp.shared.sg"] = rn(1, width)
        p += "mix."
        h, kv, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        rows = {"q": h * d, "k": kv * d, "v": kv * dv}
        if kind == "attention":
            del rows["v"]
        if "kv_from" in m:
            rows = {"q": h * d}
        for n, c in rows.items():
            out[p + n] = rn(c, width, std=1.5 * width ** -0.5)
            if kind == "attention":
                out[f"{p}{n}.conv"] = rn(c, m["conv"], std=0.7)
            else:
                out[f"{p}{n}.b"] = rn(c, std=0.4)
        out[p + "o"] = rn(width, h * dv)
        if kind == "attention_2":
            out.update({p + "o.b": rn(width, std=0.4), p + "g": rn(h * dv, width)})
        elif kind == "attention_3":
            out.update({p + "g": rn(h, width), p + "sink": rn(h, std=1.5)})
    return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}
