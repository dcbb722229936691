"""Small Rasezen models with weights of the tests' own making (nothing here comes from the package's initialiser)."""
from __future__ import annotations

import copy

import torch


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24, identity=1, scale=1.7, shared=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity, "scale": scale},
            "shared": None if shared is None else {"ff": shared}}


def state_layer(heads=6, groups=3, state=20, vdim=12, taps=4, norm_groups=4, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": taps,
                                                    "norm_groups": norm_groups}}


def window_layer(heads=6, kv=2, dim=28, vdim=20, size=37, rot=10, base=500.0, scale=0.3, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                                                       "mask": {"size": size}, "rot": {"base": base, "dims": rot}}}


def config(layers, width=88, vocab=96, eps=1e-4):
    return {"architecture": "Rasezen", "layers": copy.deepcopy(layers), "width": width, "vocab": vocab, "norm": {"eps": eps}}


CONFIGS = {
    # sizes off every multiple, a layer without feed-forward, norm groups across heads, experts with and without identity and shared ones
    "several": config([state_layer(mlp=moe()), window_layer(mlp=dense()), state_layer(heads=5, groups=1, state=33, vdim=9, taps=2, norm_groups=3),
                       window_layer(heads=5, kv=5, dim=17, vdim=40, size=130, rot=16, mlp=moe(7, 3, 13, 3, 0.6, None)),
                       window_layer(heads=4, kv=1, dim=20, vdim=20, size=2, rot=20, mlp=moe(4, 4, 30, 0, 1.0, 33)),
                       state_layer(heads=4, groups=4, state=16, vdim=32, taps=5, norm_groups=1, mlp=dense(33))]),
    # nearly everything one: single heads, states and experts, one tap, a window that sees the token itself alone, a width that is no multiple of 8
    "ones": config([state_layer(1, 1, 1, 4, 1, 1, moe(1, 1, 30, 1, 1.0, 1)), window_layer(1, 1, 8, 8, 1, 2, scale=1.0, mlp=moe(1, 2, 1, 1, 1.0, None)),
                    state_layer(1, 1, 8, 16, 1, 1, None), window_layer(1, 1, 8, 8, 70, 8, scale=1.0, mlp=dense(1))], width=30, vocab=50),
    # a window wider than a page, heads above 128, several tiles of values and states, more router outputs than lanes
    "wide": config([state_layer(heads=4, groups=2, state=128, vdim=64, taps=4, norm_groups=2, mlp=moe(37, 4, 40, 6, 2.0, 64)),
                    window_layer(heads=6, kv=2, dim=136, vdim=72, size=150, rot=64, mlp=dense(96)),
                    state_layer(heads=2, groups=1, state=64, vdim=96, taps=3, norm_groups=6, mlp=moe(30, 1, 72, 34, 1.0, 16))], width=160, vocab=130),
    # what the tensor-core kernels do not take: more than eight heads per KV head, heads above 256; many states and value columns
    "large": config([window_layer(heads=18, kv=2, dim=16, vdim=24, size=64, rot=8, mlp=dense(40)),
                     state_layer(heads=2, groups=2, state=200, vdim=136, taps=4, norm_groups=2, mlp=None),
                     window_layer(heads=2, kv=1, dim=264, vdim=264, size=300, rot=264, mlp=moe(3, 2, 8, 2))], width=64, vocab=60),
}


def tensors(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    """bf16 checkpoint tensors, every constant away from its neutral value."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s, std=None, mean=0.0: torch.randn(*s, generator=g) * (s[-1] ** -0.5 if std is None else std) + mean
    uniform = lambda lo, hi, n: torch.rand(n, generator=g) * (hi - lo) + lo
    one = lambda mean: torch.tensor(mean) + torch.rand((), generator=g) * 0.5
    width, out = cfg["width"], {}
    out["embed"], out["head"] = rn(cfg["vocab"], width, std=1.0), rn(cfg["vocab"], width, std=2.0 * width ** -0.5)
    out["final.norm"] = one(0.6)

    def unit(p, ff):
        out.update({p + "gate": rn(ff, width, std=1.5 * width ** -0.5), p + "up": rn(ff, width, std=1.5 * width ** -0.5), p + "down": rn(width, ff)})

    for i, layer in enumerate(cfg["layers"]):
        p, m, ff = f"l{i}.", layer["mixer"], layer["mlp"]
        out[p + "norm1"] = one(0.8)
        if ff and ff["kind"] == "dense":
            out.update({p + "mlp.up": rn(ff["ff"], width, std=1.5 * width ** -0.5), p + "mlp.down": rn(width, ff["ff"]),
                        p + "mlp.act": torch.tensor([-1.3, 0.4]) + rn(2, std=0.2)})
        elif ff:
            r = ff["router"]
            outputs = r["experts"] + r["identity"]
            out.update({p + "mlp.router": rn(outputs, width, std=3.0 * width ** -0.5), p + "mlp.correction": rn(outputs, std=0.5)})
            for e in range(r["experts"]):
                unit(f"{p}mlp.e{e}.", ff["expert"]["ff"])
            if ff["shared"]:
                unit(p + "mlp.shared.", ff["shared"]["ff"])
        p += "mix."
        h, dv = m["heads"], m["vdim"]
        out[p + "o"] = rn(width, h * dv)
        if layer["type"] == "mamba2":
            channels = h * dv + 2 * m["groups"] * m["state"]
            out.update({p + "in": rn(h * dv + channels + h, width, std=1.5 * width ** -0.5), p + "conv": rn(channels, m["conv"], std=0.7),
                        p + "conv.b": rn(channels, std=0.3), p + "dt_bias": uniform(-4.0, 0.5, h), p + "A_log": uniform(-3.0, 1.5, h),
                        p + "D": uniform(0.3, 1.7, h), p + "norm": rn(h * dv, std=0.3, mean=1.0)})
            continue
        for n, c in (("q", h * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * dv)):
            out.update({p + n: rn(c, width, std=1.5 * width ** -0.5), f"{p}{n}.b": rn(c, std=0.4)})
            if n != "v":
                out[f"{p}{n}.norm"] = rn(c, std=0.3, mean=1.0)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}
