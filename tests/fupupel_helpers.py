"""Small Fupupel models with weights of the tests' own making (nothing here comes from the package's initialiser)."""
from __future__ import annotations

import copy

import torch


def scan_layer(inner=40, state=8, dt_rank=5, conv=4, mlp=None):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}, "mlp": mlp}


def both_layer(heads=4, kv_heads=2, dim=32, vdim=24, window=20, rot=16, base=10000.0, scale=0.3, softcap=6.0, r_heads=4,
               r_kv=2, r_dim=16, r_vdim=24, conv=3, ls=0.7, rs=1.3, ff=56, limit=1.5):
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit},
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                               "rot": {"base": base, "dims": rot}, "scale": scale, "softcap": softcap},
                      "right": {"heads": r_heads, "kv_heads": r_kv, "dim": r_dim, "vdim": r_vdim, "conv": conv},
                      "left_scale": ls, "right_scale": rs}}


def config(layers, width=64, vocab=96, eps=1e-5, cap=9.0):
    return {"architecture": "Fupupel", "layers": copy.deepcopy(layers), "width": width, "vocab": vocab, "norm": {"eps": eps},
            "logit_softcap": cap}


CONFIGS = {
    # grouped heads, a value size smaller than the key size, a partial rotation, sizes that are no multiple of 8
    "grouped": config([scan_layer(), both_layer(), scan_layer(inner=36, state=5, dt_rank=3, conv=2),
                       both_layer(window=7, r_heads=6, r_kv=3, r_dim=20, r_vdim=12, rot=32)]),
    # everything one: single heads, unit scales, window 1, width not a multiple of 8; a feed-forward behind a scan layer
    "ones": config([both_layer(heads=1, kv_heads=1, dim=16, vdim=16, window=1, rot=16, softcap=1.0, scale=1.0, r_heads=1, r_kv=1,
                               r_dim=8, r_vdim=8, conv=1, ls=1.0, rs=1.0, ff=None),
                    scan_layer(inner=20, state=1, dt_rank=1, conv=1, mlp={"kind": "dense", "ff": 30, "limit": 1.0})],
                   width=36, vocab=50, cap=1.0),
    # a wide window over page borders, large values, three KV heads, many states, one head group of nine
    "wide": config([both_layer(heads=9, kv_heads=1, dim=24, vdim=136, window=150, rot=8, r_heads=2, r_kv=2, r_dim=40, r_vdim=136,
                               conv=5), scan_layer(inner=48, state=33, dt_rank=9, conv=3),
                    both_layer(heads=6, kv_heads=3, dim=40, vdim=40, window=200, rot=40)], width=72, vocab=130),
}


def tensors(cfg: dict, seed: int = 0, ranks=(6, 10)) -> dict[str, torch.Tensor]:
    """bf16 checkpoint tensors: decays from fast to very slow, every constant away from its neutral value."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s, std=None, mean=0.0: torch.randn(*s, generator=g) * (s[-1] ** -0.5 if std is None else std) + mean
    un = lambda lo, hi, *s: torch.rand(*s, generator=g) * (hi - lo) + lo
    width, out = cfg["width"], {}
    out["embed"], out["head"] = rn(cfg["vocab"], width, std=1.0), rn(cfg["vocab"], width, std=2.0 * width ** -0.5)
    out["final.norm"] = rn(width, std=0.2, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            out[p + n] = rn(width, std=0.2, mean=1.0)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({p + "mlp.gate": rn(ff, width, std=1.5 * width ** -0.5), p + "mlp.up": rn(ff, width, std=1.5 * width ** -0.5),
                        p + "mlp.down": rn(width, ff)})
        p += "mix."
        if layer["type"] == "mamba1":
            inner, n, r = m["inner"], m["state"], m["dt_rank"]
            out.update({p + "in": rn(2 * inner, width), p + "conv": rn(inner, m["conv"], std=0.6), p + "conv.b": rn(inner, std=0.3),
                        p + "x": rn(r + 2 * n, inner, std=2 * inner ** -0.5), p + "dt": rn(inner, r), p + "dt.b": un(-6.0, 0.5, inner),
                        p + "A_log": un(-3.0, 2.0, inner, n), p + "D": rn(inner), p + "o": rn(width, inner)})
            continue
        a, r = m["left"], m["right"]
        out.update({p + "left.q": rn(a["heads"] * a["dim"], width, std=2 * width ** -0.5),
                    p + "left.k": rn(a["kv_heads"] * a["dim"], width, std=2 * width ** -0.5),
                    p + "left.v": rn(a["kv_heads"] * a["vdim"], width), p + "left.o": rn(width, a["heads"] * a["vdim"])})
        p += "right."
        for n, c in (("q", r["kv_heads"] * r["dim"]), ("k", r["kv_heads"] * r["dim"]), ("v", r["heads"] * r["vdim"])):
            out[p + n], out[p + n + ".conv"] = rn(c, width), rn(c, r["conv"], std=0.7)
        out.update({p + "b": rn(r["heads"], width), p + "A_log": un(-4.0, 1.0, r["heads"]),
                    p + "dt_bias": un(-5.0, 0.0, r["heads"] * r["dim"]), p + "norm": rn(r["vdim"], std=0.2, mean=1.0),
                    p + "a1": rn(ranks[0], width), p + "a2": rn(r["heads"] * r["dim"], ranks[0]), p + "g1": rn(ranks[1], width),
                    p + "g2": rn(r["heads"] * r["vdim"], ranks[1]), p + "o": rn(width, r["heads"] * r["vdim"])})
    return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}
