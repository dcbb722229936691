"""Feeding kernels with ragged steps: portions of several sequences, single-token steps, slots out of order."""
from __future__ import annotations

import torch


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rel(got, want):
    want = want.double()
    return float((got.double().cpu() - want).abs().max() / want.abs().max().clamp(min=1e-6))


def cuts(total, portions):
    out, at = [], 0
    while at < total:
        n = min(portions[len(out) % len(portions)], total - at)
        out.append((at, at + n))
        at += n
    return out


def ragged_steps(lens, portions):
    """Steps of a batch of sequences fed in portions; a sequence that has ended brings no row."""
    plans = [cuts(n, portions[i % len(portions)]) for i, n in enumerate(lens)]
    for k in range(max(len(p) for p in plans)):
        yield [(i, *plans[i][k]) for i in range(len(lens)) if k < len(plans[i])]


def run_steps(cuda, lens, portions, call):
    """Drives ``call(step, cu or None, positions, slots)``; single-token steps go without boundaries."""
    slots_of = [len(lens) - i for i in range(len(lens))]
    for step in ragged_steps(lens, portions):
        pos = torch.cat([torch.arange(a, b) for _, a, b in step]).to(cuda)
        single = all(b - a == 1 for _, a, b in step)
        cu = None if single else torch.tensor([0] + list(torch.tensor([b - a for _, a, b in step]).cumsum(0)), dtype=torch.int32, device=cuda)
        slots = torch.tensor([slots_of[i] for i, _, _ in step], dtype=torch.int32, device=cuda)
        call(step, cu, pos, slots)


PORTIONS = {"whole": [[10 ** 6]], "single": [[1]], "twos": [[2]], "mixed": [[5, 1, 33, 2], [1], [2, 3, 64]], "long": [[70, 1, 1, 40]]}
