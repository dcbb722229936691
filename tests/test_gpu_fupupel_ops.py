"""The kernels of the mixer branches, each against the plain oracle: ragged portions with carried state, single-token steps,
slots that are used again, sizes off every multiple."""
import math

import pytest
import torch

from mini_vllm_b200 import ops
from mini_vllm_b200.models.layers.rotary import build_cos_sin_cache
from oracle import fupupel as plain
from tests.step_helpers import PORTIONS, gen, rel, run_steps

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
TOL = {BF: 2e-2, F32: 2e-5}


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("taps,channels,bias", [(4, 64, True), (3, 30, False), (2, 8, True), (1, 16, False), (6, 24, True), (9, 12, True)])
@pytest.mark.parametrize("portions", ["whole", "single", "twos", "mixed"])
def test_short_conv(cuda, dtype, taps, channels, bias, portions):
    g, lens = gen(1), [70, 3, 129, 1]
    w, b = torch.randn(channels, taps, generator=g).to(dtype), torch.randn(channels, generator=g).to(dtype) if bias else None
    us = [torch.randn(n, channels, generator=g).to(dtype) for n in lens]
    want = [plain.silu(plain.causal_conv(u.double(), w.double(), None if b is None else b.double())) for u in us]
    state = torch.full((len(lens) + 2, taps - 1, channels), 7.0, dtype=dtype, device=cuda)     # leftovers of earlier owners
    wd, bd = w.flip(1).T.contiguous().to(cuda), None if b is None else b.to(cuda)
    got = [torch.empty_like(w) for w in want]

    def step(entries, cu, pos, slots):
        wide = torch.cat([us[i][a:e] for i, a, e in entries])
        packed = torch.cat([wide, torch.zeros(wide.shape[0], 8, dtype=dtype)], dim=1).to(cuda)[:, :channels]      # a row stride of its own
        out = ops.short_conv_silu(packed, wd, bd, state if taps > 1 else None, slots, cu, pos).cpu()
        at = 0
        for i, a, e in entries:
            got[i][a:e] = out[at:at + e - a].double()
            at += e - a
    run_steps(cuda, lens, PORTIONS[portions], step)
    assert max(rel(x, y) for x, y in zip(got, want)) < (1e-2 if dtype == BF else 1e-5)


def scan_inputs(g, lens, inner, n, dtype):
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    seqs = [{"u": mk(t, inner), "dt": mk(t, inner), "z": mk(t, inner), "b": mk(t, n), "c": mk(t, n)} for t in lens]
    bias = torch.rand(inner, generator=g) * 7 - 6.5
    a = -torch.exp(torch.rand(inner, n, generator=g) * 5 - 3)
    return seqs, bias, a, torch.randn(inner, generator=g)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("inner,n", [(40, 16), (33, 5), (128, 20), (20, 40), (12, 100), (9, 130), (70, 1)])
@pytest.mark.parametrize("portions", ["whole", "single", "mixed", "long"])
def test_selective_scan(cuda, dtype, inner, n, portions):
    g, lens = gen(2), [70, 3, 300, 1]
    seqs, bias, a, d = scan_inputs(g, lens, inner, n, dtype)
    want = []
    for s in seqs:
        x = {k: v.double() for k, v in s.items()}
        y, _ = plain.selective_scan(x["u"], plain.softplus(x["dt"] + bias.double()), a.double(), x["b"], x["c"], d.double())
        want.append(y * plain.silu(x["z"]))
    np_ = -(-n // 4) * 4
    al = torch.zeros(inner, np_)
    al[:, :n] = a / math.log(2.0)
    state = torch.full((len(lens) + 2, inner, np_), float("nan"), device=cuda)
    got = [torch.empty_like(w) for w in want]
    biasd, ald, dd = bias.to(cuda), al.to(cuda), d.to(cuda)

    def step(entries, cu, pos, slots):
        pk = {k: torch.cat([seqs[i][k][s:e] for i, s, e in entries]).to(cuda) for k in seqs[0]}
        bc = torch.cat([pk["b"], pk["c"]], dim=1)
        out = torch.full_like(pk["u"], float("nan"))
        ops.selective_scan(pk["u"], pk["dt"], pk["z"], bc[:, :n], bc[:, n:], biasd, ald, dd, out, state, slots, cu, pos)
        at = 0
        for i, s, e in entries:
            got[i][s:e] = out[at:at + e - s].double().cpu()
            at += e - s
    run_steps(cuda, lens, PORTIONS[portions], step)
    assert max(rel(x, y) for x, y in zip(got, want)) < TOL[dtype]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 64, 40), (3, 3, 20, 12), (2, 1, 128, 128), (2, 2, 40, 136), (1, 1, 200, 24), (6, 2, 8, 50),
                                               (2, 2, 96, 96)])
@pytest.mark.parametrize("portions", ["whole", "single", "mixed", "long"])
def test_gated_delta(cuda, dtype, heads, kv, dim, vdim, portions):
    g, lens, eps = gen(3), [70, 3, 150, 1], 1e-5
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    seqs = [{"q": mk(t, kv, dim), "k": mk(t, kv, dim), "v": mk(t, heads, vdim), "a": mk(t, heads * dim), "b": mk(t, heads),
             "gate": mk(t, heads * vdim)} for t in lens]
    # decays from almost none to one that wipes a row out within a token or two
    ea, db, nw = torch.exp(torch.rand(heads, generator=g) * 6 - 3), torch.rand(heads * dim, generator=g) * 7 - 6, torch.rand(vdim, generator=g) + 0.5
    ea[0] = 40.0 if heads > 1 else ea[0]
    want = []
    for s in seqs:
        x, t = {k: v.double() for k, v in s.items()}, s["q"].shape[0]
        unit = lambda y: y / torch.sqrt((y * y).sum(-1, keepdim=True) + 1e-6)
        q, k = unit(x["q"]) * dim ** -0.5, unit(x["k"])
        gd = torch.exp(-ea.double()[:, None] * plain.softplus(x["a"] + db.double()).view(t, heads, dim))
        beta = torch.sigmoid(x["b"])
        o = torch.stack([plain.delta_rule(q[:, h // (heads // kv)], k[:, h // (heads // kv)], x["v"][:, h], gd[:, h], beta[:, h])[0]
                         for h in range(heads)], dim=1)
        want.append(plain.rms_norm(o, nw.double(), eps) * torch.sigmoid(x["gate"]).view(t, heads, vdim) * 1.3)
    state = torch.zeros(len(lens) + 2, heads, dim, -(-vdim // 4) * 4, device=cuda).fill_(3.0)
    got = [torch.empty_like(w) for w in want]
    ead, dbd, nwd = ea.to(cuda), db.to(cuda), nw.to(cuda)

    def step(entries, cu, pos, slots):
        pk = {k: torch.cat([seqs[i][k][s:e] for i, s, e in entries]).to(cuda) for k in seqs[0]}
        rows = pk["q"].shape[0]
        qkv = torch.cat([pk["q"].flatten(1), pk["k"].flatten(1), pk["v"].flatten(1)], dim=1)
        q, k = qkv[:, :kv * dim].view(rows, kv, dim) if rows == 1 else qkv[:, :kv * dim].unflatten(1, (kv, dim)), qkv[:, kv * dim:2 * kv * dim].unflatten(1, (kv, dim))
        v = qkv[:, 2 * kv * dim:].unflatten(1, (heads, vdim))
        out = torch.full((rows, heads, vdim), float("nan"), dtype=dtype, device=cuda)
        ops.gated_delta(q, k, v, pk["a"], pk["b"], pk["gate"], ead, dbd, nwd, out, state, slots, cu, pos, dim ** -0.5, eps, 1.3)
        at = 0
        for i, s, e in entries:
            got[i][s:e] = out[at:at + e - s].double().cpu()
            at += e - s
    run_steps(cuda, lens, PORTIONS[portions], step)
    # (a row whose o is all but zero is scaled up by its norm: judged by the largest value of the whole)
    assert max(rel(x, y) for x, y in zip(got, want)) < (TOL[dtype] if dtype == BF else 1e-4)


# ---- attention: cap, window, factor, any head layout ---------------------------------------------------------
def window_case(g, lens, heads, kv, d, dtype):
    return [(torch.randn(n, heads, d, generator=g).to(dtype), torch.randn(n, kv, d, generator=g).to(dtype),
             torch.randn(n, kv, d, generator=g).to(dtype)) for n in lens]


def plant_key(q, k, dist, strength=6.0):
    """Make the key ``dist`` tokens back stand out for the last query of a sequence, in every head: whether it is seen decides
    the output."""
    i = q.shape[0] - 1
    if i - dist < 0:
        return
    per = q.shape[1] // k.shape[1]
    for h in range(k.shape[1]):
        u = q[i, h * per].float()
        k[i - dist, h] = (u / u.norm() * strength).to(k.dtype)


@pytest.mark.parametrize("heads,kv,d,window,cap", [(4, 2, 128, 80, 18.0), (3, 3, 128, 33, 5.0), (8, 1, 256, 128, 30.0), (6, 3, 128, None, 50.0),
                                                   (4, 2, 128, 129, 0.0), (4, 4, 128, 1, 2.0)])
@pytest.mark.parametrize("edge", [-1, 0])
def test_capped_window_attention_prefill_and_decode(cuda, heads, kv, d, window, cap, edge):
    """edge 0: the planted key is just outside the window; -1: just inside."""
    g, lens, scale, factor = gen(4), [130, 1, 300, 257, 40], 0.4, 0.75
    seqs = window_case(g, lens, heads, kv, d, BF)
    for q, k, _ in seqs:
        plant_key(q, k, (window or 120) + edge)
    want = [plain.attention(q.double(), k.double(), v.double(), scale, cap, window) * factor for q, k, v in seqs]
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=cuda)
    q, k, v = (torch.cat([s[j] for s in seqs]).to(cuda) for j in range(3))
    left = -1 if window is None else window - 1
    got = ops.prefill_attn(q, k, v, cu, cu, max(lens), scale, left, softcap=cap, out_scale=factor).cpu()
    assert rel(got, torch.cat(want)) < 2e-2
    pos = torch.cat([torch.arange(n) for n in lens]).to(cuda)
    got = ops.any_attn(q, k, v, pos, scale, left, cu_seqlens_q=cu, cu_seqlens_k=cu, softcap=cap, out_scale=factor).cpu()
    assert rel(got, torch.cat(want)) < 1e-2
    # the last token of every sequence through the paged decode kernels; unwritten slots hold NaNs
    bs = 128
    nblk = [-(-n // bs) for n in lens]
    order = torch.randperm(sum(nblk), generator=g).tolist()
    table = torch.full((len(lens), max(nblk)), -1, dtype=torch.int32)
    kp = torch.full((sum(nblk), bs, kv, d), float("nan"), dtype=BF)
    vp, at = kp.clone(), 0
    for i, (n, (_, ks, vs)) in enumerate(zip(lens, seqs)):
        for j in range(nblk[i]):
            table[i, j] = order[at]
            kp[order[at], :min(bs, n - j * bs)] = ks[j * bs:(j + 1) * bs]
            vp[order[at], :min(bs, n - j * bs)] = vs[j * bs:(j + 1) * bs]
            at += 1
    kp, vp, table = kp.to(cuda), vp.to(cuda), table.to(cuda)
    last = torch.stack([s[0][-1] for s in seqs]).to(cuda)
    n = torch.tensor(lens, dtype=torch.int32, device=cuda)
    status = ops.new_status(cuda)
    wl = torch.stack([w[-1] for w in want])
    ws = ops.decode_workspace(len(lens), heads, d, cuda)
    ops.decode_plan(n, left, heads, kv, d, ws, block_table=table, block_size=bs)
    got = ops.decode_attn(last, kp, vp, n, table, scale, left, ws, status=status, softcap=cap, out_scale=factor)
    assert rel(got, wl) < 2e-2
    got = ops.any_attn(last, kp, vp, (n - 1).long(), scale, left, block_table=table, cache_seqlens=n, softcap=cap, out_scale=factor,
                       status=status)
    assert rel(got, wl) < 1e-2
    # portions through the pool: the second half of each sequence with the first half cached
    half = [x // 2 for x in lens]
    cq = torch.tensor([0] + list(torch.tensor([x - h for x, h in zip(lens, half)]).cumsum(0)), dtype=torch.int32, device=cuda)
    q2 = torch.cat([s[0][h:] for s, h in zip(seqs, half)]).to(cuda)
    got = ops.prefill_attn(q2, kp, vp, cq, cu, max(x - h for x, h in zip(lens, half)), scale, left, block_table=table, softcap=cap,
                           out_scale=factor, status=status)
    assert rel(got, torch.cat([w[h:] for w, h in zip(want, half)])) < 2e-2
    ops.check_status(status)


@pytest.mark.parametrize("heads,kv,d", [(9, 1, 48), (4, 2, 272), (2, 2, 528), (6, 3, 16)])
def test_any_attention_in_fp32(cuda, heads, kv, d):
    g, lens = gen(5), [130, 1, 67]
    seqs = window_case(g, lens, heads, kv, d, F32)
    want = torch.cat([plain.attention(q.double(), k.double(), v.double(), 0.2, 7.0, 50) for q, k, v in seqs])
    cu = torch.tensor([0, 130, 131, 198], dtype=torch.int32, device=cuda)
    q, k, v = (torch.cat([s[j] for s in seqs]).to(cuda) for j in range(3))
    pos = torch.cat([torch.arange(n) for n in lens]).to(cuda)
    got = ops.any_attn(q, k, v, pos, 0.2, 49, cu_seqlens_q=cu, cu_seqlens_k=cu, softcap=7.0)
    assert rel(got, want) < 1e-5


def test_scores_do_not_lose_the_cap_far_out(cuda):
    """Scores a hundred times the cap: tanh saturates, so keys on either side of it must come out equal and finite."""
    q = torch.full((2, 1, 128), 8.0, dtype=BF, device=cuda)
    k = torch.stack([torch.full((1, 128), 8.0), torch.full((1, 128), 4.0)]).to(BF).to(cuda)
    v = torch.stack([torch.full((1, 128), 1.0), torch.full((1, 128), 3.0)]).to(BF).to(cuda)
    cu = torch.tensor([0, 2], dtype=torch.int32, device=cuda)
    out = ops.prefill_attn(q, k, v, cu, cu, 2, 1.0, -1, softcap=25.0)
    assert torch.allclose(out[1].float(), torch.full_like(out[1], 2.0).float(), atol=1e-2)


# ---- rotation ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,d", [(16, 32), (32, 32), (2, 48), (0, 16)])
def test_rotation_of_laid_out_heads_keeps_every_score(cuda, dims, d):
    """The branch lays rotated pairs out at (i, i + D/2): scores after the kernel equal those of the plain rotation."""
    from mini_vllm_b200.models.layers.branches import AttentionBranch
    from mini_vllm_b200.models.layers.rotary import RotaryEmbedding
    g, t, padded, base = gen(6), 90, 128, 5000.0
    br = AttentionBranch(1, 1, d, d, 1.0, RotaryEmbedding(dims, t, base, head_dim=padded), dims, padded)
    place = br._layout()
    q, k = torch.randn(t, 1, d, generator=g), torch.randn(t, 1, d, generator=g)
    want = plain.rotate(q.double(), dims, base)[:, 0] @ plain.rotate(k.double(), dims, base)[:, 0].T
    lay = lambda x, dt: torch.zeros(t, 1, padded).index_copy(2, place, x).to(dt).to(cuda)
    pos, table = torch.arange(t, device=cuda), br.rotary.cos_sin_cache.to(cuda)
    for dt, write in ((F32, ops.rope_kv_write_f32), (BF, ops.rope_kv_write)):
        qd, kd = lay(q, dt), lay(k, dt)
        write(qd, kd, kd, pos, table, None, None, None, k_in_place=True)
        got = qd[:, 0].double().cpu() @ kd[:, 0].double().cpu().T
        assert rel(got, want) < (2e-2 if dt == BF else 1e-5)


def test_rotation_table_far_out():
    t = build_cos_sin_cache(8, 60000, 10000.0, head_dim=16)
    f = 10000.0 ** (-2.0 * torch.arange(4, dtype=torch.float64) / 8)
    assert (t[59999, :4].double() - torch.cos(59999 * f)).abs().max() < 1e-6 and (t[:, 4:8] == 1).all() and (t[:, 12:] == 0).all()


# ---- glue ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width", [36, 64, 320, 2048, 5000, 30])
def test_residual_norms(cuda, dtype, width):
    g, rows, eps = gen(7), 9, 1e-5
    x, y = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g).to(dtype)
    w, yw = (torch.rand(width, generator=g) + 0.5).to(dtype), (torch.rand(width, generator=g) + 0.5).to(dtype)
    tol = 1e-2 if dtype == BF else 1e-5
    new = x.double() + plain.rms_norm(y.double(), yw.double(), eps)
    xd = x.to(cuda)
    out = ops.residual_norm(xd, y.to(cuda), w.to(cuda), eps, y_weight=yw.to(cuda))
    assert rel(xd, new) < 1e-6 and rel(out, plain.rms_norm(new, w.double(), eps)) < tol
    xd = x.to(cuda)
    ends = torch.tensor([0, 3, 4, 9], dtype=torch.int32, device=cuda)
    out = ops.residual_norm(xd, y.to(cuda), w.to(cuda), eps, row_ends=ends)
    assert torch.equal(xd.cpu(), x) and rel(out, plain.rms_norm(x.double() + y.double(), w.double(), eps)[[2, 3, 8]]) < tol
    assert ops.residual_norm(xd, y.to(cuda), w.to(cuda), eps, row_ends=ends[:1]).shape == (0, width)
    table, ids = torch.randn(50, width, generator=g).to(dtype), torch.tensor([0, 49, 7, 7])
    x0, h0 = ops.embed_norm(ids.to(cuda), table.to(cuda), w.to(cuda), eps)
    assert torch.equal(x0.cpu(), table[ids].float()) and rel(h0, plain.rms_norm(table[ids].double(), w.double(), eps)) < tol


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("inter", [24, 30, 384])
def test_clamped_glu(cuda, dtype, inter):
    gu = (torch.randn(7, 2 * inter, generator=gen(8)) * 4).to(dtype)
    gu[0, :4] = torch.tensor([1e4, -1e4, -60.0, 2.0])
    want = plain.clamped_glu(gu[:, :inter].double(), gu[:, inter:].double(), 1.5)
    assert rel(ops.clamped_glu(gu.to(cuda), inter, 1.5, 1.702), want) < (1e-2 if dtype == BF else 1e-6)


def test_capped_logits_and_fp32_argmax(cuda):
    x = torch.randn(5, 1003, generator=gen(9)) * 30
    assert rel(ops.cap_logits(x.to(cuda), 12.0, F32), plain.soft_cap(x.double(), 12.0)) < 1e-6
    assert torch.equal(ops.cap_logits(x.to(cuda), 0.0, F32).cpu(), x)
    y = x.clone()
    y[0, 700] = y[0, 3] = 1e3                                   # a tie: the lower column wins
    y[1, 1002] = 1e3
    table, index = torch.zeros(9, dtype=torch.int64, device=cuda), torch.tensor([8, 1, 2, 3, 0], dtype=torch.int32, device=cuda)
    tok = ops.argmax_f32(y.to(cuda), table, index).cpu()
    assert torch.equal(tok, y.argmax(-1)) and tok[0] == 3 and table.cpu()[8] == 3 and table.cpu()[0] == tok[4]
