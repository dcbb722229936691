"""The kernels of the Vebonex design, each against the plain oracle: ragged portions with carried state, single-token steps, slots and
blocks that are used again, sizes off every multiple, gates at their extremes."""
import pytest
import torch

from mini_vllm_b200 import ops
from oracle import vebonex as plain
from tests.step_helpers import PORTIONS, gen, rel, run_steps

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
SIZES = [(3, 20, 28), (2, 64, 40), (2, 128, 128), (1, 8, 8), (2, 40, 136), (1, 200, 24), (5, 7, 50), (2, 96, 260)]


def packed(seqs, entries, names, cuda):
    """Rows of a step side by side, as views of one packed projection."""
    parts = [torch.cat([seqs[i][n][a:e] for i, a, e in entries]).flatten(1) for n in names]
    wide = torch.cat(parts + [torch.zeros_like(parts[0])[:, :3]], dim=1).to(cuda)
    return dict(zip(names, wide.split([p.shape[1] for p in parts] + [3], dim=1)))


def collect(got, entries, out):
    at = 0
    for i, a, e in entries:
        got[i][a:e] = out[at:at + e - a].double().cpu()
        at += e - a


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,dim,vdim", SIZES)
@pytest.mark.parametrize("portions", list(PORTIONS))
def test_gated_linear(cuda, dtype, heads, dim, vdim, portions):
    g, lens, eps, tau = gen(3), [70, 3, 150, 1], 1e-5, 5.0
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    seqs = [{"q": mk(t, heads, dim), "k": mk(t, heads, dim), "v": mk(t, heads, vdim), "a": mk(t, heads * dim), "gate": mk(t, heads * vdim)} for t in lens]
    # channels that keep everything beside channels that a token or two wipe out
    bias, nw = torch.rand(heads * dim, generator=g) * 14 - 6, torch.rand(vdim, generator=g) + 0.5
    bias[::5], bias[1::7] = -400.0, 30.0
    want = []
    for s in seqs:
        x, t = {k: v.double() for k, v in s.items()}, s["q"].shape[0]
        alpha = torch.exp(plain.log_sigmoid(x["a"] + bias.double()) / tau).view(t, heads, dim)
        o = torch.stack([plain.gated_linear(x["q"][:, h] * dim ** -0.5, x["k"][:, h], x["v"][:, h], alpha[:, h])[0] for h in range(heads)], dim=1)
        want.append(plain.rms_norm(o, nw.double(), eps) * plain.silu(x["gate"]).view(t, heads, vdim))
    state = torch.full((len(lens) + 2, heads, dim, -(-vdim // 4) * 4), 3.0, device=cuda)      # leftovers of earlier owners
    got, status = [torch.empty_like(w) for w in want], ops.new_status(cuda)
    bd, nwd = bias.to(cuda), nw.to(cuda)

    def step(entries, cu, pos, slots):
        pk = packed(seqs, entries, ["q", "k", "v", "a", "gate"], cuda)
        q, k = (pk[n].unflatten(1, (heads, dim)) for n in "qk")
        out = torch.full((pos.numel(), heads, vdim), float("nan"), dtype=dtype, device=cuda)
        ops.gated_linear(q, k, pk["v"].unflatten(1, (heads, vdim)), pk["a"], bd, tau, pk["gate"], nwd, out, state, slots, cu, pos, dim ** -0.5, eps,
                         status=status)
        collect(got, entries, out)
    run_steps(cuda, lens, PORTIONS[portions], step)
    ops.check_status(status)
    assert max(rel(x, y) for x, y in zip(got, want)) < (2e-2 if dtype == BF else 1e-4)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,dim,vdim", SIZES)
@pytest.mark.parametrize("portions", list(PORTIONS))
@pytest.mark.parametrize("cap,swing", [(15.0, 3.0), (90.0, 60.0), (1.0, 1.0)])
def test_mlstm(cuda, dtype, heads, dim, vdim, portions, cap, swing):
    """swing 60 under a cap of 90: exponents whose unscaled exponentials leave fp32."""
    g, lens, eps = gen(4), [70, 3, 150, 1], 1e-5
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    seqs = [{"q": mk(t, heads, dim), "k": mk(t, heads, dim), "v": mk(t, heads, vdim), "f": mk(t, heads) * swing, "i": mk(t, heads) * swing,
             "gate": mk(t, heads * vdim)} for t in lens]
    fb, ib, nw = torch.rand(heads, generator=g) * 6, torch.rand(heads, generator=g) * 4 - 3, torch.rand(heads * vdim, generator=g) + 0.5
    want = []
    for s in seqs:
        x, t = {k: v.double() for k, v in s.items()}, s["q"].shape[0]
        i, f = plain.soft_cap(x["i"] + ib.double(), cap), plain.log_sigmoid(plain.soft_cap(x["f"] + fb.double(), cap))
        o = torch.stack([plain.mlstm_memory(x["q"][:, h] * dim ** -0.5, x["k"][:, h], x["v"][:, h], i[:, h], f[:, h])[0] for h in range(heads)], dim=1)
        want.append((plain.rms_norm(o, None, eps).flatten(1) * nw.double() * torch.sigmoid(x["gate"])).view(t, heads, vdim))
    n = len(lens) + 2
    states = (torch.full((n, heads, dim, -(-vdim // 4) * 4), 3.0, device=cuda), torch.full((n, heads, dim), 2.0, device=cuda),
              torch.full((n, heads), 9.0, device=cuda))
    got, status = [torch.empty_like(w) for w in want], ops.new_status(cuda)
    fbd, ibd, nwd = fb.to(cuda), ib.to(cuda), nw.to(cuda)

    def step(entries, cu, pos, slots):
        pk = packed(seqs, entries, ["q", "k", "v", "f", "i", "gate"], cuda)
        q, k = (pk[n].unflatten(1, (heads, dim)) for n in "qk")
        out = torch.full((pos.numel(), heads, vdim), float("nan"), dtype=dtype, device=cuda)
        ops.mlstm(q, k, pk["v"].unflatten(1, (heads, vdim)), pk["f"], fbd, pk["i"], ibd, cap, pk["gate"], nwd, out, states, slots, cu, pos,
                  dim ** -0.5, eps, status=status)
        collect(got, entries, out)
    run_steps(cuda, lens, PORTIONS[portions], step)
    ops.check_status(status)
    # a head whose o is all but zero (a denominator of e^{-m}, far above the memory) is scaled up by its norm
    assert max(rel(x, y) for x, y in zip(got, want)) < (3e-2 if dtype == BF else 1e-3 if swing > 10 else 3e-4)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_mlstm_denominator_floor_and_sign(cuda, dtype):
    """One key, three queries: n . q far above the floor, far below it (o is then o's numerator times e^m), and negative."""
    d = 8
    q = torch.zeros(3, 1, d)
    q[:, 0, 0] = torch.tensor([64.0, 1e-3, -64.0])
    k, v = torch.zeros(3, 1, d), torch.zeros(3, 1, d)
    k[0, 0, 0], v[0, 0, :2] = 1.0, torch.tensor([2.0, -1.0])
    f, i = torch.full((3, 1), 50.0), torch.tensor([[-2.0], [-40.0], [-40.0]])
    out, zero = torch.empty(3, 1, d, dtype=dtype, device=cuda), torch.zeros(1, device=cuda)
    x = [t.to(dtype).to(cuda) for t in (q, k, v, f, i)]
    ops.mlstm(*x[:3], x[3], zero, x[4], zero, 1e4, torch.full((3, d), 40.0, dtype=dtype, device=cuda), torch.ones(d, device=cuda), out, None, None,
              torch.tensor([0, 3], dtype=torch.int32, device=cuda), torch.arange(3, device=cuda), 1.0, 1.0)
    # eps 1 in the norm keeps the size of o visible
    o, _ = plain.mlstm_memory(x[0].double().cpu()[:, 0], x[1].double().cpu()[:, 0], x[2].double().cpu()[:, 0], i[:, 0].double(),
                              plain.log_sigmoid(f[:, 0].double()))
    want = plain.rms_norm(o, None, 1.0)
    assert want[0, 0] > 0.9 and want[2, 0] < -0.9 and abs(float(want[1, 0])) < 0.01
    for t in range(3):
        assert rel(out[t, 0], want[t]) < (1e-2 if dtype == BF else 1e-5)


# ---- streams, norms, activation -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width,groups", [(72, 3), (30, 1), (30, 5), (160, 20), (2048, 8), (5000, 4), (64, 64)])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 7, 16])
def test_hyper_streams(cuda, dtype, width, groups, streams):
    g, rows, eps = gen(7), 9, 1e-5
    X, y = torch.randn(rows, streams, width, generator=g), torch.randn(rows, width, generator=g).to(dtype)
    X[:, :, :width // groups] *= 30                                              # groups of very different size
    mix, wo, wi = torch.randn(streams, streams, generator=g), torch.randn(streams, generator=g), torch.randn(streams, generator=g)
    w, tol = (torch.rand(width, generator=g) + 0.5).to(dtype), 1e-2 if dtype == BF else 2e-5
    dev = [t.to(cuda) for t in (mix, wo, wi, w)]
    new = plain.connect_out(X.double().transpose(0, 1), y.double(), mix.double(), wo.double())
    h = plain.rms_norm(plain.connect_in(new, wi.double()), w.double(), eps, groups)
    xd = X.to(cuda)
    out = ops.hyper_norm(xd, y.to(cuda), *dev, eps, groups)
    assert rel(xd.transpose(0, 1), new) < 1e-5 and rel(out, h) < tol
    xd = X.to(cuda)
    ends = torch.tensor([0, 3, 4, 9], dtype=torch.int32, device=cuda)
    out = ops.hyper_norm(xd, y.to(cuda), dev[0], dev[1], None, dev[3], eps, groups, row_ends=ends)
    assert torch.equal(xd.cpu(), X) and rel(out, plain.rms_norm(new.sum(0), w.double(), eps, groups)[[2, 3, 8]]) < tol
    assert ops.hyper_norm(xd, y.to(cuda), dev[0], dev[1], None, dev[3], eps, groups, row_ends=ends[:1]).shape == (0, width)
    table, pos, ids, at = (torch.randn(50, width, generator=g).to(dtype), torch.randn(40, width, generator=g).to(dtype),
                           torch.tensor([0, 49, 7, 7]), torch.tensor([39, 0, 5, 6]))
    x0, h0 = ops.hyper_embed_norm(ids.to(cuda), at.to(cuda), table.to(cuda), pos.to(cuda), streams, dev[2], dev[3], eps, groups)
    first = table[ids].float() + pos[at].float()
    assert all(torch.equal(x0[:, s].cpu(), first) for s in range(streams))
    u = first.double() * wi.double().sum()
    assert rel(h0, plain.rms_norm(u, w.double(), eps, groups)) < max(tol, 1e-3)   # (the weights' sum may cancel)


def test_positions_outside_the_table_are_reported(cuda):
    status, w = ops.new_status(cuda), torch.ones(8, device=cuda)
    ops.hyper_embed_norm(torch.tensor([1], device=cuda), torch.tensor([4], device=cuda), torch.zeros(3, 8, device=cuda), torch.zeros(4, 8, device=cuda), 2,
                         torch.ones(2, device=cuda), w, 1e-5, 1, status=status)
    with pytest.raises(Exception, match="position"):
        ops.check_status(status)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("cols,pad", [(56, 56), (30, 32), (1, 8), (384, 384), (9216, 9216)])
def test_poly_norm(cuda, dtype, cols, pad):
    z = (torch.randn(7, pad, generator=gen(8)) * 2).to(dtype)
    z[1] *= 1e-4                                                                  # eps is of the row's own size here
    z[2] *= 1e4
    act = torch.tensor([0.6, -0.4, 0.3, 0.25])
    out = ops.poly_norm(z.to(cuda), cols, act.to(cuda), 1e-6)
    want = plain.poly_norm(z[:, :cols].double(), act.double(), 1e-6)
    assert max(rel(out[t, :cols], want[t]) for t in range(7)) < (1e-2 if dtype == BF else 1e-5)
    assert (out[:, cols:] == 0).all()


# ---- latents --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("qr,qp,kr,kp", [(36, 40, 50, 64), (96, 96, 128, 128), (5, 8, 4, 8), (1536, 1536, 512, 512)])
def test_latent_norms_write_and_gather(cuda, dtype, qr, qp, kr, kp):
    g, lens, bs, eps = gen(9), [150, 1, 37], 128, 1e-5
    t = sum(lens)
    q, c = torch.randn(t, qr, generator=g).to(dtype), (torch.randn(t, kr, generator=g) * 4).to(dtype)
    qw, cw = (torch.rand(qr, generator=g) + 0.5).to(dtype), (torch.rand(kr, generator=g) + 0.5).to(dtype)
    table = torch.tensor([[4, 1], [3, -1], [0, -1]], dtype=torch.int32)
    slots = torch.cat([torch.tensor([int(table[s, j // bs]) * bs + j % bs for j in range(n)]) for s, n in enumerate(lens)]).int()
    cache, status = torch.full((5, bs, kp), float("nan"), dtype=dtype, device=cuda), ops.new_status(cuda)
    wide = torch.cat([q, torch.zeros(t, 3, dtype=dtype), c], dim=1).to(cuda)
    qo, co = ops.latent_norm(wide[:, :qr], qw.to(cuda), qp, wide[:, qr + 3:], cw.to(cuda), kp, eps, cache, slots.to(cuda), status=status)
    tol = 1e-2 if dtype == BF else 1e-5
    assert rel(qo[:, :qr], plain.rms_norm(q.double(), qw.double(), eps)) < tol and (qo[:, qr:] == 0).all()
    assert rel(co[:, :kr], plain.rms_norm(c.double(), cw.double(), eps)) < tol and (co[:, kr:] == 0).all()
    assert torch.equal(cache.view(-1, kp)[slots.long().to(cuda)], co)
    assert torch.isnan(cache).sum() == (5 * bs - t) * kp                         # nothing else was written
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=cuda)
    assert torch.equal(ops.gather_latents(cache, table.to(cuda), cu, t, status=status), co)
    same, none = ops.latent_norm(wide[:, :qr], qw.to(cuda), qp, None, None, 0, eps)
    assert torch.equal(same, qo) and none is None
    ops.check_status(status)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("cols", [120, 30, 2048])
def test_output_gate(cuda, dtype, cols):
    o, z = torch.randn(9, cols, generator=gen(10)).to(dtype), (torch.randn(9, cols + 8, generator=gen(11)) * 8).to(dtype)
    z[0, 0], z[0, 1] = 200.0, -200.0
    out = ops.gate_mul(o.to(cuda), z.to(cuda)[:, 8:], torch.empty(9, cols, dtype=dtype, device=cuda))
    assert rel(out, o.double() * torch.sigmoid(z[:, 8:].double())) < (1e-2 if dtype == BF else 1e-6)


def latent_case(g, lens, heads, width, bs, cuda, far=None):
    """Queries [heads, B, width], a pool whose unused rows are NaN, its table, and the answers; ``far``: this many tokens from the start
    one key is made to win every softmax."""
    nblk = [-(-n // bs) for n in lens]
    order = torch.randperm(sum(nblk), generator=g).tolist()
    table = torch.full((len(lens), max(max(nblk), 1)), -1, dtype=torch.int32)
    pool, at, scale = torch.full((max(sum(nblk), 1), bs, width), float("nan"), dtype=BF), 0, width ** -0.5
    q, want = torch.randn(heads, len(lens), width, generator=g).to(BF), torch.zeros(heads, len(lens), width, dtype=torch.float64)
    for i, n in enumerate(lens):
        c = torch.randn(n, width, generator=g)
        if far is not None and n > far:
            u = q[:, i].float().mean(0)
            q[:, i] = (q[:, i].float() + 2 * u / u.norm() * width ** 0.5).to(BF)
            c[far] = u / u.norm() * width ** 0.5
        c = c.to(BF)
        for j in range(nblk[i]):
            table[i, j] = order[at]
            pool[order[at], :min(bs, n - j * bs)] = c[j * bs:(j + 1) * bs]
            at += 1
        if n:
            s = q[:, i].double() @ c.double().T * scale
            want[:, i] = torch.softmax(s, dim=-1) @ c.double()
    return q.to(cuda), pool.to(cuda), table.to(cuda), torch.tensor(lens, dtype=torch.int32, device=cuda), scale, want


@pytest.mark.parametrize("width", ops.LATENT_WIDTHS)
@pytest.mark.parametrize("heads", [1, 8, 16, 17, 33, 64])
@pytest.mark.parametrize("lens", [[1, 63, 64, 65, 0, 128, 300, 2], [2000], [700, 5, 1500, 0, 130]])
def test_latent_decode(cuda, width, heads, lens):
    for far in (None, 0, 61):
        q, pool, table, n, scale, want = latent_case(gen(heads + width), lens, heads, width, 128, cuda, far)
        ws, status = ops.decode_workspace(len(lens), heads, width, cuda), ops.new_status(cuda)
        for _ in range(2):                                                       # the second call finds its counters as the first left them
            ops.latent_decode_plan(n, table, 128, heads, width, ws)
            out = ops.latent_decode(q, pool, n, table, scale, ws, status=status)
            assert rel(out, want) < 1.5e-2
        ops.check_status(status)
        again = ops.latent_decode(q, pool, n, table, scale, ws, status=status)
        assert torch.equal(again, out)
        pos = (n - 1).clamp(min=0).long()
        got = ops.any_attn(q.transpose(0, 1).contiguous(), pool.unsqueeze(2), pool.unsqueeze(2), pos, scale, block_table=table, cache_seqlens=n)
        assert rel(got.transpose(0, 1), want) < 1e-2


def test_latent_decode_of_many_unequal_sequences(cuda):
    """Some sequences split over CTAs, some not, at once; each row as if it were alone."""
    g = gen(21)
    lens = [int(x) for x in torch.randint(1, 900, (100,), generator=g)] + [5000]
    q, pool, table, n, scale, want = latent_case(g, lens, 16, 192, 256, cuda)
    ws = ops.decode_workspace(len(lens), 16, 192, cuda)
    ops.latent_decode_plan(n, table, 256, 16, 192, ws)
    out = ops.latent_decode(q, pool, n, table, scale, ws)
    assert rel(out, want) < 1.5e-2
    for i in (0, 57, 100):
        ws1 = ops.decode_workspace(1, 16, 192, cuda)
        ops.latent_decode_plan(n[i:i + 1].contiguous(), table[i:i + 1], 256, 16, 192, ws1)
        alone = ops.latent_decode(q[:, i:i + 1].contiguous(), pool, n[i:i + 1].contiguous(), table[i:i + 1], scale, ws1)
        assert rel(alone[:, 0], out[:, i].cpu()) < 1e-2


def test_latent_decode_refuses_what_it_does_not_know(cuda):
    q, pool, table, n, scale, _ = latent_case(gen(1), [5], 2, 64, 128, cuda)
    ws = ops.decode_workspace(1, 2, 96, cuda)
    with pytest.raises(Exception, match="unsupported"):
        ops.latent_decode(torch.zeros(2, 1, 96, dtype=BF, device=cuda), torch.zeros(1, 128, 96, dtype=BF, device=cuda), n, table, scale, ws)
    status = ops.new_status(cuda)
    bad = torch.full_like(table, 99)
    ops.latent_decode_plan(n, bad, 128, 2, 64, ws)
    ops.latent_decode(q, pool, n, bad, scale, ws, status=status)                 # the block is not in the pool: zeros, and a report
    with pytest.raises(Exception, match="block"):
        ops.check_status(status)
