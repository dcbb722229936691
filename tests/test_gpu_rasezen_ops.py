"""The kernels of the Rasezen design, each against the plain oracle: the state-space recurrence in whole prompts, portions and single
tokens, the norm behind its gate, row and value norms with the rotation and the cache write, xIELU, corrected softmax routing with identity
experts, and the residual update that adds a token's own row."""
import math

import pytest
import torch

from mini_vllm_b200 import ops
from mini_vllm_b200.models.layers.rotary import build_cos_sin_cache
from oracle import rasezen as plain
from tests.step_helpers import PORTIONS, gen, rel, run_steps

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


# ---- state space ---------------------------------------------------------------------------------------------------
def run_state_space(cuda, seqs, heads, dt_bias, a, d, portions, dtype, slots=True):
    """The sequences' outputs through the kernel, fed in portions over uncleared slots."""
    n, vdim = seqs[0]["b"].shape[2], seqs[0]["x"].shape[2]
    state = torch.full((len(seqs) + 2, heads, n, -(-vdim // 4) * 4), 3.0, device=cuda) if slots else None      # leftovers of earlier owners
    got, status = [torch.full(s["x"].shape, math.nan, dtype=torch.float64) for s in seqs], ops.new_status(cuda)
    consts = [t.float().to(cuda) for t in (dt_bias, a / math.log(2.0), d)]

    def step(entries, cu, pos, slot):
        flat = [torch.cat([seqs[i][k][lo:hi] for i, lo, hi in entries]).flatten(1) for k in ("x", "b", "c", "dt")]
        pad = [-(-f.shape[1] // 8) * 8 for f in flat]                # blocks of a packed projection start at multiples of 8
        wide = torch.cat([torch.nn.functional.pad(f, (0, p - f.shape[1])) for f, p in zip(flat, pad)], dim=1).to(cuda)
        x, b, c, dt = (v[:, :f.shape[1]] for v, f in zip(wide.split(pad, dim=1), flat))
        out = torch.full((pos.numel(), pad[0]), math.nan, dtype=dtype, device=cuda)[:, :flat[0].shape[1]].unflatten(1, (heads, vdim))
        ops.state_space(x.unflatten(1, (heads, vdim)), *(t.unflatten(1, (-1, n)) for t in (b, c)), dt, *consts, out, state, slot if slots else None,
                        cu, pos, longest=max(hi - lo for _, lo, hi in entries) if cu is not None else 0, status=status)
        at = 0
        for i, lo, hi in entries:
            got[i][lo:hi] = out[at:at + hi - lo].double().cpu()
            at += hi - lo
    run_steps(cuda, [s["x"].shape[0] for s in seqs], PORTIONS[portions] if isinstance(portions, str) else portions, step)
    ops.check_status(status)
    return got


def want_state_space(s, dt_bias, a, d):
    x = {k: v.double() for k, v in s.items()}
    return plain.state_space(x["x"], x["b"], x["c"], plain.softplus(x["dt"] + dt_bias.double()), a.double(), d.double())


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,groups,n,vdim", [(4, 2, 16, 16), (3, 3, 20, 12), (4, 1, 128, 64), (2, 1, 56, 32), (5, 1, 7, 9), (2, 2, 256, 40),
                                                 (1, 1, 1, 1), (6, 2, 64, 136), (80, 8, 24, 56), (2, 1, 180, 72)])
@pytest.mark.parametrize("portions", list(PORTIONS))
def test_state_space(cuda, dtype, heads, groups, n, vdim, portions):
    g = gen(heads + n)
    lens = [70, 3, 150, 1] if heads < 50 else [70, 1, 129]
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    seqs = [{"x": mk(t, heads, vdim), "b": mk(t, groups, n), "c": mk(t, groups, n), "dt": mk(t, heads)} for t in lens]
    # heads that keep everything beside heads that a token or two wipe out
    dt_bias, a, d = torch.rand(heads, generator=g) * 5 - 4, -torch.exp(torch.rand(heads, generator=g) * 6 - 4), torch.randn(heads, generator=g)
    got = run_state_space(cuda, seqs, heads, dt_bias, a, d, portions, dtype)
    for x, s in zip(got, seqs):
        assert rel(x, want_state_space(s, dt_bias, a, d)) < (6e-3 if dtype == BF else 2e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dt_bias,log_a", [(-30.0, 0.0), (40.0, 3.0), (0.0, -20.0), (5.0, -4.0), (-6.0, 5.0)])
def test_state_space_at_its_extremes(cuda, dtype, dt_bias, log_a):
    """Steps of nothing, decays to zero within a token (exponents far below what fp32 holds), and memories that lose nothing."""
    g, heads = gen(5), 2
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    seqs = [{"x": mk(t, heads, 40), "b": mk(t, 1, 24), "c": mk(t, 1, 24), "dt": mk(t, heads)} for t in (200, 65)]
    bias, a, d = torch.full((heads,), dt_bias), torch.full((heads,), -math.exp(log_a)), torch.tensor([0.0, 1.0])
    for portions in ("whole", "single", "long"):
        for x, s in zip(run_state_space(cuda, seqs, heads, bias, a, d, portions, dtype), seqs):
            want = want_state_space(s, bias, a, d)
            assert torch.isfinite(x).all() and rel(x, want) < (6e-3 if dtype == BF else 2e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("at", [0, 1, 15, 16, 62, 63, 64, 65, 127, 128, 190])
def test_a_remembered_token(cuda, dtype, at):
    """One token writes along a direction of its own, the later ones elsewhere; the last token asks for it.  Its place takes every side of
    a chunk's edge, in whole prompts and in portions that cut there."""
    g, n, vdim, t = gen(at), 32, 16, 200
    x, b, c = torch.randn(t, 1, vdim, generator=g) * 0.1, torch.zeros(t, 1, n), torch.zeros(t, 1, n)
    b[:, 0, 1:] = torch.randn(t, n - 1, generator=g)
    b[at], x[at] = torch.eye(n)[:1], torch.linspace(1, 2, vdim)
    c[192:, 0, 0] = 1.0                                              # the queries at the end see that direction alone
    s = {"x": x.to(dtype), "b": b.to(dtype), "c": c.to(dtype), "dt": torch.zeros(t, 1, dtype=dtype)}
    bias, a, d = torch.tensor([-3.0]), torch.tensor([-0.05]), torch.tensor([0.0])
    want = want_state_space(s, bias, a, d)
    assert want[192:].abs().min() > 0.02
    for portions in ([[10 ** 6]], [[max(at, 1), 1, 2]], [[at + 1, 63]], [[1]]):
        got = run_state_space(cuda, [s], 1, bias, a, d, portions, dtype)[0]
        assert rel(got[192:], want[192:]) < (5e-3 if dtype == BF else 1e-5)


@pytest.mark.parametrize("heads,groups,n,vdim", [(2, 1, 16, 16), (3, 1, 40, 72), (2, 2, 128, 24)])
@pytest.mark.parametrize("portions,slots", [([[10 ** 6]], True), ([[10 ** 6]], False), ([[1100, 64, 300], [70, 1], [1], [1200]], True)])
def test_long_sequences_in_segments(cuda, heads, groups, n, vdim, portions, slots):
    """Long sequences beside short ones are cut into segments that are walked at once: the same outputs, and the same state for what
    follows, as one by one."""
    from mini_vllm_b200 import _cabi
    g, lens = gen(n), [1500, 71, 1, 1290]
    assert _cabi.load().mvb_state_space_scratch_bytes(0, sum(lens), len(lens), max(lens), heads, n, vdim, 1) > 0
    mk = lambda *s: torch.randn(*s, generator=g).to(BF)
    seqs = [{"x": mk(t, heads, vdim), "b": mk(t, groups, n), "c": mk(t, groups, n), "dt": mk(t, heads)} for t in lens]
    dt_bias, a, d = torch.full((heads,), -3.0), -torch.exp(torch.linspace(-9, 1, heads)), torch.ones(heads)      # from long memories to short
    for x, s in zip(run_state_space(cuda, seqs, heads, dt_bias, a, d, portions, BF, slots=slots), seqs):
        assert rel(x, want_state_space(s, dt_bias, a, d)) < 6e-3


@pytest.mark.parametrize("dtype", [BF, F32])
def test_state_space_without_state(cuda, dtype):
    """No slots (a step of prompts that nobody continues): every sequence starts from zero and nothing is kept."""
    g = gen(8)
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    seqs = [{"x": mk(t, 2, 24), "b": mk(t, 1, 16), "c": mk(t, 1, 16), "dt": mk(t, 2)} for t in (90, 2)]
    bias, a, d = torch.zeros(2), torch.tensor([-0.3, -2.0]), torch.ones(2)
    for x, s in zip(run_state_space(cuda, seqs, 2, bias, a, d, "whole", dtype, slots=False), seqs):
        assert rel(x, want_state_space(s, bias, a, d)) < (6e-3 if dtype == BF else 2e-5)


def test_state_space_refuses_what_it_does_not_know(cuda):
    from mini_vllm_b200._cabi import KernelError
    z = lambda *s: torch.zeros(*s, dtype=BF, device=cuda)
    one = torch.ones(2, device=cuda)
    with pytest.raises(KernelError):
        ops.state_space(z(1, 2, 8), z(1, 1, 264), z(1, 1, 264), z(1, 2), one, -one, one, z(1, 2, 8), None, None, None,
                        torch.zeros(1, dtype=torch.int64, device=cuda))


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width,groups", [(1, 1), (72, 4), (96, 1), (256, 2), (1000, 5), (4096, 1), (4096, 8), (24, 24), (9000, 1), (3000, 2)])
def test_gated_group_norm(cuda, dtype, width, groups):
    g, rows, eps = gen(width), 19, 1e-2
    y, z = ((torch.randn(rows, width, generator=g) * s).to(dtype) for s in (1.0, 3.0))
    y[3], z[4] = 0, -90.0
    w = torch.randn(width, generator=g)
    want = plain.gated_group_norm(y.double(), z.double(), w.double(), groups, eps)
    zd = torch.nn.functional.pad(z, (0, 8)).to(cuda)[:, :width]
    out = torch.empty(rows, width + 8, dtype=dtype, device=cuda)[:, :width]
    got = ops.gated_group_norm(y.to(cuda), zd, w.to(cuda), out, groups, eps)
    assert rel(got, want) < (6e-3 if dtype == BF else 1e-5)


# ---- row and value norms with the rotation ----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,vdim,rot,d,hq,hkv", [(44, 44, 44, 128, 3, 1), (100, 60, 20, 128, 6, 3), (128, 128, 128, 128, 16, 8), (200, 130, 64, 256, 5, 5),
                                                   (40, 48, 8, 48, 4, 2), (264, 264, 264, 272, 2, 1), (1, 1, 0, 16, 1, 1), (128, 128, 64, 128, 96, 32)])
@pytest.mark.parametrize("form", ["both", "rows", "values"])
def test_row_norm_rotation_and_write(cuda, dtype, dim, vdim, rot, d, hq, hkv, form):
    """Padded heads: the cache and the rows hold what the plain norms and rotation give; the mean runs over used coordinates only."""
    g, t, eps = gen(dim), 21, 1e-2
    r, half = rot // 2, d // 2
    free = [j for j in range(d) if not (j < r or half <= j < half + r)]
    place = torch.tensor(list(range(r)) + [half + i for i in range(r)] + free[:dim - rot])
    mk = lambda *s: torch.randn(*s, generator=g).to(dtype)
    q, k, v, qw, kw = mk(t, hq, dim) * 3, mk(t, hkv, dim), mk(t, hkv, vdim) * 5, mk(hq, dim) + 1, mk(hkv, dim) - 1
    turn = lambda x, w: plain.rotate_half((plain.over_rms(x.double().flatten(1), eps) * w.double().flatten()).view(x.shape) if form != "values" else x.double(),
                                          rot, 700.0)
    want_q, want_k, want_v = turn(q, qw), turn(k, kw), plain.over_rms(v.double(), eps) if form != "rows" else v.double()

    def padded(x, at):
        out = torch.zeros(*x.shape[:-1], d, dtype=dtype)
        out[..., at] = x
        return out.to(cuda)
    vplace = torch.arange(vdim)
    weights = (padded(qw, place).flatten(), padded(kw, place).flatten()) if form != "values" else (None, None)
    norm = ops.RowNorm(*weights, hq * dim, hkv * dim, vdim if form != "rows" else 0, eps)
    table = build_cos_sin_cache(rot, 64, 700.0, head_dim=d).to(cuda) if rot else None
    slots = (torch.arange(t) * 2 + 1).to(torch.int32)
    slots[4] = -1
    used, tol = slots >= 0, 1e-2 if dtype == BF else 1e-5
    for in_place in (True, False):
        packed = torch.cat([padded(q, place), padded(k, place), padded(v, vplace), torch.ones(t, 1, d, dtype=dtype, device=cuda)], dim=1)
        qd, kd, vd = packed[:, :hq], packed[:, hq:hq + hkv], packed[:, hq + hkv:hq + 2 * hkv]
        kc, vc = (torch.zeros(3, 16, hkv, d, dtype=dtype, device=cuda) for _ in range(2))
        status = ops.new_status(cuda)
        ops.row_norm_rope_kv_write(qd, kd, vd, norm, torch.arange(t, device=cuda), table, slots.to(cuda), kc, vc, kv_in_place=in_place, status=status)
        ops.check_status(status)
        assert rel(qd[:, :, place.to(cuda)], want_q) < tol
        assert rel(kd[:, :, place.to(cuda)], want_k if in_place else k.double()) < tol
        assert rel(vd[:, :, :vdim], want_v if in_place else v.double()) < tol
        assert (packed[:, -1] == 1).all() and (vd[:, :, vdim:] == 0).all()
        rows = slots[used].long().to(cuda)
        assert rel(kc.view(-1, hkv, d)[rows][:, :, place.to(cuda)], want_k[used]) < tol
        assert rel(vc.view(-1, hkv, d)[rows][:, :, :vdim], want_v[used]) < tol
        others = torch.ones(48, dtype=torch.bool, device=cuda)
        others[rows] = False
        assert (kc.view(48, -1)[others] == 0).all() and (vc.view(48, -1)[others] == 0).all()


def test_positions_outside_the_table_are_reported(cuda):
    from mini_vllm_b200._cabi import KernelError
    x = lambda h: torch.ones(2, h, 128, dtype=BF, device=cuda)
    status, table = ops.new_status(cuda), build_cos_sin_cache(128, 4, 700.0, head_dim=128).to(cuda)
    ops.row_norm_rope_kv_write(x(2), x(1), x(1), ops.RowNorm(None, None, 256, 128, 0, 1e-5), torch.tensor([1, 4], device=cuda), table, None, None, None,
                               status=status)
    with pytest.raises(KernelError, match="position"):
        ops.check_status(status)


# ---- feed-forwards -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("cols", [8, 33, 1000, 5000])
def test_xielu(cuda, dtype, cols):
    g = gen(cols)
    z = (torch.randn(11, cols, generator=g) * torch.logspace(-4, 1, 11)[:, None]).to(dtype)
    z[0, :8] = torch.tensor([0.0, -0.25, -0.2501, 0.25, -80.0, 30.0, -1e-6, 1e-6])
    p, q = torch.tensor(-0.7, dtype=torch.float64), torch.tensor(1.1, dtype=torch.float64)
    act = torch.stack([plain.softplus(p), 0.5 + plain.softplus(q)]).float().to(cuda)
    out = torch.full((11, cols + 8), math.nan, dtype=dtype, device=cuda)
    got = ops.xielu(z.to(cuda), act, out=out[:, :cols]).double().cpu()
    want = plain.xielu(z.double(), p, q)
    assert ((got - want).abs() <= (4e-3 if dtype == BF else 1e-6) * (want.abs() + z.double().abs())).all()
    assert torch.isnan(out[:, cols:]).all()


def expert_feed(cuda, dtype, w, *args, **kw):
    from mini_vllm_b200.models.layers.feedforward import ExpertFeed
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        with torch.device(cuda):
            feed = ExpertFeed(*args, **kw)
    finally:
        torch.set_default_dtype(prev)
    feed.load(lambda n: w[n].to(cuda))
    return feed


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("tokens,experts,identity,top,width,inter", [
    (1, 1, 1, 1, 64, 8), (1, 8, 2, 10, 72, 40), (7, 33, 4, 4, 30, 17), (300, 5, 0, 1, 200, 96), (513, 12, 5, 3, 136, 136), (64, 300, 30, 6, 64, 24),
    (700, 4, 28, 2, 64, 100), (40, 1, 40, 3, 256, 130)])
def test_experts_with_identity(cuda, dtype, tokens, experts, identity, top, width, inter):
    """Corrected softmax scores choose, plain ones weigh; identity experts give the token's own row; the stream gets it all."""
    g, scale, outputs = gen(tokens + experts), 1.6, experts + identity
    h = torch.randn(tokens, width, generator=g).to(dtype)
    w = {"router": (torch.randn(outputs, width, generator=g) * 2 * width ** -0.5).to(dtype), "correction": torch.randn(outputs, generator=g) * 0.3}
    for e in range(experts):
        w.update({f"e{e}.gate": (torch.randn(inter, width, generator=g) * 2 * width ** -0.5).to(dtype),
                  f"e{e}.up": (torch.randn(inter, width, generator=g) * 2 * width ** -0.5).to(dtype),
                  f"e{e}.down": (torch.randn(width, inter, generator=g) * inter ** -0.5).to(dtype)})
    wd = {k: v.double() for k, v in w.items()}
    m = {"router": {"experts": experts, "identity": identity, "top": top, "scale": scale}, "expert": {"ff": inter}}
    want = plain.experts(h.double(), wd, "", m)
    feed = expert_feed(cuda, dtype, w, width, inter, experts, top, softmax=True, corrected=True, scale=scale, weigh_output=True, identity=identity)
    status, hd = ops.new_status(cuda), h.to(cuda)
    x0, y = torch.randn(tokens, width, generator=g), torch.randn(tokens, width, generator=g).to(dtype)
    for _ in range(3):                                               # later calls find the counters as the first left them
        r = feed.routed(hd, status)
        taken = r.slots[r.slots >= 0]
        assert sorted(taken.tolist()) == list(range(taken.numel()))
        x, ones = x0.to(cuda), torch.ones(width, dtype=dtype, device=cuda)
        ops.residual_norm_pair(x, y.to(cuda), ones, None, 1e-5, r.rows, r.slots, own=r.own, own_weights=r.own_weights, status=status)
        assert rel(x.double().cpu() - x0.double() - y.double(), want) < (2e-2 if dtype == BF else 2e-5)
    ops.check_status(status)
    assert int(feed.counters.abs().sum()) == 0


@pytest.mark.parametrize("softmax", [True, False])
def test_the_correction_moves_the_choice_and_not_the_weight(cuda, softmax):
    logits = torch.tensor([[3.0, 2.0, 1.0, 0.0, -1.0], [0.0, 0.0, 0.0, 5.0, 9.0]], device=cuda)
    h, counters = torch.ones(2, 8, device=cuda), torch.zeros(4, dtype=torch.int32, device=cuda)
    score = torch.softmax(logits, -1) if softmax else torch.sigmoid(logits)
    correction = torch.tensor([-3.0, 0.0, 0.0, 2.0, 1.0], device=cuda)
    _, rows = ops.moe_sort(h, logits, 2, counters, ops.Routing(softmax, correction, 2.0, 2))      # experts 0..2, identity 3 and 4
    assert (rows.slots == -1).all()
    assert torch.allclose(rows.identity, 2 * (score[:, 3] + score[:, 4]), rtol=1e-6)
    _, rows = ops.moe_sort(h, logits, 2, counters, ops.Routing(softmax, None, 1.0, 2))
    assert (rows.slots[0] >= 0).all() and rows.identity[0] == 0
    assert torch.allclose(rows.weights[rows.slots[0].long()], score[0, :2], rtol=1e-6)


def test_experts_in_a_graph_follow_the_tokens(cuda):
    """Group sizes and identity choices are data: the captured products follow another routing at every replay."""
    g, width, inter, experts, top, n = gen(2), 128, 64, 6, 2, 48
    w = {"router": torch.randn(experts + 2, width, generator=g) * width ** -0.5, "correction": torch.zeros(experts + 2)}
    for e in range(experts):
        w.update({f"e{e}.gate": torch.randn(inter, width, generator=g) * width ** -0.5, f"e{e}.up": torch.randn(inter, width, generator=g) * width ** -0.5,
                  f"e{e}.down": torch.randn(width, inter, generator=g) * inter ** -0.5})
    feed = expert_feed(cuda, BF, w, width, inter, experts, top, softmax=True, corrected=True, weigh_output=True, identity=2)
    h, zero, ones = torch.randn(n, width, generator=g).to(BF).to(cuda), torch.zeros(n, width, dtype=BF, device=cuda), torch.ones(width, dtype=BF, device=cuda)

    def run():
        x, r = torch.zeros(n, width, device=cuda), feed.routed(h, None)
        ops.residual_norm_pair(x, zero, ones, None, 1e-5, r.rows, r.slots, own=r.own, own_weights=r.own_weights)
        return x
    run()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        x = run()
    for k in range(5):
        h.copy_((torch.randn(n, width, generator=g) + (3 * (k % 2)) * w["router"][k + 3]).to(BF).to(cuda))
        graph.replay()
        assert torch.equal(x, run())


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width", [30, 72, 1000, 4096])
def test_own_rows_in_the_residual_update(cuda, dtype, width):
    g, rows = gen(width), 9
    mk = lambda *s: torch.randn(*s, generator=g)
    x, y, own, extra = mk(rows, width), mk(rows, width).to(dtype), mk(rows, width).to(dtype), mk(6, -(-width // 8) * 8).to(dtype)
    weights, index = mk(rows), torch.tensor([[-1, i % 6, -1] for i in range(rows)], dtype=torch.int32)
    weights[2] = 0.0
    want = x.double() + y.double() + weights.double()[:, None] * own.double() + extra[index[:, 1].long(), :width].double()
    w, xd, status = torch.full((width,), 0.5).to(dtype).to(cuda), x.to(cuda), ops.new_status(cuda)
    args = dict(extra=extra.to(cuda)[:, :width], extra_index=index.to(cuda), own=own.to(cuda), own_weights=weights.to(cuda), status=status)
    ends = torch.tensor([0, 3, rows], dtype=torch.int32, device=cuda)
    last, _ = ops.residual_norm_pair(xd, y.to(cuda), w, None, 1e-3, row_ends=ends, **args)
    norm = plain.scalar_norm(want, torch.tensor(0.5, dtype=torch.float64), 1e-3)
    tol = 1e-2 if dtype == BF else 1e-5
    assert torch.equal(xd.cpu(), x) and rel(last, norm[[2, rows - 1]]) < tol
    out, _ = ops.residual_norm_pair(xd, y.to(cuda), w, None, 1e-3, **args)
    assert rel(xd, want) < 1e-6 and rel(out, norm) < tol
    ops.check_status(status)
