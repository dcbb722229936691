"""The kernels of the Sunulorn design, each against the plain oracle: attention with sinks, kept first tokens, a bias by distance and head
gates in prompts, portions and decoding; the rotation with a norm behind it; the convolution that copies its keys; the paired norms; the
experts' routing and grouped products."""
import math

import pytest
import torch

from mini_vllm_b200 import ops
from mini_vllm_b200.models.layers.rotary import build_cos_sin_cache
from oracle import sunulorn as plain
from tests.step_helpers import PORTIONS, gen, ragged_steps, rel, run_steps

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
BS = 128                                       # tokens of a page

FORMS = {                                      # window, kept first tokens, sinks, slopes, head gate
    "sink": (None, 0, True, False, False), "distance": (None, 0, False, True, False), "all": (None, 0, True, True, True),
    "kept": (45, 25, False, False, False), "kept-page": (50, 128, True, False, True), "kept-far": (130, 300, False, False, False),
    "kept-one": (1, 1, True, True, False), "window": (129, 0, True, True, True), "gate": (None, 0, False, False, True),
}


class Case:
    """Sequences with their answers, and a pool of pages whose unused rows are NaN."""

    def __init__(self, cuda, lens, heads, kv, d, dtype, form, seed=0, planted=(), steep=False):
        g = gen(seed)
        self.cuda, self.lens, self.heads, self.kv, self.d, self.dtype = cuda, lens, heads, kv, d, dtype
        self.window, self.keep, sink, slope, gate = FORMS[form]
        self.scale = d ** -0.5
        self.sinks = torch.randn(heads, generator=g) * 2 if sink else None
        self.slopes = torch.tensor([plain.alibi_slope(h, heads) for h in range(heads)]) * (4 if steep else 1) if slope else None
        mk = lambda *s: torch.randn(*s, generator=g)
        self.seqs, self.want = [], []
        for n in lens:
            q, k, v = mk(n, heads, d), mk(n, kv, d), mk(n, kv, d)
            for j in planted:                  # a key that stands out for every query, with a value that says so
                if j < n:
                    u = mk(d)
                    u = u / u.norm() * d ** 0.5
                    q = q + 0.8 * u
                    k[j], v[j] = 1.2 * u, v[j] * 4 + 2
            s = {"q": q.to(dtype), "k": k.to(dtype), "v": v.to(dtype), "gate": mk(n, heads).to(dtype)}
            self.seqs.append(s)
            x = {a: b.double() for a, b in s.items()}
            o = plain.attention(x["q"], x["k"], x["v"], self.scale, plain.visible(n, self.window, self.keep),
                                None if self.sinks is None else self.sinks.double(), None if self.slopes is None else self.slopes.tolist())
            self.want.append(o * torch.sigmoid(x["gate"])[:, :, None] if gate else o)
        self.gated = gate
        nblk = [-(-n // BS) for n in lens]
        order = torch.randperm(sum(nblk), generator=g).tolist()
        self.table, at = torch.full((len(lens), max(nblk)), -1, dtype=torch.int32), 0
        for i, b in enumerate(nblk):
            self.table[i, :b] = torch.tensor(order[at:at + b])
            at += b
        self.pool = torch.full((2, sum(nblk), BS, kv, d), float("nan"), dtype=dtype, device=cuda)

    def extras(self, rows):
        put = lambda t: None if t is None else t.float().to(self.cuda)
        gate = torch.cat([rows, rows], dim=1).to(self.cuda)[:, :self.heads] if self.gated else None          # (a row stride of its own)
        return ops.AttnExtras(put(self.sinks), put(self.slopes), gate, self.keep)

    def store(self, i, a, e):
        for t in range(a, e):
            blk = int(self.table[i, t // BS])
            for c, n in enumerate("kv"):
                self.pool[c, blk, t % BS] = self.seqs[i][n][t].to(self.cuda)

    def run(self, portions, tensor_cores, dense=False):
        """Worst error over all rows, fed in ``portions``: prompt portions through the prefill kernel, single tokens through decode."""
        wl, cuda = -1 if self.window is None else self.window - 1, self.cuda
        status, worst = ops.new_status(cuda), 0.0
        for step in ragged_steps(self.lens, portions):
            cat = lambda n: torch.cat([self.seqs[i][n][a:e] for i, a, e in step])
            q, ex = cat("q").to(cuda), self.extras(cat("gate"))
            for i, a, e in step:
                self.store(i, a, e)
            table = self.table[[i for i, _, _ in step]].to(cuda)
            ends = torch.tensor([e for _, _, e in step], dtype=torch.int32, device=cuda)
            cu = lambda ns: torch.tensor([0] + list(torch.tensor(ns).cumsum(0)), dtype=torch.int32, device=cuda)
            pos = torch.cat([torch.arange(a, e) for _, a, e in step]).to(cuda)
            q_lens = [e - a for _, a, e in step]
            single = max(q_lens) == 1
            if not tensor_cores:
                out = ops.any_attn(q, self.pool[0], self.pool[1], pos, self.scale, wl, cu_seqlens_q=None if single else cu(q_lens),
                                   block_table=table, cache_seqlens=ends if single else None, status=status, extras=ex)
            elif single:
                ws = ops.decode_workspace(len(step), self.heads, self.d, cuda)
                ops.decode_plan(ends, wl, self.heads, self.kv, self.d, ws, block_table=table, block_size=BS, keep_first=self.keep)
                out = ops.decode_attn(q, self.pool[0], self.pool[1], ends, table, self.scale, wl, ws, status=status, extras=ex)
            else:
                kw = {"block_table": table}
                k, v = self.pool[0], self.pool[1]
                if dense:
                    kw, k, v = {}, cat("k").to(cuda), cat("v").to(cuda)
                cq, ck = cu(q_lens), cu([e for _, _, e in step])
                out = ops.prefill_attn(q, k, v, cq, ck, max(q_lens), self.scale, wl, status=status, extras=ex, **kw)
                items = ops.build_prefill_items(q_lens, [e for _, _, e in step], ops.prefill_item_rows(self.heads, self.kv, self.d))
                again = ops.prefill_attn(q, k, v, cq, ck, 10 * max(q_lens), self.scale, wl, status=status, extras=ex,
                                         items=torch.from_numpy(items).to(cuda), **kw)
                assert torch.equal(out, again)
            at = 0
            for i, a, e in step:
                worst = max(worst, rel(out[at:at + e - a], self.want[i][a:e]) if e > a else 0.0)
                at += e - a
        ops.check_status(status)
        return worst


SPLITS = {"whole": [[10 ** 6]], "twos": [[2]], "portions": [[130, 1, 70, 2], [2, 3, 128]], "single": [[127, 1, 1, 1, 1, 1, 1, 1]]}


@pytest.mark.parametrize("form", list(FORMS))
@pytest.mark.parametrize("heads,kv,d", [(4, 2, 128), (3, 3, 128), (6, 2, 256), (8, 1, 128)])
def test_attention_on_the_tensor_cores(cuda, form, heads, kv, d):
    lens = [1, 2, 65, 190, 700]
    case = Case(cuda, lens, heads, kv, d, BF, form, seed=heads)
    assert case.run(SPLITS["whole"], True, dense=True) < 2.5e-2
    for name in ("whole", "portions"):
        assert case.run(SPLITS[name], True) < 2.5e-2, name


@pytest.mark.parametrize("form", list(FORMS))
@pytest.mark.parametrize("heads,kv,d,dtype", [(4, 2, 128, BF), (3, 1, 40, F32), (18, 2, 16, BF), (2, 1, 264, F32)])
def test_attention_of_any_layout(cuda, form, heads, kv, d, dtype):
    case = Case(cuda, [1, 2, 65, 190, 430], heads, kv, d, dtype, form, seed=d)
    for name in ("whole", "portions"):
        assert case.run(SPLITS[name], False) < (1.5e-2 if dtype == BF else 2e-5), name


@pytest.mark.parametrize("form", ["kept", "kept-page", "kept-far", "window", "sink", "all"])
@pytest.mark.parametrize("planted", [(0,), (24,), (25,), (127,), (128,), (299,), (300,), (360,)])
@pytest.mark.parametrize("tensor_cores", [True, False])
def test_a_key_that_stands_out(cuda, form, planted, tensor_cores):
    """It decides the output of every row that sees it and of no other: at the kept tokens' end, at page borders, and where it falls out of the
    window while tokens are decoded one by one."""
    case = Case(cuda, [470], 4, 2, 128, BF, form, seed=7, planted=planted)
    for portions in ([[10 ** 6]], [[planted[0] + 20] + [1] * 60 + [2, 130, 5]], [[100, 33, 2, 200]]):
        assert case.run(portions, tensor_cores) < 2.5e-2, portions


@pytest.mark.parametrize("form", ["distance", "all"])
def test_steep_distances(cuda, form):
    """Far keys vanish altogether, near ones stand hundreds of units above them; with and without a sink."""
    case = Case(cuda, [5, 900], 2, 2, 128, BF, form, seed=3, steep=True)
    for name in ("whole", "single"):
        assert case.run([[700] + SPLITS["single"][0]] if name == "single" else SPLITS["whole"], True) < 2.5e-2


def test_sinks_of_all_sizes(cuda):
    """From a sink that takes everything to one that takes nothing, in whole and split sequences."""
    lens = [1, 40, 3000, 2]
    for sinks in ([-1e4, -30.0, 0.0, 8.0], [40.0, 300.0, 1e4, -300.0]):
        case = Case(cuda, lens, 4, 2, 128, BF, "sink", seed=5)
        case.sinks = torch.tensor(sinks)
        for i, s in enumerate(case.seqs):
            x = {a: b.double() for a, b in s.items()}
            case.want[i] = plain.attention(x["q"], x["k"], x["v"], case.scale, plain.visible(lens[i], None, 0), case.sinks.double())
        assert all(torch.isfinite(w).all() for w in case.want)
        assert case.run([[10 ** 6]], True) < 2.5e-2
        assert case.run([[39], [39], [2999], [1]], True) < 2.5e-2 and case.run([[10 ** 6]], False) < 2.5e-2


def test_decode_of_many_unequal_sequences(cuda):
    """Windows with kept tokens whose tiles are split over many CTAs, padding rows, and each row as if it were alone."""
    g = gen(31)
    lens = [int(x) for x in torch.randint(1, 600, (90,), generator=g)] + [5000]
    case = Case(cuda, lens, 4, 2, 128, BF, "kept-far", seed=9)
    q = torch.cat([s["q"][-1:] for s in case.seqs]).to(cuda)
    for i, s in enumerate(case.seqs):
        for b in range(-(-lens[i] // BS)):
            for c, n in enumerate("kv"):
                part = s[n][b * BS:(b + 1) * BS].to(cuda)
                case.pool[c, int(case.table[i, b]), :part.shape[0]] = part
    n = torch.tensor(lens, dtype=torch.int32, device=cuda)
    n[3], table = 0, case.table.to(cuda)                             # a padding row
    wl, ex = case.window - 1, case.extras(torch.zeros(len(lens), 4, dtype=BF))

    def decode(q, n, table):
        ws = ops.decode_workspace(n.numel(), 4, 128, cuda)
        ops.decode_plan(n, wl, 4, 2, 128, ws, block_table=table, block_size=BS, keep_first=case.keep)
        return ops.decode_attn(q, case.pool[0], case.pool[1], n, table, case.scale, wl, ws, extras=ex)
    out = decode(q, n, table)
    want = torch.stack([w[-1] for w in case.want])
    want[3] = 0
    assert rel(out, want) < 2.5e-2 and out[3].abs().max() == 0
    for i in (0, 50, 90):
        assert rel(decode(q[i:i + 1], n[i:i + 1].contiguous(), table[i:i + 1]), out[i:i + 1].cpu()) < 1e-2


# ---- rotation with a norm behind it, convolution ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,rot,d", [(44, 44, 128), (100, 20, 128), (128, 128, 128), (200, 64, 256), (40, 8, 48), (264, 264, 272), (1, 0, 16)])
@pytest.mark.parametrize("norm", [True, False])
def test_rotation_and_norm(cuda, dtype, dim, rot, d, norm):
    """Padded heads (rotated pairs laid out at i and i + d/2): the cache and the rows hold what the plain rotation and norm give."""
    g, t, hq, hkv, eps = gen(dim), 37, 3, 2, 1e-2
    r, half = rot // 2, d // 2
    free = [j for j in range(d) if not (j < r or half <= j < half + r)]
    place = torch.tensor(list(range(r)) + [half + i for i in range(r)] + free[:dim - rot])
    x, v = torch.randn(t, hq + hkv, dim, generator=g).to(dtype), torch.randn(t, hkv, d, generator=g).to(dtype)
    want = plain.rotate(x.double(), rot, 700.0, False)
    want = plain.rms_norm(want, None, eps) if norm else want
    wide = torch.zeros(t, hq + hkv, d, dtype=dtype)
    wide[:, :, place] = x
    table = build_cos_sin_cache(rot, 64, 700.0, head_dim=d).to(cuda) if rot else None
    pos = torch.arange(t, device=cuda)
    slots = (torch.arange(t) * 2 + 1).to(torch.int32)
    slots[4] = -1
    for in_place in (True, False):
        packed = torch.cat([wide, torch.ones(t, 1, d, dtype=dtype)], dim=1).to(cuda)
        q, k, vd = packed[:, :hq], packed[:, hq:hq + hkv], v.to(cuda)
        kc, vc = (torch.zeros(5, 16, hkv, d, dtype=dtype, device=cuda) for _ in range(2))
        status = ops.new_status(cuda)
        ops.rope_norm_kv_write(q, k, vd, pos, table, slots.to(cuda), kc, vc, k_in_place=in_place, norm_dim=dim if norm else 0, eps=eps, status=status)
        ops.check_status(status)
        tol = 1e-2 if dtype == BF else 1e-5
        assert rel(q[:, :, place.to(cuda)], want[:, :hq]) < tol
        assert rel(k[:, :, place.to(cuda)], want[:, hq:] if in_place else x[:, hq:].double()) < tol
        used = slots >= 0
        rows = kc.view(-1, hkv, d)[slots[used].long().to(cuda)]
        assert rel(rows[:, :, place.to(cuda)], want[used, hq:]) < tol
        assert torch.equal(vc.view(-1, hkv, d)[slots[used].long().to(cuda)].cpu(), v[used])
    alone = wide[:, :hq].contiguous().to(cuda)                       # q alone: a layer with borrowed keys
    ops.rope_norm_kv_write(alone, None, None, pos, table, None, None, None, norm_dim=dim if norm else 0, eps=eps)
    assert rel(alone[:, :, place.to(cuda)], want[:, :hq]) < tol


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("taps,channels,copies", [(4, 64, 24), (3, 30, 10), (1, 16, 16), (6, 24, 0), (9, 12, 4)])
@pytest.mark.parametrize("portions", ["whole", "single", "twos", "mixed"])
def test_convolution_without_activation(cuda, dtype, taps, channels, copies, portions):
    g, lens = gen(1), [70, 3, 129, 1]
    w = torch.randn(channels, taps, generator=g).to(dtype)
    us = [torch.randn(n, channels, generator=g).to(dtype) for n in lens]
    want = [plain.causal_conv(u.double(), w.double()) for u in us]
    want = [torch.cat([y, y[:, channels - copies:]], dim=1) for y in want]
    state = torch.full((len(lens) + 2, taps - 1, channels), 7.0, dtype=dtype, device=cuda)     # leftovers of earlier owners
    wd, got = w.flip(1).T.contiguous().to(cuda), [torch.empty_like(w) for w in want]

    def step(entries, cu, pos, slots):
        out = ops.short_conv(torch.cat([us[i][a:e] for i, a, e in entries]).to(cuda), wd, None, state if taps > 1 else None, slots, cu, pos,
                             copies=copies).cpu()
        at = 0
        for i, a, e in entries:
            got[i][a:e] = out[at:at + e - a].double()
            at += e - a
    run_steps(cuda, lens, PORTIONS[portions], step)
    assert max(rel(x, y) for x, y in zip(got, want)) < (1e-2 if dtype == BF else 1e-5)


# ---- norms, gated units ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width", [30, 72, 256, 1000, 4096])
@pytest.mark.parametrize("top", [0, 1, 3])
def test_paired_norms(cuda, dtype, width, top):
    g, rows, eps = gen(width), 23, 1e-3
    mk = lambda *s: torch.randn(*s, generator=g)
    table, ids = mk(11, width).to(dtype), torch.randint(0, 11, (rows,), generator=g)
    w1, w2, y = (mk(width) + 1).to(dtype), (mk(width) + 1).to(dtype), mk(rows, width).to(dtype)
    tol = 1e-2 if dtype == BF else 1e-5
    x, a, b = ops.embed_norm_pair(ids.to(cuda), table.to(cuda), 2.7, w1.to(cuda), w2.to(cuda), eps)
    want = table[ids].double() * 2.7
    assert rel(x, want) < 1e-6 and rel(a, plain.rms_norm(want, w1.double(), eps)) < tol and rel(b, plain.rms_norm(want, w2.double(), eps)) < tol
    extra = mk(rows * max(top, 1), -(-width // 8) * 8).to(dtype)
    index = torch.randperm(rows * max(top, 1), generator=g)[:rows * top].view(rows, top).to(torch.int32)
    add = extra[index.long()][..., :width].double().sum(1) if top else 0
    want = want + y.double() + add
    ex = dict(extra=extra.to(cuda)[:, :width], extra_index=index.to(cuda)) if top else {}
    ends = torch.tensor([0, 5, 6, rows], dtype=torch.int32, device=cuda)
    before = x.clone()
    last, none = ops.residual_norm_pair(x, y.to(cuda), w1.to(cuda), None, eps, row_ends=ends, **ex)
    assert none is None and torch.equal(x, before)
    assert rel(last, plain.rms_norm(want, w1.double(), eps)[[4, 5, rows - 1]]) < tol
    a, b = ops.residual_norm_pair(x, y.to(cuda), w1.to(cuda), w2.to(cuda), eps, **ex)
    assert rel(x, want) < 1e-6 and rel(a, plain.rms_norm(want, w1.double(), eps)) < tol and rel(b, plain.rms_norm(want, w2.double(), eps)) < tol


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("inter", [8, 33, 1000])
def test_gated_units(cuda, dtype, inter):
    g = gen(inter)
    z, s = (torch.randn(9, 2 * inter, generator=g) * 3).to(dtype), torch.randn(9, 3, generator=g).to(dtype)
    gate, up = z.double().split(inter, dim=1)
    tol = 1e-2 if dtype == BF else 1e-5
    assert rel(ops.glu(z.to(cuda), inter), plain.silu(gate) * up) < tol
    cg, cu = gate.clamp(max=1.5), up.clamp(-1.5, 1.5)
    want = cg * torch.sigmoid(0.9 * cg) * (cu + 2) * torch.sigmoid(s[:, 1:2].double())
    out = torch.empty(9, inter + 7, dtype=dtype, device=cuda)
    assert rel(ops.glu(z.to(cuda), inter, 1.5, 0.9, 2.0, row_gate=s.to(cuda)[:, 1], out=out[:, :inter]), want) < tol


# ---- experts -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("tokens,experts,top,width,inter", [
    (1, 1, 1, 64, 8), (1, 8, 2, 72, 40), (7, 33, 4, 30, 17), (300, 5, 1, 200, 96), (513, 12, 3, 136, 136), (64, 300, 6, 64, 24),
    (2000, 4, 2, 64, 300), (40, 3, 3, 256, 130), (129, 1, 1, 64, 64)])
@pytest.mark.parametrize("skew", [False, True])
def test_experts(cuda, dtype, tokens, experts, top, width, inter, skew):
    g, limit = gen(tokens + experts), 0.9
    h = torch.randn(tokens, width, generator=g).to(dtype)
    router = torch.randn(experts, width, generator=g) * 2 * width ** -0.5
    if skew:                                                         # nearly everybody wants the same few
        router = router + torch.linspace(1, 0, experts)[:, None] * h.float().mean(0) * 3
    w = {"router": router.to(dtype)}
    for e in range(experts):
        w.update({f"e{e}.gate": (torch.randn(inter, width, generator=g) * 2 * width ** -0.5).to(dtype),
                  f"e{e}.up": (torch.randn(inter, width, generator=g) * 2 * width ** -0.5).to(dtype),
                  f"e{e}.down": (torch.randn(width, inter, generator=g) * inter ** -0.5).to(dtype)})
    logits = h.double() @ w["router"].double().T
    scores = torch.sigmoid(logits)
    want = torch.zeros(tokens, width, dtype=torch.float64)
    chosen = torch.topk(logits, top, dim=1)
    for e in range(experts):
        rows = (chosen.indices == e).any(1)
        if rows.any():
            want[rows] += plain.clamped(scores[rows, e:e + 1] * h[rows].double(), {k: v.double() for k, v in w.items()}, f"e{e}.", limit)

    from mini_vllm_b200.models.layers.feedforward import ExpertFeed
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        with torch.device(cuda):
            feed = ExpertFeed(width, inter, experts, top, limit, 1.702, 1.0)
    finally:
        torch.set_default_dtype(prev)
    feed.load(lambda n: w[n].to(cuda))
    status, hd = ops.new_status(cuda), h.to(cuda)
    for _ in range(3):                                               # later calls find the counters as the first left them
        out = feed.routed(hd, status)
        y, slots = out.rows, out.slots
        assert sorted(slots.flatten().tolist()) == list(range(tokens * top))
        got = y[slots.flatten().long()].view(tokens, top, width).double().sum(1)
        assert rel(got, want) < (2e-2 if dtype == BF else 2e-5)
    ops.check_status(status)
    assert int(feed.counters.abs().sum()) == 0


def test_experts_in_a_graph_follow_the_tokens(cuda):
    """Group sizes are data: the captured products follow another routing at every replay."""
    from mini_vllm_b200.models.layers.feedforward import ExpertFeed
    g, width, inter, experts, top, n = gen(2), 128, 64, 8, 2, 48
    prev = torch.get_default_dtype()
    torch.set_default_dtype(BF)
    try:
        with torch.device(cuda):
            feed = ExpertFeed(width, inter, experts, top, 1.0, 1.702, 1.0)
    finally:
        torch.set_default_dtype(prev)
    for p in feed.parameters():
        p.copy_((torch.randn(p.shape, generator=g) * p.shape[-1] ** -0.5).to(cuda))
    h = torch.randn(n, width, generator=g).to(BF).to(cuda)
    feed.routed(h, None)
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        out = feed.routed(h, None)
    for k in range(4):
        h.copy_((torch.randn(n, width, generator=g) + (3 * (k % 2)) * feed.router[k].float().cpu()).to(BF).to(cuda))
        graph.replay()
        got = out.rows[out.slots.flatten().long()].view(n, top, width).float().sum(1)
        again = feed.routed(h, None)
        assert torch.equal(got, again.rows[again.slots.flatten().long()].view(n, top, width).float().sum(1))
