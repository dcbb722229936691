"""Rasezen through the engine's own step, cache and scheduler: whole prompts, portions, mixed batches, reused memory and greedy
generation, against the plain oracle on small models with weights of the tests' making."""
import random
from functools import lru_cache

import pytest
import torch

from mini_vllm_b200.config import Config, SamplingParams
from oracle.rasezen import OracleRasezen
from tests.replay_helpers import assert_tokens, feed, make_engine, portions, row_errors, write_checkpoint
from tests.rasezen_helpers import CONFIGS, config, dense, moe, state_layer, tensors, window_layer

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
# bf16: a token whose experts nearly tie may take another one than the oracle, so the median and a wide cap; fp32 is the sharp comparison
TOL = {BF: 0.9, F32: 5e-5}
MEDIAN_TOL = {BF: 0.025, F32: 5e-6}
LENS = [1, 2, 3, 23, 130, 257, 410]


@lru_cache(maxsize=None)
def reference(name):
    """(config, tensors, prompts, logits of every position in float64)"""
    cfg, rnd = CONFIGS[name], random.Random(name)
    w = tensors(cfg, seed=len(name))
    prompts = [[rnd.randrange(cfg["vocab"]) for _ in range(n)] for n in LENS]
    model = OracleRasezen(w, cfg)
    return cfg, w, prompts, [model.forward(p) for p in prompts]


@pytest.fixture(scope="module", params=[(n, d) for n in CONFIGS for d in (BF, F32)], ids=lambda p: f"{p[0]}-{str(p[1])[6:]}")
def served(request, cuda, tmp_path_factory):
    name, dtype = request.param
    ref = reference(name)
    eng = make_engine(write_checkpoint(tmp_path_factory.mktemp("m") / name, ref[0], ref[1]), dtype)
    yield eng, dtype, ref
    del eng
    torch.cuda.empty_cache()


def check(got, want, dtype):
    errs = {i: row_errors(g, want[i][:g.shape[0]]) for i, g in got.items()}
    for i, e in errs.items():
        assert e.max() < TOL[dtype], (i, int(e.argmax()), float(e.max()))
    assert torch.cat(list(errs.values())).median() < MEDIAN_TOL[dtype]


def test_whole_prompts_alone(served):
    eng, dtype, (_, _, prompts, want) = served
    check(feed(eng, prompts, [[(i, len(p))] for i, p in enumerate(prompts)]), want, dtype)


def test_token_by_token(served):
    eng, dtype, (_, _, prompts, want) = served
    check(feed(eng, prompts, [[(i, 1)] for i in (0, 2, 3, 5) for _ in prompts[i]]), want, dtype)


@pytest.mark.parametrize("sizes", [[2], [100, 69, 2, 3, 1], [128], [127, 2, 1, 1, 130]])
def test_portions(served, sizes):
    eng, dtype, (_, _, prompts, want) = served
    picked = [5] if sizes == [2] else [4, 6]
    check(feed(eng, prompts, [[(i, n)] for i in picked for n in portions(len(prompts[i]), sizes)]), want, dtype)


def test_mixed_batches_with_reused_blocks_and_slots(served):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, end, and leave their blocks and slot to the next;
    the pool holds four requests at a time."""
    eng, dtype, (_, _, prompts, want) = served
    rnd, todo, live, plan = random.Random(3), [6, 0, 4, 5, 2, 3, 1], {}, []
    while todo or live:
        while todo and len(live) < 4:
            i = todo.pop(0)
            live[i] = len(prompts[i])
        step = []
        for i in sorted(live, key=lambda _: rnd.random()):
            if rnd.random() < 0.25 and len(live) > 1:
                continue                                             # left out of this step
            n = min(live[i], rnd.choice([1, 1, 1, 2, 3, 16, 64, 128]))
            step.append((i, n))
            live[i] -= n
        live = {i: n for i, n in live.items() if n}
        if step:
            plan.append(step)
    got = feed(eng, prompts, plan)
    check(got, want, dtype)
    alone = feed(eng, prompts, [[(i, len(prompts[i]))] for i in (4, 6)])     # the same positions however they were cut
    for i in (4, 6):
        assert row_errors(got[i], alone[i].double()).max() < TOL[dtype]


def window_model(size):
    """One attention layer whose keys answer every query at token 7 alone: its embedding has a direction that the key projection turns into
    one coordinate, where the queries look; every other token's key stands in another coordinate."""
    cfg = config([window_layer(heads=2, kv=1, dim=16, vdim=16, size=size, rot=8, scale=0.7)], width=64, vocab=40)
    w, g = tensors(cfg, seed=9), torch.Generator().manual_seed(1)
    u, up = torch.zeros(64), torch.zeros(64)
    u[:32], up[32:] = torch.randn(32, generator=g), torch.rand(32, generator=g) + 0.5
    w["embed"] = (up + torch.randn(40, 64, generator=g) * 0.1 + (torch.arange(40) == 7)[:, None] * 6 * u / u.norm()).to(BF)
    w["l0.norm1"] = torch.tensor(1.0, dtype=BF)
    q, k = torch.zeros(2, 16, 64), torch.randn(16, 64, generator=g) * 0.02
    q[:, 15, 32:], k[15] = 1.0, u / u.norm() * 8
    w["l0.mix.q"], w["l0.mix.k"] = q.flatten(0, 1).to(BF), k.to(BF)
    w["l0.mix.q.b"], w["l0.mix.k.b"] = torch.zeros(32, dtype=BF), (torch.arange(16) == 14).to(BF)
    w["l0.mix.q.norm"], w["l0.mix.k.norm"] = torch.ones(32, dtype=BF), torch.ones(16, dtype=BF)
    return cfg, w


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("size,at", [(60, 0), (60, 67), (60, 68), (60, 127), (60, 128), (128, 130), (129, 127), (1, 200), (2, 255), (300, 90)])
def test_the_edge_of_the_window(cuda, tmp_path, dtype, size, at):
    """A key that stands out shows in every token of its window and in none behind it: from a prompt, from portions that cut at the edge, and
    from decoding, at both sides of a page border."""
    cfg, w = window_model(size)
    rnd, n = random.Random(2), at + size + 6
    prompt = [rnd.randrange(8, 40) for _ in range(n)]
    without, prompt[at] = list(prompt), 7
    model = OracleRasezen(w, cfg)
    want = model.forward(prompt)
    shown = row_errors(model.forward(without), want)
    assert shown[at:at + size].min() > 0.02 and shown[at + size:].max() < 1e-9 and (at == 0 or shown[:at].max() < 1e-9)
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype)
    edge = at + size
    for plan in ([[(0, n)]], [[(0, edge - 1)]] + [[(0, 1)]] * 7, [[(0, edge)], [(0, 6)]], [[(0, k)] for k in portions(n, [50, 2])]):
        got = row_errors(feed(eng, [prompt], plan)[0], want)
        assert got.max() < (0.05 if dtype == BF else 5e-5)
        assert (got[at:edge] < 0.5 * shown[at:edge]).all()


@pytest.mark.parametrize("dtype", [BF, F32])
def test_a_memory_that_reaches_back_to_the_first_token(cuda, tmp_path, dtype):
    """State-space layers that forget next to nothing: hundreds of tokens later the first one still shows, whatever lies between was fed how,
    and a slot's earlier owner does not."""
    cfg = config([state_layer(heads=4, groups=2, state=24, vdim=16, taps=3, norm_groups=2), state_layer(heads=2, groups=1, state=64, vdim=32)], vocab=40)
    w, u = tensors(cfg, seed=5), torch.zeros(88)
    u[:44] = torch.randn(44, generator=torch.Generator().manual_seed(1))
    u = u / u.norm()
    embed = w["embed"].float()
    w["embed"] = (embed - (embed @ u)[:, None] * u + (torch.arange(40) == 7)[:, None] * 20 * u).to(BF)
    w["l0.mix.in"][-4:] = u.to(BF)                                   # the first layer's steps: long for token 7, short for the others
    for k in w:
        if k.endswith("A_log"):
            w[k] = torch.full_like(w[k], -9.0)
        elif k.endswith("dt_bias"):
            w[k] = torch.full_like(w[k], -5.0)
    rnd = random.Random(6)
    prompt = [7] + [rnd.randrange(8, 40) for _ in range(420)]
    model = OracleRasezen(w, cfg)
    want = model.forward(prompt)
    shown = row_errors(model.forward([8] + prompt[1:]), want)[400:]
    assert shown.min() > 0.02
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype)
    feed(eng, [[9] * 200], [[(0, 200)]])                             # leaves its state behind in the slot
    for plan in ([[(0, 421)]], [[(0, 1)]] + [[(0, 420)]], [[(0, 400)]] + [[(0, 1)]] * 21, [[(0, k)] for k in portions(421, [63, 2, 65])]):
        got = row_errors(feed(eng, [prompt], plan)[0], want)
        assert got.max() < (0.05 if dtype == BF else 5e-5) and (got[400:] < 0.6 * shown).all()


def test_long_decoding_from_graphs(cuda, tmp_path):
    """Hundreds of decoded tokens over page borders and past the window."""
    cfg = config([state_layer(mlp=moe()), window_layer(size=100, mlp=dense()), window_layer(heads=4, kv=4, size=257, mlp=moe(3, 1))], vocab=60)
    w = tensors(cfg, seed=4)
    rnd = random.Random(7)
    prompt = [rnd.randrange(60) for _ in range(520)]
    want = OracleRasezen(w, cfg).forward(prompt)
    for dtype in (BF, F32):
        eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype)
        check(feed(eng, [prompt], [[(0, 3)]] + [[(0, 1)]] * 517), [want], dtype)
        del eng


@pytest.mark.parametrize("name", ["several", "wide", "ones"])
def test_residual_stream_of_every_layer(cuda, tmp_path, name):
    cfg, w, prompts, _ = reference(name)
    streams, taps = [], []
    OracleRasezen(w, cfg).forward(prompts[4], streams)
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), F32)
    eng.executor.model.residual_tap = lambda i, x: taps.append(x.clone())
    feed(eng, prompts, [[(4, len(prompts[4]))]])
    assert len(taps) == len(streams)
    for t, s in zip(taps, streams):
        assert (t.double().cpu() - s).abs().max() < 2e-5 * s.abs().max()


# ---- greedy generation through Engine.generate and the scheduler -----------------------------------------------
GREEDY = [state_layer(mlp=dense()), window_layer(size=20, mlp=moe()), state_layer(heads=4, groups=1, state=16, vdim=24, norm_groups=2, mlp=moe(6, 1))]


def greedy_case(n, seed, lens, new, layers=GREEDY, width=88):
    cfg = config(layers, vocab=70, width=width)
    w = tensors(cfg, seed=seed)
    rnd = random.Random(seed)
    prompts = [[rnd.randrange(70) for _ in range(rnd.choice(lens))] for _ in range(n)]
    model = OracleRasezen(w, cfg)
    return cfg, w, prompts, [model.greedy(p, new) for p in prompts]


@pytest.mark.parametrize("dtype,margin", [(F32, 1e-3), (BF, 0.5)])
@pytest.mark.parametrize("extra", [{}, {"enable_mixed_steps": True}, {"enable_chunked_prefill": True, "max_num_batched_tokens": 48},
                                   {"enable_chunked_prefill": True, "enable_mixed_steps": True, "max_num_batched_tokens": 33},
                                   {"use_cuda_graph": False, "fused_greedy_head": False}], ids=["plain", "mixed", "chunked", "chunked-mixed", "eager"])
@pytest.mark.parametrize("pipelined", [True, False])
def test_greedy_generation(cuda, tmp_path, dtype, margin, extra, pipelined):
    cfg, w, prompts, want = greedy_case(7, 11, [1, 5, 30, 75], 12)
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype, blocks=4, slots=3, **extra)     # three live at a time at most
    out = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True), use_tqdm=not pipelined)
    assert all(len(o["tokens"]) == 12 for o in out)
    compared = assert_tokens([o["tokens"] for o in out], want, margin)
    assert compared >= (80 if dtype == F32 else 4)
    bm = eng.scheduler.block_manager
    assert bm.num_free_blocks == bm.capacity and bm.state_slots.num_free == 3


def test_preempted_requests_start_over(cuda, tmp_path):
    """Too few blocks for three requests that each grow into a second: somebody is preempted, loses slot and blocks, and is computed again
    from its first token."""
    cfg, w, prompts, want = greedy_case(3, 13, [120, 126], 12)
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), F32, blocks=4, slots=3)
    preempted, preempt = [], eng.scheduler.preempt
    eng.scheduler.preempt = lambda r: (preempted.append(r.id), preempt(r))[1]
    out = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True), use_tqdm=False)
    assert preempted and assert_tokens([o["tokens"] for o in out], want, 1e-3) > 20


def test_prefix_cache_of_attention_layers(cuda, tmp_path):
    """A model without state-space layers holds no state: prompts that begin alike share blocks of normalised keys and values."""
    layers = [window_layer(mlp=moe()), window_layer(size=150, heads=4, mlp=dense())]
    cfg, w, prompts, _ = greedy_case(1, 19, [260], 1, layers)
    prompts = [prompts[0], prompts[0][:256] + [3, 4, 5], prompts[0][:128] + [9] * 40]
    path, got = write_checkpoint(tmp_path / "m", cfg, w), {}
    for cached in (True, False):
        eng, hits, got[cached] = make_engine(path, F32, enable_prefix_cache=cached), 0, []
        for p in prompts:
            req = eng.submit(p, SamplingParams(max_tokens=6, ignore_eos=True))
            eng.step()
            hits += req.num_cached_tokens
            while not eng.finished:
                eng.step()
            got[cached].append(req.completion_tokens)
        assert hits == (256 + 128 if cached else 0)
        eng.executor.check_device_status()
    model = OracleRasezen(w, cfg)
    assert got[True] == got[False] and assert_tokens(got[True], [model.greedy(p, 6) for p in prompts], 1e-3) >= 12


def test_prefix_cache_is_refused_with_state(cuda):
    from mini_vllm_b200.config import rasezen_shape
    from mini_vllm_b200.engine.engine import Engine
    with pytest.raises(ValueError, match="state"):
        Engine(Config(hf_config=rasezen_shape([state_layer()], 64, 96), enable_prefix_cache=True))


def test_sampling_and_random_init(cuda):
    from mini_vllm_b200.config import rasezen_shape
    from mini_vllm_b200.engine.engine import Engine
    eng = Engine(Config(hf_config=rasezen_shape(GREEDY, 64, 96), kv_cache_num_blocks=8, max_num_batched_seqs=4, seed=3))
    out = eng.generate([[1, 2, 3], [4]], SamplingParams(max_tokens=6, ignore_eos=True, temperature=0.8, top_k=20, top_p=0.9), use_tqdm=False)
    assert all(len(o["tokens"]) == 6 and all(0 <= t < 96 for t in o["tokens"]) for o in out)


def test_trace_program(cuda, tmp_path):
    """bin/trace_run end to end: acknowledgements, files only where something is wanted, exit code."""
    import json
    import subprocess
    from pathlib import Path

    import numpy as np
    cfg, w, prompts, want = reference("several")
    path = write_checkpoint(tmp_path / "m", cfg, w)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": prompts[4][:50], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": prompts[2], "want": [2]}, {"id": "a", "tokens": prompts[4][50:], "want": [0, 79]}],
              "end": ["a", "b"]}]
    r = subprocess.run([str(Path(__file__).resolve().parent.parent / "bin" / "trace_run"), "--model", path, "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "256"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True,
                       timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    assert not (tmp_path / "0.f32").exists()
    got = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4").reshape(3, -1))
    assert row_errors(got, torch.stack([want[2][2], want[4][50], want[4][129]])).max() < 5e-5


def test_command_line_generation(cuda, tmp_path, capsys):
    import json

    from mini_vllm_b200.__main__ import main
    cfg, w, prompts, want = greedy_case(2, 17, [5, 9], 6)
    path = write_checkpoint(tmp_path / "m", cfg, w)
    args = ["--model", path, "--dtype", "float32", "--max-tokens", "6", "--ignore-eos", "--max-model-len", "256", "--chunked-prefill"]
    assert main(args + [x for p in prompts for x in ("--prompt", " ".join(map(str, p)))]) == 0
    out = [json.loads(x)["tokens"] for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    assert assert_tokens(out, want, 1e-3) > 4
