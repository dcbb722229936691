"""Vebonex through the engine's own step, cache and scheduler: whole prompts, portions, mixed batches, reused memory and greedy
generation, against the plain oracle on small models with weights of the tests' making."""
import random
from functools import lru_cache

import pytest
import torch

from mini_vllm_b200.config import Config, SamplingParams
from oracle.vebonex import OracleVebonex
from tests.replay_helpers import assert_tokens, feed, make_engine, portions, row_errors, write_checkpoint
from tests.vebonex_helpers import CONFIGS, config, gla_layer, latent_layer, lstm_layer, tensors

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
# bf16: heads whose output is all but zero are scaled up by their norm, so single positions of these tiny models stray above the mean;
# fp32 is the sharp comparison
TOL = {BF: 0.35, F32: 1e-4}
MEAN_TOL = {BF: 0.03, F32: 2e-5}
LENS = [1, 2, 3, 23, 130, 257, 310]


@lru_cache(maxsize=None)
def reference(name):
    """(config, tensors, prompts, logits of every position in float64)"""
    cfg, rnd = CONFIGS[name], random.Random(name)
    w = tensors(cfg, seed=len(name))
    prompts = [[rnd.randrange(cfg["vocab"]) for _ in range(n)] for n in LENS]
    model = OracleVebonex(w, cfg)
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
    assert torch.cat(list(errs.values())).mean() < MEAN_TOL[dtype]


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


def far_key_model(layers, borrowed):
    """Token 7's latent wins every softmax of the attention layers (its embedding and the key and query projections share a direction), and
    its value says so."""
    cfg = config(layers, width=64, vocab=40, streams=2, groups=1, max_positions=700)
    w = tensors(cfg, seed=9)
    g = torch.Generator().manual_seed(1)
    u = torch.randn(64, generator=g)
    u = u / u.norm()
    w["pos"] = w["pos"] * 0.2
    w["embed"] = (torch.rand(40, 64, generator=g) * 0.5 + 0.5 + (torch.arange(40) == 7)[:, None] * 9 * u).to(torch.bfloat16)
    owner = 0
    dkv = torch.randn(50, 64, generator=g) * 0.05
    dkv[3] = u * 3
    w[f"l{owner}.mix.dkv"] = dkv.to(torch.bfloat16)
    for i in (owner, borrowed):
        m = cfg["layers"][i]["mixer"]
        uk = torch.zeros(m["heads"], m["dim"], 50)
        uk[:, 0, 3] = 3.0
        uq = torch.zeros(m["heads"], m["dim"], m["q_rank"])
        uq[:, 0] = torch.randn(m["q_rank"], generator=g).abs() * 0.3
        w[f"l{i}.mix.uk"], w[f"l{i}.mix.uq"] = uk.flatten(0, 1).to(torch.bfloat16), uq.flatten(0, 1).to(torch.bfloat16)
        w[f"l{i}.mix.dq"] = (torch.randn(m["q_rank"], 64, generator=g) * 0.02 + 0.2).to(torch.bfloat16)      # a latent that is all positive
    return cfg, w


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("at", [0, 1, 127, 128, 255])
def test_a_far_key_is_found(cuda, tmp_path, dtype, at):
    """Whatever lies between: at the start, on both sides of a page border; from a prompt, from portions and from decoding, directly and
    through a layer that borrows the latents."""
    layers = [latent_layer(scale=1.0, ff=None), gla_layer(ff=None), latent_layer(heads=2, dim=16, vdim=24, q_rank=20, scale=1.0, kv_from=0, ff=None)]
    cfg, w = far_key_model(layers, 2)
    rnd = random.Random(2)
    prompt = [rnd.randrange(8, 40) for _ in range(400)]
    prompt[at] = 7
    model = OracleVebonex(w, cfg)
    want = model.forward(prompt)
    without = list(prompt)
    without[at] = 8
    assert row_errors(model.forward(without)[390:], want[390:]).min() > 0.2, "the key does not show"
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype)
    for plan in ([[(0, 400)]], [[(0, 380)]] + [[(0, 1)]] * 20, [[(0, n)] for n in portions(400, [50, 2])]):
        check(feed(eng, [prompt], plan), [want], dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_a_memory_reaches_far_back(cuda, tmp_path, dtype):
    """Decays that keep everything: the first token's write is still read hundreds of tokens later, and a lost state would show."""
    cfg = config([lstm_layer(heads=2, ff=None), gla_layer(heads=2, tau=16.0, ff=None)], width=64, vocab=40, streams=2, groups=1)
    w = tensors(cfg, seed=5)
    w["l0.mix.f.b"], w["l1.mix.a2.b"] = torch.full((2,), 7.0, dtype=BF), torch.full((40,), 25.0, dtype=BF)
    w["l0.mix.i"], w["l0.mix.f"] = w["l0.mix.i"] * 0, w["l0.mix.f"] * 0
    w["embed"] = w["embed"] * 0.3
    w["embed"][7] = w["embed"][7] * 30
    w["pos"] = w["pos"] * 0.3
    rnd = random.Random(4)
    prompt = [7] + [rnd.randrange(8, 40) for _ in range(330)]
    model = OracleVebonex(w, cfg)
    want = model.forward(prompt)
    assert row_errors(model.forward([8] + prompt[1:])[300:], want[300:]).max() > 0.02, "the first token does not show"
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype)
    for plan in ([[(0, 331)]], [[(0, 2)]] + [[(0, 1)]] * 329, [[(0, n)] for n in portions(331, [17, 2, 1])]):
        check(feed(eng, [prompt], plan), [want], dtype)


def test_long_decoding_from_graphs(cuda, tmp_path):
    """Hundreds of decoded tokens over block borders, with slow decays that remember the start."""
    cfg = config([lstm_layer(), latent_layer(), gla_layer(tau=40.0), latent_layer(kv_from=1)], vocab=60)
    w = tensors(cfg, seed=4)
    w["l0.mix.f.b"] = torch.full((3,), 6.5, dtype=torch.bfloat16)
    rnd = random.Random(7)
    prompt = [rnd.randrange(60) for _ in range(520)]
    want = OracleVebonex(w, cfg).forward(prompt)
    for dtype in (BF, F32):
        eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype)
        check(feed(eng, [prompt], [[(0, 3)]] + [[(0, 1)]] * 517), [want], dtype)
        del eng


@pytest.mark.parametrize("name", ["shared", "wide"])
def test_residual_streams_of_every_layer(cuda, tmp_path, name):
    cfg, w, prompts, _ = reference(name)
    streams, taps = [], []
    OracleVebonex(w, cfg).forward(prompts[4], streams)
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), F32)
    eng.executor.model.residual_tap = lambda i, x: taps.append(x.clone())
    feed(eng, prompts, [[(4, len(prompts[4]))]])
    assert len(taps) == len(streams)
    for t, s in zip(taps, streams):
        assert (t.double().cpu() - s).abs().max() < 3e-5 * s.abs().max()


# ---- greedy generation through Engine.generate and the scheduler -----------------------------------------------
GREEDY = [lstm_layer(), latent_layer(), gla_layer(), latent_layer(heads=2, kv_from=1)]


def greedy_case(n, seed, lens, new, layers=GREEDY):
    cfg = config(layers, vocab=70)
    w = tensors(cfg, seed=seed)
    rnd = random.Random(seed)
    prompts = [[rnd.randrange(70) for _ in range(rnd.choice(lens))] for _ in range(n)]
    model = OracleVebonex(w, cfg)
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


def test_preempted_requests_start_over_from_zero_state(cuda, tmp_path):
    """Too few blocks for three requests that each grow into a second: somebody is preempted, loses slot and blocks, and is computed again
    from its first token."""
    cfg, w, prompts, want = greedy_case(3, 13, [120, 126], 12)
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), F32, blocks=4, slots=3)
    preempted, preempt = [], eng.scheduler.preempt
    eng.scheduler.preempt = lambda r: (preempted.append(r.id), preempt(r))[1]
    out = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True), use_tqdm=False)
    assert preempted and assert_tokens([o["tokens"] for o in out], want, 1e-3) > 20


@pytest.mark.parametrize("dtype,margin", [(F32, 1e-3), (BF, 0.5)])
def test_prefix_cache_over_latents(cuda, tmp_path, dtype, margin):
    """A model whose layers all cache latents has no state: prompts that begin alike share blocks."""
    layers = [latent_layer(), latent_layer(heads=2, kv_from=0)]
    cfg, w, prompts, _ = greedy_case(1, 19, [260], 1, layers)
    prompts = [prompts[0], prompts[0][:256] + [3, 4, 5], prompts[0][:128] + [9] * 40]
    model = OracleVebonex(w, cfg)
    want = [model.greedy(p, 6) for p in prompts]
    eng = make_engine(write_checkpoint(tmp_path / "m", cfg, w), dtype, enable_prefix_cache=True)
    got, hits = [], 0
    for p in prompts:
        req = eng.submit(p, SamplingParams(max_tokens=6, ignore_eos=True))
        eng.step()
        hits += req.num_cached_tokens
        while not eng.finished:
            eng.step()
        got.append(req.completion_tokens)
    assert hits == 256 + 128 and assert_tokens(got, want, margin) >= (12 if dtype == F32 else 1)
    eng.executor.check_device_status()


def test_prefix_cache_is_refused_with_state(cuda):
    from mini_vllm_b200.config import vebonex_shape
    from mini_vllm_b200.engine.engine import Engine
    with pytest.raises(ValueError, match="state"):
        Engine(Config(hf_config=vebonex_shape([gla_layer()], 64, 96), enable_prefix_cache=True))


def test_sampling_and_random_init(cuda):
    from mini_vllm_b200.config import vebonex_shape
    from mini_vllm_b200.engine.engine import Engine
    eng = Engine(Config(hf_config=vebonex_shape(GREEDY, 64, 96, groups=2), kv_cache_num_blocks=8, max_num_batched_seqs=4, seed=3))
    out = eng.generate([[1, 2, 3], [4]], SamplingParams(max_tokens=6, ignore_eos=True, temperature=0.8, top_k=20, top_p=0.9), use_tqdm=False)
    assert all(len(o["tokens"]) == 6 and all(0 <= t < 96 for t in o["tokens"]) for o in out)


def test_trace_program(cuda, tmp_path):
    """bin/trace_run end to end: acknowledgements, files only where something is wanted, exit code."""
    import json
    import subprocess
    from pathlib import Path

    import numpy as np
    cfg, w, prompts, want = reference("shared")
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
    assert row_errors(got, torch.stack([want[2][2], want[4][50], want[4][129]])).max() < 1e-4


def test_command_line_generation(cuda, tmp_path, capsys):
    import json

    from mini_vllm_b200.__main__ import main
    cfg, w, prompts, want = greedy_case(2, 17, [5, 9], 6)
    path = write_checkpoint(tmp_path / "m", cfg, w)
    args = ["--model", path, "--dtype", "float32", "--max-tokens", "6", "--ignore-eos", "--max-model-len", "256", "--chunked-prefill"]
    assert main(args + [x for p in prompts for x in ("--prompt", " ".join(map(str, p)))]) == 0
    out = [json.loads(x)["tokens"] for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    assert assert_tokens(out, want, 1e-3) > 4
