"""Host side of the Fupupel design (no GPU): configuration reader, weight layout, state slots, chunked scheduling, and the plain
oracle checked against itself."""
import random
from types import SimpleNamespace

import pytest
import torch

from mini_vllm_b200.config import Config, SamplingParams
from mini_vllm_b200.engine.request import Request
from mini_vllm_b200.kvcache.block_manager import KVCacheBlockManager
from mini_vllm_b200.kvcache.state_slots import StateSlots
from mini_vllm_b200.scheduler.batch import Batch
from mini_vllm_b200.scheduler.scheduler import Scheduler
from oracle import fupupel as plain
from tests.fupupel_helpers import CONFIGS, both_layer, config, scan_layer, tensors
from tests.replay_helpers import write_checkpoint
from tests.test_host_engine_loop import StandInExecutor, make_engine


def test_config_reader_takes_ranks_from_the_tensors(tmp_path):
    cfg = CONFIGS["grouped"]
    path = write_checkpoint(tmp_path / "m", cfg, tensors(cfg, ranks=(7, 11)))
    hf = Config(model=path, max_model_len=777).hf_config
    assert hf.architectures == ["Fupupel"] and hf.dtype == torch.bfloat16 and hf.max_position_embeddings == 777
    right = hf.layers[1]["mixer"]["right"]
    assert (right["decay_rank"], right["gate_rank"]) == (7, 11)
    assert "decay_rank" not in cfg["layers"][1]["mixer"]["right"]
    assert Config(model=path, dtype=torch.float32).hf_config.dtype == torch.float32


def cpu_model(cfg, weights, dtype=torch.float32):
    from mini_vllm_b200.config.native import fupupel_config
    from mini_vllm_b200.models.models import get_model_class
    hf = fupupel_config(cfg, {k: list(v.shape) for k, v in weights.items()}, dtype)
    model = get_model_class("Fupupel")(hf)
    model.load_weights(weights.items())
    return model


def test_weights_that_are_missing_or_unknown_are_refused():
    cfg = CONFIGS["grouped"]
    w = tensors(cfg)
    with pytest.raises(KeyError, match="l1.mix.right.g2"):
        cpu_model(cfg, {k: v for k, v in w.items() if k != "l1.mix.right.g2"})
    with pytest.raises(KeyError, match="extra"):
        cpu_model(cfg, {**w, "extra": torch.zeros(1)})
    with pytest.raises(ValueError, match="mamba9"):
        cpu_model({**cfg, "layers": [{"type": "mamba9", "mixer": {}, "mlp": None}]}, w)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_packed_projections_hold_every_weight_once(name, dtype):
    """The padded, permuted, concatenated projections are the checkpoint's matrices: same energy, blocks at multiples of 8."""
    cfg = CONFIGS[name]
    w = tensors(cfg)
    model = cpu_model(cfg, w, dtype)
    for i, layer in enumerate(model.layers):
        p = f"l{i}.mix."
        ins = ["in"] if cfg["layers"][i]["type"] == "mamba1" else [f"left.{n}" for n in "qkv"] + [f"right.{n}" for n in ("q", "k", "v", "b", "a1", "g1")]
        outs = ["o"] if cfg["layers"][i]["type"] == "mamba1" else ["left.o", "right.o"]
        for got, names in ((layer.mixer.in_proj, ins), (layer.mixer.out_proj, outs)):
            want = sum(float(w[p + n].double().pow(2).sum()) for n in names)
            assert float(got.double().pow(2).sum()) == pytest.approx(want, rel=1e-6)
        assert all(s % 8 == 0 for s in layer.mixer.in_sizes + layer.mixer.out_sizes)


def test_state_slots_lowest_first_and_never_twice():
    s = StateSlots(3)
    assert [s.take(), s.take(), s.take()] == [0, 1, 2] and s.num_free == 0
    with pytest.raises(RuntimeError):
        s.take()
    s.give(1)
    assert s.take() == 1
    s.give(2)
    with pytest.raises(AssertionError):
        s.give(2)


def test_block_manager_hands_out_slots_with_blocks():
    bm = KVCacheBlockManager(8, 128, state_slots=StateSlots(1))
    a, b = Request([1] * 200), Request([1] * 3)
    bm.allocate_blocks_for_prefill(a)
    assert a.state_slot == 0 and len(a.blocks) == 2 and not bm.can_allocate_new_block(b)
    a.tokens += [1] * 100
    a.state = Request.RUNNING
    assert bm.can_allocate_new_block(a)                              # it has its slot already
    bm.extend(a)
    assert len(a.blocks) == 3
    with pytest.raises(RuntimeError):
        bm.extend(b)
    bm.deallocate(a)
    assert a.state_slot == -1 and bm.num_free_blocks == 8
    bm.extend(b)
    assert b.state_slot == 0 and len(b.blocks) == 1


def scheduler(**kw):
    return Scheduler(SimpleNamespace(**{**dict(max_num_batched_seqs=4, max_num_batched_tokens=50, eos_token_ids=set(), kv_cache_num_blocks=20,
                                               kv_cache_block_size=128, enable_chunked_prefill=True, num_state_slots=3), **kw}))


def test_prompts_enter_in_portions_of_the_token_budget():
    sch = scheduler()
    reqs = [Request([1] * n, SamplingParams(max_tokens=2, ignore_eos=True)) for n in (120, 10, 60, 5)]
    for r in reqs:
        sch.submit(r)
    seen = []
    while not sch.finished:
        b = sch.schedule()
        if b.type == Batch.PREFILL:
            seen.append([(reqs.index(r), r.num_cached_tokens, r.step_len, p) for r, p in zip(b.requests, b.partial)])
            assert b.prefill_tokens == sum(r.step_len - r.num_cached_tokens for r in b.requests) <= 50
        sch.update(b, [9] * len(b.requests))
    assert seen[0] == [(0, 0, 50, True)] and seen[1] == [(0, 50, 100, True)]
    assert seen[2] == [(0, 100, 120, False), (1, 0, 10, False), (2, 0, 20, True)]
    assert seen[3] == [(2, 20, 60, False)]                           # three slots are taken: the fourth prompt waits for one
    assert seen[4] == [(3, 0, 5, False)]
    assert all(r.num_completion_tokens == 2 for r in reqs)
    assert sch.block_manager.num_free_blocks == 20 and sch.block_manager.state_slots.num_free == 3


@pytest.mark.parametrize("mixed", [False, True])
@pytest.mark.parametrize("blocks", [40, 7])
def test_pipelined_loop_with_portions_gives_the_plain_completions(mixed, blocks):
    """Portions, preemption and EOS under the run-ahead loop: a portion yields no token, whatever the executor returns for it."""
    rnd = random.Random(3 + blocks)
    prompts = [[rnd.randrange(1, 50) for _ in range(rnd.randrange(3, 400))] for _ in range(16)]
    params = [SamplingParams(max_tokens=rnd.randrange(2, 45), ignore_eos=(i % 5 == 4)) for i in range(len(prompts))]

    def run(chunked, pipelined):
        eng = make_engine(mixed, blocks)
        eng.config.max_num_batched_tokens = 90 if chunked else 2048
        eng.config.enable_chunked_prefill, eng.config.num_state_slots = chunked, 4
        eng.scheduler = Scheduler(eng.config)
        assert isinstance(eng.executor, StandInExecutor)
        out = eng.generate(prompts, params, use_tqdm=not pipelined)
        bm = eng.scheduler.block_manager
        assert bm.num_free_blocks == blocks and bm.state_slots.num_free == 4
        return [o["tokens"] for o in out]
    want = run(False, False)
    assert run(True, True) == want and run(True, False) == want


def test_pool_size_of_a_trace():
    from mini_vllm_b200.trace import BLOCK, pool_blocks
    rnd = random.Random(1)
    for _ in range(200):                                             # four requests that fill the stated tokens always fit
        lens = [rnd.randrange(1, 900) for _ in range(4)]
        stated = sum(-(-n // 64) * 64 for n in lens)
        assert sum(-(-n // BLOCK) for n in lens) <= pool_blocks(stated) <= stated // BLOCK + 2


# ---- the oracle against itself -----------------------------------------------------------------------------------
def test_oracle_recurrences_carry_their_state():
    g = torch.Generator().manual_seed(0)
    rn = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    u, dt, a, b, c, d = rn(9, 4), rn(9, 4).abs(), -rn(4, 3).abs(), rn(9, 3), rn(9, 3), rn(4)
    whole, end = plain.selective_scan(u, dt, a, b, c, d)
    y1, s = plain.selective_scan(u[:5], dt[:5], a, b[:5], c[:5], d)
    y2, s = plain.selective_scan(u[5:], dt[5:], a, b[5:], c[5:], d, s)
    assert torch.allclose(torch.cat([y1, y2]), whole) and torch.allclose(s, end)
    q, k, v, gd, beta = rn(9, 4), rn(9, 4), rn(9, 3), torch.rand(9, 4, generator=g, dtype=torch.float64), torch.rand(9, generator=g, dtype=torch.float64)
    whole, end = plain.delta_rule(q, k, v, gd, beta)
    o1, s = plain.delta_rule(q[:2], k[:2], v[:2], gd[:2], beta[:2])
    o2, s = plain.delta_rule(q[2:], k[2:], v[2:], gd[2:], beta[2:], s)
    assert torch.allclose(torch.cat([o1, o2]), whole) and torch.allclose(s, end)


def test_oracle_write_is_seen_by_its_own_read_and_an_erased_value_is_gone():
    k = torch.tensor([[1.0, 0.0], [1.0, 0.0]], dtype=torch.float64)
    v = torch.tensor([[5.0], [7.0]], dtype=torch.float64)
    one = torch.ones(2, dtype=torch.float64)
    o, _ = plain.delta_rule(k, k, v, torch.ones(2, 2, dtype=torch.float64), one)
    assert o[:, 0].tolist() == [5.0, 7.0]                            # full step size: the second write replaces the first


def test_oracle_window_and_conv_edges():
    q = torch.ones(6, 1, 2, dtype=torch.float64)
    v = torch.eye(6, dtype=torch.float64)[:, None]
    out = plain.attention(q, q, v, 1.0, None, 3)
    assert (out[5, 0] > 0).tolist() == [False, False, False, True, True, True]
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=torch.float64)
    w = torch.tensor([[2.0, 3.0]], dtype=torch.float64)
    assert plain.causal_conv(u, w, None)[:, 0].tolist() == [3.0, 32.0, 320.0]


def test_oracle_is_causal():
    cfg = config([scan_layer(), both_layer()])
    m = plain.OracleFupupel(tensors(cfg), cfg)
    toks = list(range(20))
    assert torch.allclose(m.forward(toks)[:11], m.forward(toks[:11]))
