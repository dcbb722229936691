"""Host side of the Vebonex design (no GPU): configuration reader, weight layout, shared latents, limits, and the plain oracle checked
against itself."""
from types import SimpleNamespace

import pytest
import torch

from mini_vllm_b200.config import Config, SamplingParams
from oracle import vebonex as plain
from tests.replay_helpers import write_checkpoint
from tests.vebonex_helpers import CONFIGS, config, gla_layer, latent_layer, lstm_layer, tensors

F64 = torch.float64


def test_config_reader(tmp_path):
    cfg = CONFIGS["shared"]
    path = write_checkpoint(tmp_path / "m", cfg, tensors(cfg, decay_rank=7))
    hf = Config(model=path, max_model_len=777).hf_config
    assert hf.architectures == ["Vebonex"] and hf.dtype == torch.bfloat16 and (hf.streams, hf.norm_groups) == (3, 3)
    assert hf.max_position_embeddings == hf.learned_positions == 600                 # the table's size, whatever the engine allows
    assert hf.layers[1]["mixer"]["decay_rank"] == 7 and "decay_rank" not in cfg["layers"][1]["mixer"]
    assert Config(model=path, dtype=torch.float32).hf_config.dtype == torch.float32


def cpu_model(cfg, weights, dtype=torch.float32):
    from mini_vllm_b200.config.native import vebonex_config
    from mini_vllm_b200.models.models import get_model_class
    hf = vebonex_config(cfg, {k: list(v.shape) for k, v in weights.items()}, dtype)
    model = get_model_class("Vebonex")(hf)
    model.load_weights(weights.items())
    return model


def test_weights_that_are_missing_or_unknown_are_refused():
    cfg = CONFIGS["shared"]
    w = tensors(cfg)
    for name in ("l2.mix.uk", "l1.hc2.mix", "pos", "l0.mlp.act"):
        with pytest.raises(KeyError, match=name):
            cpu_model(cfg, {k: v for k, v in w.items() if k != name})
    with pytest.raises(KeyError, match="l2.mix.dkv"):                                # layer 2 borrows: it has none of its own
        cpu_model(cfg, {**w, "l2.mix.dkv": w["l0.mix.dkv"]})
    with pytest.raises(ValueError, match="mamba9"):
        cpu_model({**cfg, "layers": [{"type": "mamba9", "mixer": {}, "mlp": None}]}, w)


@pytest.mark.parametrize("bad", [[latent_layer(kv_from=0)], [latent_layer(), latent_layer(kv_from=0), latent_layer(kv_from=1)],
                                 [lstm_layer(), latent_layer(kv_from=0)], [latent_layer(), latent_layer(kv_rank=20, kv_from=0)],
                                 [latent_layer(kv_from=1), latent_layer()]])
def test_latents_can_only_come_from_an_earlier_layer_that_makes_them(bad):
    cfg = config(bad)
    with pytest.raises(ValueError, match="latents"):
        cpu_model(cfg, tensors(cfg))
    with pytest.raises(ValueError, match="groups"):
        cpu_model({**CONFIGS["shared"], "norm": {"eps": 1e-5, "groups": 5}}, tensors(CONFIGS["shared"]))


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_packed_projections_hold_every_weight_once(name, dtype):
    """The padded, concatenated projections are the checkpoint's matrices: same energy, blocks at multiples of 8."""
    cfg = CONFIGS[name]
    w = tensors(cfg)
    energy = lambda *ts: sum(float(t.double().pow(2).sum()) for t in ts)
    for i, layer in enumerate(cpu_model(cfg, w, dtype).layers):
        p, kind, branch = f"l{i}.mix.", cfg["layers"][i]["type"], layer.mixer.branches["mixer"]
        ins = {"mlstm": ["q", "k", "v", "g", "i", "f"], "gla": ["q", "k", "v", "g", "a1"], "latent_attention": ["dq", "g", "dkv"]}[kind]
        assert energy(layer.mixer.in_proj) == pytest.approx(energy(*(w[p + n] for n in ins if p + n in w)), rel=1e-6)
        assert energy(layer.mixer.out_proj) == pytest.approx(energy(w[p + "o"]), rel=1e-6)
        assert all(s % 8 == 0 for s in layer.mixer.in_sizes + layer.mixer.out_sizes)
        if kind == "latent_attention":
            assert energy(branch.q_up, branch.kv_up) == pytest.approx(energy(w[p + "uq"], w[p + "uk"], w[p + "uv"]), rel=1e-6)
            assert all(s % 8 == 0 for s in branch.in_sizes)
            assert hasattr(branch, "latent_cache") == ("kv_from" not in cfg["layers"][i]["mixer"])


def test_only_models_with_state_hold_state_slots():
    cfg = CONFIGS["large"]
    assert not cpu_model(cfg, tensors(cfg)).recurrent
    cfg = CONFIGS["ones"]
    assert cpu_model(cfg, tensors(cfg)).recurrent


def test_requests_beyond_the_position_table_are_refused():
    from mini_vllm_b200.engine.engine import Engine
    eng = Engine.__new__(Engine)
    taken = []
    eng.config, eng.scheduler = SimpleNamespace(hf_config=SimpleNamespace(learned_positions=20)), SimpleNamespace(submit=taken.append)
    eng.submit([1] * 15, SamplingParams(max_tokens=6))                               # the last token is never fed back
    with pytest.raises(ValueError, match="positions"):
        eng.submit([1] * 15, SamplingParams(max_tokens=7))
    assert len(taken) == 1


# ---- the oracle against itself ---------------------------------------------------------------------------------
def randn(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def test_oracle_recurrences_carry_their_state():
    q, k, v, a = randn(9, 4), randn(9, 4, seed=1), randn(9, 3, seed=2), torch.rand(9, 4, dtype=F64)
    whole, end = plain.gated_linear(q, k, v, a)
    o1, s = plain.gated_linear(q[:2], k[:2], v[:2], a[:2])
    o2, s = plain.gated_linear(q[2:], k[2:], v[2:], a[2:], s)
    assert torch.allclose(torch.cat([o1, o2]), whole) and torch.allclose(s, end)
    i, f = randn(9, seed=3) * 3, plain.log_sigmoid(randn(9, seed=4))
    whole, end = plain.mlstm_memory(q, k, v, i, f)
    o1, s = plain.mlstm_memory(q[:5], k[:5], v[:5], i[:5], f[:5])
    o2, s = plain.mlstm_memory(q[5:], k[5:], v[5:], i[5:], f[5:], s)
    assert torch.allclose(torch.cat([o1, o2]), whole) and all(torch.allclose(x, y) for x, y in zip(s, end))


def test_oracle_running_maximum_only_rescales():
    """Without the maximum the memory is a plain decayed sum; the floor of the denominator is then 1."""
    q, k, v, i, f = randn(12, 4), randn(12, 4, seed=1), randn(12, 3, seed=2), randn(12, seed=3) * 4, plain.log_sigmoid(randn(12, seed=4))
    got, (_, _, m) = plain.mlstm_memory(q, k, v, i, f)
    s, n = torch.zeros(4, 3, dtype=F64), torch.zeros(4, dtype=F64)
    for t in range(12):
        s, n = f[t].exp() * s + i[t].exp() * k[t][:, None] * v[t], f[t].exp() * n + i[t].exp() * k[t]
    want = s.T @ q[11] / torch.maximum((n @ q[11]).abs(), torch.ones((), dtype=F64))
    assert torch.allclose(got[11], want, rtol=1e-5)
    assert m >= i[11]


def test_oracle_poly_norm_and_grouped_norm():
    z = torch.tensor([[1.0, -2.0, 3.0]], dtype=F64)
    rms = lambda v: v / (v * v).mean().sqrt()
    want = 2 * rms(z) + 3 * rms(z ** 2) + 5 * rms(z ** 3) + 7
    assert torch.allclose(plain.poly_norm(z, torch.tensor([2.0, 3.0, 5.0, 7.0], dtype=F64), 0.0), want)
    x = torch.tensor([[3.0, 3.0, -8.0, 8.0]], dtype=F64)
    assert torch.allclose(plain.rms_norm(x, None, 0.0, 2), torch.tensor([[1.0, 1.0, -1.0, 1.0]], dtype=F64))


def test_oracle_streams_mix_from_row_to_column():
    X, y = torch.tensor([[[1.0]], [[10.0]]], dtype=F64), torch.tensor([[100.0]], dtype=F64)
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64)
    new = plain.connect_out(X, y, mix, torch.tensor([0.0, 1.0], dtype=F64))
    assert new.flatten().tolist() == [31.0, 142.0]
    assert plain.connect_in(X, torch.tensor([2.0, 5.0], dtype=F64)).item() == 52.0


def test_oracle_is_causal():
    cfg = config([latent_layer(), gla_layer(), lstm_layer(), latent_layer(kv_from=0)])
    m = plain.OracleVebonex(tensors(cfg), cfg)
    toks = list(range(20))
    assert torch.allclose(m.forward(toks)[:11], m.forward(toks[:11]))
