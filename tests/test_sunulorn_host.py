"""Host side of the Sunulorn design (no GPU): configuration reader, weight layout, borrowed keys, and the plain oracle checked against itself
and against mistakes planted in it."""
import pytest
import torch

from mini_vllm_b200 import ops
from mini_vllm_b200.config import Config, sunulorn_shape
from mini_vllm_b200.models.layers.branches import AttentionBranch, alibi_slopes
from oracle import sunulorn as plain
from tests.replay_helpers import row_errors, write_checkpoint
from tests.sunulorn_helpers import CONFIGS, config, conv_layer, dense, distance_layer, moe, tensors, window_layer

F64 = torch.float64


def test_config_reader(tmp_path):
    cfg = CONFIGS["several"]
    path = write_checkpoint(tmp_path / "m", cfg, tensors(cfg))
    hf = Config(model=path, max_model_len=777).hf_config
    assert hf.architectures == ["Sunulorn"] and hf.dtype == torch.bfloat16 and hf.embedding_scale == 3.3
    assert hf.max_position_embeddings == 777 and hf.rms_norm_eps == 1e-5 and hf.layers == cfg["layers"]
    assert Config(model=path, dtype=torch.float32).hf_config.dtype == torch.float32


def cpu_model(cfg, weights, dtype=torch.float32):
    from mini_vllm_b200.config.native import sunulorn_config
    from mini_vllm_b200.models.models import get_model_class
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        model = get_model_class("Sunulorn")(sunulorn_config(cfg, None, dtype))
    finally:
        torch.set_default_dtype(prev)
    model.load_weights(weights.items())
    return model


def test_weights_that_are_missing_or_unknown_are_refused():
    cfg = CONFIGS["several"]
    w = tensors(cfg)
    for name in ("l1.mix.k.conv", "l0.mlp.e3.up", "l0.mlp.shared.sg", "l3.mix.o.b", "l2.mix.sink", "l2.norm2", "l2.mix.q.b"):
        with pytest.raises(KeyError, match=name):
            cpu_model(cfg, {k: v for k, v in w.items() if k != name})
    for name in ("l2.mix.k", "l1.mix.v", "l4.norm2", "l3.mlp.shared.sg"):              # borrowed; keys that are values; no feed-forward; none shared
        with pytest.raises(KeyError, match=name):
            cpu_model(cfg, {**w, name: w["l0.mix.k"]})
    with pytest.raises(ValueError, match="attention_9"):
        cpu_model({**cfg, "layers": [{"type": "attention_9", "mixer": conv_layer()["mixer"], "mlp": None}]}, w)
    with pytest.raises(ValueError, match="sparse"):
        cpu_model(config([conv_layer(mlp={"kind": "sparse"})]), w)
    with pytest.raises(ValueError, match="experts"):
        cpu_model(config([conv_layer(mlp=moe(3, 4))]), w)


@pytest.mark.parametrize("bad", [[distance_layer(kv_from=0)], [distance_layer(), distance_layer(kv_from=0), distance_layer(kv_from=1)],
                                 [conv_layer(), distance_layer(kv_from=0)], [distance_layer(), distance_layer(dim=20, kv_from=0)],
                                 [distance_layer(), distance_layer(heads=6, kv=2, kv_from=0)], [distance_layer(kv_from=1), distance_layer()]])
def test_keys_can_only_come_from_an_earlier_layer_that_makes_them(bad):
    with pytest.raises(ValueError, match="keys"):
        cpu_model(config(bad), tensors(config(bad)))


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_packed_projections_hold_every_weight_once(name, dtype):
    """The padded, concatenated projections are the checkpoint's matrices: same energy, blocks at multiples of 8."""
    cfg = CONFIGS[name]
    w = tensors(cfg)
    energy = lambda *ts: sum(float(t.double().pow(2).sum()) for t in ts)
    of = lambda *names: energy(*(w[n] for n in names if n in w))
    for i, layer in enumerate(cpu_model(cfg, w, dtype).layers):
        p, mixer = f"l{i}.mix.", layer.mixer
        branch, mlp = mixer.branches["mixer"], cfg["layers"][i]["mlp"]
        assert energy(mixer.in_proj) == pytest.approx(of(*(p + n for n in "qkvg")), rel=1e-6)
        downs = [] if mlp is None else ["mlp.down"] if mlp["kind"] == "dense" else ["mlp.shared.down"]
        assert energy(mixer.out_proj) == pytest.approx(of(p + "o", *(f"l{i}.{n}" for n in downs)), rel=1e-6)
        if branch.in_bias:
            assert energy(mixer.in_bias) == pytest.approx(of(*(f"{p}{n}.b" for n in "qkv")), rel=1e-6)
        if branch.taps:
            assert energy(branch.conv_weight) == pytest.approx(of(p + "q.conv", p + "k.conv"), rel=1e-6)
        assert all(s % 8 == 0 for s in mixer.in_sizes + mixer.out_sizes + branch.in_sizes)
        assert hasattr(branch.attn, "k_cache") == ("kv_from" not in cfg["layers"][i]["mixer"])
        if mlp is not None and mlp["kind"] == "moe":
            names = [f"l{i}.mlp.e{e}." for e in range(mlp["router"]["experts"])]
            assert energy(mixer.feed.gate_up) == pytest.approx(of(*(n + k for n in names for k in ("gate", "up"))), rel=1e-6)
            assert energy(mixer.feed.down) == pytest.approx(of(*(n + "down" for n in names)), rel=1e-6)


@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("dim,rot,d", [(20, 20, 32), (28, 10, 128), (9, 0, 16)])
def test_laid_out_heads_pair_the_rotated_coordinates(interleaved, dim, rot, d):
    b = AttentionBranch(2, 1, dim, dim, 1.0, None, rot, d, interleaved=interleaved)
    place = b._layout().tolist()
    assert len(set(place)) == dim and all(0 <= p < d for p in place)
    for i in range(rot // 2):
        u, v = (2 * i, 2 * i + 1) if interleaved else (i, i + rot // 2)
        assert place[u] == i and place[v] == i + d // 2
    for p in place[rot:]:                                                            # what is not rotated shares no angle
        assert p % (d // 2) >= rot // 2


def test_slopes_of_any_head_count():
    for heads in (1, 3, 8, 12):
        want = [plain.alibi_slope(h, heads) for h in range(heads)]
        assert torch.allclose(alibi_slopes(heads).double(), torch.tensor(want, dtype=F64), rtol=1e-7)
    assert alibi_slopes(8).tolist() == [2.0 ** -(h + 1) for h in range(8)]


def test_only_convolutions_hold_state():
    assert cpu_model(CONFIGS["several"], tensors(CONFIGS["several"])).recurrent
    cfg = config([distance_layer(mlp=dense()), window_layer()])
    assert not cpu_model(cfg, tensors(cfg)).recurrent
    assert not cpu_model(CONFIGS["ones"], tensors(CONFIGS["ones"])).recurrent            # one tap: nothing is carried


def test_random_weights_have_the_checkpoint_s_names():
    cfg = CONFIGS["several"]
    hf = sunulorn_shape(cfg["layers"], cfg["width"], cfg["vocab"], dtype=torch.float32)
    from mini_vllm_b200.models.models import get_model_class
    model = get_model_class("Sunulorn")(hf)
    shapes = {k: tuple(v.shape) for k, v in model.random_tensors(1)}
    assert shapes == {k: tuple(v.shape) for k, v in tensors(cfg).items()}
    model.init_random(1)


def test_tiles_grow_with_the_rows_per_expert():
    assert [ops.moe_block_rows(r, 8, torch.bfloat16) for r in (8, 120, 128, 320, 60000)] == [32, 32, 64, 128, 128]
    assert ops.moe_block_rows(60000, 8, torch.float32) == 64


# ---- the oracle against itself, and against planted mistakes ------------------------------------------------------------
def randn(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def test_oracle_is_causal():
    cfg = CONFIGS["several"]
    m = plain.OracleSunulorn(tensors(cfg), cfg)
    toks = list(range(60))
    assert torch.allclose(m.forward(toks)[:47], m.forward(toks[:47]))


def test_oracle_sink_is_a_key_without_a_value():
    q, k, v, s = randn(6, 1, 4), randn(6, 1, 4, seed=1), randn(6, 1, 3, seed=2), torch.tensor([0.7], dtype=F64)
    seen = plain.visible(6, None, 0)
    got = plain.attention(q, k, v, 0.5, seen, s)
    for t in range(6):
        e = torch.exp(q[t, 0] @ k[:t + 1, 0].T * 0.5)
        assert torch.allclose(got[t, 0], (e @ v[:t + 1, 0]) / (e.sum() + s.exp()))


def test_oracle_window_keeps_first_tokens():
    seen = plain.visible(30, 5, 3)
    assert seen[20].nonzero().flatten().tolist() == [0, 1, 2, 16, 17, 18, 19, 20]
    assert seen[4].nonzero().flatten().tolist() == [0, 1, 2, 3, 4] and seen[1].nonzero().flatten().tolist() == [0, 1]


def test_oracle_rotation_layouts():
    z = randn(5, 1, 6)
    perm = [0, 2, 1, 3, 4, 5]                                                        # interleaved pairs of 4 -> halves
    assert torch.allclose(plain.rotate(z, 4, 50.0, True)[..., perm], plain.rotate(z[..., perm], 4, 50.0, False))
    assert torch.equal(plain.rotate(z, 4, 50.0, True)[..., 4:], z[..., 4:])


def test_oracle_experts_weigh_the_input():
    h, w = randn(1, 3), {"router": randn(1, 3, seed=1), "e0.gate": randn(2, 3, seed=2), "e0.up": randn(2, 3, seed=3), "e0.down": randn(3, 2, seed=4)}
    m = {"expert": {"limit": 0.5}, "router": {"experts": 1, "top": 1}}
    x = torch.sigmoid(h @ w["router"].T) * h
    g, u = torch.clamp(x @ w["e0.gate"].T, max=0.5), torch.clamp(x @ w["e0.up"].T, -0.5, 0.5)
    assert torch.allclose(plain.experts(h, w, "", m), (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w["e0.down"].T)


MISTAKES = {
    "window one wider": lambda c: c["layers"][3]["mixer"]["mask"].update(size=38),
    "one more kept": lambda c: c["layers"][3]["mixer"]["mask"].update(keep_first=10),
    "no kept": lambda c: c["layers"][3]["mixer"]["mask"].update(keep_first=0),
    "limit": lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.9),
    "shared limit": lambda c: c["layers"][0]["mlp"]["shared"].update(limit=1.0),
    "one expert fewer": lambda c: c["layers"][0]["mlp"]["router"].update(top=1),
    "rotation": lambda c: c["layers"][1]["mixer"]["rot"].update(base=450.0),
    "scale": lambda c: c["layers"][2]["mixer"].update(scale=0.33),
    "borrowed elsewhere": lambda c: c["layers"][6]["mixer"].pop("kv_from"),
    "embedding": lambda c: c["embedding"].update(scale=3.0),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_mistakes_show_in_the_logits(name):
    """What the engine's tests allow between product and oracle is far less than any of these."""
    import copy
    cfg = CONFIGS["several"]
    w, wrong = tensors(cfg, seed=7), copy.deepcopy(cfg)
    MISTAKES[name](wrong)
    if name == "borrowed elsewhere":
        w = {**w, **{f"l6.mix.{n}": w[f"l5.mix.{n}"].flip(0) for n in ("k", "v", "k.b", "v.b")}}
    toks = [(7 * i * i + 3 * i) % 96 for i in range(80)]
    want = plain.OracleSunulorn(w, cfg).forward(toks)
    assert row_errors(plain.OracleSunulorn(w, wrong).forward(toks), want).max() > 3e-3
