"""Host side of the Rasezen design (no GPU): configuration reader, weight layout, what is refused, and the plain oracle checked against itself
and against mistakes planted in it."""
import copy

import pytest
import torch

from mini_vllm_b200.config import Config, rasezen_shape
from mini_vllm_b200.models.layers.branches import AttentionBranch, StateSpaceBranch
from mini_vllm_b200.models.layers.feedforward import ExpertFeed
from oracle import rasezen as plain
from tests.rasezen_helpers import CONFIGS, config, dense, moe, state_layer, tensors, window_layer
from tests.replay_helpers import row_errors, write_checkpoint

F64 = torch.float64


def test_config_reader(tmp_path):
    cfg = CONFIGS["several"]
    path = write_checkpoint(tmp_path / "m", cfg, tensors(cfg))
    hf = Config(model=path, max_model_len=777).hf_config
    assert hf.architectures == ["Rasezen"] and hf.dtype == torch.bfloat16 and hf.layers == cfg["layers"]
    assert hf.max_position_embeddings == 777 and hf.rms_norm_eps == 1e-4 and (hf.hidden_size, hf.vocab_size) == (88, 96)
    assert Config(model=path, dtype=torch.float32).hf_config.dtype == torch.float32


def cpu_model(cfg, weights, dtype=torch.float32):
    from mini_vllm_b200.config.native import rasezen_config
    from mini_vllm_b200.models.models import get_model_class
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        model = get_model_class("Rasezen")(rasezen_config(cfg, None, dtype))
    finally:
        torch.set_default_dtype(prev)
    model.load_weights(weights.items())
    return model


def test_weights_that_are_missing_or_unknown_are_refused():
    cfg = CONFIGS["several"]
    w = tensors(cfg)
    for name in ("l0.mix.conv.b", "l0.mlp.e3.up", "l0.mlp.correction", "l1.mix.q.norm", "l1.mix.v.b", "l1.mlp.act", "l2.mix.A_log", "l5.norm1"):
        with pytest.raises(KeyError, match=name):
            cpu_model(cfg, {k: v for k, v in w.items() if k != name})
    for name in ("l0.norm2", "l0.mlp.e5.up", "l3.mlp.shared.up", "l1.mix.o.b", "l2.mlp.up"):      # one norm; identity; none shared; no bias; no feed-forward
        with pytest.raises(KeyError, match=name):
            cpu_model(cfg, {**w, name: w["l1.mix.k"]})
    with pytest.raises(ValueError, match="mamba9"):
        cpu_model(config([{**state_layer(), "type": "mamba9"}]), w)
    with pytest.raises(ValueError, match="sparse"):
        cpu_model(config([state_layer(mlp={"kind": "sparse"})]), w)
    with pytest.raises(ValueError, match="experts"):
        cpu_model(config([state_layer(mlp=moe(3, 5, identity=1))]), w)
    for bad in (state_layer(heads=6, groups=4), state_layer(heads=6, vdim=12, norm_groups=5)):
        with pytest.raises(ValueError, match="groups"):
            cpu_model(config([bad]), w)
    with pytest.raises(ValueError, match="epsilon"):
        AttentionBranch(2, 1, 8, 8, 1.0, None, 0, 16, norm_eps=1e-5, row_norm_eps=1e-5)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_packed_projections_hold_every_weight_once(name, dtype):
    """The padded, concatenated projections are the checkpoint's matrices: same energy, blocks at multiples of 8."""
    cfg = CONFIGS[name]
    w = tensors(cfg)
    energy = lambda *ts: sum(float(t.double().pow(2).sum()) for t in ts)
    of = lambda *names: energy(*(w[n] for n in names if n in w))
    same = lambda t, *names: energy(t) == pytest.approx(of(*names), rel=1e-6)
    model = cpu_model(cfg, w, dtype)
    assert (model.norm == w["final.norm"]).all()
    for i, layer in enumerate(model.layers):
        p, mixer, mlp = f"l{i}.mix.", layer.mixer, cfg["layers"][i]["mlp"]
        branch, connection = mixer.branches["mixer"], layer.connections[0]
        assert (connection.norm == w[f"l{i}.norm1"]).all() and connection.feed_norm is None
        if isinstance(branch, StateSpaceBranch):
            assert same(mixer.in_proj, p + "in") and same(branch.conv_weight, p + "conv") and same(branch.conv_bias, p + "conv.b")
        else:
            assert same(mixer.in_proj, *(p + n for n in "qkv")) and same(mixer.in_bias, *(f"{p}{n}.b" for n in "qkv"))
            assert same(branch.q_norm, p + "q.norm") and same(branch.k_norm, p + "k.norm")
        downs = [] if mlp is None else ["mlp.down"] if mlp["kind"] == "dense" else ["mlp.shared.down"]
        assert same(mixer.out_proj, p + "o", *(f"l{i}.{n}" for n in downs))
        assert all(s % 8 == 0 for s in mixer.in_sizes + mixer.out_sizes + branch.in_sizes)
        if mlp is not None and mlp["kind"] == "moe":
            names = [f"l{i}.mlp.e{e}." for e in range(mlp["router"]["experts"])]
            assert same(mixer.feed.gate_up, *(n + k for n in names for k in ("gate", "up"))) and same(mixer.feed.down, *(n + "down" for n in names))
            assert mixer.feed.router.shape[0] == mixer.feed.correction.numel() == len(names) + mlp["router"]["identity"]
        elif mlp is not None:
            p, q = w[f"l{i}.mlp.act"].double()
            assert torch.allclose(mixer.feed.act.double(), torch.stack([plain.softplus(p), 0.5 + plain.softplus(q)]), rtol=1e-6)


def test_state_space_rows_and_channels_keep_their_places():
    """z | x | B | C | dt in the projection, x | B | C in the convolution, each block padded to a multiple of 8."""
    b = StateSpaceBranch(5, 1, 3, 3, 2, 1, 1e-5)
    names = {"in": torch.arange(15 + 21 + 5).float()[:, None] + 1, "conv": torch.arange(21.0)[:, None] * 2 + torch.tensor([[0.0, 1.0]]) + 1,
             "conv.b": torch.arange(21.0) + 1, "o": torch.ones(1, 15), "A_log": torch.zeros(5), "dt_bias": torch.zeros(5), "D": torch.ones(5),
             "norm": torch.ones(15)}
    rows, cols = b.load(lambda n: names[n])
    assert rows.flatten().tolist() == [*range(1, 16), 0, *range(16, 31), 0, 31, 32, 33, *[0] * 5, 34, 35, 36, *[0] * 5, *range(37, 42), 0, 0, 0]
    assert b.conv_bias.tolist() == [*range(1, 16), 0, 16, 17, 18, *[0] * 5, 19, 20, 21, *[0] * 5]
    assert b.conv_weight[0, :3].tolist() == [2, 4, 6] and b.conv_weight[1, :3].tolist() == [1, 3, 5]      # the token itself first
    assert cols.shape == (1, 16) and cols[0, 15] == 0


def test_only_state_space_layers_hold_state():
    assert cpu_model(CONFIGS["several"], tensors(CONFIGS["several"])).recurrent
    cfg = config([window_layer(mlp=dense()), window_layer(size=4)])
    assert not cpu_model(cfg, tensors(cfg)).recurrent
    specs = StateSpaceBranch(4, 2, 10, 6, 3, 1, 1e-5).state_specs(torch.bfloat16)
    assert specs == {"conv_state": ((2, 24 + 2 * 24), torch.bfloat16), "memory": ((4, 10, 8), torch.float32)}


@pytest.mark.parametrize("name", ["several", "wide"])
def test_random_weights_have_the_checkpoint_s_names(name):
    cfg = CONFIGS[name]
    hf = rasezen_shape(cfg["layers"], cfg["width"], cfg["vocab"], dtype=torch.float32)
    from mini_vllm_b200.models.models import get_model_class
    model = get_model_class("Rasezen")(hf)
    shapes = {k: tuple(v.shape) for k, v in model.random_tensors(1)}
    assert shapes == {k: tuple(v.shape) for k, v in tensors(cfg).items()}
    model.init_random(1)


def test_the_earlier_routing_is_the_default():
    feed = ExpertFeed(16, 8, 4, 2, 1.0, 1.7, 1.0)
    assert feed.correction is None and not feed.weigh_output and feed.routing.identity == 0 and not feed.routing.softmax and feed.routing.scale == 1.0


# ---- the oracle against itself, and against planted mistakes ------------------------------------------------------------
def randn(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def test_oracle_is_causal():
    cfg = CONFIGS["several"]
    m = plain.OracleRasezen(tensors(cfg), cfg)
    toks = list(range(60))
    assert torch.allclose(m.forward(toks)[:47], m.forward(toks[:47]))


def test_oracle_state_space_is_a_sum_over_the_past():
    """Unrolled: y_t = sum_s (c_t . b_s) dt_s e^{a (dt_{s+1} + .. + dt_t)} x_s + d x_t, head by head with its group's b and c."""
    t, heads, groups = 9, 4, 2
    x, b, c, dt = randn(t, heads, 3), randn(t, groups, 5, seed=1), randn(t, groups, 5, seed=2), randn(t, heads, seed=3).exp()
    a, d = -randn(heads, seed=4).exp(), randn(heads, seed=5)
    y = plain.state_space(x, b, c, dt, a, d)
    for h in range(heads):
        for i in range(t):
            want = d[h] * x[i, h]
            for s in range(i + 1):
                want = want + (c[i, h // 2] @ b[s, h // 2]) * dt[s, h] * torch.exp(a[h] * dt[s + 1:i + 1, h].sum()) * x[s, h]
            assert torch.allclose(y[i, h], want)


def test_oracle_norm_comes_behind_the_gate():
    y, z, w = randn(2, 6), randn(2, 6, seed=1), randn(6, seed=2)
    u = y * z * torch.sigmoid(z)
    want = torch.cat([u[:, :3] / (u[:, :3].pow(2).mean(1, keepdim=True) + 0.1).sqrt(), u[:, 3:] / (u[:, 3:].pow(2).mean(1, keepdim=True) + 0.1).sqrt()], 1)
    assert torch.allclose(plain.gated_group_norm(y, z, w, 2, 0.1), want * w)


def test_oracle_xielu():
    p, q = torch.tensor(0.3, dtype=F64), torch.tensor(-0.8, dtype=F64)
    for z in (-3.0, -1e-4, 0.0, 0.7):
        z = torch.tensor(z, dtype=F64)
        want = torch.log(1 + p.exp()) * z * z + z / 2 if z > 0 else (0.5 + torch.log(1 + q.exp())) * (z.exp() - 1 - z) + z / 2
        assert torch.allclose(plain.xielu(z, p, q), want, atol=1e-15)


def test_oracle_window_and_rotation():
    seen = plain.in_window(30, 5)
    assert seen[20].nonzero().flatten().tolist() == [16, 17, 18, 19, 20] and seen[1].nonzero().flatten().tolist() == [0, 1]
    assert torch.equal(plain.in_window(9, 1), torch.eye(9, dtype=torch.bool))
    z = randn(5, 1, 6)
    r = plain.rotate_half(z, 4, 50.0)
    assert torch.equal(r[..., 4:], z[..., 4:]) and torch.equal(r[0], z[0])
    assert torch.allclose(r[..., [0, 2]].norm(dim=-1), z[..., [0, 2]].norm(dim=-1))


def test_oracle_choice_and_weights():
    z, correction = torch.tensor([2.0, 1.0, 0.0, -1.0], dtype=F64), torch.tensor([-1.0, 0.0, 0.0, 0.5], dtype=F64)
    ids, s = plain.choose(z, correction, 2)
    assert ids.tolist() == [3, 1] and torch.allclose(s, torch.softmax(z, 0)[[3, 1]])


MISTAKES = {
    "window one wider": lambda c, w: c["layers"][4]["mixer"]["mask"].update(size=3),
    "rotation base": lambda c, w: c["layers"][1]["mixer"]["rot"].update(base=450.0),
    "rotated dims": lambda c, w: c["layers"][1]["mixer"]["rot"].update(dims=8),
    "scale": lambda c, w: c["layers"][1]["mixer"].update(scale=0.33),
    "norm groups": lambda c, w: c["layers"][0]["mixer"].update(norm_groups=6),
    "groups": lambda c, w: w.update({"l0.mix.in": torch.cat([w["l0.mix.in"][:144], w["l0.mix.in"][164:204], w["l0.mix.in"][144:164], w["l0.mix.in"][204:]])}),
    "router scale": lambda c, w: c["layers"][0]["mlp"]["router"].update(scale=1.5),
    "one expert fewer": lambda c, w: c["layers"][0]["mlp"]["router"].update(top=1),
    "no correction": lambda c, w: w.update({"l0.mlp.correction": torch.zeros(6)}),
    "conv bias": lambda c, w: w.update({"l0.mix.conv.b": torch.zeros(192)}),
    "value bias": lambda c, w: w.update({"l1.mix.v.b": torch.zeros(40)}),
    "skip": lambda c, w: w.update({"l2.mix.D": torch.zeros(5)}),
    "activation": lambda c, w: w.update({"l1.mlp.act": w["l1.mlp.act"].flip(0)}),
    "eps": lambda c, w: c["norm"].update(eps=1e-2),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_mistakes_show_in_the_logits(name):
    """What the engine's tests allow between product and oracle is far less than any of these."""
    cfg = CONFIGS["several"]
    w = tensors(cfg, seed=7)
    wrong, ww = copy.deepcopy(cfg), dict(w)
    MISTAKES[name](wrong, ww)
    toks = [(7 * i * i + 3 * i) % 96 for i in range(80)]
    want = plain.OracleRasezen(w, cfg).forward(toks)
    assert row_errors(plain.OracleRasezen(ww, wrong).forward(toks), want).max() > 3e-3
