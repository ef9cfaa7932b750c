"""The Nagavik decoder without a GPU: configuration faults, tensor names and shapes, cache entries, what is taken into a
weight when it is loaded, and the plain implementation against hand-made cases."""
import copy

import numpy as np
import pytest
import torch

import nagavik_tiny as nt
import plain_nagavik as plain
from alpacca_b200.config import ConfigError, config_from_dict
from alpacca_b200.engine.loading import build_model, random_model
from alpacca_b200.parts.base import KVSpec, StateSpec


@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_tensor_names_and_shapes(name):
    model = build_model(copy.deepcopy(nt.CONFIGS[name]), torch.float32, "cpu", 128)
    specs = {s.name: tuple(s.shape) for s in model.param_specs() if not s.absent}
    assert specs == nt.tensor_shapes(nt.CONFIGS[name])


def test_random_configurations_are_valid_and_differ():
    seen = set()
    for seed in range(40):
        cfg = nt.random_config(seed)
        model = build_model(copy.deepcopy(cfg), torch.float32, "cpu", 128)
        specs = {s.name: tuple(s.shape) for s in model.param_specs() if not s.absent}
        assert specs == nt.tensor_shapes(cfg), seed
        seen.add(str(cfg["layers"]))
    assert len(seen) == 40


def test_cache_entries():
    model = build_model(copy.deepcopy(nt.TINY_A), torch.float32, "cpu", 256)
    assert model.cache_entry_specs() == [
        StateSpec((4, 16, 12), torch.float32), StateSpec((3, 48 + 64), torch.float32), KVSpec(2, 16, None, value_heads=2, value_dim=24),
        StateSpec((6, 24, 8), torch.float32), StateSpec((1, 48 + 144), torch.float32), KVSpec(1, 20, None, value_heads=1, value_dim=12)]
    assert model.entries_of_run == [[0, 1], [2], [3, 4], [5]]
    # one tap keeps no inputs
    b = build_model(copy.deepcopy(nt.TINY_B), torch.float32, "cpu", 256)
    assert b.entries_of_run == [[0], [1], [2, 3]] and b.cache_entry_specs()[1] == StateSpec((3, 5, 20), torch.float32)


def test_positions_bounds_and_the_configuration_written_back():
    cfg = config_from_dict(copy.deepcopy(nt.TINY_B))
    assert cfg.max_positions == 260 and build_model(cfg, torch.float32, "cpu", 1000).opts.max_positions == 260
    assert config_from_dict(cfg.to_dict()) == cfg and cfg.logit_softcap is None
    a = build_model(copy.deepcopy(nt.TINY_A), torch.float32, "cpu", 64)
    att = a.spec.layers[1].mixer
    assert att.bound[1] == 3.0 and att.bound[0].tolist() == pytest.approx([2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8])
    six = a.spec.layers[3].mixer.bound[0].tolist()
    assert six == pytest.approx([2.0 ** (-8 * h / 6) for h in range(1, 7)])
    assert a.spec.head.softcap == 9.0 and build_model(copy.deepcopy(nt.TINY_B), torch.float32, "cpu", 64).spec.layers[0].mixer.bound[1] == 0.0


def test_what_loading_lays_out():
    """The layer scale is in the weight of the norm after the sub-layer; stacked experts are padded with units that add
    nothing; the convolution's weights are turned over."""
    model = random_model(copy.deepcopy(nt.TINY_A), 3, torch.float32, "cpu", 64, std=0.3)
    from alpacca_b200.weights import RandomSource
    src = RandomSource(model.param_specs(), 3, torch.float32, std=0.3)
    blk = model.spec.layers[0]
    assert torch.allclose(blk.post1.weight, src.get("l0.norm1b") * src.get("l0.ls1"))
    assert torch.allclose(blk.post2.weight, src.get("l0.norm2b") * src.get("l0.ls2"))
    assert torch.equal(blk.mixer.conv, src.get("l0.mix.conv").t())
    ffn = blk.ffn
    up, down = ffn.up.view(6, 32, 40), ffn.down.view(6, 40, 32)
    assert torch.equal(up[4, :20], src.get("l0.mlp.e4.up")) and torch.equal(down[4, :, :20], src.get("l0.mlp.e4.down"))
    assert not up[:, 20:].any() and not down[:, :, 20:].any()


def test_gated_experts_are_laid_out_in_groups():
    from alpacca_b200.parts import BuildOptions, ScoredExperts
    from alpacca_b200.weights import Fetcher, RandomSource
    part = ScoredExperts(BuildOptions(torch.float32, "cpu", 64), 12, 20, 3, 2, "m", activation="silu", shared_inner=8,
                         expert_names=("e{}.gate", "e{}.up", "e{}.down"), shared_names=("shared.gate", "shared.up", "shared.down"))
    src = RandomSource(part.param_specs(), 5, torch.float32)
    part.load(Fetcher(src, "cpu", torch.float32))
    w = part.up.view(3, 4, 2, 8, 12)
    assert torch.equal(w[1, 1, 0], src.get("m.e1.gate")[8:16]) and torch.equal(w[1, 2, 1, :4], src.get("m.e1.up")[16:20])
    assert part.shared_up.shape == (32, 12) and torch.equal(part.shared_up[8:16], src.get("m.shared.up"))


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="gla"), "not supported"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mixer"].update(groups=3), "share"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=5), "norm"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "share"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "chosen"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "shared.ff"),
    (lambda c: c["layers"][2]["mlp"].update(kind="swiglu"), "dense"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c.update(logit_softcap=-1), "logit_softcap"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_faults_are_named(change, word):
    cfg = copy.deepcopy(nt.TINY_A)
    change(cfg)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(cfg)


def test_parts_refuse_what_they_cannot_do():
    from alpacca_b200.parts import BuildOptions, MapsAttention, StateSpaceMixer
    o = BuildOptions(torch.float32, "cpu", 64)
    with pytest.raises(ValueError, match="slopes"):
        MapsAttention(o, 8, 2, 1, 4, 4, None, "m", 1.0, 1e-5, slopes=[0.5])
    with pytest.raises(ValueError, match="fixed"):
        MapsAttention(o, 8, 2, 1, 4, 4, None, "m", 1.0, 1e-5, sink=True, fixed_sink=0.0)
    with pytest.raises(ValueError, match="penalty"):
        MapsAttention(o, 8, 2, 1, 4, 4, None, "m", 1.0, 1e-5, softcap=3.0, distance=("r1", "r2"))
    with pytest.raises(ValueError, match="parts"):
        StateSpaceMixer(o, 8, 2, 5, 4, 1, 2, 4, 1e-5, "m")
    with pytest.raises(ValueError, match="convolution"):
        StateSpaceMixer(o, 8, 2, 4, 4, 1, 18, 1, 1e-5, "m")


# -- the plain implementation against cases made by hand -------------------------------------------------------
def test_plain_convolution_and_walk():
    x = np.arange(1.0, 6.0)[:, None] * np.array([[1.0, 10.0]])
    y = plain.causal_conv(x, np.array([[0.5, 0.0, 1.0], [1.0, 1.0, 1.0]]), np.array([0.0, 7.0]))
    assert np.allclose(y[:, 0], [1, 2, 3.5, 5, 6.5]) and np.allclose(y[:, 1], 7 + np.array([10, 30, 60, 90, 120]))
    # one head, state of one number: S_t = a S + dt b x, y = c S + D x with a = exp(-2 dt)
    dt = np.array([[0.5], [0.1], [1.0]])
    y, S = plain.ssm_walk(np.array([1.0, 2.0, 3.0]).reshape(3, 1, 1), np.array([1.0, -1.0, 2.0]).reshape(3, 1, 1),
                          np.array([1.0, 1.0, 10.0]).reshape(3, 1, 1), dt, np.log([2.0]), np.array([100.0]), 1)
    s = [0.5]
    s.append(np.exp(-0.2) * s[0] - 0.2)
    s.append(np.exp(-2.0) * s[1] + 6.0)
    assert np.allclose(y[:, 0, 0], [s[0] + 100, s[1] + 200, 10 * s[2] + 300]) and np.allclose(S, s[2])


def test_plain_heads_read_their_group():
    rng = np.random.default_rng(0)
    x, B, C = rng.normal(size=(4, 4, 3)), rng.normal(size=(4, 2, 5)), rng.normal(size=(4, 2, 5))
    dt, A, D = rng.uniform(0.1, 1, (4, 4)), rng.normal(size=4), np.zeros(4)
    y, _ = plain.ssm_walk(x, B, C, dt, A, D, 2)
    for a in range(4):
        one, _ = plain.ssm_walk(x[:, a:a + 1], B[:, a // 2:a // 2 + 1], C[:, a // 2:a // 2 + 1], dt[:, a:a + 1], A[a:a + 1], D[:1], 1)
        assert np.allclose(one[:, 0], y[:, a])


def test_plain_gate_comes_before_the_norm():
    y, z = np.array([[3.0, 4.0, 1.0, 0.0]]), np.array([[1.0, -1.0, 2.0, 5.0]])
    u = y * z / (1 + np.exp(-z))
    got = plain.gated_group_norm(y, z, np.array([1.0, 1.0, 2.0, 2.0]), 2, 0.0)
    assert np.allclose(got[0, :2], u[0, :2] / np.sqrt((u[0, :2] ** 2).mean()))
    assert np.allclose(got[0, 2:], 2 * u[0, 2:] / np.sqrt((u[0, 2:] ** 2).mean()))


def test_plain_attention_weights():
    q, k = np.array([[0.0], [2.0], [1.0]]), np.array([[1.0], [3.0], [-1.0]])
    p = plain.attention_weights(q, k, 0.5, 2.0, 0.25)
    s = np.array([2 * np.tanh(0.5 / 2) - 0.5, 2 * np.tanh(1.5 / 2) - 0.25, 2 * np.tanh(-0.5 / 2)])
    assert np.allclose(p[2], np.exp(s) / (1 + np.exp(s).sum())) and np.allclose(p[0], [0.5, 0, 0])
    assert np.allclose(plain.slopes(4), [0.25, 0.0625, 2.0 ** -6, 2.0 ** -8])


def test_plain_experts_take_the_weight_on_their_input():
    h, one = np.array([[2.0]]), np.ones((1, 1))
    w = {"router": np.array([[1.0], [-1.0], [0.5]])}
    for e in range(3):
        w.update({f"e{e}.up": one, f"e{e}.down": one * (e + 1)})
    s = 1 / (1 + np.exp(-np.array([2.0, 1.0])))
    got = plain.experts(h, w, {"router": {"experts": 3, "top": 2}})
    assert np.allclose(got, (2 * s[0]) ** 2 * 1 + (2 * s[1]) ** 2 * 3)
    w.update({"shared.up": -one, "shared.down": one})
    assert np.allclose(plain.experts(h, w, {"router": {"experts": 3, "top": 2}, "shared": {"ff": 1}}), got)
    assert np.allclose(plain.gelu_tanh(np.array([0.0, 1.0, -1.0])), [0.0, 0.84119199, -0.15880801])
