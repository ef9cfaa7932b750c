"""The Ponusun decoder without a GPU: configuration faults, tensor names and shapes, the schedule and its cache entries,
random weights, and the plain implementation against hand-made cases."""
import copy

import numpy as np
import pytest
import torch

import plain_ponusun as plain
import ponusun_tiny as pt
from alpacca_b200.config import ConfigError, config_from_dict
from alpacca_b200.engine.loading import build_model, random_model
from alpacca_b200.parts.base import KVSpec, StateSpec


@pytest.mark.parametrize("name", list(pt.CONFIGS))
def test_tensor_names_and_shapes(name):
    model = build_model(copy.deepcopy(pt.CONFIGS[name]), torch.float32, "cpu", 128)
    specs = {s.name: tuple(s.shape) for s in model.param_specs() if not s.absent}
    assert specs == pt.tensor_shapes(pt.CONFIGS[name])


def test_random_configurations_are_valid_and_differ():
    seen = set()
    for seed in range(40):
        cfg = pt.random_config(seed)
        model = build_model(copy.deepcopy(cfg), torch.float32, "cpu", 128)
        specs = {s.name: tuple(s.shape) for s in model.param_specs() if not s.absent}
        assert specs == pt.tensor_shapes(cfg), seed
        seen.add(str(cfg["layers"]))
    assert len(seen) == 40


def test_schedule_and_cache_entries():
    model = build_model(copy.deepcopy(pt.TINY_A), torch.float32, "cpu", 256)
    runs = model.spec.schedule
    assert [r.layer for r in runs] == [0, 1, 2, 3] and [r.reads_entry_of for r in runs] == [None, 0, None, 0]
    specs = model.cache_entry_specs()
    # every run keeps the convolution's rows itself; keys and values belong to the owner, kept for the widest reader
    conv = StateSpec((3, 40), torch.float32)
    assert specs == [conv, KVSpec(2, 16, 130, value_heads=2, value_dim=24), conv, conv,
                     KVSpec(1, 32, 5, value_heads=1, value_dim=16), conv]
    assert model.entries_of_run == [[0, 1], [2, 1], [3, 4], [5, 1]]
    # one tap keeps nothing; an owner without a window keeps everything
    b = build_model(copy.deepcopy(pt.TINY_B), torch.float32, "cpu", 256)
    assert b.cache_entry_specs()[0] == KVSpec(3, 20, None, value_heads=3, value_dim=12)
    assert b.entries_of_run == [[0], [1], [0], [2]]
    # a reader without a window makes its owner keep everything
    cfg = copy.deepcopy(pt.TINY_A)
    del cfg["layers"][1]["mixer"]["mask"]
    assert build_model(cfg, torch.float32, "cpu", 64).cache_entry_specs()[1].window is None


def test_the_position_table_bounds_the_sequences():
    cfg = config_from_dict(copy.deepcopy(pt.TINY_B))
    assert cfg.max_positions == 260 and build_model(cfg, torch.float32, "cpu", 1000).opts.max_positions == 260
    assert cfg.to_dict()["max_positions"] == 260 and config_from_dict(cfg.to_dict()) == cfg


def test_random_weights_are_usable():
    model = random_model(copy.deepcopy(pt.TINY_A), 3, torch.float32, "cpu", 64)
    for layer in (model.spec.layers[0], model.spec.layers[3]):
        table = layer.ffn.table
        assert int(table.min()) >= 0 and int(table.max()) < layer.ffn.E
        assert all(len(set(row)) == layer.ffn.top for row in table.tolist())
        assert len(set(map(tuple, table.tolist()))) > 1
        assert float(layer.mixer.penalty.min()) >= 0.0
        assert abs(float(layer.average.coef[-1]) - 1.0) < 0.2


def test_a_table_that_names_no_expert_is_refused():
    from alpacca_b200.parts import BuildOptions, TableExperts
    from alpacca_b200.weights import Fetcher, RandomSource
    from alpacca_b200.weights.loader import WeightError
    part = TableExperts(BuildOptions(torch.float32, "cpu", 64), 16, 8, 3, 2, 20, "m")
    src = RandomSource(part.param_specs(), 0, torch.float32)
    get = src.get
    src.get = lambda n: get(n) + 1 if n == "m.table" else get(n)
    with pytest.raises(WeightError, match="outside"):
        part.load(Fetcher(src, "cpu", torch.float32))


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="gla"), "not supported"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "share"),
    (lambda c: c["layers"][0]["mixer"].update(mask={}), "size"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(dim=8), "must equal those of layer 0"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "chosen"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "shared.ff"),
    (lambda c: c["layers"][2]["mlp"].update(kind="swiglu"), "dense"),
    (lambda c: c["canon"].pop("taps"), "taps"),
    (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_faults_are_named(change, word):
    cfg = copy.deepcopy(pt.TINY_A)
    change(cfg)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(cfg)


# -- the plain implementation against cases made by hand -------------------------------------------------------
def test_plain_convolution_and_average():
    x = np.arange(1.0, 6.0)[:, None] * np.array([[1.0, 10.0]])
    y = plain.input_conv(x, np.array([[0.5, 0.0, 1.0], [1.0, 1.0, 1.0]]))
    assert np.allclose(y[:, 0], x[:, 0] + [1, 2, 3.5, 5, 6.5]) and np.allclose(y[:, 1], x[:, 1] + [10, 30, 60, 90, 120])
    a, b, c = (np.full((2, 3), v) for v in (1.0, 10.0, 100.0))
    assert np.allclose(plain.depth_average([a, b, c], [0.5, -1.0, 2.0]), 0.5 - 10.0 + 200.0)
    with pytest.raises(ValueError):
        plain.depth_average([a, b], [1.0, 2.0, 3.0])


def test_plain_norm_over_whole_rows():
    mx = {"kv_heads": 2, "dim": 2, "vdim": 1}
    h = np.array([[3.0, 4.0]])
    w = {"k": np.array([[1.0, 0], [0, 1.0], [0, 0], [0, 0]]), "k.norm": np.array([1.0, 2.0, 1.0, 1.0]),
         "v": np.array([[1.0, 0], [0, 1.0]])}
    k, v = plain.keys_values(h, w, mx, 0.0)
    r = np.sqrt(25.0 / 4)                      # four numbers under one root, not two and two
    assert np.allclose(k[0], [[3 / r, 8 / r], [0, 0]]) and np.allclose(v[0, :, 0], [3, 4])


def test_plain_attention_penalty_and_window():
    rng = np.random.default_rng(1)
    T, mx = 6, {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.5, "mask": {"size": 3}}
    h = rng.normal(size=(T, 5))
    w = {"q": rng.normal(size=(8, 5)), "q.norm": rng.uniform(0.5, 2, 8), "k": rng.normal(size=(4, 5)), "k.norm": np.ones(4),
         "v": rng.normal(size=(3, 5)), "o": np.eye(6), "r1": np.array([0.7, 2.0]), "r2": np.array([0.3, 1.5])}
    kept = plain.keys_values(h, w, mx, 1e-5)
    got = plain.attention(h, w, mx, 1e-5, kept).reshape(T, 2, 3)
    q = plain.rms_norm(h @ w["q"].T, w["q.norm"], 1e-5).reshape(T, 2, 4)
    s = np.array([q[4, 1] @ kept[0][j, 0] * 0.5 - 2.0 * np.log(1 + 1.5 * (4 - j)) for j in (2, 3, 4)])
    p = np.exp(s) / np.exp(s).sum()
    assert np.allclose(got[4, 1], sum(a * kept[1][j, 0] for a, j in zip(p, (2, 3, 4))))
    assert np.allclose(got[0], kept[1][0])


def test_plain_experts_and_gelu():
    assert np.allclose(plain.gelu(np.array([0.0, 1.0, -1.0])), [0.0, 0.8413447460685429, -0.15865525393145707])
    h = np.array([[1.0], [2.0]])
    one = np.ones((1, 1))
    w = {f"e{e}.{n}": one * (e + 1 if n == "down" else 1) for e in range(3) for n in ("gate", "up", "down")}
    w.update({"table": np.array([[0, 2], [1, 2], [2, 1]]), "shared.gate": one, "shared.up": one, "shared.down": 10 * one,
              "shared.sg": 0 * one})
    mlp = {"router": {"experts": 3, "top": 2}, "shared": {"ff": 1}}
    a = plain.silu(h) * h
    assert np.allclose(plain.experts(h, [1, 0], w, mlp)[:, 0], [a[0, 0] * (2 + 3) / 2 + 5 * a[0, 0],
                                                                a[1, 0] * (1 + 3) / 2 + 5 * a[1, 0]])
