"""Nagavik configurations drawn at random from fixed seeds (`nagavik_tiny.random_config`): 1 to 6 layers in any order;
state-space mixers of 1 to 12 heads in 1 to 3 groups with states of 3 to 128 and values of 4 to 64, convolutions over 1 to 7
tokens, norms in 1 to 8 parts; attention of 1 to 15 heads on 1 to 3 key/value heads with key sizes 8 to 128 and value sizes
of their own, bounded or not; 1 to 9 experts of which some or all are chosen, with and without a shared one; layers without
a feed-forward; widths that are no multiples of 8, 4 or 2.  Each whole beside another request, in portions, and with its last
tokens one by one, in both precisions."""
import functools

import numpy as np
import pytest

import plain_nagavik as plain
import nagavik_tiny as nt
from test_gpu_nagavik import check

pytestmark = pytest.mark.gpu

SEEDS = list(range(20))


@functools.lru_cache(maxsize=None)
def case_of(seed):
    cfg = nt.random_config(seed)
    weights = nt.make_weights(cfg, 600 + seed)
    rng = np.random.default_rng(seed)
    toks, other = rng.integers(0, cfg["vocab"], 150).tolist(), rng.integers(0, cfg["vocab"], 30).tolist()
    return cfg, weights, toks, other, plain.forward(cfg, weights, toks), plain.forward(cfg, weights, other)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", SEEDS)
def test_random_configuration(tmp_path, seed, dtype):
    from alpacca_b200.engine.engine import Engine
    from alpacca_b200.engine.loading import load_model_dir
    from alpacca_b200.engine.step import StepEntry
    cfg, weights, toks, other, want, want_other = case_of(seed)
    folder = nt.write_model_dir(tmp_path / "m", cfg, weights)
    eng = Engine(load_model_dir(folder, dtype, "cuda", max_positions=512), max_tokens=1024, max_slots=3)

    def run(entries):
        out = eng.step([StepEntry(s, t, list(range(len(t)))) for s, t in entries]).cpu().numpy()
        eng.wait()
        return out
    a, b = eng.alloc_slot(), eng.alloc_slot()
    both = run([(b, other), (a, toks)])
    check(both[:30], want_other, dtype, f"seed {seed}: the short request of a batch")
    check(both[30:], want, dtype, f"seed {seed}: whole")
    eng.free_slot(a)
    eng.free_slot(b)
    a = eng.alloc_slot()
    got = [run([(a, toks[:3])]), run([(a, toks[3:5])]), run([(a, toks[5:70])]), run([(a, toks[70:110])])]
    got += [run([(a, [t])]) for t in toks[110:]]
    check(np.concatenate(got), want, dtype, f"seed {seed}: in portions and token by token")
    eng.free_slot(a)
    eng.cache.check()
