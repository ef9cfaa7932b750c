"""The Nagavik decoder in the engine against the plain implementation (tests/plain_nagavik.py): whole prompts, decoding
through pages and states, prompts in portions, unequal batches, slots and pages used again, long decoding across page and
chunk borders, the first tokens, greedy generation through the package's entry point (with sequences that end at stop
tokens), the command line and trace replay."""
import functools
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import plain_nagavik as plain
import nagavik_tiny as nt

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
DTYPES = ("float32", "bfloat16")
WEIGHTS = {name: nt.make_weights(cfg, seed) for (name, cfg), seed in zip(nt.CONFIGS.items(), (51, 52, 53))}


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("nagavik")
    return {name: nt.write_model_dir(root / name, nt.CONFIGS[name], w) for name, w in WEIGHTS.items()}


@functools.lru_cache(maxsize=None)
def _plain(name, tokens):
    return plain.forward(nt.CONFIGS[name], WEIGHTS[name], list(tokens))


def plain_logits(name, tokens):
    return _plain(name, tuple(int(t) for t in tokens))


def check(got, want, dtype, what):
    """32-bit: every logit.  bfloat16: by position (root mean square over the vocabulary, mean taken off, as a share of
    the logits' spread): rounding may turn an expert's choice at single positions, whose results the layers behind carry to
    the tokens after; a wrong key, state, tap or weight moves most positions by more."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    spread = max(float(want.std()), 1e-30)
    d = got - want
    if dtype == "float32":
        assert np.abs(d).max() <= 1e-4 * spread and np.abs(d).mean() <= 1e-5 * spread, \
            f"{what}: max |diff| {np.abs(d).max():.3e}, mean {np.abs(d).mean():.3e}, spread {spread:.3e}"
        return
    e = np.sqrt(((d - d.mean(axis=1, keepdims=True)) ** 2).mean(axis=1)) / spread
    over = int((e > 0.1).sum())
    assert e.mean() <= 0.03 and over <= max(1, int(0.04 * len(e))) and e.max() <= 0.5, \
        f"{what}: by position, mean {e.mean():.4f}, {over} of {len(e)} over 0.1, largest {e.max():.3f} of the spread"


def some_tokens(name, n, seed):
    return np.random.default_rng(seed).integers(0, nt.CONFIGS[name]["vocab"], n).tolist()


_ENGINES: dict = {}


def engine_of(dirs, name, dtype, max_tokens=2048, max_slots=6):
    from alpacca_b200.engine.engine import Engine
    from alpacca_b200.engine.loading import load_model_dir
    key = (name, dtype, max_tokens, max_slots)
    if key not in _ENGINES:
        _ENGINES[key] = Engine(load_model_dir(dirs[name], dtype, "cuda", max_positions=1024), max_tokens=max_tokens, max_slots=max_slots)
    return _ENGINES[key]


def run(eng, slot, tokens, want=None):
    from alpacca_b200.engine.step import StepEntry
    want = list(range(len(tokens))) if want is None else want
    out = eng.step([StepEntry(slot, tokens, want)]).cpu().numpy()
    eng.wait()
    return out


def in_cuts(eng, toks, cuts):
    s = eng.alloc_slot()
    try:
        got, at = [], 0
        for n in cuts:
            got.append(run(eng, s, toks[at:at + n]))
            at += n
        assert at == len(toks)
        return np.concatenate(got)
    finally:
        eng.free_slot(s)
        eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_whole_prompt(dirs, name, dtype):
    toks = some_tokens(name, 220, 1)
    check(in_cuts(engine_of(dirs, name, dtype), toks, (220,)), plain_logits(name, toks), dtype, f"{name} whole")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_prompt_then_long_decoding(dirs, name, dtype):
    """50 tokens at once, then 190 one by one: page borders are passed while decoding, and from the third step on the steps
    are graph replays."""
    toks = some_tokens(name, 240, 2)
    check(in_cuts(engine_of(dirs, name, dtype), toks, (50,) + (1,) * 190), plain_logits(name, toks), dtype, f"{name} decode")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_token_by_token_from_the_first(dirs, name, dtype):
    toks = some_tokens(name, 80, 4)
    check(in_cuts(engine_of(dirs, name, dtype), toks, (1,) * 80), plain_logits(name, toks), dtype, f"{name} token by token")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(nt.CONFIGS))
@pytest.mark.parametrize("cuts", [(2, 3, 59, 1, 64, 2, 19), (63, 2, 63, 22), (1, 1, 2, 126, 20), (65, 85), (2,) * 40,
                                  (3, 1, 1, 4, 1, 2, 140)])
def test_prompt_in_portions(dirs, name, dtype, cuts):
    toks = some_tokens(name, sum(cuts), 3)
    check(in_cuts(engine_of(dirs, name, dtype), toks, cuts), plain_logits(name, toks), dtype, f"{name} portions")


@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_the_cut_does_not_change_a_result(dirs, name):
    """32-bit: the logits of a prompt in one piece, in portions and token by token agree to rounding with each other."""
    toks = some_tokens(name, 100, 5)
    eng = engine_of(dirs, name, "float32")
    whole = in_cuts(eng, toks, (100,))
    for cuts in ((37, 63), (1,) * 100, (2,) * 50):
        assert np.abs(in_cuts(eng, toks, cuts) - whole).max() <= 2e-5 * whole.std()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_unequal_batch_against_each_alone(dirs, name, dtype):
    """Four prompts of 1, 70, 33 and 140 tokens in one step, then decoded together; the shorter requests end first."""
    from alpacca_b200.engine.step import StepEntry
    eng = engine_of(dirs, name, dtype)
    full = [some_tokens(name, n, 10 + i) for i, n in enumerate((9, 78, 39, 160))]
    first = (1, 70, 33, 140)
    slots = [eng.alloc_slot() for _ in full]
    try:
        got = [[] for _ in full]
        out = eng.step([StepEntry(s, t[:n], list(range(n))) for s, t, n in zip(slots, full, first)]).cpu().numpy()
        at = 0
        for i, n in enumerate(first):
            got[i].append(out[at:at + n])
            at += n
        pos = list(first)
        while any(p < len(t) for p, t in zip(pos, full)):
            live = [i for i in range(len(full)) if pos[i] < len(full[i])]
            out = eng.step([StepEntry(slots[i], [full[i][pos[i]]], [0]) for i in live]).cpu().numpy()
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1])
                pos[i] += 1
        eng.wait()
        for i, t in enumerate(full):
            check(np.concatenate(got[i]), plain_logits(name, t), dtype, f"{name} batch row {i}")
    finally:
        for s in slots:
            eng.free_slot(s)
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "c"])
def test_many_sequences_decoded_together(dirs, name, dtype):
    """Forty prompts of one to five tokens in one step, then six steps of all forty (the experts' grouped products in a step
    of one token each, from the third step on a graph replay with other tokens)."""
    from alpacca_b200.engine.step import StepEntry
    eng = engine_of(dirs, name, dtype, max_tokens=64 * 40, max_slots=40)
    full = [some_tokens(name, 7 + i % 5, 500 + i) for i in range(40)]
    slots = [eng.alloc_slot() for _ in full]
    try:
        got = [[] for _ in full]
        out = eng.step([StepEntry(s, t[:-6], list(range(len(t) - 6))) for s, t in zip(slots, full)]).cpu().numpy()
        at = 0
        for i, t in enumerate(full):
            got[i].append(out[at:at + len(t) - 6])
            at += len(t) - 6
        for k in range(6, 0, -1):
            out = eng.step([StepEntry(s, [t[-k]], [0]) for s, t in zip(slots, full)]).cpu().numpy()
            for i in range(40):
                got[i].append(out[i:i + 1])
        eng.wait()
        want = np.concatenate([plain_logits(name, t) for t in full])
        check(np.concatenate([np.concatenate(g) for g in got]), want, dtype, f"{name} forty together")
    finally:
        for s in slots:
            eng.free_slot(s)
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "c"])
def test_slots_and_pages_used_again(dirs, name, dtype):
    """A cache of five pages and two slots: every new sequence gets a slot and pages that another one has just given back,
    with its keys still in the pages and its matrices and inputs still among the states."""
    eng = engine_of(dirs, name, dtype, max_tokens=320, max_slots=2)
    for k, n in enumerate((130, 100, 3, 128, 65)):
        toks = some_tokens(name, n, 20 + k)
        s = eng.alloc_slot()
        other = eng.alloc_slot() if n <= 100 else None
        try:
            cut = max(1, n - 3)
            got = [run(eng, s, toks[:cut])]
            if other is not None:
                run(eng, other, some_tokens(name, 40, 99))       # a neighbour that writes pages and states too
            for p in range(cut, n):
                got.append(run(eng, s, [toks[p]]))
            check(np.concatenate(got), plain_logits(name, toks), dtype, f"{name} reuse {k}")
        finally:
            eng.free_slot(s)
            if other is not None:
                eng.free_slot(other)
        eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_first_tokens(dirs, name, dtype):
    toks = some_tokens(name, 5, 30)
    for cuts in ((5,), (1, 1, 1, 1, 1), (1, 2, 2), (2, 1, 2), (3, 2), (1, 4)):
        check(in_cuts(engine_of(dirs, name, dtype), toks, cuts), plain_logits(name, toks), dtype, f"{name} first tokens {cuts}")


def test_wanted_places_only(dirs):
    eng = engine_of(dirs, "b", "float32")
    toks = some_tokens("b", 90, 31)
    want = [0, 17, 63, 64, 89]
    s = eng.alloc_slot()
    try:
        check(run(eng, s, toks, want), plain_logits("b", toks)[want], "float32", "wanted places")
    finally:
        eng.free_slot(s)


def test_no_more_tokens_than_positions(dirs):
    """The table of positions ends the sequences: its last row is used, one token more is refused before any launch."""
    from alpacca_b200.cache import CacheFull
    n = nt.TINY_B["max_positions"]
    eng = engine_of(dirs, "b", "float32")
    toks = some_tokens("b", n, 33)
    s = eng.alloc_slot()
    try:
        check(np.concatenate([run(eng, s, toks[:n - 1]), run(eng, s, toks[n - 1:])]), plain_logits("b", toks), "float32", "the last place")
        with pytest.raises(CacheFull):
            run(eng, s, [1])
    finally:
        eng.free_slot(s)


@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_the_stream_after_every_layer(dirs, name):
    from alpacca_b200.engine.step import StepEntry
    eng = engine_of(dirs, name, "float32")
    toks = some_tokens(name, 40, 32)
    trace, seen = [], []
    plain.forward(nt.CONFIGS[name], WEIGHTS[name], toks, trace=trace)
    layers = eng.model.spec.layers

    def spy(original):
        def forward(stream, ctx, cache, write_cache=True):
            original(stream, ctx, cache, write_cache)
            assert stream.delta is None and stream.owed is None
            seen.append(stream.residual[:ctx.n_tokens].double().cpu().numpy())
        return forward
    s = eng.alloc_slot()
    try:
        for blk in layers:
            blk.forward = spy(blk.forward)
        eng.forget_graphs()
        eng.step([StepEntry(s, toks, [])])
        eng.wait()
    finally:
        for blk in layers:
            del blk.forward
        eng.free_slot(s)
        eng.forget_graphs()
    assert len(seen) == len(trace) == len(layers)
    for i, (a, b) in enumerate(zip(seen, trace)):
        assert np.abs(a - b).max() <= 2e-5 * max(1.0, np.abs(b).max()), f"stream after layer {i}"


def plain_greedy(name, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(plain_logits(name, toks)[-1])))
    return toks[len(prompt):]


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_greedy_generation_through_the_entry_point(dirs, name, graphs):
    """`Model.load` + `generate` (the scheduler, the graph decoder with its padded rows, the device sampler) give the plain
    implementation's greedy tokens, for prompts of unequal lengths that end at different steps."""
    from alpacca_b200.api import Model, generate
    from alpacca_b200.sampling import SamplerParams
    model = Model.load(dirs[name], n_ctx=256, dtype="float32", max_batch=4, progress=False)
    if not graphs:
        model.use_graphs = False
    prompts = [some_tokens(name, n, 40 + i) for i, n in enumerate((5, 70, 1))]
    res = generate(model, prompts, SamplerParams.greedy(), n_predict=12)
    for p, r in zip(prompts, res):
        assert r.token_ids == plain_greedy(name, p, 12)
    again = generate(model, prompts[::-1], SamplerParams.greedy(), n_predict=4)      # the same slots once more
    for p, r in zip(prompts[::-1], again):
        assert r.token_ids == plain_greedy(name, p, 4)


@pytest.mark.parametrize("name", list(nt.CONFIGS))
def test_generation_with_stop_tokens(dirs, name):
    """A stop token ends one sequence while steps run ahead for all of them: what the others keep per sequence must not
    move on twice.  The stop token is one that the greedy run of one prompt meets early and the others do not."""
    from alpacca_b200.api import Model, generate
    from alpacca_b200.sampling import SamplerParams
    model = Model.load(dirs[name], n_ctx=256, dtype="float32", max_batch=4, progress=False)
    prompts = [some_tokens(name, n, 140 + i) for i, n in enumerate((6, 40, 3, 17))]
    full = [plain_greedy(name, p, 16) for p in prompts]
    done = 0
    for i in range(len(prompts)):
        for at in (3, 5, 8):
            stop = full[i][at]
            ends = [f.index(stop) if stop in f else None for f in full]
            if sum(e is None for e in ends) < 2:
                continue
            res = generate(model, prompts, SamplerParams.greedy(), n_predict=16, stop_token_ids=[stop])
            for f, e, r in zip(full, ends, res):
                assert r.token_ids == (f if e is None else f[:e])
            done += 1
    assert done >= 2


def test_generation_in_bfloat16_runs(dirs):
    from alpacca_b200.api import Model, generate
    from alpacca_b200.sampling import SamplerParams
    model = Model.load(dirs["b"], n_ctx=256, dtype="bfloat16", max_batch=4, progress=False)
    res = generate(model, [some_tokens("b", 30, 50), some_tokens("b", 2, 51)], SamplerParams(temperature=0.8, seed=3), n_predict=20)
    assert all(len(r.token_ids) == 20 and all(0 <= t < nt.CONFIGS["b"]["vocab"] for t in r.token_ids) for r in res)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(dirs, dtype, tmp_path):
    name = "a"
    a, b = some_tokens(name, 70, 60), some_tokens(name, 9, 61)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]},
                                     {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:67], "want": [0]},
                                     {"id": "b", "tokens": b[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[67:68], "want": [0]},
                                     {"id": "b", "tokens": b[8:9], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[68:70], "want": [1]}], "end": ["a"]}]
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(dirs[name]), "--dtype", dtype,
                           "--out", str(out), "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [ln for ln in proc.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    V = nt.CONFIGS[name]["vocab"]
    pa, pb = plain_logits(name, a), plain_logits(name, b)
    want = {0: np.stack([pa[0], pa[65], pb[6]]), 1: pa[66:67], 2: np.stack([pa[67], pb[8]]), 3: pa[69:70]}
    for i, w in want.items():
        check(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V), w, dtype, f"trace replay, step {i}")


def test_run_command(dirs):
    """`python -m alpacca_b200 run` with a Nagavik folder: two prompts as one batch, greedy, in 32-bit."""
    name = "c"
    prompts = [some_tokens(name, 6, 70), some_tokens(name, 2, 71)]
    text = " / ".join(" ".join(map(str, p)) for p in prompts)
    proc = subprocess.run([sys.executable, "-m", "alpacca_b200", "run", str(dirs[name]), text, "--temp", "0",
                           "--repeat-penalty", "1.0", "--n-predict", "5", "--dtype", "float32", "--ctx", "64"],
                          capture_output=True, text=True, timeout=600, cwd=str(ROOT))
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [ln for ln in proc.stdout.splitlines() if ln.strip()]
    assert [[int(t) for t in ln.split()] for ln in lines] == [plain_greedy(name, p, 5) for p in prompts]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "c"])
def test_prompt_steps_replayed_from_their_graph(dirs, name, dtype):
    """Five prompt steps of one shape on empty slots: the second is captured, the later ones are replays with other tokens
    (hence other experts), slots and pages, and every one gives the plain logits."""
    from alpacca_b200.engine.step import StepEntry
    eng = engine_of(dirs, name, dtype)
    held = eng.alloc_slot()          # shifts the slots of the later rounds
    for k in range(5):
        a, b = some_tokens(name, 70, 300 + k), some_tokens(name, 9, 320 + k)
        if k == 3:
            eng.free_slot(held)
            held = None
        sa, sb = eng.alloc_slot(), eng.alloc_slot()
        out = eng.step([StepEntry(sa, a, list(range(70))), StepEntry(sb, b, list(range(9)))]).cpu().numpy()
        eng.wait()
        check(out[:70], plain_logits(name, a), dtype, f"{name} replayed prompt step {k}")
        check(out[70:], plain_logits(name, b), dtype, f"{name} replayed prompt step {k}, second prompt")
        eng.free_slot(sa)
        eng.free_slot(sb)
    assert len(eng._graphs) >= 1
