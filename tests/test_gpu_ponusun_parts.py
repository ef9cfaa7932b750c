"""Each mechanism of the Ponusun decoder alone, against its function in tests/plain_ponusun.py: the embedding with learned
positions, the input convolution with its kept rows, the kernel after a sub-layer (norm, addition, product per row,
average over depth, the next convolution), the attention with a norm over whole rows and a penalty on distance (also on
another layer's keys), the plain feed-forward, the experts chosen by token id beside a shared one, the bound on the
logits.  Sizes differ from test to test; inputs are made so that faults show."""
import math

import numpy as np
import pytest
import torch

import plain_ponusun as plain
from helpers import PartHarness, load_part

pytestmark = pytest.mark.gpu

TOL = {"float32": (2e-4, 2e-5), "bfloat16": (0.2, 0.02)}      # (largest, mean) |difference| as shares of the spread
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = ["float32", "bfloat16"]


def close(got, want, dtype, what, tol=None):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    spread = max(float(want.std()), 1e-30)
    d = np.abs(got - want) / spread
    big, mean = tol or TOL[dtype]
    assert d.max() <= big and d.mean() <= mean, f"{what}: max {d.max():.3e} mean {d.mean():.3e} of the spread"


def opts_of(dtype, max_positions=1024):
    from alpacca_b200.parts import BuildOptions
    return BuildOptions(dtype=DT[dtype], device="cuda", max_positions=max_positions)


def hidden(rng, n, width, dtype):
    """Activations [n, width] that both precisions hold exactly."""
    x = torch.from_numpy(rng.normal(0.0, 1.0, (n, width)).astype(np.float32)).to(torch.bfloat16)
    return x.to(DT[dtype]).cuda().contiguous(), x.double().numpy()


def dev(a):
    return torch.from_numpy(np.asarray(a, np.float32)).cuda().contiguous()


def f64(a):
    return dev(a).double().cpu().numpy()


def short(weights, prefix):
    return {k[len(prefix) + 1:]: v for k, v in weights.items() if k.startswith(prefix + ".")}


# ---------------------------------------------------------------------------------------------------------------
# embedding, convolution, the kernel after a sub-layer
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [24, 37, 1032])
def test_embedding_with_positions(dtype, width):
    from alpacca_b200.engine.step import StepEntry
    from alpacca_b200.parts import PositionTable, TokenEmbedding
    emb = TokenEmbedding(opts_of(dtype, 150), 90, width, "embed", weight_suffix="", positions=PositionTable(opts_of(dtype, 150), 200, width, "pos"))
    w = load_part(emb, seed=width, dtype=dtype, std=1.0)
    hs = PartHarness([], dtype, max_positions=150)
    rng = np.random.default_rng(width)
    toks = [rng.integers(0, 90, 100).tolist(), rng.integers(0, 90, 41).tolist()]
    got, at = [[], []], [0, 0]
    slots = [hs.cache.alloc_slot() for _ in toks]
    for cut in ((2, 40), (60, 1), (38, 0)):
        live = [i for i in range(2) if cut[i]]
        entries = [StepEntry(slots[i], toks[i][at[i]:at[i] + cut[i]], []) for i in live]
        ctx = hs.builder.build(entries, at if len(live) == 2 else [at[i] for i in live], hs.cache)
        out = emb.forward(ctx.tokens, ctx.n_tokens, ctx=ctx).double().cpu().numpy()
        r = 0
        for i in live:
            got[i].append(out[r:r + cut[i]])
            r += cut[i]
            at[i] += cut[i]
    for i in range(2):
        want = plain.embed(toks[i], w)
        assert np.abs(np.concatenate(got[i]) - want).max() <= 1e-6 * np.abs(want).max()      # one float32 addition
    with pytest.raises(ValueError, match="rows"):
        PositionTable(opts_of(dtype, 201), 200, width, "pos")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,taps", [(40, 3), (37, 2), (1032, 5), (64, 1), (24, 9)])
def test_input_convolution_in_portions(dtype, width, taps):
    """Two sequences side by side, one of them starting later, in portions down to one token (shorter than what the
    convolution keeps), and a slot that is used again: every token's taps reach over the portions' borders."""
    from alpacca_b200.parts import InputConv
    part = InputConv(opts_of(dtype), width, taps, "c")
    w = load_part(part, seed=taps, dtype=dtype, std=0.5)["c"]
    spec = part.cache_spec()
    assert (spec is None) == (taps == 1)
    hs = PartHarness([spec] if spec is not None else [], dtype)
    rng = np.random.default_rng(width)
    for again in range(2):
        x = [rng.normal(0, 1, (n, width)).astype(np.float32) for n in (41, 30)]
        slots = [hs.cache.alloc_slot() for _ in x]
        got, at = [[], []], [0, 0]
        for cut in ((1, 7), (1, 1), (2, 2), (3, 1), (12, 0), (1, 9), (4, 2), (17, 8)):
            live = [i for i in range(2) if cut[i]]
            ctx = hs.step([(slots[i], cut[i]) for i in live])
            rows = dev(np.concatenate([x[i][at[i]:at[i] + cut[i]] for i in live]))
            keep = rows.clone()
            out = part.forward(rows, ctx, hs.cache.entry_view(0, ctx.block_tables) if spec is not None else None)
            hs.done()
            assert torch.equal(rows, keep)
            out, r = out.float().cpu().numpy(), 0
            for i in live:
                got[i].append(out[r:r + cut[i]])
                r += cut[i]
                at[i] += cut[i]
        for i in range(2):
            close(np.concatenate(got[i]), plain.input_conv(x[i].astype(np.float64), w), dtype, f"convolution {i}",
                  tol=(5e-6, 5e-7) if dtype == "float32" else (0.03, 0.003))
        for s in slots:
            hs.cache.free_slot(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,taps", [(40, 2), (64, 3), (1032, 4), (37, 3), (24, 6)])
def test_input_convolution_of_many_tokens(dtype, width, taps):
    """Steps of hundreds of tokens, whose rows are walked in runs: sequences that start and end inside a run, some of one
    or two tokens, continued by a second such step."""
    from alpacca_b200.parts import InputConv
    part = InputConv(opts_of(dtype), width, taps, "c")
    w = load_part(part, seed=taps, dtype=dtype, std=0.5)["c"]
    hs = PartHarness([part.cache_spec()], dtype, max_slots=8)
    rng = np.random.default_rng(width)
    lens = [(131, 1), (1, 200), (2, 1), (1, 2), (90, 3), (3, 77), (40, 8), (8, 64)]
    x = [rng.normal(0, 1, (sum(n), width)).astype(np.float32) for n in lens]
    slots = [hs.cache.alloc_slot() for _ in x]
    got, at = [[] for _ in x], [0] * len(x)
    for step in range(2):
        ctx = hs.step([(s, n[step]) for s, n in zip(slots, lens)])
        out = part.forward(dev(np.concatenate([x[i][at[i]:at[i] + lens[i][step]] for i in range(len(x))])), ctx,
                           hs.cache.entry_view(0, ctx.block_tables)).float().cpu().numpy()
        hs.done()
        r = 0
        for i, n in enumerate(lens):
            got[i].append(out[r:r + n[step]])
            r += n[step]
            at[i] += n[step]
    for i in range(len(x)):
        close(np.concatenate(got[i]), plain.input_conv(x[i].astype(np.float64), w), dtype, f"convolution {i}",
              tol=(5e-6, 5e-7) if dtype == "float32" else (0.03, 0.003))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [37, 256, 1000, 2048, 4100, 9000])
def test_the_kernel_after_a_sublayer(dtype, width):
    """Every use of the kernel: the plain addition with the product per row and the cast; the average over 0 to 7 earlier
    results; and, for steps of one token per sequence, the next convolution with its kept rows, which then hold exactly
    what the convolution's own kernel would have left."""
    from alpacca_b200 import ops
    rng = np.random.default_rng(width)
    T, eps = 6, 1e-5
    hs = PartHarness([], dtype, max_slots=T)
    slots = [hs.cache.alloc_slot() for _ in range(T)]
    ctx = hs.step([(s, 1) for s in slots])
    x, w, g = rng.normal(0, 2, (T, width)), rng.uniform(0.5, 1.5, width), rng.normal(0, 1, width) / math.sqrt(width)
    for y_dtype in ("float32", "bfloat16"):
        y, y64 = hidden(rng, T, width, y_dtype)
        v64 = f64(x) + plain.rms_norm(y64, f64(w), eps)
        v, dots, out = torch.empty(T, width, device="cuda"), torch.empty(T, device="cuda"), torch.empty(T, width, device="cuda", dtype=DT[dtype])
        ops.post_norm_stream(dev(x), y, dev(w), eps, ctx, v_out=v, dot_weight=dev(g), dots=dots, out=out)
        close(v.cpu().numpy(), v64, "float32", "the stream", tol=(5e-6, 5e-7))
        close(out.float().cpu().numpy(), v64, dtype, "its cast", tol=(5e-6, 5e-7) if dtype == "float32" else (0.02, 0.003))
        assert np.abs(dots.double().cpu().numpy() - v64 @ f64(g)).max() <= 2e-5 * max(1.0, np.abs(v64 @ f64(g)).max())
    for n, taps in ((0, 1), (1, 2), (2, 3), (7, 4)):
        y, y64 = hidden(rng, T, width, "float32")
        coef, cw = rng.normal(0, 1, n + 1), rng.normal(0, 0.5, (width, taps))
        hist = rng.normal(0, 1, (n + 1, T, width))
        hist[n] = x
        h = dev(hist)
        state = dev(rng.normal(0, 1, (T + 2, max(taps - 1, 1), width)))
        state_b = state.clone()
        out = torch.empty(T, width, device="cuda", dtype=DT[dtype])
        avg = torch.empty(T, width, device="cuda")
        wt = dev(cw.T)
        # v in place of row n of the history, as the block does
        ops.post_norm_stream(h[n], y, dev(w), eps, ctx, v_out=h[n], history=h, n_history=n, coef=dev(coef), avg_out=avg,
                             out=out, conv=(wt, state[:, :taps - 1].contiguous() if taps == 1 else state))
        v64 = f64(x) + plain.rms_norm(y64, f64(w), eps)
        m64 = plain.depth_average([f64(r) for r in hist[:n]] + [v64], f64(coef))
        close(h[n].cpu().numpy(), v64, "float32", "the result", tol=(5e-6, 5e-7))
        close(avg.cpu().numpy(), m64, "float32", f"the average over {n} earlier results", tol=(1e-5, 1e-6))
        alone = torch.empty_like(out)
        ops.input_conv(avg, wt, state_b if taps > 1 else None, alone, ctx)
        assert torch.equal(alone, out) and torch.equal(state, state_b), "the convolution inside and by itself"
        kept = state_b[:T].double().cpu().numpy() if taps > 1 else None
        if taps > 1:
            assert np.array_equal(kept[:, -1], avg.double().cpu().numpy())


# ---------------------------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------------------------
SHAPES = [  # heads, kv heads, dim, vdim, window: which kernels they take in bfloat16
    (4, 2, 16, 24, None),        # tiles of rows; value size of its own
    (6, 3, 32, 32, 20),          # tiles of rows and the decode kernel
    (8, 2, 64, 64, 100),         # the tcgen05 kernel for long prompts
    (4, 2, 128, 128, None),      # tcgen05 and the streamed decode kernel
    (12, 3, 128, 128, 65),
    (16, 1, 64, 64, 130),        # 16 heads on one key/value head: the widest table of penalties
    (34, 2, 64, 64, 40),         # 17 heads per group: more than the tables hold
    (3, 3, 20, 12, 7),           # the 32-bit kernel
    (5, 1, 72, 40, 1),           # a token sees itself alone
    (2, 2, 256, 16, 50),
]


def attention_part(shape, dtype, width, seed, own_kv=True, prefix="m", keep=None):
    from alpacca_b200.parts import MapsAttention
    H, G, D, V, window = shape
    part = MapsAttention(opts_of(dtype), width, H, G, D, V, None, prefix, 1.3 / math.sqrt(D), 1e-5, window=window,
                         keep_window=keep, qk_norm=True, qk_norm_rows=True, distance=("r1", "r2"), own_kv=own_kv,
                         out_dtype=torch.float32)
    w = load_part(part, seed=seed, dtype=dtype, std=0.4)
    # penalties of some powers of e over the windows, one head with nearly none
    rng = np.random.default_rng(seed)
    r = np.stack([rng.uniform(0.5, 2.0, H), rng.uniform(0.05, 0.5, H)])
    r[0, H // 2] = 0.02
    part.penalty = dev(r)
    w = short(w, prefix)
    w["r1"], w["r2"] = f64(r)
    mx = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": 1.3 / math.sqrt(D)}
    if window:
        mx["mask"] = {"size": window}
    return part, w, mx


def feed(part, hs, slot, x, cuts, entry=0, write_cache=True):
    out, at = [], 0
    for n in cuts:
        ctx = hs.step([(slot, n)])
        out.append(part.forward(x[at:at + n].contiguous(), ctx, hs.cache.entry_view(entry, ctx.block_tables), write_cache).float().cpu().numpy())
        hs.done()
        at += n
    assert at == x.shape[0]
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("cuts", [(230,), (2, 61, 1, 2, 64, 100), (150,) + (1,) * 80])
def test_attention(dtype, shape, cuts):
    part, w, mx = attention_part(shape, dtype, 48, sum(shape[:4]))
    hs = PartHarness([part.cache_spec()], dtype)
    x, x64 = hidden(np.random.default_rng(3), 230, 48, dtype)
    s = hs.cache.alloc_slot()
    got = feed(part, hs, s, x, cuts)
    close(got, plain.attention(x64, w, mx, 1e-5, plain.keys_values(x64, w, mx, 1e-5)), dtype, f"attention {shape} {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(6, 3, 32, 32, 20), (8, 2, 64, 64, None), (4, 2, 128, 128, 150), (4, 2, 16, 48, 70)])
def test_attention_of_unequal_requests(dtype, shape):
    """Three requests in one step, then decoded together: each as if alone."""
    part, w, mx = attention_part(shape, dtype, 40, 5)
    hs = PartHarness([part.cache_spec()], dtype)
    rng = np.random.default_rng(4)
    xs = [hidden(rng, n, 40, dtype) for n in (1, 200, 66)]
    first = (1, 180, 40)
    xs[0] = hidden(rng, 27, 40, dtype)
    slots = [hs.cache.alloc_slot() for _ in xs]
    got = [[] for _ in xs]
    counts = [first] + [(1, 1, 1)] * 20 + [(1, 0, 1)] * 6
    at = [0, 0, 0]
    for cut in counts:
        live = [i for i in range(3) if cut[i]]
        ctx = hs.step([(slots[i], cut[i]) for i in live])
        rows = torch.cat([xs[i][0][at[i]:at[i] + cut[i]] for i in live]).contiguous()
        out = part.forward(rows, ctx, hs.cache.entry_view(0, ctx.block_tables), True).float().cpu().numpy()
        hs.done()
        r = 0
        for i in live:
            got[i].append(out[r:r + cut[i]])
            r += cut[i]
            at[i] += cut[i]
    for i in range(3):
        x64 = xs[i][1][:at[i]]
        close(np.concatenate(got[i]), plain.attention(x64, w, mx, 1e-5, plain.keys_values(x64, w, mx, 1e-5)), dtype, f"request {i}")


def planted(shape, dtype, places, asking, n, r1=0.0, r2=0.0):
    """An attention whose token at `asking` has a query that meets the keys at `places` far above all others (equal
    scores there): width = dim, W_q and W_k copy their input into every head, values carry the key's place."""
    H, G, D, V, window = shape
    part, w, mx = attention_part(shape, dtype, D + 1, 1)
    eye = np.concatenate([np.eye(D), np.zeros((D, 1))], axis=1)
    lift = np.zeros((V, D + 1))
    lift[:, D] = 1.0                                   # every value dim is the last input
    rng = np.random.default_rng(9)
    wq, wk, wv = np.tile(eye, (H, 1)), np.tile(eye, (G, 1)), np.tile(lift, (G, 1))
    part.qkv.weight.copy_(dev(np.concatenate([wq, wk, wv])).to(DT[dtype]))
    part.out.weight.copy_(dev(np.eye(D + 1, H * V)).to(DT[dtype]))
    part.q_weight.fill_(1.0)
    part.k_weight.fill_(1.0)
    part.penalty = dev(np.stack([np.full(H, r1), np.full(H, r2)]))
    x = rng.normal(0, 1, (n, D + 1))
    # the asking query and the planted keys point along one direction; all other keys have nothing of it
    d = np.zeros(D)
    d[0] = math.sqrt(D)
    x[:, 0] = 0.0
    x[asking, :D] = d
    for p in places:
        if p != asking:
            x[p, :D] = d
    x[:, D] = np.arange(n) % 61 / 8.0
    part.scale = mx["scale"] = 16.0 / D                # a planted key scores 16, others 0
    x = torch.from_numpy(x.astype(np.float32)).to(torch.bfloat16)
    w = {"q": wq, "k": wk, "v": wv, "q.norm": np.ones(H * D), "k.norm": np.ones(G * D), "o": np.eye(D + 1, H * V),
         "r1": np.full(H, r1), "r2": np.full(H, r2)}
    return part, w, mx, x.to(DT[dtype]).cuda().contiguous(), x.double().numpy()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("shape,window", [((4, 2, 64, 64), 5), ((4, 2, 64, 64), 64), ((4, 2, 64, 64), 65), ((4, 2, 128, 128), 130),
                                          ((2, 2, 32, 32), 63), ((2, 1, 16, 32), 66), ((3, 1, 24, 24), 9)])
def test_window_edges_with_a_planted_key(dtype, decode, shape, window):
    """The key at distance window - 1 takes all the weight; the key at distance window is not seen at all."""
    n, asking = 400, 331
    for inside in (True, False):
        place = asking - window + (1 if inside else 0)
        part, w, mx, x, x64 = planted(shape + (window,), dtype, [place], asking, n)
        hs = PartHarness([part.cache_spec()], dtype)
        s = hs.cache.alloc_slot()
        got = feed(part, hs, s, x, (300,) + (1,) * 100 if decode else (n,))
        want = plain.attention(x64, w, mx, 1e-5, plain.keys_values(x64, w, mx, 1e-5))
        close(got[asking - 3:asking + window + 3], want[asking - 3:asking + window + 3], dtype, f"window {window}, inside {inside}",
              tol=(2e-4, 2e-5) if dtype == "float32" else (0.05, 0.02))
        own, far = x64[asking, -1], x64[place, -1]
        seen = (own + far) / 2 if inside and place != asking else own
        if window > 1:
            assert abs(got[asking, 0] - seen) < 0.1, (window, inside, got[asking, 0], seen)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("shape", [(4, 2, 64, 64), (4, 2, 128, 128), (2, 2, 32, 32), (2, 1, 16, 32), (3, 1, 24, 24)])
def test_far_keys_and_the_penalty(dtype, decode, shape):
    """Keys far away, on the last place of a page and the first of the next, next to the asking token, on the sequence's
    first token: without a penalty each planted key shares the weight with the asking token's own; with one, the shares
    are (1 + r2 distance)^(-r1) to 1."""
    n, asking = 700, 668
    for place in (0, 1, 63, 64, 127, 128, 639, 640, 667):
        for r1, r2 in ((0.0, 0.0), (0.8, 0.05)):
            part, w, mx, x, x64 = planted(shape + (None,), dtype, [place], asking, n, r1, r2)
            hs = PartHarness([part.cache_spec()], dtype, max_tokens=64 * 20)
            s = hs.cache.alloc_slot()
            got = feed(part, hs, s, x, (660,) + (1,) * 40 if decode else (n,))
            share = (1.0 + r2 * (asking - place)) ** -r1
            own, far = x64[asking, -1], x64[place, -1]
            seen = (own + share * far) / (1.0 + share)
            assert abs(got[asking, 0] - seen) < (0.02 if dtype == "float32" else 0.08), (place, r1, got[asking, 0], seen)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(6, 2, 32, 32), (8, 2, 64, 64), (4, 2, 128, 128), (3, 1, 20, 12), (4, 2, 16, 48)])
@pytest.mark.parametrize("window,reading", [(70, 30), (30, 70), (None, 65), (64, None)])
def test_a_layer_that_reads_another_layers_keys(dtype, shape, window, reading):
    """The reader has other heads, its own window and penalty; it writes nothing; what the owner keeps covers both."""
    H, G, D, V = shape
    keep = "all" if window is None or reading is None else max(window, reading)
    owner, w1, mx1 = attention_part(shape + (window,), dtype, 40, 7, keep=keep)
    reader, w2, mx2 = attention_part((H + G, G, D, V, reading), dtype, 40, 8, own_kv=False, prefix="n", keep=keep)
    assert owner.cache_spec() == reader.cache_spec()
    assert [p.name for p in reader.param_specs()] == ["n.q.norm", "n.r1", "n.r2", "n.q", "n.o"]
    hs = PartHarness([owner.cache_spec()], dtype)
    rng = np.random.default_rng(11)
    a, a64 = hidden(rng, 200, 40, dtype)
    b, b64 = hidden(rng, 200, 40, dtype)
    s = hs.cache.alloc_slot()
    got1, got2, at = [], [], 0
    for n in (2, 90, 1, 1, 60) + (1,) * 46:
        ctx = hs.step([(s, n)])
        view = hs.cache.entry_view(0, ctx.block_tables)
        got1.append(owner.forward(a[at:at + n].contiguous(), ctx, view, True).float().cpu().numpy())
        before = (view.k.clone(), view.v.clone())
        got2.append(reader.forward(b[at:at + n].contiguous(), ctx, view, False).float().cpu().numpy())
        assert torch.equal(before[0], view.k) and torch.equal(before[1], view.v)
        hs.done()
        at += n
    kept = plain.keys_values(a64, w1, mx1, 1e-5)
    close(np.concatenate(got1), plain.attention(a64, w1, mx1, 1e-5, kept), dtype, "the owner")
    close(np.concatenate(got2), plain.attention(b64, w2, mx2, 1e-5, kept), dtype, "the reader")
    with pytest.raises(ValueError, match="writes no cache"):
        reader.forward(b[:1].contiguous(), hs.step([(s, 1)]), hs.cache.entry_view(0, ctx.block_tables), True)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pairing,n_rot", [("llama", 12), ("neox", 32), (None, 0)])
def test_norm_over_whole_rows_with_a_rotation(dtype, pairing, n_rot):
    """The prepared rows themselves: one root mean square over all heads, then the rotation of each head; sizes that
    take the kernel of 16-byte pieces and ones that do not."""
    from alpacca_b200 import ops
    from alpacca_b200.parts import KVSpec, RotaryEncoding
    for H, G, D, V in ((6, 3, 32, 16), (5, 1, 36, 20), (40, 8, 128, 128)):
        opts = opts_of(dtype)
        rot = RotaryEncoding(opts, D, min(n_rot, D), 100.0, pairing).rotation() if pairing else None
        hs = PartHarness([KVSpec(G, D, None, value_heads=G, value_dim=V)], dtype)
        rng = np.random.default_rng(H)
        N = H * D + G * D + G * V
        buf, b64 = hidden(rng, 70, N, dtype)
        qw, kw = rng.uniform(0.5, 1.5, H * D), rng.uniform(0.5, 1.5, G * D)
        s = hs.cache.alloc_slot()
        ctx = hs.step([(s, 70)])
        view = hs.cache.entry_view(0, ctx.block_tables)
        ops.attention_prepare(buf, (0, H * D, H * D + G * D), H, G, 1, D, V, view, ctx, q_weight=dev(qw), k_weight=dev(kw),
                              eps=1e-5, rot=rot, norm_rows=True)
        q = plain.rms_norm(b64[:, :H * D], f64(qw), 1e-5).reshape(70, H, D)
        k = plain.rms_norm(b64[:, H * D:H * D + G * D], f64(kw), 1e-5).reshape(70, G, D)
        if rot is not None:
            c, sn = rot[0][:70].double().cpu().numpy()[:, None], rot[1][:70].double().cpu().numpy()[:, None]
            n = rot[2]
            for z in (q, k):
                u, v = (z[..., 0:n:2].copy(), z[..., 1:n:2].copy()) if pairing == "llama" else (z[..., :n // 2].copy(), z[..., n // 2:n].copy())
                if pairing == "llama":
                    z[..., 0:n:2], z[..., 1:n:2] = u * c - v * sn, v * c + u * sn
                else:
                    z[..., :n // 2], z[..., n // 2:n] = u * c - v * sn, v * c + u * sn
        tol = (2e-5, 2e-6) if dtype == "float32" else (0.03, 0.004)
        close(buf[:, :H * D].float().cpu().numpy(), q.reshape(70, -1), dtype, "queries", tol=tol)
        pages = view.block_table[0].cpu().tolist()
        keys = np.stack([view.k[pages[p // 64], :, p % 64].float().cpu().numpy() for p in range(70)])
        vals = np.stack([view.v[pages[p // 64], :, p % 64].float().cpu().numpy() for p in range(70)])
        close(keys, k, dtype, "keys", tol=tol)
        assert np.array_equal(vals.reshape(70, -1).astype(np.float64), b64[:, -G * V:])


# ---------------------------------------------------------------------------------------------------------------
# feed-forwards, logits
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 8, 9, 40, 1100])
@pytest.mark.parametrize("width,ff", [(48, 100), (64, 88), (40, 33)])
def test_plain_feed_forward(dtype, rows, width, ff):
    from alpacca_b200.parts import PlainFeedForward
    part = PlainFeedForward(opts_of(dtype, 2048), width, ff, "m", out_dtype=torch.float32)
    w = short(load_part(part, seed=ff, dtype=dtype, std=0.25), "m")
    hs = PartHarness([], dtype, max_positions=2048)
    x, x64 = hidden(np.random.default_rng(rows), rows, width, dtype)
    got = part.forward(x, hs.step([(hs.cache.alloc_slot(), rows)]))
    assert got.dtype == torch.float32
    close(got.cpu().numpy(), plain.dense(x64, w), dtype, "feed-forward", tol=(2e-5, 2e-6) if dtype == "float32" else (0.05, 0.005))


MOES = [  # width, experts, ff, top, shared
    (40, 6, 20, 3, 28), (64, 5, 24, 5, None), (48, 3, 9, 2, 17), (128, 16, 64, 4, 96), (37, 1, 8, 1, 8), (256, 8, 40, 1, 200),
    (136, 70, 24, 6, 72),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 7, 9, 32, 33, 260, 1100])
@pytest.mark.parametrize("width,E,ff,top,shared", MOES)
def test_experts_by_token(dtype, rows, width, E, ff, top, shared):
    """Few rows (skinny products), many (grouped products, experts that nobody chose among them) and sizes that take the
    kernels per pair, with the gate's logit formed by the part itself and handed over."""
    from alpacca_b200 import ops
    from alpacca_b200.engine.step import StepEntry
    from alpacca_b200.parts import TableExperts
    vocab = 30
    part = TableExperts(opts_of(dtype, 2048), width, ff, E, top, vocab, "m", shared_inner=shared or 0)
    w = short(load_part(part, seed=E, dtype=dtype, std=0.3), "m")
    rng = np.random.default_rng(rows)
    hs = PartHarness([], dtype, max_positions=2048)
    toks = rng.integers(0, vocab if rows > 40 else 4, rows).tolist()
    ctx = hs.builder.build([StepEntry(hs.cache.alloc_slot(), toks, [])], [0], hs.cache)
    x, x64 = hidden(rng, rows, width, dtype)
    mlp = {"router": {"experts": E, "top": top}, "shared": {"ff": shared} if shared else None}
    want = plain.experts(x64, toks, w, mlp)
    tol = (2e-5, 2e-6) if dtype == "float32" else (0.06, 0.006)
    close(part.forward(x, ctx).cpu().numpy(), want, dtype, "experts", tol=tol)
    if shared:
        assert np.abs(plain.shared_expert(x64, w)).mean() > 0.05 * np.abs(want).mean()
        z = dev(x64 @ w["shared.sg"][0])
        close(part.forward(x, ctx, gate_logits=z).cpu().numpy(), want, dtype, "experts, gate handed over", tol=tol)
    # the same experts behind a choice that a router would hand over
    idx = part.table[torch.tensor(toks, device="cuda").long()].contiguous()
    out = torch.empty((rows, width), dtype=torch.float32, device="cuda")
    share = rng.uniform(0.2, 1.5, (rows, top))
    ops.moe_shared_experts(x, part.gate_up, part.down, E, top, out, ctx, choice=(idx, dev(share)), shared=part.shared_weights(),
                           gate_logits=dev(x64 @ w["shared.sg"][0]) if shared else None)
    want = plain.shared_expert(x64, w) if shared else np.zeros((rows, width))
    for t in range(rows):
        for k, e in enumerate(idx[t].tolist()):
            want[t] += f64(share)[t, k] * plain.gated(x64[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    close(out.cpu().numpy(), want, dtype, "experts behind a router's choice", tol=tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 8, 20])
def test_bounded_logits(dtype, rows):
    from alpacca_b200.parts import VocabHead
    cap = 3.0
    part = VocabHead(opts_of(dtype), 131, 48, "head", weight_suffix="", softcap=cap)
    w = load_part(part, seed=1, dtype=dtype, std=0.5)["head"]
    x, x64 = hidden(np.random.default_rng(rows), rows, 48, dtype)
    raw = x64 @ w.T
    assert np.abs(raw).max() > 2 * cap                      # far into the bend
    got = part.forward(x, n_rows=rows).cpu().numpy()
    assert np.abs(got - cap * np.tanh(raw / cap)).max() <= 2e-5 * cap
