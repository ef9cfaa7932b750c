"""Each mechanism of the Nagavik decoder alone, against its function in tests/plain_nagavik.py: the scaled embedding with
learned positions, the state-space mixer in its three forms (chunks, steps, walk) with its convolution and its gated norm, the
attention with bounded scores, slopes and a fixed sink, the gated feed-forward with biases, the experts whose weights multiply
their inputs, the layer scale.  Sizes differ from test to test; inputs are made so that faults show."""
import math

import numpy as np
import pytest
import torch

import plain_nagavik as plain
from helpers import PartHarness, load_part
from test_gpu_ponusun_parts import DT, DTYPES, close, dev, f64, feed, hidden, opts_of, short

pytestmark = pytest.mark.gpu


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [24, 37, 1032])
def test_scaled_embedding_with_positions(dtype, width):
    from alpacca_b200.engine.step import StepEntry
    from alpacca_b200.parts import PositionTable, TokenEmbedding
    emb = TokenEmbedding(opts_of(dtype, 150), 90, width, "embed", weight_suffix="", scale=2.5,
                         positions=PositionTable(opts_of(dtype, 150), 200, width, "pos"))
    w = load_part(emb, seed=width, dtype=dtype, std=1.0)
    hs = PartHarness([], dtype, max_positions=150)
    toks = np.random.default_rng(width).integers(0, 90, 143).tolist()
    slot, got, at = hs.cache.alloc_slot(), [], 0
    for n in (2, 1, 40, 100):
        ctx = hs.builder.build([StepEntry(slot, toks[at:at + n], [])], [at], hs.cache)
        got.append(emb.forward(ctx.tokens, ctx.n_tokens, ctx=ctx).double().cpu().numpy())
        at += n
    want = plain.embed(toks, w, 2.5)
    assert np.abs(np.concatenate(got) - want).max() <= 1e-6 * np.abs(want).max()


# ---------------------------------------------------------------------------------------------------------------
# the state-space mixer
# ---------------------------------------------------------------------------------------------------------------
SSM_SHAPES = [  # heads, vdim, state, groups, taps, norm parts
    (4, 32, 64, 2, 4, 2),          # chunks and steps
    (2, 64, 128, 1, 3, 1),
    (3, 40, 144, 3, 2, 5),         # more than eight row tiles of the state; a ragged tile of columns
    (6, 8, 16, 2, 5, 3),           # 16 columns per CTA; any number of taps
    (2, 128, 32, 2, 4, 4),
    (4, 20, 24, 4, 4, 2),          # no chunks (the state is no multiple of 16), steps
    (2, 7, 5, 1, 1, 7),            # the walk alone; one tap
    (3, 13, 33, 1, 9, 1),
    (2, 72, 256, 1, 17, 2),
]


def ssm_part(shape, dtype, width, seed):
    from alpacca_b200.parts import StateSpaceMixer
    H, V, N, G, taps, parts = shape
    part = StateSpaceMixer(opts_of(dtype), width, H, V, N, G, taps, parts, 1e-5, "m", out_dtype=torch.float32)
    w = short(load_part(part, seed=seed, dtype=dtype, std=0.3), "m")
    # decays over a few tokens to thousands, step sizes of 0.02 to 0.6
    rng = np.random.default_rng(seed)
    A, dt = rng.uniform(math.log(0.003), math.log(3.0), H), np.exp(rng.uniform(math.log(0.02), math.log(0.6), H))
    part.A_log, part.dt_bias = dev(A), dev(np.log(np.expm1(dt)))
    w["A_log"], w["dt_bias"] = f64(A), f64(np.log(np.expm1(dt)))
    return part, w, {"heads": H, "vdim": V, "state": N, "groups": G, "norm_groups": parts}


class SsmFeed:
    """Feeds a mixer that keeps one or two states."""

    def __init__(self, part, dtype, max_slots=4):
        self.part, self.hs = part, PartHarness(part.cache_specs(), dtype, max_slots=max_slots)

    def step(self, seqs, rows):
        ctx = self.hs.step(seqs)
        views = [self.hs.cache.entry_view(i, ctx.block_tables) for i in range(len(self.part.cache_specs()))]
        out = self.part.forward(rows.contiguous(), ctx, views if len(views) > 1 else views[0]).float().cpu().numpy()
        self.hs.done()
        return out

    def run(self, slot, x, cuts):
        out, at = [], 0
        for n in cuts:
            out.append(self.step([(slot, n)], x[at:at + n]))
            at += n
        assert at == x.shape[0]
        return np.concatenate(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SSM_SHAPES)
@pytest.mark.parametrize("cuts", [(230,), (2, 61, 1, 2, 64, 100), (150,) + (1,) * 80, (2,) * 30 + (65, 63, 1, 1, 40)])
def test_state_space_mixer(dtype, shape, cuts):
    """Whole, in portions across the chunks' borders, and decoded; the slot has been used by another sequence before."""
    part, w, mx = ssm_part(shape, dtype, 48, sum(shape))
    f = SsmFeed(part, dtype)
    rng = np.random.default_rng(3)
    x, x64 = hidden(rng, 230, 48, dtype)
    s = f.hs.cache.alloc_slot()
    f.run(s, hidden(rng, 70, 48, dtype)[0], (66, 1, 3))
    f.hs.cache.free_slot(s)
    assert f.hs.cache.alloc_slot() == s
    close(f.run(s, x, cuts), plain.mamba2(x64, w, mx, 1e-5), dtype, f"state-space {shape} {cuts[:3]}")


@pytest.mark.parametrize("shape", SSM_SHAPES[:6])
def test_the_forms_agree_closely(shape):
    """bfloat16, the recurrence alone: chunks against the exact sums over the same rounded rows.  Everything but those rows
    enters with 16 bits, so the difference is far below a bfloat16's rounding."""
    from alpacca_b200 import ops
    H, V, N, G, _, _ = shape
    if not ops.ssm_chunks_supports(N, V, H, G):
        pytest.skip("these sizes have no chunks")
    rng = np.random.default_rng(N)
    hs = PartHarness([], "bfloat16")
    lens = (197, 1, 64, 130)
    slots = [hs.cache.alloc_slot() for _ in lens]
    ctx = hs.step(list(zip(slots, lens)))
    T = sum(lens)
    xbc, xbc64 = hidden(rng, T, H * V + 2 * G * N, "bfloat16")
    dt = rng.uniform(0.01, 0.7, (T, H)).astype(np.float32)
    A, D = rng.uniform(math.log(0.003), math.log(8.0), H), rng.normal(0, 1, H)
    ld = -np.exp(f64(A)) * dt.astype(np.float64)
    start = rng.normal(0, 1, (len(slots), H, N, V)).astype(np.float32)
    state = dev(start)
    y = torch.empty(T, H * V, device="cuda")
    ops.ssm_chunks(xbc, dev(ld), dev(dt), dev(D), state, y, ctx, H, G, N, V)
    at = 0
    for i, n in enumerate(lens):
        x = xbc64[at:at + n, :H * V].reshape(n, H, V)
        B, C = (xbc64[at:at + n, H * V + k * G * N:H * V + (k + 1) * G * N].reshape(n, G, N) for k in (0, 1))
        S, want = start[slots[i]].astype(np.float64), np.zeros((n, H, V))
        for t in range(n):
            for a in range(H):
                S[a] = np.exp(f64(ld[at + t])[a]) * S[a] + float(dt[at + t, a]) * np.outer(B[t, a // (H // G)], x[t, a])
                want[t, a] = S[a].T @ C[t, a // (H // G)] + f64(D)[a] * x[t, a]
        got = y[at:at + n].double().cpu().numpy().reshape(n, H, V)
        close(got, want, "float32", f"read-outs of sequence {i}", tol=(4e-4, 4e-5))
        close(state[slots[i]].double().cpu().numpy(), S, "float32", f"state of sequence {i}", tol=(4e-4, 4e-5))
        at += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [SSM_SHAPES[0], SSM_SHAPES[3], SSM_SHAPES[5], SSM_SHAPES[7]])
def test_unequal_requests_together(dtype, shape):
    """Three requests in one step, then decoded together, one of them ending early: each as if alone."""
    part, w, mx = ssm_part(shape, dtype, 40, 5)
    f = SsmFeed(part, dtype)
    rng = np.random.default_rng(4)
    xs = [hidden(rng, n, 40, dtype) for n in (27, 206, 60)]
    slots = [f.hs.cache.alloc_slot() for _ in xs]
    got, at = [[] for _ in xs], [0, 0, 0]
    for cut in [(1, 180, 40)] + [(1, 1, 1)] * 20 + [(1, 1, 0)] * 6:
        live = [i for i in range(3) if cut[i]]
        out = f.step([(slots[i], cut[i]) for i in live], torch.cat([xs[i][0][at[i]:at[i] + cut[i]] for i in live]))
        r = 0
        for i in live:
            got[i].append(out[r:r + cut[i]])
            r += cut[i]
            at[i] += cut[i]
    assert at == [27, 206, 60]
    for i in range(3):
        close(np.concatenate(got[i]), plain.mamba2(xs[i][1], w, mx, 1e-5), dtype, f"request {i}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [(400,), (64, 64, 2, 126, 143, 1), (100,) + (1,) * 300])
@pytest.mark.parametrize("shape", [(2, 32, 64, 1, 2, 1), (2, 8, 20, 2, 1, 2)])
def test_a_token_far_back_is_still_in_the_state(dtype, cuts, shape):
    """No decay to speak of: what the fifth token wrote is all that the last one reads, 390 tokens later and over every
    border; with a decay of 1 % per token it has fallen to exp(-0.01 * 390)."""
    H, V, N, G, taps, parts = shape
    inner, gn = H * V, G * N
    for rate in (1e-6, 0.01):
        part, w, mx = ssm_part(shape, dtype, 8, 1)
        W = np.zeros((2 * inner + 2 * gn + H, 8))
        W[:inner, 4] = 1.0                       # the gate: the same everywhere
        W[inner:2 * inner, 0] = np.linspace(0.5, 2.0, inner)        # x, B, C: one input channel each
        W[2 * inner:2 * inner + gn, 1] = 1.0
        W[2 * inner + gn:2 * inner + 2 * gn, 2] = 1.0
        part.proj.weight.zero_()
        part.proj.weight[:W.shape[0]].copy_(dev(W).to(DT[dtype]))
        part.conv.zero_()
        part.conv[-1].fill_(1.0)
        part.conv_bias.zero_()
        part.skip.zero_()
        part.A_log, part.dt_bias = dev(np.full(H, math.log(rate))), dev(np.full(H, math.log(math.e - 1)))       # step size 1
        conv = np.zeros((inner + 2 * gn, taps))
        conv[:, -1] = 1.0
        w.update({"in": W, "conv": conv, "conv.b": np.zeros(inner + 2 * gn), "D": np.zeros(H), "A_log": np.full(H, math.log(rate)),
                  "dt_bias": np.full(H, math.log(math.e - 1))})
        x = np.zeros((400, 8))
        x[:, 4] = 1.0
        x[4, 0] = x[4, 1] = 4.0                  # writes
        x[395, 2] = 4.0                          # reads
        h = torch.from_numpy(x).to(DT[dtype]).cuda().contiguous()
        # without the norm the size of what is read shows: the kernel's eps is raised until it is all that counts
        part.eps = 1e12
        f = SsmFeed(part, dtype)
        got = f.run(f.hs.cache.alloc_slot(), h, cuts)
        want = plain.mamba2(x, w, mx, 1e12)
        spread = np.abs(want).max()
        assert np.abs(got - want).max() <= (1e-4 if dtype == "float32" else 0.02) * spread
        assert np.abs(want[395]).max() == spread and np.abs(np.delete(want, 395, 0)).max() == 0


@pytest.mark.parametrize("out_dtype", DTYPES)
@pytest.mark.parametrize("H,V,parts", [(4, 9, 6), (8, 64, 1), (5, 16, 5), (64, 64, 2), (16, 1024, 1), (3, 40, 2), (1, 7, 1)])
def test_gate_and_norm(out_dtype, H, V, parts):
    """Parts of every size, and the kept inputs moved on by one token."""
    from alpacca_b200 import ops
    rng = np.random.default_rng(H + V)
    T, G, N, taps, eps, inner = 5, 1, 3, 4, 1e-3, H * V
    hs = PartHarness([], max_slots=T + 2)
    held_slot = hs.cache.alloc_slot()
    slots = [hs.cache.alloc_slot() for _ in range(T)]
    ctx = hs.step([(s, 1) for s in slots])
    ld = 2 * inner + 2 * G * N + H
    proj, y, w = rng.normal(0, 1.5, (T, ld)), rng.normal(0, 2, (T, inner)), rng.uniform(0.5, 1.5, inner)
    y[1] *= 1e-3                                             # eps matters here
    kept = dev(rng.normal(0, 1, (T + 2, taps - 1, inner + 2 * G * N)))
    before = kept.clone()
    out = torch.empty(T, inner, dtype=DT[out_dtype], device="cuda")
    pr = dev(proj)
    ops.ssm_gate_norm(dev(y), pr, dev(w), parts, eps, out, ctx, H, G, N, V, taps, conv_state=kept)
    want = plain.gated_group_norm(f64(y), f64(proj)[:, :inner], f64(w), parts, eps)
    close(out.float().cpu().numpy(), want, out_dtype, "gate and norm", tol=(1e-5, 1e-6) if out_dtype == "float32" else (0.06, 0.003))
    for i, s in enumerate(slots):
        assert torch.equal(kept[s, :2], before[s, 1:]) and torch.equal(kept[s, 2], pr[i, inner:2 * inner + 2 * G * N])
    assert torch.equal(kept[held_slot], before[held_slot]) and torch.equal(kept[T + 1], before[T + 1])


# ---------------------------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------------------------
ATT_SHAPES = [  # heads, kv heads, dim, vdim, softcap
    (4, 2, 16, 24, 3.0),          # tiles of rows; value size of its own
    (6, 3, 32, 32, None),         # the decode kernel
    (8, 2, 64, 64, 2.0),          # the tcgen05 kernel for long prompts
    (4, 2, 128, 128, 5.0),        # tcgen05 and the streamed decode kernel
    (12, 1, 128, 128, None),
    (34, 2, 64, 64, 4.0),         # 17 heads per group
    (3, 3, 20, 12, 1.5),          # the 32-bit kernel
    (5, 1, 72, 40, 50.0),
    (2, 2, 256, 16, 2.0),
]


def attention_part(shape, dtype, width, seed):
    from alpacca_b200.parts import MapsAttention, alibi_slopes
    H, G, D, V, cap = shape
    scale = 1.7 / math.sqrt(D)
    part = MapsAttention(opts_of(dtype), width, H, G, D, V, None, "m", scale, 1e-5, qk_norm=True, qk_norm_rows=True,
                         softcap=cap, slopes=alibi_slopes(H), fixed_sink=0.0, out_dtype=torch.float32)
    w = short(load_part(part, seed=seed, dtype=dtype, std=0.4), "m")
    return part, w, {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale, "softcap": cap}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", ATT_SHAPES)
@pytest.mark.parametrize("cuts", [(230,), (2, 61, 1, 2, 64, 100), (150,) + (1,) * 80])
def test_attention(dtype, shape, cuts):
    part, w, mx = attention_part(shape, dtype, 48, sum(shape[:4]))
    hs = PartHarness([part.cache_spec()], dtype)
    x, x64 = hidden(np.random.default_rng(3), 230, 48, dtype)
    got = feed(part, hs, hs.cache.alloc_slot(), x, cuts)
    close(got, plain.attention(x64, w, mx, 1e-5), dtype, f"attention {shape} {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(6, 3, 32, 32, 2.0), (8, 2, 64, 64, None), (4, 2, 128, 128, 3.0), (4, 2, 16, 48, 6.0)])
def test_attention_of_unequal_requests(dtype, shape):
    """Three requests in one step, then decoded together; pages of an earlier sequence are used again."""
    part, w, mx = attention_part(shape, dtype, 40, 5)
    hs = PartHarness([part.cache_spec()], dtype, max_tokens=64 * 8)
    rng = np.random.default_rng(4)
    s = hs.cache.alloc_slot()
    feed(part, hs, s, hidden(rng, 300, 40, dtype)[0], (300,))
    hs.cache.free_slot(s)
    xs = [hidden(rng, n, 40, dtype) for n in (27, 200, 66)]
    slots = [hs.cache.alloc_slot() for _ in xs]
    got, at = [[] for _ in xs], [0, 0, 0]
    for cut in [(1, 180, 40)] + [(1, 1, 1)] * 20 + [(1, 0, 1)] * 6:
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
        close(np.concatenate(got[i]), plain.attention(xs[i][1][:at[i]], w, mx, 1e-5), dtype, f"request {i}")


def planted(shape, dtype, places, asking, n, slopes, score):
    """An attention whose token at `asking` meets the keys at `places` with `score` and all others with 0; the values of the
    planted tokens are 1, all others 0.  width = dim + 1, W_q and W_k copy their input into every head."""
    H, G, D, V, cap = shape
    part, w, mx = attention_part(shape, dtype, D + 1, 1)
    eye = np.concatenate([np.eye(D), np.zeros((D, 1))], axis=1)
    lift = np.zeros((V, D + 1))
    lift[:, D] = 1.0
    part.qkv.weight.copy_(dev(np.concatenate([np.tile(eye, (H, 1)), np.tile(eye, (G, 1)), np.tile(lift, (G, 1))])).to(DT[dtype]))
    part.out.weight.copy_(dev(np.eye(D + 1, H * V)).to(DT[dtype]))
    part.q_weight.fill_(1.0)
    part.k_weight.fill_(1.0)
    part.bound = (dev(slopes), part.bound[1])
    x = np.random.default_rng(9).normal(0, 1, (n, D + 1))
    d = np.zeros(D)
    d[0] = math.sqrt(D)
    x[:, 0] = 0.0
    x[:, D] = 0.0
    x[asking, :D] = d
    for p in places:
        x[p, :D] = d
        x[p, D] = 1.0
    part.scale = score / D
    x = torch.from_numpy(x.astype(np.float32)).to(torch.bfloat16)
    return part, x.to(DT[dtype]).cuda().contiguous()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("shape", [(4, 2, 64, 64), (4, 2, 128, 128), (2, 2, 32, 32), (2, 1, 16, 32), (3, 1, 24, 24), (10, 2, 48, 112)])
def test_planted_keys_fall_with_their_distance(dtype, decode, shape):
    """Keys on the first token, at page borders, next to the asking one and 668 tokens back, each alone: its weight is
    e^s / (1 + sum), s the bounded score less slope times distance, beside the other keys (score 0 less the same penalty) and
    the sink.  The bound is taken before the penalty."""
    n, asking, cap, score = 700, 668, 6.0, 11.0
    H = shape[0]
    slopes = f64(np.array([0.02 / (h + 1) for h in range(H)]))
    top = cap * math.tanh(score / cap)
    dist = np.arange(asking + 1)
    for place in (0, 63, 64, 127, 320, 639, 640, 667):
        part, x = planted(shape + (cap,), dtype, [place], asking, n, slopes, score)
        hs = PartHarness([part.cache_spec()], dtype)
        cuts = (asking,) + (1,) + (n - asking - 1,) if decode else (n,)
        got = feed(part, hs, hs.cache.alloc_slot(), x, cuts)[asking]
        V = shape[3]
        for h in range(H):
            if h * V >= got.shape[0]:
                break                                        # the output shows the first heads' values alone
            e = np.exp(-slopes[h] * dist)
            e[0] = math.exp(top)                             # the asking token meets its own key
            e[asking - place] = math.exp(top - slopes[h] * (asking - place))
            want = e[asking - place] / (1.0 + e.sum())
            assert abs(got[h * V] - want) <= (2e-5 if dtype == "float32" else 0.012) * max(want, 0.05), (place, h)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("shape", [(4, 2, 64, 64), (4, 2, 128, 128), (2, 2, 32, 32), (2, 1, 16, 32), (3, 1, 24, 24)])
def test_the_sink_takes_its_share(dtype, decode, shape):
    """Scores far below 0 (steep slopes): the token's own key and the sink are all that is left; own scores of 0 and of the
    bound leave 1/2 and e^c / (1 + e^c)."""
    n = 150
    for cap, score in ((3.0, 0.0), (1.0, 40.0), (2.0, -40.0)):
        asking = 140
        part, x = planted(shape + (cap,), dtype, [asking], asking, n, np.full(shape[0], 30.0), score)
        hs = PartHarness([part.cache_spec()], dtype)
        got = feed(part, hs, hs.cache.alloc_slot(), x, (asking, 1, n - asking - 1) if decode else (n,))[asking, 0]
        s = math.exp(cap * math.tanh(score / cap))
        assert abs(got - s / (1 + s)) <= (1e-5 if dtype == "float32" else 0.005), (cap, score)


def test_long_streamed_decoding():
    """2,000 tokens of context, chunks merged in a cluster and through memory: bounded scores, slopes and the sink."""
    from alpacca_b200 import ops
    shape = (8, 2, 128, 128, 4.0)
    part, w, mx = attention_part(shape, "bfloat16", 40, 8)
    hs = PartHarness([part.cache_spec()], "bfloat16", max_tokens=64 * 40, max_positions=2100)
    x, x64 = hidden(np.random.default_rng(6), 2003, 40, "bfloat16")
    part.bound = (dev(np.linspace(0.0005, 0.01, 8)), 4.0)
    got = feed(part, hs, hs.cache.alloc_slot(), x, (2000, 1, 1, 1))[2000:]
    old, plain.slopes = plain.slopes, lambda H: f64(np.linspace(0.0005, 0.01, 8))
    try:
        want = plain.attention(x64, w, mx, 1e-5)[2000:]
    finally:
        plain.slopes = old
    close(got, want, "bfloat16", "2,000 tokens back")
    assert ops._stream_plan(1, 8, 2, 128, 32, 148) is not None


# ---------------------------------------------------------------------------------------------------------------
# feed-forwards, layer scale
# ---------------------------------------------------------------------------------------------------------------
class Ctx:
    def __init__(self, n):
        self.n_tokens = n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 7, 8, 13, 40, 300, 1100])
def test_gated_feed_forward_with_biases(dtype, n):
    from alpacca_b200.parts import SwiGLU
    for width, ff in ((48, 88), (64, 53)):
        part = SwiGLU(opts_of(dtype), width, ff, "m", bias=True, names=("gate", "up", "down"), weight_suffix="",
                      bias_suffix=".b", activation="gelu_tanh", out_dtype=torch.float32)
        w = short(load_part(part, seed=n, dtype=dtype, std=0.3), "m")
        x, x64 = hidden(np.random.default_rng(n), n, width, dtype)
        close(part.forward(x, Ctx(n)).float().cpu().numpy()[:n], plain.dense(x64, w), dtype, f"dense {n} {ff}",
              tol=None if dtype == "float32" else (0.1, 0.01))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 5, 8, 16, 31, 33, 200, 1100])
def test_experts_with_weights_on_their_inputs(dtype, n):
    from alpacca_b200.parts import ScoredExperts
    for width, ff, E, top, shared in ((48, 40, 6, 2, 72), (64, 32, 5, 5, 0), (40, 21, 9, 1, 19), (36, 16, 3, 2, 8), (128, 64, 150, 3, 16)):
        part = ScoredExperts(opts_of(dtype), width, ff, E, top, "m", weight_in=True, shared_inner=shared)
        w = short(load_part(part, seed=E, dtype=dtype, std=0.3), "m")
        x, x64 = hidden(np.random.default_rng(n), n, width, dtype)
        mlp = {"router": {"experts": E, "top": top}, "shared": {"ff": shared} if shared else None}
        close(part.forward(x, Ctx(n)).float().cpu().numpy()[:n], plain.experts(x64, w, mlp), dtype, f"experts {n} of {E}",
              tol=None if dtype == "float32" else (0.15, 0.01))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [3, 20, 150])
@pytest.mark.parametrize("gated,weight_in,renorm,act", [(False, False, True, "relu2"), (True, False, False, "silu"), (True, True, False, "gelu"),
                                                        (False, True, True, "gelu")])
def test_other_experts_of_the_same_part(dtype, n, gated, weight_in, renorm, act):
    """Gates, weights on the output, renormalised weights and other activations: options that another design may take."""
    from alpacca_b200.parts import ScoredExperts
    names = dict(expert_names=("e{}.gate", "e{}.up", "e{}.down"), shared_names=("shared.gate", "shared.up", "shared.down")) if gated else {}
    part = ScoredExperts(opts_of(dtype), 48, 24, 5, 2, "m", activation=act, renorm=renorm, weight_in=weight_in, shared_inner=40, **names)
    w = short(load_part(part, seed=7, dtype=dtype, std=0.3), "m")
    x, h = hidden(np.random.default_rng(n), n, 48, dtype)
    f = {"relu2": plain.relu_squared, "silu": plain.silu,
         "gelu": lambda z: 0.5 * z * (1 + np.vectorize(math.erf)(z / math.sqrt(2)))}[act]

    def one(v, p):
        inner = f(v @ w[p + "gate"].T) * (v @ w[p + "up"].T) if gated else f(v @ w[p + "up"].T)
        return inner @ w[p + "down"].T
    chosen, weight = plain.route(h, w["router"], 2)
    if renorm:
        weight = weight / weight.sum(axis=1, keepdims=True)
    want = one(h, "shared.")
    for t in range(n):
        for e, s in zip(chosen[t], weight[t]):
            want[t] += one(s * h[t], f"e{e}.") if weight_in else s * one(h[t], f"e{e}.")
    close(part.forward(x, Ctx(n)).float().cpu().numpy()[:n], want, dtype, "experts", tol=None if dtype == "float32" else (0.15, 0.01))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [37, 64, 2056])
def test_layer_scale_after_the_norm(dtype, width):
    """A block whose sub-layer is the identity: x + scale * norm(norm(x)), between rows whose size differs."""
    from alpacca_b200.parts import HiddenStream, Mixer, RMSNorm, SandwichBlock

    class Same(Mixer):
        def forward(self, h, ctx, cache, write_cache=True):
            return h.float()
    o = opts_of(dtype)
    blk = SandwichBlock(RMSNorm(o, width, 1e-4, "n1", weight_suffix=""), Same(),
                        RMSNorm(o, width, 1e-4, "n1b", weight_suffix="", columns="ls"))
    w = load_part(blk, seed=2, dtype=dtype, std=0.5)
    x = np.random.default_rng(0).normal(0, 1, (5, width)) * np.array([[1.0], [10.0], [0.01], [3.0], [100.0]])
    hs = PartHarness([], dtype, max_slots=5)
    ctx = hs.step([(hs.cache.alloc_slot(), 1) for _ in range(5)])
    stream = HiddenStream(dev(x))
    blk.forward(stream, ctx, None)
    h = plain.rms_norm(f64(x), w["n1"], 1e-4)
    want = plain.rms_norm(h, w["n1b"], 1e-4) * w["ls"]
    close(stream.residual.double().cpu().numpy() - f64(x), want, dtype, "layer scale", tol=(3e-5, 3e-6) if dtype == "float32" else (0.03, 0.004))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 8, 14, 60])
def test_plain_feed_forward_with_the_square_of_relu(dtype, n):
    from alpacca_b200.parts import PlainFeedForward
    part = PlainFeedForward(opts_of(dtype), 48, 37, "m", activation="relu2", out_dtype=torch.float32)
    w = short(load_part(part, seed=n, dtype=dtype, std=0.3), "m")
    x, x64 = hidden(np.random.default_rng(n), n, 48, dtype)
    close(part.forward(x, Ctx(n)).float().cpu().numpy()[:n], plain.expert(x64, w["up"], w["down"]), dtype, "squared ReLU",
          tol=None if dtype == "float32" else (0.1, 0.01))
