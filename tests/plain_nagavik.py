"""A plain, slow implementation of the Nagavik decoder in NumPy float64: whole sequences, no cache, no batches, one
function per mechanism.  It shares no code with the package; the tests hold the package to it.

A model is (config dict, {tensor name: array}).  Layer i's tensors are `l<i>.norm1`, `l<i>.norm1b`, `l<i>.norm2`,
`l<i>.norm2b`, `l<i>.ls1`, `l<i>.ls2`, `l<i>.mix.*`, `l<i>.mlp.*`; linear weights are [out, in].

    start:   x = embed[token] * scale + pos[place]
    layer i: x <- x + ls1 * N1b(mixer(N1(x)));   x <- x + ls2 * N2b(ff(N2(x)))     (no second half without a ff)
    N(v):    v / sqrt(mean(v^2) + eps) * w
    end:     logits = cap * tanh(head N_final(x) / cap)
"""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def bounded(x, cap):
    return cap * np.tanh(x / cap)


def embed(tokens, W, scale):
    tokens = np.asarray(tokens, np.int64)
    return W["embed"][tokens] * scale + W["pos"][:len(tokens)]


# -- attention ----------------------------------------------------------------------------------------------------
def slopes(n_heads):
    return np.array([2.0 ** (-8.0 * (a + 1) / n_heads) for a in range(n_heads)])


def attention_weights(q, k, scale, cap, slope):
    """[T, T] of one head: q, k [T, D].  One more term, exp(0), stands in every row's sum."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    if cap is not None:
        s = bounded(s, cap)
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    s = np.where(dist >= 0, s - slope * dist, -np.inf)
    m = np.maximum(s.max(axis=1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=1, keepdims=True))


def attention(h, w, mx, eps):
    T = h.shape[0]
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, H, D)
    k = rms_norm(h @ w["k"].T, w["k.norm"], eps).reshape(T, G, D)
    v = (h @ w["v"].T).reshape(T, G, V)
    slope, cap = slopes(H), mx.get("softcap")
    out = np.zeros((T, H, V))
    for a in range(H):
        g = a // (H // G)
        out[:, a] = attention_weights(q[:, a], k[:, g], float(mx["scale"]), cap, slope[a]) @ v[:, g]
    return out.reshape(T, H * V) @ w["o"].T


# -- the state-space mixer ----------------------------------------------------------------------------------------
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K] (the last one meets the token itself), zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = np.tile(bias, (T, 1)).astype(np.float64)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def ssm_walk(x, B, C, dt, A_log, D, groups):
    """x [T, H, V], B and C [T, G, N], dt [T, H] (after softplus); token by token.  y [T, H, V] and the last state."""
    T, H, V = x.shape
    N = B.shape[2]
    S = np.zeros((H, N, V))
    y = np.zeros((T, H, V))
    for t in range(T):
        for a in range(H):
            g = a // (H // groups)
            S[a] = math.exp(-math.exp(A_log[a]) * dt[t, a]) * S[a] + dt[t, a] * np.outer(B[t, g], x[t, a])
            y[t, a] = S[a].T @ C[t, g] + D[a] * x[t, a]
    return y, S


def gated_group_norm(y, z, w, parts, eps):
    """(y silu(z)) in equal parts, each by its own root mean square, times w."""
    T, n = y.shape
    u = (y * silu(z)).reshape(T, parts, n // parts)
    u = u / np.sqrt(np.mean(u * u, axis=-1, keepdims=True) + eps)
    return u.reshape(T, n) * w


def mamba2(h, w, mx, eps):
    T = h.shape[0]
    H, V, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * V
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].reshape(T, H, V)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    y, _ = ssm_walk(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"], G)
    return gated_group_norm(y.reshape(T, inner), z, w["norm"], mx["norm_groups"], eps) @ w["o"].T


# -- feed-forwards ------------------------------------------------------------------------------------------------
def dense(h, w):
    return (gelu_tanh(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def expert(h, up, down):
    return relu_squared(h @ up.T) @ down.T


def route(h, router, top):
    """(chosen experts [T, top], their weights [T, top]): the largest sigmoids, as they are."""
    s = sigmoid(h @ router.T)
    order = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return order, np.take_along_axis(s, order, axis=1)


def experts(h, w, mlp):
    """A chosen expert reads its weight times h."""
    chosen, weight = route(h, w["router"], mlp["router"]["top"])
    out = np.zeros((h.shape[0], w["e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], weight[t]):
            out[t] += expert(s * h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    if mlp.get("shared"):
        out += expert(h, w["shared.up"], w["shared.down"])
    return out


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


MIXERS = {"attention": attention, "mamba2": mamba2}


def forward(config, weights, tokens, trace=None):
    """Logits [T, vocab] of the whole sequence `tokens`.  `trace`: a list that gets the stream after every layer."""
    W = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = embed(tokens, W, float(config["embedding"]["scale"]))
    for i, layer in enumerate(config["layers"]):
        p, mlp = f"l{i}.", layer.get("mlp")
        y = MIXERS[layer["type"]](rms_norm(x, W[p + "norm1"], eps), _sub(W, p + "mix."), layer["mixer"], eps)
        x = x + W[p + "ls1"] * rms_norm(y, W[p + "norm1b"], eps)
        if mlp is not None:
            h, ff = rms_norm(x, W[p + "norm2"], eps), _sub(W, p + "mlp.")
            y = dense(h, ff) if mlp["kind"] == "dense" else experts(h, ff, mlp)
            x = x + W[p + "ls2"] * rms_norm(y, W[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x.copy())
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    cap = config.get("logit_softcap")
    return logits if cap is None else bounded(logits, float(cap))
