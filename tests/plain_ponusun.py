"""A plain, slow implementation of the Ponusun decoder in NumPy float64: whole sequences, no cache, no batches, one
function per mechanism.  It shares no code with the package; the tests hold the package to it.

A model is (config dict, {tensor name: array}).  Layer i's tensors are `l<i>.norm1`, `l<i>.norm2`, `l<i>.canon1`,
`l<i>.dwa`, `l<i>.mix.*`, `l<i>.mlp.*`; linear weights are [out, in].

    start:   X_0 = embed[token] + pos[place]
    layer i: h = x + conv(x);  y = x + N1(mixer(h));  X_(i+1) = y + N2(ff(y))  (without a ff: y)
             x <- sum_(j <= i+1) dwa[j] X_j
    N(v):    v / sqrt(mean(v^2) + eps) * w
    end:     logits = cap * tanh(head N_final(x) / cap)
"""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def embed(tokens, W):
    tokens = np.asarray(tokens, np.int64)
    return W["embed"][tokens] + W["pos"][:len(tokens)]


def input_conv(x, taps):
    """x + conv(x): x [T, E], taps [E, K]; the last tap meets the token itself, zeros stand before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = np.array(x, dtype=np.float64, copy=True)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def depth_average(history, coef):
    return sum(float(c) * x for c, x in zip(coef, history, strict=True))


def distance_penalty(r1, r2, T):
    """[H, T, T]: r1_h ln(1 + r2_h (i - j)) where j <= i."""
    d = np.maximum(np.arange(T)[:, None] - np.arange(T)[None, :], 0).astype(np.float64)
    return r1[:, None, None] * np.log1p(r2[:, None, None] * d[None])


def keys_values(h, w, mx, eps):
    T, G = h.shape[0], mx["kv_heads"]
    k = rms_norm(h @ w["k"].T, w["k.norm"], eps).reshape(T, G, mx["dim"])
    return k, (h @ w["v"].T).reshape(T, G, mx["vdim"])


def attention(h, w, mx, eps, kept):
    """`kept`: (keys, values) of this layer or of the layer it reads."""
    T = h.shape[0]
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    k, v = kept
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, H, D)
    bias = distance_penalty(w["r1"], w["r2"], T)
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = j <= i
    if mx.get("mask"):
        seen &= (i - j) < mx["mask"]["size"]
    out = np.zeros((T, H, V))
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * float(mx["scale"]) - bias[a]
        s = np.where(seen, s, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, a] = (e / e.sum(axis=1, keepdims=True)) @ v[:, g]
    return out.reshape(T, H * V) @ w["o"].T


def dense(h, w):
    return gelu(h @ w["up"].T) @ w["down"].T


def gated(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def experts(h, tokens, w, mlp):
    """The experts of a token stand in a table; all of a token's experts weigh the same."""
    table = np.asarray(w["table"], np.int64)
    top = mlp["router"]["top"]
    out = np.zeros((h.shape[0], w["e0.down"].shape[0]))
    for t, tok in enumerate(tokens):
        for e in table[tok]:
            out[t] += gated(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]) / top
    if mlp.get("shared"):
        out += shared_expert(h, w)
    return out


def shared_expert(h, w):
    return sigmoid(h @ w["shared.sg"].T) * gated(h, w["shared.gate"], w["shared.up"], w["shared.down"])


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, trace=None):
    """Logits [T, vocab] of the whole sequence `tokens`.  `trace`: a list that gets the stream after every layer."""
    W = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, cap = float(config["norm"]["eps"]), float(config["logit_softcap"])
    x = embed(tokens, W)
    history, kept = [x], {}
    for i, layer in enumerate(config["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        mix = _sub(W, p + "mix.")
        h = input_conv(x, W[p + "canon1"])
        if mx.get("kv_from") is None:
            kept[i] = keys_values(h, mix, mx, eps)
        y = attention(h, mix, mx, eps, kept[i if mx.get("kv_from") is None else mx["kv_from"]])
        x = x + rms_norm(y, W[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            ff = _sub(W, p + "mlp.")
            y = dense(x, ff) if mlp["kind"] == "dense" else experts(x, tokens, ff, mlp)
            x = x + rms_norm(y, W[p + "norm2"], eps)
        history.append(x)
        x = depth_average(history, W[p + "dwa"])
        if trace is not None:
            trace.append(x.copy())
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    return cap * np.tanh(logits / cap)
