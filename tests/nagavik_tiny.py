"""Small Nagavik configurations and weights for the tests.

The configurations differ from each other in every size and constant, and within one no two sizes that could be confused
are equal by accident.  State-space layers with 1 to 4 groups, convolutions over 1 to 6 tokens, norms in 1 to 7 parts, state
and value sizes that take the kernels in chunks, in steps and the walk, and ones that do not; attention with one key/value
head for all, one each, groups in between, key and value sizes apart and equal, with and without a bound on the scores; one
expert of several, several, all of them, with and without a shared one; layers without a feed-forward.

`make_weights` draws values that a bfloat16 holds exactly, so that the plain implementation, the 32-bit engine and the
bfloat16 engine read the same numbers.  Scales are chosen so that faults show: norm weights and layer scales away from 1,
convolution taps of the order of 1, decays from a few tokens to thousands, step sizes of 0.02 to 0.6.  Routers: a token's
embedding carries one of a few directions, which the router's rows meet with well separated weights, so that rounding of the
activations seldom turns a choice.
"""
from __future__ import annotations

import numpy as np

from ponusun_tiny import bf16_exact, write_model_dir  # noqa: F401


def _ssm(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": mlp}


def _att(heads, kv_heads, dim, vdim, scale, softcap=None, mlp=None):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        mx["softcap"] = softcap
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def _model(vocab, width, positions, eps, scale, cap, layers):
    return {"architecture": "Nagavik", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "logit_softcap": cap, "layers": layers}


TINY_A = _model(101, 40, 300, 1e-5, 2.5, 9.0, [
    _ssm(4, 12, 16, 2, 4, 2, _moe(20, 6, 2, 28)),
    _att(4, 2, 16, 24, 0.3, 3.0, None),
    _ssm(6, 8, 24, 3, 2, 1, _dense(52)),
    _att(6, 1, 20, 12, 0.22, 30.0, _moe(12, 5, 5)),
])

TINY_B = _model(67, 64, 260, 1e-6, 0.7, None, [
    _att(3, 3, 24, 40, 0.25, None, _dense(100)),
    _ssm(3, 20, 5, 1, 1, 3, _moe(9, 3, 1, 17)),
    _ssm(2, 7, 16, 2, 5, 7, None),
])

# sizes of the tensor-core kernels
TINY_C = _model(131, 48, 280, 1e-5, 1.5, 4.0, [
    _ssm(4, 32, 64, 1, 4, 4, _moe(16, 8, 1, 40)),
    _att(4, 2, 64, 64, 0.15, 6.0, _dense(24)),
    _ssm(2, 72, 128, 2, 3, 2, _moe(32, 7, 4, 8)),
    _att(8, 1, 128, 128, 0.12, 2.0, None),
    _ssm(4, 16, 144, 4, 6, 1, _dense(88)),
])

CONFIGS = {"a": TINY_A, "b": TINY_B, "c": TINY_C}


def tensor_shapes(config) -> dict:
    E, V = config["width"], config["vocab"]
    out = {"embed": (V, E), "pos": (config["max_positions"], E), "final.norm": (E,), "head": (V, E)}
    for i, layer in enumerate(config["layers"]):
        p, mx, mlp, m = f"l{i}", layer["mixer"], layer["mlp"], f"l{i}.mix"
        out.update({f"{p}.norm1": (E,), f"{p}.norm1b": (E,), f"{p}.ls1": (E,)})
        H, Vd = mx["heads"], mx["vdim"]
        if layer["type"] == "mamba2":
            inner, c = H * Vd, H * Vd + 2 * mx["groups"] * mx["state"]
            out.update({f"{m}.in": (inner + c + H, E), f"{m}.conv": (c, mx["conv"]), f"{m}.conv.b": (c,),
                        f"{m}.dt_bias": (H,), f"{m}.A_log": (H,), f"{m}.D": (H,), f"{m}.norm": (inner,), f"{m}.o": (E, inner)})
        else:
            G, D = mx["kv_heads"], mx["dim"]
            out.update({f"{m}.q": (H * D, E), f"{m}.k": (G * D, E), f"{m}.v": (G * Vd, E), f"{m}.q.norm": (H * D,),
                        f"{m}.k.norm": (G * D,), f"{m}.o": (E, H * Vd)})
        if mlp is None:
            continue
        out.update({f"{p}.norm2": (E,), f"{p}.norm2b": (E,), f"{p}.ls2": (E,)})
        f = f"{p}.mlp"
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            out.update({f"{f}.gate": (F, E), f"{f}.gate.b": (F,), f"{f}.up": (F, E), f"{f}.up.b": (F,), f"{f}.down": (E, F),
                        f"{f}.down.b": (E,)})
            continue
        n, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        out[f"{f}.router"] = (n, E)
        for e in range(n):
            out.update({f"{f}.e{e}.up": (F, E), f"{f}.e{e}.down": (E, F)})
        if mlp.get("shared"):
            S = mlp["shared"]["ff"]
            out.update({f"{f}.shared.up": (S, E), f"{f}.shared.down": (E, S)})
    return out


CLASSES = 4        # directions that a token's embedding may carry


def make_weights(config, seed: int, std: float = 0.1) -> dict:
    rng = np.random.default_rng(seed)
    E = config["width"]
    directions = rng.choice([-1.0, 1.0], (CLASSES, E))
    out = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            x = rng.normal(0.0, 0.6, shape) + 1.5 * directions[rng.integers(0, CLASSES, shape[0])]
        elif name == "pos":
            x = rng.normal(0.0, 0.7, shape)
        elif last == "router":
            levels = np.stack([rng.permutation(np.linspace(-2.0, 2.0, shape[0])) for _ in range(CLASSES)], axis=1)
            x = levels @ directions / E * 1.5
        elif last in ("norm", "norm1", "norm2", "norm1b", "norm2b"):
            x = rng.uniform(0.6, 1.6, shape)
        elif last in ("ls1", "ls2"):
            x = rng.uniform(0.3, 1.2, shape)
        elif last == "conv":
            x = rng.normal(0.0, 0.5, shape)
        elif last == "b":
            x = rng.normal(0.0, 0.3, shape)
        elif last == "A_log":
            x = rng.uniform(np.log(0.003), np.log(3.0), shape)
        elif last == "dt_bias":
            dt = np.exp(rng.uniform(np.log(0.02), np.log(0.6), shape))
            x = np.log(np.expm1(dt))
        elif name == "head":
            x = rng.normal(0.0, 0.5 * (48.0 / E) ** 0.5, shape)
        elif last == "D":
            x = rng.uniform(0.3, 1.5, shape)
        else:
            x = rng.normal(0.0, std * (48.0 / shape[-1]) ** 0.5 * 1.5, shape)
        out[name] = bf16_exact(np.asarray(x, np.float32))
    return out


def random_config(seed: int) -> dict:
    """A configuration drawn from a fixed seed: 1 to 6 layers in any order, sizes of every kind."""
    rng = np.random.default_rng(7000 + seed)

    def pick(*xs):
        return xs[int(rng.integers(0, len(xs)))]

    def mlp():
        kind = pick("none", "dense", "moe", "moe")
        if kind == "none":
            return None
        if kind == "dense":
            return _dense(pick(24, 33, 64, 130))
        n = pick(1, 2, 3, 5, 9)
        return _moe(pick(8, 12, 21, 36), n, int(rng.integers(1, n + 1)), pick(None, 8, 19, 44))

    layers = []
    for _ in range(int(rng.integers(1, 7))):
        if rng.random() < 0.55:
            groups = pick(1, 2, 3)
            heads, vdim = groups * pick(1, 2, 4), pick(4, 6, 8, 16, 24, 40, 64)
            parts = [p for p in (1, 2, 3, 4, 6, 8) if heads * vdim % p == 0]
            layers.append(_ssm(heads, vdim, pick(3, 8, 16, 32, 48, 80, 128), groups, pick(1, 2, 3, 4, 5, 7), pick(*parts), mlp()))
            continue
        kv, dim = pick(1, 2, 3), pick(8, 12, 16, 32, 48, 64, 72, 128)
        vdim = dim if rng.random() < 0.5 else pick(8, 16, 24, 80)
        layers.append(_att(kv * pick(1, 2, 3, 5), kv, dim, vdim, float(pick(0.1, 0.2, 0.35)), pick(None, 1.5, 5.0, 25.0), mlp()))
    return _model(pick(97, 150, 257), pick(24, 37, 56, 64, 100, 200), pick(160, 513), float(pick(1e-6, 1e-5, 1e-3)),
                  float(pick(0.5, 1.0, 3.0)), pick(None, 3.0, 15.0, 50.0), layers)
