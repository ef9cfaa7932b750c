"""Small Ponusun configurations and weights for the tests.

The configurations differ from each other in every size and constant, and within one no two sizes that could be confused
are equal by accident (key and value sizes, expert and shared-expert sizes, head counts).  Windows of 1 to 130 tokens,
shorter than a page, longer than a page, none; layers that read an earlier layer's keys with a window smaller AND larger
than the owner's, two layers that read one owner, an owner that is not the layer right before; convolutions over 1 to 5
tokens; as many key/value heads as heads, one for all, groups in between; one expert of several, all experts chosen, a
layer of experts without a shared one, layers without a feed-forward, inner sizes that are no multiples of 8; head sizes
that take the tensor-core kernels in bfloat16 and ones that do not.

`make_weights` draws values that a bfloat16 holds exactly, so that the plain implementation, the 32-bit engine and the
bfloat16 engine read the same numbers.  Scales are chosen so that faults show: norm weights away from 1, convolution taps
of the order of 1, averages with weights of both signs on every earlier result, penalties that make a key's weight fall by
some powers of e over a window (and nearly none in one head of each layer).
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np


def _layer(heads, kv_heads, dim, vdim, scale, window=None, kv_from=None, mlp=None):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        mx["mask"] = {"size": window}
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def _model(vocab, width, positions, eps, taps, cap, layers):
    return {"architecture": "Ponusun", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
            "canon": {"taps": taps}, "logit_softcap": cap, "layers": layers}


TINY_A = _model(101, 40, 300, 1e-5, 4, 9.0, [
    _layer(4, 2, 16, 24, 0.3, window=70, mlp=_moe(20, 6, 3, 28)),
    _layer(6, 2, 16, 24, 0.22, window=33, kv_from=0, mlp=None),
    _layer(2, 1, 32, 16, 0.4, window=5, mlp=_dense(52)),
    _layer(2, 2, 16, 24, 0.35, window=130, kv_from=0, mlp=_moe(12, 4, 1, 36)),
])

TINY_B = _model(67, 64, 260, 1e-6, 1, 25.0, [
    _layer(3, 3, 20, 12, 0.25, mlp=_dense(100)),
    _layer(5, 1, 24, 40, 0.5, window=64, mlp=_moe(24, 5, 5)),
    _layer(6, 3, 20, 12, 0.3, window=65, kv_from=0, mlp=_moe(9, 3, 2, 17)),
    _layer(1, 1, 8, 8, 0.6, window=1, mlp=None),
])

# sizes of the tensor-core kernels: equal key and value sizes (the decode kernels), a head size of 64
TINY_C = _model(131, 48, 280, 1e-5, 5, 4.0, [
    _layer(6, 3, 32, 32, 0.2, window=20, mlp=_dense(88)),
    _layer(4, 2, 64, 64, 0.15, mlp=_moe(16, 8, 2, 40)),
    _layer(9, 3, 32, 32, 0.24, window=100, kv_from=0, mlp=_moe(32, 7, 4, 8)),
    _layer(8, 2, 64, 64, 0.13, window=90, kv_from=1, mlp=_dense(24)),
    _layer(4, 4, 16, 48, 0.3, window=17, mlp=_moe(16, 2, 1, 24)),
])

CONFIGS = {"a": TINY_A, "b": TINY_B, "c": TINY_C}


def bf16_exact(x):
    """Rounds float32 values to the nearest bfloat16 (ties to even), returned as float32."""
    shape = np.shape(x)
    x = np.ascontiguousarray(x, dtype=np.float32).reshape(-1)
    bits = x.view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).reshape(shape)


def tensor_shapes(config) -> dict:
    E, V = config["width"], config["vocab"]
    out = {"embed": (V, E), "pos": (config["max_positions"], E), "final.norm": (E,), "head": (V, E)}
    for i, layer in enumerate(config["layers"]):
        p, mx, mlp = f"l{i}", layer["mixer"], layer["mlp"]
        H, G, D, Vd = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        m = f"{p}.mix"
        out.update({f"{p}.norm1": (E,), f"{p}.canon1": (E, config["canon"]["taps"]), f"{p}.dwa": (i + 2,),
                    f"{m}.q": (H * D, E), f"{m}.q.norm": (H * D,), f"{m}.r1": (H,), f"{m}.r2": (H,), f"{m}.o": (E, H * Vd)})
        if mx.get("kv_from") is None:
            out.update({f"{m}.k": (G * D, E), f"{m}.k.norm": (G * D,), f"{m}.v": (G * Vd, E)})
        if mlp is None:
            continue
        out[f"{p}.norm2"] = (E,)
        f = f"{p}.mlp"
        if mlp["kind"] == "dense":
            out.update({f"{f}.up": (mlp["ff"], E), f"{f}.down": (E, mlp["ff"])})
            continue
        n, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        out[f"{f}.table"] = (V, mlp["router"]["top"])
        for e in range(n):
            out.update({f"{f}.e{e}.gate": (F, E), f"{f}.e{e}.up": (F, E), f"{f}.e{e}.down": (E, F)})
        if mlp.get("shared"):
            S = mlp["shared"]["ff"]
            out.update({f"{f}.shared.gate": (S, E), f"{f}.shared.up": (S, E), f"{f}.shared.down": (E, S),
                        f"{f}.shared.sg": (1, E)})
    return out


def make_weights(config, seed: int, std: float = 0.1) -> dict:
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        if last == "table":
            n = config["layers"][int(name[1:name.index(".")])]["mlp"]["router"]["experts"]
            out[name] = np.stack([rng.permutation(n)[:shape[1]] for _ in range(shape[0])]).astype(np.int32)
            continue
        if name == "embed":
            x = rng.normal(0.0, 1.0, shape)
        elif name == "pos":
            x = rng.normal(0.0, 0.7, shape)
        elif last in ("norm", "norm1", "norm2"):
            x = rng.uniform(0.6, 1.6, shape)
        elif last == "canon1":
            x = rng.normal(0.0, 0.5, shape)
        elif last == "dwa":
            x = rng.normal(0.0, 0.4, shape)
            x[-1] = rng.uniform(0.8, 1.3)
        elif last == "r1":
            x = rng.uniform(0.6, 2.2, shape)
            x[int(rng.integers(0, shape[0]))] = 0.05
        elif last == "r2":
            x = rng.uniform(0.08, 0.6, shape)
        else:
            x = rng.normal(0.0, std * (48.0 / shape[-1]) ** 0.5 * 1.5, shape)
        out[name] = bf16_exact(np.asarray(x, np.float32))
    return out


def write_model_dir(path, config, weights) -> Path:
    """config.json + model.safetensors (bfloat16, tables int32), through the package's writer."""
    import torch
    from alpacca_b200.weights import write_safetensors
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(config))
    entries = []
    for n, w in weights.items():
        if w.dtype == np.int32:
            entries.append((n, "I32", tuple(w.shape), (lambda w=w: torch.from_numpy(np.array(w)))))
        else:
            entries.append((n, "BF16", tuple(w.shape), (lambda w=w: torch.from_numpy(np.array(w)).to(torch.bfloat16))))
    write_safetensors(path / "model.safetensors", entries)
    return path


def random_config(seed: int) -> dict:
    """A configuration drawn from a fixed seed: 1 to 6 layers in any order, sizes of every kind."""
    rng = np.random.default_rng(9000 + seed)

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

    layers, owners = [], []
    for i in range(int(rng.integers(1, 7))):
        window = pick(None, 1, 3, 17, 63, 64, 65, 100)
        if owners and rng.random() < 0.4:
            o = layers[pick(*owners)]["mixer"]
            j = next(k for k in owners if layers[k]["mixer"] is o)
            layers.append(_layer(o["kv_heads"] * pick(1, 2, 3), o["kv_heads"], o["dim"], o["vdim"], float(pick(0.2, 0.4)),
                                 window, j, mlp()))
            continue
        kv, dim = pick(1, 2, 3), pick(8, 12, 16, 32, 48, 64, 72, 128)
        vdim = dim if rng.random() < 0.5 else pick(8, 16, 24, 80)
        layers.append(_layer(kv * pick(1, 2, 3, 5), kv, dim, vdim, float(pick(0.15, 0.3, 0.5)), window, None, mlp()))
        owners.append(i)
    return _model(pick(97, 150, 257), pick(24, 37, 56, 64, 100, 200), pick(160, 513), float(pick(1e-6, 1e-5, 1e-3)),
                  pick(1, 2, 3, 4, 6), float(pick(3.0, 15.0, 50.0)), layers)
