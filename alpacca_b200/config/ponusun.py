"""The configuration of the Ponusun decoder, by its config.json keys.

    {"architecture": "Ponusun", "vocab": V, "width": E, "max_positions": P, "norm": {"eps": e}, "canon": {"taps": n},
     "logit_softcap": c,
     "layers": [{"type": "attention", "mixer": {...}, "mlp": {...} | null}, ...]}

A layer's mixer sizes:
    attention   heads, kv_heads, dim, vdim, scale, mask: {size} (may be left out: every earlier token is seen),
                kv_from: j (may be left out; the layer then has no keys and values of its own and reads those of the
                earlier layer j)
and its feed-forward: {"kind": "dense", "ff": F}, or {"kind": "moe", "expert": {"ff": F}, "router": {"experts": n,
"top": k}, "shared": {"ff": S}} (shared may be left out).  Every size and constant is read from here; `max_positions` is
the number of learned positions and the longest sequence.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .base import ModelConfig
from .lefatar import _check_keys, _is_int, _is_num

ATTENTION = {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float}


@dataclass(frozen=True)
class PonusunConfig(ModelConfig):
    vocab: int = None
    width: int = None
    max_positions: int = None
    norm: dict = field(default_factory=dict)
    canon: dict = field(default_factory=dict)
    logit_softcap: float = None
    layers: list = field(default_factory=list)
    bos_token_id: int | None = None
    eos_token_id: int | list | None = None

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def stop_tokens(self) -> tuple[int, ...]:
        e = self.eos_token_id
        if e is None:
            return ()
        return tuple(e) if isinstance(e, (list, tuple)) else (int(e),)

    @property
    def bos_token(self) -> int | None:
        return self.bos_token_id

    def to_dict(self) -> dict:
        out = super().to_dict()
        out.pop("architectures", None)
        out = {"architecture": self.architecture, **out}
        for key in ("bos_token_id", "eos_token_id"):
            if out.get(key) is None:
                out.pop(key, None)
        return out

    def validate(self) -> list[str]:
        bad: list[str] = []
        for name in ("vocab", "width", "max_positions"):
            v = getattr(self, name)
            if not (_is_int(v) and v > 0):
                bad.append(f"key '{name}' must be a positive integer, got {v!r}")
        if not (isinstance(self.norm, dict) and _is_num(self.norm.get("eps")) and self.norm["eps"] >= 0):
            bad.append("norm.eps must be a number that is not negative")
        _check_keys("canon", self.canon, {"taps": int}, bad)
        if not (_is_num(self.logit_softcap) and self.logit_softcap > 0):
            bad.append("logit_softcap must be a positive number")
        if not isinstance(self.layers, list) or not self.layers:
            bad.append("'layers' must be a list with at least one layer")
            return bad
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict):
                bad.append(f"{where} must be an object")
                continue
            if layer.get("type") != "attention":
                bad.append(f"{where}.type {layer.get('type')!r} is not supported (supported: attention)")
                continue
            mx = layer.get("mixer")
            if _check_keys(f"{where}.mixer", mx, ATTENTION, bad):
                if mx["heads"] % mx["kv_heads"]:
                    bad.append(f"{where}.mixer: {mx['heads']} heads cannot share {mx['kv_heads']} key/value heads")
                if mx.get("mask") is not None:
                    _check_keys(f"{where}.mixer.mask", mx["mask"], {"size": int}, bad)
                j = mx.get("kv_from")
                if j is not None:
                    other = self.layers[j].get("mixer") if _is_int(j) and 0 <= j < i and isinstance(self.layers[j], dict) else None
                    if not isinstance(other, dict) or other.get("kv_from") is not None:
                        bad.append(f"{where}.mixer.kv_from {j!r} must name an earlier layer with keys and values of its own")
                    elif any(other.get(k) != mx.get(k) for k in ("kv_heads", "dim", "vdim")):
                        bad.append(f"{where}.mixer: kv_heads, dim and vdim must equal those of layer {j}, whose keys and "
                                   "values it reads")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
                bad.append(f"{where}.mlp must be null or an object of kind 'dense' or 'moe'")
                continue
            if mlp["kind"] == "dense":
                _check_keys(f"{where}.mlp", mlp, {"ff": int}, bad)
                continue
            if _check_keys(f"{where}.mlp", mlp, {"expert": dict, "router": dict}, bad):
                _check_keys(f"{where}.mlp.expert", mlp["expert"], {"ff": int}, bad)
                if _check_keys(f"{where}.mlp.router", mlp["router"], {"experts": int, "top": int}, bad) \
                        and mlp["router"]["top"] > mlp["router"]["experts"]:
                    bad.append(f"{where}.mlp.router: {mlp['router']['top']} of {mlp['router']['experts']} experts cannot be "
                               "chosen")
            if mlp.get("shared") is not None:
                _check_keys(f"{where}.mlp.shared", mlp["shared"], {"ff": int}, bad)
        for t in self.stop_tokens if not bad else ():
            if not 0 <= t < self.vocab:
                bad.append(f"eos_token_id {t} lies outside the vocabulary of {self.vocab}")
        return bad
