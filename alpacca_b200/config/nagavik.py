"""The configuration of the Nagavik decoder, by its config.json keys.

    {"architecture": "Nagavik", "vocab": V, "width": E, "max_positions": P, "norm": {"eps": e}, "embedding": {"scale": s},
     "logit_softcap": c, "layers": [{"type": "mamba2" | "attention", "mixer": {...}, "mlp": {...} | null}, ...]}

A layer's mixer sizes:
    mamba2      heads, vdim, state, groups, conv (taps), norm_groups
    attention   heads, kv_heads, dim, vdim, scale, softcap
and its feed-forward: {"kind": "dense", "ff": F}, or {"kind": "moe", "expert": {"ff": F}, "router": {"experts": n,
"top": k}, "shared": {"ff": S}}.  The two bounds (`softcap`, `logit_softcap`) and `shared` may be left out or null.  Every
size and constant is read from here; `max_positions` is the number of learned positions and the longest sequence.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .base import ModelConfig
from .lefatar import _check_keys, _is_int, _is_num

MIXERS = {
    "mamba2": {"heads": int, "vdim": int, "state": int, "groups": int, "conv": int, "norm_groups": int},
    "attention": {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float},
}


def _bad_bound(v) -> bool:
    return v is not None and not (_is_num(v) and v > 0)


@dataclass(frozen=True)
class NagavikConfig(ModelConfig):
    vocab: int = None
    width: int = None
    max_positions: int = None
    norm: dict = field(default_factory=dict)
    embedding: dict = field(default_factory=dict)
    logit_softcap: float | None = None
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
        _check_keys("embedding", self.embedding, {"scale": float}, bad)
        if _bad_bound(self.logit_softcap):
            bad.append("logit_softcap must be a positive number")
        if not isinstance(self.layers, list) or not self.layers:
            bad.append("'layers' must be a list with at least one layer")
            return bad
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict):
                bad.append(f"{where} must be an object")
                continue
            kind = layer.get("type")
            if kind not in MIXERS:
                bad.append(f"{where}.type {kind!r} is not supported (supported: {', '.join(sorted(MIXERS))})")
                continue
            self._check_mixer(f"{where}.mixer", kind, layer.get("mixer"), bad)
            self._check_mlp(f"{where}.mlp", layer.get("mlp"), bad)
        for t in self.stop_tokens if not bad else ():
            if not 0 <= t < self.vocab:
                bad.append(f"eos_token_id {t} lies outside the vocabulary of {self.vocab}")
        return bad

    @staticmethod
    def _check_mixer(where: str, kind: str, mx, bad: list) -> None:
        if not _check_keys(where, mx, MIXERS[kind], bad):
            return
        if kind == "attention":
            if mx["heads"] % mx["kv_heads"]:
                bad.append(f"{where}: {mx['heads']} heads cannot share {mx['kv_heads']} key/value heads")
            if _bad_bound(mx.get("softcap")):
                bad.append(f"{where}.softcap must be a positive number")
            return
        if mx["heads"] % mx["groups"]:
            bad.append(f"{where}: {mx['heads']} heads cannot share {mx['groups']} groups")
        if mx["heads"] * mx["vdim"] % mx["norm_groups"]:
            bad.append(f"{where}: {mx['heads'] * mx['vdim']} columns cannot be normed in {mx['norm_groups']} equal parts")

    @staticmethod
    def _check_mlp(where: str, mlp, bad: list) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            bad.append(f"{where} must be null or an object of kind 'dense' or 'moe'")
            return
        if mlp["kind"] == "dense":
            _check_keys(where, mlp, {"ff": int}, bad)
            return
        if _check_keys(where, mlp, {"expert": dict, "router": dict}, bad):
            _check_keys(f"{where}.expert", mlp["expert"], {"ff": int}, bad)
            if _check_keys(f"{where}.router", mlp["router"], {"experts": int, "top": int}, bad) \
                    and mlp["router"]["top"] > mlp["router"]["experts"]:
                bad.append(f"{where}.router: {mlp['router']['top']} of {mlp['router']['experts']} experts cannot be chosen")
        if mlp.get("shared") is not None:
            _check_keys(f"{where}.shared", mlp["shared"], {"ff": int}, bad)
