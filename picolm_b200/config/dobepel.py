"""Typed configuration of the Dobepel design: a decoder whose layers are listed one by one in config.json, each with a
pair of mixers side by side (softmax attention with a linear distance penalty behind a window, and linear attention
with a constant decay a head) and a dense or routed feed-forward (or none), norms on both sides of every sublayer, and
an embedding of token pairs beside the tokens'.

config.json keys: `architecture` ("Dobepel"), `vocab`, `width`, `norm.eps`, `residual_mult` (default 1),
`embedding.bigram: {buckets, mul_prev, mul_cur}`, and `layers`: a list of `{"type": "parallel", "mixer": {...},
"mlp": null | {...}}` with
  mixer  {left: {heads, kv_heads, dim, vdim, scale, mask?: {size, keep_first?}}, right: {heads, dim, vdim, decay: [...]}}
  mlp    {"kind": "dense", "ff"} or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared"?: {"ff"}}
Every size and constant is read from there, per layer; nothing is assumed equal between layers.  A left mixer without
`mask` sees every earlier key.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .llama import ConfigError

ARCHITECTURE = "Dobepel"
MIXER_TYPES = ("parallel",)
MLP_KINDS = ("dense", "moe")


def _need(d, key: str, where: str):
    if not isinstance(d, Mapping) or key not in d:
        raise ConfigError(f"config.json: {where} lacks the key {key!r}")
    return d[key]


def _positive(v, what: str, kind=int):
    try:
        out = kind(v)
    except (TypeError, ValueError):
        raise ConfigError(f"config.json: {what} must be a number, not {v!r}") from None
    if not out > 0:
        raise ConfigError(f"config.json: {what} must be positive")
    return out


def _number(v, what: str, kind=float):
    try:
        return kind(v)
    except (TypeError, ValueError):
        raise ConfigError(f"config.json: {what} must be a number, not {v!r}") from None


def _plain(v):
    if isinstance(v, Mapping):
        return {k: _plain(x) for k, x in v.items()}
    if isinstance(v, (list, tuple)):
        return [_plain(x) for x in v]
    return v


def _read_left(m, where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _positive(_need(m, k, where), f"{where}.{k}") for k in ("heads", "kv_heads", "dim", "vdim")}
    out["scale"] = _positive(_need(m, "scale", where), f"{where}.scale", float)
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads is not a multiple of kv_heads")
    mask = m.get("mask")
    if mask is not None:
        keep = _number(mask.get("keep_first", 0), f"{where}.mask.keep_first", int)
        if keep < 0:
            raise ConfigError(f"config.json: {where}.mask.keep_first must not be negative")
        out["mask"] = {"size": _positive(_need(mask, "size", f"{where}.mask"), f"{where}.mask.size"), "keep_first": keep}
    return out


def _read_right(m, where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _positive(_need(m, k, where), f"{where}.{k}") for k in ("heads", "dim", "vdim")}
    decay = _need(m, "decay", where)
    if not isinstance(decay, (list, tuple)) or len(decay) != out["heads"]:
        raise ConfigError(f"config.json: {where}.decay must be a list with one number per head")
    out["decay"] = [_number(d, f"{where}.decay") for d in decay]
    if any(not 0.0 <= d <= 1.0 for d in out["decay"]):
        raise ConfigError(f"config.json: {where}.decay must lie in [0, 1]")
    return out


def _read_mlp(mlp, where: str) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}.kind={kind!r} is not known ({', '.join(MLP_KINDS)})")
    if kind == "dense":
        return {"kind": kind, "ff": _positive(_need(mlp, "ff", where), f"{where}.ff")}
    router = _need(mlp, "router", where)
    out: Dict[str, Any] = {
        "kind": kind,
        "expert": {"ff": _positive(_need(_need(mlp, "expert", where), "ff", f"{where}.expert"), f"{where}.expert.ff")},
        "router": {k: _positive(_need(router, k, f"{where}.router"), f"{where}.router.{k}") for k in ("experts", "top")}}
    if out["router"]["top"] > out["router"]["experts"]:
        raise ConfigError(f"config.json: {where}.router.top exceeds the number of experts")
    if mlp.get("shared") is not None:
        out["shared"] = {"ff": _positive(_need(mlp["shared"], "ff", f"{where}.shared"), f"{where}.shared.ff")}
    return out


@dataclass(frozen=True)
class DobepelLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": _plain(self.mixer), "mlp": _plain(self.mlp)}


@dataclass(frozen=True)
class DobepelConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    bigram: Mapping[str, int]                  # buckets, mul_prev, mul_cur
    layers: Tuple[DobepelLayer, ...]
    architecture: str = ARCHITECTURE

    @staticmethod
    def from_dict(raw: Mapping[str, Any]) -> "DobepelConfig":
        vocab = _positive(_need(raw, "vocab", "the model"), "vocab")
        width = _positive(_need(raw, "width", "the model"), "width")
        eps = _number(_need(_need(raw, "norm", "the model"), "eps", "norm"), "norm.eps")
        if eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        mult = _number(raw.get("residual_mult", 1.0), "residual_mult")
        b = _need(_need(raw, "embedding", "the model"), "bigram", "embedding")
        bigram = {"buckets": _positive(_need(b, "buckets", "embedding.bigram"), "embedding.bigram.buckets")}
        for k in ("mul_prev", "mul_cur"):
            bigram[k] = _number(_need(b, k, "embedding.bigram"), f"embedding.bigram.{k}", int)
        entries = _need(raw, "layers", "the model")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]"
            kind = _need(e, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type={kind!r} is not known ({', '.join(MIXER_TYPES)})")
            m = _need(e, "mixer", where)
            mixer = {"left": _read_left(_need(m, "left", f"{where}.mixer"), f"{where}.mixer.left"),
                     "right": _read_right(_need(m, "right", f"{where}.mixer"), f"{where}.mixer.right")}
            layers.append(DobepelLayer(kind, mixer, _read_mlp(e.get("mlp"), f"{where}.mlp")))
        return DobepelConfig(vocab, width, eps, mult, bigram, tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult, "embedding": {"bigram": dict(self.bigram)},
                "layers": [layer.to_dict() for layer in self.layers]}

    def replace(self, **kw) -> "DobepelConfig":
        return dataclasses.replace(self, **kw)
