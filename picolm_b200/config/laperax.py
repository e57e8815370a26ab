"""Typed configuration of the Laperax design: a decoder whose layers are listed one by one in config.json, each with one
norm in front of a mixer and a mixture of experts side by side (or of a mixer alone), and one of three mixers: linear
attention with a constant decay a head over rotated queries and keys, softmax attention over a sliding window with
normed queries and keys, and a delta rule with one decay a head.

config.json keys: `architecture` ("Laperax"), `vocab`, `width`, `norm.eps`, `logit_scale`, `logit_softcap`, and `layers`: a
list of `{"type": "retention" | "attention" | "delta", "mixer": {...}, "mlp": null | {...}}` with
  retention  {heads, dim, vdim, decay: [...], rot?: {base, dims}}
  attention  {heads, kv_heads, dim, vdim, scale, rot?: {base, dims}, mask?: {size}}
  delta      {heads, kv_heads, dim, vdim, conv}
  mlp        {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "scale"}}
Every size and constant is read from there, per layer; nothing is assumed equal between layers.  A mixer without `rot`
rotates nothing, attention without `mask` sees every earlier key.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .dobepel import _need, _number, _plain, _positive
from .llama import ConfigError

ARCHITECTURE = "Laperax"
MLP_KINDS = ("moe",)


def _sizes(m, keys, where: str) -> Dict[str, Any]:
    out = {k: _positive(_need(m, k, where), f"{where}.{k}") for k in keys}
    if "kv_heads" in out and out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads is not a multiple of kv_heads")
    return out


def _read_rot(m, where: str) -> Optional[Dict[str, Any]]:
    rot = m.get("rot")
    if rot is None:
        return None
    dims = _number(_need(rot, "dims", f"{where}.rot"), f"{where}.rot.dims", int)
    if dims < 0 or dims % 2 or dims > m["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
    return {"base": _positive(_need(rot, "base", f"{where}.rot"), f"{where}.rot.base", float), "dims": dims} if dims else None


def _read_retention(m, where: str) -> Dict[str, Any]:
    out = _sizes(m, ("heads", "dim", "vdim"), where)
    decay = _need(m, "decay", where)
    if not isinstance(decay, (list, tuple)) or len(decay) != out["heads"]:
        raise ConfigError(f"config.json: {where}.decay must be a list with one number per head")
    out["decay"] = [_number(d, f"{where}.decay") for d in decay]
    if any(not 0.0 <= d <= 1.0 for d in out["decay"]):
        raise ConfigError(f"config.json: {where}.decay must lie in [0, 1]")
    out["rot"] = _read_rot(m, where)
    return out


def _read_attention(m, where: str) -> Dict[str, Any]:
    out = _sizes(m, ("heads", "kv_heads", "dim", "vdim"), where)
    out["scale"] = _positive(_need(m, "scale", where), f"{where}.scale", float)
    out["rot"] = _read_rot(m, where)
    mask = m.get("mask")
    out["mask"] = None if mask is None else {"size": _positive(_need(mask, "size", f"{where}.mask"), f"{where}.mask.size")}
    return out


def _read_delta(m, where: str) -> Dict[str, Any]:
    return _sizes(m, ("heads", "kv_heads", "dim", "vdim", "conv"), where)


MIXERS = {"retention": _read_retention, "attention": _read_attention, "delta": _read_delta}


def _read_mlp(mlp, where: str) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}.kind={kind!r} is not known ({', '.join(MLP_KINDS)})")
    router = _need(mlp, "router", where)
    out: Dict[str, Any] = {
        "kind": kind,
        "expert": {"ff": _positive(_need(_need(mlp, "expert", where), "ff", f"{where}.expert"), f"{where}.expert.ff")},
        "router": {k: _positive(_need(router, k, f"{where}.router"), f"{where}.router.{k}") for k in ("experts", "top")}}
    out["router"]["scale"] = _number(_need(router, "scale", f"{where}.router"), f"{where}.router.scale")
    if out["router"]["top"] > out["router"]["experts"]:
        raise ConfigError(f"config.json: {where}.router.top exceeds the number of experts")
    return out


@dataclass(frozen=True)
class LaperaxLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": {k: _plain(v) for k, v in self.mixer.items() if v is not None}, "mlp": _plain(self.mlp)}


@dataclass(frozen=True)
class LaperaxConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    logit_softcap: float
    layers: Tuple[LaperaxLayer, ...]
    architecture: str = ARCHITECTURE

    @staticmethod
    def from_dict(raw: Mapping[str, Any]) -> "LaperaxConfig":
        vocab = _positive(_need(raw, "vocab", "the model"), "vocab")
        width = _positive(_need(raw, "width", "the model"), "width")
        eps = _number(_need(_need(raw, "norm", "the model"), "eps", "norm"), "norm.eps")
        if eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        scale = _number(_need(raw, "logit_scale", "the model"), "logit_scale")
        cap = _positive(_need(raw, "logit_softcap", "the model"), "logit_softcap", float)
        entries = _need(raw, "layers", "the model")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]"
            kind = _need(e, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}.type={kind!r} is not known ({', '.join(MIXERS)})")
            mixer = MIXERS[kind](_need(e, "mixer", where), f"{where}.mixer")
            layers.append(LaperaxLayer(kind, mixer, _read_mlp(e.get("mlp"), f"{where}.mlp")))
        return LaperaxConfig(vocab, width, eps, scale, cap, tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap,
                "layers": [layer.to_dict() for layer in self.layers]}

    def replace(self, **kw) -> "LaperaxConfig":
        return dataclasses.replace(self, **kw)
