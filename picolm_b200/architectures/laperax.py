"""Laperax as a layout of parts: every layer is a `parallel_norm` arrangement with one norm whose rows both sublayers read,
around one of three mixers (`retention`; `attention` over a window, its queries and keys normed without weights;
`gated_delta` with one decay a head and a full gate) and a `routed_mlp` of ungated experts, or none.  The embedding
passes a norm, the logits a factor and a soft cap.
This file only fills `PartSpec`s from `LaperaxConfig` and names the tensors (`l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `embed`,
`embed.norm`, `final.norm`, `head`); the parts know nothing of the design.
"""
from __future__ import annotations

from ..config.laperax import ARCHITECTURE, LaperaxConfig
from ..config.registry import register_architecture
from ..config.spec import ModelSpec, PartSpec
from ..parts.block import parallel_norm_layer

UNIT_NORM_EPS = 1e-6             # inside the root where the delta rule's queries and keys are made unit vectors


def _norm(cfg: LaperaxConfig, prefix: str) -> PartSpec:
    return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "name": ""}, prefix=prefix)


def _position(m) -> PartSpec:
    rot = m.get("rot")
    if rot is None:
        return PartSpec("none")
    return PartSpec("rope", {"head_dim": m["dim"], "rotary_dim": rot["dims"], "theta": rot["base"], "scaling": None,
                             "pairing": "half", "max_positions": 1 << 30})


def _mixer_spec(cfg: LaperaxConfig, layer) -> PartSpec:
    m, d = layer.mixer, cfg.width
    if layer.type == "retention":
        return PartSpec("retention", {"hidden_size": d, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"],
                                      "decay": list(m["decay"]), "eps": cfg.norm_eps, "position": _position(m)}, prefix="mix")
    if layer.type == "attention":
        return PartSpec("attention", {
            "hidden_size": d, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "value_dim": m["vdim"], "scale": m["scale"], "window": m["mask"]["size"] if m.get("mask") else None,
            "position": _position(m), "qk_norm": {"eps": cfg.norm_eps, "per_head": True, "weights": False},
            "q_name": "q", "k_name": "k", "v_name": "v", "o_name": "o"}, prefix="mix")
    if layer.type == "delta":
        return PartSpec("gated_delta", {
            "hidden_size": d, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
            "conv": m["conv"], "eps": cfg.norm_eps, "l2_eps": UNIT_NORM_EPS, "decay": "head", "gate": "full",
            "gate_activation": "silu"}, prefix="mix")
    raise ValueError(f"no mixer of type {layer.type!r}")


def _feed_forward_spec(cfg: LaperaxConfig, mlp) -> PartSpec:
    return PartSpec("routed_mlp", {
        "hidden_size": cfg.width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
        "expert_size": mlp["expert"]["ff"], "route_scale": mlp["router"]["scale"], "activation": "relu2",
        "router_name": "router", "expert_prefix": "e", "up_name": "up", "down_name": "down"}, prefix="mlp")


def laperax_spec(cfg: LaperaxConfig) -> ModelSpec:
    layers = [parallel_norm_layer(prefix=f"l{i}", mixer=_mixer_spec(cfg, layer), mixer_norm=_norm(cfg, "norm1"),
                                  feed_forward=_feed_forward_spec(cfg, layer.mlp) if layer.mlp is not None else None)
              for i, layer in enumerate(cfg.layers)]
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed",
                                               "norm": {"name": "embed.norm", "eps": cfg.norm_eps}}),
        layers=tuple(layers), schedule=tuple(range(len(layers))),
        final_norm=_norm(cfg, "final.norm"),
        lm_head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "head",
                                     "scale": cfg.logit_scale, "softcap": cfg.logit_softcap}),
        max_positions=1 << 30)


register_architecture(ARCHITECTURE, LaperaxConfig.from_dict, laperax_spec)
