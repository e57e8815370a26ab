"""Dobepel as a layout of parts: every layer is a `sandwich_norm` arrangement whose closing norms carry the model's
residual factor, around a pair of mixers (`parallel`: `attention` with slopes and a window that keeps the first
positions, beside `lightning`), each half behind a norm of its own, and a feed-forward (`mlp` with the exact GELU, or
`routed_mlp` by biased logits with a shared expert) or none; the embedding adds a row for the pair with the token before.
This file only fills `PartSpec`s from `DobepelConfig` and names the tensors (`l<i>.norm1`, `l<i>.norm1b`, `l<i>.mix.*`,
`l<i>.norm2`, `l<i>.norm2b`, `l<i>.mlp.*`, `embed`, `bigram`, `final.norm`, `head`); the parts know nothing of the design.
"""
from __future__ import annotations

from ..config.dobepel import ARCHITECTURE, DobepelConfig
from ..config.registry import register_architecture
from ..config.spec import ModelSpec, PartSpec
from ..parts.block import sandwich_norm_layer

JOIN_SCALE = 0.5                 # the pair's result is the mean of its halves
SLOPE_OCTAVES = 8.0              # the heads' slopes fall geometrically from 2^(-8/H) to 2^-8


def _norm(cfg: DobepelConfig, prefix: str, scale: float = 1.0) -> PartSpec:
    params = {"size": cfg.width, "eps": cfg.norm_eps, "name": ""}
    if scale != 1.0:
        params["scale"] = scale
    return PartSpec("rmsnorm", params, prefix=prefix)


def _mixer_spec(cfg: DobepelConfig, m) -> PartSpec:
    left, right, d = m["left"], m["right"], cfg.width
    H = left["heads"]
    mask = left.get("mask") or {}
    attention = PartSpec("attention", {
        "hidden_size": d, "num_heads": H, "num_kv_heads": left["kv_heads"], "head_dim": left["dim"], "value_dim": left["vdim"],
        "scale": left["scale"], "window": mask.get("size"), "keep_first": mask.get("keep_first", 0),
        "slopes": [2.0 ** (-SLOPE_OCTAVES * (h + 1) / H) for h in range(H)],
        "q_name": "q", "k_name": "k", "v_name": "v", "o_name": "o"}, prefix="left")
    lightning = PartSpec("lightning", {"hidden_size": d, "heads": right["heads"], "dim": right["dim"], "vdim": right["vdim"],
                                       "decay": list(right["decay"]), "eps": cfg.norm_eps}, prefix="right")
    return PartSpec("parallel", {"left": attention, "right": lightning, "left_scale": JOIN_SCALE, "right_scale": JOIN_SCALE,
                                 "left_norm": _norm(cfg, "left.out"), "right_norm": _norm(cfg, "right.out")}, prefix="mix")


def _feed_forward_spec(cfg: DobepelConfig, mlp) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("mlp", {"hidden_size": cfg.width, "intermediate_size": mlp["ff"], "activation": "gelu_erf",
                                "up_name": "up", "down_name": "down"}, prefix="mlp")
    shared = {"size": mlp["shared"]["ff"], "prefix": "shared", "gate": None} if mlp.get("shared") else None
    return PartSpec("routed_mlp", {
        "hidden_size": cfg.width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
        "expert_size": mlp["expert"]["ff"], "route_scale": 1.0, "groups": None, "scores": "logits",
        "router_name": "router", "correction_name": "router.b", "expert_prefix": "e", "gate_name": "gate", "up_name": "up",
        "down_name": "down", "shared": shared}, prefix="mlp")


def dobepel_spec(cfg: DobepelConfig) -> ModelSpec:
    layers, ignored = [], []
    for i, layer in enumerate(cfg.layers):
        ff = {}
        if layer.mlp is not None:
            ff = dict(feed_forward=_feed_forward_spec(cfg, layer.mlp), feed_forward_norm=_norm(cfg, "norm2"),
                      feed_forward_post_norm=_norm(cfg, "norm2b", cfg.residual_mult))
        else:
            ignored.append(rf"^l{i}\.norm2b?$")              # a layer that only mixes has no use for them
        layers.append(sandwich_norm_layer(prefix=f"l{i}", mixer=_mixer_spec(cfg, layer.mixer), mixer_norm=_norm(cfg, "norm1"),
                                          mixer_post_norm=_norm(cfg, "norm1b", cfg.residual_mult), **ff))
    b = cfg.bigram
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_pair_embedding", {
            "vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed", "pair_name": "bigram",
            "buckets": b["buckets"], "mul_prev": b["mul_prev"], "mul_cur": b["mul_cur"]}),
        layers=tuple(layers), schedule=tuple(range(len(layers))),
        final_norm=_norm(cfg, "final.norm"),
        lm_head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "head"}),
        max_positions=1 << 30, ignored_tensors=tuple(ignored))


register_architecture(ARCHITECTURE, DobepelConfig.from_dict, dobepel_spec)
