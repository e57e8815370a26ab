"""The two ends of the model: token embedding and LM head.

Embedding: `x = float(embed[token])`, no scale (picolm/model_core.c:1785-1786).
Head: `logits = W x`, fp32, no bias, no soft-cap unless a design asks for one (picolm/model_core.c:2220); with
tied embeddings W is the embedding matrix itself (picolm/safetensors.c:248-251).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..cache.spec import CacheSpec
from .base import Part, WeightSpec, register_part


@register_part("embedding", "token_embedding")
class TokenEmbedding(Part):
    """params: vocab_size, hidden_size, name (absolute tensor name), scale (optional: the rows are multiplied by it
    in float32 as they enter the stream; the reference has none), norm (optional, in place of a scale: {"name" (absolute
    tensor name of the weight [hidden_size]), "eps"}: the rows pass that RMS norm as they enter the stream)."""

    def __init__(self, params, runtime):
        super().__init__(params, runtime)
        self.norm: Optional[dict] = self.params.get("norm")
        if self.norm is not None and float(self.params.get("scale", 1.0)) != 1.0:
            raise ValueError("token_embedding: a scale in front of a norm does nothing; give one of them")

    def weight_specs(self):
        specs = {self.params["name"]: WeightSpec((self.params["vocab_size"], self.params["hidden_size"]))}
        if self.norm is not None:
            specs[self.norm["name"]] = WeightSpec((self.params["hidden_size"],), init="ones_normal")
        return specs

    def load(self, tensors):
        self.table = tensors[self.params["name"]]
        if self.norm is not None:
            self.norm_weight = tensors[self.norm["name"]]
            if self.norm_weight.dtype != self.table.dtype:
                self.table, self.norm_weight = self.table.to(torch.float32), self.norm_weight.to(torch.float32)

    graph_safe = True
    graph_safe_prompts = True

    def forward(self, step):
        if self.norm is not None:
            return ops.embed_norm(step.tok_ids, self.table, self.norm_weight, float(self.norm["eps"]))
        return ops.embed(step.tok_ids, self.table, scale=float(self.params.get("scale", 1.0)))


@register_part("embedding", "token_pair_embedding")
class TokenPairEmbedding(Part):
    """The token's row of one table plus a row of a second one that the pair (token before, token) picks:
    `(before * mul_prev + token * mul_cur) mod buckets`, and the extra row `buckets` for a sequence's first token.  The
    token before is part of a sequence's state (`cache_specs`).  params: vocab_size, hidden_size, name and pair_name
    (absolute tensor names), buckets, mul_prev, mul_cur, scale (optional, as `token_embedding`'s)."""

    graph_safe = True
    graph_safe_prompts = True

    def weight_specs(self):
        p = self.params
        return {p["name"]: WeightSpec((p["vocab_size"], p["hidden_size"])),
                p["pair_name"]: WeightSpec((p["buckets"] + 1, p["hidden_size"]))}

    def load(self, tensors):
        self.table, self.pairs = tensors[self.params["name"]], tensors[self.params["pair_name"]]
        if self.table.dtype != self.pairs.dtype:
            self.table, self.pairs = self.table.to(torch.float32), self.pairs.to(torch.float32)

    def cache_specs(self):
        return [CacheSpec.state((1,), dtype="int32")]

    def forward(self, step, caches):
        p = self.params
        return ops.embed_pair(step, self.table, self.pairs, caches[0].state, p["mul_prev"], p["mul_cur"],
                              scale=float(p.get("scale", 1.0)))


@register_part("head", "lm_head")
class LMHead(Part):
    """params: vocab_size, hidden_size, name (absolute tensor name; the
    embedding's own name when the two are tied), scale (optional: the logits are multiplied by it), softcap (optional:
    then `softcap * tanh(logits / softcap)`)."""

    def weight_specs(self):
        return {self.params["name"]: WeightSpec((self.params["vocab_size"], self.params["hidden_size"]))}

    def load(self, tensors):
        self.weight = tensors[self.params["name"]]

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def forward(self, h_rows):
        logits = ops.linear(h_rows, self.weight, torch.float32)
        scale, cap = float(self.params.get("scale") or 1.0), self.params.get("softcap")
        if cap is not None:
            return ops.squash(logits, scale, float(cap))
        return logits if scale == 1.0 else logits.mul_(scale)
