"""The two ends of the model: token embedding and LM head.

Embedding: `x = float(embed[token])`, no scale (picolm/model_core.c:1785-1786).
Head: `logits = W x`, fp32, no bias, no soft-cap (picolm/model_core.c:2220); with
tied embeddings W is the embedding matrix itself (picolm/safetensors.c:248-251).
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache.spec import CacheSpec
from .base import Part, WeightSpec, register_part


@register_part("embedding", "token_embedding")
class TokenEmbedding(Part):
    """params: vocab_size, hidden_size, name (absolute tensor name), scale (optional: the rows are multiplied by it
    in float32 as they enter the stream; the reference has none)."""

    def weight_specs(self):
        return {self.params["name"]: WeightSpec((self.params["vocab_size"], self.params["hidden_size"]))}

    def load(self, tensors):
        self.table = tensors[self.params["name"]]

    graph_safe = True
    graph_safe_prompts = True

    def forward(self, step):
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
    embedding's own name when the two are tied)."""

    def weight_specs(self):
        return {self.params["name"]: WeightSpec((self.params["vocab_size"], self.params["hidden_size"]))}

    def load(self, tensors):
        self.weight = tensors[self.params["name"]]

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def forward(self, h_rows):
        return ops.linear(h_rows, self.weight, torch.float32)
