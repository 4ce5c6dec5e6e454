"""An embedding with a term for the pair of the token before and the token.

The stream starts as  table[token] * scale + pairs[row],  row = (token before * mul_prev + token * mul_cur) mod buckets;
a request's first token, which has none before it, takes the last row of the [buckets + 1, hidden] table.  The token
before a portion's first is part of the request's state (one integer in its slot), read and moved on by the kernel
that makes the rows, so that a token which was sampled on the device is known to the next step as well.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import CacheNeed, Part, PartSpec, Runtime, TensorSpec, register_part


@register_part("embedding", "bigram")
class BigramEmbedding(Part):
    """params: ``hidden``, ``buckets``, ``mul_prev``, ``mul_cur``.  Tensor: ``pairs`` [buckets + 1, hidden]."""

    STATE = "last_token"

    def __init__(self, spec: PartSpec, runtime: Runtime):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.buckets = int(p["hidden"]), int(p["buckets"])
        self.mul_prev, self.mul_cur = int(p["mul_prev"]), int(p["mul_cur"])
        if self.buckets < 1:
            raise ValueError(f"buckets={self.buckets} must be positive")
        self.pairs = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {"pairs": TensorSpec((self.buckets + 1, self.hidden))}

    def load(self, tensors) -> None:
        self.pairs = self._to_compute(tensors["pairs"])

    def cache_need(self) -> CacheNeed:
        return CacheNeed(states=((self.STATE, (1,), torch.int32),))

    def start_stream(self, token_ids, table, scale: float, ctx, cache):
        return self.rt.ops.embed_bigram(token_ids, table, scale, self.pairs, self.mul_prev, self.mul_cur, ctx, cache.states[self.STATE])
