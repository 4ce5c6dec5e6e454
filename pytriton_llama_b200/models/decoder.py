"""A decoder-only model assembled from a ``ModelSpec``: embedding, blocks run in the listed order,
final norm and LM head on the wanted rows only.

lite_llama/models/llama.py:189-223 is the same pipeline for one architecture with the LM head
over every position (:221); here only the rows whose logits are asked for reach the head.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..parts.base import CacheNeed, Part, Runtime, TensorSpec, build_part
from .spec import ModelSpec


def _walk(part: Part, spec, prefix: str = ""):
    """Yields (part, spec) of a part and all parts nested in it."""
    yield part, spec
    for name, child in part.children().items():
        yield from _walk(child, spec.parts[name])


class DecoderModel:
    EMBEDDING_ENTRY = -1     # the cache entry that holds the per-request states of the embedding part

    def __init__(self, spec: ModelSpec, runtime: Runtime):
        spec.validate()
        self.spec = spec
        self.rt = runtime
        self.blocks = [build_part("block", b, runtime) for b in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, runtime)
        self.embedding_norm = build_part("norm", spec.embedding_norm, runtime) if spec.embedding_norm is not None else None
        self.embedding_part = build_part("embedding", spec.embedding_part, runtime) if spec.embedding_part is not None else None
        self.embedding: Optional[torch.Tensor] = None
        self.lm_head: Optional[torch.Tensor] = None

    def _roots(self):
        roots = [(b, s) for b, s in zip(self.blocks, self.spec.layers)] + [(self.final_norm, self.spec.final_norm)]
        if self.embedding_norm is not None:
            roots.append((self.embedding_norm, self.spec.embedding_norm))
        if self.embedding_part is not None:
            roots.append((self.embedding_part, self.spec.embedding_part))
        return roots

    def any_part(self, predicate) -> bool:
        """True if ``predicate`` holds for a part of the model (nested parts included)."""
        return any(predicate(part) for root, rspec in self._roots() for part, _ in _walk(root, rspec))

    # ------------------------------------------------------------------ tensors
    def expected_tensors(self) -> Dict[str, TensorSpec]:
        """Checkpoint name -> spec of every tensor the model reads."""
        out: Dict[str, TensorSpec] = {
            self.spec.embedding: TensorSpec((self.spec.vocab_size, self.spec.hidden_size)),
        }
        if self.spec.lm_head is not None:
            out[self.spec.lm_head] = TensorSpec((self.spec.vocab_size, self.spec.hidden_size))
        for shared in self.spec.shared_tensors.values():
            out[shared.name] = shared.spec
        for root, rspec in self._roots():
            for part, pspec in _walk(root, rspec):
                for local, ts in part.tensor_specs().items():
                    out[pspec.tensors[local]] = ts
        return out

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        """``tensors``: checkpoint name -> CPU tensor, already checked against ``expected_tensors``."""
        rt = self.rt
        self.embedding = tensors[self.spec.embedding].to(device=rt.device, dtype=rt.dtype).contiguous()
        if self.spec.lm_head is None:
            self.lm_head = self.embedding
        else:
            self.lm_head = tensors[self.spec.lm_head].to(device=rt.device, dtype=rt.dtype).contiguous()
        for key, shared in self.spec.shared_tensors.items():
            rt.shared[key] = tensors[shared.name].to(device=rt.device, dtype=rt.dtype).contiguous()
        roots = self._roots()
        for root, rspec in roots:
            for part, pspec in _walk(root, rspec):
                specs = part.tensor_specs()
                if specs:
                    part.load({local: tensors.get(pspec.tensors[local]) for local in specs})
        for root, rspec in roots:                      # members first: a part made of others joins what they loaded
            for part, _ in reversed(list(_walk(root, rspec))):
                if hasattr(part, "after_load"):
                    part.after_load()

    # ------------------------------------------------------------------ cache
    def cache_entries(self) -> Dict[int, CacheNeed]:
        """Cache entry id -> what the layers that use it need."""
        out: Dict[int, CacheNeed] = {}
        for e in self.spec.run_order:
            need = self.blocks[e.layer].cache_need()
            if e.cache in out and out[e.cache].group_key() != need.group_key():
                try:        # (runs that only differ in how far back they look share what the farthest-looking needs)
                    need = out[e.cache].merged(need)
                except ValueError:
                    raise ValueError(f"cache entry {e.cache} is used by layers with different needs") from None
                out[e.cache] = need
            out.setdefault(e.cache, need)
        if self.embedding_part is not None:
            out[self.EMBEDDING_ENTRY] = self.embedding_part.cache_need()
        return out

    # ------------------------------------------------------------------ forward
    def forward(self, token_ids: torch.Tensor, ctx, cache_views, logit_rows: Optional[torch.Tensor]):
        """token_ids int32 [T]; ``cache_views(entry, write)`` gives the LayerCacheView of a run;
        returns float32 logits [len(logit_rows), vocab] (None when no row is wanted)."""
        ops = self.rt.ops
        begin = getattr(ops, "begin_forward", None)
        if begin is not None:
            begin()             # (what an operator set keeps per step, such as rotary angles, starts afresh)
        ctx.tokens = token_ids
        if self.embedding_part is not None:
            if self.spec.position_vector is not None or self.embedding_norm is not None:
                raise ValueError("an embedding part goes with neither a position vector nor an embedding norm")
            x, residual = None, self.embedding_part.start_stream(token_ids, self.embedding, self.spec.embedding_scale, ctx,
                                                                 cache_views(self.EMBEDDING_ENTRY, True))
        elif self.spec.position_vector is not None or self.spec.embedding_scale != 1.0:
            # scaled rows plus the position vector, in float32: this is the stream itself, nothing is left to add
            if self.spec.position_vector not in (None, "sinusoidal"):
                raise ValueError(f"unknown position vector {self.spec.position_vector!r}")
            x, residual = None, ops.embed_scaled(token_ids, self.embedding, self.spec.embedding_scale, ctx.positions,
                                                 self.spec.position_base if self.spec.position_vector else 0.0)
        elif self.embedding_norm is not None:
            # the normed rows, in float32, are the stream itself
            x, residual = None, self.embedding_norm.start_stream(ops.embed(token_ids, self.embedding))
        else:
            x, residual = ops.embed(token_ids, self.embedding), None
        run = self.spec.run_order
        for i, e in enumerate(run):
            block = self.blocks[e.layer]
            kw = {}
            if i + 1 < len(run) and getattr(block, "takes_next_norm", False):
                # the norm that reads the residual after this block (the final norm selects rows and does its own work)
                kw["next_norm"] = getattr(self.blocks[run[i + 1].layer], "norm1", None)
            x, residual = block.forward(x, residual, ctx, cache_views(e.cache, e.write), **kw)
        if logit_rows is None or logit_rows.numel() == 0:
            return None
        y, _ = self.final_norm.forward(x, residual, rows=logit_rows)
        logits = ops.linear(y, self.lm_head, out_dtype=torch.float32)
        if self.spec.logit_softcap > 0:
            ops.softcap(logits, self.spec.logit_softcap)
        return logits
