"""A decoder described as data: which parts each layer has and in which order layers run.
(lite_llama writes the same arrangement as code: ``LlamaDecoderLayer`` with its two norms, attention
and feed-forward, and ``LlamaModel`` with a ``ModuleList`` of them run in order,
lite_llama/models/llama.py:122-163,165-225.)"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

from ..parts.base import PartSpec, TensorSpec


@dataclass
class RunEntry:
    """One run of a layer.  ``cache`` names the cache entry it uses (entries are numbered by the
    model; two runs that name the same entry share keys and values).  ``write`` is False when the
    run only reads what another run stored in that entry."""
    layer: int
    cache: int
    write: bool = True


@dataclass(frozen=True)
class SharedTensor:
    """A tensor of the checkpoint that belongs to no single layer."""
    name: str                           # checkpoint name
    spec: TensorSpec


@dataclass
class ModelSpec:
    architecture: str
    hidden_size: int
    vocab_size: int
    embedding: str                      # checkpoint name of the [vocab, hidden] table
    layers: List[PartSpec]              # block specs (each with nested norm/mixer/ffn specs)
    run_order: List[RunEntry]
    final_norm: PartSpec
    lm_head: Optional[str]              # checkpoint name, or None when tied to the embedding
    initializer_range: float = 0.02
    eos_token_ids: List[int] = field(default_factory=list)
    max_position_embeddings: Optional[int] = None
    embedding_scale: float = 1.0        # the looked-up row is multiplied by this
    position_vector: Optional[str] = None   # "sinusoidal": entry 2i, 2i+1 of the stream get sin, cos(p * base^(-2i/width)) added
    position_base: float = 10000.0
    logit_softcap: float = 0.0          # > 0: logits <- cap * tanh(logits / cap)
    embedding_part: Optional[PartSpec] = None   # an embedding part that makes the stream from the scaled rows (and a state of its own)
    embedding_norm: Optional[PartSpec] = None   # a norm part the looked-up rows pass before they become the stream
    shared_tensors: Dict[str, "SharedTensor"] = field(default_factory=dict)   # read by parts of every layer (Runtime.shared)

    def validate(self) -> None:
        n = len(self.layers)
        writers: Dict[int, int] = {}
        for i, e in enumerate(self.run_order):
            if not 0 <= e.layer < n:
                raise ValueError(f"run_order[{i}] names layer {e.layer}, but there are {n} layers")
            if e.write:
                writers.setdefault(e.cache, i)
        for i, e in enumerate(self.run_order):
            if not e.write and (e.cache not in writers or writers[e.cache] > i):
                raise ValueError(f"run_order[{i}] reads cache entry {e.cache} before any run writes it")
