"""Typed configuration of the Nesisun decoder, read from its config.json.

A Nesisun model starts its stream from a scaled embedding and a row looked up by the pair of the token before and the
token.  A layer has one norm, and a mixer and a feed-forward that both read its output and are added together.  The
mixer is grouped-query softmax attention whose values are its keys as projected (with biases on both projections), a
rotation of neighbouring pairs on the first ``rot.dims`` entries of every head, a sliding window that always keeps the
first tokens of the sequence, and a learned sink score per head in the softmax's denominator.  A layer's feed-forward is
dense (gated, gelu), a routed mixture of clamped gated experts some of which may hand their input on unchanged, or
absent.  A layer may use the tensors of another (``weights_of``) with a cache of its own.  Keys of the file:

    architecture, vocab, width, norm.eps, embedding.scale, embedding.bigram.{buckets, mul_prev, mul_cur},
    layers[i].type, layers[i].mixer.{...}, layers[i].mlp (null, or {kind: dense, ff}, or {kind: moe, expert.{ff, limit},
    router.{experts, identity, top, scale}}), layers[i].weights_of
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Dict, List, Optional, Tuple, Union

from .lilenex import DenseMlpConfig, _optional_int
from .llama import ConfigError
from .tibepel import _need, _positive_int


def _integer(d, key, where) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or int(v) != v:
        raise ConfigError(f"{where}{key} must be an integer, got {v!r}")
    return int(v)


@dataclass(frozen=True)
class NeighbourRotation:
    """Entries 2i and 2i + 1 of the first ``dims`` of a head turn by position * base^(-2i/dims)."""
    dims: int
    base: float

    @classmethod
    def from_dict(cls, d, where, head_dim) -> Optional["NeighbourRotation"]:
        if d is None:
            return None
        dims = _positive_int(d, "dims", where)
        if dims % 2 or dims > head_dim:
            raise ConfigError(f"{where}dims={dims} must be even and at most the head size {head_dim}")
        base = float(_need(d, "base", where))
        if not base > 0:
            raise ConfigError(f"{where}base must be positive, got {base}")
        return cls(dims, base)

    def to_dict(self):
        return {"base": self.base, "dims": self.dims}


@dataclass(frozen=True)
class KeyValueAttentionConfig:
    """Mixer of an ``attention`` layer: the values are the keys before their rotation."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int                 # 0: every earlier position is seen
    keep_first: int             # positions below this are always seen
    rot: Optional[NeighbourRotation]

    @classmethod
    def from_dict(cls, d, where) -> "KeyValueAttentionConfig":
        heads, kv = _positive_int(d, "heads", where), _positive_int(d, "kv_heads", where)
        if heads % kv:
            raise ConfigError(f"{where}heads={heads} is no multiple of kv_heads={kv}")
        dim = _positive_int(d, "dim", where)
        if _positive_int(d, "vdim", where) != dim:
            raise ConfigError(f"{where}vdim={d['vdim']} must equal dim={dim}: the values are the keys")
        mask = d.get("mask") or {}
        return cls(heads, kv, dim, float(_need(d, "scale", where)), _optional_int(mask, "size", where + "mask."),
                   _optional_int(mask, "keep_first", where + "mask."), NeighbourRotation.from_dict(d.get("rot"), where + "rot.", dim))

    def to_dict(self):
        d = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.dim}
        if self.window:
            d["mask"] = {"keep_first": self.keep_first, "size": self.window}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class ClampedMoeConfig:
    ff: int
    limit: float
    experts: int
    identity: int               # experts after those that have no weights and hand their input on
    top: int
    scale: float                # factor on the routing weights

    @classmethod
    def from_dict(cls, d, where) -> "ClampedMoeConfig":
        expert, router = _need(d, "expert", where), _need(d, "router", where)
        limit = float(_need(expert, "limit", where + "expert."))
        if not limit > 0:
            raise ConfigError(f"{where}expert.limit must be positive, got {limit}")
        experts, top = _positive_int(router, "experts", where + "router."), _positive_int(router, "top", where + "router.")
        identity = _optional_int(router, "identity", where + "router.")
        if top > experts + identity:
            raise ConfigError(f"{where}router.top={top} exceeds the {experts + identity} experts")
        return cls(_positive_int(expert, "ff", where + "expert."), limit, experts, identity, top, float(router.get("scale", 1.0)))

    def to_dict(self):
        router = {"experts": self.experts, "scale": self.scale, "top": self.top}
        if self.identity:
            router["identity"] = self.identity
        return {"expert": {"ff": self.ff, "limit": self.limit}, "kind": "moe", "router": router}


def _mlp_from_dict(d, where):
    if d is None:
        return None
    kind = _need(d, "kind", where)
    if kind == "dense":
        return DenseMlpConfig(_positive_int(d, "ff", where))
    if kind == "moe":
        return ClampedMoeConfig.from_dict(d, where)
    raise ConfigError(f"{where}kind={kind!r} is not supported (known: dense, moe)")


@dataclass(frozen=True)
class NesisunLayerConfig:
    type: str
    mixer: KeyValueAttentionConfig
    mlp: Union[None, DenseMlpConfig, ClampedMoeConfig]
    weights_of: Optional[int]   # the layer whose tensors this one uses; None: its own

    def to_dict(self):
        d = {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(), "type": self.type}
        if self.weights_of is not None:
            d["weights_of"] = self.weights_of
        return d


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int

    @classmethod
    def from_dict(cls, d, where) -> Optional["BigramConfig"]:
        if d is None:
            return None
        return cls(_positive_int(d, "buckets", where), _integer(d, "mul_prev", where), _integer(d, "mul_cur", where))

    def to_dict(self):
        return {"buckets": self.buckets, "mul_cur": self.mul_cur, "mul_prev": self.mul_prev}


@dataclass(frozen=True)
class NesisunConfig:
    vocab: int
    width: int
    layers: Tuple[NesisunLayerConfig, ...]
    norm_eps: float
    embedding_scale: float
    bigram: Optional[BigramConfig]
    initializer_range: float = 0.02
    eos_token_id: Union[None, int, List[int]] = None

    @classmethod
    def from_dict(cls, data: Dict[str, Any]) -> "NesisunConfig":
        raw_layers = _need(data, "layers", "")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]."
            kind = _need(L, "type", where)
            if kind != "attention":
                raise ConfigError(f"{where}type={kind!r} is not supported (known: attention)")
            owner = L.get("weights_of")
            layers.append(NesisunLayerConfig(kind, KeyValueAttentionConfig.from_dict(_need(L, "mixer", where), where + "mixer."),
                                             _mlp_from_dict(L.get("mlp"), where + "mlp."),
                                             None if owner is None else _integer(L, "weights_of", where)))
        for i, L in enumerate(layers):
            if L.weights_of is None:
                continue
            where, j = f"layers[{i}].", L.weights_of
            if not 0 <= j < len(layers) or layers[j].weights_of is not None:
                raise ConfigError(f"{where}weights_of={j} must name a layer that has tensors of its own")
            if (L.mixer, L.mlp) != (layers[j].mixer, layers[j].mlp):
                raise ConfigError(f"{where}mixer and mlp must equal those of layer {j}, whose tensors it uses")
        eps = float(_need(_need(data, "norm", ""), "eps", "norm."))
        if not eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {eps}")
        emb = data.get("embedding") or {}
        eos = data.get("eos_token_id")
        return cls(vocab=_positive_int(data, "vocab", ""), width=_positive_int(data, "width", ""), layers=tuple(layers), norm_eps=eps,
                   embedding_scale=float(emb.get("scale", 1.0)), bigram=BigramConfig.from_dict(emb.get("bigram"), "embedding.bigram."),
                   initializer_range=float(data.get("initializer_range", 0.02)),
                   eos_token_id=[int(e) for e in eos] if isinstance(eos, (list, tuple)) else eos)

    @classmethod
    def from_folder(cls, folder: Union[str, Path]) -> "NesisunConfig":
        return cls.from_dict(json.loads((Path(folder) / "config.json").read_text()))

    def to_dict(self) -> Dict[str, Any]:
        emb: Dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = self.bigram.to_dict()
        d = {"architecture": "Nesisun", "embedding": emb, "layers": [L.to_dict() for L in self.layers], "norm": {"eps": self.norm_eps},
             "vocab": self.vocab, "width": self.width, "initializer_range": self.initializer_range}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    @property
    def eos_token_ids(self) -> List[int]:
        if self.eos_token_id is None:
            return []
        return [self.eos_token_id] if isinstance(self.eos_token_id, int) else list(self.eos_token_id)
