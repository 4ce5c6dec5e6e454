"""Typed configuration of the Gepilix decoder, read from its config.json.

A Gepilix model is a list of layers of three types.  ``parallel`` runs a softmax attention inside blocks of positions
(biases, no rotation, one gate per head) beside a gated linear recurrence per channel behind a short convolution, and
takes the mean of their outputs, each normed over the model width.  ``parallel_2`` runs a windowed softmax attention
with rotated halves beside a state-space recurrence with one decay per head and token, and adds them with fixed
scales.  ``wkv`` is a recurrence with a matrix state per head that decays per key channel, fed by mixes of a token and
the one before it.  Scores pass a tanh cap.  A layer's feed-forward is dense (the square of relu), a routed mixture of
gated experts with a shared one, or absent.  Norms are tanh(alpha x) w + b, and each sub-layer's result is multiplied
by a vector before it is added.  Keys of the file:

    architecture, vocab, width, norm.eps, layers[i].type, layers[i].mixer.{...},
    layers[i].mlp (null, or {kind: dense, ff}, or {kind: moe, expert.ff, router.{experts, top}, shared.ff})
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Dict, List, Optional, Tuple, Union

from .lilenex import DenseMlpConfig
from .llama import ConfigError
from .podizen import _heads
from .tibepel import _need, _positive_int


def _positive(d, key, where) -> float:
    v = float(_need(d, key, where))
    if not v > 0:
        raise ConfigError(f"{where}{key} must be positive, got {v}")
    return v


@dataclass(frozen=True)
class ScaledRotation:
    """Entry i of the first ``dims`` of a head is paired with entry i + dims/2; the pair turns by position * f_i,
    f_i = base^(-2i/dims), slowed by ``factor`` where its wavelength is above original/low, kept below
    original/high and mixed in between (``factor`` 1: kept everywhere)."""
    dims: int
    base: float
    factor: float = 1.0
    low: float = 1.0
    high: float = 1.0
    original: float = 1.0

    @classmethod
    def from_dict(cls, d, where, head_dim) -> Optional["ScaledRotation"]:
        if d is None:
            return None
        dims = _positive_int(d, "dims", where)
        if dims % 2 or dims > head_dim:
            raise ConfigError(f"{where}dims={dims} must be even and at most the head size {head_dim}")
        base = _positive(d, "base", where)
        s = d.get("scaling")
        if s is None:
            return cls(dims, base)
        return cls(dims, base, *(_positive(s, k, where + "scaling.") for k in ("factor", "low", "high", "original")))

    def to_dict(self):
        d = {"base": self.base, "dims": self.dims}
        if self != ScaledRotation(self.dims, self.base):
            d["scaling"] = {"factor": self.factor, "high": self.high, "low": self.low, "original": self.original}
        return d


@dataclass(frozen=True)
class CappedAttentionConfig:
    """Left member of ``parallel`` and ``parallel_2``: ``size`` is the block length or the window."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    size: int
    rot: Optional[ScaledRotation]

    @classmethod
    def from_dict(cls, d, where) -> "CappedAttentionConfig":
        heads, kv = _heads(d, where)
        dim = _positive_int(d, "dim", where)
        return cls(heads, kv, dim, _positive_int(d, "vdim", where), float(_need(d, "scale", where)), _positive(d, "softcap", where),
                   _positive_int(_need(d, "mask", where), "size", where + "mask."), ScaledRotation.from_dict(d.get("rot"), where + "rot.", dim))

    def to_dict(self):
        d = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "mask": {"size": self.size}, "scale": self.scale,
             "softcap": self.softcap, "vdim": self.vdim}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class LinearUnitConfig:
    """Right member of ``parallel``: ``width`` channels whose gates come from ``blocks`` square matrices."""
    width: int
    blocks: int
    conv: int

    @classmethod
    def from_dict(cls, d, where) -> "LinearUnitConfig":
        width, blocks = _positive_int(d, "width", where), _positive_int(d, "blocks", where)
        if width % blocks:
            raise ConfigError(f"{where}width={width} is no multiple of blocks={blocks}")
        return cls(width, blocks, _positive_int(d, "conv", where))

    def to_dict(self):
        return {"blocks": self.blocks, "conv": self.conv, "width": self.width}


@dataclass(frozen=True)
class StateSpaceConfig:
    """Right member of ``parallel_2``."""
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int

    @classmethod
    def from_dict(cls, d, where) -> "StateSpaceConfig":
        c = cls(*(_positive_int(d, k, where) for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv")))
        if c.heads % c.groups:
            raise ConfigError(f"{where}heads={c.heads} is no multiple of groups={c.groups}")
        if c.heads * c.vdim % c.norm_groups:
            raise ConfigError(f"{where}heads*vdim={c.heads * c.vdim} is no multiple of norm_groups={c.norm_groups}")
        return c

    def to_dict(self):
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups, "state": self.state,
                "vdim": self.vdim}


@dataclass(frozen=True)
class NormedMeanConfig:
    """Mixer of a ``parallel`` layer."""
    left: CappedAttentionConfig
    right: LinearUnitConfig

    @classmethod
    def from_dict(cls, d, where) -> "NormedMeanConfig":
        left = CappedAttentionConfig.from_dict(_need(d, "left", where), where + "left.")
        if left.rot is not None:
            raise ConfigError(f"{where}left.rot: this attention is not rotated")
        return cls(left, LinearUnitConfig.from_dict(_need(d, "right", where), where + "right."))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class ScaledSumConfig:
    """Mixer of a ``parallel_2`` layer."""
    left: CappedAttentionConfig
    right: StateSpaceConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d, where) -> "ScaledSumConfig":
        return cls(CappedAttentionConfig.from_dict(_need(d, "left", where), where + "left."),
                   StateSpaceConfig.from_dict(_need(d, "right", where), where + "right."),
                   float(_need(d, "left_scale", where)), float(_need(d, "right_scale", where)))

    def to_dict(self):
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(), "right_scale": self.right_scale}


@dataclass(frozen=True)
class WkvConfig:
    """Mixer of a ``wkv`` layer (the decay projection's inner size is the checkpoint's)."""
    heads: int
    dim: int

    @classmethod
    def from_dict(cls, d, where) -> "WkvConfig":
        return cls(_positive_int(d, "heads", where), _positive_int(d, "dim", where))

    def to_dict(self):
        return {"dim": self.dim, "heads": self.heads}


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    top: int
    shared_ff: int              # 0: no shared expert

    @classmethod
    def from_dict(cls, d, where) -> "ExpertsConfig":
        router = _need(d, "router", where)
        experts, top = _positive_int(router, "experts", where + "router."), _positive_int(router, "top", where + "router.")
        if top > experts:
            raise ConfigError(f"{where}router.top={top} exceeds router.experts={experts}")
        shared = d.get("shared")
        return cls(_positive_int(_need(d, "expert", where), "ff", where + "expert."), experts, top,
                   _positive_int(shared, "ff", where + "shared.") if shared else 0)

    def to_dict(self):
        d = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


def _mlp(d, where) -> Union[None, DenseMlpConfig, ExpertsConfig]:
    if d is None:
        return None
    kind = _need(d, "kind", where)
    if kind == "dense":
        return DenseMlpConfig(_positive_int(d, "ff", where))
    if kind == "moe":
        return ExpertsConfig.from_dict(d, where)
    raise ConfigError(f"{where}kind={kind!r} is not supported (known: dense, moe)")


_MIXERS = {"parallel": NormedMeanConfig, "parallel_2": ScaledSumConfig, "wkv": WkvConfig}


@dataclass(frozen=True)
class GepilixLayerConfig:
    type: str
    mixer: Union[NormedMeanConfig, ScaledSumConfig, WkvConfig]
    mlp: Union[None, DenseMlpConfig, ExpertsConfig]

    def to_dict(self):
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(), "type": self.type}


@dataclass(frozen=True)
class GepilixConfig:
    vocab: int
    width: int
    layers: Tuple[GepilixLayerConfig, ...]
    norm_eps: float
    initializer_range: float = 0.02
    eos_token_id: Union[None, int, List[int]] = None

    @classmethod
    def from_dict(cls, data: Dict[str, Any]) -> "GepilixConfig":
        raw_layers = _need(data, "layers", "")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]."
            kind = _need(L, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}type={kind!r} is not supported (known: {sorted(_MIXERS)})")
            layers.append(GepilixLayerConfig(kind, _MIXERS[kind].from_dict(_need(L, "mixer", where), where + "mixer."),
                                             _mlp(L.get("mlp"), where + "mlp.")))
        eos = data.get("eos_token_id")
        return cls(vocab=_positive_int(data, "vocab", ""), width=_positive_int(data, "width", ""), layers=tuple(layers),
                   norm_eps=_positive(_need(data, "norm", ""), "eps", "norm."), initializer_range=float(data.get("initializer_range", 0.02)),
                   eos_token_id=[int(e) for e in eos] if isinstance(eos, (list, tuple)) else eos)

    @classmethod
    def from_folder(cls, folder: Union[str, Path]) -> "GepilixConfig":
        return cls.from_dict(json.loads((Path(folder) / "config.json").read_text()))

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": "Gepilix", "layers": [L.to_dict() for L in self.layers], "norm": {"eps": self.norm_eps},
             "vocab": self.vocab, "width": self.width, "initializer_range": self.initializer_range}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    @property
    def eos_token_ids(self) -> List[int]:
        if self.eos_token_id is None:
            return []
        return [self.eos_token_id] if isinstance(self.eos_token_id, int) else list(self.eos_token_id)
