"""The Gepilix decoder (architecture name "Gepilix") as a ``ModelSpec``.

Layer i (tensors ``l<i>.*``) is a pre-norm block whose norms have no statistics (tanh(alpha x) w + b) and whose sub-layers'
results are multiplied by a vector each (``ls1``, ``ls2``).  The mixer is the mean of the normed outputs of a block-wise softmax
attention and a gated linear recurrence (``parallel``), the scaled sum of a windowed softmax attention and a state-space
recurrence (``parallel_2``), or RWKV-style time mixing (``wkv``).  The feed-forward is the square of relu, a routed mixture
of gated experts with a shared one, or absent.  The logits come from ``final.norm`` and the table ``head``.
"""
from __future__ import annotations

from ..config.gepilix import (CappedAttentionConfig, GepilixConfig, LinearUnitConfig, NormedMeanConfig, ScaledRotation, ScaledSumConfig,
                              StateSpaceConfig, WkvConfig)
from ..config.lilenex import DenseMlpConfig
from ..parts.base import PartSpec
from .spec import ModelSpec, RunEntry

DECAY_LIMIT = 8.0       # a channel of the gated linear recurrence decays by exp(-DECAY_LIMIT * softplus(lam)) per token at most


def _names(prefix: str, *locals_: str):
    return {n: prefix + n for n in locals_}


def _rotation(rot: ScaledRotation, head_dim: int):
    if rot is None:
        return {}
    scaling = None
    if rot.factor != 1.0:
        scaling = {"rope_type": "llama3", "factor": rot.factor, "low_freq_factor": rot.low, "high_freq_factor": rot.high,
                   "original_max_position_embeddings": rot.original}
    return {"position": PartSpec("rope", {"head_dim": head_dim, "theta": rot.base, "scaling": scaling, "rotary_dim": rot.dims})}


def _attention(width: int, m: CappedAttentionConfig, p: str, **options) -> PartSpec:
    names = ["q", "k", "v", "o"] + (["q.b", "k.b", "v.b"] if options.get("bias") else []) + (["g"] if options.get("gate") else [])
    return PartSpec("window_attention",
                    {"hidden": width, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale,
                     "softcap": m.softcap, "qk_norm_eps": 0.0, "own_kv": True, **options},
                    _names(p, *names), _rotation(m.rot, m.dim))


def _linear_unit(width: int, m: LinearUnitConfig, p: str) -> PartSpec:
    return PartSpec("gated_lru", {"hidden": width, "width": m.width, "blocks": m.blocks, "taps": m.conv, "decay_limit": DECAY_LIMIT},
                    _names(p, "y", "y.b", "x", "x.b", "conv", "conv.b", "ra", "ra.b", "ri", "ri.b", "lam", "o"))


def _state_space(width: int, m: StateSpaceConfig, p: str, eps: float) -> PartSpec:
    return PartSpec("state_space", {"hidden": width, "heads": m.heads, "value_dim": m.vdim, "state": m.state, "groups": m.groups,
                                    "norm_groups": m.norm_groups, "taps": m.conv, "norm_eps": eps},
                    _names(p, "in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o"))


def _mixer(width: int, m, p: str, eps: float) -> PartSpec:
    if isinstance(m, NormedMeanConfig):
        return PartSpec("parallel", {"hidden": width, "combine": "normed_mean", "norm_eps": eps},
                        {"left.out": p + "left.out", "right.out": p + "right.out"},
                        {"left": _attention(width, m.left, p + "left.", chunk=m.left.size, bias=True, gate="head"),
                         "right": _linear_unit(width, m.right, p + "right.")})
    if isinstance(m, ScaledSumConfig):
        return PartSpec("parallel", {"hidden": width, "scales": {"left": m.left_scale, "right": m.right_scale}},
                        parts={"left": _attention(width, m.left, p + "left.", window=m.left.size),
                               "right": _state_space(width, m.right, p + "right.", eps)})
    wkv: WkvConfig = m
    return PartSpec("wkv", {"hidden": width, "heads": wkv.heads, "head_dim": wkv.dim, "norm_eps": eps},
                    _names(p, "mu.r", "mu.k", "mu.v", "mu.g", "mu.w", "r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o"))


def _feed_forward(width: int, m, p: str) -> PartSpec:
    if isinstance(m, DenseMlpConfig):
        return PartSpec("relu2_mlp", {"hidden": width, "inter": m.ff}, _names(p, "up", "down"))
    names = ["router", "router.b"] + [f"e{i}.{w}" for i in range(m.experts) for w in ("gate", "up", "down")]
    if m.shared_ff:
        names += ["shared.gate", "shared.up", "shared.down"]
    # the softmax over the chosen logits alone is the softmax over all of them, divided by the chosen ones' sum
    return PartSpec("routed_experts", {"hidden": width, "inter": m.ff, "experts": m.experts, "top": m.top, "shared_inter": m.shared_ff,
                                       "scale_input": False, "score": "softmax", "renormalise": True, "router_bias": True},
                    _names(p, *names))


def gepilix_spec(cfg: GepilixConfig, norm_init: str = "ones") -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("tanh_norm", {"width": W, "init": norm_init}, {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"})

    layers = []
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"norm1": norm(p + "norm1"), "mixer": _mixer(W, L.mixer, p + "mix.", eps)}
        tensors = {"scale1": p + "ls1"}
        if L.mlp is not None:
            parts.update({"norm2": norm(p + "norm2"), "ffn": _feed_forward(W, L.mlp, p + "mlp.")})
            tensors["scale2"] = p + "ls2"
        layers.append(PartSpec("pre_norm", {"layer_scale": W}, tensors, parts))
    return ModelSpec(architecture="Gepilix", hidden_size=W, vocab_size=cfg.vocab, embedding="embed", layers=layers,
                     run_order=[RunEntry(layer=i, cache=i) for i in range(len(layers))], final_norm=norm("final.norm"), lm_head="head",
                     initializer_range=cfg.initializer_range, eos_token_ids=cfg.eos_token_ids)
