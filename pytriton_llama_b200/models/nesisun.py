"""The Nesisun decoder (architecture name "Nesisun") as a ``ModelSpec``.

The stream starts as embed[token] * scale plus a row of ``bigram`` chosen by the token before and the token.  A layer
(tensors ``l<i>.*``) is a ``shared_norm`` block: ``norm1``, and on its output a windowed softmax attention that keeps the
first positions, with biases, a learned sink and values that are its keys before their rotation, beside a gated gelu
feed-forward, routed clamped experts, or nothing.  A layer with ``weights_of`` is one more run of the block of the layer
it names, with a cache entry of its own.  The logits come from ``final.norm`` and the table ``head``.
"""
from __future__ import annotations

from ..config.lilenex import DenseMlpConfig
from ..config.nesisun import ClampedMoeConfig, KeyValueAttentionConfig, NesisunConfig
from ..parts.base import PartSpec
from .spec import ModelSpec, RunEntry

EXPERT_ALPHA, EXPERT_SHIFT = 1.702, 1.0     # an expert's inner value: g sigmoid(EXPERT_ALPHA g) (u + EXPERT_SHIFT)


def _names(prefix: str, *locals_: str):
    return {n: prefix + n for n in locals_}


def _attention(width: int, m: KeyValueAttentionConfig, p: str) -> PartSpec:
    parts = {}
    if m.rot is not None:
        parts["position"] = PartSpec("rotary_pairs", {"head_dim": m.dim, "dims": m.rot.dims, "base": m.rot.base, "scaling": None})
    return PartSpec("window_attention",
                    {"hidden": width, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.dim, "scale": m.scale,
                     "window": m.window, "keep_first": m.keep_first, "qk_norm_eps": 0.0, "own_kv": True, "bias": True,
                     "values_are_keys": True, "sink": "learned"},
                    _names(p, "q", "q.b", "k", "k.b", "sink", "o"), parts)


def _feed_forward(width: int, mlp, p: str) -> PartSpec:
    if isinstance(mlp, DenseMlpConfig):
        return PartSpec("gated_mlp", {"hidden": width, "inter": mlp.ff, "act": "gelu_tanh"}, _names(p, "gate", "up", "down"))
    m: ClampedMoeConfig = mlp
    names = ["router", "correction"] + [f"e{i}.{w}" for i in range(m.experts) for w in ("gate", "up", "down")]
    return PartSpec("routed_experts",
                    {"hidden": width, "inter": m.ff, "experts": m.experts, "identity": m.identity, "top": m.top, "scale_input": False,
                     "score": "softmax", "renormalise": True, "correction": True, "weight_scale": m.scale,
                     "clamped": (m.limit, EXPERT_ALPHA, EXPERT_SHIFT)}, _names(p, *names))


def nesisun_spec(cfg: NesisunConfig, norm_init: str = "ones") -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps

    def norm(weight: str) -> PartSpec:
        return PartSpec("rmsnorm", {"width": W, "eps": eps, "init": norm_init}, {"weight": weight})

    layers, block_of = [], {}
    for i, L in enumerate(cfg.layers):
        if L.weights_of is not None:
            continue
        p = f"l{i}."
        parts = {"norm1": norm(p + "norm1"), "mixer": _attention(W, L.mixer, p + "mix.")}
        if L.mlp is not None:
            parts["ffn"] = _feed_forward(W, L.mlp, p + "mlp.")
        block_of[i] = len(layers)
        layers.append(PartSpec("shared_norm", parts=parts))
    run_order = [RunEntry(layer=block_of[i if L.weights_of is None else L.weights_of], cache=i) for i, L in enumerate(cfg.layers)]
    embedding = None
    if cfg.bigram is not None:
        b = cfg.bigram
        embedding = PartSpec("bigram", {"hidden": W, "buckets": b.buckets, "mul_prev": b.mul_prev, "mul_cur": b.mul_cur}, {"pairs": "bigram"})
    return ModelSpec(architecture="Nesisun", hidden_size=W, vocab_size=cfg.vocab, embedding="embed", layers=layers, run_order=run_order,
                     final_norm=norm("final.norm"), lm_head="head", embedding_scale=cfg.embedding_scale, embedding_part=embedding,
                     initializer_range=cfg.initializer_range, eos_token_ids=cfg.eos_token_ids)
