"""RWKV-style time mixing: a matrix state per head that decays per key channel, and a bonus for the current token.

With h the mixer's input and h' the token's before it (zeros at position 0), each of r, k, v, g and w reads its own mix
m_s = h + (h' - h) * mu_s.  r, k, v = W m (heads x head_dim each);  the decay of head and key channel is
w = exp(-exp(W_w2 tanh(W_w1 m_w) + w0)).  Per head

    o = (S + diag(u) k v^T)^T r,  then  S <- diag(w) S + k v^T

so a token sees itself with the weight u and its predecessors through S.  o is divided by its root mean square per
head, multiplied by ``norm`` (one weight per channel of every head) and silu(W_g m_g), and projected by W_o.
S [heads, head_dim, head_dim] and the last token's h are per-request state (float32, zero before position 0).  The
projections run in the compute type (W_w1 gives float32); tanh, the second decay product, the exponentials, the
state and the read-out are float32.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import CacheNeed, Part, PartSpec, Runtime, TensorSpec, register_part

MIXES = ("r", "k", "v", "g", "w")


@register_part("mixer", "wkv")
class WKV(Part):
    """params: ``hidden``, ``heads``, ``head_dim``, ``norm_eps``; optional ``decay_rank`` (the inner size of the decay
    projection when weights are drawn at random; a checkpoint's own size is taken as it is).  Tensors: ``mu.r`` .. ``mu.w`` [hidden],
    ``r``, ``k``, ``v``, ``g`` [heads*head_dim, hidden], ``w1`` [rank, hidden], ``w2`` [heads*head_dim, rank], ``w0``, ``norm``
    [heads*head_dim], ``u`` [heads, head_dim], ``o`` [hidden, heads*head_dim]."""

    def __init__(self, spec: PartSpec, runtime: Runtime):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.heads, self.d = int(p["hidden"]), int(p["heads"]), int(p["head_dim"])
        self.norm_eps = float(p["norm_eps"])
        self.rank = int(p.get("decay_rank") or 16)

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        n, W = self.heads * self.d, self.hidden
        out = {f"mu.{s}": TensorSpec((W,), "uniform", lo=0.0, hi=1.0) for s in MIXES}
        out.update({s: TensorSpec((n, W)) for s in "rkvg"})
        out.update({"w1": TensorSpec((-self.rank, W)), "w2": TensorSpec((n, -self.rank)), "w0": TensorSpec((n,), "uniform", lo=-5.0, hi=0.5),
                    "u": TensorSpec((self.heads, self.d), "uniform", lo=-1.0, hi=1.0), "norm": TensorSpec((n,), "ones"),
                    "o": TensorSpec((W, n))})
        return out

    def load(self, t) -> None:
        if t["w1"].shape[0] != t["w2"].shape[1]:
            raise ValueError(f"the decay projections do not fit: w1 is {list(t['w1'].shape)}, w2 is {list(t['w2'].shape)}")
        self.mu = self._to_f32(torch.stack([t[f"mu.{s}"] for s in MIXES]))
        self.w_rkvg = self._to_compute(torch.stack([t[s] for s in "rkvg"]))          # [4, n, hidden]: one matrix per mix
        self.w_w1, self.w_w2 = self._to_compute(t["w1"]), self._to_f32(t["w2"])     # the second, small product runs in float32
        self.w_bias, self.u, self.norm_w = self._to_f32(t["w0"]), self._to_f32(t["u"].reshape(-1)), self._to_f32(t["norm"])
        self.w_o = self._to_compute(t["o"])

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kind="none", states=(("last", (self.hidden,)), ("S", (self.heads, self.d, self.d))))

    takes_tail = True

    def forward(self, x, ctx, cache, tail=None):
        ops = self.rt.ops
        H, d = self.heads, self.d
        mixes = ops.token_shift(x, self.mu, cache.states["last"], ctx)               # [5, T, hidden]
        rkvg = ops.linear_each(mixes[:4], self.w_rkvg)                                # [4, T, n]
        decay = ops.lowrank_tanh_linear(ops.linear(mixes[4], self.w_w1, out_dtype=torch.float32), 0, self.w_w2, decay_bias=self.w_bias)
        o = ops.wkv_scan(rkvg, decay, self.u, cache.states["S"], ctx, H, d)
        out = ops.empty((x.shape[0], H * d), self.rt.dtype)
        ops.gated_head_norm(o, self.norm_w, self.norm_eps, rkvg[3], 0, H, d, out, 0, 1.0, weight_per_head=True)
        return ops.linear(out, self.w_o) if tail is None else tail.product(out, self.w_o)
