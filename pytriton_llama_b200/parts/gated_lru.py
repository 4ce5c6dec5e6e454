"""A gated linear recurrence per channel behind a short convolution, beside a gelu branch.

With h the mixer's input:  y = gelu_tanh(W_y h + b_y);  u = conv(W_x h + b_x), causal and per channel with a bias of its
own.  u is cut into ``blocks`` equal parts; per part b two square matrices give  r = sigmoid(R_b u_b + b_r)  and
i = sigmoid(I_b u_b + b_i).  With log a = -``decay_limit`` * r * softplus(lam), per channel

    S <- a S + sqrt(1 - a^2) * i * u        output W_o (S * y)

S and the last ``taps - 1`` inputs of the convolution are per-request state (float32, zero before position 0).  The
projections, the convolution's result and the blocks' products take the compute type (the products give float32); gates,
decays and the state are float32, with 1 - a^2 worked out from log a.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import CacheNeed, Part, PartSpec, Runtime, TensorSpec, register_part


@register_part("mixer", "gated_lru")
class GatedLRU(Part):
    """params: ``hidden``, ``width``, ``blocks``, ``taps``, ``decay_limit``.  Tensors: ``y``, ``x`` [width, hidden], ``y.b``,
    ``x.b`` [width], ``conv`` [width, taps], ``conv.b`` [width], ``ra``, ``ri`` [blocks, width/blocks, width/blocks],
    ``ra.b``, ``ri.b`` [blocks, width/blocks], ``lam`` [width], ``o`` [hidden, width]."""

    def __init__(self, spec: PartSpec, runtime: Runtime):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.width, self.blocks, self.taps = int(p["hidden"]), int(p["width"]), int(p["blocks"]), int(p["taps"])
        self.decay_limit = float(p["decay_limit"])
        if self.width % self.blocks:
            raise ValueError(f"{self.width} channels in {self.blocks} blocks")
        self.inner_width = self.width
        self.output_bias = None
        self.w_o = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        n, B, W = self.width, self.blocks, self.hidden
        s = n // B
        bias, gate = TensorSpec((n,), "zeros_jitter"), TensorSpec((B, s, s))
        return {"y": TensorSpec((n, W)), "y.b": bias, "x": TensorSpec((n, W)), "x.b": bias,
                "conv": TensorSpec((n, self.taps), "uniform", lo=-0.5, hi=0.5), "conv.b": bias, "ra": gate, "ri": gate,
                "ra.b": TensorSpec((B, s), "zeros_jitter"), "ri.b": TensorSpec((B, s), "zeros_jitter"),
                "lam": TensorSpec((n,), "uniform", lo=-6.0, hi=-1.0), "o": TensorSpec((W, n))}

    def load(self, t) -> None:
        self.w_yx = self._to_compute(torch.cat([t["y"], t["x"]], dim=0))
        self.y_bias, self.x_bias = self._to_f32(t["y.b"]), self._to_f32(t["x.b"])
        self.conv_w, self.conv_b = self._to_f32(t["conv"]), self._to_f32(t["conv.b"])
        self.w_gates = self._to_compute(torch.cat([t["ra"], t["ri"]], dim=1))               # per block its r rows, then its i rows
        self.gate_bias = self._to_f32(torch.stack([t["ra.b"].reshape(-1), t["ri.b"].reshape(-1)]))
        # decay_limit * softplus(lam), worked out once in 64 bits
        lam = t["lam"].to(torch.float64)
        self.rate = self._to_f32(self.decay_limit * (lam.clamp(min=0) + torch.log1p(torch.exp(-lam.abs()))))
        self.w_o = self._to_compute(t["o"])

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kind="none", states=(("conv", (max(self.taps - 1, 1), self.width)), ("S", (self.width,))))

    def write_inner(self, x, ctx, cache, out, column: int, scale: float) -> None:
        ops = self.rt.ops
        yx = ops.linear(x, self.w_yx)                                       # [T, y branch | x branch], before their biases
        u = ops.causal_conv(yx, self.width, self.width, self.conv_w, self.conv_b, cache.states["conv"], ctx, silu=False, in_bias=self.x_bias)
        ops.gated_lru(u, self.w_gates, self.gate_bias, self.rate, yx, self.y_bias, cache.states["S"], ctx, out, column, scale)

    def forward(self, x, ctx, cache):
        out = self.rt.ops.empty((x.shape[0], self.inner_width), self.rt.dtype)
        self.write_inner(x, ctx, cache, out, 0, 1.0)
        return self.rt.ops.linear(out, self.w_o)
