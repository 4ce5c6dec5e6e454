"""State-space recurrence with one decay per head and token (the mixer of Mamba's second form).

With inner = heads * value_dim, N = ``state`` and ``groups`` pairs of B and C shared by heads / groups heads each:
W_in h = [z: inner | x: inner | B: groups*N | C: groups*N | dt: heads];  x, B and C pass one causal convolution per channel
(with bias) and silu;  dt <- softplus(dt + dt_bias).  Per head

    S <- exp(-exp(A_log) dt) S + dt * B x^T        y = S^T C + D x

The heads' y side by side, multiplied by silu(z), are divided by their root mean square in ``norm_groups`` equal parts,
multiplied by ``norm`` and projected by W_o.  S [heads, N, value_dim] and the last ``taps - 1`` inputs of the
convolution are per-request state (float32, zero before position 0).  The projections and the convolution run in the
compute type (dt's rows give float32); step sizes, decays, the state, the gate and the norm are float32.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import CacheNeed, Part, PartSpec, Runtime, TensorSpec, register_part


@register_part("mixer", "state_space")
class StateSpace(Part):
    """params: ``hidden``, ``heads``, ``value_dim``, ``state``, ``groups``, ``norm_groups``, ``taps``, ``norm_eps``.  Tensors: ``in``
    [2*inner + 2*groups*state + heads, hidden], ``conv`` [inner + 2*groups*state, taps], ``conv.b``, ``dt_bias``, ``A_log``, ``D``
    [heads], ``norm`` [inner], ``o`` [hidden, inner]."""

    def __init__(self, spec: PartSpec, runtime: Runtime):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.heads, self.dv, self.state = int(p["hidden"]), int(p["heads"]), int(p["value_dim"]), int(p["state"])
        self.groups, self.norm_groups, self.taps = int(p["groups"]), int(p["norm_groups"]), int(p["taps"])
        self.norm_eps = float(p["norm_eps"])
        self.inner = self.heads * self.dv
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError(f"{self.heads} heads in {self.groups} groups, {self.inner} channels in {self.norm_groups} parts")
        self.conv_channels = self.inner + 2 * self.groups * self.state
        self.inner_width = self.inner
        self.output_bias = None
        self.w_o = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        H, c, W = self.heads, self.conv_channels, self.hidden
        return {"in": TensorSpec((self.inner + c + H, W)), "conv": TensorSpec((c, self.taps), "uniform", lo=-0.5, hi=0.5),
                "conv.b": TensorSpec((c,), "zeros_jitter"), "dt_bias": TensorSpec((H,), "uniform", lo=-4.0, hi=-1.0),
                "A_log": TensorSpec((H,), "uniform", lo=0.0, hi=2.5), "D": TensorSpec((H,), "ones_jitter"),
                "norm": TensorSpec((self.inner,), "ones"), "o": TensorSpec((W, self.inner))}

    def load(self, t) -> None:
        n = self.inner + self.conv_channels
        self.w_zxbc, self.w_dt = self._to_compute(t["in"][:n]), self._to_compute(t["in"][n:])
        self.conv_w, self.conv_b = self._to_f32(t["conv"]), self._to_f32(t["conv.b"])
        self.dt_bias, self.D, self.norm_w = self._to_f32(t["dt_bias"]), self._to_f32(t["D"]), self._to_f32(t["norm"])
        self.rate = torch.exp(self._to_f32(t["A_log"]))
        self.w_o = self._to_compute(t["o"])

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kind="none", states=(("conv", (max(self.taps - 1, 1), self.conv_channels)), ("S", (self.heads, self.state, self.dv))))

    def write_inner(self, x, ctx, cache, out, column: int, scale: float) -> None:
        ops = self.rt.ops
        zxbc = ops.linear(x, self.w_zxbc)
        dt = ops.linear(x, self.w_dt, out_dtype=torch.float32)                 # [T, heads], before its bias
        xbc = ops.causal_conv(zxbc, self.inner, self.conv_channels, self.conv_w, self.conv_b, cache.states["conv"], ctx, silu=True)
        y = ops.state_space_scan(xbc, dt, self.dt_bias, self.rate, self.D, cache.states["S"], ctx, self.heads, self.groups, self.state, self.dv)
        ops.gated_group_norm(y, zxbc, 0, self.norm_w, self.norm_eps, self.norm_groups, out, column, scale)

    def forward(self, x, ctx, cache):
        out = self.rt.ops.empty((x.shape[0], self.inner_width), self.rt.dtype)
        self.write_inner(x, ctx, cache, out, 0, 1.0)
        return self.rt.ops.linear(out, self.w_o)
