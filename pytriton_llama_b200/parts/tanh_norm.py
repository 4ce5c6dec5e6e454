"""A norm without statistics: y = tanh(alpha * s) * weight + bias, entry by entry, s being the residual sum.

The sub-layer's output, times a vector where the layer has one, is added to the float32 residual first.  alpha is
one number.  Sum, tanh and y are float32 in every compute type; y is rounded once.  Because no entry waits for another,
the product (or sum) that makes a sub-layer's output can add it and work the norm out in its own last step: the
``tail_*`` methods.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Part, PartSpec, Runtime, ScaledOutput, TensorSpec, register_part


@register_part("norm", "tanh_norm")
class TanhNorm(Part):
    """params: ``width``; optional ``init`` (how random-weights mode draws the weight).
    Tensors: ``weight``, ``bias`` [width], ``alpha`` []."""

    def __init__(self, spec: PartSpec, runtime: Runtime):
        super().__init__(spec, runtime)
        self.width = int(spec.params["width"])
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None
        self.alpha = 1.0

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {"weight": TensorSpec((self.width,), init=self.spec.params.get("init", "ones")),
                "bias": TensorSpec((self.width,), init="zeros_jitter"), "alpha": TensorSpec((), "uniform", lo=0.3, hi=0.8)}

    def load(self, tensors) -> None:
        self.weight, self.bias = self._to_f32(tensors["weight"]), self._to_f32(tensors["bias"])
        self.alpha = float(tensors["alpha"])

    @property
    def params(self):
        """(alpha, weight, bias), as the operators take them."""
        return self.alpha, self.weight, self.bias

    def forward(self, x, residual, rows=None):
        """``x``: an output to add (a ``ScaledOutput``: times its scale), None, or this norm's result made ahead of time."""
        scale = None
        if hasattr(x, "materialise"):
            if x.weight is self.weight and rows is None:
                return x.materialise(), residual
            x = None
        elif isinstance(x, ScaledOutput):
            x, scale = x.x, x.scale
        return self.rt.ops.add_tanh_norm(x, residual, self.params, scale=scale, rows=rows, dtype=self.rt.dtype)

    def tail_add(self, out, residual, scale):
        return self.rt.ops.add_tanh_norm(out, residual, self.params, scale=scale, dtype=self.rt.dtype)[0]

    def tail_product(self, inner, w, residual, scale):
        return self.rt.ops.linear_add_tanh_norm(inner, w, residual, self.params, scale)

    def tail_members(self, outs, eps, residual, scale):
        return self.rt.ops.add_tanh_norm(None, residual, self.params, scale=scale, dtype=self.rt.dtype, members=(outs, eps))[0]

    def tail_experts(self, rows, shared, residual, scale):
        return self.rt.ops.combine_experts_tanh_norm(rows, shared, residual, self.params, scale)
