"""How norm, mixer, norm and feed-forward sit around the residual stream.

lite_llama/models/llama.py:136-162: pre-norm block.  The stream is carried as two tensors: the
output of the last sub-layer (not yet added) and the float32 residual; each norm first adds the
former into the latter.  The block returns its feed-forward output un-added, so the next block's
first norm (or the model's final norm, :219) folds it in.  With a scale per sub-layer the block completes the
stream itself and hands the next norm's result on.  ``SharedNormBlock`` is the arrangement with one norm whose
output both sub-layers read.
"""
from __future__ import annotations

import os

import torch

from .base import (NormedInput, Part, PartSpec, Runtime, ScaledOutput, Tail, TensorSpec, build_part, register_part,
                   side_stream)


@register_part("block", "pre_norm")
class PreNormBlock(Part):
    """Nested parts: ``norm1``, ``mixer``; ``norm2`` and ``ffn`` (both or neither: a layer without a
    feed-forward); optionally ``token_input``, which comes last.

    params: optional ``layer_scale`` (the stream's width): each sub-layer's result is multiplied entry by entry by a
    vector before it is added, tensors ``scale1`` (mixer) and ``scale2`` (feed-forward).  The norms are then of a kind
    with ``tail_add`` and the like (``tanh_norm``)."""

    def __init__(self, spec: PartSpec, runtime: Runtime):
        super().__init__(spec, runtime)
        self.norm1 = build_part("norm", spec.parts["norm1"], runtime)
        self.mixer = build_part("mixer", spec.parts["mixer"], runtime)
        if ("norm2" in spec.parts) != ("ffn" in spec.parts):
            raise ValueError("a block has both norm2 and ffn, or neither")
        self.norm2 = build_part("norm", spec.parts["norm2"], runtime) if "norm2" in spec.parts else None
        self.ffn = build_part("ffn", spec.parts["ffn"], runtime) if "ffn" in spec.parts else None
        self.token_input = build_part("token_input", spec.parts["token_input"], runtime) if "token_input" in spec.parts else None
        last = self.ffn if self.ffn is not None else self.mixer
        if self.token_input is None and getattr(last, "output_bias_spec", False):
            raise ValueError("a block whose last projection leaves its bias out needs a token_input that adds it")
        self.scale_width = int(spec.params.get("layer_scale") or 0)
        self.scale1 = self.scale2 = None
        if self.scale_width and (self.token_input is not None or not hasattr(self.norm1, "tail_add")):
            raise ValueError("a layer scale goes with norms that add a scaled output, and with no token_input")

    takes_next_norm = True   # forward() accepts the norm part that follows the block

    def children(self):
        parts = {"norm1": self.norm1, "mixer": self.mixer, "norm2": self.norm2, "ffn": self.ffn, "token_input": self.token_input}
        return {k: v for k, v in parts.items() if v is not None}

    def tensor_specs(self):
        if not self.scale_width:
            return {}
        # drawn at random: around one, so that a scale that is left out or swapped shows
        names = ["scale1"] + (["scale2"] if self.ffn is not None else [])
        return {n: TensorSpec((self.scale_width,), "uniform", lo=0.5, hi=1.5) for n in names}

    def load(self, tensors) -> None:
        if self.scale_width:
            self.scale1 = self._to_f32(tensors["scale1"])
            self.scale2 = self._to_f32(tensors["scale2"]) if self.ffn is not None else None

    def cache_need(self):
        return self.mixer.cache_need()

    def _forward_scaled(self, x, residual, ctx, cache, next_norm):
        y, residual = self.norm1.forward(x, residual)
        y = self._run_scaled(self.mixer, y, residual, self.scale1, self.norm2 if self.ffn is not None else next_norm, ctx, cache)
        if self.ffn is not None:
            y, _ = self.norm2.forward(y, residual)
            y = self._run_scaled(self.ffn, y, residual, self.scale2, next_norm)
        return y, residual

    @staticmethod
    def _run_scaled(part, y, residual, scale, following, *args):
        """``part``'s output times ``scale`` into the stream, and the following norm's result; without a norm that
        follows (the model's last layer) the output and its scale, for the final norm to add to the rows it takes."""
        if not hasattr(following, "tail_add"):
            return ScaledOutput(part.forward(y, *args), scale)
        tail = Tail(following, residual, scale)
        if getattr(part, "takes_tail", False):
            return NormedInput(part.forward(y, *args, tail=tail), following.weight)
        return NormedInput(tail.output(part.forward(y, *args)), following.weight)

    def forward(self, x, residual, ctx, cache, next_norm=None):
        """``x`` may be None: the previous sub-layer then already added its output into ``residual``.
        Mixers and feed-forwards that set ``fuses_residual`` get the residual and may do the same.
        Those that also set ``emits_normed`` are told which norm reads the residual next
        (``next_norm``: the norm part that follows this block, if any) and may return that norm's
        prepared input; a sub-layer reads such an input only if it sets ``accepts_normed``."""
        if self.scale_width:
            return self._forward_scaled(x, residual, ctx, cache, next_norm)
        y, residual = self.norm1.forward(x, residual)
        a = self._run(self.mixer, y, residual, self.norm2, ctx, cache)
        bias = getattr(self.mixer, "output_bias", None)
        if self.ffn is not None:
            y, residual = self.norm2.forward(a, residual, bias=bias) if bias is not None else self.norm2.forward(a, residual)
            a = self._run(self.ffn, y, residual, None if self.token_input is not None else next_norm)
            bias = getattr(self.ffn, "output_bias", None)
        if self.token_input is None:
            return a, residual
        self.token_input.apply(residual, a, bias, ctx)      # adds a (+ bias) and its own term into the stream
        return None, residual

    @staticmethod
    def _run(part, y, residual, following_norm, *args):
        if hasattr(y, "materialise") and not getattr(part, "accepts_normed", False):
            y = y.materialise()
        kw = {}
        if getattr(part, "fuses_residual", False):
            kw["residual"] = residual
            if getattr(part, "emits_normed", False) and getattr(following_norm, "deferrable", False):
                kw["next_norm"] = (following_norm.weight, following_norm.eps)
        return part.forward(y, *args, **kw)


@register_part("block", "shared_norm")
class SharedNormBlock(Part):
    """One norm, both sub-layers on its output, both outputs added into the stream: with h = norm1(x),
    x <- x + (mixer(h) + ffn(h)).

    Nested parts: ``norm1``, ``mixer``, optionally ``ffn``.  The mixer has ``write_inner`` (its heads' outputs into columns
    of a buffer), ``inner_width`` and ``w_o``.  A feed-forward with ``write_inner`` as well (a gated MLP) shares one output
    product with the mixer: the inputs of both last projections lie side by side in one buffer, their weights side by side
    in one matrix, and the product's sum over them is the layer's addition to the stream.  One with ``begin`` and
    ``finish`` (routed experts) adds the mixer's output, its own and the next norm up in its last kernel.

    On a CUDA device the two sub-layers run side by side in time: the feed-forward on a second stream that starts when
    the normed input is ready and is joined before the sum.  ``PTL_PARALLEL_STREAMS=0`` runs them one after the other."""

    takes_next_norm = True

    def __init__(self, spec: PartSpec, runtime: Runtime):
        super().__init__(spec, runtime)
        self.norm1 = build_part("norm", spec.parts["norm1"], runtime)
        self.mixer = build_part("mixer", spec.parts["mixer"], runtime)
        self.ffn = build_part("ffn", spec.parts["ffn"], runtime) if "ffn" in spec.parts else None
        self.routed = self.ffn is not None and hasattr(self.ffn, "begin")
        if self.ffn is not None and not self.routed and not hasattr(self.ffn, "write_inner"):
            raise ValueError(f"a feed-forward of kind {spec.parts['ffn'].kind!r} cannot stand beside a mixer")
        if self.routed:
            self.norm1.deferrable = False      # experts and router read the normed input itself, not a product's preparation of it
        self.w_out = None
        self.mixer_column, self.padded = 0, False

    def children(self):
        parts = {"norm1": self.norm1, "mixer": self.mixer, "ffn": self.ffn}
        return {k: v for k, v in parts.items() if v is not None}

    def cache_need(self):
        return self.mixer.cache_need()

    def after_load(self) -> None:
        self.w_out = self.mixer.w_o
        if self.ffn is None or self.routed:
            return
        # the feed-forward's columns first; both parts start at multiples of 8 columns (with zeros between, in the buffer
        # and in the weight), so that the kernels that write them keep their alignment
        pad = lambda w: torch.nn.functional.pad(w, (0, -w.shape[1] % 8))
        f, m = pad(self.ffn.w_down), pad(self.mixer.w_o)
        self.padded = f.shape[1] != self.ffn.inner_width or m.shape[1] != self.mixer.inner_width
        self.mixer_column = f.shape[1]
        self.w_out = torch.cat([f, m], dim=1).contiguous()
        self.ffn.w_down = self.mixer.w_o = None          # the joint weight is the one that is used

    def forward(self, x, residual, ctx, cache, next_norm=None):
        ops = self.rt.ops
        y, residual = self.norm1.forward(x, residual)
        prepared = y
        if hasattr(y, "materialise") and (isinstance(y, NormedInput) or self.routed):
            y = prepared = y.materialise()
        T, dtype = prepared.shape[0], self.rt.dtype
        width = self.mixer.inner_width
        if self.ffn is None:
            out = ops.empty((T, width), dtype)
            self.mixer.write_inner(y, ctx, cache, out, 0, 1.0)
            return self._add(out, self.w_out, residual, next_norm), residual
        fork = self.rt.device.type == "cuda" and os.environ.get("PTL_PARALLEL_STREAMS", "1") != "0"
        if self.routed:
            begun = self._beside(fork, lambda: self.ffn.begin(y))
            out = ops.empty((T, width), dtype)
            self.mixer.write_inner(y, ctx, cache, out, 0, 1.0)
            add = ops.linear_add(out, self.w_out, residual)            # None: already added
            self._join(fork)
            following = (next_norm.weight, next_norm.eps) if self._plain_rms(next_norm) else None
            normed = self.ffn.finish(begun, residual, add=add, next_norm=following)
            return (NormedInput(normed, next_norm.weight) if normed is not None else None), residual
        out = ops.empty((T, self.w_out.shape[1]), dtype)
        if self.padded:
            out.zero_()
        self._beside(fork, lambda: self.ffn.write_inner(y, out, 0))
        self.mixer.write_inner(y, ctx, cache, out, self.mixer_column, 1.0)
        self._join(fork)
        return self._add(out, self.w_out, residual, next_norm), residual

    def _add(self, out, weight, residual, next_norm):
        ops = self.rt.ops
        if self._plain_rms(next_norm) and getattr(next_norm, "deferrable", False) and getattr(ops, "fuses_next_norm", False):
            return ops.linear_add(out, weight, residual, next_norm=(next_norm.weight, next_norm.eps))
        return ops.linear_add(out, weight, residual)

    @staticmethod
    def _plain_rms(norm) -> bool:
        return norm is not None and hasattr(norm, "deferrable")

    def _beside(self, fork: bool, run):
        if not fork:
            return run()
        stream = side_stream(self.rt)
        ready = torch.cuda.Event()
        ready.record(torch.cuda.current_stream(self.rt.device))
        stream.wait_event(ready)
        with torch.cuda.stream(stream):
            return run()

    def _join(self, fork: bool) -> None:
        if fork:
            torch.cuda.current_stream(self.rt.device).wait_stream(side_stream(self.rt))
