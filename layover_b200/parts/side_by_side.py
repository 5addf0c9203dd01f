"""Mixers that run side by side on the same input."""

from __future__ import annotations

import torch

from ..weights.loader import TensorSpec
from .base import Part, build_part, register_mixer
from .norm import Deferred, DeferredMean


@register_mixer("side_by_side")
class SideBySide(Part):
    """Several mixers read the same input; the result is the mean of their outputs, each RMS-normed over the model
    width with a weight of its own first: (1 / n) sum_i w_i * m_i(h) * rsqrt(mean(m_i(h)^2) + eps).

    `combine` = "sum" instead: the result is the plain sum of the mixers' outputs (each may scale its own). The mixers
    must be `stackable`: their input matrices are stacked into one product, each works on its part of that product's
    rows and leaves its heads' outputs in its part of one row, and one product with their output matrices side by side
    is the sum.

    The mean is not computed here: the outputs are handed on as a `DeferredMean`, and the norm of the stream that
    follows norms each, averages, adds and norms the sum in one kernel (a block whose norm comes after the sum).
    Each mixer keeps a cache or state of its own: `cache_need()` is the tuple of theirs and the cache view that
    `forward` receives has one view per mixer in `parts`.

    params: hidden, combine ("mean" or "sum"), eps (for the mean), mixers (a list of (mixer PartSpec, tensor-name prefix below this part's prefix, name of
    its output-norm weight relative to this part's prefix, None with a sum))."""

    def __init__(self, params, prefix):
        super().__init__(params, prefix)
        self.combine = params.get("combine", "mean")
        if self.combine not in ("mean", "sum"):
            raise ValueError(f"side_by_side: combine is 'mean' or 'sum', got {self.combine!r}")
        self.require("hidden", "mixers", *(["eps"] if self.combine == "mean" else []))
        self.hidden, self.eps = int(params["hidden"]), float(params.get("eps", 0.0))
        self.mixers, self.weight_names = [], []
        for spec, sub_prefix, weight in params["mixers"]:
            self.mixers.append(build_part("mixer", spec, prefix + sub_prefix))
            if self.combine == "mean":
                self.weight_names.append(prefix + weight)
        if not self.mixers:
            raise ValueError("side_by_side: at least one mixer")
        if self.combine == "sum" and not all(getattr(m, "stackable", False) for m in self.mixers):
            raise ValueError("side_by_side: a sum needs mixers whose products can be stacked")
        self.weights = self.w_in = self.w_o = None

    def parts(self):
        return list(self.mixers)

    def tensor_specs(self):
        specs = [spec for mixer in self.mixers for spec in mixer.tensor_specs()]
        return specs + [TensorSpec(name, (self.hidden,), kind="vector", init="ones") for name in self.weight_names]

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        for mixer in self.mixers:
            mixer.bind(tensors, runtime)
        self.weights = [tensors[name] for name in self.weight_names]
        if self.combine == "sum":
            self._stack()

    def _stack(self):
        """One input matrix (the mixers' rows below one another) and one output matrix (theirs side by side, its rows
        padded to whole 16-byte pieces); `spans` says which part of either product's row is whose."""
        at_in = at_out = 0
        self.spans = []
        for m in self.mixers:
            self.spans.append((at_in, at_in + m.w_in.shape[0], at_out, at_out + m.w_o.shape[1]))
            at_in, at_out = self.spans[-1][1], self.spans[-1][3]
        self.w_in = torch.cat([m.w_in for m in self.mixers], dim=0).contiguous()
        self.out_width, self.out_room = at_out, -(-at_out // 8) * 8
        stacked = torch.zeros((self.hidden, self.out_room), dtype=self.w_in.dtype, device=self.w_in.device)
        for m, (_, _, begin, end) in zip(self.mixers, self.spans):
            stacked[:, begin:end] = m.w_o
            m.w_in = m.w_o = None
        self.w_o = stacked[:, :at_out]

    def cache_need(self):
        return tuple(mixer.cache_need() for mixer in self.mixers)

    def _forward_sum(self, h, batch, cache):
        proj = self.runtime.linear(h, self.w_in, out_dtype=torch.float32)
        mixed = torch.empty((h.shape[0], self.out_room), dtype=h.dtype, device=h.device)
        for mixer, view, (in0, in1, out0, out1) in zip(self.mixers, cache.parts, self.spans):
            mixer.mix(proj[:, in0:in1], batch, view, mixed[:, out0:out1])
        return self.runtime.linear(mixed[:, :self.out_width], self.w_o)

    def forward(self, h, batch, cache):
        if self.combine == "sum":
            return self._forward_sum(h, batch, cache)
        outputs = [mixer.forward(h, batch, view) for mixer, view in zip(self.mixers, cache.parts)]
        return DeferredMean(tuple(Deferred(o, w, self.eps) for o, w in zip(outputs, self.weights)), 1.0 / len(outputs))
