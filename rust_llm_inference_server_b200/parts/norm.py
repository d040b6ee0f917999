"""Norms over the float32 residual stream: RMSNorm (crates/model/src/layers.rs:103-146) and the dynamic tanh."""

from __future__ import annotations

import numpy as np
import torch

from .. import ops
from ..ops.profile import span
from .base import Norm, register_norm


class RMSNorm(Norm):
    """y = x / sqrt(mean(x^2) + eps) * w.  eps is used as a float32 (layers.rs:115); the sum of
    squares and the scale are float32; the weight is held in float32 (an exact widening).  A spec
    with an `offset` (a weight stored around zero) has it added once at load time, in float32."""

    graph_safe = True    # launches depend on the step's device arrays and shapes only

    def __init__(self, spec, dtype, device):
        self.dim = spec.dim
        self.eps = float(np.float32(spec.eps))
        self.weight_name = spec.weight
        self.offset = float(getattr(spec, "offset", 0.0))
        self.dtype = dtype
        self.weight = None

    def tensors(self) -> dict:
        return {self.weight_name: (self.dim,)}

    def load(self, src) -> None:
        self.weight = src.get(self.weight_name, "vector")
        if self.offset:
            self.weight = (self.weight + self.offset).contiguous()

    def forward(self, resid, delta, step):
        out = step.buffer("norm_out", (resid.shape[0], self.dim), self.dtype)
        with span("residual add + rms norm"):
            return ops.rmsnorm(resid, self.weight, self.eps, out, delta)

    def forward_rows(self, resid, delta, step, rows):
        out = step.buffer("norm_rows_out", (rows.shape[0], self.dim), self.dtype)
        with span("residual add + rms norm"):
            return ops.rmsnorm(resid, self.weight, self.eps, out, delta, rows)

    def sink(self, resid, step):
        if not ops.fuses_norms(resid.shape[0], self.dtype, self.dim):
            return None
        return ops.ResidualSink(resid, self.weight, self.eps)


    def stream_norm(self):
        """This norm as `ops.stream_mix` takes it."""
        return ops.StreamNorm("rmsnorm", self.weight, eps=self.eps)


class LayerNorm(Norm):
    """y = (x - mean) / sqrt(variance + eps) * w, mean and variance of the row in float32, no bias.  (Its weight is `gain`:
    the arrangements that take an RMS norm apart themselves ask for a `weight`.)"""

    graph_safe = True

    def __init__(self, spec, dtype, device):
        self.dim = spec.dim
        self.eps = float(np.float32(spec.eps))
        self.weight_name = spec.weight
        self.dtype = dtype
        self.gain = None

    def tensors(self) -> dict:
        return {self.weight_name: (self.dim,)}

    def load(self, src) -> None:
        self.gain = src.get(self.weight_name, "vector").contiguous()

    def forward(self, resid, delta, step):
        out = step.buffer("norm_out", (resid.shape[0], self.dim), self.dtype)
        with span("residual add + layer norm"):
            return ops.layer_norm(resid, self.gain, self.eps, out, delta)

    def forward_rows(self, resid, delta, step, rows):
        out = step.buffer("norm_rows_out", (rows.shape[0], self.dim), self.dtype)
        with span("residual add + layer norm"):
            return ops.layer_norm(resid, self.gain, self.eps, out, delta, rows)

    def sink(self, resid, step):
        if not ops.fuses_norms(resid.shape[0], self.dtype, self.dim):
            return None
        return ops.ResidualSink(resid, self.gain, self.eps, centred=True)


class DynamicTanh(Norm):
    """y = tanh(alpha x) * w + b, in float32: no mean and no variance, so nothing of a row has to be known before its
    entries can be written (and a product's epilogue can apply it, see `ops.StreamsSink`)."""

    graph_safe = True

    def __init__(self, spec, dtype, device):
        self.dim = spec.dim
        self.spec = spec
        self.dtype = dtype

    def tensors(self) -> dict:
        s = self.spec
        return {s.weight: (s.dim,), s.bias: (s.dim,), s.alpha: ()}

    def load(self, src) -> None:
        s = self.spec
        self.weight = src.get(s.weight, "vector").contiguous()
        self.bias = src.get(s.bias, "vector").contiguous()
        self.alpha = float(src.get(s.alpha, "vector").reshape(-1)[0].item())

    def stream_norm(self):
        return ops.StreamNorm("dynamic_tanh", self.weight, self.bias, self.alpha)

    @staticmethod
    def _one(delta, step):
        """Two additions of a block whose sublayers stand side by side as one."""
        if not isinstance(delta, tuple):
            return delta
        out = step.buffer("delta_sum", tuple(delta[0].shape), delta[0].dtype)
        return ops.sum_norm(None, 0.0, [(d, None, 1.0) for d in delta], None, 0.0, out=out)

    def forward(self, resid, delta, step):
        delta = self._one(delta, step)
        out = step.buffer("norm_out", (resid.shape[0], self.dim), self.dtype)
        with span("residual add + dynamic tanh"):
            return ops.stream_mix(resid, 1, y=delta, x_out=resid.unsqueeze(1) if delta is not None else None,
                                  norm=self.stream_norm(), h=out)

    def forward_rows(self, resid, delta, step, rows):
        delta = self._one(delta, step)
        out = step.buffer("norm_rows_out", (rows.shape[0], self.dim), self.dtype)
        with span("residual add + dynamic tanh"):
            return ops.stream_mix(resid, 1, y=delta, norm=self.stream_norm(), h=out, rows=rows)


register_norm("rmsnorm", RMSNorm)
register_norm("layer_norm", LayerNorm)
register_norm("dynamic_tanh", DynamicTanh)
