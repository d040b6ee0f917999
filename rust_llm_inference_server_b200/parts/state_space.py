"""The state-space mixer of Mamba-2: a linear recurrence over a float32 state per request with one decay a token and
head, behind a short causal convolution."""

from __future__ import annotations

import numpy as np
import torch

from .. import ops
from ..ops.profile import span
from .base import Mixer, StateSpec, register_mixer


class StateSpace(Mixer):
    """z | x | B | C | dt come from one projection.  One kernel applies the convolution (its tail of taps - 1 inputs is part
    of the request's state) with its bias and silu, and the step sizes' softplus; a second one walks the step's tokens per
    (request, head): S <- exp(-exp(a_log) dt) S + dt B x^T, y = S^T C + skip x.  y is gated by silu(z), normed in equal
    parts and projected.  Everything between the two projections is float32."""

    graph_safe = True

    def __init__(self, spec, dtype, device):
        self.spec = spec
        self.dtype = dtype
        if spec.n_heads % spec.n_groups:
            raise ValueError(f"{spec.n_heads} heads are not a multiple of {spec.n_groups} groups")
        if spec.conv < 1:
            raise ValueError(f"a convolution has at least one tap, got {spec.conv}")
        self.inner = spec.n_heads * spec.v_dim
        if self.inner % spec.norm_groups:
            raise ValueError(f"{spec.norm_groups} parts do not divide {self.inner} channels")
        self.eps = float(np.float32(spec.eps))
        self.channels = self.inner + 2 * spec.n_groups * spec.n_state
        self.dt_off = self.inner + self.channels
        self.rows = self.dt_off + spec.n_heads
        self.state_floats = ops.conv_recurrence_state_floats(spec.n_heads, spec.n_groups, spec.n_state, spec.v_dim, spec.conv)

    def tensors(self) -> dict:
        s = self.spec
        out = {s.in_proj: (self.rows, s.hidden), s.conv_weight: (self.channels, s.conv), s.a_log: (s.n_heads,),
               s.dt_bias: (s.n_heads,), s.skip: (s.n_heads,), s.out_norm: (self.inner,), s.o_proj: (s.hidden, self.inner)}
        if s.conv_bias is not None:
            out[s.conv_bias] = (self.channels,)
        return out

    def load(self, src) -> None:
        s = self.spec
        w = src.get(s.in_proj)
        pad = -w.shape[0] % 8             # rows of the projection's result stay 16-byte multiples
        if pad:
            w = torch.cat([w, w.new_zeros((pad, w.shape[1]))], dim=0)
        self.w_in = w.contiguous()
        self.conv_w = src.get(s.conv_weight, "vector").contiguous()
        self.conv_b = src.get(s.conv_bias, "vector").contiguous() if s.conv_bias is not None else None
        self.a_log, self.dt_bias, self.skip, self.out_norm = (src.get(n, "vector").contiguous()
                                                              for n in (s.a_log, s.dt_bias, s.skip, s.out_norm))
        self.w_o = src.get(s.o_proj).contiguous()

    def state_spec(self):
        return StateSpec((self.state_floats,), torch.float32)

    def fuses_norms(self, step) -> bool:
        return ops.fuses_norms(step.n_tokens, self.dtype, self.spec.hidden, self.inner)

    def forward(self, x, step, cache, state, writes_cache=True, sink=None):
        s = self.spec
        T = x.shape[0]
        with span("z|x|B|C|dt proj"):
            proj = ops.linear(x, self.w_in)
        o = step.buffer("state_space_o", (T, self.inner), torch.float32)
        with span("conv + state space"):
            ops.state_space(proj, self.inner, self.dt_off, self.conv_w, self.conv_b, self.a_log, self.dt_bias, self.skip, state,
                            o, step, s.n_heads, s.n_groups, s.n_state, s.v_dim, s.conv)
        y = step.buffer("state_space_y", (T, self.inner), self.dtype)
        with span("gate * norm"):
            ops.gate_group_norm(o, proj[:, :self.inner], self.out_norm, self.eps, y, s.norm_groups)
        with span("o proj"):
            return ops.linear(y, self.w_o, sink=sink)


register_mixer("state_space", StateSpace)
