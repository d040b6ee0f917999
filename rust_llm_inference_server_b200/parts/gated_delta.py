"""The gated delta rule: a linear recurrence over a float32 state per request whose update corrects the
state towards the token's value along its key, behind short causal convolutions of q, k and v."""

from __future__ import annotations

import numpy as np
import torch

from .. import ops
from ..ops.profile import span
from .base import Mixer, StateSpec, register_mixer


class GatedDeltaRule(Mixer):
    """q | k | v | gate | beta logits | decay logits come from one stacked projection.  One kernel applies the
    convolutions (their tail of taps - 1 inputs is part of the request's state), silu, the unit norms of q and k,
    the sigmoid of beta and the decay g = exp(-exp(a_log) softplus(. + dt_bias)); a second one walks the step's
    tokens per (request, head): S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q.  The heads' outputs are
    normed per head, gated by silu(W_g h) (or sigmoid) and projected.  Everything between the two projections is float32.

    Decay logits or gate logits through a low rank (`decay_down`, `gate_down`): the first projection's rows begin with the
    low-rank vectors of both, and one more product over them, block-diagonal, makes the logits of both."""

    graph_safe = True

    def __init__(self, spec, dtype, device):
        self.spec = spec
        self.dtype = dtype
        if spec.n_heads % spec.n_qk_heads:
            raise ValueError(f"{spec.n_heads} heads are not a multiple of {spec.n_qk_heads} query/key heads")
        if spec.conv < 1:
            raise ValueError(f"a convolution has at least one tap, got {spec.conv}")
        if spec.decay_down is not None and not spec.channel_decay:
            raise ValueError("decay logits through a low rank go with a decay a channel")
        if spec.gate_act not in ops.GATE_ACTIVATIONS:
            raise ValueError(f"unknown gate activation {spec.gate_act!r}; known: {sorted(ops.GATE_ACTIVATIONS)}")
        self.eps = float(np.float32(spec.eps))
        self.qk, self.hv = spec.n_qk_heads * spec.dim, spec.n_heads * spec.v_dim
        self.decays = spec.n_heads * (spec.dim if spec.channel_decay else 1)
        self.channels = 2 * self.qk + self.hv
        self.state_floats = ops.conv_recurrence_state_floats(spec.n_heads, spec.n_qk_heads, spec.dim, spec.v_dim, spec.conv)

    def tensors(self) -> dict:
        s = self.spec
        out = {s.q_proj: (self.qk, s.hidden), s.k_proj: (self.qk, s.hidden), s.v_proj: (self.hv, s.hidden),
               s.q_conv: (self.qk, s.conv), s.k_conv: (self.qk, s.conv), s.v_conv: (self.hv, s.conv),
               s.beta_proj: (s.n_heads, s.hidden), s.a_log: (s.n_heads,), s.dt_bias: (self.decays,),
               s.out_norm: (s.v_dim,), s.o_proj: (s.hidden, self.hv)}
        for proj, down, rows in ((s.decay_proj, s.decay_down, self.decays), (s.gate_proj, s.gate_down, self.hv)):
            out[proj] = (rows, s.hidden if down is None else None)
            if down is not None:
                out[down] = (None, s.hidden)
        return out

    def load(self, src) -> None:
        s = self.spec
        # the projection's rows: [low-rank vectors, padded to whole 16-byte vectors | q | k | v | gate | beta | decay | pad]
        low, ups = [], []
        for proj, down in ((s.decay_proj, s.decay_down), (s.gate_proj, s.gate_down)):
            if down is not None:
                d, u = src.get(down), src.get(proj)
                if d.shape[0] != u.shape[1]:
                    raise ValueError(f"{down} has {d.shape[0]} rows and {proj} {u.shape[1]} columns")
                low.append(d)
                ups.append(u)
        stack = list(low)
        rank = sum(d.shape[0] for d in low)
        if low and rank % 8:
            stack.append(low[0].new_zeros((-rank % 8, s.hidden)))
        self.low_cols = rank + (-rank % 8)
        self.w_up = None
        if low:
            self.w_up = torch.zeros((sum(u.shape[0] for u in ups), self.low_cols), dtype=low[0].dtype, device=low[0].device)
            r = c = 0
            for u in ups:
                self.w_up[r:r + u.shape[0], c:c + u.shape[1]] = u
                r, c = r + u.shape[0], c + u.shape[1]
        self.qkv_off = at = self.low_cols
        stack += [src.get(s.q_proj), src.get(s.k_proj), src.get(s.v_proj)]
        at += self.channels
        # where the logits lie: (in the product over the low-rank vectors, column)
        self.decay_at = self.gate_at = None
        up_at = 0
        if s.decay_down is not None:
            self.decay_at, up_at = (True, up_at), up_at + self.decays
        if s.gate_down is not None:
            self.gate_at = (True, up_at)
        else:
            self.gate_at = (False, at)
            stack.append(src.get(s.gate_proj))
            at += self.hv
        self.b_off = at
        stack.append(src.get(s.beta_proj))
        at += s.n_heads
        if s.decay_down is None:
            self.decay_at = (False, at)
            stack.append(src.get(s.decay_proj))
            at += self.decays
        if at % 8:                        # rows of the stacked projection stay 16-byte multiples
            stack.append(stack[-1].new_zeros((-at % 8, s.hidden)))
        self.w_in = torch.cat(stack, dim=0).contiguous()
        self.conv_w = torch.cat([src.get(s.q_conv, "vector"), src.get(s.k_conv, "vector"),
                                 src.get(s.v_conv, "vector")], dim=0).contiguous()
        self.a_log = src.get(s.a_log, "vector").contiguous()
        self.dt_bias = src.get(s.dt_bias, "vector").contiguous()
        self.out_norm = src.get(s.out_norm, "vector").contiguous()
        self.w_o = src.get(s.o_proj).contiguous()

    def state_spec(self):
        return StateSpec((self.state_floats,), torch.float32)

    def fuses_norms(self, step) -> bool:
        return ops.fuses_norms(step.n_tokens, self.dtype, self.spec.hidden, self.hv)

    def forward(self, x, step, cache, state, writes_cache=True, sink=None):
        s = self.spec
        T = x.shape[0]
        with span("q|k|v|gate|beta|decay proj"):
            proj = ops.linear(x, self.w_in)
        up = None
        if self.w_up is not None:
            with span("low-rank decay|gate proj"):
                up = ops.linear(proj[:, :self.low_cols], self.w_up)

        def logits(at, width):
            return (up if at[0] else proj)[:, at[1]:at[1] + width]

        o = step.buffer("gated_delta_o", (T, self.hv), torch.float32)
        args = (state, o, step, s.n_heads, s.n_qk_heads, s.dim, s.v_dim, s.conv, s.unit_eps, float(s.dim) ** -0.5)
        with span("conv + delta rule"):
            if s.channel_decay:
                ops.channel_delta(proj, self.qkv_off, self.b_off, logits(self.decay_at, self.decays), self.conv_w,
                                  self.a_log, self.dt_bias, *args)
            else:
                ops.gated_delta(proj, self.qkv_off, self.b_off, self.decay_at[1], self.conv_w, self.a_log, self.dt_bias, *args)
        y = step.buffer("gated_delta_y", (T, self.hv), self.dtype)
        with span("head norm * gate"):
            ops.head_norm_gate(o, self.out_norm, self.eps, y, s.n_heads, gate=logits(self.gate_at, self.hv),
                               activation=s.gate_act)
        with span("o proj"):
            return ops.linear(y, self.w_o, sink=sink)


register_mixer("gated_delta", GatedDeltaRule)
