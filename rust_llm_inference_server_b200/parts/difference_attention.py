"""Causal grouped-query attention with two maps a head whose outputs are taken off each other, normed a head and gated."""

from __future__ import annotations

import numpy as np
import torch

from .. import ops
from ..ops.profile import span
from .base import KVCacheSpec, ProjectedMixer, build_position, register_mixer, stack_rows


class DifferenceAttention(ProjectedMixer):
    """One stacked product makes q | k | v | gate logits; one kernel turns q and k and stores keys and values in the paged
    cache (a key head's two vectors are one cached row); one kernel (two where a decoded context is cut into pieces) does both
    maps, their difference, its norm and the gate; then the output projection.  Rotation, scores, softmax, value sums,
    difference, norm and gate are float32.  lambda is one number a layer, worked out at load time."""

    graph_safe = True
    MAPS = 2

    def __init__(self, spec, dtype, device):
        self.spec = spec
        self.dtype = dtype
        if spec.n_heads % spec.n_kv_heads:
            raise ValueError(f"{spec.n_heads} query heads are not a multiple of {spec.n_kv_heads} key/value heads")
        if spec.dim > 256 or spec.v_dim > 256:
            raise ValueError(f"attention kernels take head sizes up to 256, got {spec.dim} / {spec.v_dim}")
        if len(spec.lambdas) != 4:
            raise ValueError("lambda is made of four vectors")
        self.eps = float(np.float32(spec.eps))
        self.cap = float(spec.soft_cap) if spec.soft_cap is not None else 0.0
        if spec.soft_cap is not None and not self.cap > 0:
            raise ValueError(f"the cap of the scores must be positive, got {spec.soft_cap}")
        self.window = int(spec.window) if spec.window else 0
        self.k_off = spec.n_heads * 2 * spec.dim
        self.v_off = self.k_off + spec.n_kv_heads * 2 * spec.dim
        self.g_off = self.v_off + spec.n_kv_heads * spec.v_dim
        self.rotation, self.rot_half = None, False
        if spec.rotation is not None:
            pos = build_position(spec.rotation, dtype, device)
            if getattr(pos, "pairing", None) not in ("adjacent", "half") or not hasattr(pos, "rotation"):
                raise ValueError("this mixer takes a rotary spec with pairing 'adjacent' or 'half'")
            self.rotation, self.rot_half = pos.rotation(), pos.pairing == "half"
            if self.rotation[1] > spec.dim:
                raise ValueError(f"the rotation covers {self.rotation[1]} entries, a map has {spec.dim}")
        self.lam = 0.0

    @property
    def inner(self) -> int:
        return self.spec.n_heads * self.spec.v_dim

    def tensors(self) -> dict:
        s = self.spec
        out = {s.q_proj: (s.n_heads * 2 * s.dim, s.hidden), s.k_proj: (s.n_kv_heads * 2 * s.dim, s.hidden),
               s.v_proj: (s.n_kv_heads * s.v_dim, s.hidden), s.o_proj: (s.hidden, s.n_heads * s.v_dim)}
        out.update({name: (s.dim,) for name in s.lambdas})
        if s.head_gate is not None:
            out[s.head_gate] = (s.n_heads, s.hidden)
        return out

    def load(self, src) -> None:
        s = self.spec
        names = [s.q_proj, s.k_proj, s.v_proj] + ([s.head_gate] if s.head_gate is not None else [])
        self.w_in = stack_rows([src.get(n) for n in names])
        self.w_o = src.get(s.o_proj).contiguous()
        q1, k1, q2, k2 = (src.get(n, "vector").double() for n in s.lambdas)
        self.lam = float((torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum())).item()) + float(s.offset)

    def cache_spec(self):
        s = self.spec
        return KVCacheSpec(s.n_kv_heads, 2 * s.dim, s.window, v_head_dim=s.v_dim if s.v_dim != 2 * s.dim else None)

    @property
    def prefill_tile(self):
        return ops.prefill_tile() if ops.difference_prefill_takes_mma(self.dtype, self.spec.dim, self.spec.v_dim) else None

    def launch_variant(self, step):
        s = self.spec
        if not step.n_decode or not ops.difference_decode_takes_mma(self.dtype, s.n_heads, s.n_kv_heads, s.dim, s.v_dim):
            return None
        return ops.difference_decode_pieces(step.n_decode, s.n_kv_heads, s.v_dim, step.max_decode_ctx, self.window)

    def mix(self, proj, step, cache, state, writes_cache=True):
        s = self.spec
        T = proj.shape[0]
        q = step.buffer("attn_q", (T, s.n_heads * 2 * s.dim), self.dtype)
        with span("rope + kv write"):
            ops.qk_norm_store(proj, 0, self.k_off, self.v_off, None, None, self.eps, None, 0.0, q, cache.k, cache.v,
                              step.slots[cache.group] if writes_cache else None, s.n_heads, s.n_kv_heads, s.dim, s.v_dim,
                              cache.page_size, rotation=self.rotation, positions=step.positions, rot_half=self.rot_half,
                              maps=self.MAPS)
        o = step.buffer("attn_o", (T, self.inner), self.dtype)
        gate = proj[:, self.g_off:self.g_off + s.n_heads] if s.head_gate is not None else None
        with span("attention"):
            ops.attention_difference(q, cache.k, cache.v, o, gate, step, cache.group, s.n_heads, s.n_kv_heads, s.dim, s.v_dim,
                                     cache.page_size, float(s.scale), self.cap, self.lam, float(s.out_scale), self.eps,
                                     self.window)
        return o


register_mixer("difference_attention", DifferenceAttention)
