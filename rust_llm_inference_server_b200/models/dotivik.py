"""The Dotivik decoder as a description: layers whose two sublayers read one layer norm side by side, x += mixer(h) + ff(h),
with two kinds of mixer.  "attention": grouped-query attention with two maps a head whose outputs are taken off each other and
normed a head, scores capped by tanh, part of every map rotated in neighbouring pairs, a gate a head.  "latent_attention": keys
and values as linear maps of a small cached latent beside a rotated key part that all heads share, over a sliding window, with
queries straight from the input and a gate a head.  Feed-forwards are units gated by the tanh form of gelu.  A stretch of
layers may run several times in a row with the same tensors and a cache a pass; every pass starts with a linear map of the
stream beside the embedding's row.  The logits come from the embedding table.  This file holds no size: everything comes from
DotivikConfig and the order of its layers.
"""

from __future__ import annotations

from ..config.dotivik_config import ARCHITECTURE, DotivikConfig
from ..config.registry import register_architecture
from ..parts.spec import (GELU_TANH, DifferenceAttentionSpec, EmbeddingSpec, LatentAttentionSpec, LayerCall, LayerNormSpec,
                          LayerSpec, LMHeadSpec, ModelSpec, StreamJoinSpec, SwiGLUSpec, YarnRopeSpec)

LOOP_INPUT = "loop.in"


def _mixer(cfg: DotivikConfig, layer, q: str):
    m = layer.mixer
    if layer.type == "attention":
        return DifferenceAttentionSpec(
            hidden=cfg.width, n_heads=m.heads, n_kv_heads=m.kv_heads, dim=m.dim, v_dim=m.vdim, scale=m.scale, eps=cfg.eps,
            q_proj=q + "q", k_proj=q + "k", v_proj=q + "v", o_proj=q + "o", lambdas=(q + "lq1", q + "lk1", q + "lq2", q + "lk2"),
            offset=m.diff, out_scale=1.0 - m.diff, soft_cap=m.softcap,
            rotation=YarnRopeSpec(m.rot.dims, m.rot.base, pairing="adjacent"), head_gate=q + "g")
    return LatentAttentionSpec(
        hidden=cfg.width, n_heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, v_dim=m.vdim, q_rank=None, kv_rank=m.kv_rank,
        scale=m.scale, eps=cfg.eps, q_down=None, q_norm=None, q_up=q + "q", kv_down=q + "dkv", kv_norm=q + "dkv.norm",
        k_up=q + "uk", v_up=q + "uv", o_proj=q + "o", position=YarnRopeSpec(m.rot.dims, m.rot.base), window=m.window,
        head_gate=q + "g")


def describe_dotivik(cfg: DotivikConfig) -> ModelSpec:
    W = cfg.width
    norm = lambda name: LayerNormSpec(W, cfg.eps, name)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        q = p + "mlp."
        ff = SwiGLUSpec(W, layer.ff, q + "gate", q + "up", q + "down", **GELU_TANH) if layer.ff is not None else None
        layers.append(LayerSpec(norm1=norm(p + "norm1"), mixer=_mixer(cfg, layer, p + "mix."), norm2=None, feed_forward=ff,
                                arrangement="parallel"))
    # every pass of the loop is a call of its own, with a cache slot of its own, and starts with the same map
    join = StreamJoinSpec(W, LOOP_INPUT)
    order = tuple(LayerCall(i, run, entry=join if starts else None) for run, (i, starts) in enumerate(cfg.runs()))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden=W, embedding=EmbeddingSpec(cfg.vocab, W, "embed"), layers=tuple(layers), order=order,
        final_norm=norm("final.norm"), lm_head=LMHeadSpec(cfg.vocab, W, "embed"), max_positions=cfg.max_positions,
        ignorable=(LOOP_INPUT,), eos_token_ids=tuple(cfg.eos_token_ids))


def dotivik_tensor_kinds(cfg: DotivikConfig) -> dict:
    """{name: (shape, kind)} of every checkpoint tensor, for the random-weights mode.  Kinds: "matrix" N(0, 0.02); "norm"
    N(1, 0.02); "offset" N(0, 0.1) for the vectors that lambda is made of."""
    W = cfg.width
    out = {"embed": ((cfg.vocab, W), "matrix"), "final.norm": ((W,), "norm")}
    if cfg.loop is not None:
        out[LOOP_INPUT] = ((W, 2 * W), "matrix")
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        q = p + "mix."
        out[p + "norm1"] = ((W,), "norm")
        if layer.type == "attention":
            rows = (("q", m.heads * 2 * m.dim), ("k", m.kv_heads * 2 * m.dim), ("v", m.kv_heads * m.vdim))
            for name in ("lq1", "lk1", "lq2", "lk2"):
                out[q + name] = ((m.dim,), "offset")
        else:
            rows = (("q", m.heads * (m.dim + m.rot_dim)), ("dkv", m.kv_rank + m.rot_dim))
            out[q + "dkv.norm"] = ((m.kv_rank,), "norm")
            out[q + "uk"] = ((m.heads * m.dim, m.kv_rank), "matrix")
            out[q + "uv"] = ((m.heads * m.vdim, m.kv_rank), "matrix")
        for name, n in rows + (("g", m.heads),):
            out[q + name] = ((n, W), "matrix")
        out[q + "o"] = ((W, m.heads * m.vdim), "matrix")
        if layer.ff is not None:
            for name, n, k in (("gate", layer.ff, W), ("up", layer.ff, W), ("down", W, layer.ff)):
                out[p + "mlp." + name] = ((n, k), "matrix")
    return out


register_architecture(ARCHITECTURE, DotivikConfig.from_dict, describe_dotivik, dotivik_tensor_kinds)
