"""The Papulix decoder as a description: pre-norm sublayers over several residual streams (hyper-connections) under a
dynamic tanh, with three kinds of mixer.  "attention": causal grouped-query attention without positions, queries and
keys normed over their whole projections, a softmax with one added to its denominator, and a sigmoid gate on every output
channel.  "channel_delta": a gated delta rule behind short convolutions with a decay a head and key channel, decay and
output gate through low-rank maps.  "mamba2": the state-space dual form of Mamba-2.  Feed-forwards are silu-gated units
with biases.  A stretch of layers may run several times in a row with the same tensors and a cache or state a pass.  This
file holds no size: everything comes from PapulixConfig and the order of its layers.
"""

from __future__ import annotations

from ..config.papulix_config import ARCHITECTURE, PapulixConfig
from ..config.registry import register_architecture
from ..parts.spec import (BiasedAttentionSpec, DynamicTanhSpec, EmbeddingSpec, GatedDeltaSpec, HyperSpec, LayerCall, LayerSpec,
                          LMHeadSpec, ModelSpec, StateSpaceSpec, SwiGLUSpec)

# The design fixes these: the score of the softmax's sink (exp of it is the one in the denominator), and the epsilon
# under the root of the unit norms of the delta rule's queries and keys.
SINK_SCORE = 0.0
UNIT_EPS = 1e-6


def _norm(cfg: PapulixConfig, name: str) -> DynamicTanhSpec:
    return DynamicTanhSpec(cfg.width, name, name + ".b", name + ".alpha")


def _hyper(cfg: PapulixConfig, p: str) -> HyperSpec:
    return HyperSpec(cfg.streams, p + "in", p + "out", p + "mix")


def _mixer(cfg: PapulixConfig, layer, q: str):
    m = layer.mixer
    if layer.type == "attention":
        return BiasedAttentionSpec(
            hidden=cfg.width, n_heads=m.heads, n_kv_heads=m.kv_heads, dim=m.dim, v_dim=m.vdim, scale=m.scale, eps=cfg.eps,
            q_proj=q + "q", k_proj=q + "k", v_proj=q + "v", o_proj=q + "o", q_norm=q + "q.norm", k_norm=q + "k.norm",
            norm_over="projection", sink_score=SINK_SCORE, out_gate=q + "g")
    if layer.type == "channel_delta":
        return GatedDeltaSpec(
            hidden=cfg.width, n_heads=m.heads, n_qk_heads=m.kv_heads, dim=m.dim, v_dim=m.vdim, conv=m.conv, eps=cfg.eps,
            q_proj=q + "q", k_proj=q + "k", v_proj=q + "v", q_conv=q + "q.conv", k_conv=q + "k.conv", v_conv=q + "v.conv",
            beta_proj=q + "b", decay_proj=q + "a2", decay_down=q + "a1", a_log=q + "A_log", dt_bias=q + "dt_bias",
            gate_proj=q + "g2", gate_down=q + "g1", gate_act="sigmoid", out_norm=q + "norm", o_proj=q + "o",
            unit_eps=UNIT_EPS, channel_decay=True)
    return StateSpaceSpec(
        hidden=cfg.width, n_heads=m.heads, n_groups=m.groups, n_state=m.state, v_dim=m.vdim, conv=m.conv,
        norm_groups=m.norm_groups, eps=cfg.eps, in_proj=q + "in", conv_weight=q + "conv", conv_bias=q + "conv.b",
        a_log=q + "A_log", dt_bias=q + "dt_bias", skip=q + "D", out_norm=q + "norm", o_proj=q + "o")


def _feed_forward(cfg: PapulixConfig, ff, p: str):
    if ff is None:
        return None
    return SwiGLUSpec(cfg.width, ff, p + "gate", p + "up", p + "down", gate_bias=p + "gate.b", up_bias=p + "up.b",
                      down_bias=p + "down.b")


def describe_papulix(cfg: PapulixConfig) -> ModelSpec:
    W = cfg.width
    layers, unread = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ff = _feed_forward(cfg, layer.ff, p + "mlp.")
        layers.append(LayerSpec(
            norm1=_norm(cfg, p + "norm1"), mixer=_mixer(cfg, layer, p + "mix."), norm2=_norm(cfg, p + "norm2") if ff else None,
            feed_forward=ff, arrangement="hyper", hyper1=_hyper(cfg, p + "hc1."), hyper2=_hyper(cfg, p + "hc2.") if ff else None))
        if ff is None:      # a checkpoint may carry what a layer without a feed-forward does not read
            unread += [p + n for n in ("norm2", "norm2.b", "norm2.alpha", "hc2.in", "hc2.out", "hc2.mix")]
    # every pass of the loop is a call of its own, with cache slot and state of its own
    order = tuple(LayerCall(layer, run) for run, layer in enumerate(cfg.run_order()))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden=W, embedding=EmbeddingSpec(cfg.vocab, W, "embed", scale=cfg.embedding_scale),
        layers=tuple(layers), order=order, final_norm=_norm(cfg, "final.norm"),
        lm_head=LMHeadSpec(cfg.vocab, W, "head", logit_scale=cfg.logit_scale), max_positions=cfg.max_positions,
        ignorable=tuple(unread), eos_token_ids=tuple(cfg.eos_token_ids))


def papulix_tensor_kinds(cfg: PapulixConfig) -> dict:
    """{name: (shape, kind)} of every checkpoint tensor, for the random-weights mode.  Kinds: "matrix" N(0, 0.02);
    "norm" N(1, 0.02), also for the coefficients of the streams and the scalars of the norms; "offset" N(0, 0.1) for
    biases, decay logarithms and step biases; "taps" N(0, 0.5) for the short convolutions; "mixing" for the streams'
    mixing matrices, N(0, 0.1) around the identity.  The ranks of the low-rank maps are the heads' widths."""
    W, S = cfg.width, cfg.streams
    out = {"embed": ((cfg.vocab, W), "matrix"), "head": ((cfg.vocab, W), "matrix")}

    def norm(name):
        out[name] = ((W,), "norm")
        out[name + ".b"] = ((W,), "offset")
        out[name + ".alpha"] = ((), "norm")

    def hyper(p):
        out[p + "in"] = ((S,), "norm")
        out[p + "out"] = ((S,), "norm")
        out[p + "mix"] = ((S, S), "mixing")

    norm("final.norm")
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        q = p + "mix."
        norm(p + "norm1")
        hyper(p + "hc1.")
        if layer.type == "attention":
            rows = (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim), ("g", m.heads * m.vdim))
            for name, n in rows:
                out[q + name] = ((n, W), "matrix")
            out[q + "q.norm"] = ((m.heads * m.dim,), "norm")
            out[q + "k.norm"] = ((m.kv_heads * m.dim,), "norm")
            inner = m.heads * m.vdim
        elif layer.type == "channel_delta":
            inner = m.heads * m.vdim
            for name, n in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", inner)):
                out[q + name] = ((n, W), "matrix")
                out[q + name + ".conv"] = ((n, m.conv), "taps")
            out[q + "b"] = ((m.heads, W), "matrix")
            out[q + "A_log"] = ((m.heads,), "offset")
            out[q + "norm"] = ((m.vdim,), "norm")
            out[q + "a1"] = ((m.dim, W), "matrix")
            out[q + "a2"] = ((m.heads * m.dim, m.dim), "matrix")
            out[q + "dt_bias"] = ((m.heads * m.dim,), "offset")
            out[q + "g1"] = ((m.vdim, W), "matrix")
            out[q + "g2"] = ((inner, m.vdim), "matrix")
        else:
            inner = m.inner
            out[q + "in"] = ((inner + m.channels + m.heads, W), "matrix")
            out[q + "conv"] = ((m.channels, m.conv), "taps")
            out[q + "conv.b"] = ((m.channels,), "offset")
            for name, kind in (("dt_bias", "offset"), ("A_log", "offset"), ("D", "norm")):
                out[q + name] = ((m.heads,), kind)
            out[q + "norm"] = ((inner,), "norm")
        out[q + "o"] = ((W, inner), "matrix")
        if layer.ff is None:
            continue
        norm(p + "norm2")
        hyper(p + "hc2.")
        q = p + "mlp."
        for name, n, k in (("gate", layer.ff, W), ("up", layer.ff, W), ("down", W, layer.ff)):
            out[q + name] = ((n, k), "matrix")
            out[q + name + ".b"] = ((n,), "offset")
    return out


register_architecture(ARCHITECTURE, PapulixConfig.from_dict, describe_papulix, papulix_tensor_kinds)
