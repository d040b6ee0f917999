"""The Papulix decoder restated plainly in float64 numpy: whole sequences, no cache, no batching, one function per
mechanism.  It shares no code with the package; the tests compare the package against it.

`forward(cfg, w, tokens)` takes the dictionary of a config.json, a dictionary name -> float array of the
checkpoint's tensors, and one sequence of token ids; it returns the logits of every position and the sum of the
residual streams after every run of a layer.
"""

from __future__ import annotations

import numpy as np


_coarse = [lambda x: x]

UNIT_EPS = 1e-6


class coarse_products:
    """Within this context every matrix product takes its inputs, and leaves its result, through `fn` (the
    rounding of a narrower number type), and so do the queries, keys and values that attention keeps;
    everything else stays float64.  It models what rounding alone does to the logits: the tests take their
    tolerance for a narrow type from it."""

    def __init__(self, fn):
        self.fn = fn

    def __enter__(self):
        _coarse.append(self.fn)

    def __exit__(self, *exc):
        _coarse.pop()


def kept(x):
    return _coarse[-1](x)


def linear(h, weight, exact_result=False):
    y = kept(h) @ weight.T
    return y if exact_result else kept(y)


def rms_norm(x, weight, eps):
    """x divided by its root mean square over the last axis (eps under the root), times the weight."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


# ---- norm and residual streams ----------------------------------------------------------------------


def dynamic_tanh(x, w, name):
    return np.tanh(float(np.reshape(w[name + ".alpha"], -1)[0]) * x) * w[name] + w[name + ".b"]


def stream_input(streams, coef):
    """What a sublayer reads: the streams weighed, [S, T, W] -> [T, W]."""
    return np.einsum("s,stw->tw", coef, streams)


def stream_update(streams, mix, out, y):
    """x_t <- sum_s mix[s, t] x_s + out[t] y, with the old x_s on the right (rows of mix are sources, columns targets)."""
    return np.einsum("st,sjw->tjw", mix, streams) + out[:, None, None] * y[None]


# ---- short convolution ------------------------------------------------------------------------------


def short_conv(x, taps, bias=None):
    """y[t, c] = silu(sum_j taps[c, j] x[t - (n - 1) + j, c] + bias[c]), zeros before the start."""
    T, C = x.shape
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, C)), x], axis=0)
    y = sum(padded[j:j + T] * taps[:, j] for j in range(n))
    return silu(y if bias is None else y + bias)


# ---- the delta rule with a decay a channel ----------------------------------------------------------


def channel_decay_delta(q, k, v, beta, g):
    """q, k, g [T, d], v [T, dv], beta [T] of one head: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o =
    S^T q."""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def channel_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(linear(h, w[p + "q"]), w[p + "q.conv"]).reshape(T, G, d)
    k = short_conv(linear(h, w[p + "k"]), w[p + "k.conv"]).reshape(T, G, d)
    v = short_conv(linear(h, w[p + "v"]), w[p + "v.conv"]).reshape(T, H, dv)
    q = q / np.sqrt(np.sum(q * q, axis=-1, keepdims=True) + UNIT_EPS) * d ** -0.5
    k = k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + UNIT_EPS)
    beta = sigmoid(linear(h, w[p + "b"]))
    step = softplus(linear(linear(h, w[p + "a1"]), w[p + "a2"]) + w[p + "dt_bias"]).reshape(T, H, d)
    g = np.exp(-np.exp(w[p + "A_log"])[None, :, None] * step)
    o = np.stack([channel_decay_delta(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], beta[:, i], g[:, i])
                  for i in range(H)], axis=1)
    gate = sigmoid(linear(linear(h, w[p + "g1"]), w[p + "g2"])).reshape(T, H, dv)
    y = rms_norm(o, w[p + "norm"], eps) * gate
    return linear(y.reshape(T, H * dv), w[p + "o"])


# ---- the state-space mixer --------------------------------------------------------------------------


def state_space(x, B, C, dt, log_a, D):
    """x [T, P], B, C [T, N], dt [T] of one head: S <- exp(log_a dt) S + dt B x^T; y = S^T C + D x."""
    S = np.zeros((B.shape[1], x.shape[1]))
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(log_a * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        out[t] = S.T @ C[t] + D * x[t]
    return out


def gated_group_norm(y, z, weight, groups, eps):
    """y silu(z), then each of `groups` equal parts divided by its own root mean square, times the weight."""
    T, W = y.shape
    y = (y * silu(z)).reshape(T, groups, W // groups)
    return rms_norm(y, 1.0, eps).reshape(T, W) * weight


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = linear(h, w[p + "in"])
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = short_conv(xbc, w[p + "conv"], w[p + "conv.b"])
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    y = np.stack([state_space(x[:, i], B[:, i // (H // G)], C[:, i // (H // G)], dt[:, i],
                              -np.exp(w[p + "A_log"][i]), w[p + "D"][i]) for i in range(H)], axis=1)
    y = gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps)
    return linear(y, w[p + "o"])


# ---- attention --------------------------------------------------------------------------------------


def softmax_plus_one(s):
    """exp(s_j) / (1 + sum exp(s_j))."""
    top = max(float(s.max()), 0.0)
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum())


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = kept(rms_norm(linear(h, w[p + "q"]), w[p + "q.norm"], eps)).reshape(T, H, d)
    k = kept(rms_norm(linear(h, w[p + "k"]), w[p + "k.norm"], eps)).reshape(T, G, d)
    v = linear(h, w[p + "v"]).reshape(T, G, dv)
    out = np.zeros((T, H, dv))
    for hd in range(H):
        g = hd // (H // G)
        scores = (q[:, hd] @ k[:, g].T) * float(m["scale"])
        for i in range(T):
            out[i, hd] = softmax_plus_one(scores[i, :i + 1]) @ v[:i + 1, g]
    gate = sigmoid(linear(h, w[p + "g"]))
    return linear(out.reshape(T, H * dv) * gate, w[p + "o"])


# ---- feed-forward and the model ---------------------------------------------------------------------


def gated_unit(h, w, p):
    gate = linear(h, w[p + "gate"], exact_result=True) + w[p + "gate.b"]
    up = linear(h, w[p + "up"], exact_result=True) + w[p + "up.b"]
    return linear(silu(gate) * up, w[p + "down"]) + w[p + "down.b"]


MIXERS = {"channel_delta": channel_delta, "mamba2": mamba2, "attention": attention}


def run_order(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if loop is None:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def run_layer(streams, layer, w, p, eps):
    u = dynamic_tanh(stream_input(streams, w[p + "hc1.in"]), w, p + "norm1")
    y = MIXERS[layer["type"]](u, w, p + "mix.", layer["mixer"], eps)
    streams = stream_update(streams, w[p + "hc1.mix"], w[p + "hc1.out"], y)
    if layer.get("mlp") is not None:
        u = dynamic_tanh(stream_input(streams, w[p + "hc2.in"]), w, p + "norm2")
        streams = stream_update(streams, w[p + "hc2.mix"], w[p + "hc2.out"], gated_unit(u, w, p + "mlp."))
    return streams


def forward(cfg, w, tokens):
    """(logits [T, vocab], [sum of the streams after every run of a layer])."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    streams = np.stack([x] * int(cfg["streams"]))
    after = []
    for i in run_order(cfg):
        streams = run_layer(streams, cfg["layers"][i], w, f"l{i}.", eps)
        after.append(streams.sum(axis=0))
    h = dynamic_tanh(streams.sum(axis=0), w, "final.norm")
    return linear(h, w["head"], exact_result=True) * float(cfg["logit_scale"]), after
