"""The Dotivik decoder restated plainly in float64 numpy: whole sequences, no cache, no batching, one function per
mechanism.  It shares no code with the package; the tests compare the package against it.

`forward(cfg, w, tokens)` takes the dictionary of a config.json, a dictionary name -> float array of the
checkpoint's tensors, and one sequence of token ids; it returns the logits of every position and the residual stream
after every run of a layer.
"""

from __future__ import annotations

import numpy as np


_coarse = [lambda x: x]


class coarse_products:
    """Within this context every matrix product takes its inputs, and leaves its result, through `fn` (the
    rounding of a narrower number type), and so do the rotated queries and keys, the softmax weights and what the
    heads hand on; everything else stays float64.  It models what rounding alone does to the logits: the tests take
    their tolerance for a narrow type from it."""

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


# ---- norms, gates ------------------------------------------------------------------------------------


def layer_norm(x, weight, eps):
    """Mean taken off, divided by the standard deviation (of the squared deviations' mean, eps under the root)."""
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


# ---- rotations ---------------------------------------------------------------------------------------


def angles(n_positions, rot):
    """[positions, dims / 2]"""
    dims = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * np.arange(dims // 2) / dims)
    return np.arange(n_positions)[:, None] * f[None, :]


def rotate_neighbours(x, rot):
    """x [T, heads, d]: entries 2i and 2i + 1 of the first `dims` turn together."""
    a = angles(x.shape[0], rot)[:, None, :]
    n = 2 * a.shape[-1]
    out = x.copy()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:n:2] = v * np.cos(a) + u * np.sin(a)
    return out


def rotate_halves(x, rot):
    """x [T, heads, d]: entries i and i + dims / 2 of the first `dims` turn together."""
    a = angles(x.shape[0], rot)[:, None, :]
    h = a.shape[-1]
    out = x.copy()
    u, v = x[..., :h], x[..., h:2 * h]
    out[..., :h] = u * np.cos(a) - v * np.sin(a)
    out[..., h:2 * h] = v * np.cos(a) + u * np.sin(a)
    return out


# ---- attention ---------------------------------------------------------------------------------------


def softmax(s):
    """Over the last axis; a hidden key has a score of minus infinity."""
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def capped(s, cap):
    return cap * np.tanh(s / cap)


def softmax_attention(q, k, v, score, window=None):
    """One head: q, k [T, d], v [T, dv]; `score` turns raw products into scores; each row sees the keys up to itself,
    the last `window` of them where one is given."""
    i, j = np.arange(q.shape[0])[:, None], np.arange(k.shape[0])[None, :]
    seen = (j <= i) if window is None else (j <= i) & (i - j < int(window))
    return kept(softmax(np.where(seen, score(q @ k.T), -np.inf))) @ v


def head_weight(w, p, diff):
    """The number by which the second map's output is multiplied before it is taken off the first's."""
    return float(np.exp(np.sum(w[p + "lq1"] * w[p + "lk1"])) - np.exp(np.sum(w[p + "lq2"] * w[p + "lk2"])) + diff)


def difference_of_maps(a1, a2, lam, diff, eps):
    """One head: a1 - lam a2, divided by its root mean square, times 1 - diff."""
    return rms_norm(a1 - lam * a2, 1.0, eps) * (1.0 - diff)


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = kept(rotate_neighbours(linear(h, w[p + "q"]).reshape(T, H * 2, d), m["rot"])).reshape(T, H, 2, d)
    k = kept(rotate_neighbours(linear(h, w[p + "k"]).reshape(T, G * 2, d), m["rot"])).reshape(T, G, 2, d)
    v = linear(h, w[p + "v"]).reshape(T, G, dv)
    gate = sigmoid(linear(h, w[p + "g"]))
    lam = head_weight(w, p, m["diff"])
    score = lambda raw: capped(raw * m["scale"], m["softcap"])
    out = np.zeros((T, H, dv))
    for i in range(H):
        g = i // (H // G)
        maps = [softmax_attention(q[:, i, j], k[:, g, j], v[:, g], score) for j in (0, 1)]
        out[:, i] = difference_of_maps(maps[0], maps[1], lam, m["diff"], eps) * gate[:, i:i + 1]
    return linear(out.reshape(T, H * dv), w[p + "o"])


def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = linear(h, w[p + "q"]).reshape(T, H, d + dr)
    z = linear(h, w[p + "dkv"])
    c = kept(rms_norm(z[:, :r], w[p + "dkv.norm"], eps))
    k_rot = kept(rotate_halves(z[:, None, r:], m["rot"]))[:, 0]
    q_rot = kept(rotate_halves(q[..., d:], m["rot"]))
    k_plain = linear(c, w[p + "uk"]).reshape(T, H, d)
    v = linear(c, w[p + "uv"]).reshape(T, H, dv)
    gate = sigmoid(linear(h, w[p + "g"]))
    out = np.zeros((T, H, dv))
    for i in range(H):
        qi = np.concatenate([q[:, i, :d], q_rot[:, i]], axis=1)
        ki = np.concatenate([k_plain[:, i], k_rot], axis=1)
        out[:, i] = softmax_attention(qi, ki, v[:, i], lambda raw: raw * m["scale"], m["mask"]["size"]) * gate[:, i:i + 1]
    return linear(out.reshape(T, H * dv), w[p + "o"])


# ---- feed-forward and the model ----------------------------------------------------------------------


def gated_unit(h, w, p):
    return linear(gelu_tanh(linear(h, w[p + "gate"])) * linear(h, w[p + "up"]), w[p + "down"])


MIXERS = {"attention": attention, "latent_attention": latent_attention}


def runs(cfg):
    """(layer, whether a pass of the loop starts with it) in the order in which they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    middle = [(i, i == a) for i in range(a, b)] * int(loop["times"])
    return [(i, False) for i in range(a)] + middle + [(i, False) for i in range(b, n)]


def pass_input(x, x0, weight):
    """What a pass of the loop starts from: a linear map of the stream beside the embedding's row."""
    return linear(np.concatenate([x, x0], axis=-1), weight, exact_result=True)


def run_layer(x, layer, w, p, eps):
    h = layer_norm(x, w[p + "norm1"], eps)
    y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
    if layer.get("mlp") is not None:
        y = y + gated_unit(h, w, p + "mlp.")
    return x + y


def forward(cfg, w, tokens):
    """(logits [T, vocab], [the residual stream after every run of a layer])."""
    eps = float(cfg["norm"]["eps"])
    x0 = w["embed"][np.asarray(tokens)]
    x, after = x0, []
    for i, starts_pass in runs(cfg):
        if starts_pass:
            x = pass_input(x, x0, w["loop.in"])
        x = run_layer(x, cfg["layers"][i], w, f"l{i}.", eps)
        after.append(x)
    return linear(layer_norm(x, w["final.norm"], eps), w["embed"], exact_result=True), after
