"""Small Papulix configurations and weights for the tests.  The weights are drawn here (not by the package's
random-weights mode) so that attention is peaked and its sink felt, the recurrences' states live for tens of tokens, and
the streams differ: a key that is missed, a lost state, a convolution input, a gate, bias or coefficient that is left out
moves the logits far beyond rounding."""

from __future__ import annotations

import json
import os

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, scale, ff=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale},
            "mlp": dense(ff)}


def channel_delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": dense(ff)}


def mamba2(heads, vdim, state, groups, norm_groups, conv, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                        "norm_groups": norm_groups, "conv": conv}, "mlp": dense(ff)}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def model(vocab, width, eps, emb_scale, logit_scale, streams, layers, loop=None):
    out = {"architecture": "Papulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": emb_scale},
           "logit_scale": logit_scale, "streams": streams, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # every kind of mixer with and without a feed-forward, a loop in the middle over two kinds, three streams
    "A": model(211, 96, 1e-5, 2.0, 1.5, 3, [
        mamba2(6, 16, 24, 3, 2, 4, 40),
        attention(4, 2, 16, 24, 0.5),
        channel_delta(4, 2, 16, 8, 3, 56),
        attention(3, 3, 24, 8, 0.4, 24),
        mamba2(4, 8, 16, 1, 4, 2),
    ], (1, 3, 2)),
    # ones: one stream, one head, one tap, one group, constants of 1, no loop
    "B": model(97, 64, 1e-6, 1.0, 1.0, 1, [
        channel_delta(1, 1, 8, 16, 1, 32),
        mamba2(1, 24, 8, 1, 1, 1),
        attention(1, 1, 8, 8, 1.0, 48),
        channel_delta(3, 1, 24, 8, 5),
        mamba2(5, 8, 12, 5, 5, 3, 24),
    ]),
    # head sizes that the tensor-core attention takes, the whole stack three times
    "C": model(157, 128, 1e-5, 3.0, 0.7, 2, [
        attention(4, 2, 64, 32, 0.25, 128),
        channel_delta(2, 2, 64, 64, 4, 128),
        mamba2(8, 32, 64, 2, 1, 4),
        attention(2, 1, 128, 64, 0.18),
    ], (0, 4, 3)),
    # sizes that are multiples of nothing in particular, four streams, a loop over the last layer
    "D": model(131, 100, 1e-4, 1.7, 3.0, 4, [
        attention(5, 5, 20, 12, 0.45, 50),
        channel_delta(6, 3, 12, 20, 4, 38),
        mamba2(6, 10, 20, 2, 3, 4, 52),
    ], (2, 3, 4)),
    # wide enough for the tcgen05 products over prompts; five streams; the loop at the start
    "E": model(89, 320, 1e-5, 2.5, 2.2, 5, [
        channel_delta(4, 2, 32, 64, 4, 256),
        mamba2(10, 32, 48, 5, 5, 4, 384),
        attention(4, 2, 64, 64, 0.25, 128),
    ], (0, 2, 2)),
    # larger: eight query heads of 128 to a key/value head with values of 96, a delta rule with more columns than rows,
    # one group for twelve heads
    "F": model(1000, 384, 1e-6, 4.0, 1.2, 2, [
        attention(8, 1, 128, 96, 0.18, 512),
        channel_delta(3, 3, 96, 128, 4, 256),
        mamba2(12, 64, 128, 1, 3, 4),
    ], (1, 2, 2)),
}
SEEDS = {"A": 3, "B": 5, "C": 8, "D": 15, "E": 21, "F": 34}
RANKS = {"A": (12, 16), "B": (1, 3), "C": (16, 8), "D": (5, 11), "E": (32, 24), "F": (24, 40)}


def run_order(cfg: dict) -> list:
    n = len(cfg["layers"])
    if cfg.get("loop") is None:
        return list(range(n))
    a, b, times = (cfg["loop"][k] for k in ("start", "stop", "times"))
    return [*range(a), *(list(range(a, b)) * times), *range(b, n)]


def tensor_shapes(cfg: dict, ranks=(8, 8)) -> dict:
    """Names and shapes, listed here independently of the package; `ranks`: of the decay's and of the gate's low-rank maps."""
    W, S = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W)}

    def norm(name):
        out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q = p + "mix."
        norm(p + "norm1")
        out.update({p + "hc1.in": (S,), p + "hc1.out": (S,), p + "hc1.mix": (S, S)})
        H, dv = m["heads"], m["vdim"]
        if l["type"] == "attention":
            G, d = m["kv_heads"], m["dim"]
            out.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * dv, W), q + "q.norm": (H * d,),
                        q + "k.norm": (G * d,), q + "g": (H * dv, W)})
        elif l["type"] == "channel_delta":
            G, d, n = m["kv_heads"], m["dim"], m["conv"]
            ra, rg = ranks
            out.update({q + "q": (G * d, W), q + "q.conv": (G * d, n), q + "k": (G * d, W), q + "k.conv": (G * d, n),
                        q + "v": (H * dv, W), q + "v.conv": (H * dv, n), q + "b": (H, W), q + "A_log": (H,), q + "norm": (dv,),
                        q + "a1": (ra, W), q + "a2": (H * d, ra), q + "dt_bias": (H * d,), q + "g1": (rg, W),
                        q + "g2": (H * dv, rg)})
        else:
            N, G, n = m["state"], m["groups"], m["conv"]
            C = H * dv + 2 * G * N
            out.update({q + "in": (H * dv + C + H, W), q + "conv": (C, n), q + "conv.b": (C,), q + "dt_bias": (H,),
                        q + "A_log": (H,), q + "D": (H,), q + "norm": (H * dv,)})
        out[q + "o"] = (W, H * dv)
        if l["mlp"] is None:
            continue
        ff, u = l["mlp"]["ff"], p + "mlp."
        norm(p + "norm2")
        out.update({p + "hc2.in": (S,), p + "hc2.out": (S,), p + "hc2.mix": (S, S), u + "gate": (ff, W), u + "gate.b": (ff,),
                    u + "up": (ff, W), u + "up.b": (ff,), u + "down": (W, ff), u + "down.b": (W,)})
    return out


def draw_weights(cfg: dict, seed: int, ranks=(8, 8)) -> dict:
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, ranks).items():
        last = name.split(".")[-1]
        z = rng.standard_normal(shape)
        if last == "A_log":
            x = rng.uniform(-3.5, -0.5, shape)             # decays between a few and a hundred tokens
        elif last == "dt_bias":
            x = rng.uniform(-1.5, 1.0, shape)
        elif last == "D":
            x = 0.7 + 0.3 * z
        elif last == "alpha":
            x = rng.uniform(0.4, 0.9, shape) / cfg["streams"]      # some entries saturate, most do not
        elif last == "conv":
            x = 0.3 + 0.6 * z
        elif last == "mix" and len(shape) == 2 and "hc" in name:
            x = 0.75 * np.eye(shape[0]) + 0.25 * z / np.sqrt(shape[0])
        elif ".hc" in name and last == "in":
            x = (1.0 + 0.5 * z) / np.sqrt(shape[0])
        elif ".hc" in name and last == "out":
            x = 1.0 + 0.4 * z
        elif last == "b" and len(shape) == 1:
            x = 0.4 * z                                    # biases of norms, projections and convolutions
        elif len(shape) == 2:
            x = z * 0.7 if last == "embed" else z / np.sqrt(shape[1])
        else:
            x = 1.0 + 0.2 * z                              # norm weights
        out[name] = torch.from_numpy(np.asarray(x, dtype=np.float32).reshape(shape)).to(torch.bfloat16)
    return out


def make_dir(root: str, which: str, cfg: dict | None = None, seed: int | None = None, edit=None) -> str:
    """Writes config.json and model.safetensors (with the `safetensors` package) once; `edit(weights)` may
    change tensors before they are stored."""
    from safetensors.torch import save_file
    out = os.path.join(root, f"papulix_{which}")
    if not os.path.isfile(os.path.join(out, "model.safetensors")):
        os.makedirs(out, exist_ok=True)
        cfg = cfg or CONFIGS[which]
        w = draw_weights(cfg, SEEDS.get(which, 0) if seed is None else seed, RANKS.get(which, (8, 8)))
        if edit is not None:
            edit(w)
        save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(out, "model.safetensors"))
        with open(os.path.join(out, "config.json"), "w") as f:
            json.dump(cfg, f)
    return out


def plain_weights(model_dir: str) -> dict:
    from safetensors.torch import load_file
    return {k: v.to(torch.float64).numpy() for k, v in load_file(os.path.join(model_dir, "model.safetensors")).items()}


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)
