"""Small Dotivik configurations and weights for the tests.  The weights are drawn here (not by the package's random-weights
mode) so that attention is peaked and its scores reach the cap, the two maps differ, and gates and the looped passes matter: a
key that is missed, a window one token off, a cap, gate, norm or pass input that is left out moves the logits far beyond
rounding."""

from __future__ import annotations

import json
import os

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, scale, cap, diff, rot, ff=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "softcap": cap, "diff": diff, "rot": {"dims": rot[0], "base": rot[1]}}, "mlp": dense(ff)}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window, base, ff=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale, "mask": {"size": window}, "rot": {"dims": rot_dim, "base": base}},
            "mlp": dense(ff)}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def model(vocab, width, eps, layers, loop=None):
    out = {"architecture": "Dotivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # both mixers with and without a feed-forward, a loop in the middle, windows shorter than a page and longer than two
    "A": model(211, 96, 1e-5, [
        latent(3, 16, 8, 24, 40, 0.3, 7, 10000.0, 40),
        attention(4, 2, 16, 24, 0.5, 6.0, 0.4, (8, 500.0)),
        latent(5, 8, 16, 8, 24, 0.35, 37, 3000.0),
        attention(3, 3, 24, 8, 0.4, 30.0, 0.8, (24, 10000.0), 56),
    ], (1, 3, 2)),
    # ones: one head, a window of one token, one pair rotated, a loop that runs once, constants of 1
    "B": model(97, 64, 1e-6, [
        attention(1, 1, 8, 16, 1.0, 1.0, 0.5, (2, 100.0), 32),
        latent(1, 8, 2, 8, 16, 1.0, 1, 50.0, 48),
        attention(3, 1, 8, 8, 0.6, 9.0, 0.0, (8, 1000.0)),
    ], (0, 1, 1)),
    # sizes that the tensor-core kernels take (also padded ones), the whole stack three times
    "C": model(157, 128, 1e-5, [
        attention(4, 2, 64, 128, 0.2, 20.0, 0.3, (32, 20000.0), 128),
        latent(6, 32, 32, 32, 64, 0.25, 100, 10000.0, 128),
        attention(8, 1, 40, 72, 0.25, 70.0, 0.6, (20, 10000.0), 64),
    ], (0, 3, 3)),
    # sizes that are multiples of nothing in particular, no loop
    "D": model(131, 100, 1e-4, [
        attention(5, 5, 20, 12, 0.45, 12.0, 0.2, (12, 700.0), 50),
        latent(7, 12, 6, 10, 36, 0.4, 23, 900.0, 38),
    ]),
    # wide enough for the tcgen05 products over prompts; more heads than a tile of 16; the loop at the end
    "E": model(89, 320, 1e-5, [
        latent(18, 16, 16, 16, 128, 0.3, 150, 10000.0, 256),
        attention(6, 3, 56, 96, 0.22, 50.0, 0.35, (28, 50000.0), 384),
        latent(4, 64, 32, 64, 256, 0.15, 64, 2000.0, 128),
    ], (1, 3, 2)),
    # ten query heads to a key/value head, wider maps than the tensor-core kernels take, a window longer than the prompts
    "F": model(300, 192, 1e-6, [
        attention(10, 1, 32, 64, 0.3, 15.0, 0.1, (16, 10000.0), 96),
        attention(2, 1, 72, 136, 0.2, 10.0, 0.5, (72, 10000.0), 64),
        latent(2, 128, 64, 128, 512, 0.12, 5000, 10000.0, 96),
    ], (0, 1, 4)),
}
SEEDS = {"A": 3, "B": 5, "C": 8, "D": 15, "E": 21, "F": 34}


def runs(cfg: dict) -> list:
    n = len(cfg["layers"])
    if cfg.get("loop") is None:
        return list(range(n))
    a, b, times = (cfg["loop"][k] for k in ("start", "stop", "times"))
    return [*range(a), *(list(range(a, b)) * times), *range(b, n)]


def tensor_shapes(cfg: dict) -> dict:
    """Names and shapes, listed here independently of the package."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    if cfg.get("loop") is not None:
        out["loop.in"] = (W, 2 * W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q = p + "mix."
        H, dv, d = m["heads"], m["vdim"], m["dim"]
        out[p + "norm1"] = (W,)
        if l["type"] == "attention":
            G = m["kv_heads"]
            out.update({q + "q": (2 * H * d, W), q + "k": (2 * G * d, W), q + "v": (G * dv, W)})
            out.update({q + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")})
        else:
            r, dr = m["kv_rank"], m["rot_dim"]
            out.update({q + "q": (H * (d + dr), W), q + "dkv": (r + dr, W), q + "dkv.norm": (r,), q + "uk": (H * d, r),
                        q + "uv": (H * dv, r)})
        out.update({q + "g": (H, W), q + "o": (W, H * dv)})
        if l["mlp"] is not None:
            ff, u = l["mlp"]["ff"], p + "mlp."
            out.update({u + "gate": (ff, W), u + "up": (ff, W), u + "down": (W, ff)})
    return out


def draw_weights(cfg: dict, seed: int) -> dict:
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        z = rng.standard_normal(shape)
        if last in ("lq1", "lk1", "lq2", "lk2"):
            x = 0.7 * z / np.sqrt(shape[0]) + (0.05 if last[2] == "1" else 0.0)
        elif len(shape) == 1:
            x = 1.0 + 0.2 * z                              # norm weights
        elif last == "embed":
            x = z + 0.3                                    # rows whose mean is not zero
        elif name == "loop.in":
            x = z / np.sqrt(shape[1])
        else:
            x = z / np.sqrt(shape[1])
        out[name] = torch.from_numpy(np.asarray(x, dtype=np.float32).reshape(shape)).to(torch.bfloat16)
    return out


def make_dir(root: str, which: str, cfg: dict | None = None, seed: int | None = None, edit=None) -> str:
    """Writes config.json and model.safetensors (with the `safetensors` package) once; `edit(weights)` may
    change tensors before they are stored."""
    from safetensors.torch import save_file
    out = os.path.join(root, f"dotivik_{which}")
    if not os.path.isfile(os.path.join(out, "model.safetensors")):
        os.makedirs(out, exist_ok=True)
        cfg = cfg or CONFIGS[which]
        w = draw_weights(cfg, SEEDS.get(which, 0) if seed is None else seed)
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
