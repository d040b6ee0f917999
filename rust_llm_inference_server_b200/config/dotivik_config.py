"""Typed configuration of the Dotivik decoder, read from its `config.json`.

The file lists the layers one by one; every size and every constant that can differ between two models of the
design comes from it:

    {"architecture": "Dotivik", "vocab": V, "width": W, "norm": {"eps": e},
     "loop": {"start": a, "stop": b, "times": n} | absent,
     "layers": [{"type": "attention" | "latent_attention", "mixer": {...}, "mlp": {"kind": "dense", "ff": F} | null}, ...]}

type "attention": mixer {heads, kv_heads, dim, vdim, scale, softcap, diff, rot {dims, base}}.
type "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, scale, mask {size}, rot {dims, base}}.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .lasapel_config import UNBOUNDED_POSITIONS, _float, _int    # the shared field readers
from .model_config import ConfigError
from .papulix_config import _grouped, _mlp, _obj

ARCHITECTURE = "Dotivik"


@dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float

    @staticmethod
    def from_dict(d: dict, where: str, most: int) -> "RotationConfig":
        out = RotationConfig(_int(d, "dims", where), _float(d, "base", where))
        if out.dims % 2 or out.dims > most:
            raise ConfigError(f"config.json: {where}: {out.dims} rotated entries of {most} cannot be paired")
        if not out.base > 0:
            raise ConfigError(f"config.json: {where}.base must be positive")
        return out


@dataclass(frozen=True)
class DifferenceAttentionConfig:
    """The mixer of an "attention" layer."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    diff: float
    rot: RotationConfig

    @staticmethod
    def from_dict(d: dict, where: str) -> "DifferenceAttentionConfig":
        heads, kv = _grouped(d, where, "kv_heads")
        dim, cap = _int(d, "dim", where), _float(d, "softcap", where)
        if not cap > 0:
            raise ConfigError(f"config.json: {where}.softcap must be positive")
        return DifferenceAttentionConfig(heads, kv, dim, _int(d, "vdim", where), _float(d, "scale", where), cap,
                                         _float(d, "diff", where), RotationConfig.from_dict(_obj(d, "rot", where), where + ".rot", dim))


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int
    rot: RotationConfig

    @staticmethod
    def from_dict(d: dict, where: str) -> "LatentAttentionConfig":
        rot_dim = _int(d, "rot_dim", where)
        rot = RotationConfig.from_dict(_obj(d, "rot", where), where + ".rot", rot_dim)
        if rot.dims != rot_dim:
            raise ConfigError(f"config.json: {where}: all of the {rot_dim} shared entries are rotated, not {rot.dims}")
        return LatentAttentionConfig(_int(d, "heads", where), _int(d, "dim", where), rot_dim, _int(d, "vdim", where),
                                     _int(d, "kv_rank", where), _float(d, "scale", where),
                                     _int(_obj(d, "mask", where), "size", where + ".mask"), rot)


@dataclass(frozen=True)
class DotivikLayer:
    type: str
    mixer: object                    # DifferenceAttentionConfig | LatentAttentionConfig
    ff: Optional[int]                # None: no feed-forward


@dataclass(frozen=True)
class DotivikConfig:
    architecture = ARCHITECTURE

    vocab: int
    width: int
    eps: float
    layers: tuple
    loop: Optional[tuple]            # (start, stop, times): layers start .. stop - 1 run `times` times in a row; None: no loop
    eos_token_ids: tuple = ()
    bos_token_id: Optional[int] = None
    max_positions: int = UNBOUNDED_POSITIONS     # the design has no positional table and no limit of its own

    MIXERS = {"attention": DifferenceAttentionConfig, "latent_attention": LatentAttentionConfig}

    def runs(self) -> tuple:
        """(layer, whether it starts a pass of the loop) in the order in which the layers run."""
        start, stop, times = self.loop or (0, 0, 0)
        one_pass = tuple((i, i == start) for i in range(start, stop))
        return tuple((i, False) for i in range(start)) + one_pass * times + tuple((i, False) for i in range(stop, len(self.layers)))

    @classmethod
    def from_dict(cls, d: dict) -> "DotivikConfig":
        vocab, width = _int(d, "vocab", "config"), _int(d, "width", "config")
        eps = _float(_obj(d, "norm", "config"), "eps", "norm")
        if not eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]"
            if not isinstance(entry, dict) or not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"config.json: {where} must be an object with 'type' and 'mixer'")
            kind = entry.get("type")
            if kind not in cls.MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not one of {sorted(cls.MIXERS)}")
            layers.append(DotivikLayer(kind, cls.MIXERS[kind].from_dict(entry["mixer"], where + ".mixer"),
                                       _mlp(entry.get("mlp"), where + ".mlp")))
        loop = None
        if d.get("loop") is not None:
            lp = _obj(d, "loop", "config")
            loop = (_int(lp, "start", "loop", 0), _int(lp, "stop", "loop", 0), _int(lp, "times", "loop", 0))
            if not loop[0] <= loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop[0]} .. {loop[1] - 1} of {len(layers)}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else (eos,)))
        return cls(vocab, width, eps, tuple(layers), loop, eos_ids, d.get("bos_token_id"))
