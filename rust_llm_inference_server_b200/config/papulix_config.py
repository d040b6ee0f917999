"""Typed configuration of the Papulix decoder, read from its `config.json`.

The file lists the layers one by one; every size and every constant that can differ between two models of the
design comes from it:

    {"architecture": "Papulix", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "logit_scale": c, "streams": S, "loop": {"start": a, "stop": b, "times": n} | absent,
     "layers": [{"type": "attention" | "channel_delta" | "mamba2", "mixer": {...}, "mlp": {...} | null}, ...]}

type "attention": mixer {heads, kv_heads, dim, vdim, scale}.
type "channel_delta": mixer {heads, kv_heads, dim, vdim, conv}; the ranks of its low-rank maps are the tensors'.
type "mamba2": mixer {heads, vdim, state, groups, norm_groups, conv}.
mlp: kind "dense" {ff}.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .lasapel_config import UNBOUNDED_POSITIONS, _float, _int    # the shared field readers
from .model_config import ConfigError

ARCHITECTURE = "Papulix"


def _obj(d, key: str, where: str) -> dict:
    v = d.get(key) if isinstance(d, dict) else None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _grouped(d: dict, where: str, groups: str) -> tuple:
    heads, n = _int(d, "heads", where), _int(d, groups, where)
    if heads % n:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {n} {groups}")
    return heads, n


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float

    @staticmethod
    def from_dict(d: dict, where: str) -> "AttentionConfig":
        heads, kv = _grouped(d, where, "kv_heads")
        return AttentionConfig(heads, kv, _int(d, "dim", where), _int(d, "vdim", where), _float(d, "scale", where))


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @staticmethod
    def from_dict(d: dict, where: str) -> "ChannelDeltaConfig":
        heads, kv = _grouped(d, where, "kv_heads")
        return ChannelDeltaConfig(heads, kv, _int(d, "dim", where), _int(d, "vdim", where), _int(d, "conv", where))


@dataclass(frozen=True)
class StateSpaceConfig:
    """The mixer of a "mamba2" layer."""
    heads: int
    groups: int
    vdim: int
    state: int
    norm_groups: int
    conv: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """What passes the convolution: x, B and C."""
        return self.inner + 2 * self.groups * self.state

    @staticmethod
    def from_dict(d: dict, where: str) -> "StateSpaceConfig":
        heads, groups = _grouped(d, where, "groups")
        out = StateSpaceConfig(heads, groups, _int(d, "vdim", where), _int(d, "state", where), _int(d, "norm_groups", where),
                               _int(d, "conv", where))
        if out.inner % out.norm_groups:
            raise ConfigError(f"config.json: {where}: norm_groups {out.norm_groups} does not divide {out.inner} channels")
        return out


def _mlp(d, where: str) -> Optional[int]:
    """The width of a dense feed-forward, or None for a layer without one."""
    if d is None:
        return None
    if not isinstance(d, dict) or d.get("kind") != "dense":
        raise ConfigError(f"config.json: {where} must be null or an object of kind 'dense'")
    return _int(d, "ff", where)


@dataclass(frozen=True)
class PapulixLayer:
    type: str
    mixer: object                    # AttentionConfig | ChannelDeltaConfig | StateSpaceConfig
    ff: Optional[int]                # None: no feed-forward


@dataclass(frozen=True)
class PapulixConfig:
    architecture = ARCHITECTURE

    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_scale: float
    streams: int
    layers: tuple
    loop: tuple                      # (start, stop, times): layers start .. stop - 1 run `times` times in a row
    eos_token_ids: tuple = ()
    bos_token_id: Optional[int] = None
    max_positions: int = UNBOUNDED_POSITIONS     # the design has no positional table and no limit of its own

    MIXERS = {"attention": AttentionConfig, "channel_delta": ChannelDeltaConfig, "mamba2": StateSpaceConfig}

    def run_order(self) -> tuple:
        """The layers in the order in which they run."""
        start, stop, times = self.loop
        n = len(self.layers)
        return tuple(range(start)) + tuple(range(start, stop)) * times + tuple(range(stop, n))

    @classmethod
    def from_dict(cls, d: dict) -> "PapulixConfig":
        vocab, width = _int(d, "vocab", "config"), _int(d, "width", "config")
        eps = _float(_obj(d, "norm", "config"), "eps", "norm")
        if not eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        emb = d.get("embedding")
        scale = _float(emb, "scale", "embedding") if isinstance(emb, dict) and emb.get("scale") is not None else 1.0
        logit_scale = _float(d, "logit_scale", "config") if d.get("logit_scale") is not None else 1.0
        streams = _int(d, "streams", "config")
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
            layers.append(PapulixLayer(kind, cls.MIXERS[kind].from_dict(entry["mixer"], where + ".mixer"),
                                       _mlp(entry.get("mlp"), where + ".mlp")))
        loop = (0, 0, 1)
        if d.get("loop") is not None:
            lp = _obj(d, "loop", "config")
            loop = (_int(lp, "start", "loop", 0), _int(lp, "stop", "loop", 0), _int(lp, "times", "loop", 0))
            if not loop[0] <= loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop[0]} .. {loop[1] - 1} of {len(layers)}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else (eos,)))
        return cls(vocab, width, eps, scale, logit_scale, streams, tuple(layers), loop, eos_ids, d.get("bos_token_id"))
