"""Typed configuration of the Fetitar decoder, read from config.json's own keys.

config.json of this architecture is nested: ``layers`` lists the layers in order, each with its ``type`` ("attention" or
"latent_attention"), the mixer's sizes (``mixer``; ``mask.size`` is its window, absent: every earlier key; ``v_mix`` of an attention:
its values take part in the value mixing) and its feed-forward (``mlp``: ``kind`` "dense" with ``ff``; null: none).
``embedding.scale`` multiplies the token embedding, ``embedding.bigram`` (``buckets``, ``mul_prev``, ``mul_cur``) describes the table of
token pairs (absent: none), ``norm.eps`` is every norm's eps, ``vocab`` and ``width`` are the global sizes.  The design states no
position limit: ``max_positions`` is an optional key.  Every size and constant is taken from there; nothing is assumed about
their values.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from ..errors import ConfigError
from .kubedra import _get
from .semanex import DEFAULT_MAX_POSITIONS, _positive


def _window(d, where):
    """The window's size, or None for every earlier key."""
    mask = d.get("mask")
    if not mask:
        return None
    size = _get(mask, "size", int, where + ".mask")
    _positive(where + ".mask", size)
    return size


def _scale(d, where):
    scale = _get(d, "scale", float, where)
    if scale <= 0:
        raise ConfigError(f"config.json: {where}.scale must be positive")
    return scale


@dataclass(frozen=True)
class YarnConfig:
    factor: float
    original: float                       # the length the frequencies were made for
    fast: float                           # turns over that length above which a frequency stays
    slow: float                           # ... and below which it is divided by the factor

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(*(_get(d, key, float, where) for key in ("factor", "original", "fast", "slow")))
        if min(cfg.factor, cfg.original, cfg.fast, cfg.slow) <= 0:
            raise ConfigError(f"config.json: {where}: factor, original, fast and slow must be positive")
        return cfg

    def to_dict(self):
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float
    scaling: Optional[YarnConfig] = None

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(_get(d, "dims", int, where), _get(d, "base", float, where),
                  YarnConfig.from_dict(d["scaling"], where + ".scaling") if d.get("scaling") else None)
        if cfg.dims < 0 or cfg.dims % 2 or cfg.base <= 1:
            raise ConfigError(f"config.json: {where}: dims must be even and base above 1")
        return cfg

    def to_dict(self):
        return {"dims": self.dims, "base": self.base, **({"scaling": self.scaling.to_dict()} if self.scaling else {})}


@dataclass(frozen=True)
class SlopedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None
    v_mix: bool = False

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(*(_get(d, key, int, where) for key in ("heads", "kv_heads", "dim", "vdim")), _scale(d, where), _window(d, where),
                  bool(d.get("v_mix", False)))
        _positive(where, cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim)
        if cfg.heads % cfg.kv_heads:
            raise ConfigError(f"config.json: {where}: heads must be a multiple of kv_heads")
        return cfg

    def to_dict(self):
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "v_mix": self.v_mix,
                **({"mask": {"size": self.window}} if self.window else {})}


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int                              # unrotated query/key channels per head
    rot_dim: int                          # rotated ones, their keys shared by the heads
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotationConfig
    window: Optional[int] = None

    @classmethod
    def from_dict(cls, d, where):
        if not isinstance(d.get("rot"), dict):
            raise ConfigError(f"config.json: {where} lacks its rotation")
        cfg = cls(*(_get(d, key, int, where) for key in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")), _scale(d, where),
                  RotationConfig.from_dict(d["rot"], where + ".rot"), _window(d, where))
        _positive(where, cfg.heads, cfg.dim, cfg.rot_dim, cfg.vdim, cfg.q_rank, cfg.kv_rank)
        if cfg.rot.dims > cfg.rot_dim:
            raise ConfigError(f"config.json: {where}.rot: {cfg.rot.dims} rotated channels of {cfg.rot_dim}")
        return cfg

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": self.rot.to_dict(),
                **({"mask": {"size": self.window}} if self.window else {})}


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(*(_get(d, key, int, where) for key in ("buckets", "mul_prev", "mul_cur")))
        _positive(where, cfg.buckets)
        return cfg

    def to_dict(self):
        return {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}


_MIXERS = {"attention": SlopedAttentionConfig, "latent_attention": LatentConfig}


@dataclass(frozen=True)
class FetitarLayerConfig:
    type: str
    mixer: object
    ff: Optional[int]                     # the feed-forward's hidden width; None: no feed-forward

    @classmethod
    def from_dict(cls, d, where):
        kind = _get(d, "type", str, where)
        if kind not in _MIXERS:
            raise ConfigError(f"config.json: {where}.type = {kind!r}; known: {sorted(_MIXERS)}")
        if not isinstance(d.get("mixer"), dict):
            raise ConfigError(f"config.json: {where} lacks its mixer's sizes")
        ff = None
        if d.get("mlp"):
            if _get(d["mlp"], "kind", str, where + ".mlp") != "dense":
                raise ConfigError(f"config.json: {where}.mlp.kind = {d['mlp']['kind']!r}; known: 'dense'")
            ff = _get(d["mlp"], "ff", int, where + ".mlp")
            _positive(where + ".mlp", ff)
        return cls(kind, _MIXERS[kind].from_dict(d["mixer"], where + ".mixer"), ff)

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": {"kind": "dense", "ff": self.ff} if self.ff else None}


@dataclass(frozen=True)
class FetitarConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple                         # of FetitarLayerConfig
    embedding_scale: float = 1.0
    bigram: Optional[BigramConfig] = None
    max_positions: Optional[int] = None
    bos_token_id: Optional[int] = None
    eos_token_id: tuple = ()
    architecture: str = "Fetitar"

    @classmethod
    def from_dict(cls, d):
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks its list of layers")
        eos = d.get("eos_token_id")
        eos = () if eos is None else tuple(int(t) for t in (eos if isinstance(eos, (list, tuple)) else [eos]))
        embedding = d.get("embedding") or {}
        cfg = cls(_get(d, "vocab", int, "config"), _get(d, "width", int, "config"), _get(d.get("norm"), "eps", float, "norm"),
                  tuple(FetitarLayerConfig.from_dict(layer, f"layers[{i}]") for i, layer in enumerate(layers)),
                  _get(embedding, "scale", float, "embedding", default=1.0, required=False),
                  BigramConfig.from_dict(embedding["bigram"], "embedding.bigram") if embedding.get("bigram") else None,
                  _get(d, "max_positions", int, "config", required=False), _get(d, "bos_token_id", int, "config", required=False), eos)
        if min(cfg.vocab, cfg.width) <= 0 or cfg.eps <= 0 or (cfg.max_positions is not None and cfg.max_positions <= 0):
            raise ConfigError("config.json: vocab, width, norm.eps and max_positions must be positive")
        shapes = {(layer.mixer.kv_heads, layer.mixer.vdim) for layer in cfg.layers if layer.type == "attention" and layer.mixer.v_mix}
        if len(shapes) > 1:
            raise ConfigError("config.json: layers whose values mix have the same kv_heads and vdim")
        return cfg

    def to_dict(self):
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "embedding": {"scale": self.embedding_scale, **({"bigram": self.bigram.to_dict()} if self.bigram else {})},
               "layers": [layer.to_dict() for layer in self.layers]}
        if self.max_positions is not None:
            out["max_positions"] = self.max_positions
        if self.bos_token_id is not None:
            out["bos_token_id"] = self.bos_token_id
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out

    def positions(self):
        return self.max_positions or DEFAULT_MAX_POSITIONS
