"""Typed configuration of the Semanex decoder, read from config.json's own keys.

config.json of this architecture is nested: ``layers`` lists the layers in order, each with its ``type`` ("latent_attention" or
"parallel"), the mixer's sizes (``mixer``; a parallel layer's has ``left``, ``right`` and their weights ``left_scale``,
``right_scale``) and its feed-forward (``mlp``: ``kind`` "dense" with ``ff``; null: none).  ``canon.taps`` is the length of the
convolution in front of every mixer, ``postln_alpha`` the stream's factor in every sum, ``embedding.scale`` multiplies the
embedding, ``norm.eps`` is every norm's eps, ``vocab`` and ``width`` are the global sizes.  The design states no position limit:
``max_positions`` is an optional key.  Every size and constant is taken from there; nothing is assumed about their values.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from ..errors import ConfigError
from .kubedra import _get

DEFAULT_MAX_POSITIONS = 65536


def _positive(where, *sizes):
    if min(sizes) <= 0:
        raise ConfigError(f"config.json: {where}: sizes must be positive")


@dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(_get(d, "dims", int, where), _get(d, "base", float, where))
        if cfg.dims < 0 or cfg.dims % 2 or cfg.base <= 0:
            raise ConfigError(f"config.json: {where}: dims must be even and base positive")
        return cfg

    def to_dict(self):
        return {"dims": self.dims, "base": self.base}


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

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(*(_get(d, key, int, where) for key in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")),
                  _get(d, "scale", float, where), RotationConfig.from_dict(d.get("rot"), where + ".rot"))
        _positive(where, cfg.heads, cfg.dim, cfg.rot_dim, cfg.vdim, cfg.q_rank, cfg.kv_rank)
        if cfg.rot.dims > cfg.rot_dim:
            raise ConfigError(f"config.json: {where}.rot: {cfg.rot.dims} rotated channels of {cfg.rot_dim}")
        if cfg.scale <= 0:
            raise ConfigError(f"config.json: {where}.scale must be positive")
        return cfg

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class CappedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float] = None       # None: scores are not capped

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(*(_get(d, key, int, where) for key in ("heads", "kv_heads", "dim", "vdim")), _get(d, "scale", float, where),
                  _get(d, "softcap", float, where, required=False))
        _positive(where, cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim)
        if cfg.heads % cfg.kv_heads:
            raise ConfigError(f"config.json: {where}: heads must be a multiple of kv_heads")
        if cfg.scale <= 0 or (cfg.softcap is not None and cfg.softcap <= 0):
            raise ConfigError(f"config.json: {where}: scale and softcap must be positive")
        return cfg

    def to_dict(self):
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        return out


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int                             # value channels per head
    state: int
    groups: int                           # heads of a group share B and C
    conv: int                             # taps of the short convolution
    norm_groups: int

    @classmethod
    def from_dict(cls, d, where):
        cfg = cls(*(_get(d, key, int, where) for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        _positive(where, cfg.heads, cfg.vdim, cfg.state, cfg.groups, cfg.conv, cfg.norm_groups)
        if cfg.heads % cfg.groups or (cfg.heads * cfg.vdim) % cfg.norm_groups:
            raise ConfigError(f"config.json: {where}: heads must be a multiple of groups, heads * vdim of norm_groups")
        return cfg

    def to_dict(self):
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class ParallelConfig:
    left: CappedAttentionConfig
    right: StateSpaceConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d, where):
        if not isinstance(d.get("left"), dict) or not isinstance(d.get("right"), dict):
            raise ConfigError(f"config.json: {where} lacks its left or right mixer")
        return cls(CappedAttentionConfig.from_dict(d["left"], where + ".left"), StateSpaceConfig.from_dict(d["right"], where + ".right"),
                   _get(d, "left_scale", float, where), _get(d, "right_scale", float, where))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}


_MIXERS = {"latent_attention": LatentConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class SemanexLayerConfig:
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
class SemanexConfig:
    vocab: int
    width: int
    eps: float
    alpha: float                          # postln_alpha
    taps: int                             # canon.taps
    layers: tuple                         # of SemanexLayerConfig
    embedding_scale: float = 1.0
    max_positions: Optional[int] = None
    bos_token_id: Optional[int] = None
    eos_token_id: tuple = ()
    architecture: str = "Semanex"

    @classmethod
    def from_dict(cls, d):
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks its list of layers")
        eos = d.get("eos_token_id")
        eos = () if eos is None else tuple(int(t) for t in (eos if isinstance(eos, (list, tuple)) else [eos]))
        cfg = cls(_get(d, "vocab", int, "config"), _get(d, "width", int, "config"), _get(d.get("norm"), "eps", float, "norm"),
                  _get(d, "postln_alpha", float, "config"), _get(d.get("canon"), "taps", int, "canon"),
                  tuple(SemanexLayerConfig.from_dict(layer, f"layers[{i}]") for i, layer in enumerate(layers)),
                  _get(d.get("embedding"), "scale", float, "embedding", default=1.0, required=False),
                  _get(d, "max_positions", int, "config", required=False), _get(d, "bos_token_id", int, "config", required=False), eos)
        if min(cfg.vocab, cfg.width, cfg.taps) <= 0 or cfg.eps <= 0 or (cfg.max_positions is not None and cfg.max_positions <= 0):
            raise ConfigError("config.json: vocab, width, norm.eps, canon.taps and max_positions must be positive")
        return cfg

    def to_dict(self):
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "postln_alpha": self.alpha, "canon": {"taps": self.taps}, "embedding": {"scale": self.embedding_scale},
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
