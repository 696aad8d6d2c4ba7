"""Configuration of the Kikopel decoder, from its ``config.json``.

``config.json`` lists the layers one by one (``layers``: ``type``, the mixer's sizes and
constants under ``mixer``, the feed-forward under ``mlp`` or null), and model-wide ``vocab``,
``width``, ``norm.eps``, ``residual_mult``, ``embedding.scale`` and ``embedding.bigram``
(``buckets``, ``mul_prev``, ``mul_cur``).  Layer types: ``latent_attention`` (``heads``, ``dim``,
``rot_dim``, ``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot``: ``base``, ``dims``;
``mask``: ``size``) and ``hgrn2`` (``heads``, ``dim``, ``vdim``).  Feed-forwards: ``dense`` (``ff``).
Nothing here has a default that stands for a size: what the file does not give is an error, except
the options a model may leave out (``mlp``, ``mask``, ``embedding``, ``embedding.bigram``, ``residual_mult``).
"""
from __future__ import annotations

import dataclasses
import math
from typing import Any, Dict, Mapping, Optional, Tuple

from .base import ConfigError, ModelConfig


def _num(j: Any, key: str, where: str, kind=float, positive: bool = True):
    v = j.get(key) if isinstance(j, Mapping) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or (kind is int and int(v) != v):
        raise ConfigError(f"config.json: {where}{key} is missing or no number")
    if positive and v <= 0:
        raise ConfigError(f"config.json: {where}{key} must be positive")
    return kind(v)


@dataclasses.dataclass(frozen=True)
class KikopelLatentAttention:
    heads: int
    dim: int                               # unrotated query / key numbers of a head
    rot_dim: int                           # rotated ones; the keys' are shared by the heads
    vdim: int                              # size of a value head
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    mask_size: Optional[int] = None        # positions a token sees, itself included; None: all before it

    @classmethod
    def from_json(cls, j: Any, where: str) -> "KikopelLatentAttention":
        if not isinstance(j, Mapping):
            raise ConfigError(f"config.json: {where[:-1]} is missing")
        mask, rot = j.get("mask"), j.get("rot")
        a = cls(heads=_num(j, "heads", where, int), dim=_num(j, "dim", where, int), rot_dim=_num(j, "rot_dim", where, int),
                vdim=_num(j, "vdim", where, int), q_rank=_num(j, "q_rank", where, int), kv_rank=_num(j, "kv_rank", where, int),
                scale=_num(j, "scale", where, positive=False), rot_base=_num(rot, "base", where + "rot."),
                mask_size=_num(mask, "size", where + "mask.", int) if mask is not None else None)
        if a.rot_dim % 2 != 0:
            raise ConfigError(f"config.json: {where}rot_dim must be even")
        if rot.get("dims") is not None and _num(rot, "dims", where + "rot.", int) != a.rot_dim:
            raise ConfigError(f"config.json: {where}rot.dims differs from rot_dim: the whole rotated part turns")
        return a

    def to_json(self) -> Dict[str, Any]:
        j = dataclasses.asdict(self)
        j["rot"] = {"base": j.pop("rot_base"), "dims": self.rot_dim}
        size = j.pop("mask_size")
        if size is not None:
            j["mask"] = {"size": size}
        return j


@dataclasses.dataclass(frozen=True)
class KikopelHgrn2:
    heads: int
    dim: int                               # key channels of a head
    vdim: int                              # value numbers of a head

    @classmethod
    def from_json(cls, j: Any, where: str) -> "KikopelHgrn2":
        if not isinstance(j, Mapping):
            raise ConfigError(f"config.json: {where[:-1]} is missing")
        return cls(*(_num(j, k, where, int) for k in ("heads", "dim", "vdim")))

    def to_json(self) -> Dict[str, Any]:
        return dataclasses.asdict(self)


_MIXERS = {"latent_attention": KikopelLatentAttention, "hgrn2": KikopelHgrn2}


@dataclasses.dataclass(frozen=True)
class KikopelLayer:
    type: str                              # a key of _MIXERS
    mixer: Any
    ff: Optional[int]                      # inner size of the feed-forward; None: the layer has none


@dataclasses.dataclass(frozen=True)
class KikopelBigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclasses.dataclass(frozen=True)
class KikopelConfig(ModelConfig):
    vocab_size: int = 0
    width: int = 0
    layers: Tuple[KikopelLayer, ...] = ()
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    bigram: Optional[KikopelBigram] = None

    @property
    def vocab(self) -> int:
        return self.vocab_size

    @property
    def max_position(self) -> int:
        return 1 << 24                     # (positions enter a float32 angle: integers are exact up to here)

    def param_count(self, tied: Optional[bool] = None) -> int:
        w = self.width
        n = 2 * self.vocab_size * w + 1 + ((self.bigram.buckets + 1) * w if self.bigram is not None else 0)
        for L in self.layers:
            m = L.mixer
            n += 1
            if L.type == "latent_attention":
                n += w * (m.q_rank + m.kv_rank + m.rot_dim + 2 * m.heads * m.vdim) + m.q_rank + m.kv_rank
                n += m.heads * ((m.dim + m.rot_dim) * m.q_rank + (m.dim + m.vdim) * m.kv_rank)
            else:
                n += w * m.heads * (2 * m.dim + 2 * m.vdim) + 2 * m.heads * m.dim + m.vdim
            if L.ff is not None:
                n += 1 + 2 * w * L.ff + 4
        return n

    @classmethod
    def from_json(cls, j: Mapping[str, Any], architecture: str) -> "KikopelConfig":
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: layers is missing or empty")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            kind = L.get("type") if isinstance(L, Mapping) else L
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is not known ({', '.join(_MIXERS)})")
            mlp, ff = L.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind is not known (dense)")
                ff = _num(mlp, "ff", where + "mlp.", int)
            layers.append(KikopelLayer(kind, _MIXERS[kind].from_json(L.get("mixer"), where + "mixer."), ff))
        emb = j.get("embedding")
        emb = emb if emb is not None else {}
        pair = emb.get("bigram")
        if pair is not None:
            where = "embedding.bigram."
            pair = KikopelBigram(_num(pair, "buckets", where, int), _num(pair, "mul_prev", where, int, positive=False),
                                 _num(pair, "mul_cur", where, int, positive=False))
            if pair.mul_prev < 0 or pair.mul_cur < 0:
                raise ConfigError("config.json: embedding.bigram's factors must not be negative")
        return cls(architecture=architecture, vocab_size=_num(j, "vocab", "", int), width=_num(j, "width", "", int),
                   layers=tuple(layers), norm_eps=_num(j.get("norm"), "eps", "norm."),
                   residual_mult=_num(j, "residual_mult", "", positive=False) if j.get("residual_mult") is not None else 1.0,
                   embedding_scale=_num(emb, "scale", "embedding.", positive=False) if emb.get("scale") is not None else 1.0,
                   bigram=pair)

    def to_json(self) -> Dict[str, Any]:
        emb: Dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = dataclasses.asdict(self.bigram)
        return {"architecture": self.architecture, "embedding": emb,
                "layers": [{"type": L.type, "mixer": L.mixer.to_json(),
                            "mlp": {"kind": "dense", "ff": L.ff} if L.ff is not None else None} for L in self.layers],
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab_size, "width": self.width}
