"""Configuration of the Saposun decoder, from its ``config.json``.

``config.json`` lists the layers one by one (``layers``: ``type``, the mixer's sizes and
constants under ``mixer``, the experts under ``mlp`` or null), and model-wide ``vocab``,
``width``, ``norm.eps`` and ``residual_mult``.  Layer types: ``latent_attention`` (``heads``,
``dim``, ``rot_dim``, ``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot``, ``mask.size``; with ``kv_from``
the number of an earlier layer whose latent it reads), ``retention`` (``heads``, ``dim``, ``vdim``,
``rot``, ``decay``: a number per head) and ``attention`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``,
``rot``, ``conv`` taps, ``softcap``, ``mask.size`` and ``mask.pool``).  The feed-forward is ``moe``: ``expert.ff``,
``router.experts``, ``router.top``.
Nothing here has a default that stands for a size: what the file does not give is an error, except
the options a model may leave out (``mlp``, ``kv_from``, ``mask``, ``mask.pool``, ``conv``, ``softcap``).
"""
from __future__ import annotations

import dataclasses
import math
from typing import Any, Dict, Mapping, Optional, Tuple

from .base import ConfigError, ModelConfig


def _num(j: Any, key: str, where: str, kind=float, positive: bool = True):
    v = j.get(key) if isinstance(j, Mapping) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (kind is int and int(v) != v) or not math.isfinite(v):
        raise ConfigError(f"config.json: {where}{key} is missing or no number")
    if positive and v <= 0:
        raise ConfigError(f"config.json: {where}{key} must be positive")
    return kind(v)


def _optional(j: Mapping[str, Any], key: str, where: str, kind=float, positive: bool = True):
    return None if j.get(key) is None else _num(j, key, where, kind, positive)


def _rotation(j: Mapping[str, Any], where: str, most: int) -> Tuple[float, int]:
    """(base, rotated elements of a head); at most ``most`` of them."""
    base, dims = _num(j.get("rot"), "base", where + "rot."), _num(j.get("rot"), "dims", where + "rot.", int)
    if dims % 2 != 0 or dims > most:
        raise ConfigError(f"config.json: {where}rot.dims must be even and at most {most}")
    return base, dims


@dataclasses.dataclass(frozen=True)
class SaposunLatent:
    heads: int
    dim: int                               # unrotated query / key elements of a head
    rot_dim: int                           # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    mask_size: Optional[int] = None        # of the window; None: every earlier position is seen
    kv_from: Optional[int] = None          # the layer whose latents and rotated key parts are read

    @classmethod
    def from_json(cls, j: Any, where: str) -> "SaposunLatent":
        if not isinstance(j, Mapping):
            raise ConfigError(f"config.json: {where[:-1]} is missing")
        rot_dim = _num(j, "rot_dim", where, int)
        base, dims = _rotation(j, where, rot_dim)
        if dims != rot_dim:
            raise ConfigError(f"config.json: {where}rot.dims must be rot_dim")
        return cls(heads=_num(j, "heads", where, int), dim=_num(j, "dim", where, int), rot_dim=rot_dim, vdim=_num(j, "vdim", where, int),
                   q_rank=_num(j, "q_rank", where, int), kv_rank=_num(j, "kv_rank", where, int), scale=_num(j, "scale", where, positive=False),
                   rot_base=base, mask_size=_num(j["mask"], "size", where + "mask.", int) if j.get("mask") is not None else None,
                   kv_from=_optional(j, "kv_from", where, int, positive=False))

    def to_json(self) -> Dict[str, Any]:
        j = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
             "kv_rank": self.kv_rank, "scale": self.scale, "rot": {"base": self.rot_base, "dims": self.rot_dim}}
        if self.mask_size is not None:
            j["mask"] = {"size": self.mask_size}
        if self.kv_from is not None:
            j["kv_from"] = self.kv_from
        return j


@dataclasses.dataclass(frozen=True)
class SaposunRetention:
    heads: int
    dim: int                               # key channels of a head
    vdim: int                              # value numbers of a head
    rot_base: float
    rot_dims: int                          # rotated elements of a query / key head, from the first
    decay: Tuple[float, ...] = ()          # a number per head

    @classmethod
    def from_json(cls, j: Any, where: str) -> "SaposunRetention":
        if not isinstance(j, Mapping):
            raise ConfigError(f"config.json: {where[:-1]} is missing")
        heads, dim = _num(j, "heads", where, int), _num(j, "dim", where, int)
        base, dims = _rotation(j, where, dim)
        decay = j.get("decay")
        if (not isinstance(decay, list) or len(decay) != heads
                or any(isinstance(a, bool) or not isinstance(a, (int, float)) or not math.isfinite(a) for a in decay)):
            raise ConfigError(f"config.json: {where}decay must list a number for each of the {heads} heads")
        return cls(heads=heads, dim=dim, vdim=_num(j, "vdim", where, int), rot_base=base, rot_dims=dims, decay=tuple(float(a) for a in decay))

    def to_json(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "rot": {"base": self.rot_base, "dims": self.rot_dims},
                "decay": list(self.decay)}


@dataclasses.dataclass(frozen=True)
class SaposunAttention:
    heads: int
    kv_heads: int
    dim: int                               # size of a query / key head
    vdim: int                              # size of a value head
    scale: float
    rot_base: float
    rot_dims: int
    conv: Optional[int] = None             # taps of the short filters of q, k and v; None: there are none
    softcap: Optional[float] = None        # scores s become softcap tanh(s / softcap)
    mask_size: Optional[int] = None        # of the window; None: every earlier position is seen
    pool: Optional[int] = None             # positions of a block that is seen by its mean once it lies before the window

    @classmethod
    def from_json(cls, j: Any, where: str) -> "SaposunAttention":
        if not isinstance(j, Mapping):
            raise ConfigError(f"config.json: {where[:-1]} is missing")
        dim = _num(j, "dim", where, int)
        base, dims = _rotation(j, where, dim)
        mask = j.get("mask")
        a = cls(heads=_num(j, "heads", where, int), kv_heads=_num(j, "kv_heads", where, int), dim=dim, vdim=_num(j, "vdim", where, int),
                scale=_num(j, "scale", where, positive=False), rot_base=base, rot_dims=dims, conv=_optional(j, "conv", where, int),
                softcap=_optional(j, "softcap", where),
                mask_size=_num(mask, "size", where + "mask.", int) if mask is not None else None,
                pool=_optional(mask, "pool", where + "mask.", int) if isinstance(mask, Mapping) else None)
        if a.heads % a.kv_heads != 0:
            raise ConfigError(f"config.json: {where}heads must be a multiple of kv_heads")
        return a

    def to_json(self) -> Dict[str, Any]:
        j: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                             "rot": {"base": self.rot_base, "dims": self.rot_dims}}
        if self.conv is not None:
            j["conv"] = self.conv
        if self.softcap is not None:
            j["softcap"] = self.softcap
        if self.mask_size is not None:
            j["mask"] = {"size": self.mask_size}
            if self.pool is not None:
                j["mask"]["pool"] = self.pool
        return j


@dataclasses.dataclass(frozen=True)
class SaposunExperts:
    ff: int                                # inner size of every expert
    experts: int
    top: int

    @classmethod
    def from_json(cls, j: Mapping[str, Any], where: str) -> "SaposunExperts":
        kind = j.get("kind") if isinstance(j, Mapping) else None
        if kind != "moe":
            raise ConfigError(f"config.json: {where}kind {kind!r} is not known (moe)")
        r = j.get("router")
        m = cls(_num(j.get("expert"), "ff", where + "expert.", int), experts=_num(r, "experts", where + "router.", int),
                top=_num(r, "top", where + "router.", int))
        if m.top > m.experts:
            raise ConfigError(f"config.json: {where}router.top is larger than the number of experts")
        return m

    def to_json(self) -> Dict[str, Any]:
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


_MIXERS = {"latent_attention": SaposunLatent, "retention": SaposunRetention, "attention": SaposunAttention}


@dataclasses.dataclass(frozen=True)
class SaposunLayer:
    type: str                                              # a key of _MIXERS
    mixer: Any
    mlp: Optional[SaposunExperts]


@dataclasses.dataclass(frozen=True)
class SaposunConfig(ModelConfig):
    vocab_size: int = 0
    width: int = 0
    layers: Tuple[SaposunLayer, ...] = ()
    norm_eps: float = 1e-6
    residual_mult: float = 1.0

    @property
    def vocab(self) -> int:
        return self.vocab_size

    @property
    def max_position(self) -> int:
        return 1 << 24                     # (positions enter a float32 angle: integers are exact up to here)

    def param_count(self, tied: Optional[bool] = None) -> int:
        """Number of parameters (every expert counted)."""
        w = self.width
        n = 2 * self.vocab_size * w + w
        for L in self.layers:
            m = L.mixer
            n += w
            if L.type == "latent_attention":
                n += m.q_rank * (w + 1 + m.heads * (m.dim + m.rot_dim)) + m.heads * (m.dim + m.vdim) * m.kv_rank + w * m.heads * m.vdim
                if m.kv_from is None:
                    n += (m.kv_rank + m.rot_dim) * w + m.kv_rank
            elif L.type == "retention":
                n += w * m.heads * (2 * m.dim + 3 * m.vdim)
            else:
                n += (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)) * (w + (m.conv or 0)) + m.heads * w + w * m.heads * m.vdim
            if L.mlp is not None:
                n += 3 * w * L.mlp.ff * L.mlp.experts + (w + 1) * L.mlp.experts
        return n

    @classmethod
    def from_json(cls, j: Mapping[str, Any], architecture: str) -> "SaposunConfig":
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: layers is missing or empty")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            kind = L.get("type") if isinstance(L, Mapping) else L
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is not known ({', '.join(sorted(_MIXERS))})")
            mixer = _MIXERS[kind].from_json(L.get("mixer"), where + "mixer.")
            if kind == "latent_attention" and mixer.kv_from is not None:
                src = layers[mixer.kv_from] if 0 <= mixer.kv_from < i else None
                if src is None or src.type != "latent_attention" or src.mixer.kv_from is not None:
                    raise ConfigError(f"config.json: {where}mixer.kv_from must name an earlier layer with latents of its own")
                s = src.mixer
                if (s.kv_rank, s.rot_dim, s.rot_base) != (mixer.kv_rank, mixer.rot_dim, mixer.rot_base):
                    raise ConfigError(f"config.json: {where}mixer reads layer {mixer.kv_from}, whose latent or rotation differs")
            mlp = L.get("mlp")
            layers.append(SaposunLayer(kind, mixer, SaposunExperts.from_json(mlp, where + "mlp.") if mlp is not None else None))
        return cls(architecture=architecture, vocab_size=_num(j, "vocab", "", int), width=_num(j, "width", "", int), layers=tuple(layers),
                   norm_eps=_num(j.get("norm"), "eps", "norm."), residual_mult=_num(j, "residual_mult", "", positive=False))

    def to_json(self) -> Dict[str, Any]:
        return {"architecture": self.architecture,
                "layers": [{"type": L.type, "mixer": L.mixer.to_json(), "mlp": L.mlp.to_json() if L.mlp is not None else None}
                           for L in self.layers],
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab_size, "width": self.width}
