"""The Saposun decoder as a model spec.

Every layer is one sum, x <- x + m (mixer(h) + ff(h)) with h = norm1(x): both sublayers read the output of the
layer's only norm.  Mixers: ``latent_attention`` (a window, no sink and no gate; a layer may read the latents that an
earlier layer cached), ``retention`` (a linear attention with a fixed decay per head, rotated queries and keys and a
gated norm of the result without a weight) or ``attention`` (short filters over the projections, values of unit root
mean square, soft-capped scores, a window beside which the blocks before it are seen by their means, a gate per head).
The feed-forward is a mixture of gated experts, chosen by corrected softmax scores and weighted by the scores
themselves, or absent.
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.base import Architecture, register_architecture
from ..config.saposun import SaposunAttention, SaposunConfig, SaposunLatent, SaposunRetention
from ..parts import latent_attention as _latent, linear_attention as _linear_attention, routed as _routed   # register the kinds  # noqa: F401
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

_LATENT_NAMES = dict(dq="dq", dq_norm="dq.norm", uq="uq", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", o="o")
_RETENTION_NAMES = dict(q="q", k="k", v="v", gate="g", o="o")
_ATTENTION_NAMES = dict(q="q", k="k", v="v", q_conv="q.conv", k_conv="k.conv", v_conv="v.conv", gate="g", o="o")
_EXPERT_NAMES = dict(gate="gate", up="up", down="down", expert="e{i}.", router="router", correction="correction")


def _latent_spec(cfg: SaposunConfig, m: SaposunLatent) -> PartSpec:
    return PartSpec("latent_attention", {
        "width": cfg.width, "heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_dim": m.vdim, "q_rank": m.q_rank,
        "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps,
        "position": PartSpec("rotary_pairs", {"head_dim": m.rot_dim, "dims": m.rot_dim, "theta": m.rot_base, "pairing": "neighbours"}),
        "window": m.mask_size, "sink": False, "gate": None, "own_kv": m.kv_from is None, "names": _LATENT_NAMES})


def _retention_spec(cfg: SaposunConfig, m: SaposunRetention) -> PartSpec:
    return PartSpec("retention", {
        "width": cfg.width, "heads": m.heads, "head_dim": m.dim, "v_dim": m.vdim, "decay": m.decay, "eps": cfg.norm_eps,
        "position": PartSpec("rotary_pairs", {"head_dim": m.dim, "dims": m.rot_dims, "theta": m.rot_base, "pairing": "halves"}),
        "names": _RETENTION_NAMES})


def _attention_spec(cfg: SaposunConfig, m: SaposunAttention) -> PartSpec:
    return PartSpec("attention", {
        "width": cfg.width, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim, "scale": m.scale,
        "bias": False, "qk_norm": None, "eps": cfg.norm_eps, "conv": m.conv, "value_norm": True, "soft_cap": m.softcap, "gate": "head",
        "position": PartSpec("rotary_pairs", {"head_dim": m.dim, "dims": m.rot_dims, "theta": m.rot_base, "pairing": "halves"}),
        "mask": None if m.mask_size is None else {"kind": "window", "size": m.mask_size, "pool": m.pool}, "names": _ATTENTION_NAMES})


_SPECS = {"latent_attention": _latent_spec, "retention": _retention_spec, "attention": _attention_spec}


def build_spec(cfg: SaposunConfig) -> ModelSpec:
    norm = PartSpec("rms", {"width": cfg.width, "eps": cfg.norm_eps, "tensor": ""})
    layers = []
    for i, L in enumerate(cfg.layers):
        ffn = PartSpec("none") if L.mlp is None else PartSpec("routed_moe", {
            "width": cfg.width, "experts": L.mlp.experts, "top": L.mlp.top, "intermediate": L.mlp.ff, "scores": "softmax",
            "correction": True, "renormalize": False, "expert": "gated", "names": _EXPERT_NAMES})
        layers.append(LayerSpec(block=PartSpec("parallel_residual", {"width": cfg.width, "factor": cfg.residual_mult}),
                                mixer=_SPECS[L.type](cfg, L.mixer), mixer_norm=norm, ffn=ffn, ffn_norm=PartSpec("none"), prefix=f"l{i}.",
                                names={"mixer": "mix.", "mixer_norm": "norm1", "ffn": "mlp.", "ffn_norm": ""}))
    spec = ModelSpec(
        architecture=cfg.architecture, vocab=cfg.vocab_size, width=cfg.width, max_position=cfg.max_position,
        embedding=PartSpec("table", {"vocab": cfg.vocab_size, "width": cfg.width, "tensor": ""}), embedding_prefix="embed",
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i, read_cache_of=getattr(L.mixer, "kv_from", None)) for i, L in enumerate(cfg.layers)),
        final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear", {"vocab": cfg.vocab_size, "width": cfg.width, "tied": False, "tensor": ""}), head_prefix="head")
    spec.validate()
    return spec


SAPOSUN = register_architecture(Architecture(names=("Saposun", "saposun"), config_cls=SaposunConfig, build_spec=build_spec))
