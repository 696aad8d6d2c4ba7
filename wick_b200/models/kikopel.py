"""The Kikopel decoder as a model spec.

The embedding's rows are multiplied by a factor and a row of a pair table joins them, chosen by the token and the one
before it.  The sublayers read the stream itself and their results are normed (by one number instead of a weight
vector) and multiplied by a factor before they join it: x <- x + m norm1(mixer(x)), then x <- x + m norm2(ff(x)).
Mixers: ``latent_attention`` (a window, no sink, an output gate per element, a rotated part of half-split pairs) or
``hgrn2`` (a linear attention whose forget factor, bounded below per channel, also says how much is written).  The
feed-forward has one inner matrix and the PolyNorm activation, or is absent.
Tensor names: ``embed``, ``bigram``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.base import Architecture, register_architecture
from ..config.kikopel import KikopelConfig
from ..parts import latent_attention as _latent, linear_attention as _linear_attention   # register the kinds  # noqa: F401
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

_LATENT_NAMES = dict(dq="dq", dq_norm="dq.norm", uq="uq", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", gate="g", o="o")
_HGRN2_NAMES = dict(q="q", forget="f", forget_bias="f.b", lower="lower", v="v", norm="norm", o="o")


def build_spec(cfg: KikopelConfig) -> ModelSpec:
    def norm(factor=1.0, optional=False):
        return PartSpec("rms", {"width": cfg.width, "eps": cfg.norm_eps, "tensor": "", "one_number": True, "factor": factor,
                                "optional": optional})

    layers = []
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        if L.type == "latent_attention":
            mixer = PartSpec("latent_attention", {
                "width": cfg.width, "heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_dim": m.vdim,
                "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps,
                "position": PartSpec("rotary_pairs", {"head_dim": m.rot_dim, "dims": m.rot_dim, "theta": m.rot_base,
                                                      "pairing": "halves"}),
                "window": m.mask_size, "sink": False, "gate": "element", "names": _LATENT_NAMES})
        else:
            mixer = PartSpec("hgrn2", {"width": cfg.width, "heads": m.heads, "head_dim": m.dim, "v_dim": m.vdim,
                                       "eps": cfg.norm_eps, "names": _HGRN2_NAMES})
        ffn = PartSpec("none") if L.ff is None else PartSpec("mlp", {
            "width": cfg.width, "intermediate": L.ff, "activation": "poly_norm", "eps": cfg.norm_eps,
            "names": {"up": "up", "down": "down", "coefficients": "act"}})
        layers.append(LayerSpec(block=PartSpec("normed_sum_residual"), mixer=mixer, mixer_norm=norm(cfg.residual_mult), ffn=ffn,
                                ffn_norm=norm(cfg.residual_mult, optional=L.ff is None), prefix=f"l{i}.",
                                names={"mixer": "mix.", "mixer_norm": "norm1", "ffn": "mlp.", "ffn_norm": "norm2"}))
    pairs = None
    if cfg.bigram is not None:
        pairs = {"tensor": "bigram", "buckets": cfg.bigram.buckets, "mul_prev": cfg.bigram.mul_prev, "mul_cur": cfg.bigram.mul_cur}
    spec = ModelSpec(
        architecture=cfg.architecture, vocab=cfg.vocab_size, width=cfg.width, max_position=cfg.max_position,
        embedding=PartSpec("table", {"vocab": cfg.vocab_size, "width": cfg.width, "tensor": "embed", "scale": cfg.embedding_scale,
                                     "pairs": pairs}),
        embedding_prefix="", layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm(), final_norm_prefix="final.norm",
        head=PartSpec("linear", {"vocab": cfg.vocab_size, "width": cfg.width, "tied": False, "tensor": ""}), head_prefix="head")
    spec.validate()
    return spec


KIKOPEL = register_architecture(Architecture(names=("Kikopel", "kikopel"), config_cls=KikopelConfig, build_spec=build_spec))
