"""The Saposun decoder and its mechanisms against the plain implementation in ``tests/plain/saposun_plain.py``: every
mechanism alone through its part or kernel, then whole models through the engine (prompts, decoding, portions, batches,
reused pages, slots and records, far tokens, window and block edges, generation).  The configurations differ from each other
in every size and option and include the values that make mechanisms vanish or coincide (a factor of one, filters of one
tap and none, blocks of one position, blocks longer than a page and longer than the window, windows of one position and of
more than the prompt, no window, no feed-forward, one head, a decay of one and of zero, widths and head sizes that are no
multiples of four)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

import wick_b200 as wick  # noqa: E402
from wick_b200 import ops  # noqa: E402
from wick_b200.engine.batch import BatchLayout, StepBatch, fill_host  # noqa: E402
from wick_b200.models.spec import PartSpec  # noqa: E402
from wick_b200.parts.base import BuildContext, FeedForward, Hidden, Mixer, build_part  # noqa: E402
from wick_b200.parts import attention as _att, latent_attention as _lat, linear_attention as _gla, routed as _moe  # noqa: E402,F401
from wick_b200.parts.standard import NoNorm, ParallelResidual  # noqa: E402
from wick_b200.weights.safetensors_io import SafeTensorsDir, write_safetensors  # noqa: E402
from helpers import random_tokens, tmp_root  # noqa: E402
from plain import saposun_plain as P  # noqa: E402

PAGE = 64
DEV = "cuda"


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=10000.0, window=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
             rot={"base": base, "dims": rot_dim})
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def ret(heads, dim, vdim, decay, base=10000.0, dims=None):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=decay, rot={"base": base, "dims": dims or dim // 2 * 2})


def att(heads, kv_heads, dim, vdim, scale, window=None, pool=None, conv=None, cap=None, base=10000.0, dims=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot={"base": base, "dims": dims or dim // 2 * 2})
    if window is not None:
        m["mask"] = {"size": window}
        if pool is not None:
            m["mask"]["pool"] = pool
    if conv is not None:
        m["conv"] = conv
    if cap is not None:
        m["softcap"] = cap
    return m


def layer(mixer, ff=None, experts=0, top=0):
    kind = "latent_attention" if "kv_rank" in mixer else ("retention" if "decay" in mixer else "attention")
    mlp = None if ff is None else {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return dict(type=kind, mixer=mixer, mlp=mlp)


# SA: small windows, a reader of other sizes, blocks of three positions
CONFIG_SA = dict(architecture="Saposun", vocab=211, width=64, norm={"eps": 1e-5}, residual_mult=0.35, layers=[
    layer(lat(3, 12, 8, 4, 28, 24, 0.3, 1000.0, 17), 56, 6, 2), layer(att(4, 2, 16, 12, 0.3, 20, 3, 4, 12.0, 700.0, 8), 48, 5, 3),
    layer(ret(3, 8, 4, [0.9, 0.5, 0.999], 300.0, 4), None), layer(lat(4, 8, 8, 12, 16, 24, 0.4, 1000.0, 70, 0), 40, 4, 4),
    layer(att(2, 1, 8, 8, 0.4, 64, 10, 2, 30.0), None), layer(ret(1, 16, 16, [1.0]), 24, 3, 1)])
# SB: a factor of one, no windows, no caps, no filters
CONFIG_SB = dict(architecture="Saposun", vocab=130, width=72, norm={"eps": 1e-3}, residual_mult=1.0, layers=[
    layer(att(6, 2, 10, 10, 0.35), 20, 7, 2), layer(lat(2, 10, 6, 8, 20, 16, 0.35), None), layer(ret(2, 24, 20, [0.97, 0.8]), 44, 2, 1),
    layer(lat(5, 4, 6, 16, 20, 16, 0.3, kv_from=1), 12, 9, 5)])
# SC: sizes that the tensor-core attentions take (keys and values of one size 64 and 128, of others, keys from the latent)
CONFIG_SC = dict(architecture="Saposun", vocab=300, width=128, norm={"eps": 1e-5}, residual_mult=0.5, layers=[
    layer(att(4, 1, 64, 64, 0.125, 70, 8, 4, 25.0), 64, 8, 2), layer(lat(2, 48, 16, 64, 96, 72, 0.125, 10000.0, 100), 64, 4, 2),
    layer(att(2, 2, 128, 128, 0.09, 100, 24, 3, 40.0, 500.0, 64), 96, 3, 2), layer(ret(2, 64, 96, [0.99, 0.9]), None),
    layer(att(3, 3, 48, 32, 0.15, 33, 70, 5, 15.0), 40, 5, 2), layer(lat(4, 32, 16, 48, 64, 72, 0.15, 10000.0, 65, 1), None)])
# SD: a width that is no multiple of eight, odd sizes, a window of one position, blocks of one position, one tap
CONFIG_SD = dict(architecture="Saposun", vocab=77, width=100, norm={"eps": 1e-6}, residual_mult=1.4, layers=[
    layer(att(5, 5, 7, 9, 0.3, 1, 1, 1, 8.0, 50.0, 6), 37, 3, 2), layer(lat(5, 7, 6, 9, 11, 13, 0.3, 50.0, 1), None),
    layer(ret(5, 9, 7, [0.3, 0.7, 0.99, 0.0, 1.0], 20.0, 8), 30, 11, 3), layer(att(3, 1, 5, 6, 0.45, 128, 65, 3, 20.0, 9.0, 2), None),
    layer(lat(2, 5, 6, 6, 10, 13, 0.4, 50.0, 200, 1), 50, 4, 1)])
CONFIGS = {"SA": CONFIG_SA, "SB": CONFIG_SB, "SC": CONFIG_SC, "SD": CONFIG_SD}
_models = {}
STD = 0.15


def write_model(cfg, d, seed=5, std=STD):
    wick.write_random_model(wick.config_from_json(cfg), seed, d, std=std)
    st = SafeTensorsDir(d)
    return {n: st.get(n).tensor() for n in st.names()}


def model(name, seed=5):
    if (name, seed) not in _models:
        d = os.path.join(tmp_root(), f"sapo-{name}-{seed}")
        _models[name, seed] = (d, write_model(CONFIGS[name], d, seed))
    return _models[name, seed]


def engine(name, dtype, max_tokens=1024, **kw):
    return wick.Engine.from_dir(model(name)[0], dtype=dtype, max_tokens=max_tokens, **kw)


_plain = {}


def plain(name, tokens):
    key = (name, tuple(tokens))
    if key not in _plain:
        _plain[key] = P.forward(CONFIGS[name], model(name)[1], list(tokens)).float()
    return _plain[key]


def tight(got, ref, dtype, what="", tol=None):
    """Every number within the dtype's rounding of the scale."""
    got, ref = got.detach().float().cpu(), ref.detach().float().cpu()
    assert got.shape == ref.shape, f"{what}: {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite"
    scale = max(1e-6, ref.abs().max().item())
    rows = (got - ref).abs().reshape(got.shape[0], -1).max(-1).values / scale
    tol = tol or (3e-5 if dtype in ("float32", torch.float32) else 2.5e-2)
    assert rows.max().item() <= tol, f"{what}: differs by {rows.max().item():.3e} of the scale {scale:.3g}, worst row {int(rows.argmax())}"


def close(got, ref, dtype, what="", tol=None):
    """float32: every row within ``tol`` of the scale.  bfloat16: with random weights a router's close call may choose another
    expert than the plain model's, which replaces a whole expert's output at that row (and, through the states, moves later
    rows a little), so the median row must be within ``tol``, nine rows in ten within three times that, and at most one row in
    twenty further than a third of the scale away; float32 is the sharp comparison."""
    got, ref = got.detach().float().cpu(), ref.detach().float().cpu()
    assert got.shape == ref.shape, f"{what}: {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite"
    scale = max(1.0, ref.abs().max().item())
    rows = (got - ref).abs().reshape(got.shape[0], -1).max(-1).values / scale
    f32 = dtype in ("float32", torch.float32)
    tol = tol or (2e-4 if f32 else 2e-2)
    if f32:
        if rows.max().item() > tol:
            raise AssertionError(f"{what}: differs by {rows.max().item():.3e} of the scale {scale:.3g}, worst row {int(rows.argmax())}")
        return
    med, q90, worst = rows.median().item(), rows.quantile(0.9).item(), rows.max().item()
    far = int((rows > 0.34).sum())
    if med > tol or q90 > 3 * tol or far > max(1, rows.numel() // 20):
        raise AssertionError(f"{what}: median {med:.3e}, nine in ten within {q90:.3e}, worst {worst:.3e} (row {int(rows.argmax())}) "
                             f"of the scale {scale:.3g}")


DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def make_batch(tokens, starts, pages, slots):
    lay = BatchLayout(len(tokens), sum(len(t) for t in tokens), max(len(p) for p in pages), 0)
    host = np.zeros(lay.size, dtype=np.int32)
    fill_host(lay, host, tokens=tokens, starts=starts, slots=slots, pages=pages, want=[[]] * len(tokens))
    return StepBatch(lay, torch.from_numpy(host).to(DEV), q_lens=[len(t) for t in tokens], starts=starts)


def seq_batch(n_new, start=0, tokens=None):
    """A step of one sequence: ``n_new`` tokens after ``start`` cached ones."""
    return make_batch([tokens or [0] * n_new], [start], [list(range(1, (start + n_new + PAGE - 1) // PAGE + 1))], [1])


def make_part(category, kind, params, dtype, tensors):
    """The part with the given tensors (local name -> float tensor), and the tensors as the part holds them (rounded to
    bfloat16 where it keeps them so), as float64 for the plain functions."""
    ctx = BuildContext(dtype=TORCH[dtype], device=torch.device(DEV))
    part = build_part(category, PartSpec(kind, params), ctx)
    specs = {s.name: s for s in part.tensor_specs()}
    assert set(specs) == set(tensors), (sorted(specs), sorted(tensors))
    for n, s in specs.items():
        assert tuple(tensors[n].shape) == tuple(s.shape), (n, tuple(tensors[n].shape), s.shape)
    held = {n: (t.to(TORCH[dtype]) if specs[n].role == "matrix" else t.float()) for n, t in tensors.items()}
    part.load(lambda n: held[n])
    for n, t in held.items():
        assert torch.equal(part.tensor(n).cpu(), t), n
    return part, {n: t.double() for n, t in held.items()}


def rnd(g, *shape, std=1.0):
    return torch.randn(*shape, generator=g) * std


LAT_NAMES = dict(dq="dq", dq_norm="dq.norm", uq="uq", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", o="o")
ATT_NAMES = dict(q="q", k="k", v="v", q_conv="q.conv", k_conv="k.conv", v_conv="v.conv", gate="g", o="o")


def lat_part(dtype, width, m, eps, g, std=0.3, change=None):
    H, d, dr, e, qr, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
    own = m.get("kv_from") is None
    t = {"dq": rnd(g, qr, width, std=std), "dq.norm": 1 + 0.3 * rnd(g, qr), "uq": rnd(g, H * (d + dr), qr, std=std),
         "uk": rnd(g, H * d, r, std=std), "uv": rnd(g, H * e, r, std=std), "o": rnd(g, width, H * e, std=std)}
    if own:
        t.update({"dkv": rnd(g, r + dr, width, std=std), "dkv.norm": 1 + 0.3 * rnd(g, r)})
    if change:
        change(t)
    params = {"width": width, "heads": H, "head_dim": d, "rot_dim": dr, "v_dim": e, "q_rank": qr, "kv_rank": r, "scale": m["scale"],
              "eps": eps, "position": PartSpec("rotary_pairs", {"head_dim": dr, "dims": dr, "theta": m["rot"]["base"], "pairing": "neighbours"}),
              "window": (m.get("mask") or {}).get("size"), "sink": False, "gate": None, "own_kv": own, "names": LAT_NAMES}
    return make_part("mixer", "latent_attention", params, dtype, t)


def ret_part(dtype, width, m, eps, g, std=0.3):
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    t = {"q": rnd(g, H * dk, width, std=std), "k": rnd(g, H * dk, width, std=std), "v": rnd(g, H * dv, width, std=std),
         "g": rnd(g, H * dv, width, std=std), "o": rnd(g, width, H * dv, std=std)}
    params = {"width": width, "heads": H, "head_dim": dk, "v_dim": dv, "decay": m["decay"], "eps": eps, "position": PartSpec(
        "rotary_pairs", {"head_dim": dk, "dims": m["rot"]["dims"], "theta": m["rot"]["base"], "pairing": "halves"}),
        "names": dict(q="q", k="k", v="v", gate="g", o="o")}
    return make_part("mixer", "retention", params, dtype, t)


def att_part(dtype, width, m, eps, g, std=0.3, change=None):
    H, G, d, e, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m.get("conv")
    t = {"q": rnd(g, H * d, width, std=std), "k": rnd(g, G * d, width, std=std), "v": rnd(g, G * e, width, std=std),
         "g": rnd(g, H, width, std=std), "o": rnd(g, width, H * e, std=std)}
    if taps:
        t.update({"q.conv": rnd(g, H * d, taps, std=taps ** -0.5), "k.conv": rnd(g, G * d, taps, std=taps ** -0.5),
                  "v.conv": rnd(g, G * e, taps, std=taps ** -0.5)})
    if change:
        change(t)
    mask = m.get("mask")
    params = {"width": width, "heads": H, "kv_heads": G, "head_dim": d, "v_dim": e, "scale": m["scale"], "eps": eps, "conv": taps,
              "value_norm": True, "soft_cap": m.get("softcap"), "gate": "head",
              "mask": None if mask is None else {"kind": "window", "size": mask["size"], "pool": mask.get("pool")},
              "position": PartSpec("rotary_pairs", {"head_dim": d, "dims": m["rot"]["dims"], "theta": m["rot"]["base"], "pairing": "halves"}),
              "names": ATT_NAMES}
    return make_part("mixer", "attention", params, dtype, t)


class View:
    def __init__(self, **kw):
        self.__dict__.update(kw)


def rows_view(part, dtype, pages=13):
    return View(rows=torch.full((pages, PAGE, part.row), float("nan"), dtype=TORCH[dtype], device=DEV))


def record_view(part, slots=3):
    """Records as the cache hands them out: NaN everywhere but in slot 1, which a sequence has just opened."""
    rec = torch.full((slots, part.record_floats()), float("nan"), device=DEV)
    rec[1].zero_()
    return View(state=rec, slots=None)


def att_view(part, dtype, pages=13):
    """What the cache hands an attention: NaN in every page and record but the one of slot 1."""
    def nans(n):
        return torch.full((pages, n), float("nan"), dtype=TORCH[dtype], device=DEV)
    views = [View(kv=nans(part.kv_heads * PAGE * (part.head_dim + part.v_dim)))]
    if part.pool:
        views.append(View(blocks=nans(part.kv_heads * ops.block_rows(part.pool) * (part.head_dim + part.v_dim))))
    if part.taps > 1:
        views.append(record_view(part))
    return views[0] if len(views) == 1 else View(parts=views)


def run_mixer(part, h, dtype, cuts, view):
    """The part's result for the rows of ``h`` fed in portions of the sizes ``cuts``: float32 [n, width]."""
    out, at = [], 0
    for n in cuts:
        x = h[at:at + n].to(DEV, TORCH[dtype]).contiguous()
        d = part.forward(x, seq_batch(n, at), view, True)
        out.append(d.sum(0) if d.dim() == 3 else d)
        at += n
    assert at == h.shape[0]
    return torch.cat(out)


def as_held(h, dtype):
    return h.to(TORCH[dtype]).double()


# ---------------------------------------------------------------------------
# mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,eps,factor,ffn", [(64, 1e-5, 0.35, "plain"), (101, 1e-2, 1.0, "none"), (6, 1e-6, -1.4, "joins"), (2304, 1e-5, 0.6, "joins"),
                                                  (72, 1e-5, 1.0, "joins")])
def test_both_sublayers_read_the_one_norm_and_their_sum_joins_the_stream_with_a_factor(dtype, width, eps, factor, ffn):
    """The block with a mixer and a feed-forward that note what they read and return given partial sums."""
    g = torch.Generator().manual_seed(width)
    ctx = BuildContext(dtype=TORCH[dtype], device=torch.device(DEV))
    n = 11
    seen, results = [], [0.5 * rnd(g, 3, n, width), 2 * rnd(g, 1, n, width)]

    class M(Mixer):
        def forward(self, x, batch, cache, write_cache):
            seen.append(x.clone())
            return results[0].to(DEV)

    class F(FeedForward):
        IS_NONE = ffn == "none"
        JOINS_BESIDE = ffn == "joins"

        def forward(self, x, batch, beside=None):
            seen.append(x.clone())
            assert (beside is not None) == self.JOINS_BESIDE
            y = results[1].to(DEV)
            return y if beside is None else ops.weighted_sum([(beside, 1.0), (y, 1.0)])

    w = 1 + 0.3 * rnd(g, width)
    norm = build_part("norm", PartSpec("rms", {"width": width, "eps": eps, "tensor": ""}), ctx)
    norm.load(lambda nm: w)
    block = ParallelResidual({"width": width, "factor": factor}, ctx, M({}, ctx), norm, F({}, ctx), NoNorm({}, ctx))
    x = 3 * rnd(g, n, width)
    h = Hidden(x.clone().to(DEV))
    for _ in range(3):
        h = block.forward(h, None, None, True)
    want, reads = x.double(), []
    for _ in range(3):
        reads.append(P.norm(want, w.double(), eps))
        want = want + factor * (results[0].double().sum(0) + (0 if ffn == "none" else results[1].double()[0]))
    per = 1 if ffn == "none" else 2
    assert len(seen) == 3 * per
    for i, s in enumerate(seen):
        tight(s, reads[i // per], "float32", f"sublayer {i} reads", 3e-6 if dtype == "float32" else 5e-3)
    rows = torch.tensor([3, 3, 10, 0], dtype=torch.int32, device=DEV)
    extra = {} if h.scale is None else {"scale": h.scale}
    tight(norm.add_forward(h.x, h.pending, torch.float32, rows, **extra), P.norm(want, w.double(), eps)[[3, 3, 10, 0]], "float32", "chosen rows", 3e-6)
    tight(h.resolved(), want, "float32", "the stream", 2e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,experts,top,ff", [(40, 7, 2, 24), (64, 12, 5, 48), (100, 3, 3, 37), (128, 16, 1, 64)])
def test_experts_chosen_by_corrected_scores_weighted_by_the_scores_themselves(dtype, width, experts, top, ff):
    g = torch.Generator().manual_seed(experts)
    t = {}
    for i in range(experts):
        t.update({f"e{i}.gate": rnd(g, ff, width, std=0.2), f"e{i}.up": rnd(g, ff, width, std=0.2), f"e{i}.down": rnd(g, width, ff, std=0.2)})
    t["router"], t["correction"] = rnd(g, experts, width, std=0.4), 0.3 * rnd(g, experts)
    part, td = make_part("ffn", "routed_moe", {"width": width, "experts": experts, "top": top, "intermediate": ff, "scores": "softmax",
                                               "correction": True, "renormalize": False, "expert": "gated", "names": dict(
                                                   gate="gate", up="up", down="down", expert="e{i}.", router="router", correction="correction")}, dtype, t)
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    for n in (1, 7, 130):
        h = as_held(rnd(g, 4 * n, width), dtype)
        s = torch.softmax(h @ td["router"].T, -1) + td["correction"]          # (rows whose choice is no close call)
        v = torch.cat([s.sort(-1, descending=True).values, torch.full((4 * n, 1), -9.0, dtype=torch.float64)], -1)
        h = h[(v[:, top - 1] - v[:, top] > 2e-3).nonzero()[:n, 0]]
        assert h.shape[0] == n
        if top < experts:                                   # the correction decides who is chosen, and weighs nothing
            assert any(set(a.tolist()) != set(b.tolist()) for a, b in zip(P.choose_experts(h @ td["router"].T, td["correction"], top)[0],
                                                                            P.choose_experts(h @ td["router"].T, 0, top)[0])) or n < 30
        ref = P.expert_ff(h, td, "", mlp)
        x = h.to(DEV, TORCH[dtype]).contiguous()
        tight(part.forward(x, seq_batch(n)).sum(0), ref, dtype, f"{n} tokens")
        beside = rnd(g, 3, n, width)
        got = part.forward(x, seq_batch(n), beside=beside.to(DEV))
        tight(got.sums()[0], ref + beside.double().sum(0), dtype, f"{n} tokens beside")


LATS = [lat(3, 12, 8, 20, 28, 24, 0.3, 1000.0, 17), lat(2, 16, 16, 16, 32, 40, 0.2, 20000.0, 64), lat(5, 7, 6, 9, 11, 13, 0.3, 50.0, 1),
        lat(4, 48, 16, 64, 96, 72, 0.125, 10000.0, 65), lat(2, 96, 32, 128, 64, 136, 0.09), lat(1, 24, 8, 40, 36, 32, 0.25, 100.0, 129),
        lat(6, 32, 64, 48, 40, 200, 0.1, 300.0, 128), lat(3, 5, 2, 6, 10, 15, 0.45, 9.0, 400)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", LATS, ids=lambda m: f"h{m['heads']}d{m['dim']}+{m['rot_dim']}v{m['vdim']}r{m['kv_rank']}w{(m.get('mask') or {}).get('size')}")
def test_latent_attention_and_a_reader_of_its_rows_in_any_portions(dtype, m):
    """The layer with latents of its own, and one of other sizes that applies its own matrices to the same rows."""
    g = torch.Generator().manual_seed(m["heads"] * 100 + m["dim"])
    width, n = 48, 210
    reader = dict(m, heads=3, dim=m["dim"] + 4, vdim=m["vdim"] + 3, q_rank=18, scale=0.2, mask={"size": 90}, kv_from=0)
    part, t = lat_part(dtype, width, m, 1e-5, g)
    part2, t2 = lat_part(dtype, width, reader, 1e-5, g)
    assert part2.cache_need() is None
    h, h2 = rnd(g, n, width), rnd(g, n, width)
    rows = P.latent_rows(as_held(h, dtype), t, "", m, 1e-5)
    ref, ref2 = P.latent_attention(as_held(h, dtype), t, "", m, 1e-5, rows), P.latent_attention(as_held(h2, dtype), t2, "", reader, 1e-5, rows)
    for cuts in ([n], [1] * 5 + [2, 60, 2, 3, 64, 74], [70] + [1] * 5 + [17, 118], [209, 1]):
        view = rows_view(part, dtype)
        outs, at = ([], []), 0
        for c in cuts:
            batch = seq_batch(c, at)
            for o, p, hh, w in ((outs[0], part, h, True), (outs[1], part2, h2, False)):
                o.append(p.forward(hh[at:at + c].to(DEV, TORCH[dtype]).contiguous(), batch, view, w).sum(0))
            at += c
        tight(torch.cat(outs[0]), ref, dtype, f"own rows, cuts {cuts[:3]}")
        tight(torch.cat(outs[1]), ref2, dtype, f"reader, cuts {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv,dims", [(3, 8, 4, 8), (2, 16, 16, 8), (1, 6, 10, 2), (2, 128, 128, 128), (4, 20, 36, 12), (1, 300, 8, 300), (2, 64, 96, 32),
                                          (5, 9, 7, 8), (3, 100, 12, 50)])
def test_retention_in_any_portions(dtype, H, dk, dv, dims):
    g = torch.Generator().manual_seed(H * 1000 + dk)
    width, n = 40, 350                                       # (a step of 192 tokens or more is scanned in chunks of 64)
    m = ret(H, dk, dv, [0.999, 0.5, 1.0, 0.0, 0.96875][:H], 700.0, dims)
    part, t = ret_part(dtype, width, m, 1e-5, g)
    h = rnd(g, n, width)
    ref = P.retention(as_held(h, dtype), t, "", m, 1e-5)
    for cuts in ([n], [1] * 6 + [2, 3, 2, 59, 64, 1, 1, 12, 200], [349, 1], [75, 75, 8, 192], [192, 158]):
        tight(run_mixer(part, h, dtype, cuts, record_view(part)), ref, dtype, f"cuts {cuts[:3]}")


@pytest.mark.parametrize("H,dk,dv,dims", [(2, 6, 3, 4), (1, 8, 12, 8), (3, 16, 4, 0)])
def test_the_recurrence_on_its_own(H, dk, dv, dims):
    """ops.retention_mix from given partial sums: the state after the step, [H][dv][dk] in the record, is the plain one."""
    g = torch.Generator().manual_seed(8)
    n = 70
    q, k, v = rnd(g, n, H * dk), rnd(g, n, H * dk), rnd(g, n, H * dv)
    whole = torch.cat([q, k, v, rnd(g, n, 5)], -1)
    a = rnd(g, n, whole.shape[1])
    parts = torch.stack([whole - a, a]).to(DEV)             # (two partial sums)
    decay = torch.tensor([0.9, 1.0, 0.25][:H])
    turned = [P.turn(x.double().view(n, H, dk), 100.0, dims, True) if dims else x.double().view(n, H, dk) for x in (q, k)]
    o, S = P.decaying_outer_products(turned[0], turned[1] * 0.3, v.double().view(n, H, dv), decay.double())
    rec = torch.full((3, H * dv * dk), float("nan"), device=DEV)
    freq = torch.tensor([100.0 ** (-2.0 * i / dims) for i in range(dims // 2)], device=DEV) if dims else None
    for cuts in ([n], [1] * 5 + [65], [2, 1, 67]):
        rec[1].zero_()
        outs, at = [], 0
        for c in cuts:
            b = seq_batch(c, at)
            cos, sin = ops.rope_table(b.positions, freq) if dims else (None, None)
            outs.append(ops.retention_mix(parts[:, at:at + c].contiguous(), heads=H, key_dim=dk, v_dim=dv, cos=cos, sin=sin, rot_dims=dims,
                                          k_scale=0.3, decay=decay.to(DEV), records=rec, batch=b))
            at += c
        tight(torch.cat(outs), o.reshape(n, H * dv), "float32", f"o, cuts {cuts[:2]}")
        tight(rec[1].view(H, dv, dk), S.transpose(1, 2), "float32", f"the record, cuts {cuts[:2]}")
        assert torch.isnan(rec[0]).all() and torch.isnan(rec[2]).all()
    got = ops.gla_norm_gate(torch.cat(outs), None, 0, H, dv, None, 1e-3, torch.float32)
    tight(got, P.rms(o, 1e-3).reshape(n, H * dv), "float32", "norm without a weight")


def test_the_state_remembers_a_token_hundreds_of_positions_back():
    """With a decay of 0.9995 the result 500 positions later moves when one early token changes, in a prompt, in portions and
    token by token, as the plain one does; with 0.5 nothing of it is left."""
    g = torch.Generator().manual_seed(3)
    width, n = 24, 520
    h = rnd(g, n, width, std=0.3)
    h2 = h.clone()
    h2[7] = 30 * rnd(g, width)
    for a, late in ((0.9995, True), (0.5, False)):
        m = ret(2, 6, 10, [a, a])
        part, t = ret_part("float32", width, m, 1e-7, g)
        ref, ref2 = (P.retention(x.double(), t, "", m, 1e-7) for x in (h, h2))
        assert bool((ref[515:] - ref2[515:]).abs().max() > 1e-2 * ref.abs().max()) == late
        for cuts in ([n], [8, 400, 112], [500] + [1] * 20):
            tight(run_mixer(part, h, "float32", cuts, record_view(part)), ref, "float32", f"cuts {cuts[:3]}", tol=2e-4)
            tight(run_mixer(part, h2, "float32", cuts, record_view(part)), ref2, "float32", f"changed, cuts {cuts[:3]}", tol=2e-4)


@pytest.mark.parametrize("H,G,d,e,taps,extra,splits", [(3, 1, 8, 4, 4, 3, 2), (2, 2, 7, 5, 2, 0, 1), (4, 2, 32, 16, 7, 4, 3), (1, 1, 4, 4, 1, 2, 1), (2, 1, 16, 16, 16, 0, 2)])
def test_the_short_filters_and_their_record(H, G, d, e, taps, extra, splits):
    """The finish kernel on given partial sums: q comes out filtered, k and v lie filtered in the cache, and the record holds the
    last inputs, oldest first, zeros before the start."""
    g = torch.Generator().manual_seed(d)
    n, W = 90, (H + G) * d + G * e
    u = rnd(g, n, W + extra)
    a = rnd(g, splits - 1, n, W + extra)
    parts, w = torch.cat([(u - a.sum(0))[None], a]).to(DEV), rnd(g, taps, W)
    ref = P.causal_filter(u[:, :W].double(), w.T.double())
    for cuts in ([n], [1] * 9 + [2, 2, 3, 64, 10], [1, 2, 87]):
        rec = torch.full((3, (taps - 1) * W), float("nan"), device=DEV)
        rec[1].zero_()
        kv = torch.full((4, G * PAGE * (d + e)), float("nan"), device=DEV)
        outs, at = [], 0
        for c in cuts:
            b = seq_batch(c, at)
            outs.append(ops.qkv_finish(parts[:, at:at + c].contiguous(), H, G, d, e, dtype=torch.float32, kv=kv, page_table=b.page_table,
                                       seq_of_token=b.seq_of_token, positions=b.positions, conv=(w.to(DEV), rec if taps > 1 else None, b)))
            at += c
            if taps > 1:
                want = torch.cat([torch.zeros(taps - 1, W), u[:at, :W]])[-(taps - 1):]
                tight(rec[1].view(taps - 1, W), want, "float32", f"record after {at}")
        tight(torch.cat(outs).view(n, -1), ref[:, :H * d], "float32", f"q, cuts {cuts[:3]}")
        keys = kv[1:3, :G * PAGE * d].view(2, G, PAGE, d).transpose(1, 2).reshape(2 * PAGE, G * d)[:n]
        vals = kv[1:3, G * PAGE * d:].view(2, G, PAGE, e).transpose(1, 2).reshape(2 * PAGE, G * e)[:n]
        tight(torch.cat([keys, vals], 1), ref[:, H * d:], "float32", f"k and v, cuts {cuts[:3]}")
        assert torch.isnan(rec[0]).all() and torch.isnan(rec[2]).all()


@pytest.mark.parametrize("width,top,splits,factor,sorted_rows", [(64, 2, 3, 0.4, False), (2048, 4, 1, 1.0, True), (4100, 1, 2, -0.7, True), (12, 33, 1, 0.5, False)])
def test_experts_sums_join_the_stream_and_its_norm_in_one_kernel(width, top, splits, factor, sorted_rows):
    g = torch.Generator().manual_seed(width)
    n, E, eps = 9, top + 2, 1e-4
    choice = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(n)]).int()
    choice[0, 0] = -1                                       # (names no expert)
    row_of = torch.randperm(3 * n * top, generator=g)[:n * top].view(n, top).int() if sorted_rows else None
    y, weight = rnd(g, 3 * n * top if sorted_rows else n * top, width), torch.rand(n, top, generator=g)
    base, x, w = rnd(g, splits, n, width), 3 * rnd(g, n, width), 1 + 0.3 * rnd(g, width)
    rows = row_of.long() if sorted_rows else torch.arange(n * top).view(n, top)
    d = (weight * (choice >= 0)).double()[:, :, None] * y.double()[rows]
    dev = lambda t: None if t is None else t.to(DEV)
    for b in (base, None):
        want = x.double() + factor * (d.sum(1) + (0 if b is None else b.double().sum(0)))
        s = ops.ExpertSum(dev(y), dev(row_of), dev(choice), dev(weight), E, dev(b))
        assert s.joins_norm()
        tight(s.sums()[0], (want - x.double()) / factor, "float32", "sums", 1e-5)
        xd = x.to(DEV)
        got = ops.moe_experts_norm(xd, s, factor, w.to(DEV), eps, torch.float32, torch.tensor([3, 3, 8, 0], dtype=torch.int32, device=DEV))
        tight(got, P.norm(want, w.double(), eps)[[3, 3, 8, 0]], "float32", "chosen rows", 3e-6)
        assert torch.equal(xd.cpu(), x)
        for dt in DTYPES:
            xd = x.to(DEV)
            tight(ops.moe_experts_norm(xd, s, factor, w.to(DEV), eps, TORCH[dt]), P.norm(want, w.double(), eps), dt, "normed", 3e-6 if dt == "float32" else 5e-3)
            tight(xd, want, "float32", "the stream", 3e-6)


ATTS = [att(4, 2, 16, 12, 0.3, 20, 3, 4, 12.0, 700.0, 8), att(2, 1, 8, 8, 0.4, 64, 10, 2, 30.0), att(5, 5, 7, 9, 0.3, 1, 1, 1, 8.0, 50.0, 6),
        att(6, 2, 10, 10, 0.35), att(4, 1, 64, 64, 0.125, 70, 8, 4, 25.0), att(2, 2, 128, 128, 0.09, 100, 24, 3, 40.0, 500.0, 64),
        att(3, 3, 48, 32, 0.15, 33, 70, 5, 15.0), att(3, 1, 5, 6, 0.45, 128, 65, 3, 20.0, 9.0, 2), att(8, 1, 64, 64, 0.125, 64, 64, 4),
        att(6, 2, 32, 48, 0.2, 17, 2, None, 10.0), att(4, 4, 64, 64, 0.2, 300, 12, 4, 20.0), att(2, 1, 64, 64, 0.2, None, None, 3, 9.0),
        att(8, 2, 24, 20, 0.2, 40, 33, 9, 6.0), att(2, 1, 256, 160, 0.06, 50, 7, 2, 20.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", ATTS, ids=lambda m: f"h{m['heads']}g{m['kv_heads']}d{m['dim']}v{m['vdim']}w{(m.get('mask') or {}).get('size')}"
                                                  f"p{(m.get('mask') or {}).get('pool')}c{m.get('conv')}")
def test_attention_with_filters_pooled_blocks_and_capped_scores_in_any_portions(dtype, m):
    g = torch.Generator().manual_seed(m["heads"] * 100 + m["dim"])
    width, n = 48, 330
    part, t = att_part(dtype, width, m, 1e-5, g)
    h = rnd(g, n, width)
    ref = P.window_attention(as_held(h, dtype), t, "", m, 1e-5)
    for cuts in ([n], [1] * 40 + [2, 3, 2, 60, 64, 2, 2, 155], [1, 2, 327], [200] + [1] * 70 + [60], [329, 1]):
        tight(run_mixer(part, h, dtype, cuts, att_view(part, dtype)), ref, dtype, f"cuts {cuts[:3]}")


def paged(x, pages, fill=float("nan")):
    """x [n, heads, size] -> [len(pages) + .. , heads, 64, size] pages with x's rows on the given pages in order."""
    n, heads, size = x.shape
    out = torch.full((max(pages) + 2, heads, PAGE, size), fill, dtype=x.dtype)
    for i in range(n):
        out[pages[i // PAGE], :, i % PAGE] = x[i]
    return out


@pytest.mark.parametrize("dtype,H,G,d,e,kind", [("float32", 4, 2, 16, 20, "rows"), ("bfloat16", 4, 2, 16, 32, "rows"), ("bfloat16", 4, 2, 48, 32, "mma"),
                                                ("bfloat16", 4, 1, 64, 64, "tc"), ("bfloat16", 2, 2, 128, 128, "tc"), ("bfloat16", 6, 2, 64, 64, "rows")])
@pytest.mark.parametrize("window,block", [(1, 1), (20, 3), (64, 64), (63, 12), (65, 10), (100, 128), (33, 65)])
def test_a_block_that_stands_out_shows_from_the_position_it_is_seen_at(dtype, H, G, d, e, kind, window, block):
    """The first key of one block is so large that the block's mean key still stands out, the block's values are large, and every
    query points that way: the result is the block's value while that token is in the window, and again from the position on
    at which the block lies wholly before the window; between the two it is not seen at all.  For blocks at the start, at
    page borders and late, in prompts from position 0, in portions, and decoded."""
    g = torch.Generator().manual_seed(window * 100 + block)
    n, scale, cap, dt = 420, d ** -0.5, 30.0, TORCH[dtype]
    pages = [5, 1, 7, 2, 3, 6, 4]
    big = rnd(g, d)
    big = big / big.norm() * d ** 0.5
    q = (0.1 * rnd(g, n, H, d) + 3 * big).to(dt)
    gate = torch.rand(n, H, generator=g)
    for blk in sorted({0, 1, 64 // block, 200 // block}):
        k, v = 0.3 * rnd(g, n, G, d), 0.3 * rnd(g, n, G, e)
        lo, hi = blk * block, min(n, (blk + 1) * block)
        k[lo] += 3 * block * big
        v[lo:hi] += 4.0
        k, v = k.to(dt), v.to(dt)
        ref = P.attend(q.double(), k.double(), v.double(), scale, window, block, cap)
        seen = hi - 1 + window                               # the first position that sees a whole block
        if hi - lo == block and seen < n:
            assert ref[lo + window - 1].mean() > 2, "the token must show while it is in the window"
            assert ref[seen].mean() > 2, "the block must show"
            assert window < 20 or block == 1 or ref[seen - 1].mean() < 1, "... and not one position early"
        ref = ref * gate.double()[:, :, None]
        kv = torch.cat([paged(k, pages).flatten(1), paged(v, pages).flatten(1)], 1).contiguous().to(DEV)
        rows = ops.block_rows(block)
        for cuts in ([n], [64, 2, 150, 204]):
            store = torch.full((kv.shape[0], G * rows * (d + e)), float("nan"), dtype=dt, device=DEV)
            outs, at = [], 0
            for c in cuts:
                b = make_batch([[0] * c], [at], [pages[:(at + c + PAGE - 1) // PAGE]], [1])
                outs.append(ops.attention_pooled(q[at:at + c].to(DEV).contiguous(), kv, b, scale, n_kv=G, v_dim=e, window=window, store=store,
                                                 block=block, soft_cap=cap, gate=gate[at:at + c].to(DEV).contiguous(), kind=kind))
                at += c
            tight(torch.cat(outs), ref, dtype, f"block {blk}, cuts {cuts}")
        # decoded alone, from the store that the portions left
        at = [i for i in (hi - 1, hi + window - 3, hi + window - 2, hi + window - 1, hi + window, n - 1) if 0 <= i < n]
        for i in at:
            b = make_batch([[0]], [i], [pages[:(i + PAGE) // PAGE]], [1])
            got = ops.attention_pooled(q[i:i + 1].to(DEV).contiguous(), kv, b, scale, n_kv=G, v_dim=e, window=window, store=store, block=block,
                                       pooled=True, soft_cap=cap, gate=gate[i:i + 1].to(DEV).contiguous())
            assert (got.cpu().double() - ref[i]).abs().max() < (3e-5 if dtype == "float32" else 2.5e-2) * ref.abs().max(), f"block {blk}, position {i} decoded"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 129])
def test_a_latent_key_that_stands_out_just_inside_and_just_outside_the_window(dtype, window):
    """The latent's first 64 rows of Wdkv are Wdq, a head's keys are that half of the latent, its values are made from the
    other half, whose rows see only what Wdq maps to zero, and there is no rotated part.  A score is then the product of two
    normed vectors of 64 numbers: about 64 * scale where h_j is h_i with the rest negated, and a few units of 8 * scale
    elsewhere; the value of such a twin is the negated value, so a result is v_i where the twin is not seen and vanishes
    where it is.  The rows are checked in a prompt, in portions and decoded alone."""
    g = torch.Generator().manual_seed(77)
    width, r, n, dr, H = 160, 64, 520, 16, 2
    m = lat(H, r, dr, 32, r, 2 * r, 0.4, 10000.0, window)

    def change(t):
        t["dkv"][:r] = t["dq"]
        nul = torch.linalg.svd(t["dq"])[2][r:]
        t["dkv"][r:2 * r] = rnd(g, r, nul.shape[0], std=0.3) @ nul
        t["dkv"][2 * r:] = 0
        t["dq.norm"], t["dkv.norm"] = torch.ones(r), torch.ones(2 * r)
        t["uk"] = torch.cat([torch.eye(r), torch.zeros(r, r)], 1).repeat(H, 1)
        t["uv"][:, :r] = 0
        t["uq"] = torch.cat([torch.eye(r), torch.zeros(dr, r)]).repeat(H, 1)

    part, t = lat_part(dtype, width, m, 1e-6, g, change=change)
    h = rnd(g, n, width)
    null = torch.linalg.svd(t["dq"])[2][r:].T.float()
    pairs = []
    for i in (70, 127, 128, 192, 255, 300, 383, 448, 511, 515):
        pairs.append((i, i - window + 1 - len(pairs) % 2))   # the oldest key that is seen, or the newest that is not
    pairs = [(i, j) for i, j in pairs if 0 <= j < i and j not in {a for a, _ in pairs}]
    for i, j in pairs:
        h[j] = h[i] - 2 * null @ (null.T @ h[i])

    def plain_of(x):
        x = as_held(x, dtype)
        return P.latent_attention(x, t, "", m, 1e-6, P.latent_rows(x, t, "", m, 1e-6))
    ref = plain_of(h)
    h2 = h.clone()
    for i, j in pairs:
        h2[j] = rnd(g, width)
    ref2 = plain_of(h2)
    for i, j in pairs:                                      # a twin that is seen matters, one that is not does not
        assert bool((ref2[i] - ref[i]).abs().max() > 0.1 * ref.abs().max()) == (i - j < window), (i, j)
    for cuts in ([n], [64, 64, 2, 190, 200], [256, 2, 262]):
        tight(run_mixer(part, h, dtype, cuts, rows_view(part, dtype)), ref, dtype, f"cuts {cuts[:3]}")
    for i, j in pairs[:7]:                                  # decoded: i alone after a prompt that ends right before it
        got = run_mixer(part, h[:i + 1], dtype, [i, 1], rows_view(part, dtype))
        tight(torch.cat([ref[:i].float(), got[i:].cpu()]), ref[:i + 1], dtype, f"position {i} decoded, its twin at {j}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("block", [1, 3, 12, 64, 65, 130])
def test_the_means_of_blocks_are_those_of_the_cached_numbers(dtype, block):
    """Sequences of unequal lengths in one step, portions that end inside blocks, pages in any order: the store holds the
    means (of the numbers as they are cached) of whole blocks only, and the array for the prompt kernels holds all of them."""
    g = torch.Generator().manual_seed(block)
    G, d, e, dt = 2, 10, 6, TORCH[dtype]
    lens, pages = [150, 3, 400], [[3, 9, 1], [6], [2, 4, 8, 5, 7, 11, 10]]
    ks, vs = [rnd(g, n, G, d).to(dt) for n in lens], [rnd(g, n, G, e).to(dt) for n in lens]
    kv = torch.full((13, G * PAGE * (d + e)), float("nan"), dtype=dt)
    for k, v, pg in zip(ks, vs, pages):
        a, b = paged(k, pg).flatten(1), paged(v, pg).flatten(1)
        kv[pg] = torch.cat([a, b], 1)[pg]
    kv = kv.to(DEV)
    rows = ops.block_rows(block)
    store = torch.full((13, G * rows * (d + e)), float("nan"), dtype=dt, device=DEV)
    done = [0, 0, 0]
    for upto in ([70, 1, 64], [131, 3, 395], [150, 3, 400]):
        new = [b - a for a, b in zip(done, upto)]
        b = make_batch([[0] * c for c in new], done, [p[:(u + PAGE - 1) // PAGE] for p, u in zip(pages, upto)], [1, 2, 3])
        flat, tiles = ops.pool_blocks(kv, store, b, n_kv=G, d=d, e=e, block=block, flat=True)
        done = upto
        for s, n in enumerate(upto):
            mk, mv = P.pooled(ks[s][:n].double(), block), P.pooled(vs[s][:n].double(), block)
            for i in range(n // block):
                page = (i * block + block - 1) // PAGE
                at = i - page * PAGE // block
                row = store[pages[s][page]].cpu()
                keys, vals = row[:G * rows * d].view(G, rows, d), row[G * rows * d:].view(G, rows, e)
                tight(keys[:, at], mk[i], dtype, f"key {s} {i}", 4e-6 if dtype == "float32" else 5e-3)
                tight(vals[:, at], mv[i], dtype, f"value {s} {i}", 4e-6 if dtype == "float32" else 5e-3)
            tile = flat.view(-1, tiles, G * PAGE * (d + e))[s].cpu()
            fk = tile[:, :G * PAGE * d].view(tiles, G, PAGE, d).transpose(1, 2).reshape(tiles * PAGE, G, d)
            if n // block:
                tight(fk[:n // block], mk, dtype, "the array", 4e-6 if dtype == "float32" else 5e-3)
            assert (fk[n // block:] == 0).all()
    assert torch.isnan(store[0]).all() and torch.isnan(store[12]).all()


def test_the_first_tokens_start_from_zeros_not_from_the_record_of_the_slots_last_user():
    g = torch.Generator().manual_seed(4)
    width, m = 24, att(2, 1, 6, 10, 0.4, 7, 3, 5, 9.0)
    part, t = att_part("float32", width, m, 1e-5, g)
    h = rnd(g, 9, width)
    ref = P.window_attention(h.double(), t, "", m, 1e-5)
    view = att_view(part, "float32")
    run_mixer(part, rnd(g, 30, width), "float32", [30], view)          # another sequence leaves its record in slot 1
    rec = view.parts[2].state
    assert rec[1].abs().max() > 0
    for cuts in ([9], [1, 1, 1, 2, 4]):
        rec[1].zero_()                                        # (what the cache does when a sequence opens in the slot)
        tight(run_mixer(part, h, "float32", cuts, view), ref, "float32", f"cuts {cuts}")
    assert torch.isnan(rec[2]).all() and torch.isnan(rec[0]).all(), "another slot's record was written"


# ---------------------------------------------------------------------------
# whole models through the engine
def step_rows(eng, s, toks, cuts):
    rows, at = [], 0
    for n in cuts:
        rows.append(eng.step([s], [toks[at:at + n]], [list(range(n))]).clone())
        at += n
    return torch.cat(rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_decoding_and_portions_agree_with_the_plain_model(name, dtype):
    toks = random_tokens(CONFIGS[name]["vocab"], 230, seed=11)
    ref = plain(name, toks)
    eng = engine(name, dtype)
    for cuts in ([230], [1] * 7 + [2, 3, 61, 2, 64, 70] + [1] * 13, [198] + [1] * 32, [2] * 40):
        s = eng.open_seq()
        got = step_rows(eng, s, toks, cuts)
        close(got, ref[:got.shape[0]], dtype, f"cuts {cuts[:3]}")
        eng.close_seq(s)
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["SA", "SC"])
def test_a_prompt_beyond_the_captured_sizes(name, dtype):
    """More tokens than a captured prompt step takes: in bfloat16 the tensor-core attention and the chunked scan."""
    toks = random_tokens(CONFIGS[name]["vocab"], 620, seed=15)
    ref = plain(name, toks)
    eng = engine(name, dtype, max_tokens=2048)
    for cuts in ([620], [600] + [1] * 20, [530, 2, 88]):
        s = eng.open_seq()
        close(step_rows(eng, s, toks, cuts), ref, dtype, f"cuts {cuts[:3]}")
        eng.close_seq(s)
    # two of them and a short one in one step
    other, short = random_tokens(CONFIGS[name]["vocab"], 530, seed=16), random_tokens(CONFIGS[name]["vocab"], 3, seed=17)
    slots = [eng.open_seq() for _ in range(3)]
    got = eng.step(slots, [other, short, toks], [[0, 529], [0, 1, 2], list(range(620))])
    close(got, torch.cat([plain(name, other)[[0, 529]], plain(name, short), ref]), dtype, "together")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_stream_after_every_layer(name, dtype):
    toks = random_tokens(CONFIGS[name]["vocab"], 90, seed=13)
    taps = []
    P.forward(CONFIGS[name], model(name)[1], toks, taps=taps)
    eng = engine(name, dtype, use_graphs=False)
    seen, fwd = [], eng.model.forward
    eng.model.forward = lambda batch, cache: fwd(batch, cache, tap=lambda i, x: seen.append(x.clone().cpu()))
    s = eng.open_seq()
    eng.step([s], [toks])
    assert len(seen) == len(taps) == len(eng.spec.schedule)
    for i, (got, ref) in enumerate(zip(seen, taps)):
        close(got, ref.float(), dtype, f"after layer {i}", 1e-4 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_passes_page_borders_and_windows(dtype):
    name = "SA"
    toks = random_tokens(CONFIGS[name]["vocab"], 270, seed=12)
    eng = engine(name, dtype)
    s = eng.open_seq()
    close(step_rows(eng, s, toks, [3] + [1] * 267), plain(name, toks), dtype, "decoded")


def test_an_early_token_shows_in_the_logits_hundreds_of_positions_later():
    """Every decay is set to 0.9995 and the early token's embedding row is large: changing token 2 moves the logits at
    position 600 (by the states and by the mean of the block that holds it), in the plain model and in the engine, for a
    prompt in one step, in portions, and decoded."""
    cfg = json.loads(json.dumps(CONFIGS["SA"]))
    for L in cfg["layers"]:
        if L["type"] == "retention":
            L["mixer"]["decay"] = [0.9995] * L["mixer"]["heads"]
    w = {k: v.clone() for k, v in model("SA")[1].items()}
    a = random_tokens(cfg["vocab"] - 1, 604, seed=14)
    a[2] = cfg["vocab"] - 1
    w["embed"][a[2]] *= 60.0
    b = list(a)
    b[2] = 17
    d = os.path.join(tmp_root(), "sapo-SA-remembers")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(d, "model.safetensors"), w)
    ra, rb = P.forward(cfg, w, a).float(), P.forward(cfg, w, b).float()
    assert (ra[600:] - rb[600:]).abs().max() > 1e-2 * ra.abs().max(), "the early token must show late"
    eng = wick.Engine.from_dir(d, dtype="float32", max_tokens=2048)
    for toks, ref in ((a, ra), (b, rb)):
        for cuts in ([604], [3, 2, 395, 200] + [1] * 4, [590] + [1] * 14):
            s = eng.open_seq()
            close(step_rows(eng, s, toks, cuts), ref, "float32", f"cuts {cuts[:3]}", 3e-4)
            eng.close_seq(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_a_batch_of_unequal_requests_equals_each_alone(name, dtype):
    cfg = CONFIGS[name]
    lens = [1, 65, 130, 9, 64]
    prompts = [random_tokens(cfg["vocab"], n + 12, seed=20 + i) for i, n in enumerate(lens)]
    eng = engine(name, dtype, max_tokens=2048)
    alone = []
    for p, n in zip(prompts, lens):
        s = eng.open_seq()
        alone.append(step_rows(eng, s, p, [n] + [1] * 12))
        eng.close_seq(s)
        close(alone[-1], plain(name, p), dtype, f"alone, {n} tokens")
    slots = [eng.open_seq() for _ in prompts]
    got = [[] for _ in prompts]
    first = eng.step(slots, [p[:n] for p, n in zip(prompts, lens)], [list(range(n)) for n in lens])
    at = 0
    for i, n in enumerate(lens):
        got[i].append(first[at:at + n].clone())
        at += n
    live = list(range(len(prompts)))
    for step in range(12):
        if step == 5:                                      # two requests end early; the others go on
            for i in (1, 3):
                eng.close_seq(slots[i])
                live.remove(i)
        out = eng.step([slots[i] for i in live], [[prompts[i][lens[i] + step]] for i in live])
        for r, i in enumerate(live):
            got[i].append(out[r:r + 1].clone())
    for i in range(len(prompts)):
        x = torch.cat(got[i])
        close(x, plain(name, prompts[i])[:x.shape[0]], dtype, f"request {i} in a batch")
        if dtype == "float32":
            tight(x, alone[i][:x.shape[0]], dtype, f"request {i} differs in a batch", 2e-5)


def poison_free(eng):
    """NaN in every page that no sequence holds, and in every record of a slot that no sequence has."""
    held = eng.cache.pages.held()
    free = [p for p in range(1, eng.cache.n_pages) if p not in held]
    idle = [s for s in range(1, eng.cache.max_seqs + 1) if s not in set(eng.cache.seqs)]
    for g in eng.cache.groups:
        if g.need.kind.startswith("paged_") and free:
            g.storage[:, torch.tensor(free, device=g.storage.device)] = float("nan")
        if g.need.kind == "state" and idle:
            g.storage[:, torch.tensor(idle, device=g.storage.device)] = float("nan")


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_slots_and_records_that_were_given_back_are_used_again(dtype):
    name = "SA"
    cfg = CONFIGS[name]
    eng = engine(name, dtype, max_tokens=320)
    a, b = random_tokens(cfg["vocab"], 150, seed=31), random_tokens(cfg["vocab"], 140, seed=32)
    s1 = eng.open_seq()
    eng.step([s1], [a])
    s2 = eng.open_seq()
    eng.step([s2], [b[:70]])
    eng.close_seq(s1)                                      # its three pages, its slot and its records come back
    poison_free(eng)
    s3 = eng.open_seq()
    assert s3 == s1
    out = eng.step([s3], [a[:100]], [list(range(100))])
    assert set(eng.cache.pages_of(s3)) & {1, 2, 3}
    close(out, plain(name, a[:100]), dtype, "in reused pages")
    rows = [eng.step([s2, s3], [[b[70 + i]], [a[100 + i]]]).clone() for i in range(30)]
    close(torch.stack([r[0] for r in rows]), plain(name, b[:100])[70:], dtype, "the request that stayed")
    close(torch.stack([r[1] for r in rows]), plain(name, a[:130])[100:], dtype, "the request in reused pages")
    eng.cache.check()


def test_a_request_starts_over_and_a_model_without_recurrences_goes_back():
    eng = engine("SA", "float32")
    toks = random_tokens(CONFIGS["SA"]["vocab"], 40, seed=33)
    s = eng.open_seq()
    first = eng.step([s], [toks]).clone()
    with pytest.raises(ValueError):
        eng.truncate_seq(s, 20)                              # (the recurrences' records hold all 40 tokens)
    eng.truncate_seq(s, 0)
    eng.step([s], [toks[:17]], [[]])
    close(eng.step([s], [toks[17:]]), first, "float32", "again", 2e-5)
    # attention without filters keeps every position; blocks that are no longer whole are made again when they are
    cfg = dict(CONFIGS["SA"], layers=[layer(lat(3, 12, 8, 4, 28, 24, 0.3, 1000.0, 17), 56, 6, 2), layer(att(4, 2, 16, 12, 0.3, 20, 7, None, 12.0), None),
                                      layer(lat(2, 8, 8, 8, 16, 24, 0.3, 1000.0, 40, 0), None)])
    d = os.path.join(tmp_root(), "sapo-SA-attention")
    w = write_model(cfg, d)
    eng = wick.Engine.from_dir(d, dtype="float32", max_tokens=512)
    toks, other = random_tokens(cfg["vocab"], 100, seed=34), random_tokens(cfg["vocab"], 50, seed=35)
    s = eng.open_seq()
    eng.step([s], [toks])
    for keep in (64, 33):
        eng.truncate_seq(s, keep)
        got = step_rows(eng, s, other, [30] + [1] * 20)
        close(got, P.forward(cfg, w, toks[:keep] + other).float()[keep:], "float32", f"back to {keep}")


@pytest.mark.parametrize("name", ["SA", "SC", "SD"])
def test_greedy_generation_through_the_library_entry(name):
    cfg = CONFIGS[name]
    prompts = [random_tokens(cfg["vocab"], n, seed=50 + n) for n in (3, 40, 71)]
    eng = engine(name, "float32")
    out = wick.generate(eng, prompts, wick.GenOptions(max_tokens=24, sampler=wick.SamplerConfig.greedy()))
    for p, r in zip(prompts, out):
        assert len(r.tokens) == 24
        ref = plain(name, list(p) + r.tokens)               # (causal: row i is the prefix's last row)
        for i, t in enumerate(r.tokens):                    # every token is the plain model's best (or ties with it)
            row = ref[len(p) - 1 + i]
            assert row[t] >= row.max() - 1e-3, (name, len(p), i)
    # more requests than run together, and limits that end some early: the slots and pages go round
    out2 = wick.generate(eng, prompts * 3, wick.GenOptions(max_tokens=9, max_batch=2, sampler=wick.SamplerConfig.greedy()))
    assert [r.tokens for r in out2] == [r.tokens[:9] for r in out] * 3
    eng_b = engine(name, "bfloat16")
    out_b = wick.generate(eng_b, prompts, wick.GenOptions(max_tokens=8, sampler=wick.SamplerConfig.greedy()))
    for p, r in zip(prompts, out_b):
        assert len(r.tokens) == 8
        ref = plain(name, list(p) + r.tokens)
        for i, t in enumerate(r.tokens):
            row = ref[len(p) - 1 + i]
            assert row[t] >= row.max() - 0.05 * row.abs().max(), (name, len(p), i)


def test_the_command_line_writes_runs_and_times_the_design(tmp_path):
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    env = dict(os.environ, PYTHONPATH=root)
    cmd = [sys.executable, os.path.join(root, "bin", "wick")]
    cfg_path, d = str(tmp_path / "cfg.json"), str(tmp_path / "m")
    with open(cfg_path, "w") as f:
        json.dump(CONFIG_SA, f)
    r = subprocess.run(cmd + ["random", d, "--config", cfg_path, "--seed", "4"], capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr
    st = SafeTensorsDir(d)
    w = {n: st.get(n).tensor() for n in st.names()}
    prompts = [[5, 17, 3], [9, 9, 200, 1, 77, 3, 3, 14]]
    r = subprocess.run(cmd + ["run", d, "--ids", "5,17,3", "--ids", "9,9,200,1,77,3,3,14", "-n", "6", "-t", "0", "-q", "f32"],
                       capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr
    assert "Saposun" in r.stderr
    lines = [json.loads(l) for l in r.stdout.strip().splitlines()]
    for p, toks in zip(prompts, lines):
        assert len(toks) == 6
        ref = P.forward(CONFIG_SA, w, p + toks).float()
        for i, t in enumerate(toks):
            row = ref[len(p) - 1 + i]
            assert row[t] >= row.max() - 1e-3, (p, i)
    args = ["run", d, "--ids", "5,17,3", "-n", "12", "-t", "0.9", "--top-k", "20", "--seed", "7", "-q", "bf16"]
    a = subprocess.run(cmd + args, capture_output=True, text=True, env=env, timeout=600)
    b = subprocess.run(cmd + args, capture_output=True, text=True, env=env, timeout=600)
    assert a.returncode == 0 and a.stdout == b.stdout, a.stderr
    r = subprocess.run(cmd + ["bench", d, "--prompt-len", "16", "-n", "4", "--batch", "2", "-q", "bf16"],
                       capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0 and "tok/s" in r.stdout, r.stderr


def test_the_trace_runner_serves_the_design():
    name = "SD"
    d = model(name)[0]
    V = CONFIGS[name]["vocab"]
    a, b = random_tokens(V, 70, seed=61), random_tokens(V, 9, seed=62)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [0, 65]}, {"id": "y", "tokens": b[:5], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:67], "want": [0]}, {"id": "y", "tokens": b[5:6], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": a[67:68], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": a[68:69], "want": [0]}], "end": ["x"]}]
    out = os.path.join(tmp_root(), "sapo-trace-out")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out,
                        "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb = plain(name, a), plain(name, b)
    read = lambda i: torch.from_numpy(np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, V))
    close(read(0), ra[[0, 65]], "float32", "step 0")
    close(read(1), torch.stack([ra[66], rb[5]]), "float32", "step 1")
    assert not os.path.exists(os.path.join(out, "2.f32"))
    close(read(3), ra[68:69], "float32", "step 3")
