"""The Kikopel decoder and its mechanisms against the plain implementation in ``tests/plain/kikopel_plain.py``: every
mechanism alone through its part or kernel, then whole models through the engine (prompts, decoding, portions, batches,
reused pages, slots and records, far tokens and window edges, generation).  The configurations differ from each other in
every size and option and include the values that make mechanisms vanish or coincide (no pair table, a pair table of one
row and the first token's, factors of one, a window of one position and of more than the prompt, no window, no
feed-forward, one head, widths and head sizes that are no multiples of four)."""
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
from wick_b200.parts import attention as _att, feedforward as _ff, latent_attention as _lat, linear_attention as _gla  # noqa: E402,F401
from wick_b200.parts.standard import NormedSumResidual  # noqa: E402
from wick_b200.weights.safetensors_io import SafeTensorsDir, write_safetensors  # noqa: E402
from helpers import random_tokens, tmp_root  # noqa: E402
from plain import kikopel_plain as P  # noqa: E402

PAGE = 64
DEV = "cuda"


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=10000.0, window=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
             rot={"base": base, "dims": rot_dim})
    if window is not None:
        m["mask"] = {"size": window}
    return m


def hg(heads, dim, vdim):
    return dict(heads=heads, dim=dim, vdim=vdim)


def layer(mixer, ff):
    kind = "latent_attention" if "kv_rank" in mixer else "hgrn2"
    return dict(type=kind, mixer=mixer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def emb(scale, buckets=None, mul_prev=0, mul_cur=0):
    e = {"scale": scale}
    if buckets is not None:
        e["bigram"] = dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)
    return e


# KA: small windows; layers without feed-forward
CONFIG_KA = dict(architecture="Kikopel", vocab=211, width=64, norm={"eps": 1e-5}, residual_mult=0.35, embedding=emb(2.0, 97, 13, 5), layers=[
    layer(hg(3, 8, 4), 80), layer(lat(3, 12, 8, 20, 28, 24, 0.3, 1000.0, 17), None), layer(lat(4, 8, 4, 12, 16, 20, 0.4, 500.0, 64), 56),
    layer(hg(1, 16, 16), None), layer(lat(2, 16, 16, 16, 32, 40, 0.2, 20000.0, 70), 128)])
# KB: no pair table, factors of one, no window
CONFIG_KB = dict(architecture="Kikopel", vocab=130, width=72, norm={"eps": 1e-3}, residual_mult=1.0, embedding=emb(1.0), layers=[
    layer(lat(6, 10, 6, 8, 20, 16, 0.35), 52), layer(hg(2, 24, 20), 44), layer(lat(1, 24, 8, 40, 36, 32, 0.25, 100.0), None)])
# KC: sizes that the tensor-core attention takes; states of 128 x 128 and 64 x 96
CONFIG_KC = dict(architecture="Kikopel", vocab=300, width=128, norm={"eps": 1e-5}, residual_mult=0.5, embedding=emb(0.8, 500, 300, 1), layers=[
    layer(lat(2, 48, 16, 64, 96, 72, 0.125, 10000.0, 100), 256), layer(hg(2, 64, 96), 192), layer(lat(4, 32, 16, 48, 64, 80, 0.15, 300.0, 65), 64),
    layer(hg(1, 128, 128), 128), layer(lat(2, 96, 32, 128, 64, 136, 0.09), 96)])
# KD: a width that is no multiple of eight, odd sizes everywhere, a window of one position, a pair table of one bucket
CONFIG_KD = dict(architecture="Kikopel", vocab=77, width=100, norm={"eps": 1e-6}, residual_mult=1.4, embedding=emb(0.5, 1, 7, 3), layers=[
    layer(lat(5, 7, 6, 9, 11, 13, 0.3, 50.0, 1), 50), layer(hg(5, 9, 7), 37), layer(lat(3, 5, 2, 6, 10, 15, 0.45, 9.0, 128), None),
    layer(hg(2, 6, 10), 90)])
CONFIGS = {"KA": CONFIG_KA, "KB": CONFIG_KB, "KC": CONFIG_KC, "KD": CONFIG_KD}
_models = {}
STD = 0.15


def write_model(cfg, d, seed=5, std=STD):
    wick.write_random_model(wick.config_from_json(cfg), seed, d, std=std)
    st = SafeTensorsDir(d)
    return {n: st.get(n).tensor() for n in st.names()}


def model(name, seed=5):
    if (name, seed) not in _models:
        d = os.path.join(tmp_root(), f"kiko-{name}-{seed}")
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
    """Whole models: rounding of several layers.  In bfloat16 at most one row in forty (a head whose sum nearly vanishes is
    normed all the same, which magnifies rounding) may be further away than the tolerance, up to four times."""
    if dtype == "float32":
        return tight(got, ref, dtype, what, tol or 2e-4)
    tol = tol or 5e-2
    tight(got, ref, dtype, what, 4 * tol)
    scale = max(1e-6, ref.abs().max().item())
    far = ((got.detach().float().cpu() - ref).abs().max(-1).values > tol * scale).sum().item()
    assert far <= max(1, ref.shape[0] // 40), f"{what}: {far} of {ref.shape[0]} rows are off by more than {tol}"


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


LAT_NAMES = dict(dq="dq", dq_norm="dq.norm", uq="uq", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", gate="g", o="o")
HG_NAMES = dict(q="q", forget="f", forget_bias="f.b", lower="lower", v="v", norm="norm", o="o")


def lat_part(dtype, width, m, eps, g, std=0.3, change=None):
    H, d, dr, e, qr, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
    t = {"dq": rnd(g, qr, width, std=std), "dq.norm": 1 + 0.3 * rnd(g, qr), "uq": rnd(g, H * (d + dr), qr, std=std),
         "dkv": rnd(g, r + dr, width, std=std), "dkv.norm": 1 + 0.3 * rnd(g, r), "uk": rnd(g, H * d, r, std=std),
         "uv": rnd(g, H * e, r, std=std), "g": rnd(g, H * e, width, std=std), "o": rnd(g, width, H * e, std=std)}
    if change:
        change(t)
    params = {"width": width, "heads": H, "head_dim": d, "rot_dim": dr, "v_dim": e, "q_rank": qr, "kv_rank": r, "scale": m["scale"],
              "eps": eps, "position": PartSpec("rotary_pairs", {"head_dim": dr, "dims": dr, "theta": m["rot"]["base"], "pairing": "halves"}),
              "window": (m.get("mask") or {}).get("size"), "sink": False, "gate": "element", "names": LAT_NAMES}
    return make_part("mixer", "latent_attention", params, dtype, t)


def hg_part(dtype, width, m, eps, g, std=0.3, change=None):
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    t = {"q": rnd(g, H * dk, width, std=std), "f": rnd(g, H * dk, width, std=std), "f.b": rnd(g, H * dk),
         "lower": torch.rand(H * dk, generator=g), "v": rnd(g, H * dv, width, std=std), "norm": 1 + 0.3 * rnd(g, dv),
         "o": rnd(g, width, H * dv, std=std)}
    if change:
        change(t)
    params = {"width": width, "heads": H, "head_dim": dk, "v_dim": dv, "eps": eps, "names": HG_NAMES}
    return make_part("mixer", "hgrn2", params, dtype, t)


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
@pytest.mark.parametrize("width,scale,buckets,mp,mc", [(64, 2.0, 97, 13, 5), (101, 1.0, 1, 3, 4), (6, 0.25, 1000, 2_000_003, 1_999_999),
                                                       (300, -1.5, 33, 0, 1), (8, 0.5, 40, 7, 0)])
def test_embedding_rows_times_a_factor_plus_the_pairs_rows(dtype, width, scale, buckets, mp, mc):
    g = torch.Generator().manual_seed(width)
    vocab, n = 5000, 210
    part, t = make_part("embedding", "table", {"vocab": vocab, "width": width, "tensor": "embed", "scale": scale, "pairs": dict(
        tensor="bigram", buckets=buckets, mul_prev=mp, mul_cur=mc)}, dtype, {"embed": rnd(g, vocab, width), "bigram": rnd(g, buckets + 1, width)})
    toks = torch.randint(0, vocab, (n,), generator=g)
    toks[:3] = vocab - 1                                    # (products beyond 32 bits for the large factors)
    ref = P.embed(toks, t["embed"], scale, t["bigram"], dict(buckets=buckets, mul_prev=mp, mul_cur=mc))
    ids = toks.tolist()
    need = part.cache_need()
    assert need.kind == "paged_rows" and need.dtype == torch.int32
    for cuts in ([n], [1] * 70 + [2, 56, 1, 1, 80], [63, 1, 1, 63, 82], [64, 64, 2, 80]):
        history = torch.full((6, PAGE, 1), 4242, dtype=torch.int32, device=DEV)
        at, out = 0, []
        for c in cuts:
            out.append(part.forward_step(seq_batch(c, at, ids[at:at + c]), View(rows=history)))
            at += c
        got = torch.cat(out)
        assert got.dtype == torch.float32
        tight(got, ref, "float32", f"cuts {cuts[:3]}", 1e-6)
        assert torch.equal(history[1:5].reshape(-1)[:n].cpu(), toks.int())
    # unequal sequences in one step, each after tokens of its own; pages in any order; the first token of each is the table's last row
    history = torch.full((9, PAGE, 1), 4242, dtype=torch.int32, device=DEV)
    seqs, pages, starts = [ids[:70], ids[70:75], ids[75:205]], [[7, 3], [5], [2, 8, 4]], [0, 0, 0]
    refs = [P.embed(torch.tensor(s), t["embed"], scale, t["bigram"], dict(buckets=buckets, mul_prev=mp, mul_cur=mc)) for s in seqs]
    first = part.forward_step(make_batch([seqs[0][:64], seqs[1][:1], seqs[2][:127]], starts, pages, [1, 2, 3]), View(rows=history))
    tight(first, torch.cat([refs[0][:64], refs[1][:1], refs[2][:127]]), "float32", "first", 1e-6)
    then = part.forward_step(make_batch([seqs[2][127:], seqs[1][1:], seqs[0][64:65]], [127, 1, 64], [pages[2], pages[1], pages[0]], [3, 2, 1]),
                             View(rows=history))
    tight(then, torch.cat([refs[2][127:], refs[1][1:], refs[0][64:65]]), "float32", "then", 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,eps,factor,ffn", [(64, 1e-5, 0.35, True), (101, 1e-2, 1.0, False), (6, 1e-6, -1.4, True), (2304, 1e-5, 0.6, True)])
def test_the_sublayers_read_the_stream_and_their_results_are_normed_by_one_number(dtype, width, eps, factor, ffn):
    """The block with a mixer and a feed-forward that note what they read and return given partial sums."""
    g = torch.Generator().manual_seed(width)
    ctx = BuildContext(dtype=TORCH[dtype], device=torch.device(DEV))
    n = 11
    seen, results = [], [0.5 * rnd(g, 3, n, width), 20 * rnd(g, 1, n, width)]

    class M(Mixer):
        def forward(self, x, batch, cache, write_cache):
            seen.append(x.clone())
            return results[0].to(DEV)

    class F(FeedForward):
        IS_NONE = not ffn

        def forward(self, x, batch):
            seen.append(x.clone())
            return results[1].to(DEV)

    norms = []
    for w in (1.7, -0.4):
        p = build_part("norm", PartSpec("rms", {"width": width, "eps": eps, "tensor": "", "one_number": True, "factor": factor}), ctx)
        assert p.tensor_specs()[0].shape == ()
        p.load(lambda nm: torch.tensor(w))
        assert p.tensor("").shape == ()
        norms.append(p)
    block = NormedSumResidual({}, ctx, M({}, ctx), norms[0], F({}, ctx), norms[1])
    x = 3 * rnd(g, n, width)
    h = Hidden(x.clone().to(DEV))
    for _ in range(2):                                      # (two such layers: the second resolves what the first left pending)
        h = block.forward(h, None, None, True)
    want, reads = x.double(), []
    for _ in range(2):
        for k in (0, 1) if ffn else (0,):
            reads.append(want.clone())
            want = want + factor * P.norm(results[k].double().sum(0), (1.7, -0.4)[k], eps)
    for i, (s, r) in enumerate(zip(seen, reads)):
        tight(s, r, "float32", f"sublayer {i} reads", 2e-6 if dtype == "float32" else 5e-3)
    tight(h.resolved(), want, "float32", "the stream", 2e-6)
    # a norm by one number after everything (what the head reads), over chosen rows with the last sum pending
    h = Hidden(x.clone().to(DEV))
    h = block.forward(h, None, None, True)
    rows = torch.tensor([3, 3, 10, 0], dtype=torch.int32, device=DEV)
    got = norms[1].add_forward(h.x, h.pending, torch.float32, rows, rms=h.rms)
    half = reads[2] if ffn else reads[1]
    tight(got, factor * P.norm(half, -0.4, eps)[[3, 3, 10, 0]], "float32", "final norm", 3e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [lat(3, 12, 8, 20, 28, 24, 0.3, 1000.0, 17), lat(2, 16, 16, 16, 32, 40, 0.2, 20000.0, 64), lat(5, 7, 6, 9, 11, 13, 0.3, 50.0, 1),
                               lat(4, 48, 16, 64, 96, 72, 0.125, 10000.0, 65), lat(2, 96, 32, 128, 64, 136, 0.09), lat(1, 24, 8, 40, 36, 32, 0.25, 100.0, 129),
                               lat(6, 32, 64, 48, 40, 200, 0.1, 300.0, 128), lat(2, 8, 8, 136, 24, 16, 0.2, 10.0, 63), lat(3, 5, 2, 6, 10, 15, 0.45, 9.0, 400),
                               lat(8, 128, 64, 112, 48, 512, 0.05, 5000.0, 70)],
                         ids=lambda m: f"h{m['heads']}d{m['dim']}+{m['rot_dim']}v{m['vdim']}r{m['kv_rank']}w{(m.get('mask') or {}).get('size')}")
def test_latent_attention_with_a_gate_per_element_in_any_portions(dtype, m):
    g = torch.Generator().manual_seed(m["heads"] * 100 + m["dim"])
    width, n = 48, 210
    part, t = lat_part(dtype, width, m, 1e-5, g)
    h = rnd(g, n, width)
    ref = P.latent_attention(as_held(h, dtype), t, "", m, 1e-5)
    for cuts in ([n], [1] * 5 + [2, 60, 2, 3, 64, 74], [70] + [1] * 5 + [17, 118], [209, 1]):
        tight(run_mixer(part, h, dtype, cuts, rows_view(part, dtype)), ref, dtype, f"cuts {cuts[:3]}")
    # the gate matters element by element, and so do the rotation's layout and the latents' norm
    flat = P.latent_attention(as_held(h, dtype), dict(t, g=torch.zeros_like(t["g"])), "", m, 1e-5)
    assert (flat - ref).abs().max() > 0.1 * ref.abs().max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 129, None])
def test_a_key_that_stands_out_just_inside_and_just_outside_the_window(dtype, window):
    """The latent's first 64 rows of Wdkv are Wdq, a head's keys are that half of the latent, its values are made from the
    other half, whose rows see only what Wdq maps to zero, and there is no rotated part.  A score is then the product of two
    normed vectors of 64 numbers: about 64 * scale where h_j is h_i with that part negated, as for j = i, and a few units of
    8 * scale elsewhere; the value of such a twin is the negated value, so a result is v_i where the twin is not seen and
    vanishes where it is.  Twins stand just inside and just outside the window, at page borders and far away; the rows are
    checked in a prompt, in portions and decoded alone."""
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
    w = window or n
    pairs = []
    for i in (70, 127, 128, 192, 255, 300, 383, 448, 511, 515):
        k = len(pairs) % 2                                  # the oldest key that is seen, or the newest that is not
        j = i - w + 1 - k
        if window is None:
            j = (3, 0, 63, 64, 1, 62, 65, 5, 129, 2)[len(pairs)]
        pairs.append((i, j))
    pairs = [(i, j) for i, j in pairs if 0 <= j < i and j not in {a for a, _ in pairs}]
    for i, j in pairs:
        h[j] = h[i] - 2 * null @ (null.T @ h[i])
    ref = P.latent_attention(as_held(h, dtype), t, "", m, 1e-6)
    h2 = h.clone()
    for i, j in pairs:
        h2[j] = rnd(g, width)
    ref2 = P.latent_attention(as_held(h2, dtype), t, "", m, 1e-6)
    for i, j in pairs:                                      # a twin that is seen matters, one that is not does not
        moved = (ref2[i] - ref[i]).abs().max() > 0.1 * ref.abs().max()
        assert bool(moved) == (i - j < w), (i, j)
    for cuts in ([n], [64, 64, 2, 190, 200], [256, 2, 262]):
        tight(run_mixer(part, h, dtype, cuts, rows_view(part, dtype)), ref, dtype, f"cuts {cuts[:3]}")
    for i, j in pairs[:7]:                                  # decoded: i alone after a prompt that ends right before it
        got = run_mixer(part, h[:i + 1], dtype, [i, 1], rows_view(part, dtype))
        tight(torch.cat([ref[:i].float(), got[i:].cpu()]), ref[:i + 1], dtype, f"position {i} decoded, its twin at {j}")


def test_the_first_token_sees_itself_alone():
    g = torch.Generator().manual_seed(2)
    width, m = 24, lat(2, 8, 4, 12, 10, 16, 0.5, 100.0, 5)
    part, t = lat_part("float32", width, m, 1e-5, g)
    h = rnd(g, 1, width)
    c = P.norm(h.double() @ t["dkv"][:16].T, t["dkv.norm"], 1e-5)
    want = (torch.sigmoid(h.double() @ t["g"].T) * (c @ t["uv"].T)) @ t["o"].T
    tight(run_mixer(part, h, "float32", [1], rows_view(part, "float32")), want, "float32", "its own value")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv", [(3, 8, 4), (2, 16, 16), (1, 6, 10), (2, 128, 128), (4, 20, 36), (1, 300, 8), (2, 64, 96), (5, 9, 7), (3, 100, 12)])
def test_hgrn2_in_any_portions(dtype, H, dk, dv):
    g = torch.Generator().manual_seed(H * 1000 + dk)
    width, n = 40, 350                                       # (a step of 192 tokens or more is scanned in chunks of 64)
    m = hg(H, dk, dv)

    def change(t):                                           # bounds of zero and near one beside those in between
        t["lower"][0], t["lower"][-1] = 0.0, 0.999

    part, t = hg_part(dtype, width, m, 1e-5, g, change=change)
    h = rnd(g, n, width)
    ref = P.hgrn2(as_held(h, dtype), t, "", m, 1e-5)
    f = P.forget_factors(as_held(h, dtype), t, "", m)
    assert f.min() < 0.3 and f.max() > 0.99
    for cuts in ([n], [1] * 6 + [2, 3, 2, 59, 64, 1, 1, 12, 200], [349, 1], [75, 75, 8, 192], [192, 158]):
        tight(run_mixer(part, h, dtype, cuts, record_view(part)), ref, dtype, f"cuts {cuts[:3]}")


@pytest.mark.parametrize("H,dk,dv", [(2, 5, 3), (1, 8, 12), (3, 16, 4)])
def test_the_recurrence_and_the_per_head_norm_on_their_own(H, dk, dv):
    """ops.hgrn2_mix from given partial sums: the state after the step, [H][dv][dk] in the record, is the plain
    recurrence's last state; logits of +-100 give factors of one and of the bound without a NaN."""
    g = torch.Generator().manual_seed(8)
    n = 70
    q, z, v = 2 * rnd(g, n, H * dk), 3 * rnd(g, n, H * dk), rnd(g, n, H * dv)
    z[5, 0], z[6, 0], q[7, 0], q[8, 0] = 100.0, -100.0, 100.0, -100.0
    bias, lower = rnd(g, H * dk), torch.rand(H * dk, generator=g)
    whole = torch.cat([q, z, v], -1)
    a = rnd(g, n, whole.shape[1])
    parts = torch.stack([whole - a, a]).to(DEV)             # (two partial sums)
    f = (lower + (1 - lower) * torch.sigmoid(z.double() + bias)).view(n, H, dk)
    o, S = P.forgetting_outer_products(P.silu(q.double()).view(n, H, dk), v.double().view(n, H, dv), f)
    rec = torch.full((3, H * dv * dk), float("nan"), device=DEV)
    for cuts in ([n], [1] * 5 + [65], [2, 1, 67]):
        rec[1].zero_()
        outs, at = [], 0
        for c in cuts:
            outs.append(ops.hgrn2_mix(parts[:, at:at + c].contiguous(), heads=H, key_dim=dk, v_dim=dv, bias=bias.to(DEV), lower=lower.to(DEV),
                                      records=rec, batch=seq_batch(c, at)))
            at += c
        tight(torch.cat(outs), o.reshape(n, H * dv), "float32", f"o, cuts {cuts[:2]}")
        tight(rec[1].view(H, dv, dk), S.transpose(1, 2), "float32", f"the record, cuts {cuts[:2]}")
        assert torch.isnan(rec[0]).all() and torch.isnan(rec[2]).all()
    w = 1 + 0.3 * rnd(g, dv)
    got = ops.gla_norm_gate(torch.cat(outs), None, 0, H, dv, w.to(DEV), 1e-3, torch.float32)
    tight(got, P.norm(o, w.double(), 1e-3).reshape(n, H * dv), "float32", "norm")


def test_the_state_remembers_a_token_hundreds_of_positions_back():
    """With bounds of 0.999 the state keeps what one early token wrote: the result 500 positions later moves when that
    token changes, in a prompt, in portions and token by token, as the plain one does; with bounds of zero and logits of
    -9 nothing of it is left a few tokens later."""
    g = torch.Generator().manual_seed(3)
    width, n, m = 24, 520, hg(2, 6, 10)

    def remembers(t):
        t["lower"] = torch.full((12,), 0.999)

    def forgets(t):
        t["lower"], t["f"], t["f.b"] = torch.zeros(12), torch.zeros_like(t["f"]), torch.full((12,), -9.0)

    part, t = hg_part("float32", width, m, 1e-7, g, change=remembers)
    h = rnd(g, n, width, std=0.3)
    h2 = h.clone()
    h2[7] = 30 * rnd(g, width)
    ref, ref2 = (P.hgrn2(x.double(), t, "", m, 1e-7) for x in (h, h2))
    assert (ref[515:] - ref2[515:]).abs().max() > 1e-2 * ref.abs().max(), "the early token must show late"
    for cuts in ([n], [8, 400, 112], [500] + [1] * 20):
        tight(run_mixer(part, h, "float32", cuts, record_view(part)), ref, "float32", f"cuts {cuts[:3]}", tol=1e-4)
        tight(run_mixer(part, h2, "float32", cuts, record_view(part)), ref2, "float32", f"changed, cuts {cuts[:3]}", tol=1e-4)
    part3, t3 = hg_part("float32", width, m, 1e-7, g, change=forgets)
    r3, r32 = (P.hgrn2(x[:40].double(), t3, "", m, 1e-7) for x in (h, h2))
    assert (r3[12:] - r32[12:]).abs().max() < 1e-9 * r3.abs().max() and (r3[7] - r32[7]).abs().max() > 1e-3
    tight(run_mixer(part3, h2[:40], "float32", [5, 1, 1, 1, 32], record_view(part3)), r32, "float32", "strong forgetting")


def test_the_first_tokens_start_from_zeros_not_from_the_record_of_the_slots_last_user():
    g = torch.Generator().manual_seed(4)
    width, m = 24, hg(2, 6, 10)
    part, t = hg_part("float32", width, m, 1e-5, g)
    h = rnd(g, 9, width)
    ref = P.hgrn2(h.double(), t, "", m, 1e-5)
    view = record_view(part)
    run_mixer(part, rnd(g, 30, width), "float32", [30], view)          # another sequence leaves its record in slot 1
    assert view.state[1].abs().max() > 0
    for cuts in ([9], [1, 1, 1, 2, 4]):
        view.state[1].zero_()                                 # (what the cache does when a sequence opens in the slot)
        tight(run_mixer(part, h, "float32", cuts, view), ref, "float32", f"cuts {cuts}")
    assert torch.isnan(view.state[2]).all() and torch.isnan(view.state[0]).all(), "another slot's record was written"


@pytest.mark.parametrize("splits,n,ff,eps", [(1, 5, 40, 1e-5), (3, 9, 37, 1e-2), (2, 3, 4096, 1e-5), (1, 2, 13000, 1e-5), (4, 2, 25604, 1e-3),
                                             (1, 2, 30001, 1e-5), (6, 1, 1, 1e-6), (1, 300, 256, 1e-5)])
def test_poly_norm(splits, n, ff, eps):
    g = torch.Generator().manual_seed(ff)
    parts = 0.7 * rnd(g, splits, n, ff)
    parts[:, 0] *= 0.02                                     # a row so small that eps shows in the means of the powers
    z = parts.double().sum(0)
    for co in (torch.tensor([0.5, -1.2, 0.8, 0.3]), torch.tensor([0.0, 0.0, 2.0, 0.0]), torch.tensor([1.0, 1.0, 1.0, 1.0])):
        ref = P.poly_norm(z, co.double(), eps)
        for dtype in DTYPES:
            tight(ops.poly_norm(parts.to(DEV), co.to(DEV), eps, TORCH[dtype]), ref, dtype, f"{co.tolist()}", 5e-6 if dtype == "float32" else 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(40, 72), (100, 50), (128, 256), (64, 33)])
def test_a_feed_forward_with_the_poly_norm_activation(dtype, width, ff):
    g = torch.Generator().manual_seed(21)
    t = {"up": rnd(g, ff, width, std=0.2), "down": rnd(g, width, ff, std=0.2), "act": torch.tensor([0.6, 0.9, -0.5, 0.2])}
    part, td = make_part("ffn", "mlp", {"width": width, "intermediate": ff, "activation": "poly_norm", "eps": 1e-4,
                                        "names": dict(up="up", down="down", coefficients="act")}, dtype, t)
    for n in (1, 7, 130):
        h = rnd(g, n, width)
        got = part.forward(h.to(DEV, TORCH[dtype]).contiguous(), seq_batch(n))
        tight(got.sum(0) if got.dim() == 3 else got, P.feed_forward(as_held(h, dtype), td, "", 1e-4), dtype, f"{n} tokens")


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
@pytest.mark.parametrize("name", ["KA", "KC"])
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
    name = "KA"
    toks = random_tokens(CONFIGS[name]["vocab"], 270, seed=12)
    eng = engine(name, dtype)
    s = eng.open_seq()
    close(step_rows(eng, s, toks, [3] + [1] * 267), plain(name, toks), dtype, "decoded")


def test_an_early_token_shows_in_the_logits_hundreds_of_positions_later():
    """Every forget factor's bound is set to 0.9995 and the early token's embedding row is large: changing token 2 moves the
    logits at position 600, in the plain model and in the engine, for a prompt in one step, in portions, and decoded."""
    cfg = CONFIGS["KA"]
    w = {k: v.clone() for k, v in model("KA")[1].items()}
    for k in list(w):
        if k.endswith(".lower"):
            w[k] = torch.full(w[k].shape, 0.9995, dtype=torch.float32)
    a = random_tokens(cfg["vocab"] - 1, 604, seed=14)
    a[2] = cfg["vocab"] - 1
    w["embed"][a[2]] *= 60.0
    b = list(a)
    b[2] = 17
    d = os.path.join(tmp_root(), "kiko-KA-remembers")
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
    """NaN (a number no token has, where integers are kept) in every page that no sequence holds, and NaN in every record of
    a slot that no sequence has."""
    held = eng.cache.pages.held()
    free = [p for p in range(1, eng.cache.n_pages) if p not in held]
    idle = [s for s in range(1, eng.cache.max_seqs + 1) if s not in set(eng.cache.seqs)]
    for g in eng.cache.groups:
        bad = float("nan") if g.dtype.is_floating_point else 987654
        if g.need.kind == "paged_rows" and free:
            g.storage[:, torch.tensor(free, device=g.storage.device)] = bad
        if g.need.kind == "state" and idle:
            g.storage[:, torch.tensor(idle, device=g.storage.device)] = bad


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_slots_and_records_that_were_given_back_are_used_again(dtype):
    name = "KA"
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
    eng = engine("KA", "float32")
    toks = random_tokens(CONFIGS["KA"]["vocab"], 40, seed=33)
    s = eng.open_seq()
    first = eng.step([s], [toks]).clone()
    with pytest.raises(ValueError):
        eng.truncate_seq(s, 20)                              # (the recurrences' records hold all 40 tokens)
    eng.truncate_seq(s, 0)
    eng.step([s], [toks[:17]], [[]])
    close(eng.step([s], [toks[17:]]), first, "float32", "again", 2e-5)
    # latent attention and the token history alone keep every position
    cfg = dict(CONFIGS["KA"], layers=[L for L in CONFIGS["KA"]["layers"] if L["type"] == "latent_attention"])
    d = os.path.join(tmp_root(), "kiko-KA-latent")
    w = write_model(cfg, d)
    eng = wick.Engine.from_dir(d, dtype="float32", max_tokens=512)
    toks, other = random_tokens(cfg["vocab"], 100, seed=34), random_tokens(cfg["vocab"], 30, seed=35)
    s = eng.open_seq()
    eng.step([s], [toks])
    for keep in (64, 33):
        eng.truncate_seq(s, keep)
        got = eng.step([s], [other], [list(range(30))])
        close(got, P.forward(cfg, w, toks[:keep] + other).float()[keep:], "float32", f"back to {keep}")


@pytest.mark.parametrize("name", ["KA", "KC", "KD"])
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
        json.dump(CONFIG_KA, f)
    r = subprocess.run(cmd + ["random", d, "--config", cfg_path, "--seed", "4"], capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr
    st = SafeTensorsDir(d)
    w = {n: st.get(n).tensor() for n in st.names()}
    prompts = [[5, 17, 3], [9, 9, 200, 1, 77, 3, 3, 14]]
    r = subprocess.run(cmd + ["run", d, "--ids", "5,17,3", "--ids", "9,9,200,1,77,3,3,14", "-n", "6", "-t", "0", "-q", "f32"],
                       capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr
    assert "Kikopel" in r.stderr
    lines = [json.loads(l) for l in r.stdout.strip().splitlines()]
    for p, toks in zip(prompts, lines):
        assert len(toks) == 6
        ref = P.forward(CONFIG_KA, w, p + toks).float()
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
    name = "KD"
    d = model(name)[0]
    V = CONFIGS[name]["vocab"]
    a, b = random_tokens(V, 70, seed=61), random_tokens(V, 9, seed=62)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [0, 65]}, {"id": "y", "tokens": b[:5], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:67], "want": [0]}, {"id": "y", "tokens": b[5:6], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": a[67:68], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": a[68:69], "want": [0]}], "end": ["x"]}]
    out = os.path.join(tmp_root(), "kiko-trace-out")
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
