"""Kikopel's configuration, its spec, the cache's bookkeeping for its token history, and the plain implementation's own
invariants (no GPU)."""
import copy
import math

import pytest
import torch

import wick_b200 as wick
from wick_b200.cache import Cache
from wick_b200.config.base import ConfigError
from wick_b200.weights.loader import WeightError, load_weights
from wick_b200.weights.safetensors_io import SafeTensorsDir, write_safetensors
from helpers import tmp_root
from plain import kikopel_plain as P

LAT = dict(heads=2, dim=6, rot_dim=4, vdim=10, q_rank=14, kv_rank=12, scale=0.3, rot={"base": 1000.0, "dims": 4}, mask={"size": 9})
HG = dict(heads=3, dim=8, vdim=4)
CONFIG = dict(architecture="Kikopel", vocab=97, width=32, norm={"eps": 1e-5}, residual_mult=0.4,
              embedding={"scale": 2.0, "bigram": {"buckets": 53, "mul_prev": 11, "mul_cur": 5}}, layers=[
    dict(type="hgrn2", mixer=HG, mlp={"kind": "dense", "ff": 40}),
    dict(type="latent_attention", mixer=LAT, mlp=None),
    dict(type="latent_attention", mixer={k: v for k, v in LAT.items() if k != "mask"}, mlp={"kind": "dense", "ff": 24}),
    dict(type="hgrn2", mixer=HG, mlp=None),
])


def test_config_round_trip_and_registry():
    cfg = wick.config_from_json(CONFIG)
    assert isinstance(cfg, wick.KikopelConfig) and cfg.vocab == 97 and len(cfg.layers) == 4
    assert cfg.residual_mult == 0.4 and cfg.embedding_scale == 2.0 and cfg.norm_eps == 1e-5
    assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (53, 11, 5)
    assert cfg.layers[1].mixer.mask_size == 9 and cfg.layers[2].mixer.mask_size is None and cfg.layers[1].ff is None
    assert cfg.layers[1].mixer.rot_base == 1000.0 and cfg.layers[0].ff == 40 and cfg.layers[3].mixer.vdim == 4
    assert wick.config_from_json(cfg.to_json()) == cfg
    assert "Kikopel" in wick.architecture_names()
    bare = copy.deepcopy(CONFIG)
    bare.pop("embedding"), bare.pop("residual_mult")
    c2 = wick.config_from_json(bare)
    assert c2.bigram is None and c2.embedding_scale == 1.0 and c2.residual_mult == 1.0
    assert wick.config_from_json(c2.to_json()) == c2


@pytest.mark.parametrize("breakage", [
    lambda c: c.pop("vocab"), lambda c: c.pop("norm"), lambda c: c["layers"][0]["mixer"].pop("vdim"), lambda c: c["layers"][0].pop("mixer"),
    lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][0]["mlp"].update(kind="gated"),
    lambda c: c["layers"][0]["mlp"].pop("ff"), lambda c: c["layers"][1]["mixer"].pop("q_rank"), lambda c: c["layers"][1]["mixer"].pop("rot"),
    lambda c: c["layers"][1]["mixer"]["rot"].pop("base"), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=2),
    lambda c: c["layers"][1]["mixer"].update(rot_dim=5, rot={"base": 10.0, "dims": 5}), lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), lambda c: c["layers"][1]["mixer"]["mask"].pop("size"),
    lambda c: c["embedding"]["bigram"].pop("buckets"), lambda c: c["embedding"]["bigram"].update(mul_cur=-1),
    lambda c: c["embedding"]["bigram"].update(buckets=0), lambda c: c.update(residual_mult="x"), lambda c: c.update(layers=[])])
def test_broken_configs_are_refused(breakage):
    c = copy.deepcopy(CONFIG)
    breakage(c)
    with pytest.raises(ConfigError):
        wick.config_from_json(c)


def test_spec_names_every_tensor():
    cfg = wick.config_from_json(CONFIG)
    spec = wick.get_architecture("Kikopel").build_spec(cfg)
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3] and spec.layers[1].ffn.kind == "none" and spec.layers[0].ffn.kind == "mlp"
    m = wick.Model(spec, torch.float32, "cpu")
    table = m.tensor_table()
    for n, shape in {"embed": (97, 32), "bigram": (54, 32), "final.norm": (), "head": (97, 32), "l0.norm1": (), "l0.norm2": (),
                     "l0.mix.q": (24, 32), "l0.mix.f": (24, 32), "l0.mix.f.b": (24,), "l0.mix.lower": (24,), "l0.mix.v": (12, 32),
                     "l0.mix.norm": (4,), "l0.mix.o": (32, 12), "l0.mlp.up": (40, 32), "l0.mlp.down": (32, 40), "l0.mlp.act": (4,),
                     "l1.mix.dq": (14, 32), "l1.mix.dq.norm": (14,), "l1.mix.uq": (20, 14), "l1.mix.dkv": (16, 32),
                     "l1.mix.dkv.norm": (12,), "l1.mix.uk": (12, 12), "l1.mix.uv": (20, 12), "l1.mix.g": (20, 32),
                     "l1.mix.o": (32, 20)}.items():
        assert table[n].shape == shape, (n, table[n].shape)
    assert table["l1.norm2"].optional and "l1.mlp.up" not in table and "l1.mix.sink" not in table
    needs = m.cache_needs()
    assert [n.kind for n in needs] == ["state", "paged_rows", "paged_rows", "state", "paged_rows"]
    assert needs[0].shape == (3 * 8 * 4,) and needs[1].shape == (16,) and needs[4].shape == (1,) and needs[4].dtype == torch.int32
    n_params = sum(math.prod(ts.shape) for name, ts in table.items() if ts.init != "absent")
    assert cfg.param_count() == n_params
    bare = copy.deepcopy(CONFIG)
    bare["embedding"].pop("bigram")
    m2 = wick.Model(wick.get_architecture("Kikopel").build_spec(wick.config_from_json(bare)), torch.float32, "cpu")
    assert "bigram" not in m2.tensor_table() and len(m2.cache_needs()) == 4


def test_the_cache_keeps_the_tokens_beside_the_rows():
    m = wick.Model(wick.get_architecture("Kikopel").build_spec(wick.config_from_json(CONFIG)), torch.bfloat16, "cpu")
    cache = Cache(m.cache_needs(), max_tokens=256, dtype=torch.bfloat16, device="cpu")
    kinds = sorted((g.need.kind, tuple(g.need.shape), len(g.entries), str(g.dtype)) for g in cache.groups)
    assert kinds == [("paged_rows", (1,), 1, "torch.int32"), ("paged_rows", (16,), 2, "torch.bfloat16"), ("state", (96,), 2, "torch.float32")]
    view = cache.view(4)
    assert view.rows.dtype == torch.int32 and view.rows.shape == (5, 64, 1)
    assert cache.bytes_per_token() == 2 * 16 * 2 + 4


def test_a_random_model_folder_loads_and_the_plain_model_is_causal():
    d = wick.write_random_model(wick.config_from_json(CONFIG), 3, tmp_root() + "/kiko-cpu", std=0.3)
    st = SafeTensorsDir(d)
    w = {n: st.get(n).tensor() for n in st.names()}
    assert "l1.norm2" not in w and w["l0.norm1"].shape == () and w["l0.mix.lower"].min() > 0 and w["l0.mix.lower"].max() < 1
    toks = list(range(40))
    taps = []
    z = P.forward(CONFIG, w, toks, taps=taps)
    assert z.shape == (40, 97) and len(taps) == 4 and torch.isfinite(z).all()
    other = list(toks)
    other[10] = 96
    z2 = P.forward(CONFIG, w, other)
    assert torch.allclose(z[:10], z2[:10], rtol=0, atol=1e-11) and all((z[i] - z2[i]).abs().max() > 1e-7 for i in range(10, 40))
    m = wick.Model(wick.get_architecture("Kikopel").build_spec(wick.config_from_json(CONFIG)), torch.float32, "cpu")
    load_weights(m, d)
    for n in ("bigram", "embed", "l1.mix.g", "l1.mix.dkv", "l0.mix.f", "l0.mix.v", "l0.mlp.act", "l0.norm1", "final.norm", "head"):
        assert torch.equal(m.tensor(n).float(), w[n].float()), n
    assert torch.allclose(m.blocks[0].mixer_norm.weight, (0.4 * w["l0.norm1"].float()).expand(32))
    assert torch.allclose(m.final_norm.weight, w["final.norm"].float().expand(32))
    w["l0.norm1"] = torch.ones(32)
    write_safetensors(d + "/model.safetensors", w)
    with pytest.raises(WeightError):
        load_weights(m, d)


def test_plain_mechanisms_on_small_cases():
    assert P.pair_rows(torch.tensor([5, 7, 7, 0]), 10, 3, 2).tolist() == [10, (15 + 14) % 10, (21 + 14) % 10, 21 % 10]
    # a pair (1, 0) at position 1 with a frequency of one turns by one radian; entry i meets entry i + dr / 2
    x = torch.zeros(2, 4).double()
    x[:, 0] = 1.0
    y = P.turn(x, 100.0)
    assert torch.allclose(y[0], x[0]) and torch.allclose(y[1], torch.tensor([math.cos(1), 0, math.sin(1), 0]).double())
    x = torch.zeros(3, 4).double()
    x[:, 3] = 1.0
    y = P.turn(x, 100.0)                                     # the second pair turns by base^(-1/2) a position, the other way round
    assert torch.allclose(y[2], torch.tensor([0, -math.sin(0.2), 0, math.cos(0.2)]).double())
    vis = P.visible(5, 2)
    assert vis.sum(1).tolist() == [1, 2, 2, 2, 2] and vis[4, 3] and not vis[4, 2] and P.visible(5, None).sum() == 15
    # one key channel and one value: f = 1/2 writes one half
    q, v, f = torch.ones(3, 1, 1).double(), torch.tensor([2.0, 4.0, 6.0]).double().view(3, 1, 1), torch.full((3, 1, 1), 0.5).double()
    o, S = P.forgetting_outer_products(q, v, f)
    assert o.flatten().tolist() == [1.0, 2.5, 4.25] and S.item() == 4.25
    # f = 1 keeps and writes nothing; the factor acts on key channels (rows)
    f2 = torch.tensor([1.0, 0.0]).double().expand(2, 1, 2)
    o2, S2 = P.forgetting_outer_products(torch.ones(2, 1, 2).double(), v[:2], f2)
    assert o2.flatten().tolist() == [2.0, 4.0] and S2.flatten().tolist() == [0.0, 4.0]
    t = {"m.f": torch.zeros(4, 3).double(), "m.f.b": torch.zeros(4).double(), "m.lower": torch.tensor([0.0, 0.2, 0.5, 1.0]).double()}
    ff = P.forget_factors(torch.ones(1, 3).double(), t, "m.", dict(heads=2, dim=2))
    assert torch.allclose(ff, torch.tensor([0.5, 0.6, 0.75, 1.0]).double().view(1, 2, 2))
    z = torch.tensor([[3.0, -4.0]]).double()
    got = P.poly_norm(z, torch.tensor([1.0, 0.0, 0.0, 0.5]).double(), 0.0)
    assert torch.allclose(got, z / math.sqrt(12.5) + 0.5)
    got = P.poly_norm(z, torch.tensor([0.0, 2.0, 1.0, 0.0]).double(), 0.0)
    want = 2 * torch.tensor([9.0, 16.0]) / math.sqrt((81 + 256) / 2) + torch.tensor([27.0, -64.0]) / math.sqrt((729 + 4096) / 2)
    assert torch.allclose(got[0], want.double())
