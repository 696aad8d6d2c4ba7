"""The Saposun configuration, its spec, tensor names and cache needs, without a GPU; and the plain implementation's own
properties (what a query sees, the filter's start, the decay)."""
import copy
import json
import os

import pytest
import torch

import wick_b200 as wick
from wick_b200.cache.cache import Cache
from wick_b200.models.model import Model
from wick_b200.parts.base import CacheNeed
from wick_b200.weights.safetensors_io import SafeTensorsDir
from plain import saposun_plain as P

MOE = {"kind": "moe", "expert": {"ff": 40}, "router": {"experts": 5, "top": 2}}
CFG = dict(architecture="Saposun", vocab=97, width=48, norm={"eps": 1e-4}, residual_mult=0.6, layers=[
    dict(type="latent_attention", mixer=dict(heads=3, dim=10, rot_dim=6, vdim=8, q_rank=20, kv_rank=14, scale=0.3, rot={"base": 500.0, "dims": 6},
                                             mask={"size": 9}), mlp=MOE),
    dict(type="attention", mixer=dict(heads=4, kv_heads=2, dim=12, vdim=10, conv=3, scale=0.25, softcap=20.0, rot={"base": 900.0, "dims": 8},
                                      mask={"size": 11, "pool": 4}), mlp=None),
    dict(type="retention", mixer=dict(heads=2, dim=8, vdim=6, decay=[0.5, 1.0], rot={"base": 100.0, "dims": 4}), mlp=MOE),
    dict(type="latent_attention", mixer=dict(heads=2, dim=4, rot_dim=6, vdim=12, q_rank=16, kv_rank=14, scale=0.4, rot={"base": 500.0, "dims": 6},
                                             mask={"size": 30}, kv_from=0), mlp=MOE),
    dict(type="attention", mixer=dict(heads=2, kv_heads=1, dim=6, vdim=6, scale=0.3, rot={"base": 50.0, "dims": 6}), mlp=MOE)])


def changed(path, value):
    c = copy.deepcopy(CFG)
    at = c
    for k in path[:-1]:
        at = at[k]
    if value is KeyError:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return c


def test_the_configuration_round_trips_and_names_its_tensors():
    cfg = wick.config_from_json(CFG)
    assert isinstance(cfg, wick.SaposunConfig) and cfg.vocab == 97 and cfg.residual_mult == 0.6
    assert wick.config_from_json(json.loads(json.dumps(cfg.to_json()))) == cfg
    model = Model(wick.get_architecture("Saposun").build_spec(cfg), torch.float32, "cpu")
    table = model.tensor_table()
    shapes = {n: tuple(s.shape) for n, s in table.items()}
    assert shapes["embed"] == shapes["head"] == (97, 48) and shapes["final.norm"] == (48,)
    assert shapes["l0.mix.dkv"] == (20, 48) and shapes["l0.mix.uq"] == (48, 20) and shapes["l0.mix.uk"] == (30, 14)
    assert not any(n.startswith("l3.mix.dkv") for n in shapes) and shapes["l3.mix.uv"] == (24, 14)
    assert shapes["l1.mix.q.conv"] == (48, 3) and shapes["l1.mix.v.conv"] == (20, 3) and shapes["l1.mix.g"] == (4, 48)
    assert "l4.mix.q.conv" not in shapes and shapes["l4.mix.g"] == (2, 48)
    assert shapes["l2.mix.g"] == (12, 48) and shapes["l2.mix.o"] == (48, 12) and "l2.mix.norm" not in shapes
    assert shapes["l2.mlp.e4.down"] == (48, 40) and shapes["l2.mlp.router"] == (5, 48) and shapes["l2.mlp.correction"] == (5,)
    assert not any(n.startswith("l1.mlp") for n in shapes) and not any("norm2" in n for n in shapes)
    total = sum(torch.Size(s).numel() for s in shapes.values())
    assert total == cfg.param_count()


@pytest.mark.parametrize("path,value", [
    (("layers",), []), (("layers", 0, "type"), "gla"), (("width",), 0), (("norm", "eps"), KeyError), (("residual_mult",), None),
    (("layers", 0, "mixer", "kv_rank"), KeyError), (("layers", 0, "mixer", "rot", "dims"), 4), (("layers", 3, "mixer", "kv_from"), 1),
    (("layers", 3, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "kv_rank"), 16), (("layers", 3, "mixer", "rot", "base"), 400.0),
    (("layers", 1, "mixer", "kv_heads"), 3), (("layers", 1, "mixer", "mask", "pool"), 0), (("layers", 1, "mixer", "rot", "dims"), 14),
    (("layers", 1, "mixer", "rot", "dims"), 3), (("layers", 1, "mixer", "mask", "size"), 2.5), (("layers", 2, "mixer", "decay"), [0.5]),
    (("layers", 2, "mixer", "decay"), [0.5, "x"]), (("layers", 0, "mlp", "kind"), "dense"), (("layers", 0, "mlp", "router", "top"), 6),
    (("layers", 1, "mixer", "scale"), True)])
def test_what_the_file_lacks_or_has_wrong_is_an_error(path, value):
    with pytest.raises(wick.ConfigError):
        wick.config_from_json(changed(path, value))


def test_the_cache_holds_rows_keys_blocks_and_records():
    spec = wick.get_architecture("Saposun").build_spec(wick.config_from_json(CFG))
    assert [e.read_cache_of for e in spec.schedule] == [None, None, None, 0, None]
    needs = Model(spec, torch.bfloat16, "cpu").cache_needs()
    assert needs[0] == CacheNeed("paged_rows", shape=(20,)) and needs[3] is None
    kv, blocks, record = needs[1].parts
    assert (kv.kind, kv.kv_heads, kv.head_dim, kv.v_head_dim) == ("paged_kv", 2, 12, 10)
    assert (blocks.kind, blocks.block, blocks.kv_heads, blocks.head_dim, blocks.v_head_dim) == ("paged_blocks", 4, 2, 12, 10)
    assert record.kind == "state" and record.shape == (2 * (48 + 24 + 20),) and record.dtype == torch.float32
    assert needs[2] == CacheNeed("state", shape=(96,), dtype=torch.float32)
    assert needs[4].kind == "paged_kv" and needs[4].v_head_dim is None
    cache = Cache(needs, max_tokens=256, dtype=torch.bfloat16, device="cpu")
    v = cache.view(1)
    assert v.parts[1].blocks.shape == (5, 2 * 16 * 22)               # 16 blocks of 4 positions end on a page of 64
    assert cache.bytes_per_token() == 2 * (20 + 2 * 22 + 12 + 2 * 16 * 22 / 64)
    assert cache.read_bytes(100, 1) == 2 * 100 * (20 + 44 + 12) + 25 * 2 * 22 * 2 + 4 * (96 + 2 * 92)


@pytest.mark.parametrize("block,rows", [(1, 64), (3, 22), (12, 6), (60, 2), (63, 2), (64, 1), (65, 1), (500, 1)])
def test_the_places_of_blocks_on_pages_are_few_and_never_shared(block, rows):
    """A block lies on the page of its last position, at the number of blocks that end there before it."""
    need = CacheNeed("paged_blocks", kv_heads=1, head_dim=2, block=block)
    cache = Cache([need], max_tokens=64, dtype=torch.float32, device="cpu")
    assert cache.view(0).blocks.shape[1] == rows * 4
    seen = set()
    for b in range(3000 // block):
        page = (b * block + block - 1) // 64
        place = b - page * 64 // block
        assert 0 <= place < rows and (page, place) not in seen
        seen.add((page, place))


def test_random_weights_are_written_and_read_back(tmp_path):
    d = str(tmp_path)
    cfg = wick.config_from_json(CFG)
    wick.write_random_model(cfg, 3, d)
    st = SafeTensorsDir(d)
    w = {n: st.get(n).tensor() for n in st.names()}
    model = Model(wick.get_architecture("Saposun").build_spec(cfg), torch.float32, "cpu")
    wick.load_weights(model, d)
    for n, t in model.tensors().items():
        assert torch.equal(t, w[n].float()), n
    out = P.forward(CFG, w, [1, 2, 3, 50, 96])
    assert out.shape == (5, 97) and torch.isfinite(out).all()


def test_what_the_plain_query_sees():
    n, size, pool = 40, 7, 5
    win, blk = P.in_window(n, size), P.sees_block(n, size, pool)
    for i in range(n):
        assert win[i].nonzero()[:, 0].tolist() == list(range(max(0, i - 6), i + 1))
        assert blk[i].nonzero()[:, 0].tolist() == [b for b in range(8) if all(not win[i, j] and j < i for j in range(5 * b, 5 * b + 5))]
    # the newest block that is seen ends right before the window, one position later the next begins to wait
    assert blk[16].nonzero()[:, 0].tolist() == [0, 1] and blk[15].nonzero()[:, 0].tolist() == [0]


def test_the_plain_filter_and_decay():
    u = torch.arange(1.0, 7.0)[:, None]
    assert P.causal_filter(u, torch.tensor([[100.0, 10.0, 1.0]]))[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0, 456.0]
    one = torch.ones(4, 2, 1)
    o, S = P.decaying_outer_products(one, one, one, torch.tensor([0.5, 1.0]))
    assert o[:, 0, 0].tolist() == [1.0, 1.5, 1.75, 1.875] and o[:, 1, 0].tolist() == [1.0, 2.0, 3.0, 4.0] and S[0, 0, 0] == 1.875
    x = torch.randn(5, 2, 6)
    for halves in (True, False):                            # only the first four elements turn; position 0 stays
        y = P.turn(x, 10.0, 4, halves)
        assert torch.equal(y[:, :, 4:], x[:, :, 4:]) and torch.equal(y[0], x[0])
        assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1)) and not torch.allclose(y[3, :, :4], x[3, :, :4])
    assert not torch.allclose(P.turn(x, 10.0, 6, True), P.turn(x, 10.0, 6, False))
