"""Host-side parts of the Poresun design: config.json parsing and validation, the registry, tensor names and shapes, the
weight layout the library reads, the distance tables, the page manager's rule for pages that several layers read, and the oracle's own
mechanisms on hand-made inputs. No GPU."""
import json
import math

import pytest
import torch

import poresun_cases as K
import poresun_oracle as O
from livecc_b200 import registry
from livecc_b200.checkpoint import seq_param_specs, synthetic_seq_tensors
from livecc_b200.config import SeqModelConfig
from livecc_b200.kv_cache import PAGE_SIZE, SeqCache, SeqStatePool

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(K.CASES))
def test_config_round_trip_and_validation(name):
    d = K.CASES[name]
    cfg = SeqModelConfig.from_json(json.loads(json.dumps(d)))
    cfg.validate()
    assert SeqModelConfig.from_json(cfg.to_json()) == cfg
    assert [L["type"] for L in cfg.to_json()["layers"]] == [L["type"] for L in d["layers"]]
    assert cfg.block == "postnorm" and cfg.norm == "rms" and cfg.dense == "clamp_glu" and cfg.tied_head and cfg.layer_scale
    assert cfg.positions is None and cfg.eps == d["norm"]["eps"] and cfg.alpha == d["postln_alpha"] and cfg.embed_scale == d["embedding"]["scale"]
    for L, e in zip(cfg.layers, d["layers"]):
        mx = e["mixer"]
        if e["type"] == "latent_attention":
            a = L.latent
            assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank) == tuple(mx[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            assert a.gate and a.gate_channel and a.rot_pairs and not a.sink and not a.window and a.rot.base == mx["rot"]["base"] and a.gate_rows == a.heads * a.vdim
        else:
            a, two = L.attn, e["type"] == "attention_2"
            assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale) == tuple(mx[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
            assert (a.window, a.softcap, a.rel_max, a.kv_from) == (mx.get("mask", {}).get("size", 0), mx.get("softcap", 0.0), mx["bias_max"], mx.get("kv_from", -1))
            assert (a.temp_coef, a.temp_every) == ((mx["q_temp"]["coef"], mx["q_temp"]["every"]) if "q_temp" in mx else (0.0, 0))
            assert a.qk_norm and a.unit_norm != two and a.rot.dims == 0 and a.gate == "none" and not a.sink and not a.value_keys and not a.bias and a.maps == 1
        mlp = e["mlp"]
        if mlp and mlp["kind"] == "moe":
            r = mlp["router"]
            assert (L.moe.experts, L.moe.top, L.moe.ff, L.moe.shared_ff) == (r["experts"], r["top"], mlp["expert"]["ff"], mlp.get("shared", {"ff": 0})["ff"])
            assert L.moe.router == "topk_softmax" and L.moe.act == "relu2" and L.moe.router_bias and L.moe.shared_gate and not L.moe.groups and L.moe.scale == 1.0
        elif mlp:
            assert (L.ff, L.ff_limit) == (mlp["ff"], mlp["limit"])
        else:
            assert not L.ff and L.moe is None


def test_random_configurations_are_valid():
    for seed in range(60):
        cfg = SeqModelConfig.from_json(K.random_config(seed))
        cfg.validate()
        assert SeqModelConfig.from_json(cfg.to_json()) == cfg


def test_bad_configurations_are_refused():
    def bad(change, case="mixed"):
        d = json.loads(json.dumps(K.CASES[case]))
        change(d)
        with pytest.raises((ValueError, NotImplementedError, KeyError)):
            SeqModelConfig.from_json(d).validate()

    bad(lambda d: d["layers"][1]["mixer"].update(kv_heads=2))                                  # 3 query heads over 2 key/value heads
    bad(lambda d: d["layers"][1]["mixer"].update(softcap=-2.0))
    bad(lambda d: d["layers"][1]["mixer"].update(bias_max=-4))
    bad(lambda d: d["layers"][0]["mixer"]["q_temp"].update(every=-1))
    bad(lambda d: d["layers"][0]["mixer"].update(kv_from=3))                                   # a later layer
    bad(lambda d: d["layers"][3]["mixer"].update(kv_from=3))                                   # itself
    bad(lambda d: d["layers"][3]["mixer"].update(kv_from=2))                                   # a latent layer
    bad(lambda d: d["layers"][3]["mixer"].update(kv_from=1))                                   # another geometry
    bad(lambda d: (d["layers"].append(K.att2(kv_from=3))))                                     # a layer without a cache of its own
    bad(lambda d: d["layers"][2]["mixer"]["rot"].update(dims=2))
    bad(lambda d: d["layers"][1]["mlp"]["router"].update(top=9))                               # 6 experts
    bad(lambda d: d["layers"][0]["mlp"].pop("limit"))
    bad(lambda d: d["layers"][0].update(type="attention_3"))
    bad(lambda d: d.update(architecture="Lugizen"))                                            # that design has no second attention mixer


def test_registry_and_tensor_names():
    assert "Poresun" in registry.architectures()
    cfg = SeqModelConfig.from_json(K.CASES["mixed"])
    names = {n: s for n, s, _ in seq_param_specs(cfg)}
    assert all(names[f"l0.{n}"] == (32,) for n in ("norm1", "norm2", "ls1", "ls2")) and names["final.norm"] == (32,) and "head" not in names
    assert names["l0.mix.q"] == (24, 32) and names["l0.mix.k"] == (12, 32) and names["l0.mix.v"] == (20, 32) and names["l0.mix.o"] == (32, 40)
    assert names["l0.mix.q.norm"] == (6,) and names["l0.mix.k.norm"] == (6,) and names["l0.mix.rel"] == (10, 4)
    assert names["l0.mlp.gate"] == (20, 32) and names["l0.mlp.up"] == (20, 32) and names["l0.mlp.down"] == (32, 20)
    assert names["l1.mix.q"] == (24, 32) and names["l1.mix.rel"] == (12, 3) and "l1.mix.q.norm" not in names and "l1.mix.g" not in names
    assert names["l1.mlp.router"] == (6, 32) and names["l1.mlp.router.b"] == (6,) and names["l1.mlp.e5.up"] == (12, 32) and "l1.mlp.e5.gate" not in names
    assert names["l1.mlp.shared.up"] == (10, 32) and names["l1.mlp.shared.sg"] == (1, 32) and "l1.mlp.correction" not in names
    assert names["l2.mix.dq"] == (9, 32) and names["l2.mix.uq"] == (30, 9) and names["l2.mix.dkv"] == (18, 32) and names["l2.mix.dkv.norm"] == (14,)
    assert names["l2.mix.uk"] == (18, 14) and names["l2.mix.uv"] == (15, 14) and names["l2.mix.g"] == (15, 32) and "l2.mix.sink" not in names
    # a layer that reads another layer's keys and values owns neither their projections nor their norm
    assert names["l3.mix.q.norm"] == (6,) and names["l3.mix.rel"] == (10, 4) and not {"l3.mix.k", "l3.mix.v", "l3.mix.k.norm"} & set(names)
    assert "l4.norm2" not in names and "l4.ls2" not in names and names["l4.ls1"] == (32,)
    t = synthetic_seq_tensors(cfg, seed=1)
    assert set(t) == set(names) and all(tuple(t[n].shape) == s for n, s in names.items())


def test_weight_layout_the_library_reads():
    from livecc_b200.seq_engine import SeqWeights

    d = K.config([K.att2(heads=3, kv_heads=1, dim=5, vdim=7, rows=6, far=12, mlp=K.dense(16, 0.5)), K.lat(heads=3, vdim=5, rank=10, rot=4, q_rank=9, mlp="moe"),
                  K.att2(heads=3, kv_heads=1, dim=5, vdim=7, kv_from=0, mlp=K.dense(12, 0.5))], width=16, vocab=41)
    cfg = SeqModelConfig.from_json(d)
    t = synthetic_seq_tensors(cfg, seed=2)
    w = SeqWeights(cfg, t, torch.float32, "cpu")
    assert not w.unused and w.head is w.embed and w.embed.shape == (48, 16) and not w.embed[41:].any()
    a, b, c = w.layers
    assert a["m_in"].shape == (32, 16) and torch.equal(a["m_in"][20:27], t["l0.mix.v"].float()) and not a["m_in"][27:].any()
    assert c["m_in"].shape == (16, 16) and torch.equal(c["m_in"][:15], t["l2.mix.q"].float()) and "m_knorm" not in c and c["m_qnorm"].shape == (5,)
    # the gate's rows start at a multiple of 8 behind [query latent | latent, key part]
    assert b["a_in"].shape == (40, 16) and torch.equal(b["a_in"][24:39], t["l1.mix.g"].float()) and not b["a_in"][23].any() and not b["a_in"][39].any()
    assert b["e_router"].shape == (8, 16) and torch.equal(b["e_router"][6], t["l1.mlp.shared.sg"].float()[0]) and torch.equal(b["e_router_bias"], t["l1.mlp.router.b"].float())
    # gate and up rows interleaved in groups of 16 where the width allows it, else one block behind the other
    assert a["ff_il16"] == 1 and torch.equal(a["ff_in"][:16], t["l0.mlp.gate"].float()) and torch.equal(a["ff_in"][16:], t["l0.mlp.up"].float())
    assert c["ff_il16"] == 0 and torch.equal(c["ff_in"][:12], t["l2.mlp.gate"].float()) and torch.equal(c["ff_in"][12:24], t["l2.mlp.up"].float())
    assert torch.equal(a["ls1"], t["l0.ls1"].float()) and torch.equal(a["ls2"], t["l0.ls2"].float())


@pytest.mark.parametrize("rows,far", [(2, 2), (2, 300), (4, 3), (8, 128), (16, 128), (16, 200), (32, 128), (32, 1000), (13, 77), (40, 700), (64, 64), (6, 3.5)])
def test_distance_tables(rows, far):
    """The table the kernels read (one entry per distance up to the first that no later distance leaves) is the bucket formula's."""
    from livecc_b200.seq_engine import distance_bias

    rel = torch.arange(rows * 3, dtype=torch.float32).reshape(rows, 3)
    t = distance_bias(rel, 3, far, "rel")
    n_max = int(far) + 40
    want = O.distance_bias(rel, far, n_max)
    got = torch.stack([t[:, min(n, t.shape[1] - 1)] for n in range(n_max + 1)])
    assert torch.equal(got, want)
    assert t.shape[1] <= far + 2 and t[0, -1] == rel[-1, 0] and (t.shape[1] < 2 or t[0, -2] != t[0, -1])
    assert [int(x) for x in t[0] / 3][: rows // 2] == list(range(rows // 2))
    for bad in ((rel[:, :2], far), (rel[:1], 5), (rel, rows // 2)):
        with pytest.raises(ValueError):
            distance_bias(bad[0], 3, bad[1], "rel")


def test_distances_whose_logarithms_meet_an_integer():
    """8 buckets from 8 to 128: powers of two of the ratio 16 ^ (1/8) land on 16, 32, 64 exactly and open a bucket there."""
    assert [O.bucket(n, 16, 128) for n in (7, 8, 15, 16, 31, 32, 63, 64, 127, 128, 10 ** 6)] == [7, 8, 9, 10, 11, 12, 13, 14, 15, 15, 15]
    assert [O.bucket(n, 32, 128) for n in (15, 16, 127, 128)] == [15, 16, 31, 31] and [O.bucket(n, 2, 9) for n in (0, 1, 2, 9)] == [0, 1, 1, 1]


def test_pages_that_several_layers_read_stay_for_the_widest():
    from livecc_b200.seq_engine import shared_mask

    def cfg(*masks):
        layers = [K.att2(window=masks[0], mlp=None)] + [K.att2(kv_from=0, window=m, mlp=None) for m in masks[1:]]
        c = SeqModelConfig.from_json(K.config(layers))
        c.validate()
        return c

    assert shared_mask(cfg(20), 0) == (20, 0) and shared_mask(cfg(20, 90, 30), 0) == (90, 0)
    assert shared_mask(cfg(20, 0), 0) == (0, 0) and shared_mask(cfg(0, 20), 0) == (0, 0)
    pool = SeqStatePool({0: (2, 6, 10, 0) + shared_mask(cfg(20, 90), 0)}, [0, 0], torch.float32, "cpu", initial_pages=8)
    c = SeqCache(pool)
    c.ensure_tokens(300)
    c.advance(300)
    assert pool.keep_from(300) == 211 and [p is None for p in c.pages] == [True] * (211 // PAGE_SIZE) + [False] * (5 - 211 // PAGE_SIZE)
    c.release()
    assert len(pool.free) == pool.num_pages


# ---- the oracle's mechanisms on hand-made inputs ----------------------------------------------------------------------------
def test_oracle_bias_lies_behind_the_cap_and_inside_the_window():
    q = torch.zeros(6, 1, 2, dtype=F64)
    v = torch.arange(6, dtype=F64).reshape(6, 1, 1)
    bias = torch.tensor([0.0, math.log(3.0), 50.0, 0.0, 0.0, 0.0, 0.0], dtype=F64).reshape(7, 1)
    o = O.softmax_attention(q, q, v, 1.0, cap=1.0, size=2, bias=bias)
    assert abs(float(o[5]) - (5 + 3 * 4) / 4) < 1e-12                     # the 50 at distance 2 is outside the window, ln 3 is not capped
    assert abs(float(O.softmax_attention(q, q, v, 1.0, size=0, bias=bias)[5]) - 3.0) < 1e-12
    assert list(O.visible(7, 3)) == [5, 6, 7] and list(O.visible(2, 0)) == [0, 1, 2] and list(O.visible(1, 5)) == [0, 1]


def test_oracle_query_temperature_steps():
    qt = {"coef": 0.5, "every": 4}
    assert [O.query_temperature(p, qt) for p in (0, 2)] == [1.0, 1.0]
    assert abs(O.query_temperature(3, qt) - (1 + 0.5 * math.log(2))) < 1e-12 and O.query_temperature(6, qt) == O.query_temperature(3, qt)
    assert abs(O.query_temperature(7, qt) - (1 + 0.5 * math.log(3))) < 1e-12


def test_oracle_rotation_pairs_neighbours():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0]]] * 3, dtype=F64)
    r = O.rotate_pairs(x, 100.0)
    assert torch.equal(r[0], x[0])
    want = torch.tensor([math.cos(2), math.sin(2), -2 * math.sin(0.2), 2 * math.cos(0.2)], dtype=F64)
    assert torch.allclose(r[2, 0], want)


def test_oracle_clamped_glu_route_and_expert():
    g, u = torch.tensor([3.0, -3.0, 0.5], dtype=F64), torch.tensor([9.0, -9.0, 0.25], dtype=F64)
    s = lambda z: z / (1 + math.exp(-1.702 * z))
    want = torch.tensor([s(2.0) * 3.0, s(-3.0) * -1.0, s(0.5) * 1.25], dtype=F64)
    assert torch.allclose(O.clamped_glu(g, u, 2.0), want)
    idx, w = O.route(torch.tensor([0.1, 2.0, -1.0, 2.0, 1.0], dtype=F64), 3)
    assert idx == [1, 3, 4] and torch.allclose(w, torch.softmax(torch.tensor([2.0, 2.0, 1.0], dtype=F64), 0))
    t = {"up": torch.tensor([[1.0], [-1.0]], dtype=F64), "down": torch.tensor([[1.0, 10.0]], dtype=F64)}
    assert O.expert(torch.tensor([[3.0], [-2.0]], dtype=F64), t, "").flatten().tolist() == [9.0, 40.0]


def test_oracle_norm_behind_the_sum():
    """One layer whose mixer's factor is zero: the stream is the embedding's scaled row, normed; alpha cancels but for eps."""
    d = K.config([K.att(mlp=None)], alpha=2.0, scale=3.0)
    t = synthetic_seq_tensors(SeqModelConfig.from_json(d), seed=3)
    t["l0.ls1"].zero_()
    _, x = O.forward(d, t, [4, 5], layer_outputs=True)
    e = t["embed"][[4, 5]].double() * 6.0
    assert torch.allclose(x[0], e / torch.sqrt(e.pow(2).mean(-1, keepdim=True) + 1e-5) * t["l0.norm1"].double())
