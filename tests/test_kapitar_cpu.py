"""Host-side parts of the Kapitar design: config.json parsing and validation, the registry, tensor names and shapes, the
weight layout the library reads, the page manager's rule for windows that keep the first tokens, and the oracle's own
mechanisms on hand-made inputs. No GPU."""
import json
import math

import pytest
import torch

import kapitar_cases as K
import kapitar_oracle as O
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
    assert cfg.block == "sandwich" and cfg.norm == "layer" and cfg.dense == "mlp" and cfg.dense_act == "relu2" and cfg.tied_head
    assert cfg.positions is None and cfg.eps == d["norm"]["eps"]
    for L, e in zip(cfg.layers, d["layers"]):
        mx = e["mixer"]
        if e["type"] == "attention":
            a, mask = L.attn, mx.get("mask", {})
            assert (a.heads, a.kv_heads, a.dim, a.vdim, a.maps) == tuple(mx[k] for k in ("heads", "kv_heads", "dim", "vdim")) + (2,)
            assert (a.window, a.keep_first, a.softcap, a.diff) == (mask.get("size", 0), mask.get("keep_first", 0), mx.get("softcap", 0.0), mx["diff"])
            assert a.bias and not a.qk_norm and not a.unit_norm and a.gate == "none" and not a.sink and a.rot.dims == 0 and not a.value_keys
        else:
            t = L.retention
            assert (t.heads, t.dim, t.vdim, t.decay) == (mx["heads"], mx["dim"], mx["vdim"], mx["decay"])
            assert t.silu and not t.key_scale and t.whole_norm and t.gate == "sigmoid" and t.rot.dims == 0
        if e["mlp"] and e["mlp"]["kind"] == "moe":
            r, g = e["mlp"]["router"], e["mlp"]["router"].get("groups", {"count": 0, "keep": 0})
            assert (L.moe.experts, L.moe.top, L.moe.ff, L.moe.groups, L.moe.keep) == (r["experts"], r["top"], e["mlp"]["expert"]["ff"], g["count"], g["keep"])
            assert L.moe.router == "sigmoid" and L.moe.act == "gelu" and L.moe.group_top == 2 and not L.moe.correction and not L.moe.shared_gate
            assert L.moe.scale == 1.0 and L.moe.shared_ff == e["mlp"].get("shared", {"ff": 0})["ff"]


def test_random_configurations_are_valid():
    for seed in range(40):
        cfg = SeqModelConfig.from_json(K.random_config(seed))
        cfg.validate()
        assert SeqModelConfig.from_json(cfg.to_json()) == cfg


def test_bad_configurations_are_refused():
    def bad(change, case="mixed"):
        d = json.loads(json.dumps(K.CASES[case]))
        change(d)
        with pytest.raises((ValueError, NotImplementedError, KeyError)):
            SeqModelConfig.from_json(d).validate()

    bad(lambda d: d["layers"][0]["mixer"].update(kv_heads=2))                                  # 3 query heads over 2 key/value heads
    bad(lambda d: d["layers"][0]["mixer"]["mask"].update(keep_first=-1))
    bad(lambda d: d["layers"][0]["mixer"].update(softcap=-2.0))
    bad(lambda d: d["layers"][1]["mixer"].update(decay=[0.5]))                                 # two heads
    bad(lambda d: d["layers"][1]["mixer"].update(decay=[0.5, 1.5]))
    bad(lambda d: d["layers"][1]["mlp"]["router"].update(top=9))                               # 6 experts
    bad(lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=4))                   # 6 experts in 4 groups
    bad(lambda d: d["layers"][1]["mlp"]["router"].update(top=5))                               # two kept groups hold 4
    bad(lambda d: d["layers"][0].update(type="retention"))                                     # (no rotation, no such mixer's keys)
    bad(lambda d: d.update(architecture="Lugizen"))                                            # that design has no lightning mixer


def test_registry_and_tensor_names():
    assert "Kapitar" in registry.architectures()
    cfg = SeqModelConfig.from_json(K.CASES["mixed"])
    names = {n: s for n, s, _ in seq_param_specs(cfg)}
    assert all(names[f"l0.{n}"] == (32,) for n in ("norm1", "norm1b", "norm2", "norm2b")) and names["final.norm"] == (32,) and "head" not in names
    assert names["l0.mix.q"] == (48, 32) and names["l0.mix.k"] == (16, 32) and names["l0.mix.v"] == (6, 32) and names["l0.mix.o"] == (32, 18)
    assert names["l0.mix.q.b"] == (48,) and names["l0.mix.k.b"] == (16,) and names["l0.mix.v.b"] == (6,) and "l0.mix.q.norm" not in names
    assert all(names[f"l0.mix.{n}"] == (8,) for n in ("lq1", "lk1", "lq2", "lk2"))
    assert names["l0.mlp.up"] == (20, 32) and names["l0.mlp.down"] == (32, 20) and "l0.mlp.gate" not in names
    assert names["l1.mix.q"] == (12, 32) and names["l1.mix.k"] == (12, 32) and names["l1.mix.v"] == (20, 32) and names["l1.mix.g"] == (20, 32)
    assert names["l1.mix.norm"] == (20,) and names["l1.mix.o"] == (32, 20) and "l1.mix.q.b" not in names
    assert names["l1.mlp.router"] == (6, 32) and names["l1.mlp.e5.up"] == (12, 32) and names["l1.mlp.e5.down"] == (32, 12)
    assert names["l1.mlp.shared.up"] == (10, 32) and "l1.mlp.shared.sg" not in names and "l1.mlp.correction" not in names and "l1.mlp.e0.gate" not in names
    assert names["l3.norm1b"] == (32,) and "l3.norm2" not in names and "l3.norm2b" not in names
    t = synthetic_seq_tensors(cfg, seed=1)
    assert set(t) == set(names) and all(tuple(t[n].shape) == s for n, s in names.items())


def test_weight_layout_the_library_reads():
    """Biases lie behind each other as the rows of the fused projection do (zeros on its padding rows), the weight of the second
    map is one number, the router has no gate row, and the head is the embedding table itself."""
    from livecc_b200.seq_engine import SeqWeights

    d = K.config([K.att(heads=3, kv_heads=1, dim=5, vdim=7, diff=0.25, mlp="moe"), K.light(mlp=None)], width=16, vocab=41)
    cfg = SeqModelConfig.from_json(d)
    t = synthetic_seq_tensors(cfg, seed=2)
    w = SeqWeights(cfg, t, torch.float32, "cpu")
    assert not w.unused and w.head is w.embed and w.embed.shape == (48, 16) and not w.embed[41:].any()
    a = w.layers[0]
    assert a["m_in"].shape == (48, 16) and torch.equal(a["m_in"][:30], t["l0.mix.q"].float()) and torch.equal(a["m_in"][40:47], t["l0.mix.v"].float())
    assert torch.equal(a["m_in_bias"][30:40], t["l0.mix.k.b"].float()) and torch.equal(a["m_in_bias"][40:47], t["l0.mix.v.b"].float()) and a["m_in_bias"][47] == 0
    assert abs(a["m_lambda"] - float(O.diff_lambda({k: v.double() for k, v in t.items()}, "l0.mix.", 0.25))) < 1e-12
    assert a["e_router"].shape == (8, 16) and not a["e_router"][6:].any() and "e_correction" not in a and a["e_up"].shape == (6, 12, 16)
    assert a["norm1b"].shape == (16,) and a["norm2b"].shape == (16,) and w.layers[1]["t_norm"].shape == (20,)
    assert w.nbytes() < sum(v.numel() * 4 for v in t.values()) + 4 * 16 * 64


def test_pages_between_the_kept_tokens_and_the_window_are_given_back():
    pool = SeqStatePool({0: (1, 16, 8, 0, 70, 5), 2: (1, 6, 4, 0, 20, 65)}, [0, 8, 0], torch.float32, "cpu", initial_pages=8)
    assert pool.keep_from(300) == 231 and pool.kept_first() == 65
    c = SeqCache(pool)
    c.ensure_tokens(300)
    first = list(c.pages)
    c.advance(300)
    # positions 0 .. 64 (pages 0 and 1) stay for good, the window starts in page 3: page 2 goes back
    assert c.pages == [first[0], first[1], None, first[3], first[4]] and 231 // PAGE_SIZE == 3 and first[2] in pool.free
    c.ensure_tokens(330)
    assert c.pages[5] == first[2] or c.pages[5] not in first      # (a freed page may come back as a later one)
    c.advance(130)
    assert c.pages[:5] == [first[0], first[1], None, None, None]
    c.release()
    assert len(pool.free) == pool.num_pages and len(set(pool.free)) == pool.num_pages
    no_window = SeqStatePool({0: (1, 16, 8, 0, 70, 5), 1: (2, 8, 4, 0, 0, 0)}, [0, 0], torch.float32, "cpu")
    assert no_window.keep_from(300) == 0
    # a window without kept tokens behaves as before, and kept tokens beyond what is cached change nothing
    assert SeqStatePool({0: (1, 4, 4, 0, 9)}, [0], torch.float32, "cpu").kept_first() == 0
    c = SeqCache(SeqStatePool({0: (1, 4, 4, 0, 9, 500)}, [0], torch.float32, "cpu", initial_pages=8))
    c.ensure_tokens(300)
    c.advance(300)
    assert c.live_pages() == 5
    c.release()


# ---- the oracle's mechanisms on hand-made inputs ----------------------------------------------------------------------------
def test_oracle_layer_norm_takes_the_mean_off():
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=F64)
    w = torch.tensor([1.0, 1.0, 2.0, 1.0], dtype=F64)
    sd = math.sqrt((4.0 + 1.0 + 0.0 + 9.0) / 4)
    assert torch.allclose(O.layer_norm(x, w, 0.0), torch.tensor([[-2.0, -1.0, 0.0, 3.0]], dtype=F64) / sd)
    assert torch.allclose(O.layer_norm(x + 100.0, w, 1e-5), O.layer_norm(x, w, 1e-5))


def test_oracle_window_keeps_the_first_positions():
    assert O.visible(7, 3, 2) == [0, 1, 5, 6, 7] and O.visible(3, 3, 2) == [0, 1, 2, 3] and O.visible(7, 3, 0) == [5, 6, 7]
    assert O.visible(2, 0, 0) == [0, 1, 2] and O.visible(7, 1, 1) == [0, 7] and O.visible(4, 2, 50) == [0, 1, 2, 3, 4]
    q = torch.zeros(8, 1, 2, dtype=F64)
    v = torch.arange(8, dtype=F64).reshape(8, 1, 1)
    assert abs(float(O.softmax_map(q, q, v, 1.0, 0.0, 3, 2)[7]) - (0 + 1 + 5 + 6 + 7) / 5) < 1e-12


def test_oracle_soft_cap_bounds_scores():
    s = torch.tensor([0.1, 5.0, -500.0], dtype=F64)
    c = O.soft_cap(s, 2.0)
    assert abs(float(c[0]) - 2 * math.tanh(0.05)) < 1e-12 and float(c[2]) == -2.0 and torch.equal(O.soft_cap(s, 0.0), s)


def test_oracle_difference_of_maps():
    a1, a2 = torch.tensor([3.0, 5.0], dtype=F64), torch.tensor([1.0, -1.0], dtype=F64)
    o = O.diff_combine(a1, a2, 0.5, 0.2, 0.0)
    d = torch.tensor([2.5, 5.5], dtype=F64)
    assert torch.allclose(o, d / math.sqrt((2.5 ** 2 + 5.5 ** 2) / 2) * 0.8)
    t = {"lq1": torch.tensor([1.0, 2.0], dtype=F64), "lk1": torch.tensor([0.5, 0.25], dtype=F64), "lq2": torch.zeros(2, dtype=F64), "lk2": torch.ones(2, dtype=F64)}
    assert abs(float(O.diff_lambda(t, "", 0.3)) - (math.e - 1.0 + 0.3)) < 1e-12


def test_oracle_decayed_sum_reads_its_own_write():
    k = torch.tensor([[1.0, 0.0], [0.0, 2.0], [1.0, 0.0]], dtype=F64)
    q = torch.tensor([[1.0, 1.0], [1.0, 1.0], [1.0, 0.0]], dtype=F64)
    v = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    assert O.decayed_sum(q, k, v, 0.5)[:, 0].tolist() == [1.0, 0.5 + 20.0, 0.25 + 100.0]


def test_oracle_groups_score_as_the_sum_of_their_two_best():
    """Group 0 holds the single best expert, groups 1 and 2 the better pairs: with one score per group the choice is another."""
    s = torch.tensor([0.9, 0.1, 0.1, 0.6, 0.55, 0.1, 0.7, 0.5, 0.0], dtype=F64)
    r = {"top": 3, "groups": {"count": 3, "keep": 2}}
    idx, w = O.route_scores(s, r)
    assert idx == [6, 3, 4] and torch.allclose(w, torch.tensor([0.7, 0.6, 0.55], dtype=F64))      # weights: the scores themselves
    assert O.route_scores(s, r, group_top=1)[0] == [0, 6, 7]
    assert O.route_scores(s, {"top": 2})[0] == [0, 6]
    assert O.route_scores(s[:3], {"top": 2, "groups": {"count": 3, "keep": 2}})[0] == [0, 1]        # groups of one expert
    assert torch.allclose(O.gelu_erf(torch.tensor([1.0], dtype=F64)), torch.tensor([0.8413447460685429], dtype=F64))
    assert O.relu2(torch.tensor([-2.0, 3.0], dtype=F64)).tolist() == [0.0, 9.0]
