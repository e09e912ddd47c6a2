"""Poresun on the GPU against the float64 oracle (tests/poresun_oracle.py): every mechanism alone and together, whole prompts
against token-by-token decoding, portions down to two tokens, batches against each request alone, pages and slots that are used
again, keys far away, at page borders and just inside / just outside the window with a sharp softmax, in a layer's own cache and in one
it shares, every bucket of the distance tables, long decoding, unusual sizes, and greedy generation through the engine's own entry
point. fp32 storage is compared tightly; bf16 storage within bf16 rounding."""
import json
import os
import subprocess

import pytest
import torch

import poresun_cases as K
import poresun_oracle as O
from livecc_b200.checkpoint import synthetic_seq_tensors, write_safetensors
from livecc_b200.config import SeqModelConfig

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 2e-5
BF16_TOL = 4e-2

_models = {}


def build(d, tensors, dtype="float32", **kw):
    from livecc_b200.seq_engine import SeqLMForCausalLM

    return SeqLMForCausalLM.from_state_dict(SeqModelConfig.from_json(d), tensors, dtype, **kw)


def make(d, seed=21):
    return synthetic_seq_tensors(SeqModelConfig.from_json(d), seed=seed)


def model_of(name, dtype="float32", seed=21):
    key = (name, dtype, seed)
    if key not in _models:
        d = K.CASES[name]
        tensors = make(d, seed)
        _models[key] = (build(d, tensors, dtype), d, tensors)
    return _models[key]


_oracle = {}


def oracle(name, toks, seed=21, **kw):
    """(logits, residual stream after every layer)"""
    key = (name, tuple(toks), seed, tuple(sorted(kw.items())))
    if key not in _oracle:
        _, d, tensors = model_of(name, "float32", seed)
        _oracle[key] = O.forward(d, tensors, toks, layer_outputs=True, **kw)
    return _oracle[key]


def rows_rel(got, want):
    got, want = got.double().cpu(), want.double()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-30)


def rel(got, want):
    """Largest row error: rms(got - want) / rms(want) over the last axis."""
    return float(rows_rel(got, want).max())


def bf16_ok(got, want, routed=False):
    """bf16 storage: the bulk of the rows stays within bf16 rounding and few rows lie beyond twice that. routed: a stack with
    routers, where a logit close to the next one can fall the other way under rounding and hand the stream another expert's row,
    which attention carries to later positions: held to rounding in the median only."""
    e = rows_rel(got, want)
    if not bool(torch.isfinite(e).all()):
        return False
    if routed:
        return float(e.median()) < BF16_TOL
    return float(e.median()) < BF16_TOL / 2 and float((e > BF16_TOL).double().mean()) <= 0.1


def run(m, toks, cuts):
    """One request through forward_step in portions ending at `cuts`; returns the logits of every position."""
    c = m.new_cache()
    rows, lo = [], 0
    for hi in list(cuts) + [len(toks)]:
        if hi <= lo:
            continue
        rows.append(m.forward_step([(c, toks[lo:hi])], [list(range(hi - lo))]).cpu())
        lo = hi
    c.release()
    return torch.cat(rows)


ALL = ["attention_only", "attention2_only", "latent_only", "dense", "moe", "mixed", "odd"]


def routed(d):
    return any(L["mlp"] and L["mlp"]["kind"] == "moe" for L in d["layers"])


# ---- every mechanism alone, and together, against the oracle ------------------------------------------------------------
@pytest.mark.parametrize("name", ALL)
def test_whole_prompt_every_layer_matches_the_oracle_fp32(name):
    m, d, _ = model_of(name)
    toks = K.tokens(150, d["vocab"])
    want_lg, want_layers = oracle(name, toks)
    c = m.new_cache()
    lg, dump = m.forward_step([(c, toks)], [list(range(len(toks)))], layer_dump=True)
    c.release()
    for li in range(len(d["layers"])):
        assert rel(dump[li], want_layers[li]) < F32_TOL, f"residual stream after layer {li}"
    assert rel(lg, want_lg) < F32_TOL


@pytest.mark.parametrize("name", ALL)
def test_bf16_storage_stays_within_rounding_on_both_linear_paths(name, monkeypatch):
    _, d, tensors = model_of(name)
    toks = K.tokens(160, d["vocab"], seed=3)
    want_lg, _ = oracle(name, toks)
    for tc in ("1", "0"):                       # tensor-core kernels where the shape allows them / CUDA-core kernels only
        monkeypatch.setenv("LIVECC_B200_SEQ_TC", tc)
        m = build(d, tensors, "bfloat16")
        assert bf16_ok(run(m, toks, []), want_lg, routed(d))
        assert bf16_ok(run(m, toks, [120] + list(range(121, 160))), want_lg, routed(d))


@pytest.mark.parametrize("name,what", [("attention_only", "bias"), ("attention_only", "softcap"), ("attention_only", "window"), ("attention2_only", "bias"),
                                       ("attention2_only", "q_temp"), ("latent_only", "rotation"), ("latent_only", "gate"), ("moe", "router_bias"),
                                       ("moe", "shared"), ("moe", "shared_gate"), ("dense", "layer_scale"), ("dense", "alpha")])
def test_each_mechanism_shows_in_these_weights(name, what):
    """An oracle that drops one mechanism is far outside the tolerance: the other tests would notice a product that left it out."""
    m, d, _ = model_of(name)
    toks = K.tokens(90, d["vocab"])
    got = run(m, toks, [])
    assert rel(got, oracle(name, toks)[0]) < F32_TOL
    assert rel(got, oracle(name, toks, leave_out=(what,))[0]) > 100 * F32_TOL


@pytest.mark.parametrize("what", ["limit", "embedding", "kv_from", "base", "bias_max", "eps"])
def test_each_constant_of_the_configuration_shows(what):
    """The product follows the constants it is given: another value moves the oracle far beyond the tolerance."""
    m, d, tensors = model_of("dense")
    toks = K.tokens(90, d["vocab"])
    other = json.loads(json.dumps(d))
    if what == "limit":
        other["layers"][1]["mlp"]["limit"] *= 1.5
    elif what == "embedding":
        other["embedding"]["scale"] *= 0.5
        other["norm"]["eps"] = 0.3              # (the first norm takes a factor off again but for eps and the sublayer beside it)
    elif what == "kv_from":
        other["layers"][3]["mixer"]["kv_from"] = None
        tensors = dict(tensors)
        for n in ("k", "v", "k.norm"):
            tensors["l3.mix." + n] = tensors["l1.mix." + n]
    elif what == "base":
        other["layers"][2]["mixer"]["rot"]["base"] = 90.0
    elif what == "bias_max":
        other["layers"][1]["mixer"]["bias_max"] = 30
    else:
        other["norm"]["eps"] = 0.02
    want = O.forward(other, tensors, toks)
    assert rel(O.forward(d, tensors, toks), want) > 100 * F32_TOL
    assert rel(run(build(other, tensors), toks, [60, 62]), want) < F32_TOL


@pytest.mark.parametrize("seed", range(16))
def test_random_configurations_in_three_schedules(seed):
    """Random stacks (tests/poresun_cases.py::random_config): the whole prompt, most of it then token by token, and portions of
    changing size down to two tokens, all against the oracle in fp32; bf16 storage runs every stack and is held to rounding
    where the stack is shallow."""
    import random

    d = K.random_config(seed)
    tensors = make(d, 30 + seed)
    rng = random.Random(seed)
    T = rng.choice([70, 150, 260])
    toks = K.tokens(T, d["vocab"], seed=60 + seed)
    want = O.forward(d, tensors, toks)
    portions, p = [], 0
    while p < T - 20:
        p += rng.choice([2, 3, 5, 16, 37, 64])
        portions.append(min(p, T - 20))
    m = build(d, tensors)
    for cuts in ([], [T - 20] + list(range(T - 19, T)), portions + list(range(T - 19, T))):
        assert rel(run(m, toks, cuts), want) < F32_TOL
    got = run(build(d, tensors, "bfloat16"), toks, portions)
    assert bool(torch.isfinite(got).all())
    if len(d["layers"]) <= 3:
        assert bf16_ok(got, want, routed(d))


# ---- prefill against decoding, portions, first tokens ---------------------------------------------------------------------
@pytest.mark.parametrize("name", ALL)
def test_token_by_token_decoding_equals_the_whole_prompt(name):
    m, d, _ = model_of(name)
    toks = K.tokens(100, d["vocab"], seed=1)
    want_lg, _ = oracle(name, toks)
    assert rel(run(m, toks, range(1, 100)), want_lg) < F32_TOL          # every token alone, from the first one
    assert rel(run(m, toks, [41] + list(range(42, 100))), want_lg) < F32_TOL


@pytest.mark.parametrize("cuts", [[2, 4, 6, 9, 11, 40, 42], [1, 3, 64, 66], [9, 10, 12, 13, 47, 49, 65], [63, 65, 67, 69], [15, 31, 33, 64, 80, 82]])
def test_portions_of_any_size_down_to_two_tokens(cuts):
    """(cuts at a window's edge, at page borders, where the temperature steps and where the attention changes kernels)"""
    for name in ("mixed", "attention2_only"):
        m, d, _ = model_of(name)
        toks = K.tokens(100, d["vocab"], seed=2)
        assert rel(run(m, toks, cuts), oracle(name, toks)[0]) < F32_TOL


def test_first_tokens_of_a_sequence():
    for name in ("mixed", "odd", "latent_only"):
        m, d, _ = model_of(name)
        for n in (1, 2, 3, 4):
            toks = K.tokens(n, d["vocab"], seed=20 + n)
            assert rel(run(m, toks, []), oracle(name, toks)[0]) < F32_TOL
            assert rel(run(m, toks, range(1, n)), oracle(name, toks)[0]) < F32_TOL


# ---- far keys, page borders, the window's edges -----------------------------------------------------------------------------
A, B, COL_A, COL_B, CH = 5, 9, 3, 11, 2


def _stand_out(tensors, d):
    """Token A (the key) and token B (the query) have embeddings in columns of their own."""
    for col in (COL_A, COL_B):
        tensors["embed"][:, col] = 0.0
    for tok, col in ((A, COL_A), (B, COL_B)):
        tensors["embed"][tok].zero_()
        tensors["embed"][tok, col] = 2.0


def _sharp_head(tensors, p, mx, own_kv=True):
    """One key channel reads A's column only, one query channel of every head B's: B's score against A is about scale * dim, against
    every other key about 0, wherever A sits; A's value row is large, so whether A is seen moves the output by far more than the
    tolerance."""
    for h in range(mx["heads"]):
        tensors[p + "q"][h * mx["dim"] + CH].zero_()
        tensors[p + "q"][h * mx["dim"] + CH, COL_B] = 40.0
    if own_kv:
        tensors[p + "k"][CH].zero_()
        tensors[p + "k"][CH, COL_A] = 40.0
        tensors[p + "v"][:, COL_A] = 6.0


def _key_model(window=100, seed=22):
    """One sliding-window layer with soft-capped scores."""
    d = json.loads(json.dumps(K.CASES["sharp"]))
    mx = d["layers"][0]["mixer"]
    mx.pop("mask")
    if window:
        mx["mask"] = {"size": window}
    tensors = make(d, seed)
    _stand_out(tensors, d)
    _sharp_head(tensors, "l0.mix.", mx)
    return d, tensors


def _shared_key_model(mute=True, seed=23):
    """Two causal layers, the second reading the first one's keys and values. mute: the first layer's output is multiplied by zero, so
    that only the second one's queries can bring A's value to B; else the second one's is."""
    d = json.loads(json.dumps(K.CASES["sharp2"]))
    tensors = make(d, seed)
    _stand_out(tensors, d)
    tensors["l0.norm1"].fill_(1.0)
    tensors["l0.mix.q.norm"].fill_(1.0), tensors["l0.mix.k.norm"].fill_(1.0), tensors["l1.mix.q.norm"].fill_(1.0)
    _sharp_head(tensors, "l0.mix.", d["layers"][0]["mixer"])
    _sharp_head(tensors, "l1.mix.", d["layers"][1]["mixer"], own_kv=False)
    tensors["l0.ls1" if mute else "l1.ls1"].zero_()
    return d, tensors


def _latent_key_model(rotated=False, seed=24):
    """One latent-attention layer: A's latent is one channel alone, every head's first key channel reads it, B's query latent is one
    channel alone, every head's first query channel reads it (so the score does not depend on positions). rotated: the score comes
    from the shared rotated part instead, whose pair (0, 1) is given a frequency of 1: it depends on the distance as cos does."""
    d = json.loads(json.dumps(K.CASES["sharp_latent"]))
    mx = d["layers"][0]["mixer"]
    tensors = make(d, seed)
    p = "l0.mix."
    _stand_out(tensors, d)
    H, D, R, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
    tensors[p + "dkv"][CH].zero_(), tensors[p + "dq"][CH].zero_()
    tensors[p + "dkv"][CH, COL_A] = 40.0
    tensors[p + "dq"][CH, COL_B] = 40.0
    tensors[p + "dkv.norm"].fill_(1.0), tensors[p + "dq.norm"].fill_(1.0)
    if rotated:
        tensors[p + "dkv"][rank:].mul_(0.2)
        tensors[p + "dkv"][rank].zero_()
        tensors[p + "dkv"][rank, COL_A] = 2.0
    for h in range(H):
        if rotated:
            tensors[p + "uq"][h * (D + R) + D, CH] = 4.0
        else:
            tensors[p + "uq"][h * (D + R), CH] = 2.5
            tensors[p + "uk"][h * D, CH] = 2.5
    return d, tensors


def _with_key(d, n, key_at, query_at, seed):
    toks = [t if t not in (A, B) else 17 for t in K.tokens(n, d["vocab"], seed=seed)]
    toks[key_at] = A
    for q in query_at:
        toks[q] = B
    return toks


@pytest.mark.parametrize("kind", ["shared", "own", "latent", "latent_rotated", "window"])
@pytest.mark.parametrize("far_at", [0, 1, 63, 64, 65, 127, 128, 200])
def test_a_far_key_among_hundreds_at_page_borders(far_at, kind):
    """A sits once at `far_at` of 300 tokens (first tokens, just before / on / after a page border, deep inside), B queries it from the
    end: in one prompt, decoded alone, and at the start of a two-token portion; in fp32 and in bf16 on the tensor-core attention."""
    if kind == "window":
        d, tensors = _key_model(300)
    elif kind in ("shared", "own"):
        d, tensors = _shared_key_model(kind == "shared")
    else:
        d, tensors = _latent_key_model(kind == "latent_rotated")
    toks = _with_key(d, 300, far_at, [298, 299], seed=7)
    moved = list(toks)
    moved[far_at] = 17
    want = O.forward(d, tensors, toks)
    gap = rel(O.forward(d, tensors, moved)[-2:], want[-2:])
    assert gap > (50 if kind == "latent_rotated" else 500) * F32_TOL, "the far key does not stand out"
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL
    assert rel(run(m, toks, [250] + list(range(251, 300))), want) < F32_TOL
    assert rel(run(m, toks, [66, 129, 298]), want) < F32_TOL
    m = build(d, tensors, "bfloat16")
    for cuts in ([], [66, 129, 298], [250] + list(range(251, 300))):
        got = run(m, toks, cuts)
        assert bf16_ok(got, want) and rel(got[-2:], want[-2:]) < max(BF16_TOL, gap / 10)


@pytest.mark.parametrize("window", [1, 2, 7, 63, 64, 65, 100, 128, 129, 300])
@pytest.mark.parametrize("inside", [True, False])
def test_keys_just_inside_and_just_outside_the_window(window, inside):
    """The query at position i, the key at i - window + 1 (the last one the window keeps) or at i - window (the first one it drops):
    windows shorter than, equal to and longer than a page and a key tile; in one prompt, with the query decoded alone, at the
    start and at the end of short portions, and through the tiled kernels in bf16."""
    d, tensors = _key_model(window)
    n, i = 420, 401
    key_at = i - window + 1 if inside else i - window
    toks = _with_key(d, n, key_at, [i], seed=11)
    if key_at == i:
        toks[i] = A
    want = O.forward(d, tensors, toks)
    if window > 1:      # (a window of one position holds the query alone)
        gone = list(toks)
        gone[key_at] = 17
        gap = rel(O.forward(d, tensors, gone)[i:i + 1], want[i:i + 1])
        assert gap > 0.05 if inside else gap < 1e-9, "the test's key does not show the window's edge"
        assert inside or rel(O.forward(d, tensors, toks, leave_out=("window",))[i:i + 1], want[i:i + 1]) > 0.05
    m = build(d, tensors)
    for cuts in ([], [i] + list(range(i + 1, n)), [key_at + 1, i, i + 2], [i - 1, i + 1], [200, i - 30]):
        assert rel(run(m, toks, cuts), want) < F32_TOL, cuts
    bf = build(d, tensors, "bfloat16")
    for cuts in ([], [i] + list(range(i + 1, n))):
        got = run(bf, toks, cuts)
        assert bf16_ok(got, want) and rel(got[i:i + 1], want[i:i + 1]) < BF16_TOL


def test_every_position_while_the_window_leaves_the_start():
    for window in (1, 5, 30, 64, 65):
        d, tensors = _key_model(window)
        toks = _with_key(d, 150, 0, [window - 1, window, window + 1, 149], seed=15)
        toks[0] = A
        want = O.forward(d, tensors, toks)
        m = build(d, tensors)
        for cuts in ([], list(range(1, 150)), [2, 4, window, window + 2], list(range(17, 150, 17))):
            assert rel(run(m, toks, cuts), want) < F32_TOL, (window, cuts)


@pytest.mark.parametrize("kind", ["window700", "causal", "shared", "latent"])
def test_long_ranges_in_steps_of_a_few_rows_split_the_keys(kind):
    """Ranges of hundreds of keys in steps of one to three rows: the keys are split over several CTAs and merged by the last to arrive.
    The key at the range's first position, just before it, and at the edges of the splits; then through generation, where only the
    device knows the position."""
    d, tensors = {"window700": lambda: _key_model(700), "causal": lambda: _key_model(0), "shared": _shared_key_model, "latent": _latent_key_model}[kind]()
    n = 1000
    m = build(d, tensors)
    for key_at in (0, n - 1 - 700, n - 700, 383, 384, 998):
        toks = _with_key(d, n, key_at, [n - 1, n - 3], seed=13)
        want = O.forward(d, tensors, toks)
        cuts = [950, 952, 955] + list(range(956, n))
        assert rel(run(m, toks, cuts), want) < F32_TOL, key_at
        if key_at in (383, n - 700):
            assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, cuts), want)
    toks = _with_key(d, n, 300, [959], seed=14)
    new = O.greedy(d, tensors, toks[:960], 3)
    out = m.generate(torch.tensor([toks[:960]]), max_new_tokens=3, output_logits=True)
    assert out.sequences[0, 960:].tolist() == new
    assert rel(torch.stack(out.logits), O.forward(d, tensors, toks[:960] + new)[959:962]) < F32_TOL
    out.past_key_values.release()


# ---- distance tables, temperature, caps -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,far", [(2, 2), (4, 200), (16, 128), (32, 128), (13, 77), (40, 3000), (64, 64), (32, 600)])
@pytest.mark.parametrize("second", [False, True])
def test_every_bucket_of_the_distance_table(rows, far, second):
    """Scores are nearly flat (a small scale) and the table's entries are spread over +-3, so a key that met a neighbouring bucket's bias
    would show; distances inside the table's first half, at every bucket's first position and beyond the last one; prompts and few-row
    steps, tables shorter and longer than a key tile, another bias per head."""
    mk = dict(heads=4, kv_heads=2, dim=8, vdim=16, scale=0.05, rows=rows, far=far, mlp=None)
    d = K.config([K.att2(temp=None, **mk) if second else K.att(window=0, cap=2.0, **mk)], width=32, vocab=64, alpha=0.1)
    tensors = make(d, 31)
    g = torch.Generator().manual_seed(rows)
    tensors["l0.mix.rel"] = (torch.rand((rows, 4), generator=g) * 6 - 3).to(torch.bfloat16)
    toks = K.tokens(330, d["vocab"], seed=41)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    shifted = dict(tensors)
    shifted["l0.mix.rel"] = torch.roll(tensors["l0.mix.rel"], 1, 0)
    assert rel(O.forward(d, shifted, toks), want) > 100 * F32_TOL
    for cuts in ([], [300, 302, 305] + list(range(306, 330)), [63, 65, 128, 193, 195]):
        assert rel(run(m, toks, cuts), want) < F32_TOL
    bf = build(d, tensors, "bfloat16")
    assert bf16_ok(run(bf, toks, []), want) and bf16_ok(run(bf, toks, [250, 300] + list(range(301, 330))), want)


@pytest.mark.parametrize("dist", [0, 1, 5, 6, 63, 64, 65, 100, 127, 128, 129, 191, 255, 256])
def test_one_distance_stands_out(dist):
    """A table with a row per distance whose row `dist` alone is large: every position's output is then nearly the value `dist` tokens
    back, whatever tile, page, split or portion it lies in; a bias read one place off would bring another token's value."""
    d = K.config([K.att2(heads=2, kv_heads=1, dim=8, vdim=8, scale=0.02, temp=None, rows=600, far=400, mlp=None)], width=16, vocab=64, alpha=0.2)
    tensors = make(d, 32)
    t = torch.zeros(600, 2)
    t[dist, 0], t[dist, 1] = 14.0, 11.0
    tensors["l0.mix.rel"] = t.to(torch.bfloat16)
    toks = K.tokens(400, d["vocab"], seed=42)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    for cuts in ([], [dist + 1, dist + 3, 330], [300] + list(range(301, 400))):
        assert rel(run(m, toks, cuts), want) < F32_TOL
    bf = build(d, tensors, "bfloat16")
    for cuts in ([], [300] + list(range(301, 400))):
        assert float((rows_rel(run(bf, toks, cuts), want) > 2 * BF16_TOL).double().mean()) < 0.02


@pytest.mark.parametrize("coef,every", [(0.7, 1), (0.3, 7), (2.0, 64), (0.5, 100), (1.0, 5000), (-0.2, 20)])
def test_the_query_temperature_steps_where_it_should(coef, every):
    d = K.config([K.att2(heads=4, kv_heads=2, dim=8, vdim=8, scale=0.5, temp=(coef, every), mlp=None),
                  K.att2(heads=4, kv_heads=2, dim=8, vdim=8, scale=0.5, temp=(coef / 2, every + 1), kv_from=0, mlp=None)], width=32, vocab=64, alpha=0.3)
    tensors = make(d, 33)
    toks = K.tokens(215, d["vocab"], seed=43)
    want = O.forward(d, tensors, toks)
    off = [json.loads(json.dumps(d)) for _ in range(2)]
    for o, e in zip(off, (every + 1, every + 2)):
        o["layers"][0]["mixer"]["q_temp"]["every"] = e
    if every < 100:
        assert all(rel(O.forward(o, tensors, toks), want) > 100 * F32_TOL for o in off)
    m = build(d, tensors)
    for cuts in ([], list(range(1, 215)), [every - 1, every, every + 2], [98, 100, 102, 199, 201]):
        assert rel(run(m, toks, [c for c in cuts if c < 215]), want) < F32_TOL
    assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, [100] + list(range(190, 215))), want)


@pytest.mark.parametrize("cap,scale", [(0.5, 2.0), (20.0, 0.14), (3.0, 10.0), (0.0, 1.0), (1000.0, 1.0)])
def test_soft_caps_from_saturated_to_open(cap, scale):
    d = K.config([K.att(heads=2, kv_heads=1, dim=16, vdim=8, window=50, cap=cap, scale=scale, mlp=None)], width=32, vocab=64)
    tensors = make(d, 27)
    toks = K.tokens(130, d["vocab"], seed=57)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    tol = F32_TOL * (10 if scale >= 5 else 1)        # large scores: the exponentials amplify the products' rounding
    assert rel(run(m, toks, []), want) < tol
    assert rel(run(m, toks, [100, 103] + list(range(110, 130))), want) < tol
    bf = run(build(d, tensors, "bfloat16"), toks, [])
    assert bool(torch.isfinite(bf).all()) and (scale >= 5 or bf16_ok(bf, want))


# ---- keys and values of another layer ---------------------------------------------------------------------------------------------
def test_layers_that_share_a_cache_keep_the_pages_the_widest_needs():
    """The owner sees 20 positions, one reader 150, another 40 (with query heads of its own number): pages go back only behind the widest
    one; every layer keeps its own window, temperature and bias table."""
    geo = dict(kv_heads=2, dim=6, vdim=10, mlp=None)
    d = K.config([K.att2(heads=4, window=20, **geo), K.att(heads=3, window=9, mlp="dense"), K.att2(heads=4, window=150, kv_from=0, temp=(0.9, 30), rows=24, far=140, **geo),
                  K.att2(heads=2, window=40, kv_from=0, **geo)], width=24, alpha=0.6)
    tensors = make(d, 34)
    toks = K.tokens(420, d["vocab"], seed=44)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    for cuts in ([], [64, 66, 130, 200, 330, 332], [380] + list(range(381, 420))):
        assert rel(run(m, toks, cuts), want) < F32_TOL
    c = m.new_cache()
    m.forward_step([(c, toks[:400])])
    assert [p is None for p in c.pages] == [True, True, True, False, False, False, False]      # position 251 onwards: page 3
    assert sorted(m.pool.k) == [0, 1] and rel(m.forward_step([(c, toks[400:])], [list(range(20))]), want[400:]) < F32_TOL
    c.release()
    without = json.loads(json.dumps(d))
    without["layers"][2]["mixer"]["mask"]["size"] = 100
    assert rel(O.forward(without, tensors, toks)[-20:], want[-20:]) > 100 * F32_TOL


# ---- heads, widths, experts -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dim,vdim,heads,kv", [(136, 40, 2, 1), (72, 136, 4, 2), (128, 128, 2, 1), (128, 256, 2, 2), (300, 24, 1, 1), (64, 300, 2, 1), (20, 129, 3, 3),
                                               (24, 16, 4, 1), (13, 22, 2, 2), (40, 600, 1, 1), (1, 1, 2, 1), (2, 3, 8, 2)])
@pytest.mark.parametrize("second", [False, True])
def test_attention_heads_of_many_sizes(dim, vdim, heads, kv, second):
    """Values up to 128 channels (two groups of warps on alternate key tiles), up to 256 (one group), beyond, beyond what the key-split
    kernel takes, and head sizes that are not multiples of 8 or 16."""
    mk = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=dim ** -0.5, rows=20, far=150, mlp=None)
    d = K.config([K.att2(**mk), K.att2(kv_from=0, **mk)] if second else [K.att(window=90, cap=30.0, **mk)], width=32, vocab=64)
    tensors = make(d, 24)
    toks = K.tokens(215, d["vocab"], seed=52)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL
    assert rel(run(m, toks, [64, 128, 129, 193] + list(range(205, 215))), want) < F32_TOL
    m = build(d, tensors, "bfloat16")
    assert bf16_ok(run(m, toks, []), want)
    assert bf16_ok(run(m, toks, [64, 129, 193] + list(range(194, 215))), want)


@pytest.mark.parametrize("heads,dim,rot,vdim,rank,q_rank", [(4, 32, 16, 32, 64, 40), (2, 64, 32, 48, 128, 96), (3, 5, 2, 7, 9, 11), (1, 128, 64, 128, 192, 64),
                                                            (2, 24, 8, 20, 260, 30), (6, 16, 12, 33, 64, 24), (2, 8, 40, 40, 64, 8)])
def test_latent_attention_of_many_sizes(heads, dim, rot, vdim, rank, q_rank):
    """Gated value up-projections as one batched tensor-core product (latents of 64 k channels, 8-aligned values of 32 channels or more) and
    in the CUDA-core kernels' stores (everything else, and few rows); gate blocks whose first row needs padding."""
    d = K.config([K.lat(heads=heads, dim=dim, rot=rot, vdim=vdim, rank=rank, q_rank=q_rank, scale=(dim + rot) ** -0.5, mlp=None)], width=64, vocab=64)
    tensors = make(d, 25)
    tensors["l0.mix.g"] *= 3.0
    toks = K.tokens(140, d["vocab"], seed=53)
    want = O.forward(d, tensors, toks)
    assert rel(O.forward(d, tensors, toks, leave_out=("gate",)), want) > 100 * F32_TOL
    assert rel(O.forward(d, tensors, toks, leave_out=("rotation",)), want) > 100 * F32_TOL
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL
    assert rel(run(m, toks, [33, 35, 60, 61, 100] + list(range(120, 140))), want) < F32_TOL
    m = build(d, tensors, "bfloat16")
    assert bf16_ok(run(m, toks, []), want)
    assert bf16_ok(run(m, toks, [64, 129] + list(range(130, 140))), want)


@pytest.mark.parametrize("width", [1, 30, 1028, 2050, 5000])
def test_rows_of_many_widths(width):
    """The post-norm kernel's forms: one to sixteen pieces per thread, four columns a piece or one, rows beyond what a thread keeps;
    behind a mixer, a dense and a routed feed-forward."""
    d = K.config([K.att(heads=1, dim=4, vdim=4, mlp=K.dense(16)), K.att2(heads=1, kv_heads=1, dim=4, vdim=4, mlp=K.moe(experts=2, top=1, ff=8, shared=8)),
                  K.lat(heads=1, mlp=K.moe(experts=40, top=35, ff=4, shared=0))], width=width, vocab=30, alpha=0.7)
    tensors = make(d, 35)
    toks = K.tokens(40, d["vocab"], seed=59)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < 2 * F32_TOL
    assert rel(run(m, toks, [30] + list(range(31, 40))), want) < 2 * F32_TOL
    if width > 1:
        assert bool(torch.isfinite(run(build(d, tensors, "bfloat16"), toks, [20])).all())


@pytest.mark.parametrize("ff,limit", [(16, 0.3), (48, 7.0), (64, 0.5), (72, 0.5), (20, 1.0), (1, 0.4)])
def test_clamped_dense_feed_forward(ff, limit, monkeypatch):
    """Interleaved rows (widths of 16 k: the activation in the product's epilogue or store), separate blocks (other widths: a row kernel
    behind the product), few and many rows, clamps that bite and clamps that hardly do."""
    d = K.config([K.att(mlp=K.dense(ff, limit))], width=64, vocab=64, alpha=0.4)
    tensors = make(d, 36)
    tensors["l0.mlp.gate"] *= 2.0
    tensors["l0.mlp.up"] *= 2.0
    toks = K.tokens(90, d["vocab"], seed=45)
    want = O.forward(d, tensors, toks)
    other = json.loads(json.dumps(d))
    other["layers"][0]["mlp"]["limit"] = 1.3 * limit
    assert limit > 5 or rel(O.forward(other, tensors, toks), want) > 50 * F32_TOL
    cuts = [50, 52, 60] + list(range(70, 90))
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL and rel(run(m, toks, cuts), want) < F32_TOL
    for tc in ("1", "0"):
        monkeypatch.setenv("LIVECC_B200_SEQ_TC", tc)
        m = build(d, tensors, "bfloat16")
        assert bf16_ok(run(m, toks, []), want) and bf16_ok(run(m, toks, cuts), want)


def test_router_bias_chooses_and_weighs():
    """Router rows shaped so that every token's logits alone favour the first experts and the bias turns the choice; the weights are the
    softmax over the chosen logits with their bias, and the shared expert's gate has none."""
    d = K.config([K.att(mlp=K.moe(experts=5, top=2, ff=8, shared=6))], width=16, vocab=40, alpha=0.3)
    tensors = make(d, 37)
    tensors["l0.mlp.router"] *= 0.2
    tensors["l0.mlp.router.b"] = torch.tensor([-3.0, -2.0, 1.0, 2.5, 0.5]).to(torch.bfloat16)
    toks = K.tokens(200, d["vocab"], seed=56)
    want = O.forward(d, tensors, toks)
    assert rel(O.forward(d, tensors, toks, leave_out=("router_bias",)), want) > 100 * F32_TOL
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL                                   # few rows and many rows: both router kernels
    assert rel(run(m, toks, [100, 102] + list(range(180, 200))), want) < F32_TOL
    flat = dict(tensors)
    flat["l0.mlp.router"] = torch.zeros_like(tensors["l0.mlp.router"])              # the choice is the bias's alone, for every token
    assert rel(run(build(d, flat), toks, []), O.forward(d, flat, toks)) < F32_TOL


def test_many_rows_per_expert_and_experts_without_rows():
    """300 rows over 33 experts (top 5) and over 2 experts (top 1): lists longer than one tile, lists of a few rows, empty lists; the same
    rows decoded one by one take the few-row kernel."""
    m, d, _ = model_of("odd")
    toks = K.tokens(300, d["vocab"], seed=53)
    want = oracle("odd", toks)[0]
    assert rel(run(m, toks, []), want) < F32_TOL
    assert rel(run(m, toks, [280, 290] + list(range(291, 300))), want) < F32_TOL


def test_the_whole_stack_on_the_tensor_cores(monkeypatch):
    """bf16 storage with enough rows and aligned shapes: projections, latent products, the gated value up-projection, the dense
    feed-forward with its clamp and the padded expert lists all take tensor-core kernels. Against the oracle, against the CUDA-core
    route, and with the prompt cut so that later portions take the few-row route."""
    layers = [K.att(heads=4, kv_heads=2, dim=16, vdim=32, window=64, mlp=K.moe(experts=6, top=2, ff=72, shared=64)),
              K.att2(heads=4, kv_heads=1, dim=32, vdim=16, mlp=K.dense(144, 1.0)),
              K.lat(heads=4, dim=32, rot=16, vdim=32, rank=64, q_rank=72, mlp=K.moe(experts=9, top=1, ff=64, shared=0)),
              K.att2(heads=4, kv_heads=1, dim=32, vdim=16, kv_from=1, mlp=K.moe(experts=4, top=4, ff=80, shared=72))]
    d = K.config(layers, width=64, vocab=64)
    tensors = make(d, 25)
    toks = K.tokens(400, d["vocab"], seed=54)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors, "bfloat16")
    n0 = m.kernel_launches()
    got = run(m, toks, [])
    assert m.kernel_launches() - n0 < 70, "the step took the per-list kernels"
    assert bf16_ok(got, want, routed=True)
    assert bf16_ok(run(m, toks, [300, 390, 395]), want, routed=True)
    monkeypatch.setenv("LIVECC_B200_SEQ_TC", "0")
    assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, []), want, routed=True)
    assert rel(run(build(d, tensors, "float32"), toks, []), want) < F32_TOL


# ---- batches, pages and slots that are used again -----------------------------------------------------------------------------
def test_a_batch_of_unequal_requests_equals_each_alone():
    m, d, _ = model_of("mixed")
    reqs = [K.tokens(n, d["vocab"], seed=30 + n) for n in (57, 9, 130)]
    alone = [run(m, t, []) for t in reqs]
    caches = [m.new_cache() for _ in reqs]
    # step 1: unequal prompt portions; step 2: one decodes, one continues its prompt, one finishes
    cut = [40, 8, 70]
    lg1 = m.forward_step([(c, t[:k]) for c, t, k in zip(caches, reqs, cut)], [list(range(k)) for k in cut]).cpu()
    lg2 = m.forward_step([(c, t[k:]) for c, t, k in zip(caches, reqs, cut)], [list(range(len(t) - k)) for t, k in zip(reqs, cut)]).cpu()
    o1 = o2 = 0
    for t, k, want in zip(reqs, cut, alone):
        got = torch.cat([lg1[o1:o1 + k], lg2[o2:o2 + len(t) - k]])
        o1, o2 = o1 + k, o2 + len(t) - k
        assert rel(got, want.double()) < F32_TOL
        assert rel(got, oracle("mixed", t)[0]) < F32_TOL
    for c in caches:
        c.release()


def test_freed_pages_and_slots_are_used_again():
    d = K.config([K.att(window=70, mlp="dense"), K.att(heads=1, dim=4, vdim=4, window=20, mlp="moe"), K.att2(window=33, mlp=None), K.att2(window=50, kv_from=2, mlp=None)],
                 width=24)
    tensors = make(d, 29)
    m = build(d, tensors, max_tokens=256)
    a, b, c3 = (K.tokens(n, d["vocab"], seed=40 + n) for n in (360, 230, 33))
    want_a, want_b, want_c = (O.forward(d, tensors, t) for t in (a, b, c3))
    ca = m.new_cache()
    got_a = torch.cat([m.forward_step([(ca, a[:300])], [list(range(300))]).cpu(), m.forward_step([(ca, a[300:])], [list(range(60))]).cpu()])
    assert rel(got_a, want_a) < F32_TOL
    # 360 tokens cached, the widest window is 70: the next token reads from position 291, in page 4
    assert [p is None for p in ca.pages] == [True, True, True, True, False, False]
    slot_a, pages_a = ca.slot, [p for p in ca.pages if p is not None]
    ca.release()
    cb = m.new_cache()
    assert cb.slot == slot_a
    got_b = m.forward_step([(cb, b[:150])], [list(range(150))]).cpu()
    cc = m.new_cache()                          # a second live request while b is half way
    got_c = m.forward_step([(cc, c3)], [list(range(len(c3)))]).cpu()
    got_b = torch.cat([got_b] + [m.forward_step([(cb, b[i:i + 2])], [[0, 1]]).cpu() for i in range(150, 230, 2)])
    assert set(pages_a) & set(p for p in cb.pages + cc.pages if p is not None), "the freed pages were not handed out again"
    assert rel(got_b, want_b) < F32_TOL and rel(got_c, want_c) < F32_TOL
    cb.release(), cc.release()
    assert len(m.pool.free) == m.pool.num_pages and len(m.pool.free_slots) == m.pool.num_slots


# ---- long decoding, generation ---------------------------------------------------------------------------------------------
def test_long_prompts_and_long_decoding_stay_on_the_oracle():
    m, d, _ = model_of("odd")
    toks = K.tokens(300, d["vocab"], seed=6)
    assert rel(run(m, toks, [4] + list(range(5, 300))), oracle("odd", toks)[0]) < F32_TOL
    assert rel(run(m, toks, [100, 131, 133, 260, 292]), oracle("odd", toks)[0]) < F32_TOL


def _generating_model():
    """The residual enters with a small alpha, so that the sublayers, not the token itself, decide the
    next token under the tied head."""
    d = json.loads(json.dumps(K.CASES["mixed"]))
    d["postln_alpha"] = 0.4
    tensors = make(d, 36)
    return build(d, tensors), d, tensors


def test_greedy_generation_through_the_engine_entry_point():
    m, d, tensors = _generating_model()
    prompt = K.tokens(37, d["vocab"], seed=8)
    want = O.greedy(d, tensors, prompt, 20)
    assert len(set(want)) > 3, "the generated tokens do not vary"
    ids = torch.tensor([prompt])
    out = m.generate(ids, max_new_tokens=20, output_logits=True)
    assert out.sequences[0, :37].tolist() == prompt and out.sequences[0, 37:].tolist() == want
    full = O.forward(d, tensors, prompt + want)
    assert rel(torch.stack(out.logits), full[36:36 + 20]) < F32_TOL     # the logits of every step are the oracle's
    assert out.past_key_values.get_seq_length() == 37 + 19              # the last token is selected, not yet run
    out.past_key_values.release()
    m.use_cuda_graph = False                    # eager launches instead of graph replay, and a prompt cut into portions
    assert m.generate(ids, max_new_tokens=20, prefill_chunk=5).sequences[0, 37:].tolist() == want
    m.use_cuda_graph = True
    stop = want[6]                              # a stop id ends the call early; a second turn continues from the cache
    first = want.index(stop)
    out = m.generate(ids, max_new_tokens=20, eos_token_id=stop)
    assert out.sequences[0, 37:].tolist() == want[:first + 1]
    turn2 = out.sequences[0].tolist() + K.tokens(5, d["vocab"], seed=9)
    out2 = m.generate(torch.tensor([turn2]), past_key_values=out.past_key_values, max_new_tokens=4)
    assert out2.sequences[0, len(turn2):].tolist() == O.greedy(d, tensors, turn2, 4)
    out2.past_key_values.release()
    got = build(d, tensors, "bfloat16").generate(ids, max_new_tokens=8).sequences[0, 37:].tolist()
    assert len(got) == 8 and all(0 <= t < d["vocab"] for t in got)


def test_generation_crosses_pages_buckets_and_temperature_steps_under_graph_replay():
    """A replayed decode step was captured at position 100; 200 tokens later the windows have moved across three page borders, the
    queries' temperature has stepped 28 times and distances have left the tables. Every step's logits against the oracle over the
    generated sequence."""
    m, d, tensors = _generating_model()
    prompt = K.tokens(100, d["vocab"], seed=10)
    out = m.generate(torch.tensor([prompt]), max_new_tokens=200, eos_token_id=-1, output_logits=True)
    seq = out.sequences[0].tolist()
    assert len(seq) == 300 and seq[:100] == prompt
    assert rel(torch.stack(out.logits), O.forward(d, tensors, seq)[99:299]) < F32_TOL
    out.past_key_values.release()


@pytest.mark.parametrize("dtype,name", [("float32", "mixed"), ("bfloat16", "dense")])
def test_trace_replay_command_line(tmp_path, dtype, name):
    """(bf16 storage on a stack without routers: with only four rows compared, one router choice that falls the other way
    under rounding would decide the result.)"""
    d = K.CASES[name]
    tensors = make(d)
    mdir = tmp_path / "model"
    mdir.mkdir()
    (mdir / "config.json").write_text(json.dumps(d))
    write_safetensors(str(mdir / "model.safetensors"), tensors)
    a, b = K.tokens(50, d["vocab"], seed=50), K.tokens(7, d["vocab"], seed=51)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[33:35], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[35:], "want": [14]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b, "want": [6]}], "end": ["y"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(mdir), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                       timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (out / "1.f32").exists()
    import numpy as np

    la, lb = O.forward(d, tensors, a), O.forward(d, tensors, b)
    g0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4")).reshape(2, -1)
    g2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4")).reshape(1, -1)
    g3 = torch.from_numpy(np.fromfile(out / "3.f32", dtype="<f4")).reshape(1, -1)
    got, want = torch.cat([g0, g2, g3]), torch.cat([la[[0, 32]], la[[49]], lb[[6]]])
    assert rel(got, want) < (F32_TOL if dtype == "float32" else BF16_TOL)
