"""Kapitar on the GPU against the float64 oracle (tests/kapitar_oracle.py): every mechanism alone and together, whole prompts
against token-by-token decoding, portions down to two tokens, batches against each request alone, pages between the kept tokens
and the window, pages and slots that are used again, keys far away, at page borders, just inside / just outside the window and
among / just behind the first tokens it keeps, in either of the two maps with a sharp softmax, a first token that only the
recurrent state carries, the router's groups, long decoding, unusual sizes, and greedy generation through the engine's own
entry point. fp32 storage is compared tightly; bf16 storage within bf16 rounding."""
import json
import os
import subprocess

import pytest
import torch

import kapitar_cases as K
import kapitar_oracle as O
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


def close32(got, want):
    """fp32 storage against the oracle: every row within the tolerance, but for the few rows (at most 2 in 100) in which the two
    maps or a sublayer's output nearly cancel: the norm behind them scales such a row up, rounding included. Those stay within ten
    times the tolerance."""
    e = rows_rel(got, want)
    return float(e.max()) < 10 * F32_TOL and float((e > F32_TOL).double().mean()) <= 0.02


def bf16_ok(got, want, routed=False):
    """bf16 storage: the bulk of the rows stays within bf16 rounding and few rows lie beyond twice that. routed: a stack with
    routers, where a score close to the next one can fall the other way under rounding and hand the stream another expert's row,
    which attention and the recurrence carry to later positions: held to rounding in the median only."""
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


ALL = ["attention_only", "lightning_only", "dense", "moe", "mixed", "odd"]


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
        assert close32(dump[li], want_layers[li]), f"residual stream after layer {li}"
    assert close32(lg, want_lg)


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


@pytest.mark.parametrize("name,what", [("attention_only", "bias"), ("attention_only", "softcap"), ("attention_only", "window"), ("attention_only", "keep_first"),
                                       ("attention_only", "second_map"), ("moe", "groups"), ("moe", "group_sum"), ("moe", "shared")])
def test_each_mechanism_shows_in_these_weights(name, what):
    """An oracle that drops the projections' biases, the soft cap, the window, the kept tokens, the second map, the limit to the best
    groups, the second score of a group's sum, or the shared expert is far outside the tolerance: the other tests would notice a
    product that left any of them out."""
    m, d, _ = model_of(name)
    toks = K.tokens(90, d["vocab"])
    got = run(m, toks, [])
    assert close32(got, oracle(name, toks)[0])
    assert rel(got, oracle(name, toks, leave_out=(what,))[0]) > 100 * F32_TOL


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations_in_three_schedules(seed):
    """Random stacks (tests/kapitar_cases.py::random_config): the whole prompt, most of it then token by token, and portions of
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
        assert close32(run(m, toks, cuts), want)
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
    assert close32(run(m, toks, range(1, 100)), want_lg)          # every token alone, from the first one
    assert close32(run(m, toks, [41] + list(range(42, 100))), want_lg)


@pytest.mark.parametrize("cuts", [[2, 4, 6, 9, 11, 40, 42], [1, 3, 64, 66], [9, 10, 12, 13, 47, 49, 65], [63, 65, 67, 69], [15, 31, 33, 64, 80, 82]])
def test_portions_of_any_size_down_to_two_tokens(cuts):
    """(cuts at a window's and the kept tokens' edges, at page borders, and where the recurrence and the attention change kernels)"""
    m, d, _ = model_of("mixed")
    toks = K.tokens(100, d["vocab"], seed=2)
    assert close32(run(m, toks, cuts), oracle("mixed", toks)[0])


def test_first_tokens_of_a_sequence():
    for name in ("mixed", "odd"):
        m, d, _ = model_of(name)
        for n in (1, 2, 3, 4):
            toks = K.tokens(n, d["vocab"], seed=20 + n)
            assert rel(run(m, toks, []), oracle(name, toks)[0]) < F32_TOL
            assert rel(run(m, toks, range(1, n)), oracle(name, toks)[0]) < F32_TOL


# ---- the recurrent state ------------------------------------------------------------------------------------------------------
def test_a_first_token_that_only_the_recurrent_state_carries():
    """One lightning layer with decays of 1 and close to it: what the first token wrote is still read 190 tokens later, through every
    cut of the prompt (token by token, short portions, blocks of the sequence-parallel form); another first token moves the last
    rows by far more than the tolerance. A decay of 0 keeps a token's own write only."""
    d = K.config([K.light(heads=3, dim=20, vdim=6, decay=[1.0, 0.999, 0.995], mlp=None)], width=16, vocab=40)
    tensors = make(d, 23)
    toks = K.tokens(190, d["vocab"], seed=70)
    other = [(toks[0] + 1) % d["vocab"]] + toks[1:]
    want = O.forward(d, tensors, toks)
    assert rel(O.forward(d, tensors, other)[-3:], want[-3:]) > 100 * F32_TOL, "the first token does not reach the end"
    m = build(d, tensors)
    for cuts in ([], [1], [2, 50], [63, 127], [64, 128], [65, 129], [160] + list(range(161, 190)), list(range(1, 190))):
        assert rel(run(m, toks, cuts), want) < F32_TOL
    assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, [2, 50, 188]), want)
    d = K.config([K.light(heads=2, dim=8, vdim=4, decay=[0.0, 1e-6], mlp=None)], width=16, vocab=40)
    tensors = make(d, 24)
    assert rel(run(build(d, tensors), toks, [100, 102] + list(range(170, 190))), O.forward(d, tensors, toks)) < F32_TOL


@pytest.mark.parametrize("heads,dim,vdim", [(2, 128, 64), (4, 64, 128), (1, 200, 24), (3, 17, 130), (2, 512, 8), (8, 32, 96)])
def test_lightning_heads_of_many_sizes(heads, dim, vdim):
    d = K.config([K.light(heads=heads, dim=dim, vdim=vdim, decay=[0.5 + 0.49 * i / heads for i in range(heads)], mlp=None)], width=64, vocab=64)
    tensors = make(d, 33)
    toks = K.tokens(140, d["vocab"], seed=55)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL
    assert rel(run(m, toks, [33, 35] + list(range(120, 140))), want) < F32_TOL
    assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, [100]), want)


# ---- far keys, page borders, the window's and the kept tokens' edges ------------------------------------------------------
def _key_model(window=100, keep=6, mp=0, seed=22):
    """One attention layer whose weights make one key stand out in map `mp`: token A (the key) and token B (the query) have one-hot
    embeddings in columns of their own; one key channel of that map reads A's column, one query channel of the same map of every head
    reads B's. B's score against A is then about 30 (behind the cap), against every other key a few, wherever A sits; A's
    value row is large, so whether A is seen moves the output by far more than the tolerance."""
    d = json.loads(json.dumps(K.CASES["sharp"]))
    mx = d["layers"][0]["mixer"]
    mx["mask"] = {"size": window, "keep_first": keep}
    tensors = make(d, seed)
    A, B, ja, jb, ch = 5, 9, 3, 11, 2
    D, H = mx["dim"], mx["heads"]
    tensors["l0.norm1"].fill_(1.0)
    for col in (ja, jb):
        tensors["embed"][:, col] = 0.0
    for tok, col in ((A, ja), (B, jb)):
        tensors["embed"][tok].zero_()
        tensors["embed"][tok, col] = 2.0
    tensors["l0.mix.k"][mp * D + ch].zero_()
    tensors["l0.mix.k"][mp * D + ch, ja] = 2.3
    tensors["l0.mix.v"][:, ja] = 6.0
    for h in range(H):
        tensors["l0.mix.q"][(2 * h + mp) * D + ch].zero_()
        tensors["l0.mix.q"][(2 * h + mp) * D + ch, jb] = 2.3
    return d, tensors, A, B


def _with_key(d, n, key_at, A, B, query_at, seed):
    toks = [t if t not in (A, B) else 17 for t in K.tokens(n, d["vocab"], seed=seed)]
    toks[key_at] = A
    for q in query_at:
        toks[q] = B
    return toks


@pytest.mark.parametrize("mp", [0, 1])
@pytest.mark.parametrize("far_at", [0, 1, 62, 63, 64, 65, 127, 128, 200])
def test_a_far_key_among_hundreds_at_page_borders(far_at, mp):
    """A window of 300 over a 300-token sequence: A sits once at `far_at` (first tokens, just before / on / after a page border, deep
    inside), B queries it from the end: in one prompt, decoded alone, and at the start of a two-token portion; in fp32 and in bf16
    on the tensor-core attention; the key standing out in the first or in the second map."""
    d, tensors, A, B = _key_model(300, 0, mp)
    toks = _with_key(d, 300, far_at, A, B, [298, 299], seed=7)
    moved = list(toks)
    moved[far_at] = 17
    want = O.forward(d, tensors, toks)
    assert rel(O.forward(d, tensors, moved)[-2:], want[-2:]) > 1e3 * F32_TOL, "the far key does not stand out"
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL
    assert rel(run(m, toks, [250] + list(range(251, 300))), want) < F32_TOL
    assert rel(run(m, toks, [66, 129, 298]), want) < F32_TOL
    assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, [66, 129, 298]), want)


@pytest.mark.parametrize("window", [1, 2, 7, 63, 64, 65, 100, 128, 129, 300])
@pytest.mark.parametrize("inside", [True, False])
def test_keys_just_inside_and_just_outside_the_window(window, inside):
    """The query at position i, the key at i - window + 1 (the last one the window keeps) or at i - window (the first one it drops):
    windows shorter than, equal to and longer than a page and a key tile; in one prompt, with the query decoded alone, at the
    start and at the end of short portions, and through the tiled kernels in bf16."""
    d, tensors, A, B = _key_model(window, 6, window % 2)
    n, i = 420, 401
    key_at = i - window + 1 if inside else i - window
    toks = _with_key(d, n, key_at, A, B, [i], seed=11)
    want = O.forward(d, tensors, toks)
    other = O.forward(d, tensors, toks, leave_out=("window",))
    if window > 1:      # (a window of one position holds the query and the kept tokens)
        gap = rel(other[i:i + 1], want[i:i + 1])
        assert gap < 0.05 if inside else gap > 0.05, "the test's key does not show the window's edge"
    m = build(d, tensors)
    for cuts in ([], [i] + list(range(i + 1, n)), [key_at + 1, i, i + 2], [i - 1, i + 1], [200, i - 30]):
        assert rel(run(m, toks, cuts), want) < F32_TOL, cuts
    bf = build(d, tensors, "bfloat16")
    assert bf16_ok(run(bf, toks, []), want)
    assert bf16_ok(run(bf, toks, [i] + list(range(i + 1, n))), want)


@pytest.mark.parametrize("keep", [1, 2, 20, 63, 64, 65, 130])
@pytest.mark.parametrize("kept", [True, False])
def test_the_last_token_a_window_keeps_and_the_next_one(keep, kept):
    """A key at position keep - 1 stays visible for good, one at position `keep` leaves with the window: read from far behind (pages
    between the two have gone back), from the window's last position over it, and from the first position past it; windows that
    start inside, at the end of and behind the kept tokens while the prompt runs."""
    window = 70
    d, tensors, A, B = _key_model(window, keep, keep % 2)
    key_at = keep - 1 if kept else keep
    n, at = 420, [key_at + window - 1, key_at + window, 300, 401]
    toks = _with_key(d, n, key_at, A, B, at, seed=12)
    want = O.forward(d, tensors, toks)
    without = O.forward(d, tensors, toks, leave_out=("keep_first",))
    if kept:
        assert rel(without[401:402], want[401:402]) > 0.05, "the test's key does not show the kept tokens' edge"
    else:
        seen = list(toks)
        seen[key_at] = 17
        gone = O.forward(d, tensors, seen)
        assert rel(gone[401:402], want[401:402]) < 1e-9 and rel(gone[at[0]:at[0] + 1], want[at[0]:at[0] + 1]) > 0.05
    m = build(d, tensors)
    for cuts in ([], [401] + list(range(402, n)), [keep, keep + 2, at[0], at[1], at[1] + 2], [key_at + 1, 299, 301], list(range(40, n, 40))):
        assert rel(run(m, toks, cuts), want) < F32_TOL, cuts
    c = m.new_cache()
    m.forward_step([(c, toks[:380])])
    assert c.live_pages() == (keep + 63) // 64 + len([p for p in range((keep + 63) // 64, 6) if (p + 1) * 64 > 380 - window + 1])
    assert rel(m.forward_step([(c, toks[380:])], [list(range(40))]), want[380:]) < F32_TOL
    c.release()
    bf = build(d, tensors, "bfloat16")
    assert bf16_ok(run(bf, toks, []), want)
    assert bf16_ok(run(bf, toks, [100, 401] + list(range(402, n))), want)


def test_every_position_while_the_window_leaves_the_kept_tokens():
    """Windows shorter and longer than the kept head: every position of a prompt, decoded from the first token on, as the visible
    range goes from whole to kept head + window with a gap."""
    for window, keep in ((5, 12), (30, 4), (64, 64), (1, 1)):
        d, tensors, A, B = _key_model(window, keep)
        toks = _with_key(d, 150, keep - 1, A, B, [window + keep - 2, window + keep - 1, window + keep, 149], seed=15)
        want = O.forward(d, tensors, toks)
        m = build(d, tensors)
        for cuts in ([], list(range(1, 150)), [2, keep + 2, window + keep, window + keep + 2], list(range(17, 150, 17))):
            assert rel(run(m, toks, cuts), want) < F32_TOL, (window, keep, cuts)


@pytest.mark.parametrize("window,keep", [(700, 20), (700, 150), (0, 0)])
def test_long_windows_in_steps_of_a_few_rows_split_the_keys(window, keep):
    """A window of 700 positions (and plain causal attention) in steps of one to three rows: the keys are split over several CTAs
    and merged by the last to arrive. The key at the window's first position, just before it, at tile edges and in the kept
    head; then through generation, where only the device knows the position."""
    d, tensors, A, B = _key_model(max(window, 1), keep, 1)
    if not window:
        del d["layers"][0]["mixer"]["mask"]
    n = 1000
    m = build(d, tensors)
    for key_at in (0, 19, 20, 149, 150, n - 1 - 700, n - 700, 383, 384, 998):
        toks = _with_key(d, n, key_at, A, B, [n - 1, n - 3], seed=13)
        want = O.forward(d, tensors, toks)
        cuts = [950, 952, 955] + list(range(956, n))
        assert rel(run(m, toks, cuts), want) < F32_TOL, key_at
        if key_at in (19, n - 700):
            assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, cuts), want)
    tensors["embed"] *= 0.25                     # (tied head: let the sublayers decide the next token)
    m = build(d, tensors)
    toks = _with_key(d, n, 10, A, B, [959], seed=14)
    new = O.greedy(d, tensors, toks[:960], 4)
    out = m.generate(torch.tensor([toks[:960]]), max_new_tokens=4, output_logits=True)
    assert out.sequences[0, 960:].tolist() == new
    assert rel(torch.stack(out.logits), O.forward(d, tensors, toks[:960] + new)[959:963]) < F32_TOL
    out.past_key_values.release()


# ---- scores, heads, lambda ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cap,scale", [(0.5, 2.0), (50.0, 0.14), (3.0, 40.0), (0.0, 1.0), (1000.0, 5.0)])
def test_soft_caps_from_saturated_to_open(cap, scale):
    d = K.config([K.att(heads=2, kv_heads=1, dim=16, vdim=8, window=50, keep=3, cap=cap, scale=scale, mlp=None)], width=32, vocab=64)
    tensors = make(d, 27)
    toks = K.tokens(130, d["vocab"], seed=57)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    tol = F32_TOL * (10 if cap != 0.5 and scale >= 5 else 1)        # large scores: the exponentials amplify the products' rounding
    assert rel(run(m, toks, []), want) < tol
    assert rel(run(m, toks, [100, 103] + list(range(110, 130))), want) < tol
    bf = run(build(d, tensors, "bfloat16"), toks, [])
    assert bool(torch.isfinite(bf).all()) and (scale >= 5 or bf16_ok(bf, want))


@pytest.mark.parametrize("diff,shift", [(0.0, 0.0), (0.2, 1.0), (0.8, -1.0)])
def test_the_second_maps_weight(diff, shift):
    """lambda from below zero to above one (the vectors that make it scaled up), with and without a starting value."""
    d = K.config([K.att(heads=4, kv_heads=2, dim=8, vdim=16, diff=diff, window=40, mlp=None)], width=32, vocab=64)
    tensors = make(d, 28)
    for n in ("lq1", "lk1") if shift > 0 else ("lq2", "lk2"):
        tensors["l0.mix." + n].fill_(0.3 * abs(shift))
    toks = K.tokens(90, d["vocab"], seed=58)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    assert close32(run(m, toks, []), want)
    assert close32(run(m, toks, [60] + list(range(61, 90))), want)
    assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, [40]), want)


@pytest.mark.parametrize("dim,vdim,heads,kv", [(136, 40, 2, 1), (72, 136, 4, 2), (128, 256, 2, 1), (256, 256, 2, 2), (300, 24, 1, 1), (64, 300, 2, 1), (20, 129, 3, 3),
                                               (24, 16, 4, 1), (13, 22, 2, 2), (40, 600, 1, 1)])
def test_attention_heads_of_many_sizes(dim, vdim, heads, kv):
    """Values up to 256 channels (both maps in one tensor-core CTA), beyond (one map per CTA, the difference behind them), beyond what
    the key-split kernel takes, and head sizes that are not multiples of 8 or 16."""
    d = K.config([K.att(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, window=90, keep=10, cap=30.0, scale=dim ** -0.5, mlp=None)], width=32, vocab=64)
    tensors = make(d, 24)
    toks = K.tokens(215, d["vocab"], seed=52)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    assert rel(run(m, toks, []), want) < F32_TOL
    assert rel(run(m, toks, [64, 128, 129, 193] + list(range(205, 215))), want) < F32_TOL
    m = build(d, tensors, "bfloat16")
    assert bf16_ok(run(m, toks, []), want)
    assert bf16_ok(run(m, toks, [64, 129, 193] + list(range(194, 215))), want)


# ---- long prompts, wide rows, experts -------------------------------------------------------------------------------------
def test_long_prompts_cross_many_key_tiles_and_blocks():
    m, d, _ = model_of("odd")
    toks = K.tokens(333, d["vocab"], seed=50)
    want_lg, want_layers = oracle("odd", toks)
    c = m.new_cache()
    lg, dump = m.forward_step([(c, toks)], [list(range(333))], layer_dump=True)
    c.release()
    for li in range(len(d["layers"])):
        assert close32(dump[li], want_layers[li]), f"residual stream after layer {li}"
    assert close32(lg, want_lg)
    assert close32(run(m, toks, [100, 131, 133, 260, 292]), want_lg)


@pytest.mark.parametrize("width", [1, 30, 1028, 2050, 5000])
def test_rows_of_many_widths(width):
    """The norms' forms: one to sixteen pieces per thread, four columns a piece or one, rows beyond what a thread keeps; a mean away from
    zero (a constant added to the embedding) that the layer norms take off. (The tied head multiplies that constant with a row whose
    sum nearly cancels: the constant is kept small.)"""
    d = K.config([K.light(heads=1, dim=4, vdim=4, mlp=K.dense(8)), K.att(heads=1, dim=4, vdim=4, mlp=K.moe(experts=2, top=1, ff=8, groups=None, shared=8))],
                 width=width, vocab=30)
    tensors = make(d, 35)
    if width > 1:
        tensors["embed"] += 2.0
    toks = K.tokens(40, d["vocab"], seed=59)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors)
    if width == 1:                              # a row of one column minus its mean is zero: every norm's output is zero
        assert not bool(want.any()) and not bool(run(m, toks, [20]).any())
        return
    assert rel(run(m, toks, []), want) < 5 * F32_TOL
    assert rel(run(m, toks, [30] + list(range(31, 40))), want) < 5 * F32_TOL


def test_many_rows_per_expert_and_experts_without_rows():
    """300 rows over 33 experts (top 5 out of 7 of 11 groups) and over 2 experts (top 1): lists longer than one tile, lists of a few
    rows, empty lists; the same rows decoded one by one take the few-row kernel."""
    m, d, _ = model_of("odd")
    toks = K.tokens(300, d["vocab"], seed=53)
    want = oracle("odd", toks)[0]
    assert close32(run(m, toks, []), want)
    assert close32(run(m, toks, [280, 290] + list(range(291, 300))), want)


def test_experts_and_feed_forward_on_the_tensor_cores(monkeypatch):
    """bf16 storage with enough routed rows and 8-aligned shapes: expert lists are padded to whole 128-row tiles and both expert
    products run as one grouped tensor-core GEMM each with the gelu in the first one's epilogue; the dense feed-forward's squared
    relu and the shared expert's gelu ride in their first product. Against the oracle, against the CUDA-core route, and with the prompt
    cut so that later portions take the few-row route."""
    layers = [K.att(heads=2, kv_heads=1, dim=8, vdim=16, mlp=K.moe(experts=6, top=2, ff=72, groups=(3, 2), shared=64)),
              K.light(heads=2, dim=8, vdim=8, mlp=K.dense(136)),
              K.att(heads=4, kv_heads=2, dim=16, vdim=32, window=64, mlp=K.moe(experts=9, top=1, ff=64, groups=(3, 1), shared=0)),
              K.light(heads=2, dim=16, vdim=32, mlp=K.moe(experts=4, top=4, ff=80, groups=None, shared=72))]
    d = K.config(layers, width=64, vocab=64)
    tensors = make(d, 25)
    toks = K.tokens(400, d["vocab"], seed=54)
    want = O.forward(d, tensors, toks)
    m = build(d, tensors, "bfloat16")
    n0 = m.kernel_launches()
    got = run(m, toks, [])
    assert m.kernel_launches() - n0 < 90, "the step took the per-list kernels"
    assert bf16_ok(got, want, routed=True)
    assert bf16_ok(run(m, toks, [300, 390, 395]), want, routed=True)
    monkeypatch.setenv("LIVECC_B200_SEQ_TC", "0")
    assert bf16_ok(run(build(d, tensors, "bfloat16"), toks, []), want, routed=True)
    assert close32(run(build(d, tensors, "float32"), toks, []), want)


def test_router_groups_and_weights():
    """Router rows shaped so that the first group holds the single best expert and the other two the better pairs for every token: a
    group that scored as its best expert alone would choose otherwise; the weights are the scores as they are (their sum is not 1)."""
    d = K.config([K.light(mlp=K.moe(experts=9, top=3, ff=8, groups=(3, 2), shared=6))], width=16, vocab=40)
    tensors = make(d, 34)
    r = tensors["l0.mlp.router"]
    u = r[0].clone().float()
    tensors["l0.norm2"].fill_(1.0)
    for e, s in enumerate((1.0, -1.0, -1.2, 0.8, 0.7, -1.0, 0.9, 0.5, -1.1)):
        r[e] = (s * u).to(r.dtype)
    toks = K.tokens(60, d["vocab"], seed=56)
    want = O.forward(d, tensors, toks)
    assert rel(O.forward(d, tensors, toks, leave_out=("group_sum",)), want) > 100 * F32_TOL
    assert rel(O.forward(d, tensors, toks, leave_out=("groups",)), want) > 100 * F32_TOL
    m = build(d, tensors)
    assert close32(run(m, toks, []), want)                                   # few rows and many rows: both router kernels
    assert close32(run(m, toks, [30, 32] + list(range(40, 60))), want)
    long = K.tokens(200, d["vocab"], seed=61)
    assert close32(run(m, long, []), O.forward(d, tensors, long))


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
        assert close32(got, oracle("mixed", t)[0])
    for c in caches:
        c.release()


def test_freed_pages_and_slots_are_used_again():
    d = K.config([K.att(window=70, keep=10, mlp="dense"), K.light(mlp=None), K.att(heads=1, dim=4, vdim=4, window=20, keep=70, mlp="moe")], width=24)
    tensors = make(d, 29)
    m = build(d, tensors, max_tokens=256)
    a, b, c3 = (K.tokens(n, d["vocab"], seed=40 + n) for n in (360, 230, 33))
    want_a, want_b, want_c = (O.forward(d, tensors, t) for t in (a, b, c3))
    ca = m.new_cache()
    got_a = torch.cat([m.forward_step([(ca, a[:300])], [list(range(300))]).cpu(), m.forward_step([(ca, a[300:])], [list(range(60))]).cpu()])
    assert close32(got_a, want_a)
    # 360 tokens cached, 70 kept ones (pages 0 and 1), the widest window is 70: the next token reads from position 291, in page 4
    assert [p is None for p in ca.pages] == [False, False, True, True, False, False]
    slot_a, pages_a = ca.slot, [p for p in ca.pages if p is not None]
    ca.release()
    cb = m.new_cache()
    assert cb.slot == slot_a                    # the slot's recurrent state starts from zero again
    got_b = m.forward_step([(cb, b[:150])], [list(range(150))]).cpu()
    cc = m.new_cache()                          # a second live request while b is half way
    got_c = m.forward_step([(cc, c3)], [list(range(len(c3)))]).cpu()
    got_b = torch.cat([got_b] + [m.forward_step([(cb, b[i:i + 2])], [[0, 1]]).cpu() for i in range(150, 230, 2)])
    assert set(pages_a) & set(p for p in cb.pages + cc.pages if p is not None), "the freed pages were not handed out again"
    assert close32(got_b, want_b) and close32(got_c, want_c)
    cb.release(); cc.release()
    assert len(m.pool.free) == m.pool.num_pages and len(m.pool.free_slots) == m.pool.num_slots


# ---- long decoding, generation ---------------------------------------------------------------------------------------------
def test_long_decoding_stays_on_the_oracle():
    m, d, _ = model_of("odd")
    toks = K.tokens(300, d["vocab"], seed=6)
    assert close32(run(m, toks, [4] + list(range(5, 300))), oracle("odd", toks)[0])


def _generating_model():
    """The embedding scaled down so that the sublayers, not the token itself, decide the next token under the tied head."""
    d = K.CASES["mixed"]
    tensors = make(d, 36)
    tensors["embed"] *= 0.2
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
    assert close32(torch.stack(out.logits), full[36:36 + 20])           # the logits of every step are the oracle's
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


def test_generation_moves_the_window_across_pages_under_graph_replay():
    """A replayed decode step was captured at position 100; 200 tokens later the windows (9 positions behind 3 kept ones, 70 behind
    10) have moved across three page borders and the recurrent state has taken 200 more writes. Every step's logits against the
    oracle over the generated sequence."""
    m, d, tensors = _generating_model()
    prompt = K.tokens(100, d["vocab"], seed=10)
    out = m.generate(torch.tensor([prompt]), max_new_tokens=200, eos_token_id=-1, output_logits=True)
    seq = out.sequences[0].tolist()
    assert len(seq) == 300 and seq[:100] == prompt
    assert close32(torch.stack(out.logits), O.forward(d, tensors, seq)[99:299])
    assert [p is None for p in out.past_key_values.pages[:4]] == [False, True, True, False]
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
