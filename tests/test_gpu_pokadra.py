"""Pokadra models (differential attention under windows that keep the first tokens, on own or shared keys; minimal gated recurrences;
norms in groups behind the sub-layers, token pairs, token inputs per layer, averages over the depth) through the engine against the plain
restatement in oracle/layered.py, in f32 (tight) and in the serving format (bf16 products; f32 residual, scores, norms, recurrences).

The measure of a logits row is the rms of its error over the rms spread of the model's logits."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import layered as ref
from tests import layered_models as lm
from tests.layered_models import error, run, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# f32: rounding of a few hundred-term sums through a few layers.  bf16: activations and products rounded to 8 bits between
# the steps; what a misplaced key, a lost state or a wrong row does is many times that.
TOL = {True: 3e-5, False: 4e-2}
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])
NAMES = list(lm.POKADRA)


@pytest.fixture(scope="module")
def env():
    from mlx_llm_b200 import _lib, engine

    ctx = _lib.Context(0)
    yield ctx, engine
    ctx.close()


_models, _refs = {}, {}


def get_model(env, name, f32):
    ctx, eng = env
    if (name, f32) not in _models:
        cfg = lm.POKADRA[name]
        w = lm.pokadra_weights(cfg, seed=len(name))
        _models[name, f32] = (lm.load(eng, ctx, cfg, w, f32), cfg, w)
    return _models[name, f32]


def want_logits(name, cfg, w, n):
    """Oracle logits [n, vocab] of the test sequence (prefixes of one long sequence)."""
    if name not in _refs or len(_refs[name]) < n:
        _refs[name] = ref.forward(cfg, w, tokens(cfg, max(n, 200), 0))
    return _refs[name][:n]


CUTS = {"prompt": [170], "tokens": [], "twos": [2] * 90, "mixed": [3, 1, 2, 14, 1, 1, 17, 16, 2, 33, 5, 12, 13, 60], "borders": [15, 2, 31, 1, 64, 2, 1, 63],
        "chunks": [64, 1, 63, 2, 65]}


@BOTH
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("cuts", list(CUTS))
def test_portions_and_single_tokens(env, name, f32, cuts):
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    n = 170 if cuts != "twos" else 90
    pool = eng.BlockPool(ctx, model, 16, 11, 1)
    got = run(eng, model, pool, tokens(cfg, 200, 0)[:n], CUTS[cuts])
    e = error(got, want_logits(name, cfg, w, 200)[:n])
    pool.free()
    assert e < TOL[f32], e


@BOTH
@pytest.mark.parametrize("name", NAMES)
def test_stream_after_every_layer(env, name, f32):
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    ids = tokens(cfg, 40, 5)
    layers = []
    want = ref.forward(cfg, w, ids, layers)
    buf = np.zeros((len(layers), len(ids), cfg["width"]), np.float32)
    model.capture_residual(buf)
    pool = eng.BlockPool(ctx, model, 16, 4, 1)
    got = run(eng, model, pool, ids, [40])
    model.capture_residual(None)
    pool.free()
    assert error(got, want) < TOL[f32]  # looking does not change anything
    for i, x in enumerate(layers):
        assert np.abs(buf[i] - x).max() < (1e-5 if f32 else 3e-2) * np.abs(x).max(), i


@BOTH
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_with_reused_pages_and_slots(env, name, f32):
    """Portions beside single tokens in one step, requests that pause, end and hand their pages and slots on; the pool is as
    small as the schedule allows, so everything is used again."""
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    pool = eng.BlockPool(ctx, model, 16, 20, 3, 20)
    rng = np.random.default_rng(3)
    full = want_logits(name, cfg, w, 200)
    ids0 = tokens(cfg, 200, 0)
    todo = [(i, ids0[:n]) for i, n in enumerate([90, 33, 1, 118, 47, 2, 64, 150])]
    live, worst = {}, 0.0
    while todo or live:
        while todo and len(live) < 3 and sum(-(-len(v[0]) // 16) for v in live.values()) + -(-len(todo[0][1]) // 16) <= 20:
            i, ids = todo.pop(0)
            live[i] = [ids, eng.PagedKvCache(pool), 0]
        step, wants, meta = [], [], []
        for i, (ids, c, at) in live.items():
            if len(live) > 1 and rng.random() < 0.2 and step:
                continue  # sits this step out
            n = min(int(rng.choice([1, 1, 2, 5, 16, 40, 70])), len(ids) - at)
            want = sorted({int(x) for x in rng.integers(0, n, 3)} | {n - 1})
            step.append((ids[at:at + n], c))
            wants.append(want)
            meta.append((i, at, n, want))
        got, _ = model.step_at(step, wants)
        row = 0
        for i, at, n, want in meta:
            worst = max(worst, error(np.concatenate([got[row:row + len(want)], full]), np.concatenate([full[[at + x for x in want]], full])))
            row += len(want)
            live[i][2] = at + n
            if live[i][2] == len(live[i][0]):
                live.pop(i)[1].free()
    assert pool.stats()["free_pages"] == 20
    pool.free()
    assert worst < TOL[f32], worst


def single(eng, ctx, layers, f32, n=140, cuts=None, seed=2, width=64, vocab=70, change=None, gain=None, page=16, **kw):
    cfg = lm.pokadra(layers if isinstance(layers, list) else [layers], **{**dict(width=width, vocab=vocab, groups=4), **kw})
    w = lm.pokadra_weights(cfg, seed=seed, gain=gain)
    if change:
        change(w)
    w = {k: lm.round_bf16(v) for k, v in w.items()}
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, n, 9)
    pool = eng.BlockPool(ctx, model, page, -(-n // page), 1)
    e = error(run(eng, model, pool, ids, [n] if cuts is None else cuts), ref.forward(cfg, w, ids))
    pool.free()
    model.free()
    return e


ONE = pytest.mark.parametrize("cuts", [[140], [60, 1, 1, 1, 30, 2], []], ids=["prompt", "portions", "tokens"])
HEADS = [dict(heads=2, kv_heads=2, dim=32, vdim=32, dims=32), dict(heads=20, kv_heads=2, dim=16, vdim=8, dims=8), dict(heads=3, kv_heads=1, dim=64, vdim=128, dims=24),
         dict(heads=2, kv_heads=1, dim=134, vdim=48, dims=34), dict(heads=4, kv_heads=4, dim=128, vdim=65, dims=2), dict(heads=9, kv_heads=1, dim=128, vdim=128, dims=128),
         dict(heads=5, kv_heads=1, dim=64, vdim=192, dims=0), dict(heads=3, kv_heads=3, dim=7, vdim=11, dims=6), dict(heads=4, kv_heads=1, dim=64, vdim=128, dims=64)]


@BOTH
@ONE
@pytest.mark.parametrize("size,keep", [(1, 0), (2, 1), (16, 16), (33, 20), (128, 0), (30, 200), (1000, 3)])
@pytest.mark.parametrize("a", HEADS, ids=str)
def test_differential_attention_with_sharp_scores(env, cuts, f32, a, size, keep):
    """Scores scaled so that single keys stand out: one wrong, missing or extra key shows, in either map."""
    ctx, eng = env
    e = single(eng, ctx, (lm.differential(size=size, keep=keep, scale=1.5 * a["dim"] ** -0.5, base=200.0, **a), None), f32, cuts=cuts)
    assert e < (6e-5 if f32 else 0.1), e


def test_no_mask(env):
    """A layer without a mask sees everything."""
    ctx, eng = env
    for f32 in (True, False):
        for cuts in ([140], [60, 1, 1, 1, 30, 2]):
            kind, m = lm.differential()
            m = {k: v for k, v in m.items() if k != "mask"}
            e = single(eng, ctx, [((kind, m), None), ((kind, dict(m, kv_from=0, mask=dict(size=9, keep_first=2))), None)], f32, cuts=cuts)
            assert e < TOL[f32], e


@BOTH
@ONE
@pytest.mark.parametrize("scaling", [False, dict(factor=1.0), dict(factor=40.0, original=4096, fast=32.0, slow=1.0), dict(factor=3.0, original=20, fast=30.0, slow=25.0),
                                     dict(factor=7.0, original=60, fast=2.0, slow=0.01), dict(factor=0.5)], ids=str)
@pytest.mark.parametrize("base,dims", [(10000.0, 24), (30.0, 6), (5e6, 22)])
def test_rotation(env, base, dims, scaling, cuts, f32):
    """No scaling, one that changes nothing, ramps over many pairs, over none (both ends at one pair), cut off at either end."""
    ctx, eng = env
    a = lm.differential(base=base, dims=dims, scale=0.5, size=500, **(dict(scaling=True, **scaling) if scaling else dict(scaling=False)))
    e = single(eng, ctx, (a, None), f32, cuts=cuts)
    assert e < (6e-5 if f32 else 0.1), e


@BOTH
@pytest.mark.parametrize("what", ["equal", "first only", "second counts double", "negative", "no difference"])
def test_weight_of_the_second_map(env, what, f32):
    ctx, eng = env

    def change(w):
        for n, v in dict(zip(("lq1", "lk1", "lq2", "lk2"), {"equal": (0, 0, 0, 0), "first only": (0, 0, 1, 0.2624), "second counts double": (1, 0.5, 0, 0), "negative": (0, 0, 1, 1.2),
                                                            "no difference": (0.3, 0.3, 0.3, 0.3)}[what])).items():
            v = v * np.ones(24) if n[1] == "q" else v * np.ones(24) / 24
            w["l0.mix." + n] = v

    diff = {"equal": 0.9, "first only": 0.3, "second counts double": 0.4, "negative": 0.2, "no difference": 0.0}[what]
    for cuts in ([140], [60, 1, 1, 1, 30, 2]):
        e = single(eng, ctx, (lm.differential(diff=diff), None), f32, cuts=cuts, change=change)
        assert e < TOL[f32], e


@BOTH
def test_gate_per_head_decides(env, f32):
    """Gates near zero and near one, different from head to head and token to token."""
    ctx, eng = env
    for a in (dict(heads=4), dict(heads=6, kv_heads=1, dim=64, vdim=128)):
        for cuts in ([140], [60, 1, 1, 1, 30, 2]):
            e = single(eng, ctx, (lm.differential(**{**dict(kv_heads=2), **a}), None), f32, cuts=cuts, gain={"mix.g": 6.0})
            assert e < (6e-5 if f32 else 8e-2), e


def marked(size, keep, kv_from=False, heads=4, kv_heads=2, second=False):
    """A model whose queries all look for one marked token (7) in one map: the mark stands out by a score of ten and more."""
    a = dict(heads=heads, kv_heads=kv_heads, dim=32, vdim=16, dims=8, scale=0.5, diff=0.2)
    layers = [(lm.differential(size=5 if kv_from else size, keep=0 if kv_from else keep, **a), None)] + ([(lm.differential(size=size, keep=keep, kv_from=0, **a), None)] if kv_from else [])
    cfg = lm.pokadra(layers, width=64, vocab=64, groups=2, scale=1.0, side=4)
    w = lm.pokadra_weights(cfg, seed=4)
    E = np.zeros((64, 64))
    E[:, :32] = np.random.default_rng(0).standard_normal((64, 32))
    E[:, 40] = 4.0                # what every token's query asks with
    E[7, 41] = 30.0               # the mark
    w["embed"] = E
    w["bigram"] *= 0
    w["side.embed"] *= 0
    for i in range(len(layers)):
        p = f"l{i}.mix."
        w[f"l{i}.dwa"] = np.array([0.2] * (i + 1) + [0.8])
        w[p + "o"][40:42] = 0     # (a second layer finds both again)
        rows = np.arange(20, heads * 64, 32)  # coordinate 20 is not rotated
        w[p + "q"] *= 0.1
        w[p + "q"][rows, 40] = 8.0
        if p + "k" in w:
            w[p + "k"] *= 0.3
            w[p + "k"][20::32] = 0
            w[p + "k"][(52 if second else 20)::64, 41] = 4.0
    if kv_from:  # the first layer only provides the keys
        w["l0.mix.o"] *= 0
    return cfg, {k: lm.round_bf16(v) for k, v in w.items()}


@BOTH
@pytest.mark.parametrize("kv_from,second", [(False, False), (False, True), (True, False)], ids=["first map", "second map", "shared keys"])
@pytest.mark.parametrize("size,keep", [(3, 0), (16, 1), (17, 16), (50, 17), (127, 20), (128, 128), (129, 130), (300, 33)])
def test_edges_of_windows_and_first_tokens(env, kv_from, second, size, keep, f32):
    """The marked key lies just inside and just outside an edge of the window and of the kept first tokens: every position around it, in a
    prompt, in a later portion and when decoding, on pages of 16 and 48."""
    ctx, eng = env
    cfg, w = marked(size, keep, kv_from, second=second)
    model = lm.load(eng, ctx, cfg, w, f32)
    rng = np.random.default_rng(1)
    for mark in sorted({keep - 1, keep, keep + 1, 64, 15} - {-1}):
        edge = mark + size  # the first position that does not see the mark, unless it is one of the kept ones
        n = edge + 40
        ids = rng.integers(8, 64, n).astype(np.int32)
        ids[mark] = 7
        want = ref.forward(cfg, w, ids)
        gone = ids.copy()
        gone[mark] = 9
        other = ref.forward(cfg, w, gone)
        assert edge - 1 == mark or error(other[edge - 1:edge], want[edge - 1:edge]) > 0.05  # it decides what the last one that sees it answers ...
        for at in (edge, n - 1):
            e = error(other[at:at + 1], want[at:at + 1])
            assert e > 0.05 if mark < keep else e < 1e-9                                   # ... and later ones if and only if it is kept
        before = max(edge - 2, mark + 1)
        for page in (16, 48):
            pool = eng.BlockPool(ctx, model, page, -(-n // page), 1)
            for cuts in ([n], [max(n - 60, 2), 1, 2, 30], [mark + 1, before - mark - 1] + [1] * 5 + [2, 128] if before > mark + 1 else [mark + 1] + [1] * 5 + [60, 2, 128]):
                e = error(run(eng, model, pool, ids, cuts), want)
                assert e < (1e-4 if f32 else 0.08), (page, mark, cuts, e)
            pool.free()
    model.free()


@BOTH
@pytest.mark.parametrize("keep", [0, 200], ids=["window", "kept"])
def test_key_far_away(env, keep, f32):
    """One marked token among hundreds; moving the mark by one place must move the answer."""
    ctx, eng = env
    cfg, w = marked(30 if keep else 410, keep)
    model = lm.load(eng, ctx, cfg, w, f32)
    rng = np.random.default_rng(1)
    n = 420
    pool = eng.BlockPool(ctx, model, 16, -(-n // 16), 1)
    for mark in (3, 15, 16, 127, 128):
        ids = rng.integers(8, 64, n).astype(np.int32)
        ids[mark] = 7
        want = ref.forward(cfg, w, ids)
        moved = ids.copy()
        moved[mark], moved[mark + 1] = ids[mark + 1], 7
        assert error(ref.forward(cfg, w, moved)[mark:mark + 1], want[mark:mark + 1]) > 0.05
        for cuts in ([n], [200, 1, 2, 190], [mark + 1, 60, 2, 128, 1, 1, 1, 200]):
            e = error(run(eng, model, pool, ids, cuts), want)
            assert e < (1e-4 if f32 else 0.08), (mark, cuts, e)
    pool.free()
    model.free()


@BOTH
@ONE
def test_shared_keys_under_another_mask_and_scale(env, cuts, f32):
    """Later layers read the first layer's keys with masks, scales and weights of their own, the last one across a recurrent layer."""
    ctx, eng = env
    a = dict(heads=4, kv_heads=2, dim=24, vdim=16, dims=16)
    layers = [(lm.differential(size=10, keep=0, **a), None), (lm.differential(size=70, keep=11, kv_from=0, scale=0.6, diff=0.1, **a), None), (lm.mingru(), None),
              (lm.differential(size=33, keep=40, kv_from=0, scale=0.1, **a), None), (lm.differential(size=20, **a), None), (lm.differential(size=90, kv_from=4, **{**a, "heads": 6}), None)]
    e = single(eng, ctx, layers, f32, cuts=cuts)
    assert e < (6e-5 if f32 else 0.06), e


MEM_CUTS = pytest.mark.parametrize("cuts", [[140], [2] * 70, [64, 1, 63, 12], [11, 13, 65, 3], []], ids=["prompt", "twos", "portions", "short", "tokens"])


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("width", [1, 7, 8, 64, 250, 600])
def test_recurrence_alone(env, width, cuts, f32):
    ctx, eng = env
    e = single(eng, ctx, (lm.mingru(width), None), f32, cuts=cuts, seed=4)
    assert e < TOL[f32], e


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("bias,gain", [(12.0, 1.0), (-9.0, 1.0), (-60.0, 1.0), (None, 1.0), (0.0, 8.0)], ids=["forgets at once", "forgets slowly", "writes nothing", "both", "now and then"])
def test_gates_of_the_recurrence(env, bias, gain, cuts, f32):
    ctx, eng = env

    def change(w):
        v = w["l0.mix.z.b"]
        v[:] = bias if bias is not None else np.where(np.arange(len(v)) % 2, 12.0, -9.0)
        w["l0.mix.x.b"][::3] -= 2.0  # candidates on both sides of zero

    # (a state that nothing is written to leaves the norm behind it no digits)
    e = single(eng, ctx, (lm.mingru(90), None), f32, cuts=cuts, change=change, gain={"mix.z": gain})
    assert e < TOL[f32], e


@BOTH
def test_recurrence_over_a_long_sequence(env, f32):
    """Slow gates: the state still carries the first tokens hundreds of steps later, across every kind of cut."""
    ctx, eng = env
    cfg = lm.pokadra([(lm.mingru(64), None)], width=64, vocab=60, groups=4)
    w = lm.pokadra_weights(cfg, seed=6)
    w["l0.mix.z.b"][:] = -7.0
    w = {k: lm.round_bf16(v) for k, v in w.items()}
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, 520, 1)
    other = ids.copy()
    other[:4] = (other[:4] + 1) % 60
    want = ref.forward(cfg, w, ids)
    assert error(ref.forward(cfg, w, other)[-1:], want[-1:]) > 1e-3  # the first tokens still matter at the end
    pool = eng.BlockPool(ctx, model, 16, 33, 2)
    for cuts in ([520], [300] + [1] * 50 + [2, 3, 100], [400], [12, 52, 64, 65, 128, 11, 129]):
        e = error(run(eng, model, pool, ids, cuts), want)
        assert e < TOL[f32], (cuts, e)
    pool.free()
    model.free()


@BOTH
@pytest.mark.parametrize("pairs", [(1, 0, 0), (2, 1, 1), (97, 41, 13), (1000, 999, 0), (511, 0, 123457), (250, 4000000007, 3999999979)], ids=str)
def test_pairs_of_tokens(env, pairs, f32):
    """The previous token is part of a sequence's state: portions that start anywhere, a first token, products beyond 32 bits."""
    ctx, eng = env

    def change(w):
        w["bigram"] = np.random.default_rng(1).standard_normal(w["bigram"].shape) * 3

    for cuts in ([60], [], [2] * 30, [1, 30, 1, 1, 13]):
        e = single(eng, ctx, (lm.mingru(8), None), f32, n=60, cuts=cuts, pairs=pairs, change=change, scale=0.1)
        assert e < TOL[f32], e


@BOTH
@pytest.mark.parametrize("width,groups", [(64, 1), (64, 8), (54, 6), (57, 3), (57, 1), (1024, 128), (1024, 32), (520, 5), (2400, 25)])
def test_norms_in_groups(env, width, groups, f32):
    """Groups on both sides of the number of warps, of sizes that divide nothing; weights whose groups differ by orders of magnitude."""
    ctx, eng = env

    def change(w):
        for n in ("l0.mlp.down", "l0.mix.o", "l1.mix.o", "embed"):
            s = 10.0 ** (np.arange(width) * groups // width % 4 - 2)
            w[n] = w[n] * (s[None] if n == "embed" else s[:, None])

    layers = [(lm.mingru(24), lm.clipped(40)), (lm.differential(heads=2, kv_heads=1, dim=16, dims=8, vdim=16), None)]
    for cuts in ([20], [10, 1, 2]):
        assert single(eng, ctx, layers, f32, n=20, cuts=cuts, width=width, groups=groups, change=change) < (TOL[f32] if f32 else 6e-2)


@BOTH
@pytest.mark.parametrize("dim", [1, 5, 64, 72, 200])
def test_token_inputs(env, dim, f32):
    """Only the token inputs add to the stream."""
    ctx, eng = env

    def change(w):
        for i in range(3):
            w[f"l{i}.norm1"] *= 0
            if f"l{i}.norm2" in w:
                w[f"l{i}.norm2"] *= 0
            w[f"l{i}.side.norm"] += 1.0

    layers = [(lm.mingru(8), lm.clipped(16)), (lm.mingru(8), None), (lm.mingru(8), lm.clipped(16))]
    for cuts in ([50], [20, 1, 2, 1]):
        # (a single number per token has no more digits in bf16 than its gate)
        assert single(eng, ctx, layers, f32, n=50, cuts=cuts, side=dim, change=change, vocab=90) < TOL[f32]


@BOTH
@pytest.mark.parametrize("what", ["first", "last", "signs"])
def test_averages_over_the_depth(env, what, f32):
    """Layers that pass on the embedding output alone, their own result alone, and sums with both signs."""
    ctx, eng = env
    n = 7

    def change(w):
        rng = np.random.default_rng(3)
        for i in range(n):
            v = np.zeros(i + 2)
            if what == "first":
                v[0] = 1.5
            elif what == "last":
                v[-1] = 1.0
            else:
                v = rng.standard_normal(i + 2)
            w[f"l{i}.dwa"] = v

    layers = [(lm.mingru(16), lm.clipped(24) if i % 2 else None) for i in range(n)]
    for cuts in ([30], [10, 1, 13, 2]):
        assert single(eng, ctx, layers, f32, n=30, cuts=cuts, change=change, width=60, groups=2) < TOL[f32]


@BOTH
@pytest.mark.parametrize("ff,limit", [(8, 0.05), (100, 1.0), (70, 50.0)])
@pytest.mark.parametrize("mult", [0.05, 1.0, -0.7])
def test_feed_forward_alone(env, ff, limit, mult, f32):
    ctx, eng = env
    for cuts in ([70], [20, 1, 2]):
        e = single(eng, ctx, (lm.mingru(8), lm.clipped(ff, limit)), f32, n=70, cuts=cuts, mult=mult, change=lambda w: w["l0.norm1"].fill(0), gain={".gate": 3.0, ".up": 3.0})
        assert e < TOL[f32], e


def greedy(cfg, w, prompt, n):
    ids, margins = list(prompt), []
    for _ in range(n):
        a = np.sort(lg := ref.forward(cfg, w, ids)[-1])
        margins.append(a[-1] - a[-2])
        ids.append(int(np.argmax(lg)))
    return ids[len(prompt):], margins


@pytest.mark.parametrize("name", ["all_kinds", "odd"])
def test_greedy_generation_through_the_scheduler(env, name):
    """generate, generate_continuous (exact, throughput, chunked, more requests than lanes) and the serving form."""
    ctx, eng = env
    model, cfg, w = get_model(env, name, True)
    prompts = [tokens(cfg, n, 20 + n) for n in (1, 5, 21, 34, 16)]
    want = []
    for p in prompts:
        t, margins = greedy(cfg, w, p, 8)
        want.append(t[:next((i for i, m in enumerate(margins) if m < 1e-3), 8)])  # beyond a near-tie nothing is decided
    assert sum(len(t) for t in want) > 20
    check = lambda outs: [o.tokens[:len(t)] for o, t in zip(outs, want)] == want
    assert check([eng.generate(model, p, 8) for p in prompts])
    reqs = [eng.BatchRequest(p, 8) for p in prompts]
    for kw in (dict(max_batch=8), dict(max_batch=2), dict(max_batch=3, exactness=eng.THROUGHPUT),
               dict(max_batch=3, exactness=eng.THROUGHPUT, prefill_chunk_tokens=7)):
        assert check(eng.generate_continuous(model, reqs, eng.ContinuousConfig(block_size=16, **kw))), kw
    srv = eng.ServingEngine(model, eng.ContinuousConfig(max_batch=2, exactness=eng.THROUGHPUT, prefill_chunk_tokens=6, max_pages=12, max_blocks_per_seq=6))
    rids = [srv.submit(r) for r in reqs]
    for _ in range(200):
        if srv.step():
            break
    assert check([srv.result(r) for r in rids])
    srv.free()


@pytest.mark.parametrize("name", ["all_kinds", "tiles"])
def test_long_decoding(env, name):
    ctx, eng = env
    model, cfg, w = get_model(env, name, False)
    ids = tokens(cfg, 400, 0)
    pool = eng.BlockPool(ctx, model, 16, 25, 1)
    e = error(run(eng, model, pool, ids, [20]), want_logits(name, cfg, w, 400))
    pool.free()
    assert e < TOL[False], e


@BOTH
@pytest.mark.parametrize("name", ["odd", "tiles"])
@pytest.mark.parametrize("n", [16, 17, 32, 33, 64, 65, 100])
def test_many_sequences_in_one_step(env, name, n, f32):
    """Batches on both sides of the sizes at which products are done differently: every sequence decodes one token."""
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    full = want_logits(name, cfg, w, 200)
    ids = tokens(cfg, 200, 0)
    pool = eng.BlockPool(ctx, model, 16, 3 * n, n, 3)
    caches, lens = [eng.PagedKvCache(pool) for _ in range(n)], [3 + (7 * i) % 29 for i in range(n)]
    model.step_at([(ids[:k], c) for k, c in zip(lens, caches)], [[] for _ in lens])
    for s in range(2):
        got, _ = model.step_at([(ids[k + s:k + s + 1], c) for k, c in zip(lens, caches)], [[0]] * n)
        assert error(np.concatenate([got, full]), np.concatenate([full[[k + s for k in lens]], full])) < TOL[f32]
    for c in caches:
        c.free()
    pool.free()


def test_long_contexts_are_split_over_keys(env):
    """Windows of many work items with and without kept keys, several sequences at different places of them, alone and beside a portion:
    partial results are added up, and the maps of a head are taken off one another only then."""
    ctx, eng = env
    cfg = lm.pokadra([(lm.differential(heads=4, kv_heads=1, dim=64, vdim=128, dims=64, size=600, keep=150), None), (lm.differential(heads=6, kv_heads=2, dim=64, vdim=64, dims=64, size=650, keep=0), None),
                      (lm.differential(heads=3, kv_heads=3, dim=32, vdim=32, dims=32, size=180, keep=300), None), (lm.differential(heads=20, kv_heads=1, dim=64, vdim=64, dims=64, size=2000), None)],
                     width=96, vocab=150, groups=4)
    w = lm.pokadra_weights(cfg, seed=1)
    model = lm.load(eng, ctx, cfg, w, False)
    n = 1000
    ids = tokens(cfg, n, 0)
    full = ref.forward(cfg, w, ids)
    pool = eng.BlockPool(ctx, model, 16, 260, 6, 63)
    caches, lens = [eng.PagedKvCache(pool) for _ in range(5)], [647, 130, 990, 200, 663]
    model.step_at([(ids[:k], c) for k, c in zip(lens, caches)], [[] for _ in lens])
    extra = eng.PagedKvCache(pool)
    for s in range(6):
        got, _ = model.step_at([(ids[k + s:k + s + 1], c) for k, c in zip(lens, caches)] + [(ids[s * 40:s * 40 + 40], extra)], [[0]] * 5 + [[39]])
        assert error(got, full[[k + s for k in lens] + [s * 40 + 39]]) < TOL[False]
    for c in caches + [extra]:
        c.free()
    pool.free()
    model.free()


def test_caches(env):
    """Fork copies pages, states and the last token; a layer that reads another layer's keys has no pages of its own; a slot that is used
    again starts anew."""
    ctx, eng = env
    model, cfg, w = get_model(env, "all_kinds", True)
    assert model.state_bytes() > 0
    ids = tokens(cfg, 200, 0)[:60]
    full = want_logits("all_kinds", cfg, w, 200)
    pool = eng.BlockPool(ctx, model, 16, 12, 3)
    a = eng.PagedKvCache(pool)
    model.step_at([(ids[:37], a)], [[]])
    b = a.fork(37)
    got, _ = model.step_at([(ids[37:40], a), (ids[37:38], b)], [[2], [0]])
    assert error(got, full[[39, 37]]) < TOL[True]
    got, _ = model.step_at([(ids[38:60], b)], [[21]])
    assert error(got, full[[59]]) < TOL[True]
    a.reset()
    got, _ = model.step_at([(ids[:1], a)], [[0]])
    assert error(got, full[[0]]) < TOL[True]
    got, _ = model.step_at([(ids[1:50], a)], [[48]])
    assert error(got, full[[49]]) < TOL[True]
    a.free()
    b.free()
    pool.free()


def test_shapes_that_do_not_fit_are_refused(env):
    from mlx_llm_b200._lib import B2Error

    ctx, eng = env
    cfg = lm.POKADRA["all_kinds"]
    w = lm.pokadra_weights(cfg)
    for key, new in (("l0.mix.q", (96, 72)), ("l0.mix.lk2", (25,)), ("l1.mix.z.b", (87,)), ("l2.dwa", (3,)), ("l0.side.proj", (72, 21)), ("side.embed", (211, 100)), ("bigram", (103, 72)), ("l4.mix.k.norm", (32,)),
                     ("head", (211, 71))):
        bad = copy.copy(w)
        bad[key] = np.zeros(new)
        with pytest.raises(B2Error) as e:
            lm.load(eng, ctx, cfg, bad, True)
        assert e.value.code == -4 and key in str(e.value)
    bad = copy.copy(w)
    bad.pop("l3.mix.x.b")
    with pytest.raises(B2Error) as e:
        lm.load(eng, ctx, cfg, bad, True)
    assert "l3.mix.x.b" in str(e.value)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(env, tmp_path, dtype):
    cfg = lm.POKADRA["all_kinds"]
    w = lm.pokadra_weights(cfg, seed=11)
    lm.save(tmp_path / "m", cfg, w)
    ids = [tokens(cfg, n, n).tolist() for n in (30, 9)]
    full = [ref.forward(cfg, w, t) for t in ids]
    steps = [dict(step=0, entries=[dict(id="a", tokens=ids[0][:20], want=[0, 19]), dict(id="b", tokens=ids[1][:1], want=[])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=ids[1][1:], want=[7])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=ids[0][20:], want=[]), dict(id="c", tokens=ids[1], want=[8])], end=["a", "c"])]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    got = [np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]) for i in range(3)]
    tol = TOL[dtype == "float32"]
    assert error(got[0], full[0][[0, 19]]) < tol and error(got[1], full[1][[8]]) < tol and error(got[2], full[1][[8]]) < tol
