"""Tirezen models (retention, delta memories, capped sink attention beside a delta memory, parallel layers, a repeated
stretch of layers) through the engine against the plain restatement in oracle/layered.py, in f32 (tight) and in the serving
format (bf16 products; f32 residual, scores, recurrences).

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
# the steps; what a misplaced key, a lost state or a missing sink does is many times that.
TOL = {True: 3e-5, False: 4e-2}
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])


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
        cfg = lm.TIREZEN[name]
        w = lm.tirezen_weights(cfg, seed=len(name))
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
@pytest.mark.parametrize("name", list(lm.TIREZEN))
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
@pytest.mark.parametrize("name", ["all_kinds", "odd", "tiles"])
def test_residual_after_every_layer_run(env, name, f32):
    """A repeated layer counts each time; what comes ahead of the next pass is not in it."""
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    ids = tokens(cfg, 40, 5)
    layers = []
    ref.forward(cfg, w, ids, layers)
    assert len(layers) == len(ref.layer_runs(cfg))
    buf = np.zeros((len(layers), len(ids), cfg["width"]), np.float32)
    model.capture_residual(buf)
    pool = eng.BlockPool(ctx, model, 16, 4, 1)
    run(eng, model, pool, ids, [40])
    model.capture_residual(None)
    pool.free()
    for i, x in enumerate(layers):
        assert np.abs(buf[i] - x).max() < (2e-4 if f32 else 0.25), i


@BOTH
@pytest.mark.parametrize("name", ["all_kinds", "odd", "tiles", "uneven", "large_heads"])
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


def single(eng, ctx, layer, f32, n=140, cuts=None, seed=2, width=64, vocab=70, change=None, gain=None, loop=(0, 0, 0), page=16):
    cfg = lm.tirezen([layer], width=width, vocab=vocab, loop=loop)
    w = lm.tirezen_weights(cfg, seed=seed, gain=gain)
    if change:
        change(w)
    w = {k: lm.round_bf16(v) for k, v in w.items()}
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, n, 9)
    pool = eng.BlockPool(ctx, model, page, -(-n // page), 1)
    got = run(eng, model, pool, ids, [n] if cuts is None else cuts)
    e = error(got, ref.forward(cfg, w, ids))
    pool.free()
    model.free()
    return e


ONE = pytest.mark.parametrize("cuts", [[140], [60, 1, 1, 1, 30, 2], []], ids=["prompt", "portions", "tokens"])


def only_left(w):
    w["l0.mix.right.o"] *= 0


def only_right(w):
    w["l0.mix.left.o"] *= 0


@BOTH
@ONE
@pytest.mark.parametrize("a", [dict(heads=2, kv_heads=2, dim=32, vdim=32, dims=32), dict(heads=20, kv_heads=2, dim=16, vdim=8, dims=8), dict(heads=3, kv_heads=1, dim=64, vdim=100, dims=24),
                               dict(heads=2, kv_heads=1, dim=134, vdim=48, dims=34), dict(heads=4, kv_heads=4, dim=128, vdim=65, dims=2), dict(heads=8, kv_heads=1, dim=192, vdim=128, dims=192),
                               dict(heads=5, kv_heads=1, dim=100, vdim=192, dims=0)], ids=str)
def test_attention_with_sharp_scores(env, cuts, f32, a):
    """Large scores, so that single keys stand out: one wrong, missing or extra key shows."""
    ctx, eng = env
    e = single(eng, ctx, (lm.sides(scale=3.0 * a["dim"] ** -0.5, softcap=30.0, base=200.0, **a), None), f32, cuts=cuts, change=only_left)
    assert e < (6e-5 if f32 else 0.1), e


@BOTH
@ONE
@pytest.mark.parametrize("softcap", [0.3, 2.0, 50.0])
def test_caps(env, cuts, f32, softcap):
    """Caps far below, near and far above the scores."""
    ctx, eng = env
    e = single(eng, ctx, (lm.sides(dim=64, vdim=64, dims=64, scale=0.7, softcap=softcap), None), f32, cuts=cuts, change=only_left)
    assert e < (6e-5 if f32 else 0.1), e


@BOTH
@ONE
@pytest.mark.parametrize("sign", [1.0, -1.0])
def test_the_sink_counts(env, cuts, f32, sign):
    """Strongly negative scores: the sink takes nearly everything, so leaving it out would change the output by a factor;
    positive ones: it takes next to nothing."""
    ctx, eng = env

    def change(w):
        only_left(w)
        for n in ("q", "k"):
            w[f"l0.mix.left.{n}"] *= 0.3
            w[f"l0.mix.left.{n}.b"][:] = 1.0 if n == "q" else sign

    layer = (lm.sides(dim=32, vdim=32, dims=0, scale=0.25, softcap=12.0), None)
    cfg = lm.tirezen([layer], width=64, vocab=70)
    w = lm.tirezen_weights(cfg, seed=2)
    change(w)
    h = np.random.default_rng(0).standard_normal((20, 64))
    g = lambda n: w["l0.mix.left." + n]
    with_sink = ref.sink_attention(h, g, layer[0][1]["left"], 1e-6)
    far = np.abs(with_sink).max()
    assert far < 0.5 if sign < 0 else far > 0.5  # the sink decides
    # with the sink's share the left mixer is small; it is scaled up so that it still dominates the logits
    if sign < 0:
        layer[0][1]["left_scale"] = 40.0
    e = single(eng, ctx, layer, f32, cuts=cuts, change=change)
    assert e < (1e-4 if f32 else 0.1), e


@BOTH
def test_key_far_away(env, f32):
    """Every query looks for one marked token among hundreds; moving the mark by one place must move the answer, in a prompt,
    in a later portion and when decoding, on both sides of page and tile borders."""
    ctx, eng = env
    cfg = lm.tirezen([(lm.sides(heads=4, kv_heads=2, dim=32, vdim=16, dims=8, scale=1.0, softcap=14.0, left_scale=1.0), None)], width=64, vocab=64)
    w = lm.tirezen_weights(cfg, seed=4)
    only_left(w)
    E = np.zeros((64, 64))
    E[:, :32] = np.random.default_rng(0).standard_normal((64, 32))
    E[:, 40] = 4.0                # what every token's query asks with
    E[7, 41] = 30.0               # the mark
    w["embed"] = E
    w["l0.norm1"] = np.zeros(64)
    w["l0.mix.left.q"] *= 0.1
    w["l0.mix.left.q"][20::32, 40] = 8.0   # coordinate 20 is not rotated
    w["l0.mix.left.k"] *= 0.3
    w["l0.mix.left.k"][20::32] = 0
    w["l0.mix.left.k"][20::32, 41] = 2.0
    w["l0.mix.left.k.b"] = 0.2 * np.ones(64)
    w["l0.mix.left.q.b"] *= 0.1
    w = {k: lm.round_bf16(v) for k, v in w.items()}
    model = lm.load(eng, ctx, cfg, w, f32)
    rng = np.random.default_rng(1)
    n = 420
    for page in (16, 48):
        pool = eng.BlockPool(ctx, model, page, -(-n // page), 1)
        for mark in (3, 15, 16, 127, 128):
            ids = rng.integers(8, 64, n).astype(np.int32)
            ids[mark] = 7
            want = ref.forward(cfg, w, ids)
            moved = ids.copy()
            moved[mark], moved[mark + 1] = ids[mark + 1], 7
            assert error(ref.forward(cfg, w, moved)[mark:mark + 1], want[mark:mark + 1]) > 0.2  # the mark decides
            for cuts in ([n], [200, 1, 2, 100], [mark + 1, 60, 2, 128, 1, 1, 1, 200]):
                e = error(run(eng, model, pool, ids, cuts), want)
                assert e < (1e-4 if f32 else 0.08), (page, mark, cuts, e)
        pool.free()
    model.free()


MEM_CUTS = pytest.mark.parametrize("cuts", [[140], [2] * 70, [64, 1, 63, 12], [11, 13, 65, 3], []], ids=["prompt", "twos", "portions", "short", "tokens"])


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("m", [dict(), dict(heads=1, dim=16, vdim=16, dims=16), dict(heads=2, dim=64, vdim=128, dims=32), dict(heads=2, dim=128, vdim=40, dims=128, base=70000.0),
                               dict(heads=4, dim=33, vdim=70, dims=0, decay=[1.0, 0.5, 0.001, 0.9990234375]), dict(heads=2, dim=250, vdim=24, dims=250)], ids=str)
def test_retention_alone(env, m, cuts, f32):
    ctx, eng = env
    e = single(eng, ctx, (lm.retention(**m), None), f32, cuts=cuts)
    assert e < TOL[f32], e


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("m", [dict(), dict(heads=1, kv_heads=1, dim=16, vdim=64, conv=1), dict(heads=4, kv_heads=1, dim=64, vdim=128, conv=4), dict(heads=2, kv_heads=2, dim=128, vdim=33, conv=3),
                               dict(heads=3, kv_heads=1, dim=37, vdim=70, conv=6), dict(heads=2, kv_heads=2, dim=256, vdim=16, conv=2)], ids=str)
@pytest.mark.parametrize("kind", ["head", "channel"])
def test_delta_alone(env, kind, m, cuts, f32):
    ctx, eng = env
    layer = lm.delta(**m) if kind == "head" else lm.sides(heads=1, kv_heads=1, dim=8, vdim=8, dims=8, right={**dict(heads=6, kv_heads=3, dim=28, vdim=12, conv=2), **m})
    e = single(eng, ctx, (layer, None), f32, cuts=cuts, change=None if kind == "head" else only_right)
    assert e < TOL[f32], e


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("A,dt,gain", [(3.0, 4.0, 1.0), (-7.0, -2.0, 1.0), (0.0, None, 1.0), (2.5, -1.0, 3.0)], ids=["forgets at once", "forgets nothing", "both", "now and then"])
@pytest.mark.parametrize("kind,dim", [("head", 40), ("channel", 40), ("channel", 104)])
def test_delta_decays(env, kind, dim, A, dt, gain, cuts, f32):
    """Exponents of minus hundreds per token, of nearly nothing, both in neighbouring channels (heads), and from token to token."""
    ctx, eng = env
    p = "l0.mix." if kind == "head" else "l0.mix.right."

    def change(w):
        w[p + "A_log"][:] = A
        w[p + "dt_bias"][:] = dt if dt is not None else np.where(np.arange(len(w[p + "dt_bias"])) % 2, 60.0, -9.0)
        w[p + ("a" if kind == "head" else "a2")] *= gain
        if kind == "channel":
            only_right(w)

    m = dict(heads=4, kv_heads=2, dim=dim, vdim=24, conv=3)
    layer = lm.delta(**m) if kind == "head" else lm.sides(heads=1, kv_heads=1, dim=8, vdim=8, dims=8, right=m)
    e = single(eng, ctx, (layer, None), f32, cuts=cuts, change=change)
    assert e < TOL[f32], e


@BOTH
@pytest.mark.parametrize("ranks", [(1, 1), (70, 33), (8, 130)], ids=str)
def test_ranks_come_from_the_tensors(env, ranks, f32):
    ctx, eng = env
    cfg = lm.tirezen([(lm.sides(right=dict(heads=2, kv_heads=1, dim=24, vdim=36)), None)], width=58, vocab=60)
    w = lm.tirezen_weights(cfg, seed=5, ranks=ranks)
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, 40, 3)
    want = ref.forward(cfg, w, ids)
    pool = eng.BlockPool(ctx, model, 16, 3, 1)
    for cuts in ([40], [13, 1, 2]):
        assert error(run(eng, model, pool, ids, cuts), want) < TOL[f32]
    pool.free()
    model.free()


@BOTH
def test_delta_overwrites_what_a_key_stored(env, f32):
    """The same few tokens over and over: every key returns with another value, step sizes near one and no decay, so that the
    correction by what the state already answers is all that keeps the state from growing."""
    ctx, eng = env
    cfg = lm.tirezen([(lm.delta(heads=2, kv_heads=1, dim=64, vdim=32, conv=1), None)], width=64, vocab=6)
    w = lm.tirezen_weights(cfg, seed=3)
    w["l0.mix.A_log"][:] = -9.0
    w["l0.mix.b"] *= 4.0
    w = {k: lm.round_bf16(v) for k, v in w.items()}
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, 300, 4)
    want = ref.forward(cfg, w, ids)
    pool = eng.BlockPool(ctx, model, 16, 19, 1)
    for cuts in ([300], [40, 100, 2, 2, 90], []):
        e = error(run(eng, model, pool, ids, cuts), want)
        assert e < TOL[f32], (cuts, e)
    pool.free()
    model.free()


@BOTH
@pytest.mark.parametrize("kind", ["retention", "head", "channel"])
def test_memory_over_a_long_sequence(env, kind, f32):
    """Slow decays: the state still carries the first tokens hundreds of steps later, across every kind of cut."""
    ctx, eng = env
    layer = {"retention": lm.retention(heads=2, dim=64, vdim=16, dims=64, decay=[0.99951171875, 1.0]), "head": lm.delta(heads=2, kv_heads=1, dim=64, vdim=16, conv=3),
             "channel": lm.sides(heads=1, kv_heads=1, dim=8, vdim=8, dims=8, right=dict(heads=2, kv_heads=1, dim=64, vdim=16, conv=3))}[kind]
    cfg = lm.tirezen([(layer, None)], width=64, vocab=60)
    w = lm.tirezen_weights(cfg, seed=6)
    for k in w:
        if k.endswith("A_log"):
            w[k][:] = -6.0
        if k.endswith("dt_bias"):
            w[k][:] = -1.0
    if kind == "channel":
        only_right(w)
    w = {k: lm.round_bf16(v) for k, v in w.items()}
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, 520, 1)
    other = ids.copy()
    other[:4] = (other[:4] + 1) % 60
    want = ref.forward(cfg, w, ids)
    assert error(ref.forward(cfg, w, other)[-1:], want[-1:]) > 1e-3  # the first tokens still matter at the end
    pool = eng.BlockPool(ctx, model, 16, 33, 2)
    for cuts in ([520], [300] + [1] * 50 + [2, 3, 100], [400]):
        e = error(run(eng, model, pool, ids, cuts), want)
        assert e < TOL[f32], (cuts, e)
    pool.free()
    model.free()


@BOTH
@pytest.mark.parametrize("n,cuts", [(90, [90]), (9, [])], ids=["prompt", "tokens"])
@pytest.mark.parametrize("ff", [8, 100, 300])
def test_feed_forward_alone(env, ff, n, cuts, f32):
    """The mixer's output projection is zero, so only the feed-forward adds to the stream."""
    ctx, eng = env

    def change(w):
        w["l0.mix.o"] *= 0

    e = single(eng, ctx, (lm.retention(heads=1), lm.dense(ff)), f32, n=n, cuts=cuts, change=change, gain={"up": 3.0})
    assert e < TOL[f32], e


@BOTH
@pytest.mark.parametrize("loop", [(0, 1, 1), (0, 1, 5), (0, 2, 2), (1, 2, 3), (1, 3, 1), (2, 3, 2)], ids=str)
def test_loops(env, loop, f32):
    """Each pass has its own cache and state, vector and share of the embedding output."""
    ctx, eng = env
    layers = [(lm.retention(), None), (lm.sides(), lm.dense(48)), (lm.delta(), None)]
    cfg = lm.tirezen(layers, vocab=50, loop=loop)
    w = lm.tirezen_weights(cfg, seed=8)
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, 50, 2)
    pool = eng.BlockPool(ctx, model, 16, 4, 1)
    want = ref.forward(cfg, w, ids)
    for cuts in ([50], [20, 1, 13, 2], []):
        e = error(run(eng, model, pool, ids, cuts), want)
        assert e < TOL[f32], (cuts, e)
    pool.free()
    model.free()


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


@pytest.mark.parametrize("name", ["tiles", "uneven"])
def test_long_contexts_are_split_over_keys(env, name):
    """Decoding several sequences with contexts of many chunks, alone and beside a portion: partial results are added up."""
    ctx, eng = env
    model, cfg, w = get_model(env, name, False)
    n = 700
    ids = tokens(cfg, n, 0)
    full = want_logits(name, cfg, w, n)
    pool = eng.BlockPool(ctx, model, 16, 160, 5, 60)
    caches, lens = [eng.PagedKvCache(pool) for _ in range(4)], [690, 130, 517, 200]
    model.step_at([(ids[:k], c) for k, c in zip(lens, caches)], [[] for _ in lens])
    extra = eng.PagedKvCache(pool)
    for s in range(6):
        got, _ = model.step_at([(ids[k + s:k + s + 1], c) for k, c in zip(lens, caches)] + [(ids[s * 40:s * 40 + 40], extra)], [[0]] * 4 + [[39]])
        assert error(got, full[[k + s for k in lens] + [s * 40 + 39]]) < TOL[False]
    for c in caches + [extra]:
        c.free()
    pool.free()


def test_caches(env):
    """Fork copies pages and states of every run; the prefix cache reuses a stored sequence only where its state is."""
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
    got, _ = model.step_at([(ids[:50], a)], [[49]])
    assert error(got, full[[49]]) < TOL[True]
    a.free()
    b.free()
    pool.free()


def test_shapes_that_do_not_fit_are_refused(env):
    from mlx_llm_b200._lib import B2Error

    ctx, eng = env
    cfg = lm.TIREZEN["odd"]
    w = lm.tirezen_weights(cfg)
    for key, new in (("l0.mix.right.a2", (3, 7)), ("head", (97, 50)), ("l1.mix.k.conv", (9, 4)), ("loop.step", (1, 53))):
        bad = copy.copy(w)
        bad[key] = np.zeros(new)
        with pytest.raises(B2Error) as e:
            lm.load(eng, ctx, cfg, bad, True)
        assert e.value.code == -4 and key in str(e.value)
    bad = copy.copy(w)
    bad.pop("l2.mix.g")
    with pytest.raises(B2Error) as e:
        lm.load(eng, ctx, cfg, bad, True)
    assert "l2.mix.g" in str(e.value)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(env, tmp_path, dtype):
    cfg = lm.TIREZEN["all_kinds"]
    w = lm.tirezen_weights(cfg, seed=11)
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
