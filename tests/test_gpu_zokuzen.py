"""Zokuzen models (time mixing with a bonus, windowed latent attention, chunked attention on own or shared keys, residual streams,
mixtures with identity and shared experts) through the engine against the plain restatement in oracle/layered.py, in f32 (tight)
and in the serving format (bf16 products; f32 residual, scores, routing, recurrences).

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
# the steps; what a misplaced key, a lost state or a wrong expert does is many times that.
TOL = {True: 3e-5, False: 4e-2}
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])
NAMES = list(lm.ZOKUZEN)
# (weights whose first tokens do not read out nearly nothing: the norm behind a memory would blow bf16 rounding up)
SEEDS = dict(all_kinds=10, odd=4, tiles=7, uneven=8, large_heads=12)


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
        cfg = lm.ZOKUZEN[name]
        w = lm.zokuzen_weights(cfg, seed=SEEDS[name])
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
def test_sum_of_the_streams_after_every_layer(env, name, f32):
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


def single(eng, ctx, layers, f32, n=140, cuts=None, seed=2, width=64, vocab=70, change=None, gain=None, streams=2, page=16, **kw):
    cfg = lm.zokuzen(layers if isinstance(layers, list) else [layers], width=width, vocab=vocab, streams=streams)
    w = lm.zokuzen_weights(cfg, seed=seed, gain=gain, **kw)
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


@BOTH
@ONE
@pytest.mark.parametrize("size", [1, 2, 16, 33, 128, 1000])
@pytest.mark.parametrize("a", [dict(heads=2, dim=32, vdim=32), dict(heads=20, dim=16, vdim=8), dict(heads=3, dim=40, vdim=100, kv_rank=130), dict(heads=1, dim=130, vdim=65, kv_rank=9),
                               dict(heads=40, dim=8, vdim=6), dict(heads=2, dim=192, vdim=128, kv_rank=520)], ids=str)
def test_windowed_latent_attention_with_sharp_scores(env, cuts, f32, a, size):
    """Queries scaled so that single keys stand out: one wrong, missing or extra key shows."""
    ctx, eng = env
    e = single(eng, ctx, (lm.window(size=size, **{**dict(kv_rank=64), **a}), None), f32, cuts=cuts, gain={".q": 4.0})
    assert e < (6e-5 if f32 else 0.1), e


@BOTH
@ONE
@pytest.mark.parametrize("size", [1, 2, 16, 33, 128, 1000])
@pytest.mark.parametrize("a", [dict(heads=2, kv_heads=2, dim=32, vdim=32, dims=32), dict(heads=20, kv_heads=2, dim=16, vdim=8, dims=8), dict(heads=3, kv_heads=1, dim=64, vdim=100, dims=24),
                               dict(heads=2, kv_heads=1, dim=134, vdim=48, dims=34), dict(heads=4, kv_heads=4, dim=128, vdim=65, dims=2), dict(heads=8, kv_heads=1, dim=192, vdim=128, dims=192),
                               dict(heads=5, kv_heads=1, dim=100, vdim=192, dims=0)], ids=str)
def test_chunked_attention_with_sharp_scores(env, cuts, f32, a, size):
    ctx, eng = env
    e = single(eng, ctx, (lm.chunk(size=size, scale=1.5 * a["dim"] ** -0.5, base=200.0, **a), None), f32, cuts=cuts)
    assert e < (6e-5 if f32 else 0.1), e


def marked(kind, size, kv_from=False):
    """A model whose queries all look for one marked token (7): the mark stands out by a score of ten and more."""
    if kind == "window":
        layers = [(lm.window(heads=2, dim=16, vdim=16, kv_rank=32, size=size), None)]
    else:
        a = dict(heads=4, kv_heads=2, dim=32, vdim=16, dims=8, scale=0.5)
        layers = [(lm.chunk(size=5 if kv_from else size, **a), None)] + ([(lm.chunk(size=size, kv_from=0, **a), None)] if kv_from else [])
    cfg = lm.zokuzen(layers, width=64, vocab=64, streams=2)
    w = lm.zokuzen_weights(cfg, seed=4)
    E = np.zeros((64, 64))
    E[:, :32] = np.random.default_rng(0).standard_normal((64, 32))
    E[:, 40] = 4.0                # what every token's query asks with
    E[7, 41] = 30.0               # the mark
    w["embed"] = E
    for i in range(len(layers)):
        p = f"l{i}.mix."
        w[f"l{i}.norm1"] = np.zeros(64)
        w[p + "o"][40:42] = 0     # (a second layer finds both again)
        w[p + "q"] *= 0.1
        if kind == "window":
            w[p + "q"][[0, 16], 40] = 8.0
            w[p + "dkv"] *= 0.3
            w[p + "dkv"][0] = 0
            w[p + "dkv"][0, 41] = 2.0  # latent 0 is the mark
            w[p + "uk"] *= 0.1
            w[p + "uk"][[0, 16], 0] = 3.0
        else:
            w[p + "q"][20::32, 40] = 8.0  # coordinate 20 is not rotated
            if p + "k" in w:
                w[p + "k"] *= 0.3
                w[p + "k"][20::32] = 0
                w[p + "k"][20::32, 41] = 2.0
    if kv_from:  # the first layer only provides the keys
        w["l0.mix.o"] *= 0
    return cfg, {k: lm.round_bf16(v) for k, v in w.items()}


@BOTH
@pytest.mark.parametrize("kind,kv_from", [("window", False), ("chunk", False), ("chunk", True)], ids=["window", "chunk", "shared keys"])
@pytest.mark.parametrize("size", [3, 16, 17, 50, 127, 128, 129, 300])
def test_edges_of_windows_and_chunks(env, kind, kv_from, size, f32):
    """The marked key lies just inside and just outside an edge: every position around it, in a prompt, in a later portion and
    when decoding, on pages of 16 and 48."""
    ctx, eng = env
    cfg, w = marked(kind, size, kv_from)
    model = lm.load(eng, ctx, cfg, w, f32)
    rng = np.random.default_rng(1)
    n = 420
    for page in (16, 48):
        pool = eng.BlockPool(ctx, model, page, -(-n // page), 1)
        for mark in ((3, 15, 64) if kind == "window" else (size - 1, size, 2 * size - 1)):
            edge = mark + size if kind == "window" else (mark // size + 1) * size  # the first position that does not see the mark
            if edge >= n:
                continue
            ids = rng.integers(8, 64, n).astype(np.int32)
            ids[mark] = 7
            want = ref.forward(cfg, w, ids)
            gone = ids.copy()
            gone[mark] = 9
            other = ref.forward(cfg, w, gone)
            assert edge - 1 == mark or error(other[edge - 1:edge], want[edge - 1:edge]) > 0.2  # it decides what the last one that sees it answers ...
            assert error(other[edge:edge + 1], want[edge:edge + 1]) < 1e-9                     # ... and nothing after that
            before = max(edge - 2, mark + 1)
            for cuts in ([n], [200, 1, 2, 100], [mark + 1, before - mark - 1] + [1] * 5 + [2, 128] if before > mark + 1 else [mark + 1] + [1] * 5 + [60, 2, 128]):
                e = error(run(eng, model, pool, ids, cuts), want)
                assert e < (1e-4 if f32 else 0.08), (page, mark, cuts, e)
        pool.free()
    model.free()


@BOTH
@pytest.mark.parametrize("kind,kv_from", [("window", False), ("chunk", False), ("chunk", True)], ids=["window", "chunk", "shared keys"])
def test_key_far_away(env, kind, kv_from, f32):
    """One marked token among hundreds; moving the mark by one place must move the answer."""
    ctx, eng = env
    cfg, w = marked(kind, 410, kv_from)
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
        assert error(ref.forward(cfg, w, moved)[mark:mark + 1], want[mark:mark + 1]) > 0.2
        for cuts in ([n], [200, 1, 2, 100], [mark + 1, 60, 2, 128, 1, 1, 1, 200]):
            e = error(run(eng, model, pool, ids, cuts), want)
            assert e < (1e-4 if f32 else 0.08), (mark, cuts, e)
    pool.free()
    model.free()


@BOTH
@ONE
def test_shared_keys_under_another_mask_and_scale(env, cuts, f32):
    """Two later layers read the first layer's keys with masks of their own, the last one across a layer that keeps none."""
    ctx, eng = env
    a = dict(heads=4, kv_heads=2, dim=24, vdim=16, dims=16)
    layers = [(lm.chunk(size=10, **a), None), (lm.chunk(size=70, kv_from=0, scale=0.6, **a), None), (lm.wkv(), None), (lm.chunk(size=33, kv_from=0, scale=0.1, **a), None),
              (lm.chunk(size=20, **a), None), (lm.chunk(size=90, kv_from=4, **{**a, "heads": 6}), None)]
    e = single(eng, ctx, layers, f32, cuts=cuts)
    assert e < (6e-5 if f32 else 0.06), e


MEM_CUTS = pytest.mark.parametrize("cuts", [[140], [2] * 70, [64, 1, 63, 12], [11, 13, 65, 3], []], ids=["prompt", "twos", "portions", "short", "tokens"])


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("m", [dict(), dict(heads=1, dim=16), dict(heads=2, dim=64), dict(heads=1, dim=128), dict(heads=3, dim=33), dict(heads=2, dim=104), dict(heads=4, dim=7), dict(heads=1, dim=230)],
                         ids=str)
def test_time_mixing_alone(env, m, cuts, f32):
    ctx, eng = env
    e = single(eng, ctx, (lm.wkv(**m), None), f32, cuts=cuts, seed=4)
    assert e < TOL[f32], e


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("dim", [20, 40, 104])
@pytest.mark.parametrize("w0,gain", [(5.0, 1.0), (12.0, 1.0), (-9.0, 1.0), (None, 1.0), (0.0, 6.0)], ids=["forgets at once", "exponents beyond f32", "forgets nothing", "both", "now and then"])
def test_decays_of_the_time_mixing(env, dim, w0, gain, cuts, f32):
    """Exponents of minus hundreds per token (and beyond what an exponential takes), of nearly nothing, both in neighbouring
    channels, and from token to token."""
    ctx, eng = env

    def change(w):
        v = w["l0.mix.w0"]
        v[:] = w0 if w0 is not None else np.where(np.arange(len(v)) % 2, 5.0, -9.0)
        w["l0.mix.w2"] *= gain

    e = single(eng, ctx, (lm.wkv(heads=2, dim=dim), None), f32, cuts=cuts, change=change)
    assert e < TOL[f32], e


@BOTH
@MEM_CUTS
@pytest.mark.parametrize("what", ["bonus", "state", "shift"])
def test_parts_of_the_time_mixing_decide(env, what, cuts, f32):
    """bonus: the current token's weight is large; state: it is zero, so the first token reads nothing; shift: every input is the
    token before's."""
    ctx, eng = env

    def change(w):
        if what == "shift":
            for n in "rkvgw":
                w["l0.mix.mu." + n][:] = 1.0
        else:
            w["l0.mix.u"][:] = 8.0 if what == "bonus" else 0.0

    e = single(eng, ctx, (lm.wkv(heads=2, dim=40), None), f32, cuts=cuts, change=change)
    assert e < TOL[f32], e


@BOTH
@pytest.mark.parametrize("rank", [1, 8, 70, 130])
def test_rank_comes_from_the_tensors(env, rank, f32):
    ctx, eng = env
    for cuts in ([40], [13, 1, 2]):
        assert single(eng, ctx, (lm.wkv(), None), f32, n=40, cuts=cuts, width=58, rank=rank) < TOL[f32]


@BOTH
def test_time_mixing_over_a_long_sequence(env, f32):
    """Slow decays: the state still carries the first tokens hundreds of steps later, across every kind of cut."""
    ctx, eng = env
    cfg = lm.zokuzen([(lm.wkv(heads=2, dim=32), None)], width=64, vocab=60)
    w = lm.zokuzen_weights(cfg, seed=6)
    w["l0.mix.w0"][:] = -8.0
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


def quiet_mixer(w):
    for k in w:
        if k.endswith(".mix.o"):
            w[k] *= 0


MIXTURES = [dict(), dict(experts=1, identity=0, top=1), dict(experts=2, identity=2, top=4), dict(experts=9, identity=5, top=6, ff=8, shared=200), dict(experts=4, identity=0, top=2, ff=100, shared=None),
            dict(experts=3, identity=70, top=2, scale=0.3), dict(experts=40, identity=8, top=8, ff=64, scale=2.5), dict(experts=4, identity=4, top=1, shared=None)]


@BOTH
@pytest.mark.parametrize("n,cuts", [(90, [90]), (200, [200]), (9, [])], ids=["prompt", "long", "tokens"])
@pytest.mark.parametrize("f", MIXTURES, ids=str)
def test_mixture_alone(env, f, n, cuts, f32):
    """The mixer's output projection is zero, so only the feed-forward adds to the streams."""
    ctx, eng = env
    e = single(eng, ctx, (lm.wkv(heads=1), lm.mixture(**f)), f32, n=n, cuts=cuts, change=quiet_mixer, gain={".up": 3.0})
    assert e < TOL[f32], e


@pytest.mark.parametrize("f", MIXTURES, ids=str)
def test_corrections_move_the_choice_only(env, f):
    """Corrections and scores of the same size (f32, where no choice here is a close call); the weights stay the scores'."""
    ctx, eng = env
    cfg = lm.zokuzen([(lm.wkv(heads=1), lm.mixture(**f))], width=64, vocab=70)
    w = lm.zokuzen_weights(cfg, seed=3, decide=False)
    ids = tokens(cfg, 60, 3)
    r = cfg["layers"][0]["mlp"]["router"]
    # the router's inputs, from the restatement
    gaps, real = [], ref.softmax_router

    def watch(z, corr, top, scale):
        s = np.exp(z - z.max(1, keepdims=True))
        c = np.sort(s / s.sum(1, keepdims=True) + corr, 1)[:, ::-1]
        if top < c.shape[1]:
            gaps.append((c[:, top - 1] - c[:, top]).min())
        moved.append((real(z, corr, top, scale) > 0) != (real(z, 0 * corr, top, scale) > 0))
        return real(z, corr, top, scale)

    moved = []
    ref.softmax_router = watch
    try:
        want = ref.forward(cfg, w, ids)
    finally:
        ref.softmax_router = real
    assert min(gaps, default=1.0) > 2e-5
    if r["top"] < r["experts"] + r["identity"]:
        assert moved[0].any()
    model = lm.load(eng, ctx, cfg, w, True)
    pool = eng.BlockPool(ctx, model, 16, 4, 1)
    for cuts in ([60], [20, 1, 2, 17]):
        assert error(run(eng, model, pool, ids, cuts), want) < TOL[True]
    pool.free()
    model.free()


@BOTH
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8, 11, 16])
@pytest.mark.parametrize("width", [64, 54, 57])
def test_streams(env, streams, width, f32):
    ctx, eng = env
    layers = [(lm.wkv(heads=2, dim=16), lm.mixture(ff=24, shared=16)), (lm.window(heads=2, dim=16, vdim=8), None), (lm.chunk(heads=2, kv_heads=1, dim=16, dims=8), lm.mixture(ff=16, identity=0))]

    def change(w):  # mixtures of the streams that are far from the identity, also negative ones
        rng = np.random.default_rng(5)
        for k in w:
            if k == "l1.hc1.mix":
                w[k] = rng.standard_normal(w[k].shape) / streams ** 0.5
            if k == "l1.hc1.in":
                w[k] = rng.standard_normal(w[k].shape)
        w["l2.hc2.in"] = 0 * w["l2.hc2.in"]  # a sub-layer that reads nothing: its norm sees zeros
        w["l2.mlp.correction"] = np.arange(len(w["l2.mlp.correction"])) * 1.0

    for cuts in ([50], [20, 1, 13, 2]):
        assert single(eng, ctx, layers, f32, n=50, cuts=cuts, width=width, streams=streams, change=change) < TOL[f32]


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
    """Batches on both sides of the sizes at which products and launches are merged differently: every sequence decodes one token."""
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
    """Windows and chunks of many work items, several sequences at different places of them, alone and beside a portion: partial
    results are added up."""
    ctx, eng = env
    cfg = lm.zokuzen([(lm.window(heads=18, dim=64, vdim=64, kv_rank=128, size=600), None), (lm.chunk(heads=6, kv_heads=2, dim=64, vdim=64, dims=64, size=650), None),
                      (lm.window(heads=3, dim=32, vdim=32, kv_rank=64, size=180), None), (lm.chunk(heads=20, kv_heads=1, dim=64, vdim=64, dims=64, size=333), None)], width=96, vocab=150)
    w = lm.zokuzen_weights(cfg, seed=1)
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
    """Fork copies pages, states and the shift's rows; a layer that reads another layer's keys has no pages of its own."""
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
    cfg = lm.ZOKUZEN["odd"]
    w = lm.zokuzen_weights(cfg)
    for key, new in (("l1.mix.w2", (13, 5)), ("l1.mix.u", (13,)), ("l0.mix.dkv", (20, 53)), ("l2.mix.k.norm", (9,)), ("l0.hc2.mix", (2, 2)), ("l0.mlp.correction", (3,)), ("l0.mlp.shared.sg", (2, 53))):
        bad = copy.copy(w)
        bad[key] = np.zeros(new)
        with pytest.raises(B2Error) as e:
            lm.load(eng, ctx, cfg, bad, True)
        assert e.value.code == -4 and key in str(e.value)
    bad = copy.copy(w)
    bad.pop("l1.mix.mu.w")
    with pytest.raises(B2Error) as e:
        lm.load(eng, ctx, cfg, bad, True)
    assert "l1.mix.mu.w" in str(e.value)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(env, tmp_path, dtype):
    cfg = lm.ZOKUZEN["all_kinds"]
    w = lm.zokuzen_weights(cfg, seed=11)
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
