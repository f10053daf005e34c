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
