"""Layered models (latent attention, Mamba-2, routed and dense feed-forwards) through the engine against the plain
restatement in oracle/layered.py, in f32 (tight) and in the serving format (bf16 products, f32 residual / scores / state).

The measure of a logits row is the rms of its error over the rms spread of the model's logits."""
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
# f32: rounding of a few hundred-term sums through at most four layers.  bf16: activations and weights-times-activations
# rounded to 8 bits between the steps; what a misplaced key, a lost state or a wrong expert does is 10 to 100 times that.
TOL = {True: 2e-5, False: 4e-2}


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
        cfg = lm.CASES[name]
        w = lm.weights(cfg, seed=len(name))
        _models[name, f32] = (lm.load(eng, ctx, cfg, w, f32), cfg, w)
    return _models[name, f32]


def want_logits(name, cfg, w, n, seed=0):
    """Oracle logits [n, vocab] of the test sequence (a prefix of a longer one is the same, so compute it once)."""
    key = (name, seed)
    if key not in _refs or len(_refs[key]) < n:
        _refs[key] = ref.forward(cfg, w, tokens(cfg, n, seed))
    return _refs[key][:n]


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("name", list(lm.CASES))
def test_whole_prompt(env, name, f32):
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    n = 150
    pool = eng.BlockPool(ctx, model, 16, 16, 1)
    got = run(eng, model, pool, tokens(cfg, n, 0), [n])
    e = error(got, want_logits(name, cfg, w, n))
    pool.free()
    assert e < TOL[f32], e


@pytest.mark.parametrize("f32", [True, False])
def test_residual_after_every_layer(env, f32):
    ctx, eng = env
    model, cfg, w = get_model(env, "mixed", f32)
    ids = tokens(cfg, 40, 5)
    layers = []
    ref.forward(cfg, w, ids, layers)
    buf = np.zeros((len(layers), len(ids), cfg["width"]), np.float32)
    model.capture_residual(buf)
    pool = eng.BlockPool(ctx, model, 16, 4, 1)
    run(eng, model, pool, ids, [40])
    model.capture_residual(None)
    pool.free()
    for i, x in enumerate(layers):
        assert np.abs(buf[i] - x).max() < (1e-4 if f32 else 0.15), i


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("name", list(lm.CASES))
@pytest.mark.parametrize("cuts", [[], [2] * 80, [3, 1, 2, 14, 1, 1, 17, 16, 2, 33, 5], [15, 2, 31, 1, 64]], ids=["tokens", "twos", "mixed", "borders"])
def test_portions_and_single_tokens(env, name, f32, cuts):
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    n = 118
    pool = eng.BlockPool(ctx, model, 16, 8, 1)
    got = run(eng, model, pool, tokens(cfg, n, 0), cuts)
    e = error(got, want_logits(name, cfg, w, 150)[:n])
    pool.free()
    assert e < TOL[f32], e


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("name", ["mixed", "recurrent_first", "wide_heads", "big_state"])
def test_mixed_batches_with_reused_pages_and_slots(env, name, f32):
    """Portions beside single tokens in one step, requests that pause, end and hand their pages and slots on; the pool
    is as small as the schedule allows, so everything is used again."""
    ctx, eng = env
    model, cfg, w = get_model(env, name, f32)
    pool = eng.BlockPool(ctx, model, 16, 20, 3, 20)
    rng = np.random.default_rng(3)
    todo = [(i, tokens(cfg, n, 0)[:n]) for i, n in enumerate([90, 33, 1, 118, 47, 2, 64, 101])]
    live, worst = {}, 0.0
    while todo or live:
        while todo and len(live) < 3 and sum(-(-len(v[0]) // 16) for v in live.values()) + -(-len(todo[0][1]) // 16) <= 20:
            i, ids = todo.pop(0)
            live[i] = [ids, eng.PagedKvCache(pool), 0]
        step, wants, meta = [], [], []
        for i, (ids, c, at) in live.items():
            if len(live) > 1 and rng.random() < 0.2 and step:
                continue  # sits this step out
            n = min(int(rng.choice([1, 1, 2, 5, 16, 40])), len(ids) - at)
            want = sorted({int(x) for x in rng.integers(0, n, 3)} | {n - 1})
            step.append((ids[at:at + n], c))
            wants.append(want)
            meta.append((i, at, n, want))
        got, _ = model.step_at(step, wants)
        row = 0
        full = want_logits(name, cfg, w, 150)
        for i, at, n, want in meta:
            worst = max(worst, error(np.concatenate([got[row:row + len(want)], full]), np.concatenate([full[[at + x for x in want]], full])))
            row += len(want)
            live[i][2] = at + n
            if live[i][2] == len(live[i][0]):
                live.pop(i)[1].free()
    assert pool.stats()["free_pages"] == 20
    pool.free()
    assert worst < TOL[f32], worst


def single(eng, ctx, layer, f32, gain=None, n=140, cuts=None, seed=2, width=64, vocab=70, zero=()):
    cfg = lm.config([layer], width=width, vocab=vocab)
    w = lm.weights(cfg, seed=seed, gain=gain)
    for k in zero:
        w[k] = np.zeros_like(w[k])
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, n, 9)
    pool = eng.BlockPool(ctx, model, 16, -(-n // 16), 1)
    got = run(eng, model, pool, ids, cuts or [n])
    e = error(got, ref.forward(cfg, w, ids))
    pool.free()
    model.free()
    return e


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("cuts", [[140], [60, 1, 1, 1, 30, 2], []], ids=["prompt", "portions", "tokens"])
@pytest.mark.parametrize("heads,dims", [(2, dict(dim=32, rot_dim=32, vdim=32)), (20, dict(dim=16, rot_dim=8, vdim=8)), (3, dict(dim=40, rot_dim=24, vdim=100)),
                                        (2, dict(dim=100, rot_dim=34, vdim=48)), (1, dict(dim=56, rot_dim=72, vdim=65)), (40, dict(dim=8, rot_dim=4, vdim=6))])
def test_latent_attention_with_sharp_scores(env, cuts, f32, heads, dims):
    """Queries and keys scaled so that single keys stand out: one wrong, missing or extra key shows."""
    ctx, eng = env
    gain = {".q": 4.0}
    e = single(eng, ctx, (lm.latent(heads=heads, kv_rank=64, base=200.0, **dims), None), f32, gain=gain, cuts=cuts)
    assert e < (5e-5 if f32 else 0.1), e


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("rank", [9, 130, 448, 520])
def test_latent_sizes(env, rank, f32):
    """Ranks of one to several value blocks, and one beyond the tensor-core decode kernel's reach."""
    ctx, eng = env
    e = single(eng, ctx, (lm.latent(heads=3, dim=32, rot_dim=16, vdim=24, kv_rank=rank), None), f32, n=150, cuts=[100, 1, 1, 30, 2])
    assert e < TOL[f32], e


@pytest.mark.parametrize("f32", [True, False])
def test_key_far_away(env, f32):
    """Every query looks for one marked token (position 3) among hundreds; moving the mark by one place must move the
    answer, in a prompt, in a later portion and when decoding, on both sides of page and tile borders."""
    ctx, eng = env
    cfg = lm.config([(lm.latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=32), None)], width=64, vocab=64)
    w = lm.weights(cfg, seed=4)
    E = np.zeros((64, 64))
    E[:, :32] = np.random.default_rng(0).standard_normal((64, 32))
    E[:, 40] = 4.0                # what every token's query asks with
    E[7, 41] = 30.0               # the mark
    w["embed"] = lm.round_bf16(E)
    w["l0.norm1"] = np.ones(64)
    w["l0.mix.q"] *= 0.1
    w["l0.mix.q"][[0, 24], 40] = 8.0
    w["l0.mix.dkv"][0] = 0
    w["l0.mix.dkv"][0, 41] = 2.0  # latent 0 is the mark
    w["l0.mix.dkv"][1:32] *= 0.3
    w["l0.mix.uk"] *= 0.1
    w["l0.mix.uk"][[0, 16], 0] = 3.0
    w = {k: lm.round_bf16(v) for k, v in w.items()}
    model = lm.load(eng, ctx, cfg, w, f32)
    rng = np.random.default_rng(1)
    n = 420
    pool = eng.BlockPool(ctx, model, 16, -(-n // 16), 1)
    seen = []
    for mark in (3, 15, 16, 127, 128):
        ids = rng.integers(8, 64, n).astype(np.int32)
        ids[mark] = 7
        want = ref.forward(cfg, w, ids)
        moved = ids.copy()
        moved[mark], moved[mark + 1] = ids[mark + 1], 7
        assert error(ref.forward(cfg, w, moved)[mark:mark + 1], want[mark:mark + 1]) > 0.2  # the mark decides
        for cuts in ([n], [200, 1, 2, 100], [mark + 1, 60, 2, 128, 1, 1, 1, 200]):
            assert error(run(eng, model, pool, ids, cuts), want) < (5e-5 if f32 else 0.08)
        seen.append(want[-1])
    pool.free()
    model.free()


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("cuts", [[140], [2] * 70, [64, 1, 63], []], ids=["prompt", "twos", "portions", "tokens"])
@pytest.mark.parametrize("m", [dict(), dict(heads=3, groups=1, vdim=17, state=33, conv=2, norm_groups=3), dict(heads=8, groups=8, vdim=16, state=16, conv=6, norm_groups=1),
                               dict(heads=3, groups=3, vdim=80, state=64, conv=1, norm_groups=3),
                               dict(heads=2, groups=1, vdim=64, state=128, conv=4, norm_groups=1)])
def test_mamba2_alone(env, m, cuts, f32):
    ctx, eng = env
    e = single(eng, ctx, (lm.mamba(**m), None), f32, cuts=cuts)
    assert e < TOL[f32], e


@pytest.mark.parametrize("f32", [True, False])
def test_mamba2_remembers_over_a_long_sequence(env, f32):
    """Slow decays: the state still carries the first tokens hundreds of steps later, across every kind of cut."""
    ctx, eng = env
    cfg = lm.config([(lm.mamba(heads=2, vdim=16, state=32, groups=1, norm_groups=1, conv=4), None)], width=64, vocab=60)
    w = lm.weights(cfg, seed=6)
    w["l0.mix.A_log"] = lm.round_bf16(np.array([-6.0, -5.0]))
    w["l0.mix.dt_bias"] = lm.round_bf16(np.array([-1.0, -2.0]))
    model = lm.load(eng, ctx, cfg, w, f32)
    ids = tokens(cfg, 520, 1)
    other = ids.copy()
    other[:4] = (other[:4] + 1) % 60
    want = ref.forward(cfg, w, ids)
    assert error(ref.forward(cfg, w, other)[-1:], want[-1:]) > 1e-3  # the first tokens still matter at the end
    pool = eng.BlockPool(ctx, model, 16, 33, 2)
    for cuts in ([520], [300] + [1] * 50 + [2, 3, 100], [400]):
        assert error(run(eng, model, pool, ids, cuts), want) < TOL[f32]
    pool.free()
    model.free()


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("mlp,gain", [(lm.dense(100), None), (lm.moe(experts=6, top=1, ff=48, limit=0.6), {"gate": 3.0, "up": 3.0}),
                                      (lm.moe(experts=6, top=6, ff=33, limit=1.5), {"gate": 3.0, "up": 3.0}),
                                      (lm.moe(experts=40, top=5, ff=64, limit=7.0), None), (lm.moe(experts=1, top=1, ff=24, limit=0.3), None)])
@pytest.mark.parametrize("n,cuts", [(90, [90]), (9, [])], ids=["prompt", "tokens"])
def test_feed_forward_alone(env, mlp, gain, n, cuts, f32):
    """The mixer's output projection is zero, so only the feed-forward adds to the stream (limits bind on both sides)."""
    ctx, eng = env
    e = single(eng, ctx, (lm.latent(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8), mlp), f32, gain=gain, n=n, cuts=cuts, zero=("l0.mix.o",))
    assert e < TOL[f32], e


def greedy(cfg, w, prompt, n):
    ids = list(prompt)
    margins = []
    for _ in range(n):
        lg = ref.forward(cfg, w, ids)[-1]
        a = np.sort(lg)
        margins.append(a[-1] - a[-2])
        ids.append(int(np.argmax(lg)))
    return ids[len(prompt):], margins


@pytest.mark.parametrize("name", ["mixed", "recurrent_first"])
def test_greedy_generation_through_the_scheduler(env, name):
    """generate, generate_continuous (exact, throughput, chunked, more requests than lanes) and the serving form."""
    ctx, eng = env
    model, cfg, w = get_model(env, name, True)
    prompts = [tokens(cfg, n, 20 + n) for n in (1, 5, 21, 34, 16)]
    want = []
    for p in prompts:
        t, margins = greedy(cfg, w, p, 8)
        cut = next((i for i, m in enumerate(margins) if m < 1e-3), 8)  # beyond a near-tie nothing is decided
        want.append(t[:cut])
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


def test_serving_format_generates_like_itself(env):
    """bf16: the batched, chunked loop gives the single-sequence loop's tokens up to near-ties."""
    ctx, eng = env
    model, cfg, w = get_model(env, "mixed", False)
    prompts = [tokens(cfg, n, 40 + n) for n in (3, 18, 50)]
    alone = [eng.generate(model, p, 12).tokens for p in prompts]
    outs = eng.generate_continuous(model, [eng.BatchRequest(p, 12) for p in prompts],
                                   eng.ContinuousConfig(max_batch=3, block_size=16, exactness=eng.THROUGHPUT, prefill_chunk_tokens=16))
    same = sum(o.tokens[0] == a[0] for o, a in zip(outs, alone))
    assert same == 3 and all(len(o.tokens) == 12 for o in outs)


def test_long_decoding(env):
    ctx, eng = env
    model, cfg, w = get_model(env, "mixed", False)
    n = 400
    ids = tokens(cfg, n, 0)
    pool = eng.BlockPool(ctx, model, 16, 25, 1)
    got = run(eng, model, pool, ids, [20])
    e = error(got, want_logits("mixed", cfg, w, n))
    pool.free()
    assert e < TOL[False], e


def test_long_contexts_are_split_over_keys(env):
    """Decoding several sequences with contexts of many chunks: partial results are added up."""
    ctx, eng = env
    model, cfg, w = get_model(env, "wide_heads", False)
    n = 700
    ids = tokens(cfg, n, 0)
    full = want_logits("wide_heads", cfg, w, n)
    pool = eng.BlockPool(ctx, model, 16, 140, 4, 60)
    caches, lens = [eng.PagedKvCache(pool) for _ in range(4)], [690, 130, 517, 200]
    model.step_at([(ids[:k], c) for k, c in zip(lens, caches)], [[] for _ in lens])
    for s in range(6):
        got, _ = model.step_at([(ids[k + s:k + s + 1], c) for k, c in zip(lens, caches)], [[0]] * 4)
        assert error(got, full[[k + s for k in lens]]) < TOL[False]
    for c in caches:
        c.free()
    pool.free()


def test_caches_of_recurrent_models(env):
    """Fork at the end copies pages and state; earlier positions, shared blocks and roll-backs are refused; the prefix
    cache reuses a stored sequence only where its state is."""
    from mlx_llm_b200._lib import B2Error

    ctx, eng = env
    model, cfg, w = get_model(env, "mixed", True)
    assert model.state_bytes() > 0
    ids = tokens(cfg, 60, 0)
    full = want_logits("mixed", cfg, w, 150)
    pool = eng.BlockPool(ctx, model, 16, 12, 3)
    a = eng.PagedKvCache(pool)
    model.step_at([(ids[:37], a)], [[]])
    b = a.fork(37)
    got, _ = model.step_at([(ids[37:40], a), (ids[37:38], b)], [[2], [0]])
    assert error(got, full[[39, 37]]) < TOL[True]
    got, _ = model.step_at([(ids[38:60], b)], [[21]])
    assert error(got, full[[59]]) < TOL[True]
    for bad in (lambda: a.fork(20), lambda: a.truncate(20), lambda: eng.PagedKvCache.new_seeded(pool, a.block_ids()[:1])):
        with pytest.raises(B2Error) as e:
            bad()
        assert e.value.code == -5
    a.reset()
    got, _ = model.step_at([(ids[:50], a)], [[49]])
    assert error(got, full[[49]]) < TOL[True]
    a.free()
    b.free()
    pool.free()
    with pytest.raises(B2Error) as e:
        eng.generate_prompt_lookup(model, ids[:10], 4)
    assert e.value.code == -5
    pc = eng.PrefixCache(ctx, model, 2)
    one = eng.generate_cached(model, ids[:20], 4, pc).tokens
    assert one == eng.generate(model, ids[:20], 4).tokens
    longer = list(ids[:20]) + one[:3] + [5, 6]  # continues exactly where the stored sequence's state is
    assert eng.generate_cached(model, longer, 4, pc).tokens == eng.generate(model, longer, 4).tokens
    assert pc.stats()["hits"] == 1
    assert eng.generate_cached(model, ids[:12], 4, pc).tokens == eng.generate(model, ids[:12], 4).tokens
    assert pc.stats()["hits"] == 1
    pc.free()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(env, tmp_path, dtype):
    cfg = lm.CASES["recurrent_first"]
    w = lm.weights(cfg, seed=11)
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


def test_flat_models_through_the_registry(env, tmp_path):
    """A Llama-style folder opens through the same entry point, and listed positions work there too."""
    from tests import helpers as H

    ctx, eng = env
    cfg0 = H.CONFIG0
    tw = H.tiny_weights()
    ws = eng.Weights()
    ones = lambda n: np.ones(n, np.float32)
    ws.add("model.embed_tokens.weight", tw["embed"])
    ws.add("lm_head.weight", tw["lm_head"])
    ws.add("model.norm.weight", ones(cfg0["hidden"]))
    for l, lw in enumerate(tw["layers"]):
        for k, key in dict(q="self_attn.q_proj", k="self_attn.k_proj", v="self_attn.v_proj", o="self_attn.o_proj", gate="mlp.gate_proj",
                           up="mlp.up_proj", down="mlp.down_proj").items():
            ws.add(f"model.layers.{l}.{key}.weight", lw[k])
        ws.add(f"model.layers.{l}.input_layernorm.weight", ones(cfg0["hidden"]))
        ws.add(f"model.layers.{l}.post_attention_layernorm.weight", ones(cfg0["hidden"]))
    js = dict(model_type="llama", hidden_size=256, num_attention_heads=4, num_key_value_heads=2, head_dim=64, num_hidden_layers=2, intermediate_size=688,
              vocab_size=1024, rope_theta=10000.0)
    a = eng.CausalLm.from_json(ctx, ws, js)
    b = eng.CausalLm.from_weights(ctx, ws, "", eng.model_config_from_json(js))
    ids = H.config0_prompts()[1]
    pa, pb = eng.BlockPool(ctx, a, 16, 8, 1), eng.BlockPool(ctx, b, 16, 8, 1)
    ca, cb = eng.PagedKvCache(pa), eng.PagedKvCache(pb)
    rows, am = a.step_at([(ids, ca)], [[3, len(ids) - 1]])
    last, lam = b.step([(ids, cb)])
    assert not a.logits_f32() and np.array_equal(rows[1], H.bf16_to_f32_np(last[0])) and am[1] == lam[0]
    for x in (ca, cb, pa, pb, a, b, ws):
        x.free()
