"""Host-side checks of the layered models: the model registry and the reader of config.json, and the restatement the GPU
tests compare with (its mechanisms against independent formulations).  No GPU needed."""
import copy

import numpy as np
import pytest

from oracle import layered as ref
from tests import layered_models as lm


@pytest.fixture(scope="module")
def eng():
    from mlx_llm_b200 import build, engine

    build.build()
    return engine


def test_registry_names_the_family(eng):
    assert eng.model_family(lm.CASES["mixed"]) == "Zukitar"
    assert all(eng.model_family(c) == "Tirezen" for c in lm.TIREZEN.values())
    llama = dict(hidden_size=64, intermediate_size=128, num_hidden_layers=2, num_attention_heads=4, vocab_size=32)
    assert eng.model_family(llama) == "llama"


def test_registry_refuses_what_it_does_not_know(eng):
    from mlx_llm_b200._lib import B2Error

    def code(change):
        cfg = copy.deepcopy(lm.CASES["mixed"])
        change(cfg)
        with pytest.raises(B2Error) as e:
            eng.model_family(cfg)
        return e.value.code, str(e.value)

    assert code(lambda c: c.update(architecture="Other"))[0] == -5
    for change, word in ((lambda c: c.pop("logit_scale"), "logit_scale"), (lambda c: c["layers"][0].update(type="conv"), "conv"),
                         (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"), (lambda c: c["layers"][1]["mixer"].update(groups=3), "groups"),
                         (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "experts"), (lambda c: c["layers"][0]["mlp"].update(kind="x"), "kind"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot"), (lambda c: c.update(layers=[]), "layers"),
                         (lambda c: c["norm"].update(eps="small"), "eps")):
        rc, msg = code(change)
        assert rc == -4 and word in msg, msg


def test_latent_attention_absorbed_form_is_the_same():
    """Scores and outputs computed in latent coordinates equal the per-head form."""
    cfg = lm.config([(lm.latent(), None)])
    w = lm.weights(cfg, 1)
    m = cfg["layers"][0]["mixer"]
    h = np.random.default_rng(0).standard_normal((30, cfg["width"]))
    g = lambda n: w["l0.mix." + n]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(30.0)
    q = (h @ g("q").T).reshape(30, H, D + R)
    ck = h @ g("dkv").T
    c = ref.rms_norm(ck[:, :K], g("dkv.norm"), 3e-5)
    kr = ref.rotate_pairs(ck[:, K:], pos, m["rot"]["base"], R)
    out = np.zeros((30, H, V))
    for hd in range(H):
        ql = q[:, hd, :D] @ g("uk")[hd * D:(hd + 1) * D]
        qr = ref.rotate_pairs(q[:, hd, D:], pos, m["rot"]["base"], R)
        for t in range(30):
            s = (c[:t + 1] @ ql[t] + kr[:t + 1] @ qr[t]) * m["scale"]
            p = np.exp(s - s.max())
            out[t, hd] = g("uv")[hd * V:(hd + 1) * V] @ (p / p.sum() @ c[:t + 1])
    assert np.allclose(out.reshape(30, -1) @ g("o").T, ref.latent_attention(h, g, m, 3e-5))


def test_recurrence_equals_its_closed_form():
    """y_t = sum over s <= t of C_t . B_s  d_s  exp(-A sum of d over (s, t])  x_s  + D x_t."""
    rng = np.random.default_rng(2)
    T, H, P, G, N = 12, 4, 3, 2, 5
    x, B, C = rng.standard_normal((T, H, P)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, A_log, D = rng.random((T, H)), rng.standard_normal(H), rng.standard_normal(H)
    y = ref.ssd_recurrence(x, B, C, dt, A_log, D)
    for t in range(T):
        for h in range(H):
            want = D[h] * x[t, h]
            for s in range(t + 1):
                want = want + (C[t, h // 2] @ B[s, h // 2]) * dt[s, h] * np.exp(-np.exp(A_log[h]) * dt[s + 1:t + 1, h].sum()) * x[s, h]
            assert np.allclose(y[t, h], want)


def test_small_pieces():
    u, w, b = np.random.default_rng(0).standard_normal((6, 2)), np.array([[1.0, 2.0, 3.0], [0.0, 0.0, 1.0]]), np.array([0.5, 0.0])
    c = ref.causal_conv_silu(u, w, b)
    assert np.allclose(c[0, 0], ref.silu(3 * u[0, 0] + 0.5)) and np.allclose(c[4, 0], ref.silu(u[2, 0] + 2 * u[3, 0] + 3 * u[4, 0] + 0.5))
    assert np.allclose(c[:, 1], ref.silu(u[:, 1]))
    v = np.array([[[1.0, 0.0, 5.0]]])
    r = ref.rotate_pairs(v, np.array([1.0]), 100.0, 2)
    assert np.allclose(r, [[[np.cos(1.0), np.sin(1.0), 5.0]]])
    y = ref.gated_group_norm(np.ones((1, 4)), np.array([[1.0, 1.0, 2.0, 2.0]]), np.ones(4), 2, 0.0)
    assert np.allclose(y, 1.0)
    one = dict(router=dict(experts=2, top=1), expert=dict(ff=1, limit=0.5))
    W = {"router": np.array([[3.0], [-1.0]]), "e0.gate": np.array([[2.0]]), "e0.up": np.array([[-9.0]]), "e0.down": np.array([[1.0]]),
         "e1.gate": np.zeros((1, 1)), "e1.up": np.zeros((1, 1)), "e1.down": np.zeros((1, 1))}
    got = ref.routed_ff(np.array([[1.0]]), W.__getitem__, one)
    assert np.allclose(got, 0.5 / (1 + np.exp(-1.702 * 0.5)) * 0.5)  # gate cut at 0.5, up at -0.5


def test_tirezen_configurations_that_are_refused(eng):
    from mlx_llm_b200._lib import B2Error

    def sub(c, *path):
        for p in path:
            c = c[p]
        return c

    base = lm.TIREZEN["all_kinds"]
    for change, word in ((lambda c: c.pop("width"), "width"), (lambda c: sub(c, "layers", 0, "mixer", "decay").pop(), "decay"),
                         (lambda c: sub(c, "layers", 0, "mixer").update(decay=[0.5, 0.0, 0.5]), "decay"), (lambda c: sub(c, "layers", 2, "mixer").update(kv_heads=4), "kv_heads"),
                         (lambda c: sub(c, "layers", 1, "mixer", "left").update(kv_heads=3), "kv_heads"), (lambda c: sub(c, "layers", 1, "mixer", "left").pop("softcap"), "softcap"),
                         (lambda c: sub(c, "layers", 1, "mixer").pop("right"), "right"), (lambda c: sub(c, "layers", 1, "mixer").pop("left_scale"), "left_scale"),
                         (lambda c: sub(c, "layers", 0, "mixer", "rot").update(dims=22), "rot"), (lambda c: c["loop"].update(stop=5), "loop"), (lambda c: c["loop"].update(start=3), "loop"),
                         (lambda c: c["loop"].update(times=0), "times"), (lambda c: c["layers"][0].update(type="mamba2"), "mamba2"),
                         (lambda c: sub(c, "layers", 0, "mlp").update(kind="moe"), "kind")):
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(B2Error) as e:
            eng.model_family(cfg)
        assert e.value.code == -4 and word in str(e.value), str(e.value)


def test_delta_rule_solves_a_triangular_system():
    """The writes u of a stretch of tokens from a zero state: (I + A) u = beta v, A the decayed products of the keys."""
    rng = np.random.default_rng(5)
    T, D, V = 9, 4, 3
    q, k, v = rng.standard_normal((T, D)), rng.standard_normal((T, D)) * 0.5, rng.standard_normal((T, V))
    lg, beta = -rng.random((T, D)), rng.random(T)
    G = np.cumsum(lg, 0)
    pair = lambda a, t, s: (a[t] * np.exp(G[t] - G[s]) * k[s]).sum()
    A = np.array([[beta[t] * pair(k, t, s) if s < t else 0.0 for s in range(T)] for t in range(T)])
    u = np.linalg.solve(np.eye(T) + A, beta[:, None] * v)
    o = np.array([sum(pair(q, t, s) * u[s] for s in range(t + 1)) for t in range(T)])
    assert np.allclose(o, ref.decayed_memory(q, k, v, lg, beta))
    plain = np.array([sum(pair(q, t, s) * v[s] for s in range(t + 1)) for t in range(T)])
    assert np.allclose(plain, ref.decayed_memory(q, k, v, lg))


def test_pieces_of_the_capped_sink_attention():
    rng = np.random.default_rng(1)
    m = dict(heads=2, kv_heads=1, dim=4, vdim=3, rot=dict(base=10.0, dims=2), scale=0.5, softcap=1e6)
    w = dict(q=rng.standard_normal((8, 5)), k=rng.standard_normal((4, 5)), v=rng.standard_normal((3, 5)), o=np.eye(6))
    w.update({"q.b": rng.standard_normal(8), "k.b": rng.standard_normal(4), "v.b": rng.standard_normal(3), "q.norm": np.ones(4), "k.norm": np.ones(4)})
    h = rng.standard_normal((1, 5))
    out = ref.sink_attention(h, w.__getitem__, m, 0.0)[0]  # one token: weight exp(s) / (1 + exp(s)) on its own value
    v = w["v"] @ h[0] + w["v.b"]
    k = ref.rms(w["k"] @ h[0] + w["k.b"], 0.0)
    for i in range(2):
        q = ref.rms((w["q"] @ h[0] + w["q.b"])[4 * i:4 * i + 4], 0.0)
        assert np.allclose(out[3 * i:3 * i + 3], ref.sigmoid(0.5 * q @ k) * v)
    capped = ref.sink_attention(h, w.__getitem__, dict(m, softcap=1e-9), 0.0)[0]
    assert np.allclose(capped, np.concatenate([v, v]) / 2)
    r = ref.rotate_halves(np.array([[[1.0, 9.0, 0.0, 8.0, 5.0]]]), np.array([1.0]), 100.0, 4)
    a = 1.0 * 100.0 ** -0.5
    assert np.allclose(r, [[[np.cos(1.0), 9 * np.cos(a) - 8 * np.sin(a), np.sin(1.0), 8 * np.cos(a) + 9 * np.sin(a), 5.0]]])
    assert np.allclose(ref.gelu_erf(np.array([0.0, 1.0])), [0.0, 0.8413447460685429])


def test_layer_runs():
    cfg = dict(layers=[0] * 4, loop=dict(start=1, stop=3, times=2))
    assert ref.layer_runs(cfg) == [(0, -1), (1, 0), (2, 0), (1, 1), (2, 1), (3, -1)]
    assert ref.layer_runs(dict(layers=[0] * 2)) == [(0, -1), (1, -1)]


def test_zokuzen_configurations_that_are_refused(eng):
    from mlx_llm_b200._lib import B2Error

    assert all(eng.model_family(c) == "Zokuzen" for c in lm.ZOKUZEN.values())
    base = lm.ZOKUZEN["all_kinds"]
    mixer = lambda c, i: c["layers"][i]["mixer"]
    for change, word in ((lambda c: c.pop("streams"), "streams"), (lambda c: c.update(streams=0), "streams"), (lambda c: mixer(c, 1).pop("mask"), "mask"),
                         (lambda c: mixer(c, 1)["mask"].update(size=0), "size"), (lambda c: mixer(c, 1).pop("kv_rank"), "kv_rank"), (lambda c: mixer(c, 2).update(kv_heads=3), "kv_heads"),
                         (lambda c: mixer(c, 2)["rot"].update(dims=26), "rot"), (lambda c: mixer(c, 4).update(kv_from=4), "kv_from"), (lambda c: mixer(c, 4).update(kv_from=1), "kv_from"),
                         (lambda c: mixer(c, 5).update(kv_from=4), "kv_from"), (lambda c: mixer(c, 4).update(vdim=8), "kv_from"), (lambda c: c["layers"][0].update(type="retention"), "retention"),
                         (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "experts"), (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "scale"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind")):
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(B2Error) as e:
            eng.model_family(cfg)
        assert e.value.code == -4 and word in str(e.value), str(e.value)


def test_bonus_memory_equals_its_closed_form():
    """o_t = sum over s < t of (r_t . (decay over (s, t)) k_s) v_s, plus (r_t . u k_t) v_t."""
    rng = np.random.default_rng(7)
    T, D = 9, 4
    r, k, v, u = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal(D)
    w = rng.random((T, D))
    want = np.array([sum((r[t] * w[s + 1:t].prod(0) * k[s]).sum() * v[s] for s in range(t)) + (r[t] * u * k[t]).sum() * v[t] for t in range(T)])
    assert np.allclose(want, ref.bonus_memory(r, k, v, w, u))
    assert np.allclose(ref.shifted(np.array([[1.0], [2.0], [3.0]])), [[0.0], [1.0], [2.0]])


def test_masks():
    win, ch = ref.in_window(7, 3), ref.in_chunk(7, 3)
    assert [list(np.nonzero(r)[0]) for r in win] == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4], [3, 4, 5], [4, 5, 6]]
    assert [list(np.nonzero(r)[0]) for r in ch] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]


def test_pieces_of_the_mixture():
    z, c = np.log(np.array([[1.0, 2.0, 3.0, 4.0]])), np.array([0.0, 5.0, 0.0, 0.0])
    assert np.allclose(ref.softmax_router(z, 0 * c, 2, 1.0), [[0, 0, 3 / 7, 4 / 7]])
    assert np.allclose(ref.softmax_router(z, c, 2, 3.0), [[0, 3 * 2 / 6, 0, 3 * 4 / 6]])  # the correction chooses, the score weighs
    # nothing but identity experts: the input times the scale
    w = {"router": np.zeros((3, 2)), "correction": np.array([0.0, 1.0, 2.0])}
    h = np.array([[1.0, -2.0]])
    assert np.allclose(ref.mixture(h, w.__getitem__, dict(router=dict(experts=1, identity=2, top=2, scale=0.5))), 0.5 * h)


def test_connected_streams():
    X = np.array([[[1.0], [10.0]]])
    w = {"in": np.array([2.0, 3.0]), "mix": np.array([[1.0, 5.0], [7.0, 0.0]]), "out": np.array([100.0, 1000.0])}
    out = ref.connect(X, w, "", lambda u: u)  # reads 2 * 1 + 3 * 10
    assert np.allclose(out, [[[1 + 70 + 3200], [5 + 32000]]])


def test_pokadra_configurations_that_are_refused(eng):
    from mlx_llm_b200._lib import B2Error

    assert all(eng.model_family(c) == "Pokadra" for c in lm.POKADRA.values())
    base = lm.POKADRA["all_kinds"]
    mixer = lambda c, i: c["layers"][i]["mixer"]
    for change, word in ((lambda c: c.pop("residual_mult"), "residual_mult"), (lambda c: c["norm"].update(groups=5), "groups"), (lambda c: c["norm"].pop("groups"), "groups"),
                         (lambda c: c.pop("embedding"), "embedding"), (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"), (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
                         (lambda c: c["token_side"].update(dim=0), "dim"), (lambda c: mixer(c, 0).pop("diff"), "diff"), (lambda c: mixer(c, 0)["mask"].update(size=0), "size"),
                         (lambda c: mixer(c, 0)["mask"].update(keep_first=-1), "keep_first"), (lambda c: mixer(c, 0).update(kv_heads=3), "kv_heads"), (lambda c: mixer(c, 0)["rot"].update(dims=26), "rot"),
                         (lambda c: mixer(c, 0)["rot"]["scaling"].pop("slow"), "slow"), (lambda c: mixer(c, 0)["rot"]["scaling"].update(factor=0), "scaling"), (lambda c: mixer(c, 2).update(kv_from=1), "kv_from"),
                         (lambda c: mixer(c, 2).update(kv_from=2), "kv_from"), (lambda c: mixer(c, 5).update(kv_from=2), "kv_from"), (lambda c: mixer(c, 5).update(dim=16), "kv_from"),
                         (lambda c: mixer(c, 1).pop("width"), "width"), (lambda c: c["layers"][1].update(type="delta"), "delta"), (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind")):
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(B2Error) as e:
            eng.model_family(cfg)
        assert e.value.code == -4 and word in str(e.value), str(e.value)


def test_window_that_keeps_the_first_tokens():
    seen = [list(np.nonzero(r)[0]) for r in ref.in_window_or_first(7, 2, 3)]
    assert seen == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 2, 3, 4], [0, 1, 2, 4, 5], [0, 1, 2, 5, 6]]


def test_scaled_frequencies():
    rot = dict(base=100.0, dims=8)
    plain, m = ref.yarn_frequencies(rot)
    assert m == 1.0 and np.allclose(plain, [1.0, 100 ** -0.25, 0.1, 100 ** -0.75])
    # a pair whose frequency is f makes original * f / (2 pi) turns: 20, 6.32, 2, 0.63
    s = dict(factor=4.0, original=20 * 2 * np.pi, fast=20.0, slow=0.5)
    f, m = ref.yarn_frequencies(dict(rot, scaling=s))
    assert np.isclose(m, 1 + 0.1 * np.log(4.0))
    assert np.allclose(f / plain, [1.0, 1 - 0.75 / 4, 1 - 0.75 / 2, 1 - 0.75 * 3 / 4])  # the ramp goes from pair 0 to pair 3.2 rounded up
    f, _ = ref.yarn_frequencies(dict(rot, scaling=dict(s, fast=2.1, slow=1.9)))  # from pair 1 (1.96 rounded down) to pair 3 (2.04 rounded up)
    assert np.allclose(f / plain, [1.0, 1.0, 1 - 0.75 / 2, 0.25])
    v = np.array([[[1.0, 0.0, 0.0, 2.0, 5.0]]])
    r = ref.rotate_scaled(v, np.array([3.0]), dict(base=100.0, dims=4, scaling=dict(s, fast=1e-3, slow=1e-4)))
    k = 1 + 0.1 * np.log(4.0)
    assert np.allclose(r, [[[k * np.cos(3.0), k * np.sin(3.0), -2 * k * np.sin(0.3), 2 * k * np.cos(0.3), 5.0]]])


def test_pieces_of_the_differential_attention():
    rng = np.random.default_rng(1)
    m = dict(heads=2, kv_heads=1, dim=4, vdim=3, rot=dict(base=10.0, dims=2), scale=0.5, mask=dict(size=5, keep_first=1), diff=0.25)
    w = dict(q=rng.standard_normal((16, 5)), k=rng.standard_normal((8, 5)), v=rng.standard_normal((3, 5)), o=np.eye(6), g=rng.standard_normal((2, 5)), lq1=np.ones(4), lk1=np.full(4, 0.5), lq2=np.ones(4),
             lk2=np.full(4, 0.25))
    w.update({"q.norm": np.ones(4), "k.norm": np.ones(4)})
    lam = ref.difference_weight(w["lq1"], w["lk1"], w["lq2"], w["lk2"], 0.25)
    assert np.isclose(lam, np.exp(2.0) - np.exp(1.0) + 0.25)
    h = rng.standard_normal((2, 5))
    out, (k, v) = ref.differential_attention(h, w.__getitem__, m, 0.0)
    assert k.shape == (1, 2, 2, 4) and v.shape == (1, 2, 3)
    # one token: both maps answer with its value, of which 1 - lambda is left and normed
    val = w["v"] @ h[0] * (1 - lam)
    for i in range(2):
        assert np.allclose(out[0, 3 * i:3 * i + 3], ref.rms(val, 0.0) * 0.75 * ref.sigmoid(w["g"][i] @ h[0]))
    # two tokens: weights of each map by hand
    for i in range(2):
        a = []
        for j in range(2):
            q = ref.rms((w["q"] @ h[1])[8 * i + 4 * j:8 * i + 4 * j + 4], 0.0)
            q = ref.rotate_pairs(q[None, None], np.array([1.0]), 10.0, 2)[0, 0]
            e = np.exp(0.5 * k[0, j] @ q)
            a.append(e @ v[0] / e.sum())
        assert np.allclose(out[1, 3 * i:3 * i + 3], ref.rms(a[0] - lam * a[1], 0.0) * 0.75 * ref.sigmoid(w["g"][i] @ h[1]))


def test_gated_average_equals_its_closed_form():
    """S_t = sum over s <= t of z_s c_s times the product of 1 - z over (s, t]."""
    rng = np.random.default_rng(3)
    z, c = rng.random((9, 4)), rng.standard_normal((9, 4))
    want = [sum(z[s] * c[s] * (1 - z[s + 1:t + 1]).prod(0) for s in range(t + 1)) for t in range(9)]
    assert np.allclose(want, ref.gated_average(z, c))
    w = {"z": np.zeros((2, 1)), "z.b": np.array([50.0, 50.0]), "x": np.array([[1.0], [-1.0]]), "x.b": np.zeros(2), "g": np.full((2, 1), 2.0), "o": np.eye(2)}
    out = ref.min_gru(np.array([[3.0], [0.0]]), w.__getitem__, None, 0.0)  # the gate is open: the candidate alone, continuous at zero
    assert np.allclose(out, [[3.5 * ref.silu(6.0), ref.sigmoid(-3.0) * ref.silu(6.0)], [0.0, 0.0]])


def test_pieces_around_the_sub_layers():
    w = {"embed": np.arange(6.0).reshape(3, 2), "bigram": 100.0 * np.arange(8.0).reshape(4, 2)}
    x = ref.embed_pairs([2, 1, 0], w, 0.5, dict(buckets=3, mul_prev=2, mul_cur=5))  # rows 3 (no previous), (2 * 2 + 5) % 3, (1 * 2 + 0) % 3
    assert np.allclose(x, [[2 + 600, 2.5 + 700], [1, 1.5 + 100], [400, 0.5 + 500]])
    assert np.allclose(ref.group_norm(np.array([[3.0, 3.0, -0.1, 0.1]]), np.array([1.0, 2.0, 3.0, 4.0]), 2, 0.0), [[1.0, 2.0, -3.0, 4.0]])
    one = {"gate": np.array([[2.0]]), "up": np.array([[-9.0]]), "down": np.array([[1.0]])}
    assert np.allclose(ref.clipped_ff(np.array([[1.0], [-4.0]]), one.__getitem__, 0.5), [[0.5 / (1 + np.exp(-0.851)) * 0.5], [-8.0 / (1 + np.exp(1.702 * 8)) * 1.5]])
    side = {"gate": np.array([[1.0, 0.0]]), "proj": np.array([[1.0], [1.0]]), "norm": np.array([1.0, 3.0])}
    assert np.allclose(ref.token_input(np.array([[2.0, 7.0]]), np.array([[-5.0]]), side.__getitem__, 0.0), [[-1.0, -3.0]])
