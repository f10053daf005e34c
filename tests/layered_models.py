"""Small layered models for the tests: configurations, random weights (bf16 values held as float64) and loaders."""
import json
import os
import struct

import numpy as np

from tests import helpers as H


def latent(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=56, base=900.0, scale=None, dims=None):
    return ("latent_attention", dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank,
                                     rot=dict(base=base, dims=rot_dim if dims is None else dims),
                                     scale=scale if scale is not None else float((dim + rot_dim) ** -0.5)))


def mamba(heads=4, vdim=24, state=40, groups=2, norm_groups=4, conv=3):
    return ("mamba2", dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv))


def dense(ff=136):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=2, ff=72, limit=0.7):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def config(layers, width=104, vocab=333, eps=3e-5, logit_scale=0.4):
    return dict(architecture="Zukitar", width=width, vocab=vocab, norm=dict(eps=eps), logit_scale=logit_scale,
                layers=[dict(type=m[0], mixer=m[1], mlp=f) for m, f in layers])


# ---- Tirezen: retention, delta memories, capped sink attention beside a delta memory, a repeated stretch of layers ------
def retention(heads=3, dim=20, vdim=28, base=3000.0, dims=12, decay=None):
    return ("retention", dict(heads=heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=dims),
                              decay=decay or [1.0 - 2.0 ** -(2 + 3 * (i % 3)) for i in range(heads)]))


def delta(heads=6, kv_heads=3, dim=28, vdim=12, conv=2):
    return ("delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv))


def sides(heads=4, kv_heads=2, dim=24, vdim=40, dims=16, base=700.0, scale=None, softcap=4.0, left_scale=0.7, right_scale=1.3, right=None):
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=dims), scale=scale or dim ** -0.5 * 1.5, softcap=softcap)
    right = {**dict(heads=4, kv_heads=2, dim=12, vdim=20, conv=3), **(right or {})}
    return ("parallel", dict(left=left, right=right, left_scale=left_scale, right_scale=right_scale))


def tirezen(layers, width=72, vocab=211, eps=2e-5, loop=(0, 0, 0)):
    cfg = dict(architecture="Tirezen", width=width, vocab=vocab, norm=dict(eps=eps), layers=[dict(type=m[0], mixer=m[1], mlp=f) for m, f in layers])
    if loop[2]:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


def tirezen_weights(cfg, seed=0, gain=None, ranks=(7, 11)):
    """name -> float64 array of bf16 values; ranks: of the decay's and the gate's two-factor projections."""
    rng = np.random.default_rng(seed)
    w, W = {}, cfg["width"]

    def mat(name, rows, cols):
        g = next((v for k, v in (gain or {}).items() if name.endswith(k)), 1.0)
        w[name] = round_bf16(rng.standard_normal((rows, cols)) * g / np.sqrt(cols))

    def vec(name, n, mean, sd):
        w[name] = round_bf16(mean + sd * rng.standard_normal(n))

    def delta_part(p, m, low_rank):
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, c in (("q", G * D), ("k", G * D), ("v", H * V)):
            mat(p + n, c, W)
            vec(f"{p}{n}.conv", (c, m["conv"]), 0.3, 0.6)
        mat(p + "b", H, W)
        vec(p + "A_log", H, 0.0, 1.0)
        vec(p + "norm", V, 1.0, 0.2)
        if low_rank:
            mat(p + "a1", ranks[0], W), mat(p + "a2", H * D, ranks[0]), mat(p + "g1", ranks[1], W), mat(p + "g2", H * V, ranks[1])
            vec(p + "dt_bias", H * D, -2.5, 1.5)
        else:
            mat(p + "a", H, W), mat(p + "g", H * V, W)
            vec(p + "dt_bias", H, -2.5, 1.5)
        mat(p + "o", W, H * V)

    w["embed"] = round_bf16(rng.standard_normal((cfg["vocab"], W)))
    if cfg.get("loop"):
        vec("loop.step", (cfg["loop"]["times"], W), 0.0, 0.5)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W, 0.0, 0.2)
        if L["type"] == "retention":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            mat(p + "q", H * D, W), mat(p + "k", H * D, W), mat(p + "v", H * V, W), mat(p + "g", H * V, W), mat(p + "o", W, H * V)
        elif L["type"] == "delta":
            delta_part(p, m, False)
        else:
            a = m["left"]
            for n, c in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                mat(p + "left." + n, c, W)
                vec(f"{p}left.{n}.b", c, 0.0, 0.3)
            vec(p + "left.q.norm", a["dim"], 1.2, 0.3)
            vec(p + "left.k.norm", a["dim"], 1.2, 0.3)
            mat(p + "left.o", W, a["heads"] * a["vdim"])
            delta_part(p + "right.", m["right"], True)
        if L["mlp"]:
            mat(f"l{i}.mlp.up", L["mlp"]["ff"], W), mat(f"l{i}.mlp.down", W, L["mlp"]["ff"])
    vec("final.norm", W, 0.0, 0.2)
    mat("head", cfg["vocab"], W)
    return w


# ---- Zokuzen: time mixing, windowed latent and chunked attention, shared keys, residual streams, mixtures of experts --------
def wkv(heads=3, dim=20):
    return ("wkv", dict(heads=heads, dim=dim))


def window(heads=3, dim=24, vdim=40, kv_rank=56, size=21, scale=None):
    return ("latent_attention", dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, mask=dict(size=size), scale=scale or float(dim ** -0.5)))


def chunk(heads=4, kv_heads=2, dim=24, vdim=40, dims=16, base=700.0, size=27, scale=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=dims), mask=dict(size=size), scale=scale or float(dim ** -0.5 * 1.5))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return ("attention", m)


def mixture(experts=5, identity=2, top=3, ff=40, shared=56, scale=1.75):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, identity=identity, top=top, scale=scale), shared=dict(ff=shared) if shared else None)


def zokuzen(layers, width=72, vocab=211, eps=2e-5, streams=2):
    return dict(architecture="Zokuzen", width=width, vocab=vocab, norm=dict(eps=eps), streams=streams, layers=[dict(type=m[0], mixer=m[1], mlp=f) for m, f in layers])


def zokuzen_weights(cfg, seed=0, gain=None, rank=9, decide=True):
    """name -> float64 array of bf16 values; rank: of the decays' two factors.  decide: keep routing away from close calls."""
    rng = np.random.default_rng(seed)
    w, W, S = {}, cfg["width"], cfg["streams"]

    def mat(name, rows, cols):
        g = next((v for k, v in (gain or {}).items() if name.endswith(k)), 1.0)
        w[name] = round_bf16(rng.standard_normal((rows, cols)) * g / np.sqrt(cols))

    def vec(name, n, mean, sd):
        w[name] = round_bf16(mean + sd * rng.standard_normal(n))

    w["embed"] = round_bf16(rng.standard_normal((cfg["vocab"], W)))
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        for q in (1, 2) if L["mlp"] else (1,):
            vec(f"l{i}.norm{q}", W, 0.0, 0.2)
            w[f"l{i}.hc{q}.in"] = round_bf16(rng.uniform(0.1, 1.2, S) / S ** 0.5)
            w[f"l{i}.hc{q}.out"] = round_bf16(rng.uniform(0.4, 1.4, S))
            w[f"l{i}.hc{q}.mix"] = round_bf16(rng.uniform(-0.1, 0.5, (S, S)) / S + 0.7 * np.eye(S))
        if L["type"] == "wkv":
            Q = m["heads"] * m["dim"]
            for n in "rkvgw":
                w[f"{p}mu.{n}"] = round_bf16(rng.uniform(0, 1, W))
            for n in "rkvg":
                mat(p + n, Q, W)
            mat(p + "w1", rank, W), mat(p + "w2", Q, rank), mat(p + "o", W, Q)
            vec(p + "w0", Q, -2.0, 2.0)
            vec(p + "u", (m["heads"], m["dim"]), 0.5, 0.6)
            vec(p + "norm", Q, 1.0, 0.2)
        elif L["type"] == "latent_attention":
            mat(p + "q", m["heads"] * m["dim"], W), mat(p + "dkv", m["kv_rank"], W)
            vec(p + "dkv.norm", m["kv_rank"], 1.0, 0.2)
            mat(p + "uk", m["heads"] * m["dim"], m["kv_rank"]), mat(p + "uv", m["heads"] * m["vdim"], m["kv_rank"])
            mat(p + "o", W, m["heads"] * m["vdim"])
        else:
            mat(p + "q", m["heads"] * m["dim"], W)
            vec(p + "q.norm", m["heads"] * m["dim"], 1.2, 0.3)
            if m.get("kv_from") is None:
                mat(p + "k", m["kv_heads"] * m["dim"], W), mat(p + "v", m["kv_heads"] * m["vdim"], W)
                vec(p + "k.norm", m["kv_heads"] * m["dim"], 1.2, 0.3)
            mat(p + "o", W, m["heads"] * m["vdim"])
        f, p = L["mlp"], f"l{i}.mlp."
        if not f:
            continue
        n = f["router"]["experts"] + f["router"].get("identity", 0)
        mat(p + "router", n, W)
        vec(p + "correction", n, 0.0, 0.2)
        for e in range(f["router"]["experts"]):
            ff = f["expert"]["ff"]
            mat(f"{p}e{e}.gate", ff, W), mat(f"{p}e{e}.up", ff, W), mat(f"{p}e{e}.down", W, ff)
        if f.get("shared"):
            ff = f["shared"]["ff"]
            mat(p + "shared.gate", ff, W), mat(p + "shared.up", ff, W), mat(p + "shared.down", W, ff), mat(p + "shared.sg", 1, W)
    vec("final.norm", W, 0.0, 0.2)
    if decide:
        decide_mixtures(cfg, w, rng)
    return w


def decide_mixtures(cfg, w, rng, cols=8, margin=0.3):
    """As decide_routes: routers read the first few coordinates, which hold a positive multiple of the embedding's in every stream.
    One router output is always chosen and one never is (corrections beyond what a score can outweigh); among the rest every
    token has a gap."""
    routers = [(i, L["mlp"]["router"]) for i, L in enumerate(cfg["layers"]) if L["mlp"]]
    if not routers:
        return
    for k in w:
        if k.endswith((".mix.o", ".down")):
            w[k][:cols] = 0
    cut = {}
    for i, r in routers:
        n = r["experts"] + r.get("identity", 0)
        w[f"l{i}.norm2"][:cols] = 0
        z = rng.standard_normal((n, cols))
        w[f"l{i}.mlp.router"] = round_bf16(np.concatenate([z, np.zeros((n, cfg["width"] - cols))], 1))
        c = np.zeros(n)
        if n > 3 and 1 < r["top"] < n - 1:
            c[rng.permutation(n)[:2]] = 3.0, -3.0
        w[f"l{i}.mlp.correction"] = c
        cut[i] = (np.nonzero(c == 0)[0], r["top"] - int((c > 0).sum()))
    for t in range(cfg["vocab"]):
        for _ in range(100000):
            v = round_bf16(1.5 * rng.standard_normal(cols))
            gaps = [1e9]
            for i, (free, top) in cut.items():
                z = np.sort((w[f"l{i}.mlp.router"][:, :cols] @ v)[free])[::-1]
                if 0 < top < len(z):
                    gaps.append(z[top - 1] - z[top])
            if min(gaps) > margin:
                break
        w["embed"][t, :cols] = v


# ---- Pokadra: differential attention, minimal gated recurrences, norms behind the sub-layers, token pairs and token inputs, depth averages -----
def differential(heads=4, kv_heads=2, dim=24, vdim=40, dims=16, base=700.0, size=27, keep=5, diff=0.35, scale=None, kv_from=None, scaling=True, original=90, factor=6.0, fast=9.0, slow=1.5):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, diff=diff, rot=dict(base=base, dims=dims), mask=dict(size=size, keep_first=keep), scale=scale or float(dim ** -0.5))
    if scaling:
        m["rot"]["scaling"] = dict(factor=factor, original=original, fast=fast, slow=slow)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return ("attention", m)


def mingru(width=88):
    return ("mingru", dict(width=width))


def clipped(ff=136, limit=0.9):
    return dict(kind="dense", ff=ff, limit=limit)


def pokadra(layers, width=72, vocab=211, eps=2e-5, groups=3, mult=0.45, side=20, scale=0.7, pairs=(103, 29, 7)):
    return dict(architecture="Pokadra", width=width, vocab=vocab, norm=dict(eps=eps, groups=groups), residual_mult=mult, token_side=dict(dim=side),
                embedding=dict(scale=scale, bigram=dict(buckets=pairs[0], mul_prev=pairs[1], mul_cur=pairs[2])),
                layers=[dict(type=m[0], mixer=m[1], mlp=f) for m, f in layers])


def pokadra_weights(cfg, seed=0, gain=None):
    """name -> float64 array of bf16 values."""
    rng = np.random.default_rng(seed)
    w, W, D = {}, cfg["width"], cfg["token_side"]["dim"]

    def mat(name, rows, cols):
        g = next((v for k, v in (gain or {}).items() if name.endswith(k)), 1.0)
        w[name] = round_bf16(rng.standard_normal((rows, cols)) * g / np.sqrt(cols))

    def vec(name, n, mean, sd):
        w[name] = round_bf16(mean + sd * rng.standard_normal(n))

    w["embed"] = round_bf16(1.5 * rng.standard_normal((cfg["vocab"], W)))
    w["bigram"] = round_bf16(0.6 * rng.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, W)))
    w["side.embed"] = round_bf16(rng.standard_normal((cfg["vocab"], D * len(cfg["layers"]))))
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W, 1.0, 0.2)
        if L["type"] == "mingru":
            n = m["width"]
            mat(p + "z", n, W), mat(p + "x", n, W), mat(p + "g", n, W), mat(p + "o", W, n)
            vec(p + "z.b", n, -2.0, 2.5)
            vec(p + "x.b", n, 0.0, 0.3)
        else:
            H, G, d, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mat(p + "q", H * 2 * d, W), mat(p + "g", H, W), mat(p + "o", W, H * V)
            vec(p + "q.norm", d, 1.2, 0.3)
            if m.get("kv_from") is None:
                mat(p + "k", G * 2 * d, W), mat(p + "v", G * V, W)
                vec(p + "k.norm", d, 1.2, 0.3)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                vec(p + n, d, 0.0, 0.15)
        if L["mlp"]:
            ff, p = L["mlp"]["ff"], f"l{i}.mlp."
            vec(f"l{i}.norm2", W, 1.0, 0.2)
            mat(p + "gate", ff, W), mat(p + "up", ff, W), mat(p + "down", W, ff)
        mat(f"l{i}.side.gate", D, W), mat(f"l{i}.side.proj", W, D)
        vec(f"l{i}.side.norm", W, 0.5, 0.15)
        c = rng.uniform(-0.2, 0.5, i + 2)
        c[-1] += 0.6
        w[f"l{i}.dwa"] = round_bf16(c)
    vec("final.norm", W, 1.0, 0.2)
    mat("head", cfg["vocab"], W)
    return w


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


def error(got, want):
    """Worst row: rms of the error over the rms spread of the wanted logits."""
    d = got - want
    d = d - d.mean(1, keepdims=True)
    spread = np.sqrt(np.mean((want - want.mean(1, keepdims=True)) ** 2))
    return float(np.sqrt((d * d).mean(1)).max() / spread)


def run(eng, model, pool, ids, cuts, cache=None):
    """Feeds ids in portions of the given sizes, the rest one by one; logits of every position."""
    c = cache or eng.PagedKvCache(pool)
    out, at = [], 0
    while at < len(ids):
        n = min(cuts[len(out)] if len(out) < len(cuts) else 1, len(ids) - at)
        lg, _ = model.step_at([(ids[at:at + n], c)], [list(range(n))])
        out.append(lg)
        at += n
    if cache is None:
        c.free()
    return np.concatenate(out)


def round_bf16(a):
    return H.bf16_to_f32_np(H.f32_to_bf16_np(np.asarray(a, np.float32))).astype(np.float64)


def weights(cfg, seed=0, gain=None):
    """name -> float64 array of bf16 values.  gain: {name suffix: factor} on top of the 1/sqrt(inputs) scale."""
    rng = np.random.default_rng(seed)
    w, W = {}, cfg["width"]

    def mat(name, rows, cols):
        g = next((v for k, v in (gain or {}).items() if name.endswith(k)), 1.0)
        w[name] = round_bf16(rng.standard_normal((rows, cols)) * g / np.sqrt(cols))

    def vec(name, n, mean, sd):
        w[name] = round_bf16(mean + sd * rng.standard_normal(n))

    w["embed"] = round_bf16(rng.standard_normal((cfg["vocab"], W)))
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W, 1.0, 0.2)
        if L["type"] == "latent_attention":
            mat(p + "q", m["heads"] * (m["dim"] + m["rot_dim"]), W)
            mat(p + "dkv", m["kv_rank"] + m["rot_dim"], W)
            vec(p + "dkv.norm", m["kv_rank"], 1.0, 0.2)
            mat(p + "uk", m["heads"] * m["dim"], m["kv_rank"])
            mat(p + "uv", m["heads"] * m["vdim"], m["kv_rank"])
            mat(p + "o", W, m["heads"] * m["vdim"])
        else:
            inner = m["heads"] * m["vdim"]
            ch = inner + 2 * m["groups"] * m["state"]
            mat(p + "in", inner + ch + m["heads"], W)
            vec(p + "conv", (ch, m["conv"]), 0.0, 0.6)
            vec(p + "conv.b", ch, 0.0, 0.3)
            vec(p + "dt_bias", m["heads"], -2.0, 1.5)
            vec(p + "A_log", m["heads"], 0.0, 1.0)
            vec(p + "D", m["heads"], 1.0, 0.4)
            vec(p + "norm", inner, 1.0, 0.2)
            mat(p + "o", W, inner)
        f, p = L["mlp"], f"l{i}.mlp."
        if f is None:
            continue
        vec(f"l{i}.norm2", W, 1.0, 0.2)
        if f["kind"] == "dense":
            mat(p + "gate", f["ff"], W), mat(p + "up", f["ff"], W), mat(p + "down", W, f["ff"])
        else:
            mat(p + "router", f["router"]["experts"], W)
            for e in range(f["router"]["experts"]):
                ff = f["expert"]["ff"]
                mat(f"{p}e{e}.gate", ff, W), mat(f"{p}e{e}.up", ff, W), mat(f"{p}e{e}.down", W, ff)
    vec("final.norm", W, 1.0, 0.2)
    decide_routes(cfg, w, rng)
    return w


def decide_routes(cfg, w, rng, cols=8, margin=0.15):
    """Keeps routing away from close calls, which rounding may settle either way: the routers read the first few coordinates
    only, no layer writes to those, and every token's values there put a gap between the chosen experts and the rest."""
    routers = [(i, L["mlp"]["router"]) for i, L in enumerate(cfg["layers"]) if L["mlp"] and L["mlp"]["kind"] == "moe"]
    if not routers:
        return
    for k in w:
        if k.endswith((".mix.o", ".down")):
            w[k][:cols] = 0
    for i, r in routers:
        w[f"l{i}.norm2"][:cols] = 1
        z = rng.standard_normal((r["experts"], cols))
        w[f"l{i}.mlp.router"] = round_bf16(np.concatenate([z, np.zeros((r["experts"], cfg["width"] - cols))], 1))
    E = w["embed"]
    for t in range(cfg["vocab"]):
        for _ in range(100000):
            v = round_bf16(rng.standard_normal(cols))
            gaps = []
            for i, r in routers:
                z = np.sort(w[f"l{i}.mlp.router"][:, :cols] @ v)[::-1]
                gaps.append(z[r["top"] - 1] - z[r["top"]] if r["top"] < r["experts"] else 1e9)
            if min(gaps) > margin:
                break
        E[t, :cols] = v


def load(eng, ctx, cfg, w, f32):
    ws = eng.Weights()
    for k, v in w.items():
        ws.add(k, H.f32_to_bf16_np(v.astype(np.float32)), bf16=True)
    m = eng.CausalLm.from_json(ctx, ws, cfg, f32=f32)
    ws.free()
    return m


def save(path, cfg, w):
    """A folder with config.json and model.safetensors (bf16)."""
    header, blobs, off = {}, [], 0
    for k, v in w.items():
        b = H.f32_to_bf16_np(v.astype(np.float32)).tobytes()
        header[k] = dict(dtype="BF16", shape=list(v.shape), data_offsets=[off, off + len(b)])
        blobs.append(b)
        off += len(b)
    h = json.dumps(header).encode()
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)


# Designs that differ in every size and in the order of layers; dimensions that divide nothing, single groups, a mixer
# without a feed-forward, all experts chosen, a rotation narrower than its part of the head.
CASES = {
    "mixed": config([(latent(), dense()), (mamba(norm_groups=2), moe()), (latent(heads=2, base=70000.0), None), (mamba(groups=4, conv=4, norm_groups=1), dense(88))]),
    "recurrent_first": config([(mamba(heads=6, vdim=20, state=12, groups=3, norm_groups=1, conv=2), moe(experts=7, top=3)),
                               (mamba(heads=2, groups=1, conv=5, state=70), None), (latent(heads=5, dim=10, rot_dim=6, vdim=9, kv_rank=21), moe(top=1))],
                              width=60, vocab=97, eps=1e-4, logit_scale=1.7),
    "narrow_rotation": config([(latent(rot_dim=20, dims=12, vdim=17), moe(experts=3, top=3, ff=40, limit=2.5))], width=72, vocab=50),
    # head sizes of the tensor-core tiles: plain 128 | rotated 64, values 128, more than 16 (and more than 32) heads
    "wide_heads": config([(latent(heads=18, dim=128, rot_dim=64, vdim=128, kv_rank=192), dense(512)),
                          (latent(heads=33, dim=64, rot_dim=32, vdim=64, kv_rank=512), None)], width=256, vocab=400),
    # outside the expanded-key kernel's tiles: attention in latent coordinates for prompts as well
    "wide_plain": config([(latent(heads=2, dim=200, rot_dim=8, vdim=140, kv_rank=72), dense(64))], width=64, vocab=80),
    "big_state": config([(mamba(heads=4, vdim=64, state=128, groups=1, norm_groups=2, conv=4), moe(experts=16, top=4, ff=128)),
                         (mamba(heads=2, vdim=16, state=200, groups=2, norm_groups=2), dense(192))], width=128, vocab=200),
}

TIREZEN = {
    "all_kinds": tirezen([(retention(), dense(88)), (sides(), dense(136)), (delta(), None), (sides(heads=6, kv_heads=1, vdim=16, softcap=9.0, right=dict(conv=4)), dense(40))],
                         loop=(1, 3, 3)),
    # sizes that divide nothing, one head, one tap, single query groups
    "odd": tirezen([(sides(heads=5, kv_heads=5, dim=10, vdim=7, dims=4, right=dict(conv=1)), dense(33)), (delta(heads=3, kv_heads=1, dim=9, vdim=5, conv=5), dense(50)),
                    (retention(heads=1, dim=7, vdim=3, dims=6), None)], width=53, vocab=97, loop=(0, 3, 2)),
    # the tiles of the tensor-core kernels, more than eight query heads for one key head
    "tiles": tirezen([(sides(heads=10, kv_heads=1, dim=128, vdim=128, dims=128, softcap=15.0, right=dict(heads=2, kv_heads=1, dim=128, vdim=64, conv=4)), dense(512)),
                      (retention(heads=2, dim=128, vdim=128, dims=64), dense(256)), (delta(heads=2, kv_heads=2, dim=128, vdim=64, conv=4), None)],
                     width=128, vocab=300, loop=(2, 3, 1)),
    "uneven": tirezen([(sides(heads=4, kv_heads=4, dim=160, vdim=72, dims=96, softcap=3.0), None), (sides(heads=3, kv_heads=3, dim=64, vdim=144, dims=64), dense(64)),
                       (retention(heads=2, dim=48, vdim=200, dims=48), dense(72))], width=96, vocab=150),
    # beyond those kernels
    "large_heads": tirezen([(sides(heads=2, kv_heads=1, dim=232, vdim=250, dims=100, softcap=6.0), None), (delta(heads=2, kv_heads=1, dim=200, vdim=136, conv=3), dense(30))],
                           width=64, vocab=80),
}

ZOKUZEN = {
    "all_kinds": zokuzen([(wkv(), mixture()), (window(), mixture(experts=7, identity=1, top=2, scale=0.9)), (chunk(), None), (wkv(heads=2, dim=28), None),
                          (chunk(size=40, kv_from=2, scale=0.4), mixture(shared=None)), (chunk(heads=2, kv_heads=1, dim=16, vdim=32, dims=8, size=11), mixture(identity=0, top=5))],
                         streams=3),
    # sizes that divide nothing, single heads, all router outputs chosen, one stream
    "odd": zokuzen([(window(heads=5, dim=7, vdim=9, kv_rank=19, size=13), mixture(experts=3, identity=1, top=4, ff=17, shared=23)), (wkv(heads=1, dim=13), mixture(experts=4, identity=3, top=1, ff=9)),
                    (chunk(heads=3, kv_heads=1, dim=10, vdim=7, dims=4, size=37), mixture(ff=33, shared=11)), (chunk(heads=6, kv_heads=1, dim=10, vdim=7, dims=4, size=9, kv_from=2), None)],
                   width=53, vocab=97, streams=1),
    # the tiles of the tensor-core kernels
    "tiles": zokuzen([(wkv(heads=2, dim=64), mixture(experts=16, identity=4, top=4, ff=128, shared=256)), (window(heads=18, dim=128, vdim=128, kv_rank=192, size=100), mixture(experts=4, identity=0, top=2, ff=64)),
                      (chunk(heads=10, kv_heads=1, dim=128, vdim=128, dims=128, size=96), None), (wkv(heads=1, dim=128), mixture(ff=64)), (chunk(heads=5, kv_heads=1, dim=128, vdim=128, dims=64, size=150, kv_from=2), None)],
                     width=128, vocab=300, streams=4),
    "uneven": zokuzen([(window(heads=33, dim=64, vdim=64, kv_rank=512, size=130), None), (chunk(heads=4, kv_heads=4, dim=160, vdim=72, dims=96, size=128), mixture(experts=6, top=2)),
                       (wkv(heads=3, dim=48), None), (window(heads=2, dim=100, vdim=72, kv_rank=40, size=64), None)], width=96, vocab=150, streams=2),
    # beyond those kernels, many streams
    "large_heads": zokuzen([(window(heads=2, dim=200, vdim=140, kv_rank=72, size=33), None), (chunk(heads=2, kv_heads=1, dim=232, vdim=250, dims=100, size=50), mixture()), (wkv(heads=2, dim=150), None)],
                           width=64, vocab=80, streams=6),
}

POKADRA = {
    "all_kinds": pokadra([(differential(), clipped()), (mingru(), clipped(88, 1.7)), (differential(size=40, keep=17, kv_from=0, scale=0.4), None), (mingru(width=40), None),
                          (differential(heads=2, kv_heads=1, dim=16, vdim=32, dims=8, size=11, keep=0), clipped(40)), (differential(heads=6, size=200, keep=70, kv_from=0, diff=0.8), clipped(72, 0.2))]),
    # sizes that divide nothing, single heads and groups, no scaling, windows of one
    "odd": pokadra([(mingru(width=13), clipped(33)), (differential(heads=5, kv_heads=5, dim=10, vdim=7, dims=4, size=13, keep=1, scaling=False), None),
                    (differential(heads=3, kv_heads=1, dim=9, vdim=5, dims=6, size=1, keep=3), clipped(17, 4.0)), (mingru(width=97), clipped(50))],
                   width=53, vocab=97, groups=1, side=7, pairs=(1, 5, 3)),
    # the tiles of the tensor-core kernels, more than four query heads for one key head
    "tiles": pokadra([(differential(heads=10, kv_heads=1, dim=64, vdim=128, dims=64, size=100, keep=20), clipped(512)), (mingru(width=256), clipped(256)),
                      (differential(heads=4, kv_heads=2, dim=128, vdim=128, dims=32, size=150, keep=128), None), (differential(heads=4, kv_heads=2, dim=64, vdim=64, dims=64, size=96, keep=4), clipped(64)),
                      (differential(heads=5, kv_heads=1, dim=64, vdim=128, dims=64, size=300, keep=130, kv_from=0), None)], width=128, vocab=300, groups=8, side=64, mult=1.0),
    "uneven": pokadra([(differential(heads=4, kv_heads=4, dim=72, vdim=100, dims=36, size=128, keep=16), clipped(100)), (differential(heads=3, kv_heads=3, dim=100, vdim=64, dims=100, size=64, keep=33), None),
                       (mingru(width=300), None), (differential(heads=8, kv_heads=1, dim=8, vdim=8, dims=2, size=500, keep=2), clipped(24))], width=96, vocab=150, groups=12, side=130, scale=1.0),
    # beyond those kernels
    "large_heads": pokadra([(differential(heads=2, kv_heads=1, dim=136, vdim=250, dims=100, size=50, keep=9), clipped(30)), (differential(heads=2, kv_heads=2, dim=100, vdim=200, dims=8, size=33, keep=40), None)],
                           width=64, vocab=80, groups=4, side=1),
}
