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
