"""Plain numpy restatement (float64) of decoders whose layers are listed one by one in config.json: latent attention,
Mamba-2, dense gated and routed feed-forwards.  One function per mechanism, whole sequences only, no cache, no batching:
the yardstick of the layered models' tests.  Nothing here is shared with the library's own code path.

Weights are a dict name -> float array; `cfg` is the parsed config.json.
"""
import math

import numpy as np

F = np.float64


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def silu(x):
    return x / (1.0 + np.exp(-x))


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def rotate_pairs(v, pos, base, dims):
    """v [..., T, d]: coordinates (2i, 2i+1) for 2i < dims turned by pos * base^(-2i/dims)."""
    out = v.copy()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = np.cos(a), np.sin(a)
        u, w = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = u * c - w * s
        out[..., 2 * i + 1] = w * c + u * s
    return out


def latent_attention(h, g, m, eps):
    """h [T, width]; g(name) -> weight of this mixer; m: the mixer's config."""
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T, dtype=F)
    q = (h @ g("q").T).reshape(T, H, D + R).transpose(1, 0, 2)                       # [H, T, D + R]
    qn, qr = q[..., :D], rotate_pairs(q[..., D:], pos, m["rot"]["base"], m["rot"]["dims"])
    ckr = h @ g("dkv").T
    c = rms_norm(ckr[:, :K], g("dkv.norm"), eps)
    kr = rotate_pairs(ckr[:, K:], pos, m["rot"]["base"], m["rot"]["dims"])            # [T, R], one for all heads
    kn = (c @ g("uk").T).reshape(T, H, D).transpose(1, 0, 2)
    v = (c @ g("uv").T).reshape(T, H, V).transpose(1, 0, 2)
    s = (np.einsum("htd,hsd->hts", qn, kn) + np.einsum("htd,sd->hts", qr, kr)) * m["scale"]
    s = np.where(np.tril(np.ones((T, T), bool))[None], s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    p /= p.sum(-1, keepdims=True)
    o = np.einsum("hts,hsv->htv", p, v).transpose(1, 0, 2).reshape(T, H * V)
    return o @ g("o").T


def causal_conv_silu(u, w, b):
    """u [T, channels], w [channels, taps] (last column: the current token), b [channels]."""
    T, taps = u.shape[0], w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, u.shape[1]), F), u])
    return silu(sum(pad[j:j + T] * w[:, j] for j in range(taps)) + b)


def ssd_recurrence(x, B, C, dt, A_log, D):
    """x [T, heads, P], B / C [T, groups, N], dt [T, heads] -> y [T, heads, P], one token after the other."""
    T, H, P = x.shape
    of = np.arange(H) // (H // B.shape[1])                     # group of every head
    S = np.zeros((H, B.shape[2], P), F)
    y = np.zeros_like(x)
    for t in range(T):
        decay = np.exp(-np.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][of][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnp,hn->hp", S, C[t][of]) + D[:, None] * x[t]
    return y


def gated_group_norm(y, z, w, groups, eps):
    v = (y * silu(z)).reshape(y.shape[0], groups, -1)
    return rms(v, eps).reshape(y.shape) * w


def mamba2(h, g, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    zxbcdt = h @ g("in").T
    z, xbc, dt = zxbcdt[:, :inner], zxbcdt[:, inner:2 * inner + 2 * G * N], zxbcdt[:, 2 * inner + 2 * G * N:]
    xbc = causal_conv_silu(xbc, g("conv"), g("conv.b"))
    y = ssd_recurrence(xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + G * N].reshape(T, G, N),
                       xbc[:, inner + G * N:].reshape(T, G, N), softplus(dt + g("dt_bias")), g("A_log"), g("D"))
    return gated_group_norm(y.reshape(T, inner), z, g("norm"), m["norm_groups"], eps) @ g("o").T


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2}


def dense_ff(h, g):
    return (gelu_tanh(h @ g("gate").T) * (h @ g("up").T)) @ g("down").T


def clipped_expert(h, g, e, limit):
    a = np.minimum(h @ g(f"e{e}.gate").T, limit)
    u = np.clip(h @ g(f"e{e}.up").T, -limit, limit)
    return (a * sigmoid(1.702 * a) * (u + 1.0)) @ g(f"e{e}.down").T


def routed_ff(h, g, mlp):
    """Scores by a sigmoid, the best `top` experts, each fed its score times the input."""
    s = sigmoid(h @ g("router").T)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in np.argsort(-s[t], kind="stable")[:mlp["router"]["top"]]:
            out[t] += clipped_expert(s[t, e] * h[t], g, e, mlp["expert"]["limit"])
    return out


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  layers_out (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)].astype(F)
    for i, L in enumerate(cfg["layers"]):
        mix = lambda n, i=i: w[f"l{i}.mix.{n}"]
        ff = lambda n, i=i: w[f"l{i}.mlp.{n}"]
        x = x + MIXERS[L["type"]](rms_norm(x, w[f"l{i}.norm1"], eps), mix, L["mixer"], eps)
        if L.get("mlp"):
            h = rms_norm(x, w[f"l{i}.norm2"], eps)
            x = x + (dense_ff(h, ff) if L["mlp"]["kind"] == "dense" else routed_ff(h, ff, L["mlp"]))
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
