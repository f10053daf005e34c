"""Plain numpy restatement (float64) of decoders whose layers are listed one by one in config.json: latent attention,
Mamba-2, softmax attention with a cap and a sink, retention, the gated delta rule, two mixers side by side, time mixing with a
bonus for the current token, windowed latent and chunked grouped attention (also on another layer's keys), differential attention
under a window that keeps the first tokens, the minimal gated recurrence, dense (gated and plain) and routed feed-forwards, shared and
identity experts, repeated layers, several residual streams, averages over the depth, token inputs per layer, embeddings of token
pairs.  One function per mechanism, whole sequences only, no cache, no batching: the yardstick of the layered models' tests.  Nothing here is shared with the library's own code path.

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


def gelu_erf(x):
    return 0.5 * x * (1.0 + np.vectorize(math.erf)(x / math.sqrt(2.0)))


def rotate_halves(v, pos, base, dims):
    """v [..., T, d]: coordinates (i, i + dims/2) for i < dims/2 turned by pos * base^(-2i/dims)."""
    out = v.copy()
    for i in range(dims // 2):
        j = i + dims // 2
        a = pos * base ** (-2.0 * i / dims)
        out[..., i] = v[..., i] * np.cos(a) - v[..., j] * np.sin(a)
        out[..., j] = v[..., j] * np.cos(a) + v[..., i] * np.sin(a)
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


def sink_attention(h, g, m, eps):
    """Grouped-query attention: biases, per-head norms of queries and keys, rotated halves, capped scores, and a softmax
    whose denominator has one more term, exp(0)."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T, dtype=F)
    part = lambda n, heads, d: (h @ g(n).T + g(n + ".b")).reshape(T, heads, d).transpose(1, 0, 2)
    turn = lambda v: rotate_halves(v, pos, m["rot"]["base"], m["rot"]["dims"])
    q = turn(rms_norm(part("q", H, D), g("q.norm"), eps))
    k = turn(rms_norm(part("k", G, D), g("k.norm"), eps))
    v = part("v", G, V)
    out = np.zeros((T, H, V), F)
    for i in range(H):
        s = q[i] @ k[i // (H // G)].T * m["scale"]
        s = m["softcap"] * np.tanh(s / m["softcap"])
        s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
        top = np.maximum(s.max(-1, keepdims=True), 0.0)
        e = np.exp(s - top)
        out[:, i] = e / (np.exp(-top) + e.sum(-1, keepdims=True)) @ v[i // (H // G)]
    return out.reshape(T, H * V) @ g("o").T


def decayed_memory(q, k, v, log_decay, beta=None):
    """One head, one token after the other: q, k [T, D], v [T, V], log_decay [T, D].  Without beta the memory adds k v^T;
    with it, k u^T with u = beta (v - what the decayed memory answers to k).  The read-out sees the token's own write."""
    S = np.zeros((k.shape[1], v.shape[1]), F)
    out = np.zeros((k.shape[0], v.shape[1]), F)
    for t in range(k.shape[0]):
        S = np.exp(log_decay[t])[:, None] * S
        u = v[t] if beta is None else beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def retention(h, g, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    pos = np.arange(T, dtype=F)
    turn = lambda v: rotate_halves(v.reshape(T, H, D).transpose(1, 0, 2), pos, m["rot"]["base"], m["rot"]["dims"])
    q, k, v = turn(h @ g("q").T), turn(h @ g("k").T) * D ** -0.5, (h @ g("v").T).reshape(T, H, V)
    o = np.stack([decayed_memory(q[i], k[i], v[:, i], np.full((T, D), math.log(m["decay"][i]))) for i in range(H)], 1)
    return (rms(o, eps).reshape(T, H * V) * silu(h @ g("g").T)) @ g("o").T


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def gated_delta(h, g, m, eps, per_channel=False):
    """per_channel: a decay per head and key channel and a sigmoid output gate, both from low-rank projections; otherwise a
    decay per head and a silu gate."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda n: causal_conv_silu(h @ g(n).T, g(n + ".conv"), 0.0)
    q, k, v = unit(conv("q").reshape(T, G, D)) * D ** -0.5, unit(conv("k").reshape(T, G, D)), conv("v").reshape(T, H, V)
    beta = sigmoid(h @ g("b").T)
    if per_channel:
        step = softplus(h @ g("a1").T @ g("a2").T + g("dt_bias")).reshape(T, H, D)
        gate = sigmoid(h @ g("g1").T @ g("g2").T)
    else:
        step = np.repeat(softplus(h @ g("a").T + g("dt_bias"))[:, :, None], D, 2)
        gate = silu(h @ g("g").T)
    log_decay = -np.exp(g("A_log"))[:, None] * step
    o = np.stack([decayed_memory(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], log_decay[:, i], beta[:, i]) for i in range(H)], 1)
    return ((rms(o, eps) * g("norm")).reshape(T, H * V) * gate) @ g("o").T


def side_by_side(h, g, m, eps):
    left = sink_attention(h, lambda n: g("left." + n), m["left"], eps)
    right = gated_delta(h, lambda n: g("right." + n), m["right"], eps, per_channel=True)
    return m["left_scale"] * left + m["right_scale"] * right


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2, "retention": retention, "delta": gated_delta, "parallel": side_by_side}


def plain_ff(h, g):
    return gelu_erf(h @ g("up").T) @ g("down").T


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


# ---- Zokuzen ---------------------------------------------------------------------------------------------------------
def shifted(h):
    """Row t holds the previous token's h (zeros for the first token)."""
    return np.concatenate([np.zeros((1, h.shape[1]), F), h[:-1]])


def bonus_memory(r, k, v, w, u):
    """One head, one token after the other: r, k, w [T, D], v [T, D], u [D].  The read-out sees the state before the token's own
    write, plus that write weighted by u; the decay w comes after the read-out."""
    S = np.zeros((k.shape[1], v.shape[1]), F)
    out = np.zeros((k.shape[0], v.shape[1]), F)
    for t in range(k.shape[0]):
        kv = np.outer(k[t], v[t])
        out[t] = (S + u[:, None] * kv).T @ r[t]
        S = w[t][:, None] * S + kv
    return out


def time_mix(h, g, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    step = shifted(h) - h
    mixed = {n: h + step * g("mu." + n) for n in "rkvgw"}
    r, k, v = ((mixed[n] @ g(n).T).reshape(T, H, D) for n in "rkv")
    w = np.exp(-np.exp(np.tanh(mixed["w"] @ g("w1").T) @ g("w2").T + g("w0"))).reshape(T, H, D)
    o = np.stack([bonus_memory(r[:, i], k[:, i], v[:, i], w[:, i], g("u")[i]) for i in range(H)], 1)
    return (rms(o, eps).reshape(T, H * D) * g("norm") * silu(mixed["g"] @ g("g").T)) @ g("o").T


def in_window(T, size):
    """visible[i, j]: j is i or one of the size - 1 tokens before it."""
    i, j = np.arange(T)[:, None], np.arange(T)[None]
    return (j <= i) & (i - j < size)


def in_chunk(T, size):
    """visible[i, j]: j <= i lies in the same stretch of `size` tokens, counted from the sequence's start."""
    i, j = np.arange(T)[:, None], np.arange(T)[None]
    return (j <= i) & (i // size == j // size)


def softmax_attention(q, k, v, scale, visible):
    """q [H, T, D], k [G, T, D], v [G, T, V] -> [T, H * V]; query head h reads key head h // (H / G)."""
    H, T = q.shape[:2]
    out = np.zeros((T, H, v.shape[2]), F)
    for i in range(H):
        g = i // (H // k.shape[0])
        s = np.where(visible, q[i] @ k[g].T * scale, -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, i] = e / e.sum(-1, keepdims=True) @ v[g]
    return out.reshape(T, -1)


def window_latent(h, g, m, eps):
    """Latent attention whose keys and values are images of the normed latent alone, over a sliding window."""
    T = h.shape[0]
    heads = lambda x, d: x.reshape(T, m["heads"], d).transpose(1, 0, 2)
    c = rms_norm(h @ g("dkv").T, g("dkv.norm"), eps)
    return softmax_attention(heads(h @ g("q").T, m["dim"]), heads(c @ g("uk").T, m["dim"]), heads(c @ g("uv").T, m["vdim"]), m["scale"],
                             in_window(T, m["mask"]["size"])) @ g("o").T


def chunk_attention(h, g, m, eps, kv=None):
    """Grouped-query attention inside chunks; queries and keys are normed over the whole projection, then rotated.  `kv`: keys and
    values of another layer, used instead of projections of its own.  Returns the output and the keys and values it used."""
    T = h.shape[0]
    pos = np.arange(T, dtype=F)
    heads = lambda x, n, d: x.reshape(T, n, d).transpose(1, 0, 2)
    turn = lambda x: rotate_halves(x, pos, m["rot"]["base"], m["rot"]["dims"])
    q = turn(heads(rms_norm(h @ g("q").T, g("q.norm"), eps), m["heads"], m["dim"]))
    if kv is None:
        kv = (turn(heads(rms_norm(h @ g("k").T, g("k.norm"), eps), m["kv_heads"], m["dim"])), heads(h @ g("v").T, m["kv_heads"], m["vdim"]))
    return softmax_attention(q, kv[0], kv[1], m["scale"], in_chunk(T, m["mask"]["size"])) @ g("o").T, kv


def swiglu(h, g, p):
    return (silu(h @ g(p + "gate").T) * (h @ g(p + "up").T)) @ g(p + "down").T


def softmax_router(z, correction, top, scale):
    """z [T, outputs] -> weights [T, outputs], zero where not chosen: the correction moves the choice, not the weight."""
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    out = np.zeros_like(s)
    for t in range(len(z)):
        best = np.argsort(-(s[t] + correction), kind="stable")[:top]
        out[t, best] = s[t, best] / (s[t, best].sum() + 1e-20) * scale
    return out


def mixture(h, g, mlp):
    """Routed experts of which the last ones return their input, and a shared expert behind a gate."""
    r = mlp["router"]
    w = softmax_router(h @ g("router").T, g("correction"), r["top"], r["scale"])
    out = w[:, r["experts"]:].sum(1, keepdims=True) * h
    for e in range(r["experts"]):
        rows = np.nonzero(w[:, e])[0]
        if len(rows):
            out[rows] += w[rows, e:e + 1] * swiglu(h[rows], g, f"e{e}.")
    if mlp.get("shared"):
        out = out + sigmoid(h @ g("shared.sg").T) * swiglu(h, g, "shared.")
    return out


def connect(X, w, key, sublayer):
    """X [T, streams, width] -> the streams after one sub-layer: it reads a weighted sum, and its output goes to every stream
    beside a mixture ([from, to]) of the old ones."""
    y = sublayer(np.einsum("s,tsw->tw", w[key + "in"], X))
    return np.einsum("ab,taw->tbw", w[key + "mix"], X) + w[key + "out"][None, :, None] * y[:, None, :]


def forward_zokuzen(cfg, w, tokens, layers_out=None):
    eps = cfg["norm"]["eps"]
    X = np.repeat(w["embed"][np.asarray(tokens)].astype(F)[:, None, :], cfg["streams"], 1)
    stored = {}
    for i, L in enumerate(cfg["layers"]):
        mix = lambda n, i=i: w[f"l{i}.mix.{n}"]
        ff = lambda n, i=i: w[f"l{i}.mlp.{n}"]

        def mixer(u):
            h = rms_norm(u, 1.0 + w[f"l{i}.norm1"], eps)
            if L["type"] == "wkv":
                return time_mix(h, mix, L["mixer"], eps)
            if L["type"] == "latent_attention":
                return window_latent(h, mix, L["mixer"], eps)
            y, stored[i] = chunk_attention(h, mix, L["mixer"], eps, stored.get(L["mixer"].get("kv_from")))
            return y

        X = connect(X, w, f"l{i}.hc1.", mixer)
        if L.get("mlp"):
            X = connect(X, w, f"l{i}.hc2.", lambda u: mixture(rms_norm(u, 1.0 + w[f"l{i}.norm2"], eps), ff, L["mlp"]))
        if layers_out is not None:
            layers_out.append(X.sum(1))
    return rms_norm(X.sum(1), 1.0 + w["final.norm"], eps) @ w["embed"].T


# ---- Pokadra ---------------------------------------------------------------------------------------------------------
def embed_pairs(tokens, w, scale, pairs):
    """Token rows times `scale` plus one row per (previous, current) token; the first token takes the table's last row."""
    tokens = [int(t) for t in tokens]
    x = w["embed"][tokens].astype(F) * scale
    if pairs:
        rows = [pairs["buckets"]] + [(a * pairs["mul_prev"] + b * pairs["mul_cur"]) % pairs["buckets"] for a, b in zip(tokens, tokens[1:])]
        x = x + w["bigram"][rows]
    return x


def group_norm(x, w, groups, eps):
    """RMS norm of each of `groups` equal parts by itself, one weight over all."""
    return rms(x.reshape(x.shape[0], groups, -1), eps).reshape(x.shape) * w


def yarn_frequencies(rot):
    """-> (angle per position of every pair, factor of cos and sin)."""
    n, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    place = lambda turns: n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(place(s["fast"])), 0), min(math.ceil(place(s["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate_scaled(v, pos, rot):
    """v [..., T, d]: coordinates (2i, 2i+1) turned by the scaled frequencies."""
    freq, m = yarn_frequencies(rot)
    out = v.copy()
    for i, f in enumerate(freq):
        c, s = np.cos(pos * f) * m, np.sin(pos * f) * m
        out[..., 2 * i] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = v[..., 2 * i + 1] * c + v[..., 2 * i] * s
    return out


def in_window_or_first(T, size, keep):
    """visible[i, j]: j is i, one of the size - 1 tokens before it, or one of the sequence's first `keep`."""
    i, j = np.arange(T)[:, None], np.arange(T)[None]
    return (j <= i) & ((i - j < size) | (j < keep))


def difference_weight(lq1, lk1, lq2, lk2, base):
    return float(np.exp((lq1 * lk1).sum()) - np.exp((lq2 * lk2).sum()) + base)


def differential_attention(h, g, m, eps, kv=None):
    """Two softmax maps per head over the same values; the second one, weighted, is taken off the first; the difference is normed
    per head and gated by one number per head.  Returns the output and the keys and values it used."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T, dtype=F)
    maps = lambda x, n, w: rotate_scaled(rms_norm(x.reshape(T, n, 2, D), w, eps).transpose(1, 2, 0, 3), pos, m["rot"])  # [n, 2, T, D]
    q = maps(h @ g("q").T, H, g("q.norm"))
    if kv is None:
        kv = (maps(h @ g("k").T, G, g("k.norm")), (h @ g("v").T).reshape(T, G, V).transpose(1, 0, 2))
    mask = m.get("mask")
    visible = in_window_or_first(T, mask["size"], mask["keep_first"]) if mask else in_window(T, T + 1)
    a = [softmax_attention(q[:, i], kv[0][:, i], kv[1], m["scale"], visible).reshape(T, H, V) for i in (0, 1)]
    o = a[0] - difference_weight(g("lq1"), g("lk1"), g("lq2"), g("lk2"), m["diff"]) * a[1]
    o = rms(o, eps) * (1.0 - m["diff"]) * sigmoid(h @ g("g").T)[:, :, None]
    return o.reshape(T, H * V) @ g("o").T, kv


def gated_average(z, c):
    """S_t = (1 - z_t) S_(t-1) + z_t c_t from zero, all [T, width]."""
    S, out = np.zeros(z.shape[1], F), np.zeros_like(z)
    for t in range(len(z)):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return out


def min_gru(h, g, m, eps):
    u = h @ g("x").T + g("x.b")
    S = gated_average(sigmoid(h @ g("z").T + g("z.b")), np.where(u >= 0, u + 0.5, sigmoid(u)))
    return (S * silu(h @ g("g").T)) @ g("o").T


def clipped_ff(h, g, limit):
    a, u = np.minimum(h @ g("gate").T, limit), np.clip(h @ g("up").T, -limit, limit)
    return (a * sigmoid(1.702 * a) * (u + 1.0)) @ g("down").T


def token_input(x, e, g, eps):
    """What a token's own row e of the layer adds, gated by the stream."""
    return rms_norm((gelu_tanh(x @ g("gate").T) * e) @ g("proj").T, g("norm"), eps)


def forward_pokadra(cfg, w, tokens, layers_out=None):
    eps, m, groups = cfg["norm"]["eps"], cfg["residual_mult"], cfg["norm"]["groups"]
    x = embed_pairs(tokens, w, cfg["embedding"]["scale"], cfg["embedding"].get("bigram"))
    before, stored, side = [x], {}, cfg.get("token_side")
    for i, L in enumerate(cfg["layers"]):
        part = lambda p, i=i: lambda n: w[f"l{i}.{p}.{n}"]
        if L["type"] == "mingru":
            y = min_gru(x, part("mix"), L["mixer"], eps)
        else:
            y, stored[i] = differential_attention(x, part("mix"), L["mixer"], eps, stored.get(L["mixer"].get("kv_from")))
        x = x + m * group_norm(y, w[f"l{i}.norm1"], groups, eps)
        if L.get("mlp"):
            x = x + m * group_norm(clipped_ff(x, part("mlp"), L["mlp"]["limit"]), w[f"l{i}.norm2"], groups, eps)
        if side:
            n = side["dim"]
            x = x + m * token_input(x, w["side.embed"][np.asarray(tokens), i * n:(i + 1) * n], part("side"), eps)
        before.append(x)
        x = sum(c * X for c, X in zip(w[f"l{i}.dwa"], before))
        if layers_out is not None:
            layers_out.append(x.copy())
    return group_norm(x, w["final.norm"], groups, eps) @ w["head"].T


def layer_runs(cfg):
    """(layer, pass) in the order they run; pass is -1 outside the repeated stretch."""
    n, loop = len(cfg["layers"]), cfg.get("loop") or dict(start=0, stop=0, times=0)
    a, b = loop["start"], loop["stop"]
    return [(i, -1) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)] + [(i, -1) for i in range(b, n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  layers_out (a list) receives the residual stream after every layer run."""
    by_name = {"Zukitar": forward_zukitar, "Tirezen": forward_tirezen, "Zokuzen": forward_zokuzen, "Pokadra": forward_pokadra}
    return by_name[cfg["architecture"]](cfg, w, tokens, layers_out)


def forward_tirezen(cfg, w, tokens, layers_out=None):
    """Parallel layers (one norm, mixer and feed-forward both read it), norm weights around zero, a stretch of layers that runs
    several times, an output projection of its own."""
    eps = cfg["norm"]["eps"]
    first = w["embed"][np.asarray(tokens)].astype(F)
    x = first
    for i, t in layer_runs(cfg):
        L = cfg["layers"][i]
        if t >= 0 and i == cfg["loop"]["start"]:
            x = x + w["loop.step"][t] + (first if t > 0 else 0.0)
        mix = lambda n, i=i: w[f"l{i}.mix.{n}"]
        h = rms_norm(x, 1.0 + w[f"l{i}.norm1"], eps)
        y = MIXERS[L["type"]](h, mix, L["mixer"], eps)
        if L.get("mlp"):
            y = y + plain_ff(h, lambda n, i=i: w[f"l{i}.mlp.{n}"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, 1.0 + w["final.norm"], eps) @ w["head"].T


def forward_zukitar(cfg, w, tokens, layers_out=None):
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
