"""Seeded synthetic serving workloads and model shapes of the benchmark configurations.

Llama-3-8B-architecture continuous batching: 2048 requests, Poisson
arrivals at 50 req/s, prompt lengths lognormal with median 512 (sigma 1.0 — not given by the
configuration, chosen here) clipped to [16, 8192], output lengths uniform in [64, 512], prompt token
ids uniform over the vocabulary.  No public dataset is involved.
"""
import numpy as np

LLAMA3_8B = dict(num_layers=32, hidden_size=4096, num_heads=32, num_kv_heads=8, head_dim=128, intermediate_size=14336,
                 vocab_size=128256, rms_norm_eps=1e-5, rope_theta=500000.0, rope_kind=1, rope_factor=8.0, rope_low_freq_factor=1.0,
                 rope_high_freq_factor=4.0, rope_original_context=8192.0, qk_norm=0)
QWEN3_32B = dict(num_layers=64, hidden_size=5120, num_heads=64, num_kv_heads=8, head_dim=128, intermediate_size=25600,
                 vocab_size=151936, rms_norm_eps=1e-6, rope_theta=1000000.0, rope_kind=0, rope_factor=1.0, rope_low_freq_factor=1.0,
                 rope_high_freq_factor=4.0, rope_original_context=8192.0, qk_norm=1)
# a 4-layer cut of the 8B shape for quick checks (same per-layer kernels and tile shapes)
LLAMA3_8B_4L = dict(LLAMA3_8B, num_layers=4)


def serving_requests(n=2048, seed=0, rate=50.0, vocab=128256, median_prompt=512, sigma=1.0, min_prompt=16, max_prompt=8192,
                     min_out=64, max_out=512, poisson=True):
    """Returns (prompts [list of int32 arrays], max_new [n], arrival_s [n])."""
    rng = np.random.default_rng(seed)
    plen = np.clip(np.rint(np.exp(rng.normal(np.log(median_prompt), sigma, size=n))), min_prompt, max_prompt).astype(np.int64)
    out = rng.integers(min_out, max_out + 1, size=n).astype(np.int64)
    arrival = np.cumsum(rng.exponential(1.0 / rate, size=n)) if poisson else np.zeros(n)
    prompts = [rng.integers(0, vocab, size=int(p), dtype=np.int32) for p in plen]
    return prompts, out, arrival


def long_context_requests(n=512, seed=0, vocab=151936, min_prompt=1024, max_prompt=32768, max_new=256):
    """n sequences, prompt lengths uniform in [min_prompt, max_prompt], max_new outputs each,
    all present at time 0.  Returns (prompts, max_new [n], arrival_s [n])."""
    rng = np.random.default_rng(seed)
    plen = rng.integers(min_prompt, max_prompt + 1, size=n)
    prompts = [rng.integers(0, vocab, size=int(p), dtype=np.int32) for p in plen]
    return prompts, np.full(n, max_new, np.int64), np.zeros(n)


def projection_params(cfg):
    """Weights every token is multiplied with in the projections (per token: 2 flops each)."""
    h, qd, kvd, i = cfg["hidden_size"], cfg["num_heads"] * cfg["head_dim"], cfg["num_kv_heads"] * cfg["head_dim"], cfg["intermediate_size"]
    return cfg["num_layers"] * (h * (qd + 2 * kvd) + qd * h + 3 * h * i)


def step_weight_bytes(cfg, bits):
    """Bytes of weights one decode step streams: projections (quantized: bits/8 + 4 bytes per 64-group)
    plus the bf16 lm_head."""
    p = projection_params(cfg)
    per = bits / 8.0 + 4.0 / 64.0 if bits else 2.0
    return p * per + cfg["vocab_size"] * cfg["hidden_size"] * 2


def kv_bytes_per_token(cfg):
    return cfg["num_layers"] * 2 * cfg["num_kv_heads"] * cfg["head_dim"] * 2


# Layered design (latent attention + dense feed-forward, Mamba-2 + routed experts, alternating) at sizes of real models, and
# the flat decoder of equal width it is measured beside.
LAYERED_SIZES = {
    "w4096": dict(width=4096, latent=dict(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512), ff=14336,
                  mamba=dict(heads=128, vdim=64, state=128, groups=8, norm_groups=8, conv=4), experts=32, top=4, expert_ff=1792),
    "w2048": dict(width=2048, latent=dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512), ff=8192,
                  mamba=dict(heads=64, vdim=64, state=128, groups=4, norm_groups=4, conv=4), experts=32, top=4, expert_ff=1024),
}


def layered_config(size, pairs, vocab=32000):
    s = LAYERED_SIZES[size]
    lat = dict(s["latent"], rot=dict(base=500000.0, dims=s["latent"]["rot_dim"]), scale=(s["latent"]["dim"] + s["latent"]["rot_dim"]) ** -0.5)
    moe = dict(kind="moe", expert=dict(ff=s["expert_ff"], limit=7.0), router=dict(experts=s["experts"], top=s["top"]))
    layers = [dict(type="latent_attention", mixer=lat, mlp=dict(kind="dense", ff=s["ff"])), dict(type="mamba2", mixer=s["mamba"], mlp=moe)] * pairs
    return dict(architecture="Zukitar", width=s["width"], vocab=vocab, norm=dict(eps=1e-5), logit_scale=1.0, layers=layers)


# Tirezen at the same widths: half of the layers with capped sink attention beside a delta memory, the others retention and
# delta memories in turn; the feed-forward has the flat twin's inner size.
TIREZEN_SIZES = {
    "w4096": dict(heads=32, kv_heads=8, memory=dict(heads=32, kv_heads=32), delta=dict(heads=32, kv_heads=16)),
    "w2048": dict(heads=16, kv_heads=4, memory=dict(heads=16, kv_heads=16), delta=dict(heads=16, kv_heads=8)),
}


def tirezen_config(size, layers, vocab=32000):
    s, t = LAYERED_SIZES[size], TIREZEN_SIZES[size]
    left = dict(heads=t["heads"], kv_heads=t["kv_heads"], dim=128, vdim=128, rot=dict(base=500000.0, dims=128), scale=128 ** -0.5, softcap=30.0)
    sides = dict(left=left, right=dict(t["memory"], dim=128, vdim=128, conv=4), left_scale=0.5, right_scale=0.5)
    retention = dict(heads=t["heads"], dim=128, vdim=128, rot=dict(base=500000.0, dims=128), decay=[1.0 - 2.0 ** -(5 + i % 7) for i in range(t["heads"])])
    mixers = [("parallel", sides), ("retention", retention), ("parallel", sides), ("delta", dict(t["delta"], dim=128, vdim=128, conv=4))]
    mlp = dict(kind="dense", ff=s["ff"])
    return dict(architecture="Tirezen", width=s["width"], vocab=vocab, norm=dict(eps=1e-5),
                layers=[dict(type=mixers[i % 4][0], mixer=mixers[i % 4][1], mlp=mlp) for i in range(layers)])


# Zokuzen at the same widths: time mixing, windowed latent attention, time mixing, chunked attention, repeated; every second chunked
# layer reads the keys of the one before it; experts whose active part (chosen and shared) has the flat twin's inner size.
ZOKUZEN_SIZES = {
    "w4096": dict(wkv=dict(heads=64, dim=64), latent=dict(heads=32, dim=128, vdim=128, kv_rank=512), heads=32, kv_heads=8, expert_ff=1792, shared_ff=7168),
    "w2048": dict(wkv=dict(heads=32, dim=64), latent=dict(heads=16, dim=128, vdim=128, kv_rank=512), heads=16, kv_heads=4, expert_ff=1024, shared_ff=4096),
}


def zokuzen_config(size, layers, vocab=32000, streams=4):
    z, width = ZOKUZEN_SIZES[size], LAYERED_SIZES[size]["width"]
    latent = dict(z["latent"], scale=z["latent"]["dim"] ** -0.5, mask=dict(size=4096))
    attn = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=128, vdim=128, rot=dict(base=500000.0, dims=128), scale=128 ** -0.5, mask=dict(size=8192))
    mlp = dict(kind="moe", expert=dict(ff=z["expert_ff"]), router=dict(experts=32, identity=4, top=4, scale=2.0), shared=dict(ff=z["shared_ff"]))
    mixers = [("wkv", z["wkv"]), ("latent_attention", latent), ("wkv", z["wkv"]), ("attention", attn)]

    def mixer(i):
        kind, m = mixers[i % 4]
        return dict(type=kind, mixer=dict(m, kv_from=i - 4) if kind == "attention" and i // 4 % 2 else m, mlp=mlp)

    return dict(architecture="Zokuzen", width=width, vocab=vocab, norm=dict(eps=1e-5), streams=streams, layers=[mixer(i) for i in range(layers)])


# Pokadra at the same widths: differential attention (the flat twin's projections: two maps of half its key size) and minimal gated
# recurrences of the model's width in turn; every second attention layer reads the keys of the one before it; the flat twin's feed-forward.
POKADRA_SIZES = {
    "w4096": dict(heads=32, kv_heads=8, side=256),
    "w2048": dict(heads=16, kv_heads=4, side=128),
}


def pokadra_config(size, layers, vocab=32000):
    s, p = LAYERED_SIZES[size], POKADRA_SIZES[size]
    rot = dict(base=500000.0, dims=64, scaling=dict(factor=4.0, original=8192, fast=24.0, slow=2.0))
    attn = dict(heads=p["heads"], kv_heads=p["kv_heads"], dim=64, vdim=128, diff=0.4, rot=rot, scale=64 ** -0.5, mask=dict(size=4096, keep_first=64))
    mlp = dict(kind="dense", ff=s["ff"], limit=7.0)

    def layer(i):
        if i % 2:
            return dict(type="mingru", mixer=dict(width=s["width"]), mlp=mlp)
        return dict(type="attention", mixer=dict(attn, kv_from=i - 2) if i % 4 else attn, mlp=mlp)

    return dict(architecture="Pokadra", width=s["width"], vocab=vocab, norm=dict(eps=1e-5, groups=8), residual_mult=0.5, token_side=dict(dim=p["side"]),
                embedding=dict(scale=1.0, bigram=dict(buckets=16381, mul_prev=8191, mul_cur=127)), layers=[layer(i) for i in range(layers)])


def flat_twin(size, layers, vocab=32000):
    """Llama-architecture model of the same width, feed-forward and layer count, dense bf16."""
    s = LAYERED_SIZES[size]
    hq = s["width"] // 128
    return dict(num_layers=layers, hidden_size=s["width"], num_heads=hq, num_kv_heads=max(hq // 4, 1), head_dim=128, intermediate_size=s["ff"],
                vocab_size=vocab, rms_norm_eps=1e-5, rope_theta=500000.0)
