// Minimal gated recurrence: S <- (1 - z) S + z c element by element, z and c from the current token alone; the output is S silu(G).
// State and everything that enters it in f32.
//
// Portions of a few tokens go token by token, the state in registers.  Longer ones in 64-token chunks: what a stretch of tokens does to
// the state is S -> A S + B with A = prod (1 - z).  One kernel forms A and B of every chunk but the last; a second one folds the chunks
// ahead of each, and walks it with a warp per eight tokens, whose own A and B tell the next warps where they start.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

constexpr int kWarps = 8, kTokens = kMemoryChunk / kWarps, kCols = 64;  // of a chunk's block: warps, tokens of each, channels (two per lane)

template <typename T>
struct Pair;  // two channels as stored
template <>
struct Pair<uint16_t> {
    uint32_t u;
    __device__ __forceinline__ void ld(const uint16_t* p) { u = *reinterpret_cast<const uint32_t*>(p); }
    __device__ __forceinline__ float x() const { return bflo(u); }
    __device__ __forceinline__ float y() const { return bfhi(u); }
    static __device__ __forceinline__ void st(uint16_t* p, float x, float y) { *reinterpret_cast<uint32_t*>(p) = pack_bf2(x, y); }
};
template <>
struct Pair<float> {
    float2 u;
    __device__ __forceinline__ void ld(const float* p) { u = *reinterpret_cast<const float2*>(p); }
    __device__ __forceinline__ float x() const { return u.x; }
    __device__ __forceinline__ float y() const { return u.y; }
    static __device__ __forceinline__ void st(float* p, float x, float y) { *reinterpret_cast<float2*>(p) = make_float2(x, y); }
};
// ... with the fast exponential and division where the inputs are bf16
template <typename T>
__device__ __forceinline__ float sigmoid_for(float x) {
    return sizeof(T) == 2 ? __fdividef(1.0f, 1.0f + __expf(-x)) : sigmoid_f32(x);
}
template <typename T>
__device__ __forceinline__ float candidate(float u) {
    return u >= 0.f ? u + 0.5f : sigmoid_for<T>(u);
}
// a stretch of tokens, two channels: S -> a S + b
struct Stretch {
    float2 a, b;
    __device__ __forceinline__ void then(const float2& a2, const float2& b2) {
        b.x = fmaf(a2.x, b.x, b2.x), b.y = fmaf(a2.y, b.y, b2.y);
        a.x *= a2.x, a.y *= a2.y;
    }
    __device__ __forceinline__ float2 of(float2 s) const { return make_float2(fmaf(a.x, s.x, b.x), fmaf(a.y, s.y, b.y)); }
};
__device__ __forceinline__ void step(float2& S, const float2& z, const float2& c) {
    S.x = fmaf(z.x, c.x - S.x, S.x);
    S.y = fmaf(z.y, c.y - S.y, S.y);
}
__device__ __forceinline__ int channels(int width) { return (width + 7) / 8 * 8; }  // with the padding, whose inputs are zero
__device__ __forceinline__ void put_state(float* s, int c, int width, float2 v) {
    if (c < width) s[c] = v.x;
    if (c + 1 < width) s[c + 1] = v.y;
}
__device__ __forceinline__ float2 get_state(const float* s, int c, int width) { return make_float2(c < width ? s[c] : 0.f, c + 1 < width ? s[c + 1] : 0.f); }

template <typename T>
__global__ void __launch_bounds__(128) gated_average_scan_kernel(const GatedAverageParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int c = (blockIdx.x * 128 + threadIdx.x) * 2, b = blockIdx.y;
    const int start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start;
    if (n <= 0 || (p.n_chunks > 0 && n >= kMemoryChunkMin) || c >= p.ldo) return;
    T* out = reinterpret_cast<T*>(p.out) + (size_t)start * p.ldo + c;
    if (c >= channels(p.width)) {
        for (int t = 0; t < n; t++) Pair<T>::st(out + (size_t)t * p.ldo, 0.f, 0.f);
        return;
    }
    const T* in = reinterpret_cast<const T*>(p.in) + (size_t)start * p.ld + c;
    float* state = p.state + (size_t)p.seq_slot[b] * p.slot_stride;
    const float2 bz = *reinterpret_cast<const float2*>(p.z_bias + c), bu = *reinterpret_cast<const float2*>(p.u_bias + c);
    float2 S = p.context_lens[b] > n ? get_state(state, c, p.width) : make_float2(0.f, 0.f);
    for (int t = 0; t < n; t++, in += p.ld, out += p.ldo) {
        Pair<T> z, u, g;
        z.ld(in + p.z_off);
        u.ld(in + p.u_off);
        g.ld(in + p.g_off);
        step(S, make_float2(sigmoid_for<T>(z.x() + bz.x), sigmoid_for<T>(z.y() + bz.y)), make_float2(candidate<T>(u.x() + bu.x), candidate<T>(u.y() + bu.y)));
        Pair<T>::st(out, S.x * g.x() * sigmoid_for<T>(g.x()), S.y * g.y() * sigmoid_for<T>(g.y()));
    }
    put_state(state, c, p.width, S);
}

struct Chunk {
    int b, first, n, t0, cnt;  // its sequence, that one's first chunk, tokens of the portion, the chunk's first token in it, its tokens
};
__device__ __forceinline__ Chunk find_chunk(const GatedAverageParams& p, int chunk) {
    int b = -1;  // the last chunked portion that starts at or before this chunk (starts rise with the index)
    for (int i = threadIdx.x & 31; i < p.B; i += 32)
        if (p.chunk_off[i] >= 0 && p.chunk_off[i] <= chunk) b = i;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) b = max(b, __shfl_xor_sync(0xffffffffu, b, o));
    Chunk k{b, 0, 0, 0, 0};
    if (b < 0) return k;
    k.first = p.chunk_off[b];
    k.n = p.cu_seqlens[b + 1] - p.cu_seqlens[b];
    k.t0 = (chunk - k.first) * kMemoryChunk;
    k.cnt = min(kMemoryChunk, k.n - k.t0);
    return k;
}
// Gates and candidates of a warp's tokens; tokens past `cnt` leave the state alone.
template <typename T>
__device__ __forceinline__ Stretch warp_inputs(const GatedAverageParams& p, int c, size_t tok, int cnt, float2 (&z)[kTokens], float2 (&u)[kTokens]) {
    const T* in = reinterpret_cast<const T*>(p.in) + tok * p.ld + c;
    const float2 bz = *reinterpret_cast<const float2*>(p.z_bias + c), bu = *reinterpret_cast<const float2*>(p.u_bias + c);
    Pair<T> zr[kTokens], ur[kTokens];
#pragma unroll
    for (int k = 0; k < kTokens; k++)
        if (k < cnt) {
            zr[k].ld(in + (size_t)k * p.ld + p.z_off);
            ur[k].ld(in + (size_t)k * p.ld + p.u_off);
        }
    Stretch s{make_float2(1.f, 1.f), make_float2(0.f, 0.f)};
#pragma unroll
    for (int k = 0; k < kTokens; k++) {
        z[k] = u[k] = make_float2(0.f, 0.f);
        if (k < cnt) {
            z[k] = make_float2(sigmoid_for<T>(zr[k].x() + bz.x), sigmoid_for<T>(zr[k].y() + bz.y));
            u[k] = make_float2(candidate<T>(ur[k].x() + bu.x), candidate<T>(ur[k].y() + bu.y));
        }
        s.a.x *= 1.f - z[k].x;
        s.a.y *= 1.f - z[k].y;
        step(s.b, z[k], u[k]);
    }
    return s;
}
// Record of a chunk: A and B, [channels] each.  For a portion's first chunk the kept state stands in A's place: the second kernel's
// last chunk replaces the kept one while the first may still need it.
template <typename T>
__global__ void __launch_bounds__(kWarps * 32) gated_average_chunk_kernel(const GatedAverageParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    __shared__ Stretch parts[kWarps][32];
    const int chunk = blockIdx.y, W = channels(p.width), warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c = blockIdx.x * kCols + lane * 2;
    const Chunk k = find_chunk(p, chunk);
    if (k.cnt <= 0 || k.t0 + k.cnt >= k.n) return;  // (nothing follows a portion's last chunk)
    if (c < W) {
        float2 z[kTokens], u[kTokens];
        parts[warp][lane] = warp_inputs<T>(p, c, (size_t)p.cu_seqlens[k.b] + k.t0 + warp * kTokens, kTokens, z, u);
    }
    __syncthreads();
    if (warp > 0 || c >= W) return;
    Stretch s = parts[0][lane];
#pragma unroll
    for (int i = 1; i < kWarps; i++) s.then(parts[i][lane].a, parts[i][lane].b);
    if (chunk == k.first) {
        const float2 S0 = p.context_lens[k.b] > k.n ? get_state(p.state + (size_t)p.seq_slot[k.b] * p.slot_stride, c, p.width) : make_float2(0.f, 0.f);
        s.b = s.of(S0);
        s.a = S0;
    }
    float* rec = p.chunk + (size_t)chunk * 2 * W + c;
    *reinterpret_cast<float2*>(rec) = s.a;
    *reinterpret_cast<float2*>(rec + W) = s.b;
}
template <typename T>
__global__ void __launch_bounds__(kWarps * 32) gated_average_walk_kernel(const GatedAverageParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    __shared__ Stretch parts[kWarps][32], ahead[kWarps][32];
    const int chunk = blockIdx.y, W = channels(p.width), warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c = blockIdx.x * kCols + lane * 2;
    const Chunk k = find_chunk(p, chunk);
    if (k.cnt <= 0) return;
    const int cnt = min(max(k.cnt - warp * kTokens, 0), kTokens);
    const size_t tok = (size_t)p.cu_seqlens[k.b] + k.t0 + warp * kTokens;
    T* out = reinterpret_cast<T*>(p.out) + tok * p.ldo + c;
    float* state = p.state + (size_t)p.seq_slot[k.b] * p.slot_stride;
    float2 z[kTokens], u[kTokens], S = make_float2(0.f, 0.f);
    Pair<T> g[kTokens];
    if (c < W) {
        if (k.n <= kMemoryChunk && p.context_lens[k.b] > k.n) S = get_state(state, c, p.width);  // the only chunk, which replaces it below
        const T* in = reinterpret_cast<const T*>(p.in) + tok * p.ld + p.g_off + c;
#pragma unroll
        for (int i = 0; i < kTokens; i++)
            if (i < cnt) g[i].ld(in + (size_t)i * p.ld);
        parts[warp][lane] = warp_inputs<T>(p, c, tok, cnt, z, u);
        // the chunks ahead, shared out among the warps; the first one's record holds the state behind it
        Stretch s{make_float2(1.f, 1.f), make_float2(0.f, 0.f)};
        const int before = chunk - k.first, per = (before + kWarps - 1) / kWarps, end = min(before, (warp + 1) * per);
        const float* rec = p.chunk + (size_t)k.first * 2 * W + c;
#pragma unroll 8
        for (int i = warp * per; i < end; i++) {
            const float2 a = *reinterpret_cast<const float2*>(rec + (size_t)i * 2 * W);
            s.then(i == 0 ? make_float2(0.f, 0.f) : a, *reinterpret_cast<const float2*>(rec + (size_t)i * 2 * W + W));
        }
        ahead[warp][lane] = s;
    }
    __syncthreads();
    if (c >= W) {
        if (c < p.ldo)
            for (int i = 0; i < cnt; i++) Pair<T>::st(out + (size_t)i * p.ldo, 0.f, 0.f);
        return;
    }
    if (chunk > k.first) {
#pragma unroll
        for (int i = 0; i < kWarps; i++) S = ahead[i][lane].of(S);
    } else if (k.n > kMemoryChunk) {
        S = *reinterpret_cast<const float2*>(p.chunk + (size_t)k.first * 2 * W + c);
    }
    for (int i = 0; i < warp; i++) S = parts[i][lane].of(S);
#pragma unroll
    for (int i = 0; i < kTokens; i++)
        if (i < cnt) {
            step(S, z[i], u[i]);
            Pair<T>::st(out + (size_t)i * p.ldo, S.x * g[i].x() * sigmoid_for<T>(g[i].x()), S.y * g[i].y() * sigmoid_for<T>(g[i].y()));
        }
    if (k.t0 + k.cnt == k.n && cnt > 0 && k.cnt <= (warp + 1) * kTokens) put_state(state, c, p.width, S);
}

template <typename T>
int32_t launch(b2_ctx* ctx, const GatedAverageParams& p) {
    const int W = (p.width + 7) / 8 * 8;
    B2_REQUIRE(p.B <= 65535 && p.n_chunks <= 65535, B2_ERR_UNSUPPORTED, "gated average: too many sequences in one step");
    if (p.n_short > 0) {
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gated_average_scan_kernel<T>, dim3((p.ldo + 255) / 256, p.B), dim3(128), 0, ctx->stream, p));
        B2_LAUNCHED(ctx);
    }
    if (p.n_long > 0) {
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gated_average_chunk_kernel<T>, dim3((W + kCols - 1) / kCols, p.n_chunks), dim3(kWarps * 32), 0, ctx->stream, p));
        B2_LAUNCHED(ctx);
    }
    if (p.n_chunks > 0) {
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gated_average_walk_kernel<T>, dim3((p.ldo + kCols - 1) / kCols, p.n_chunks), dim3(kWarps * 32), 0, ctx->stream, p));
        B2_LAUNCHED(ctx);
    }
    return B2_OK;
}

}  // namespace

size_t b2_gated_average_chunk_floats(int width) { return (size_t)(width + 7) / 8 * 8 * 2; }
int32_t b2_gated_average_launch(b2_ctx* ctx, bool f32, const GatedAverageParams& p) {
    if (p.T <= 0) return B2_OK;
    return f32 ? launch<float>(ctx, p) : launch<uint16_t>(ctx, p);
}
