// Minimal gated recurrence: S <- (1 - z) S + z c element by element, z and c from the current token alone; the output is S silu(G).
// State and everything that enters it in f32.
//
// Portions of a few tokens go token by token, the state in registers.  Longer ones in 64-token chunks: what a chunk does to the state is
// S -> A S + B, so one kernel forms A = prod (1 - z) and B of every chunk but the last, and a second one takes each chunk's first state
// from the chunks ahead of it and walks its tokens.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

constexpr int kBatch = 8;  // tokens whose inputs are on their way together

template <typename T>
__device__ __forceinline__ float2 ld_pair(const T* p) {
    if constexpr (sizeof(T) == 2) {
        const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
        return make_float2(bflo(u), bfhi(u));
    } else {
        return *reinterpret_cast<const float2*>(p);
    }
}
template <typename T>
__device__ __forceinline__ float sigmoid_for(float x) {
    return sizeof(T) == 2 ? __fdividef(1.0f, 1.0f + __expf(-x)) : sigmoid_f32(x);
}
__device__ __forceinline__ float candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoid_f32(u); }

// Two channels of a thread over tokens [tok0, tok0 + n): OUT writes the outputs; otherwise `a` collects prod (1 - z).
template <typename T, bool OUT>
__device__ __forceinline__ void walk(const GatedAverageParams& p, int c, size_t tok0, int n, float2& S, float2& a) {
    const T* in = reinterpret_cast<const T*>(p.in) + tok0 * p.ld + c;
    T* out = reinterpret_cast<T*>(p.out) + tok0 * p.ldo + c;
    const float2 bz = *reinterpret_cast<const float2*>(p.z_bias + c), bu = *reinterpret_cast<const float2*>(p.u_bias + c);
    for (int t0 = 0; t0 < n; t0 += kBatch) {
        float2 z[kBatch], u[kBatch], g[kBatch];
#pragma unroll
        for (int k = 0; k < kBatch; k++)
            if (t0 + k < n) {
                const T* x = in + (size_t)(t0 + k) * p.ld;
                z[k] = ld_pair(x + p.z_off);
                u[k] = ld_pair(x + p.u_off);
                if constexpr (OUT) g[k] = ld_pair(x + p.g_off);
            }
#pragma unroll
        for (int k = 0; k < kBatch; k++)
            if (t0 + k < n) {
                const float zx = sigmoid_f32(z[k].x + bz.x), zy = sigmoid_f32(z[k].y + bz.y);
                S.x = fmaf(zx, candidate(u[k].x + bu.x) - S.x, S.x);
                S.y = fmaf(zy, candidate(u[k].y + bu.y) - S.y, S.y);
                if constexpr (OUT) {
                    const float ox = S.x * g[k].x * sigmoid_for<T>(g[k].x), oy = S.y * g[k].y * sigmoid_for<T>(g[k].y);
                    T* o = out + (size_t)(t0 + k) * p.ldo;
                    if constexpr (sizeof(T) == 2)
                        *reinterpret_cast<uint32_t*>(o) = pack_bf2(ox, oy);
                    else
                        *reinterpret_cast<float2*>(o) = make_float2(ox, oy);
                } else {
                    a.x *= 1.f - zx;
                    a.y *= 1.f - zy;
                }
            }
    }
}
template <typename T>
__device__ __forceinline__ void zeros(const GatedAverageParams& p, int c, size_t tok0, int n) {
    T* out = reinterpret_cast<T*>(p.out) + tok0 * p.ldo + c;
    for (int t = 0; t < n; t++, out += p.ldo) Elt<T>::st(out, 0.f), Elt<T>::st(out + 1, 0.f);
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
    if (c >= channels(p.width)) return zeros<T>(p, c, start, n);
    float* state = p.state + (size_t)p.seq_slot[b] * p.slot_stride;
    float2 S = p.context_lens[b] > n ? get_state(state, c, p.width) : make_float2(0.f, 0.f), a;
    walk<T, true>(p, c, start, n, S, a);
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
// Record of a chunk: A and B, [channels] each.  A portion's first chunk starts from the kept state, which stands in A's place: the second
// kernel's last chunk replaces the kept one while others still need it.
template <typename T>
__global__ void __launch_bounds__(128) gated_average_chunk_kernel(const GatedAverageParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int chunk = blockIdx.y, W = channels(p.width), c = (blockIdx.x * 128 + threadIdx.x) * 2;
    const Chunk k = find_chunk(p, chunk);
    if (k.cnt <= 0 || k.t0 + k.cnt >= k.n || c >= W) return;  // (nothing follows a portion's last chunk)
    float2 S = make_float2(0.f, 0.f), a = make_float2(1.f, 1.f);
    const bool first = chunk == k.first;
    if (first && p.context_lens[k.b] > k.n) S = get_state(p.state + (size_t)p.seq_slot[k.b] * p.slot_stride, c, p.width);
    const float2 S0 = S;
    walk<T, false>(p, c, (size_t)p.cu_seqlens[k.b] + k.t0, k.cnt, S, a);
    float* rec = p.chunk + (size_t)chunk * 2 * W;
    *reinterpret_cast<float2*>(rec + c) = first ? S0 : a;
    *reinterpret_cast<float2*>(rec + W + c) = S;
}
template <typename T>
__global__ void __launch_bounds__(128) gated_average_walk_kernel(const GatedAverageParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int chunk = blockIdx.y, W = channels(p.width), c = (blockIdx.x * 128 + threadIdx.x) * 2;
    const Chunk k = find_chunk(p, chunk);
    if (k.cnt <= 0 || c >= p.ldo) return;
    const size_t tok0 = (size_t)p.cu_seqlens[k.b] + k.t0;
    if (c >= W) return zeros<T>(p, c, tok0, k.cnt);
    float* state = p.state + (size_t)p.seq_slot[k.b] * p.slot_stride;
    const float* rec = p.chunk + (size_t)k.first * 2 * W + c;
    float2 S = make_float2(0.f, 0.f), a;
    if (k.n <= kMemoryChunk) {  // the only chunk
        if (p.context_lens[k.b] > k.n) S = get_state(state, c, p.width);
    } else if (chunk == k.first) {
        S = *reinterpret_cast<const float2*>(rec);
    } else {
        S = *reinterpret_cast<const float2*>(rec + W);
        const int before = chunk - k.first;
#pragma unroll 4
        for (int i = 1; i < before; i++) {
            const float2 A = *reinterpret_cast<const float2*>(rec + (size_t)i * 2 * W), Bv = *reinterpret_cast<const float2*>(rec + (size_t)i * 2 * W + W);
            S.x = fmaf(A.x, S.x, Bv.x);
            S.y = fmaf(A.y, S.y, Bv.y);
        }
    }
    walk<T, true>(p, c, tok0, k.cnt, S, a);
    if (k.t0 + k.cnt == k.n) put_state(state, c, p.width, S);
}

template <typename T>
int32_t launch(b2_ctx* ctx, const GatedAverageParams& p) {
    const int blocks = (p.ldo + 255) / 256, inner = ((p.width + 7) / 8 * 8 + 255) / 256;
    B2_REQUIRE(p.B <= 65535 && p.n_chunks <= 65535, B2_ERR_UNSUPPORTED, "gated average: too many sequences in one step");
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gated_average_scan_kernel<T>, dim3(blocks, p.B), dim3(128), 0, ctx->stream, p));
    B2_LAUNCHED(ctx);
    if (p.n_chunks > 0) {
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gated_average_chunk_kernel<T>, dim3(inner, p.n_chunks), dim3(128), 0, ctx->stream, p));
        B2_LAUNCHED(ctx);
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gated_average_walk_kernel<T>, dim3(blocks, p.n_chunks), dim3(128), 0, ctx->stream, p));
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
