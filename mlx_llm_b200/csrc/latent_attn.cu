// Attention over a shared low-rank latent (one latent vector and one rotated key part per token, shared by all heads).
//
// The keys' and values' up-projections are absorbed into the query and the output: with k_h = Wk_h c and v_h = Wv_h c,
//     q_h . k_h = (Wk_h^T q_h) . c        sum_j p_j v_hj = Wv_h (sum_j p_j c_j)
// so attention runs over the cached rows [c | rotated key] themselves, as one key/value head shared by every query head.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

// One block per token: norm of the latent, rotation of the shared key part and of every head's rotated part, cache row
// and query buffers.
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentAttnSpec a, const LatentPrepParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    __shared__ float red[33];
    const int t = blockIdx.x, R = a.kv_rank, rot = a.rot_dim, dims = a.rot.dims, half = dims / 2, W = a.row_pad();
    const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld;
    const int pos = p.positions[t], slot = p.slot_mapping[t];
    const float* ct = p.cos_t + (size_t)pos * half;
    const float* st = p.sin_t + (size_t)pos * half;
    auto turned = [&](const T* v, int d) -> float {  // element d of the rotated vector v
        const float x = Elt<T>::ld(v + d);
        if (d >= dims) return x;
        const float c = ct[d >> 1], s = st[d >> 1], o = Elt<T>::ld(v + (d ^ 1));
        return (d & 1) ? x * c + o * s : x * c - o * s;
    };
    const T* lat = row + a.heads * (a.dim + rot);
    float ss = 0.f;
    for (int i = threadIdx.x; i < R; i += blockDim.x) {
        const float v = Elt<T>::ld(lat + i);
        ss += v * v;
    }
    ss = elt_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)R + p.eps);
    if (slot >= 0) {
        T* crow = reinterpret_cast<T*>(p.cache) + (size_t)slot * W;
        for (int i = threadIdx.x; i < W; i += blockDim.x)
            Elt<T>::st(crow + i, i < R ? Elt<T>::ld(lat + i) * inv * p.c_norm[i] : (i < R + rot ? turned(lat + R, i - R) : 0.f));
    }
    T* qn = reinterpret_cast<T*>(p.q_nope) + (size_t)t * a.heads * p.dim_pad;
    for (int i = threadIdx.x; i < a.heads * p.dim_pad; i += blockDim.x) {
        const int h = i / p.dim_pad, d = i - h * p.dim_pad;
        if (d < a.dim)
            qn[i] = row[h * (a.dim + rot) + d];
        else
            Elt<T>::st(qn + i, 0.f);
    }
    T* ql = reinterpret_cast<T*>(p.q_lat) + (size_t)t * a.heads * W;
    const int tail = W - R;
    for (int i = threadIdx.x; i < a.heads * tail; i += blockDim.x) {
        const int h = i / tail, d = i - h * tail;
        Elt<T>::st(ql + (size_t)h * W + R + d, d < rot ? turned(row + h * (a.dim + rot) + a.dim, d) : 0.f);
    }
}

// Plain form: one block per (token, head), 128 keys at a time with an online softmax, everything f32.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_simple_kernel(const LatentAttnSpec a, const LatentAttnParams p) {
    pdl_wait();
    extern __shared__ float sm[];  // q [W] | acc [R] | p [128]
    __shared__ float red[33];
    const int t = blockIdx.x, h = blockIdx.y, W = a.row_pad(), R = a.kv_rank;
    float *q = sm, *acc = sm + W, *pr = acc + R;
    const int n = p.positions[t] + 1;
    const int32_t* bt = p.block_tables + (size_t)p.seq_slot[p.token_seq[t]] * p.max_blocks;
    const T* cache = reinterpret_cast<const T*>(p.cache);
    const T* qr = reinterpret_cast<const T*>(p.q_lat) + ((size_t)t * a.heads + h) * W;
    for (int i = threadIdx.x; i < W; i += 128) q[i] = Elt<T>::ld(qr + i);
    for (int i = threadIdx.x; i < R; i += 128) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    __syncthreads();
    for (int j0 = 0; j0 < n; j0 += 128) {
        const int j = j0 + threadIdx.x, cnt = min(128, n - j0);
        float s = -INFINITY;
        if (j < n) {
            const T* k = cache + ((size_t)bt[j / p.page_size] * p.page_size + j % p.page_size) * W;
            float d = 0.f;
            for (int i = 0; i < W; i += 8) {
                float v[8];
                Elt<T>::ld8(k + i, v);
#pragma unroll
                for (int e = 0; e < 8; e++) d = fmaf(q[i + e], v[e], d);
            }
            s = d * a.scale;
        }
        float mx = elt_warp_max(s);
        __syncthreads();
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])), m);
        const float alpha = expf(m - mx), e = j < n ? expf(s - mx) : 0.f;
        pr[threadIdx.x] = e;
        l = l * alpha + elt_block_sum(e, red);
        m = mx;
        for (int i = threadIdx.x; i < R; i += 128) {
            float v = acc[i] * alpha;
            for (int jj = 0; jj < cnt; jj++) {
                const int key = j0 + jj;
                v = fmaf(pr[jj], Elt<T>::ld(cache + ((size_t)bt[key / p.page_size] * p.page_size + key % p.page_size) * W + i), v);
            }
            acc[i] = v;
        }
        __syncthreads();
    }
    T* o = reinterpret_cast<T*>(p.o_lat) + ((size_t)t * a.heads + h) * p.o_pad;
    for (int i = threadIdx.x; i < p.o_pad; i += 128) Elt<T>::st(o + i, i < R ? acc[i] / l : 0.f);
}

}  // namespace

int32_t b2_latent_prep_launch(b2_ctx* ctx, bool f32, const LatentAttnSpec& a, const LatentPrepParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? latent_prep_kernel<float> : latent_prep_kernel<uint16_t>, dim3(p.T), dim3(256), 0, ctx->stream, a, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_latent_attn_simple_launch(b2_ctx* ctx, bool f32, const LatentAttnSpec& a, const LatentAttnParams& p) {
    if (p.T <= 0) return B2_OK;
    const size_t smem = (size_t)(a.row_pad() + a.kv_rank + 128) * 4;
    B2_REQUIRE(smem <= 46 * 1024, B2_ERR_UNSUPPORTED, "latent attention: the latent is too wide");
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? latent_attn_simple_kernel<float> : latent_attn_simple_kernel<uint16_t>, dim3(p.T, a.heads), dim3(128), smem,
                          ctx->stream, a, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
