// Elementwise and normalisation steps of the layered models (residual stream in f32), in bf16 or f32 storage.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

template <typename T>
__global__ void embed_residual_kernel(const T* __restrict__ table, int ld_table, const int32_t* __restrict__ ids, int width, int vocab,
                                      float* __restrict__ x, int ldx, int copies) {
    pdl_wait();
    const int t = blockIdx.x;
    int id = ids[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = Elt<T>::ld(table + (size_t)id * ld_table + i);
        for (int c = 0; c < copies; c++) x[((size_t)t * copies + c) * ldx + i] = v;
    }
}

// x += y (one row, or the sum of several), then RMS norm, one block per row.  The row is kept in shared memory between
// the two passes.
template <typename T>
__global__ void add_norm_kernel(const AddNormParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const int r = blockIdx.x, t = p.row_idx ? p.row_idx[r] : r;
    float* xr = p.x + (size_t)t * p.ldx;
    const T* emb = nullptr;
    if (p.table) emb = reinterpret_cast<const T*>(p.table) + (size_t)min(max(p.ids[t], 0), p.vocab - 1) * p.ld_table;
    float ss = 0.f;
    const bool vec = p.width % 4 == 0 && p.ldx % 4 == 0 && p.ldy % 4 == 0;
    if (vec) {
        for (int i = threadIdx.x * 4; i < p.width; i += blockDim.x * 4) {
            float4 v = *reinterpret_cast<const float4*>(xr + i);
            for (int k = 0; k < p.n_src; k++) {
                const int yr = p.y_rows ? p.y_rows[(size_t)t * p.n_src + k] : t;
                const float4 a = *reinterpret_cast<const float4*>(p.y + (size_t)yr * p.ldy + i);
                v.x += a.x, v.y += a.y, v.z += a.z, v.w += a.w;
            }
            if (p.vec) {
                const float4 a = *reinterpret_cast<const float4*>(p.vec + i);
                v.x += a.x, v.y += a.y, v.z += a.z, v.w += a.w;
            }
            if (emb) {
                float a[4];
                Elt<T>::ld4(emb + i, a);
                v.x += a[0], v.y += a[1], v.z += a[2], v.w += a[3];
            }
            if (p.write_x) *reinterpret_cast<float4*>(xr + i) = v;
            *reinterpret_cast<float4*>(row + i) = v;
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int i = threadIdx.x; i < p.width; i += blockDim.x) {
            float v = xr[i];
            for (int k = 0; k < p.n_src; k++) v += p.y[(size_t)(p.y_rows ? p.y_rows[(size_t)t * p.n_src + k] : t) * p.ldy + i];
            if (p.vec) v += p.vec[i];
            if (emb) v += Elt<T>::ld(emb + i);
            if (p.write_x) xr[i] = v;
            row[i] = v;
            ss += v * v;
        }
    }
    if (!p.w) return;
    ss = elt_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)p.width + p.eps);
    T* o = reinterpret_cast<T*>(p.out) + (size_t)r * p.ldo;
    if (p.width % 8 == 0) {  // p.ldo is a multiple of 64
        for (int i = threadIdx.x * 8; i < p.ldo; i += blockDim.x * 8) {
            float v[8];
#pragma unroll
            for (int j = 0; j < 8; j++) v[j] = i < p.width ? row[i + j] * inv * p.w[i + j] * p.out_scale : 0.f;
            Elt<T>::st8(o + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < p.ldo; i += blockDim.x) Elt<T>::st(o + i, i < p.width ? row[i] * inv * p.w[i] * p.out_scale : 0.f);
    }
}

constexpr int kStreamSources = 64;  // rows of y whose numbers are kept in shared memory
// The streams' step, one block per token: VEC columns per thread with all streams in registers (NS: their number, rounded up).
template <typename T, int NS, int VEC>
__global__ void __launch_bounds__(NS <= 4 ? 1024 : 512) stream_norm_kernel(const StreamNormParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33], mix[NS][NS], to[NS], from[NS];
    __shared__ int src[kStreamSources];
    const int n = p.streams;
    for (int i = threadIdx.x; i < NS * NS; i += blockDim.x) {  // (weights: nothing earlier writes them)
        const int a = i / NS, b = i % NS;
        mix[a][b] = p.mix && a < n && b < n ? p.mix[a * n + b] : 0.f;
        if (a == 0) {
            to[b] = p.mix && b < n ? p.to[b] : 0.f;
            from[b] = b < n ? (p.from ? p.from[b] : 1.f) : 0.f;
        }
    }
    pdl_wait();
    const int r = blockIdx.x, t = p.row_idx ? p.row_idx[r] : r;
    float* xt = p.x + (size_t)t * n * p.ldx;
    const int n_src = p.mix ? p.n_src : 0;
    if ((int)threadIdx.x < min(n_src, kStreamSources)) src[threadIdx.x] = p.y_rows ? p.y_rows[(size_t)t * n_src + threadIdx.x] : t;
    __syncthreads();
    const float pass = p.mix && p.pass ? p.pass[t] : 0.f;
    const T* h = reinterpret_cast<const T*>(p.h) + (size_t)t * p.ldh;
    auto load = [](const float* s, float (&v)[VEC]) {
        if constexpr (VEC == 4)
            Elt<float>::ld4(s, v);
        else
            v[0] = s[0];
    };
    auto store = [](float* d, const float (&v)[VEC]) {
        if constexpr (VEC == 4)
            Elt<float>::st4(d, v);
        else
            d[0] = v[0];
    };
    float ss = 0.f;
    for (int i = threadIdx.x * VEC; i < p.width; i += blockDim.x * VEC) {
        float x[NS][VEC], u[VEC];
#pragma unroll
        for (int a = 0; a < NS; a++)
            if (a < n) load(xt + (size_t)a * p.ldx + i, x[a]);
#pragma unroll
        for (int e = 0; e < VEC; e++) u[e] = 0.f;
        if (p.mix) {
            float y[VEC];
#pragma unroll
            for (int e = 0; e < VEC; e++) y[e] = 0.f;
            constexpr int FLY = 2;  // sources on their way at a time
            for (int k0 = 0; k0 < n_src; k0 += FLY) {
                float v[FLY][VEC];
#pragma unroll
                for (int k = 0; k < FLY; k++) {
                    const int yr = k0 + k >= n_src ? -1 : k0 + k < kStreamSources ? src[k0 + k] : p.y_rows[(size_t)t * n_src + k0 + k];
                    if (yr >= 0)
                        load(p.y + (size_t)yr * p.ldy + i, v[k]);
                    else
#pragma unroll
                        for (int e = 0; e < VEC; e++) v[k][e] = 0.f;
                }
#pragma unroll
                for (int k = 0; k < FLY; k++)
#pragma unroll
                    for (int e = 0; e < VEC; e++) y[e] += v[k][e];
            }
            if (pass != 0.f) {
                float v[VEC];
                if constexpr (VEC == 4)
                    Elt<T>::ld4(h + i, v);
                else
                    v[0] = Elt<T>::ld(h + i);
#pragma unroll
                for (int e = 0; e < VEC; e++) y[e] = fmaf(pass, v[e], y[e]);
            }
#pragma unroll
            for (int b = 0; b < NS; b++) {
                if (b >= n) continue;
                float v[VEC];
#pragma unroll
                for (int e = 0; e < VEC; e++) v[e] = to[b] * y[e];
#pragma unroll
                for (int a = 0; a < NS; a++)
                    if (a < n)
#pragma unroll
                        for (int e = 0; e < VEC; e++) v[e] = fmaf(mix[a][b], x[a][e], v[e]);
                if (p.write_x) store(xt + (size_t)b * p.ldx + i, v);
#pragma unroll
                for (int e = 0; e < VEC; e++) u[e] = fmaf(from[b], v[e], u[e]);
            }
        } else {
#pragma unroll
            for (int a = 0; a < NS; a++)
                if (a < n)
#pragma unroll
                    for (int e = 0; e < VEC; e++) u[e] = fmaf(from[a], x[a][e], u[e]);
        }
        if (p.sum) store(p.sum + (size_t)r * p.ldx + i, u);
        store(row + i, u);
#pragma unroll
        for (int e = 0; e < VEC; e++) ss += u[e] * u[e];
    }
    if (!p.w) return;
    ss = elt_block_sum(ss, red);  // (every read of h is behind this barrier: out may be the same row)
    const float inv = 1.0f / sqrtf(ss / (float)p.width + p.eps);
    T* o = reinterpret_cast<T*>(p.out) + (size_t)r * p.ldo;
    if (p.width % 8 == 0) {  // p.ldo is a multiple of 64
        for (int i = threadIdx.x * 8; i < p.ldo; i += blockDim.x * 8) {
            float v[8];
#pragma unroll
            for (int j = 0; j < 8; j++) v[j] = i < p.width ? row[i + j] * inv * p.w[i + j] * p.out_scale : 0.f;
            Elt<T>::st8(o + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < p.ldo; i += blockDim.x) Elt<T>::st(o + i, i < p.width ? row[i] * inv * p.w[i] * p.out_scale : 0.f);
    }
}

__device__ __forceinline__ float gate_one(const GateSpec& gs, float g, float u) {
    if (gs.act == GateAct::GeluTanh) {
        const float k = 0.7978845608028654f;  // sqrt(2 / pi)
        return 0.5f * g * (1.0f + tanhf(k * (g + 0.044715f * g * g * g))) * u;
    }
    if (gs.act == GateAct::Swish) return silu_f32(g) * u;
    g = fminf(g, gs.limit);
    u = fminf(fmaxf(u, -gs.limit), gs.limit);
    return g * sigmoid_f32(gs.alpha * g) * (u + 1.0f);
}
template <typename T>
__global__ void gate_kernel(const GateSpec gs, const GateRows a, const GateRows b, int row0) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int row = row0 + blockIdx.y;
    const bool second = row >= a.rows;
    const GateRows& g = second ? b : a;
    const int r = second ? row - a.rows : row, i = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    if (i >= g.ldo) return;
    const float s = g.row_w ? g.row_w[r] : 1.0f;
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (i < g.ff) {  // gate and up rows are padded to multiples of 64: eight columns can always be read
        float x[8], u[8];
        if (g.gu_f32) {
            const float* src = reinterpret_cast<const float*>(g.gu) + (size_t)r * g.ldg + i;
            Elt<float>::ld8(src, x);
            Elt<float>::ld8(src + g.up_off, u);
        } else {
            const T* src = reinterpret_cast<const T*>(g.gu) + (size_t)r * g.ldg + i;
            Elt<T>::ld8(src, x);
            Elt<T>::ld8(src + g.up_off, u);
        }
#pragma unroll
        for (int j = 0; j < 8; j++) v[j] = i + j >= g.ff ? 0.f : gs.scale_out ? gate_one(gs, x[j], u[j]) * s : gate_one(gs, x[j] * s, u[j] * s);
    }
    Elt<T>::st8(reinterpret_cast<T*>(g.out) + (size_t)r * g.ldo + i, v);
}

__global__ void tanh_kernel(const float* __restrict__ x, int ldx, int n, float* __restrict__ out, int ldo) {
    pdl_wait();
    for (int i = threadIdx.x; i < ldo; i += blockDim.x) out[(size_t)blockIdx.x * ldo + i] = i < n ? tanhf(x[(size_t)blockIdx.x * ldx + i]) : 0.f;
}

template <typename T>
__global__ void zero_cols_kernel(T* x, int ldx, int c0, int c1) {
    pdl_wait();
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) Elt<T>::st(x + (size_t)blockIdx.x * ldx + c, 0.f);
}

// 32 x 32 outputs per block (4 rows per thread), x and w staged 32 inputs at a time; each 32-input partial sum is added
// to the running total, which keeps the rounding error near that of a blocked sum.
__global__ void __launch_bounds__(256) linear_f32_blocked_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ w, int M, int N, int K,
                                                                 float* __restrict__ y, int ldy) {
    pdl_wait();
    __shared__ float xs[32][33], ws[32][33];
    const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5;
    const int j = blockIdx.x * 32 + tx, t0 = blockIdx.y * 32;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < K; k0 += 32) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int r = ty * 4 + i;
            xs[r][tx] = (t0 + r < M && k0 + tx < K) ? x[(size_t)(t0 + r) * ldx + k0 + tx] : 0.f;
            ws[r][tx] = (blockIdx.x * 32 + r < N && k0 + tx < K) ? w[(size_t)(blockIdx.x * 32 + r) * K + k0 + tx] : 0.f;
        }
        __syncthreads();
        float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int d = 0; d < 32; d++)
#pragma unroll
            for (int i = 0; i < 4; i++) part[i] = fmaf(xs[ty * 4 + i][d], ws[tx][d], part[i]);
#pragma unroll
        for (int i = 0; i < 4; i++) acc[i] += part[i];
        __syncthreads();
    }
    if (j >= N) return;
#pragma unroll
    for (int i = 0; i < 4; i++)
        if (t0 + ty * 4 + i < M) y[(size_t)(t0 + ty * 4 + i) * ldy + j] = acc[i];
}

__global__ void argmax_rows_f32_kernel(const float* __restrict__ logits, int ld, int vocab, int32_t* __restrict__ out) {
    pdl_wait();
    __shared__ float bv[32];
    __shared__ int bi[32];
    const float* row = logits + (size_t)blockIdx.x * ld;
    float best = -INFINITY;
    int idx = 0x7fffffff;
    for (int i = threadIdx.x * 4; i < vocab; i += blockDim.x * 4) {  // (ld is a multiple of 128) a thread's ids ascend: its first maximum is kept
        const float4 v = *reinterpret_cast<const float4*>(row + i);
        if (v.x > best) best = v.x, idx = i;
        if (i + 1 < vocab && v.y > best) best = v.y, idx = i + 1;
        if (i + 2 < vocab && v.z > best) best = v.z, idx = i + 2;
        if (i + 3 < vocab && v.w > best) best = v.w, idx = i + 3;
    }
    auto take = [&](float ov, int oi) {
        if (ov > best || (ov == best && oi < idx)) best = ov, idx = oi;
    };
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) take(__shfl_xor_sync(0xffffffffu, best, o), __shfl_xor_sync(0xffffffffu, idx, o));
    if ((threadIdx.x & 31) == 0) bv[threadIdx.x >> 5] = best, bi[threadIdx.x >> 5] = idx;
    __syncthreads();
    if (threadIdx.x < 32) {
        const int nw = blockDim.x >> 5;
        best = threadIdx.x < nw ? bv[threadIdx.x] : -INFINITY;
        idx = threadIdx.x < nw ? bi[threadIdx.x] : 0x7fffffff;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) take(__shfl_xor_sync(0xffffffffu, best, o), __shfl_xor_sync(0xffffffffu, idx, o));
        if (threadIdx.x == 0) out[blockIdx.x] = idx == 0x7fffffff ? 0 : idx;
    }
}

int threads_for(int n, int per, int cap) {
    int t = (n + per - 1) / per;
    t = (t + 31) / 32 * 32;
    return t < 32 ? 32 : (t > cap ? cap : t);
}

}  // namespace

int32_t b2_embed_residual_launch(b2_ctx* ctx, bool f32, const void* table, int ld_table, const int32_t* ids, int T, int width, int vocab, float* x,
                                 int ldx, int copies) {
    if (T <= 0) return B2_OK;
    const int th = threads_for(width, 4, 512);
    if (f32)
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, embed_residual_kernel<float>, dim3(T), dim3(th), 0, ctx->stream, (const float*)table, ld_table, ids, width, vocab, x, ldx, copies));
    else
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, embed_residual_kernel<uint16_t>, dim3(T), dim3(th), 0, ctx->stream, (const uint16_t*)table, ld_table, ids, width, vocab, x, ldx, copies));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_add_norm_launch(b2_ctx* ctx, bool f32, const AddNormParams& p) {
    if (p.rows <= 0) return B2_OK;
    const int th = threads_for(p.width, 8, 512);
    const size_t smem = ((size_t)p.width * 4 + 15) / 16 * 16;
    B2_REQUIRE(smem <= 200 * 1024, B2_ERR_UNSUPPORTED, "add_norm: the model is too wide");
    if (smem > 40 * 1024) {
        B2_SMEM_ONCE(ctx, add_norm_kernel<float>, 200 * 1024);
        B2_SMEM_ONCE(ctx, add_norm_kernel<uint16_t>, 200 * 1024);
    }
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? add_norm_kernel<float> : add_norm_kernel<uint16_t>, dim3(p.rows), dim3(th), smem, ctx->stream, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_stream_norm_launch(b2_ctx* ctx, bool f32, const StreamNormParams& p) {
    if (p.rows <= 0) return B2_OK;
    B2_REQUIRE(p.streams >= 1 && p.streams <= kMaxStreams, B2_ERR_UNSUPPORTED, "residual streams: 1 to 16");
    const bool vec = p.width % 4 == 0 && p.ldx % 4 == 0 && p.ldy % 4 == 0 && p.ldh % 4 == 0;
    const int th = threads_for(p.width, vec ? 4 : 1, p.streams <= 4 && vec && p.rows <= 2 * ctx->sm_count ? 1024 : 512);
    const size_t smem = ((size_t)p.width * 4 + 15) / 16 * 16;
    B2_REQUIRE(smem <= 200 * 1024, B2_ERR_UNSUPPORTED, "stream_norm: the model is too wide");
    auto run = [&](auto k) -> int32_t {
        if (smem > 40 * 1024) B2_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3(p.rows), dim3(th), smem, ctx->stream, p));
        B2_LAUNCHED(ctx);
        return B2_OK;
    };
    auto pick = [&](auto e) -> int32_t {
        using T = decltype(e);
        if (!vec) return run(stream_norm_kernel<T, kMaxStreams, 1>);
        if (p.streams <= 2) return run(stream_norm_kernel<T, 2, 4>);
        if (p.streams == 3) return run(stream_norm_kernel<T, 3, 4>);
        if (p.streams == 4) return run(stream_norm_kernel<T, 4, 4>);
        if (p.streams <= 8) return run(stream_norm_kernel<T, 8, 4>);
        return run(stream_norm_kernel<T, kMaxStreams, 4>);
    };
    return f32 ? pick(float{}) : pick(uint16_t{});
}
int32_t b2_tanh_launch(b2_ctx* ctx, const float* x, int ldx, int T, int n, float* out, int ldo) {
    if (T <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, tanh_kernel, dim3(T), dim3(threads_for(ldo, 1, 256)), 0, ctx->stream, x, ldx, n, out, ldo));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_gate_launch(b2_ctx* ctx, bool f32, const GateSpec& g, const GateRows& a, const GateRows& b) {
    const int rows = a.rows + b.rows, ldo = a.ldo > b.ldo ? a.ldo : b.ldo;
    if (rows <= 0) return B2_OK;
    const int th = threads_for(ldo, 8, 256);
    for (int r0 = 0; r0 < rows; r0 += 65535) {  // grid.y limit
        const dim3 grid((ldo / 8 + th - 1) / th, rows - r0 < 65535 ? rows - r0 : 65535);
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? gate_kernel<float> : gate_kernel<uint16_t>, grid, dim3(th), 0, ctx->stream, g, a, b, r0));
        B2_LAUNCHED(ctx);
    }
    return B2_OK;
}
int32_t b2_zero_cols_launch(b2_ctx* ctx, bool f32, void* x, int ldx, int c0, int c1, int rows) {
    if (rows <= 0 || c0 >= c1) return B2_OK;
    if (f32)
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, zero_cols_kernel<float>, dim3(rows), dim3(64), 0, ctx->stream, (float*)x, ldx, c0, c1));
    else
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, zero_cols_kernel<uint16_t>, dim3(rows), dim3(64), 0, ctx->stream, (uint16_t*)x, ldx, c0, c1));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_linear_f32_launch(b2_ctx* ctx, const float* x, int ldx, const float* w, int M, int N, int K, float* y, int ldy) {
    if (M <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, linear_f32_blocked_kernel, dim3((N + 31) / 32, (M + 31) / 32), dim3(256), 0, ctx->stream, x, ldx, w, M, N, K, y, ldy));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_argmax_f32_launch(b2_ctx* ctx, const float* logits, int ld, int rows, int vocab, int32_t* out) {
    if (rows <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, argmax_rows_f32_kernel, dim3(rows), dim3(1024), 0, ctx->stream, logits, ld, vocab, out));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
