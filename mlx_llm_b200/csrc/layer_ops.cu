// Elementwise and normalisation steps of the layered models (residual stream in f32), in bf16 or f32 storage.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

__device__ __forceinline__ float gelu_tanh_f32(float g) {
    const float k = 0.7978845608028654f;  // sqrt(2 / pi)
    return 0.5f * g * (1.0f + tanhf(k * (g + 0.044715f * g * g * g)));
}

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

// One block per token.  The block of a sequence's first token in the step is the only one that reads the kept token, and the one
// that replaces it.
template <typename T>
__global__ void embed_pairs_kernel(const EmbedPairsParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    __shared__ int64_t s_row;
    const int t = blockIdx.x;
    auto token = [&](int id) { return min(max(id, 0), p.vocab - 1); };
    const int id = token(p.ids[t]);
    if (p.pairs.buckets > 0) {
        if (threadIdx.x == 0) {
            const int b = p.token_seq[t], start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start;
            int prev = t > start ? token(p.ids[t - 1]) : -1;
            if (t == start) {
                float* kept = p.kept + (size_t)p.seq_slot[b] * p.slot_stride;
                if (p.context_lens[b] > n) prev = __float_as_int(*kept);
                *kept = __int_as_float(token(p.ids[start + n - 1]));
            }
            s_row = prev < 0 ? p.pairs.buckets : ((int64_t)prev * p.pairs.mul_prev + (int64_t)id * p.pairs.mul_cur) % p.pairs.buckets;
        }
        __syncthreads();
    }
    const T* a = reinterpret_cast<const T*>(p.table) + (size_t)id * p.ld_table;
    const T* b = p.pairs.buckets > 0 ? reinterpret_cast<const T*>(p.pair_table) + (size_t)s_row * p.ld_pairs : nullptr;
    T* o = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo;
    float* x = p.x + (size_t)t * p.ldx;
    if (p.width % 8 == 0) {  // (table rows and p.ldo are multiples of 64)
        for (int i = threadIdx.x * 8; i < p.ldo; i += blockDim.x * 8) {
            float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (i < p.width) {
                float u[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                Elt<T>::ld8(a + i, v);
                if (b) Elt<T>::ld8(b + i, u);
#pragma unroll
                for (int j = 0; j < 8; j++) v[j] = fmaf(v[j], p.scale, u[j]);
                Elt<float>::st8(x + i, v);
            }
            Elt<T>::st8(o + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < p.ldo; i += blockDim.x) {
            const float v = i < p.width ? fmaf(Elt<T>::ld(a + i), p.scale, b ? Elt<T>::ld(b + i) : 0.f) : 0.f;
            if (i < p.width) x[i] = v;
            Elt<T>::st(o + i, v);
        }
    }
}

// Sums of squares of `groups` equal parts of a row, by the block's warps: each group has a team of them, or each warp has groups.
// sq(i) gives column i's square, VEC columns at a time; inv[g] receives 1 / sqrt(mean + eps).  `part` holds 32 floats.
template <typename F>
__device__ __forceinline__ void group_inverses(int width, int groups, float eps, float* part, float* inv, int step, F sum_at) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5, size = width / groups;
    const int teams = min(groups, warps), team_warps = warps / teams, team = warp / team_warps, mine = warp - team * team_warps;
    if (team < teams)
        for (int g = team; g < groups; g += teams) {
            float ss = 0.f;
            for (int i = (mine * 32 + lane) * step; i < size; i += team_warps * 32 * step) ss += sum_at(g * size + i);
            ss = elt_warp_sum(ss);
            if (lane == 0) {
                if (team_warps == 1)
                    inv[g] = 1.0f / sqrtf(ss / (float)size + eps);
                else
                    part[warp] = ss;
            }
        }
    __syncthreads();
    if (team_warps > 1) {
        for (int g = threadIdx.x; g < groups; g += blockDim.x) {
            float ss = 0.f;
            for (int k = 0; k < team_warps; k++) ss += part[g * team_warps + k];
            inv[g] = 1.0f / sqrtf(ss / (float)size + eps);
        }
        __syncthreads();
    }
}

// One block per row; y stays in shared memory between the two passes.
template <typename T, int VEC>
__global__ void post_norm_kernel(const PostNormParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    extern __shared__ __align__(16) float row[];  // [width], then [groups]
    __shared__ float part[32];
    float* inv = row + (p.width + 3) / 4 * 4;
    const size_t r = blockIdx.x;
    const int size = p.width / p.groups;
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
    const float* yr = p.y + (p.y_rows ? (size_t)p.y_rows[r] : r) * p.ldy;
    group_inverses(p.width, p.groups, p.eps, part, inv, VEC, [&](int i) {
        float v[VEC], ss = 0.f;
        load(yr + i, v);
        store(row + i, v);
#pragma unroll
        for (int e = 0; e < VEC; e++) ss += v[e] * v[e];
        return ss;
    });
    const float* xr = p.x + r * p.ldx;
    T* o = p.out ? reinterpret_cast<T*>(p.out) + r * p.ldo : nullptr;
    for (int i = threadIdx.x * VEC; i < p.width; i += blockDim.x * VEC) {
        float x[VEC], y[VEC], w[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) x[e] = 0.f;
        if (p.x) load(xr + i, x);
        load(row + i, y);
        load(p.w + i, w);
        const float f = inv[i / size];  // (VEC columns lie in one group)
#pragma unroll
        for (int e = 0; e < VEC; e++) x[e] = fmaf(p.mult, y[e] * f * w[e], x[e]);
        if (p.keep) store(p.keep + r * p.ldx + i, x);
        if (p.avg) {
            const float own = p.avg[p.depth];
#pragma unroll
            for (int e = 0; e < VEC; e++) x[e] *= own;
            const float* past = p.past + r * p.ldx + i;
#pragma unroll 4
            for (int j = 0; j < p.depth; j++) {
                float v[VEC];
                load(past + j * p.past_stride, v);
#pragma unroll
                for (int e = 0; e < VEC; e++) x[e] = fmaf(p.avg[j], v[e], x[e]);
            }
        }
        if (p.x_out) store(p.x_out + r * p.ldx + i, x);
        if (o) {
            if constexpr (VEC == 4)
                Elt<T>::st4(o + i, x);
            else
                Elt<T>::st(o + i, x[0]);
        }
    }
    if (o)
        for (int i = p.width + threadIdx.x; i < p.ldo; i += blockDim.x) Elt<T>::st(o + i, 0.f);
}

// The same with groups of whole 128 columns: the row lies in registers (NV times four columns per thread), every load is on its way
// before the only barrier.
template <typename T, int NV>
__global__ void __launch_bounds__(NV <= 1 ? 1024 : 512) post_norm_rows_kernel(const PostNormParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    extern __shared__ float part[];  // [width / 128] sums of squares
    const size_t r = blockIdx.x;
    const int size = p.width / p.groups, per = size / 128, lane = threadIdx.x & 31;
    float y[NV][4], x[NV][4], w[NV][4];
    const float* yr = p.y + (p.y_rows ? (size_t)p.y_rows[r] : r) * p.ldy;
#pragma unroll
    for (int k = 0; k < NV; k++) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i < p.width) Elt<float>::ld4(yr + i, y[k]);
    }
#pragma unroll
    for (int k = 0; k < NV; k++) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        x[k][0] = x[k][1] = x[k][2] = x[k][3] = 0.f;
        if (i >= p.width) continue;
        if (p.x) Elt<float>::ld4(p.x + r * p.ldx + i, x[k]);
        Elt<float>::ld4(p.w + i, w[k]);
    }
    float past[NV][4];
#pragma unroll
    for (int k = 0; k < NV; k++) {
#pragma unroll
        for (int e = 0; e < 4; e++) past[k][e] = 0.f;
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (p.avg && i < p.width) {
            const float* src = p.past + r * p.ldx + i;
#pragma unroll 4
            for (int j = 0; j < p.depth; j++) {
                float v[4];
                Elt<float>::ld4(src + j * p.past_stride, v);
#pragma unroll
                for (int e = 0; e < 4; e++) past[k][e] = fmaf(p.avg[j], v[e], past[k][e]);
            }
        }
    }
#pragma unroll
    for (int k = 0; k < NV; k++) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i >= p.width) continue;  // (the whole warp: 128 columns)
        const float ss = elt_warp_sum(y[k][0] * y[k][0] + y[k][1] * y[k][1] + y[k][2] * y[k][2] + y[k][3] * y[k][3]);
        if (lane == 0) part[i / 128] = ss;
    }
    __syncthreads();
    const float own = p.avg ? p.avg[p.depth] : 1.f;
    T* o = p.out ? reinterpret_cast<T*>(p.out) + r * p.ldo : nullptr;
#pragma unroll
    for (int k = 0; k < NV; k++) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i >= p.width) continue;
        float ss = 0.f;
        for (int s = lane; s < per; s += 32) ss += part[i / size * per + s];
        const float f = 1.0f / sqrtf(elt_warp_sum(ss) / (float)size + p.eps);
#pragma unroll
        for (int e = 0; e < 4; e++) x[k][e] = fmaf(p.mult, y[k][e] * f * w[k][e], x[k][e]);
        if (p.keep) Elt<float>::st4(p.keep + r * p.ldx + i, x[k]);
        if (p.avg)
#pragma unroll
            for (int e = 0; e < 4; e++) x[k][e] = fmaf(own, x[k][e], past[k][e]);
        if (p.x_out) Elt<float>::st4(p.x_out + r * p.ldx + i, x[k]);
        if (o) Elt<T>::st4(o + i, x[k]);
    }
    if (o)
        for (int i = p.width + threadIdx.x; i < p.ldo; i += blockDim.x) Elt<T>::st(o + i, 0.f);
}

template <typename T>
__global__ void token_gate_kernel(const TokenGateParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int t = blockIdx.x;
    const T* e = reinterpret_cast<const T*>(p.table) + (size_t)min(max(p.ids[t], 0), p.vocab - 1) * p.ld_table + p.col0;
    for (int i = threadIdx.x; i < p.ldo; i += blockDim.x) {
        float v = 0.f;
        if (i < p.n) {
            float z = 0.f;
#pragma unroll 8
            for (int k = 0; k < p.parts; k++) z += p.z[k * p.part_stride + (size_t)t * p.ldz + i];
            v = gelu_tanh_f32(z) * Elt<T>::ld(e + i);
        }
        Elt<T>::st(reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo + i, v);
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
    if (gs.act == GateAct::GeluTanh) return gelu_tanh_f32(g) * u;
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
int32_t b2_embed_pairs_launch(b2_ctx* ctx, bool f32, const EmbedPairsParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? embed_pairs_kernel<float> : embed_pairs_kernel<uint16_t>, dim3(p.T), dim3(threads_for(p.ldo, 8, 512)), 0, ctx->stream, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_post_norm_launch(b2_ctx* ctx, bool f32, const PostNormParams& p) {
    if (p.rows <= 0) return B2_OK;
    const bool vec = (p.width / p.groups) % 4 == 0 && p.ldx % 4 == 0 && p.ldy % 4 == 0 && p.past_stride % 4 == 0;
    const int th = threads_for(p.width, vec ? 4 : 1, p.rows <= 2 * ctx->sm_count ? 1024 : 512);
    const size_t smem = ((size_t)p.width * 4 + 15) / 16 * 16 + (size_t)p.groups * 4;
    B2_REQUIRE(smem <= 200 * 1024, B2_ERR_UNSUPPORTED, "post_norm: the model is too wide");
    if (vec && (p.width / p.groups) % 128 == 0 && p.width <= 8192) {
        const int cap = p.rows <= 2 * ctx->sm_count && p.width <= 4096 ? 1024 : 512, n = (p.width / 4 + cap - 1) / cap, nv = n <= 1 ? 1 : n <= 2 ? 2 : 4;
        const int t = (p.width / 4 + nv - 1) / nv;
        auto go = [&](auto k) -> int32_t {
            B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3(p.rows), dim3((t + 31) / 32 * 32), (size_t)p.width / 128 * 4, ctx->stream, p));
            B2_LAUNCHED(ctx);
            return B2_OK;
        };
        if (f32) return nv == 1 ? go(post_norm_rows_kernel<float, 1>) : nv == 2 ? go(post_norm_rows_kernel<float, 2>) : go(post_norm_rows_kernel<float, 4>);
        return nv == 1 ? go(post_norm_rows_kernel<uint16_t, 1>) : nv == 2 ? go(post_norm_rows_kernel<uint16_t, 2>) : go(post_norm_rows_kernel<uint16_t, 4>);
    }
    auto run = [&](auto k) -> int32_t {
        if (smem > 40 * 1024) B2_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3(p.rows), dim3(th), smem, ctx->stream, p));
        B2_LAUNCHED(ctx);
        return B2_OK;
    };
    if (f32) return vec ? run(post_norm_kernel<float, 4>) : run(post_norm_kernel<float, 1>);
    return vec ? run(post_norm_kernel<uint16_t, 4>) : run(post_norm_kernel<uint16_t, 1>);
}
int32_t b2_token_gate_launch(b2_ctx* ctx, bool f32, const TokenGateParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? token_gate_kernel<float> : token_gate_kernel<uint16_t>, dim3(p.T), dim3(threads_for(p.ldo, 1, 256)), 0, ctx->stream, p));
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
