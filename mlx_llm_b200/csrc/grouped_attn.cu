// Grouped-query attention of the layered models: projections to rotated queries and cache rows, and the plain form of the
// attention.  Scores may be capped, the softmax may have a sink (exp(0) in its denominator, with no value), two maps may be taken
// off one another (differential attention).
#include <type_traits>

#include "elt.cuh"
#include "layer_kernels.h"

namespace {

constexpr int kMaxHead = 256;

// A warp per (token, head of q, k or v; with two maps, per map): bias, norm over the head, rotation of the pairs (i, i + dims/2) or
// (2i, 2i + 1), store.  A lane holds VEC consecutive values of every 32 * VEC; the rotation finds its partner in shared memory
// (N 1, VEC 4: heads of up to 128, the partner comes by shuffle; neighbours with VEC 4: the lane has both).  With a norm over all heads (ALL) a block takes eight heads of
// one token, and first the sums of squares of all its queries and of all its keys.
template <typename T, int VEC, int N, bool ALL>
__global__ void __launch_bounds__(256) gqa_prep_kernel(const GroupedAttnSpec a, const GqaPrepParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    constexpr bool SHUFFLE = N == 1 && VEC == 4;
    __shared__ __align__(16) float rows[SHUFFLE ? 1 : 8][SHUFFLE ? 4 : kMaxHead];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, QH = a.q_heads(), KH = a.k_heads(), units = QH + (p.own_kv ? KH + a.kv_heads : 0);
    const int id = blockIdx.x * 8 + warp, t = ALL ? blockIdx.y : id / units, u = ALL ? id : id - t * units;
    float all_inv[2] = {1.f, 1.f};
    if constexpr (ALL) {  // (every thread of the block: u0 the block's first unit)
        __shared__ float red[33];
        const int u0 = blockIdx.x * 8, nq = a.heads * a.dim, nk = a.kv_heads * a.dim;
        auto sum = [&](const float* bias, int off, int n) {
            const T* x = reinterpret_cast<const T*>(p.in) + (size_t)t * p.ld + off;
            float ss = 0.f;
            if constexpr (VEC == 4) {
                for (int i = threadIdx.x * 4; i < n; i += 1024) {
                    float v[4];
                    Elt<T>::ld4(x + i, v);
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        if (bias) v[e] += bias[i + e];
                        ss += v[e] * v[e];
                    }
                }
            } else {
                for (int i = threadIdx.x; i < n; i += 256) {
                    const float v = Elt<T>::ld(x + i) + (bias ? bias[i] : 0.f);
                    ss += v * v;
                }
            }
            return 1.0f / sqrtf(elt_block_sum(ss, red) / (float)n + p.eps);
        };
        if (u0 < a.heads) all_inv[0] = sum(p.q_bias, p.q_off, nq);
        if (p.own_kv && u0 + 8 > a.heads && u0 < a.heads + a.kv_heads) all_inv[1] = sum(p.k_bias, p.k_off, nk);
        if (u >= units) return;
    }
    if (t >= p.T) return;
    const int kind = u < QH ? 0 : u < QH + KH ? 1 : 2, h = kind == 0 ? u : kind == 1 ? u - QH : u - QH - KH;
    const int n = kind == 2 ? a.vdim : a.dim, padded = kind == 2 ? a.v_row() : a.k_row(), dims = kind == 2 ? 0 : a.rot.dims, half = dims / 2;
    const T* src = reinterpret_cast<const T*>(p.in) + (size_t)t * p.ld + (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + h * n;
    const float* bias = kind == 0 ? p.q_bias : kind == 1 ? p.k_bias : p.v_bias;
    const float* w = kind == 0 ? p.q_norm : kind == 1 ? p.k_norm : nullptr;
    if (ALL && w) w += h * n;
    const int slot = p.slot_mapping[t];
    T* dst;
    if (kind == 0) {
        dst = reinterpret_cast<T*>(p.q) + ((size_t)t * QH + h) * padded;
    } else {
        if (slot < 0) return;
        const size_t row = ((size_t)(slot / p.page_size) * (kind == 1 ? KH : a.kv_heads) + h) * p.page_size + slot % p.page_size;
        dst = reinterpret_cast<T*>(kind == 1 ? p.k_cache : p.v_cache) + row * padded;
    }
    float v[N][VEC], ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int d = (i * 32 + lane) * VEC;
#pragma unroll
        for (int e = 0; e < VEC; e++) v[i][e] = 0.f;
        if (d >= n) continue;
        if constexpr (VEC == 4)
            Elt<T>::ld4(src + d, v[i]);
        else
            v[i][0] = Elt<T>::ld(src + d);
        if (bias) {
            if constexpr (VEC == 4) {
                float x[4];
                Elt<float>::ld4(bias + h * n + d, x);
#pragma unroll
                for (int e = 0; e < 4; e++) v[i][e] += x[e];
            } else {
                v[i][0] += bias[h * n + d];
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; e++) ss += v[i][e] * v[i][e];
    }
    if (w) {
        const float inv = ALL ? all_inv[kind] : 1.0f / sqrtf(elt_warp_sum(ss) / (float)n + p.eps);
#pragma unroll
        for (int i = 0; i < N; i++)
#pragma unroll
            for (int e = 0; e < VEC; e++) {
                const int d = (i * 32 + lane) * VEC + e;
                if (d < n) v[i][e] = v[i][e] * inv * w[d];
            }
    }
    if (VEC == 4 && a.neighbours) {
        const float* ct = p.cos_t + (size_t)p.positions[t] * half;
        const float* st = p.sin_t + (size_t)p.positions[t] * half;
#pragma unroll
        for (int i = 0; i < N; i++)
#pragma unroll
            for (int e = 0; e < VEC - 1; e += 2) {
                const int d = (i * 32 + lane) * VEC + e;
                if (d < dims) {
                    const float c = ct[d / 2], s = st[d / 2], x = v[i][e], y = v[i][e + 1];
                    v[i][e] = x * c - y * s;
                    v[i][e + 1] = y * c + x * s;
                }
            }
    } else if constexpr (SHUFFLE) {
        if (half > 0) {  // (half is a multiple of four)
            const int d = lane * 4, src_lane = d < half ? lane + half / 4 : lane - half / 4;
            float o[4], c[4] = {1.f, 1.f, 1.f, 1.f}, sn[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int e = 0; e < 4; e++) o[e] = __shfl_sync(0xffffffffu, v[0][e], src_lane & 31);
            if (d < dims) {
                const size_t at = (size_t)p.positions[t] * half + (d < half ? d : d - half);
                Elt<float>::ld4(p.cos_t + at, c);
                Elt<float>::ld4(p.sin_t + at, sn);
#pragma unroll
                for (int e = 0; e < 4; e++) v[0][e] = d < half ? v[0][e] * c[e] - o[e] * sn[e] : v[0][e] * c[e] + o[e] * sn[e];
            }
        }
    } else if (half > 0) {
        const float* ct = p.cos_t + (size_t)p.positions[t] * half;
        const float* st = p.sin_t + (size_t)p.positions[t] * half;
#pragma unroll
        for (int i = 0; i < N; i++)
#pragma unroll
            for (int e = 0; e < VEC; e++) rows[warp][(i * 32 + lane) * VEC + e] = v[i][e];
        __syncwarp();
#pragma unroll
        for (int i = 0; i < N; i++)
#pragma unroll
            for (int e = 0; e < VEC; e++) {
                const int d = (i * 32 + lane) * VEC + e;
                if (a.neighbours) {
                    if (d < dims) v[i][e] = v[i][e] * ct[d / 2] + (d % 2 ? rows[warp][d - 1] : -rows[warp][d + 1]) * st[d / 2];
                } else if (d < half)
                    v[i][e] = v[i][e] * ct[d] - rows[warp][d + half] * st[d];
                else if (d < dims)
                    v[i][e] = v[i][e] * ct[d - half] + rows[warp][d - half] * st[d - half];
            }
    }
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int d = (i * 32 + lane) * VEC;
        if (d >= padded) continue;
        if constexpr (VEC == 4)
            Elt<T>::st4(dst + d, v[i]);
        else
            Elt<T>::st(dst + d, v[i][0]);
    }
}

// The same for rotations of neighbours (and no rotation) over heads of whole eights, without biases: LP lanes per head (per map) of
// q and k, eight values each; values go in pieces of as many.
template <typename T, int LP>
__global__ void __launch_bounds__(256) gqa_prep_rows_kernel(const GroupedAttnSpec a, const GqaPrepParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    constexpr int PIECE = LP * 8;
    const int QH = a.q_heads(), KH = a.k_heads(), vp = (a.v_row() + PIECE - 1) / PIECE, units = QH + (p.own_kv ? KH + a.kv_heads * vp : 0);
    const int id = (blockIdx.x * 256 + threadIdx.x) / LP, t = id / units, u = id - t * units;
    if (t >= p.T) return;  // (all lanes of a unit)
    const int kind = u < QH ? 0 : u < QH + KH ? 1 : 2;
    int h = kind == 0 ? u : u - QH, d = threadIdx.x % LP * 8;
    if (kind == 2) {
        h -= KH;
        d += h % vp * PIECE;
        h /= vp;
    }
    const int n = kind == 2 ? a.vdim : a.dim, padded = kind == 2 ? a.v_row() : a.k_row();
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (d < n) Elt<T>::ld8(reinterpret_cast<const T*>(p.in) + (size_t)t * p.ld + (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + h * n + d, v);
    if (kind != 2) {
        const float* w = kind == 0 ? p.q_norm : p.k_norm;
        if (w) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; e++) ss += v[e] * v[e];
            const unsigned mask = LP == 32 ? 0xffffffffu : ((1u << LP) - 1u) << ((threadIdx.x & 31) / LP * LP);
#pragma unroll
            for (int o = LP / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
            const float inv = 1.0f / sqrtf(ss / (float)n + p.eps);
            if (d < n) {
                float x[8];
                Elt<float>::ld8(w + d, x);
#pragma unroll
                for (int e = 0; e < 8; e++) v[e] *= inv * x[e];
            }
        }
        const int half = a.rot.dims / 2;
        if (d < a.rot.dims) {
            const float* ct = p.cos_t + (size_t)p.positions[t] * half + d / 2;
            const float* st = p.sin_t + (size_t)p.positions[t] * half + d / 2;
            float c[4], s[4];
            if (half % 4 == 0) {
                Elt<float>::ld4(ct, c);
                Elt<float>::ld4(st, s);
            } else {
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const bool ok = d + 2 * e < a.rot.dims;
                    c[e] = ok ? ct[e] : 1.f;
                    s[e] = ok ? st[e] : 0.f;
                }
            }
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const float x = v[2 * e], y = v[2 * e + 1];
                v[2 * e] = x * c[e] - y * s[e];
                v[2 * e + 1] = y * c[e] + x * s[e];
            }
        }
    }
    if (d >= padded) return;
    if (kind == 0) {
        Elt<T>::st8(reinterpret_cast<T*>(p.q) + ((size_t)t * QH + h) * padded + d, v);
    } else {
        const int slot = p.slot_mapping[t];
        if (slot < 0) return;
        const size_t row = ((size_t)(slot / p.page_size) * (kind == 1 ? KH : a.kv_heads) + h) * p.page_size + slot % p.page_size;
        Elt<T>::st8(reinterpret_cast<T*>(kind == 1 ? p.k_cache : p.v_cache) + row * padded + d, v);
    }
}

// Plain form: one block per (token, head), one map after the other, 128 keys at a time with an online softmax, everything f32.
template <typename T>
__global__ void __launch_bounds__(128) gqa_simple_kernel(const GroupedAttnSpec a, const GqaAttnParams p) {
    pdl_wait();
    __shared__ float q[kMaxHead], accs[2][kMaxHead], pr[128], red[33];
    const int t = blockIdx.x, h = blockIdx.y, g = h / a.group(), KR = a.k_row(), VR = a.v_row(), ps = p.page_size;
    const int n = p.positions[t] + 1, lo = a.mask.first(p.positions[t]), kept = a.mask.kept(p.positions[t]), seen = kept + n - lo;
    const int32_t* bt = p.block_tables + (size_t)p.seq_slot[p.token_seq[t]] * p.max_blocks;
    auto key = [&](int i) { return i < kept ? i : i - kept + lo; };  // the i-th visible one
    auto row = [&](int j, int heads, int hd) { return ((size_t)bt[j / ps] * heads + hd) * ps + j % ps; };
    float l = 0.f;
    for (int mp = 0; mp < a.maps; mp++) {
        float* acc = accs[mp];
        const T* qr = reinterpret_cast<const T*>(p.q) + ((size_t)t * a.q_heads() + h * a.maps + mp) * KR;
        for (int i = threadIdx.x; i < KR; i += 128) q[i] = Elt<T>::ld(qr + i);
        for (int i = threadIdx.x; i < VR; i += 128) acc[i] = 0.f;
        float m = -INFINITY;
        l = 0.f;
        __syncthreads();
        for (int j0 = 0; j0 < seen; j0 += 128) {
            const int j = j0 + threadIdx.x, cnt = min(128, seen - j0);
            float s = -INFINITY;
            if (j < seen) {
                const T* k = reinterpret_cast<const T*>(p.k_cache) + row(key(j), a.k_heads(), g * a.maps + mp) * KR;
                float d = 0.f;
                for (int i = 0; i < KR; i += 8) {
                    float v[8];
                    Elt<T>::ld8(k + i, v);
#pragma unroll
                    for (int e = 0; e < 8; e++) d = fmaf(q[i + e], v[e], d);
                }
                s = d * a.scale;
                if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
            }
            float mx = elt_warp_max(s);
            __syncthreads();
            if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = mx;
            __syncthreads();
            mx = fmaxf(fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])), m);
            const float alpha = expf(m - mx), e = j < seen ? expf(s - mx) : 0.f;
            pr[threadIdx.x] = e;
            l = l * alpha + elt_block_sum(e, red);
            m = mx;
            for (int i = threadIdx.x; i < VR; i += 128) {
                float v = acc[i] * alpha;
                for (int jj = 0; jj < cnt; jj++) v = fmaf(pr[jj], Elt<T>::ld(reinterpret_cast<const T*>(p.v_cache) + row(key(j0 + jj), a.kv_heads, g) * VR + i), v);
                acc[i] = v;
            }
            __syncthreads();
        }
        if (a.sink) l += expf(-m);
        if (a.maps == 2) {  // (a thread's own values)
            for (int i = threadIdx.x; i < a.vdim; i += 128) acc[i] /= l;
            l = 1.f;
        }
    }
    float* acc = accs[0];
    if (a.maps == 2) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < a.vdim; i += 128) {
            acc[i] -= p.lambda * accs[1][i];
            ss += acc[i] * acc[i];
        }
        l = sqrtf(elt_block_sum(ss, red) / (float)a.vdim + p.eps) / (1.f - a.diff);
    }
    if (a.head_gate) l /= sigmoid_f32(Elt<T>::ld(reinterpret_cast<const T*>(p.gate) + (size_t)t * p.ld_gate + h));
    T* o = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo + h * a.vdim;
    for (int i = threadIdx.x; i < a.vdim; i += 128) Elt<T>::st(o + i, acc[i] / l * p.out_scale);
}

}  // namespace

int32_t b2_gqa_prep_launch(b2_ctx* ctx, bool f32, const GroupedAttnSpec& a, const GqaPrepParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_REQUIRE(a.dim <= kMaxHead && a.vdim <= kMaxHead, B2_ERR_UNSUPPORTED, "grouped attention: head sizes up to 256");
    if ((a.neighbours || a.rot.dims == 0) && !a.norm_all && !p.q_bias && a.dim % 8 == 0 && a.vdim % 8 == 0 && (p.q_off | p.k_off | p.v_off | p.ld) % 8 == 0) {
        const int lp = a.k_row() <= 64 ? 8 : a.k_row() <= 128 ? 16 : 32, vp = (a.v_row() + lp * 8 - 1) / (lp * 8);
        const size_t n = (size_t)p.T * (a.q_heads() + (p.own_kv ? a.k_heads() + a.kv_heads * vp : 0)) * lp;
        auto k = lp == 8    ? (f32 ? gqa_prep_rows_kernel<float, 8> : gqa_prep_rows_kernel<uint16_t, 8>)
                 : lp == 16 ? (f32 ? gqa_prep_rows_kernel<float, 16> : gqa_prep_rows_kernel<uint16_t, 16>)
                            : (f32 ? gqa_prep_rows_kernel<float, 32> : gqa_prep_rows_kernel<uint16_t, 32>);
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, ctx->stream, a, p));
        B2_LAUNCHED(ctx);
        return B2_OK;
    }
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && p.q_off % 4 == 0 && p.k_off % 4 == 0 && p.v_off % 4 == 0 && p.ld % 4 == 0;
    const int units = a.q_heads() + (p.own_kv ? a.k_heads() + a.kv_heads : 0);
    const bool small = a.dim <= 128 && a.vdim <= 128 && (a.neighbours || a.rot.dims % 8 == 0);
    auto pick = [&](auto all) {
        constexpr bool ALL = decltype(all)::value;
        return !vec    ? (f32 ? gqa_prep_kernel<float, 1, 8, ALL> : gqa_prep_kernel<uint16_t, 1, 8, ALL>)
               : small ? (f32 ? gqa_prep_kernel<float, 4, 1, ALL> : gqa_prep_kernel<uint16_t, 4, 1, ALL>)
                       : (f32 ? gqa_prep_kernel<float, 4, 2, ALL> : gqa_prep_kernel<uint16_t, 4, 2, ALL>);
    };
    auto k = a.norm_all ? pick(std::true_type{}) : pick(std::false_type{});
    const dim3 grid = a.norm_all ? dim3((units + 7) / 8, p.T) : dim3((unsigned)(((size_t)p.T * units + 7) / 8));
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, grid, dim3(256), 0, ctx->stream, a, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_gqa_simple_launch(b2_ctx* ctx, bool f32, const GroupedAttnSpec& a, const GqaAttnParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_REQUIRE(a.dim <= kMaxHead && a.vdim <= kMaxHead, B2_ERR_UNSUPPORTED, "grouped attention: head sizes up to 256");
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? gqa_simple_kernel<float> : gqa_simple_kernel<uint16_t>, dim3(p.T, a.heads), dim3(128), 0, ctx->stream, a, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
