// Linear memories (retention, gated delta rule, time mixing with a bonus) between a layer's projections: what enters the recurrence, the recurrence
// token by token, and the input row of the output projection.
//
// Recurrent record of a sequence (f32, one slot per block-table row of the pool):
//   S     [heads][vdim][dim]
//   conv  [taps - 1][channels]   the last inputs of the convolution, oldest first; or, with a token shift, [width] the last row of
//                                the layer's normed input
// A sequence that starts in this step (nothing cached) starts from zero, whatever its slot held before.
//
// Everything that enters the recurrence besides the convolved (or plain) values is prepared and kept in f32.
#include "elt.cuh"
#include "memory.cuh"

namespace {

__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// Queries and keys of a memory without convolution: rotated (pairs (i, i + dims/2)), keys times dim^-1/2, as f32.  VEC
// consecutive values per thread.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) memory_rotate_kernel(const MemorySpec s, const MemoryParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int t = blockIdx.x, Q = s.q_cols(), D = s.dim, dims = s.rot.dims, half = dims / 2;
    const T* src = reinterpret_cast<const T*>(p.in) + (size_t)t * p.ld + p.c_off;
    const float* ct = p.cos_t + (size_t)p.positions[t] * half;
    const float* st = p.sin_t + (size_t)p.positions[t] * half;
    const float scale = rsqrtf((float)D);
    auto load = [&](const T* x, float (&v)[VEC]) {
        if constexpr (VEC == 4)
            Elt<T>::ld4(x, v);
        else
            v[0] = Elt<T>::ld(x);
    };
    for (int i = (blockIdx.y * 256 + threadIdx.x) * VEC; i < 2 * Q; i += gridDim.y * 256 * VEC) {
        const int c = i < Q ? i : i - Q, d = c % D;
        float v[VEC], o[VEC];
        load(src + i, v);
        if (d < dims) {
            const bool low = d < half;
            float cs[VEC], sn[VEC];
            load(src + (low ? i + half : i - half), o);
            if constexpr (VEC == 4) {
                Elt<float>::ld4(ct + (low ? d : d - half), cs);
                Elt<float>::ld4(st + (low ? d : d - half), sn);
            } else {
                cs[0] = ct[low ? d : d - half], sn[0] = st[low ? d : d - half];
            }
#pragma unroll
            for (int e = 0; e < VEC; e++) v[e] = low ? v[e] * cs[e] - o[e] * sn[e] : v[e] * cs[e] + o[e] * sn[e];
        }
        float* dst = (i < Q ? p.q : p.k) + (size_t)t * Q + c;
        if (i >= Q)
#pragma unroll
            for (int e = 0; e < VEC; e++) v[e] *= scale;
        if constexpr (VEC == 4)
            Elt<float>::st4(dst, v);
        else
            dst[0] = v[0];
    }
}

// Token shift: a block takes `run` tokens and 256 * VEC columns, and carries the row before along.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) token_shift_kernel(const ShiftParams p, int run) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int i = (blockIdx.x * 256 + threadIdx.x) * VEC, t0 = blockIdx.y * run, t1 = min(t0 + run, p.T);
    if (i >= p.ldo) return;
    const bool in = i < p.width;  // (VEC divides the width)
    const T* h = reinterpret_cast<const T*>(p.h) + i;
    T* out = reinterpret_cast<T*>(p.out) + i;
    auto load = [&](const T* s, float (&v)[VEC]) {
        if constexpr (VEC == 4)
            Elt<T>::ld4(s, v);
        else
            v[0] = Elt<T>::ld(s);
    };
    float mu[5][VEC], prev[VEC], cur[VEC];
#pragma unroll
    for (int j = 0; j < 5; j++)
#pragma unroll
        for (int e = 0; e < VEC; e++) mu[j][e] = in ? p.mu[(size_t)j * p.width + i + e] : 0.f;
#pragma unroll
    for (int e = 0; e < VEC; e++) prev[e] = cur[e] = 0.f;
    for (int t = t0; t < t1; t++) {
        const int b = p.token_seq[t], start = p.cu_seqlens[b];
        if (in) {
            if (t == start) {  // what the sequence's last step left, or nothing
                const bool kept = p.context_lens[b] > p.cu_seqlens[b + 1] - start;
                const float* k = p.kept + (size_t)p.seq_slot[b] * p.slot_stride + i;
#pragma unroll
                for (int e = 0; e < VEC; e++) prev[e] = kept ? k[e] : 0.f;
            } else if (t == t0) {
                load(h + (size_t)(t - 1) * p.ld_h, prev);
            }
            load(h + (size_t)t * p.ld_h, cur);
        }
#pragma unroll
        for (int j = 0; j < 5; j++) {
            float v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; e++) v[e] = fmaf(prev[e] - cur[e], mu[j][e], cur[e]);
            T* o = out + ((size_t)t * 5 + j) * p.ldo;
            if constexpr (VEC == 4)
                Elt<T>::st4(o, v);
            else
                Elt<T>::st(o, v[0]);
        }
#pragma unroll
        for (int e = 0; e < VEC; e++) prev[e] = cur[e];
    }
}

// Time mixing: logarithms -exp(z + w0) of the decays (queries and keys need no preparation).  Below e^-128 an f32 decay is zero:
// the logarithm stops there, which keeps its sums finite.
__device__ __forceinline__ float log_decay_of(float x) { return fmaxf(-expf(x), -128.f); }
__global__ void __launch_bounds__(256) memory_decay_kernel(const MemorySpec s, const MemoryParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int Q = s.q_cols(), i = blockIdx.x * 256 + threadIdx.x, t = blockIdx.y;
    if (i < Q) p.lg[(size_t)t * Q + i] = log_decay_of(reinterpret_cast<const float*>(p.dec)[(size_t)t * p.ld_dec + i] + p.dt_bias[i]);
}
// ... from the first factor's result x (f32): z = tanh(x) W2^T, bf16 operands.  Block = 16 MT tokens x 128 channels, a warp 16
// channels; 64 inputs at a time.
template <int MT>
__global__ void __launch_bounds__(256) memory_decay_tc_kernel(const MemorySpec s, const MemoryParams p) {
    constexpr int TM = 16 * MT;
    __shared__ __align__(128) uint8_t sa[TM * 128], sb[128 * 128];
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, n0 = blockIdx.x * 128, t0 = blockIdx.y * TM, mi = lane >> 3, lr = lane & 7;
    const uint32_t base_a = smem_u32(sa), base_b = smem_u32(sb);
    const uint16_t* w = reinterpret_cast<const uint16_t*>(p.low_w) + (size_t)n0 * p.low_k;  // rows padded to whole blocks
    auto load_w = [&](int k0) {
        for (int c = tid; c < 128 * 8; c += 256) cp_async16(base_b + (c >> 3) * 128 + (((c & 7) ^ ((c >> 3) & 7)) << 4), w + (size_t)(c >> 3) * p.low_k + k0 + (c & 7) * 8);
        cp_async_commit();
    };
    load_w(0);  // (weights: nothing earlier writes them)
    pdl_wait();
    float acc[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < 2; j++) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
    for (int k0 = 0; k0 < p.low_k; k0 += 64) {
        for (int c = tid; c < TM * 32; c += 256) {  // pairs of inputs
            const int r = c >> 5, x = (c & 31) * 2, col = k0 + x;
            const float* src = p.low + (size_t)(t0 + r) * p.ld_low + col;
            const bool ok = t0 + r < p.T;
            const float u = ok && col < p.rank ? tanhf(src[0]) : 0.f, v = ok && col + 1 < p.rank ? tanhf(src[1]) : 0.f;
            *reinterpret_cast<uint32_t*>(sa + r * 128 + (((x >> 3) ^ (r & 7)) << 4) + (x & 7) * 2) = pack_bf2(u, v);
        }
        cp_async_wait<0>();
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 4; k++) {
            uint32_t b0[2], b1[2];
            {
                const int r = warp * 16 + lr + (mi >> 1) * 8, ch = 2 * k + (mi & 1);
                ldmatrix_x4(b0[0], b0[1], b1[0], b1[1], base_b + r * 128 + ((ch ^ (r & 7)) << 4));
            }
#pragma unroll
            for (int i = 0; i < MT; i++) {
                const int r = i * 16 + lr + (mi & 1) * 8, ch = 2 * k + (mi >> 1);
                uint32_t f[4];
                ldmatrix_x4(f[0], f[1], f[2], f[3], base_a + r * 128 + ((ch ^ (r & 7)) << 4));
                mma_bf16_16816(acc[i][0], f, b0);
                mma_bf16_16816(acc[i][1], f, b1);
            }
        }
        __syncthreads();
        if (k0 + 64 < p.low_k) load_w(k0 + 64);
    }
    const int Q = s.q_cols();
#pragma unroll
    for (int j = 0; j < 2; j++) {
        const int col = n0 + warp * 16 + j * 8 + 2 * (lane & 3);
        if (col >= Q) continue;
        const bool two = col + 1 < Q;
        const float w0 = p.dt_bias[col], w1 = two ? p.dt_bias[col + 1] : 0.f;
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const int t = t0 + i * 16 + h * 8 + (lane >> 2);
                if (t >= p.T) continue;
                float* d = p.lg + (size_t)t * Q + col;
                const float u = log_decay_of(acc[i][j][2 * h] + w0), v = log_decay_of(acc[i][j][2 * h + 1] + w1);
                if (Q % 2 == 0) {
                    *reinterpret_cast<float2*>(d) = make_float2(u, v);
                } else {
                    d[0] = u;
                    if (two) d[1] = v;
                }
            }
    }
}

// Convolution with silu, unit vectors, decays and step sizes.  A warp takes one unit over a run of tokens: a head of q or k, a
// stretch of the values' channels, or the decays of a head (or of all heads).  TAPS 0: any number, inputs read again.
template <typename T, int TAPS, int VEC, int NCH>
__global__ void __launch_bounds__(256) memory_prep_kernel(const MemorySpec s, const MemoryParams p, int run) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, Q = s.q_cols(), C = s.channels(), V = s.heads * s.vdim;
    constexpr int SPAN = 32 * VEC * NCH;
    const int n_v = (V + SPAN - 1) / SPAN, n_conv = 2 * s.kv_heads + n_v, u = blockIdx.x * 8 + warp;
    const int t0 = blockIdx.y * run, t1 = min(t0 + run, p.T);
    const T* in = reinterpret_cast<const T*>(p.in);
    if (u >= n_conv) {
        const int h = u - n_conv;
        if (s.decay == MemDecay::PerChannel && h < s.heads) {
            const float A = -expf(p.A_log[h]);
            const T* dec = reinterpret_cast<const T*>(p.dec) + h * s.dim;
            float* lg = p.lg + h * s.dim;
            for (int d = lane * VEC; d < s.dim; d += 32 * VEC) {
                float bias[VEC];
#pragma unroll
                for (int e = 0; e < VEC; e++) bias[e] = p.dt_bias[h * s.dim + d + e];
#pragma unroll 4
                for (int t = t0; t < t1; t++) {
                    float v[VEC];
                    if constexpr (VEC == 4)
                        Elt<T>::ld4(dec + (size_t)t * p.ld_dec + d, v);
                    else
                        v[0] = Elt<T>::ld(dec + (size_t)t * p.ld_dec + d);
#pragma unroll
                    for (int e = 0; e < VEC; e++) v[e] = A * softplus_f32(v[e] + bias[e]);
                    if constexpr (VEC == 4)
                        Elt<float>::st4(lg + (size_t)t * s.decays() + d, v);
                    else
                        lg[(size_t)t * s.decays() + d] = v[0];
                }
            }
        } else if (h == (s.decay == MemDecay::PerChannel ? s.heads : 0)) {
            for (int t = t0; t < t1; t++)
                for (int i = lane; i < s.heads; i += 32) {
                    p.beta[(size_t)t * s.heads + i] = sigmoid_f32(Elt<T>::ld(in + (size_t)t * p.ld + p.b_off + i));
                    if (s.decay == MemDecay::PerHead)
                        p.lg[(size_t)t * s.heads + i] =
                            -expf(p.A_log[i]) * softplus_f32(Elt<T>::ld(reinterpret_cast<const T*>(p.dec) + (size_t)t * p.ld_dec + i) + p.dt_bias[i]);
                }
        }
        return;
    }
    // channels c0 .. c0 + n - 1 of q | k | v
    const bool is_v = u >= 2 * s.kv_heads;
    const int c0 = is_v ? 2 * Q + (u - 2 * s.kv_heads) * SPAN : u * s.dim, n = is_v ? min(SPAN, C - c0) : s.dim;
    constexpr int WT = TAPS > 0 ? TAPS : 1;
    float w[WT][NCH][VEC], win[WT][NCH][VEC];
    auto fetch = [&](int t, float (&x)[NCH][VEC]) {
        const T* r = in + (size_t)t * p.ld + p.c_off + c0;
#pragma unroll
        for (int i = 0; i < NCH; i++) {
            const int d = (i * 32 + lane) * VEC;
            if (d >= n) continue;
            if constexpr (VEC == 4)
                Elt<T>::ld4(r + d, x[i]);
            else
                x[i][0] = Elt<T>::ld(r + d);
        }
    };
#pragma unroll
    for (int j = 0; j < WT; j++)
#pragma unroll
        for (int i = 0; i < NCH; i++)
#pragma unroll
            for (int e = 0; e < VEC; e++) {
                const int d = (i * 32 + lane) * VEC + e;
                w[j][i][e] = TAPS > 0 && d < n ? p.conv_w[(size_t)j * C + c0 + d] : 0.f;
                win[j][i][e] = 0.f;
            }
    float next[NCH][VEC];  // the input of the token after this one is on its way
    if constexpr (TAPS > 0) {
        if (t0 < t1) fetch(t0, next);
    }
    int cur = -1, start = 0, before = 0;
    const float* kept = nullptr;
#pragma unroll 4
    for (int t = t0; t < t1; t++) {
        const int b = p.token_seq[t];
        if (b != cur) {
            cur = b;
            start = p.cu_seqlens[b];
            before = p.context_lens[b] - (p.cu_seqlens[b + 1] - start);  // tokens the state has seen
            kept = p.state + (size_t)p.seq_slot[b] * p.slot_stride + s.state_floats() + c0;
            if constexpr (TAPS > 1) {  // the inputs before this token: of this step, or the kept ones
#pragma unroll
                for (int j = 1; j < TAPS; j++) {
                    const int k = t - start - TAPS + j;
                    if (k >= 0) {
                        fetch(start + k, win[j]);
                    } else {
#pragma unroll
                        for (int i = 0; i < NCH; i++)
#pragma unroll
                            for (int e = 0; e < VEC; e++) {
                                const int d = (i * 32 + lane) * VEC + e;
                                win[j][i][e] = before > 0 && d < n ? kept[(size_t)(k + TAPS - 1) * C + d] : 0.f;
                            }
                    }
                }
            }
        }
        float y[NCH][VEC];
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS; j++)
#pragma unroll
                for (int i = 0; i < NCH; i++)
#pragma unroll
                    for (int e = 0; e < VEC; e++) win[j][i][e] = win[j + 1][i][e];
#pragma unroll
            for (int i = 0; i < NCH; i++)
#pragma unroll
                for (int e = 0; e < VEC; e++) win[TAPS - 1][i][e] = (i * 32 + lane) * VEC < n ? next[i][e] : 0.f;
            if (t + 1 < t1) fetch(t + 1, next);
#pragma unroll
            for (int i = 0; i < NCH; i++)
#pragma unroll
                for (int e = 0; e < VEC; e++) {
                    y[i][e] = 0.f;
#pragma unroll
                    for (int j = 0; j < TAPS; j++) y[i][e] = fmaf(w[j][i][e], win[j][i][e], y[i][e]);
                }
        } else {
#pragma unroll
            for (int i = 0; i < NCH; i++)
#pragma unroll
                for (int e = 0; e < VEC; e++) {
                    const int d = (i * 32 + lane) * VEC + e;
                    float v = 0.f;
                    for (int j = 0; d < n && j < s.conv; j++) {
                        const int k = t - start - (s.conv - 1) + j;
                        const float x = k >= 0 ? Elt<T>::ld(in + (size_t)(start + k) * p.ld + p.c_off + c0 + d) : (before > 0 ? kept[(size_t)(k + s.conv - 1) * C + d] : 0.f);
                        v = fmaf(p.conv_w[(size_t)j * C + c0 + d], x, v);
                    }
                    y[i][e] = v;
                }
        }
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NCH; i++)
#pragma unroll
            for (int e = 0; e < VEC; e++) {
                y[i][e] = (i * 32 + lane) * VEC + e < n ? silu_for<T>(y[i][e]) : 0.f;
                ss += y[i][e] * y[i][e];
            }
        if (is_v) {
            T* o = reinterpret_cast<T*>(const_cast<void*>(p.v)) + (size_t)t * p.ld_v + (c0 - 2 * Q);
#pragma unroll
            for (int i = 0; i < NCH; i++) {
                const int d = (i * 32 + lane) * VEC;
                if (d >= n) continue;
                if constexpr (VEC == 4)
                    Elt<T>::st4(o + d, y[i]);
                else
                    Elt<T>::st(o + d, y[i][0]);
            }
        } else {
            const bool is_q = u < s.kv_heads;
            float f = s.unit ? 1.0f / sqrtf(elt_warp_sum(ss) + s.unit_eps) : 1.f;
            if (is_q == s.unit) f *= rsqrtf((float)s.dim);
            float* o = (is_q ? p.q + (size_t)t * Q + c0 : p.k + (size_t)t * Q + c0 - Q);
#pragma unroll
            for (int i = 0; i < NCH; i++) {
                const int d = (i * 32 + lane) * VEC;
                if (d >= n) continue;
#pragma unroll
                for (int e = 0; e < VEC; e++) y[i][e] *= f;
                if constexpr (VEC == 4)
                    Elt<float>::st4(o + d, y[i]);
                else
                    o[d] = y[i][0];
            }
        }
    }
}

// The recurrence, token after token.  Block = (16 value rows of one head, sequence); thread = (value row, one eighth of the
// state in float4 pieces).  Tokens pass through shared memory a few at a time.  Both dots of a token -- what the decayed
// state answers to its key and to its query -- are taken together: S_new^T q = S^T q + u (k . q).  With a bonus the read-out
// comes before the decay, and the keys in k . q are weighted by it.
constexpr int SC_P = 16;
template <typename T, int K4, bool BONUS>
__global__ void __launch_bounds__(128) memory_scan_kernel(const MemorySpec s, const MemoryParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    constexpr int NP = K4 * 32, SC_T = K4 <= 4 ? 16 : 8;
    __shared__ __align__(16) float Ks[SC_T][NP], Qs[SC_T][NP], Gs[SC_T][NP];
    __shared__ float xs[SC_T][SC_P], kq[SC_T], bs[SC_T];
    const int h = blockIdx.y, b = blockIdx.z, p0 = blockIdx.x * SC_P, kh = h / (s.heads / s.kv_heads);
    const int D = s.dim, P = s.vdim, Q = s.q_cols(), V = s.heads * P;
    const int tid = threadIdx.x, pr = tid >> 3, ln = tid & 7;
    const int start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start, before = p.context_lens[b] - n;
    if (n <= 0 || (p.n_chunks > 0 && n >= kMemoryChunkMin)) return;
    float* slot = p.state + (size_t)p.seq_slot[b] * p.slot_stride;
    const bool live = p0 + pr < P, vec = D % 4 == 0;
    float* S = slot + ((size_t)h * P + p0 + pr) * D;
    float st[K4][4];
#pragma unroll
    for (int k = 0; k < K4; k++) {
        const int i0 = k * 32 + ln * 4;
        const bool ok = before > 0 && live && i0 < D;
        if (vec) {
            const float4 v = ok ? *reinterpret_cast<const float4*>(S + i0) : make_float4(0.f, 0.f, 0.f, 0.f);
            st[k][0] = v.x, st[k][1] = v.y, st[k][2] = v.z, st[k][3] = v.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++) st[k][e] = ok && i0 + e < D ? S[i0 + e] : 0.f;
        }
    }
    const T* v = reinterpret_cast<const T*>(p.v) + (size_t)h * P + p0;
    for (int t0 = 0; t0 < n; t0 += SC_T) {
        const int cnt = min(SC_T, n - t0);
        __syncthreads();
        for (int i = tid; i < cnt * NP; i += 128) {
            const int t = i / NP, c = i - t * NP;
            const size_t tok = (size_t)(start + t0 + t);
            if constexpr (BONUS) {  // straight from the projections
                const T* x = reinterpret_cast<const T*>(p.in) + tok * p.ld + p.c_off + kh * D + c;
                Ks[t][c] = c < D ? Elt<T>::ld(x + Q) : 0.f;
                Qs[t][c] = c < D ? Elt<T>::ld(x) : 0.f;
            } else {
                Ks[t][c] = c < D ? p.k[tok * Q + kh * D + c] : 0.f;
                Qs[t][c] = c < D ? p.q[tok * Q + kh * D + c] : 0.f;
            }
            float g = 1.f;
            if (c < D)
                g = s.decay == MemDecay::PerChannel ? expf(p.lg[tok * s.decays() + h * D + c]) : s.decay == MemDecay::PerHead ? expf(p.lg[tok * s.heads + h]) : p.decay[h];
            Gs[t][c] = g;
        }
        for (int i = tid; i < cnt * SC_P; i += 128) {
            const int t = i / SC_P, c = i - t * SC_P;
            xs[t][c] = p0 + c < P ? Elt<T>::ld(v + (size_t)(start + t0 + t) * p.ld_v + c) : 0.f;
        }
        if (tid < cnt && s.delta) bs[tid] = p.beta[(size_t)(start + t0 + tid) * s.heads + h];
        __syncthreads();
        {  // k . q of every token: eight threads each
            const int t = min(pr, SC_T - 1);
            float d = 0.f;
            if (t < cnt)
                for (int i = ln; i < NP; i += 8) d = fmaf(BONUS && i < D ? Ks[t][i] * p.bonus[(size_t)h * D + i] : Ks[t][i], Qs[t][i], d);
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
            if (ln == 0) kq[t] = d;
        }
        __syncthreads();
        for (int t = 0; t < cnt; t++) {
            float d1 = 0.f, d2 = 0.f;
            float4 kk[K4];
#pragma unroll
            for (int k = 0; k < K4; k++) {
                const int at = k * 32 + ln * 4;
                kk[k] = *reinterpret_cast<const float4*>(&Ks[t][at]);
                const float4 q = *reinterpret_cast<const float4*>(&Qs[t][at]), g = *reinterpret_cast<const float4*>(&Gs[t][at]);
                if constexpr (BONUS) {
                    d2 = fmaf(q.x, st[k][0], d2), st[k][0] *= g.x;
                    d2 = fmaf(q.y, st[k][1], d2), st[k][1] *= g.y;
                    d2 = fmaf(q.z, st[k][2], d2), st[k][2] *= g.z;
                    d2 = fmaf(q.w, st[k][3], d2), st[k][3] *= g.w;
                } else {
                    st[k][0] *= g.x, d1 = fmaf(kk[k].x, st[k][0], d1), d2 = fmaf(q.x, st[k][0], d2);
                    st[k][1] *= g.y, d1 = fmaf(kk[k].y, st[k][1], d1), d2 = fmaf(q.y, st[k][1], d2);
                    st[k][2] *= g.z, d1 = fmaf(kk[k].z, st[k][2], d1), d2 = fmaf(q.z, st[k][2], d2);
                    st[k][3] *= g.w, d1 = fmaf(kk[k].w, st[k][3], d1), d2 = fmaf(q.w, st[k][3], d2);
                }
            }
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) {
                if (!BONUS) d1 += __shfl_xor_sync(0xffffffffu, d1, o);
                d2 += __shfl_xor_sync(0xffffffffu, d2, o);
            }
            const float x = xs[t][pr], u = !BONUS && s.delta ? bs[t] * (x - d1) : x;
#pragma unroll
            for (int k = 0; k < K4; k++) {
                st[k][0] = fmaf(kk[k].x, u, st[k][0]);
                st[k][1] = fmaf(kk[k].y, u, st[k][1]);
                st[k][2] = fmaf(kk[k].z, u, st[k][2]);
                st[k][3] = fmaf(kk[k].w, u, st[k][3]);
            }
            if (ln == 0 && live) p.o[(size_t)(start + t0 + t) * V + h * P + p0 + pr] = fmaf(u, kq[t], d2);
        }
    }
    if (live) {
#pragma unroll
        for (int k = 0; k < K4; k++) {
            const int i0 = k * 32 + ln * 4;
            if (vec && i0 < D) {
                *reinterpret_cast<float4*>(S + i0) = make_float4(st[k][0], st[k][1], st[k][2], st[k][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (i0 + e < D) S[i0 + e] = st[k][e];
            }
        }
    }
    memory_keep_inputs<T>(s, p, b, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
}

// A warp per (token, memory head) and per (token, 256 feed-forward columns); the last unit writes the zeros between the parts.
// With heads of up to 64 values (`pairs` > 0) half a warp per head, and that many warps walk over the heads.
template <typename T>
__global__ void __launch_bounds__(256) branch_out_kernel(const BranchOutParams p, int pairs) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n_m = p.o ? (pairs > 0 ? pairs : p.heads) : 0, n_f = p.up ? (p.ff + 255) / 256 : 0;
    T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo;
    int u = blockIdx.y * 8 + warp;
    if (u < n_m && pairs > 0) {
        const int P = p.vdim, d = (lane & 15) * 4;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int h0 = u * 2; h0 < p.heads; h0 += 2 * pairs) {
            const int h = h0 + (lane >> 4);
            const bool ok = h < p.heads && d < P;
            const size_t at = (size_t)h * P + d;
            const float4 v = ok ? *reinterpret_cast<const float4*>(p.o + (size_t)t * p.heads * P + at) : zero;
            float g[4] = {0.f, 0.f, 0.f, 0.f}, w[4] = {1.f, 1.f, 1.f, 1.f};
            if (ok) Elt<T>::ld4(reinterpret_cast<const T*>(p.gate) + (size_t)t * p.ld_gate + at, g);
            if (ok && p.norm) Elt<float>::ld4(p.norm_heads ? p.norm + at : p.norm + d, w);
            float ss = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float inv = p.scale / sqrtf(ss / (float)P + p.eps);
            if (!ok) continue;
#pragma unroll
            for (int e = 0; e < 4; e++) w[e] *= inv * (p.act == MemGate::Silu ? silu_for<T>(g[e]) : sigmoid_f32(g[e]));
            const float r[4] = {v.x * w[0], v.y * w[1], v.z * w[2], v.w * w[3]};
            Elt<T>::st4(out + p.m_off + at, r);
        }
        return;
    }
    if (u < n_m) {
        const int P = p.vdim;
        const float* o = p.o + ((size_t)t * p.heads + u) * P;
        const T* z = reinterpret_cast<const T*>(p.gate) + (size_t)t * p.ld_gate + u * P;
        T* dst = out + p.m_off + u * P;
        const float* norm = p.norm && p.norm_heads ? p.norm + (size_t)u * P : p.norm;
        const bool vec = P % 4 == 0 && p.ld_gate % 4 == 0 && ((uintptr_t)p.gate & (sizeof(T) * 4 - 1)) == 0 && p.m_off % 4 == 0;
        auto gated = [&](float v, float g) { return v * (p.act == MemGate::Silu ? silu_f32(g) : sigmoid_f32(g)); };
        float ss = 0.f;
        if (vec && P <= 256) {
            float4 v[2];
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int d = (i * 32 + lane) * 4;
                v[i] = d < P ? *reinterpret_cast<const float4*>(o + d) : make_float4(0.f, 0.f, 0.f, 0.f);
                ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
            }
            const float inv = p.scale / sqrtf(elt_warp_sum(ss) / (float)P + p.eps);
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int d = (i * 32 + lane) * 4;
                if (d >= P) continue;
                float g[4], w[4] = {1.f, 1.f, 1.f, 1.f};
                Elt<T>::ld4(z + d, g);
                if (norm) Elt<float>::ld4(norm + d, w);
                const float r[4] = {gated(v[i].x * inv * w[0], g[0]), gated(v[i].y * inv * w[1], g[1]), gated(v[i].z * inv * w[2], g[2]), gated(v[i].w * inv * w[3], g[3])};
                Elt<T>::st4(dst + d, r);
            }
        } else {
            for (int d = lane; d < P; d += 32) ss += o[d] * o[d];
            const float inv = p.scale / sqrtf(elt_warp_sum(ss) / (float)P + p.eps);
            for (int d = lane; d < P; d += 32) Elt<T>::st(dst + d, gated(o[d] * inv * (norm ? norm[d] : 1.f), Elt<T>::ld(z + d)));
        }
        return;
    }
    u -= n_m;
    if (u < n_f) {
        const T* x = reinterpret_cast<const T*>(p.up) + (size_t)t * p.ld_up;
        const int c0 = u * 256 + lane * 8;
        auto gelu = [](float v) { return 0.5f * v * (1.0f + erff(v * 0.7071067811865476f)); };
        if (c0 + 8 <= p.ff && ((uintptr_t)p.up & 15) == 0 && p.ld_up % 8 == 0 && p.f_off % 8 == 0) {
            float v[8];
            Elt<T>::ld8(x + c0, v);
#pragma unroll
            for (int e = 0; e < 8; e++) v[e] = gelu(v[e]);
            Elt<T>::st8(out + p.f_off + c0, v);
        } else {
            for (int c = c0; c < min(c0 + 8, p.ff); c++) Elt<T>::st(out + p.f_off + c, gelu(Elt<T>::ld(x + c)));
        }
        return;
    }
    if (u > n_f) return;
    int at = p.att_cols;  // ends of the parts, in order
    auto zero_to = [&](int c1) {
        for (int c = at + lane; c < c1; c += 32) Elt<T>::st(out + c, 0.f);
    };
    if (p.o) zero_to(p.m_off), at = p.m_off + p.heads * p.vdim;
    if (n_f) zero_to(p.f_off), at = p.f_off + p.ff;
    zero_to(p.ldo);
}

template <typename T, int VEC, int NCH>
int32_t launch_prep(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p) {
    constexpr int SPAN = 32 * VEC * NCH;
    const int units = 2 * s.kv_heads + (s.heads * s.vdim + SPAN - 1) / SPAN + (s.decay == MemDecay::PerChannel ? s.heads : 0) + 1;
    const int bx = (units + 7) / 8, want = 12 * ctx->sm_count / bx + 1;  // blocks along the tokens
    const int run = p.T > want ? (p.T + want - 1) / want : 1;
    auto k = s.conv == 1 ? memory_prep_kernel<T, 1, VEC, NCH> : s.conv == 2 ? memory_prep_kernel<T, 2, VEC, NCH> : s.conv == 3 ? memory_prep_kernel<T, 3, VEC, NCH>
             : s.conv == 4 ? memory_prep_kernel<T, 4, VEC, NCH> : memory_prep_kernel<T, 0, VEC, NCH>;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3(bx, (p.T + run - 1) / run), dim3(256), 0, ctx->stream, s, p, run));
    B2_LAUNCHED(ctx);
    return B2_OK;
}

template <typename T>
int32_t launch_memory(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p) {
    if (s.shift > 0) {
        if (p.low) {
            const int bx = (s.q_cols() + 127) / 128;
            B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, p.T <= 16 ? memory_decay_tc_kernel<1> : memory_decay_tc_kernel<4>, dim3(bx, p.T <= 16 ? 1 : (p.T + 63) / 64), dim3(256), 0, ctx->stream,
                                  s, p));
        } else {
            B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, memory_decay_kernel, dim3((s.q_cols() + 255) / 256, p.T), dim3(256), 0, ctx->stream, s, p));
        }
        B2_LAUNCHED(ctx);
    } else if (s.conv > 0) {
        const bool vec = s.dim % 4 == 0 && (s.heads * s.vdim) % 4 == 0 && p.ld_dec % 4 == 0 && p.c_off % 4 == 0 && p.ld % 4 == 0 && p.ld_v % 4 == 0;
        if (!vec)
            B2_CHECK((launch_prep<T, 1, 8>(ctx, s, p)));
        else if (s.dim <= 128)
            B2_CHECK((launch_prep<T, 4, 1>(ctx, s, p)));
        else
            B2_CHECK((launch_prep<T, 4, 2>(ctx, s, p)));
    } else {
        const bool vec = s.dim % 4 == 0 && s.rot.dims % 8 == 0 && p.c_off % 4 == 0 && p.ld % 4 == 0;
        const int by = (2 * s.q_cols() / (vec ? 4 : 1) + 1023) / 1024;  // up to four pieces per thread
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, vec ? memory_rotate_kernel<T, 4> : memory_rotate_kernel<T, 1>, dim3(p.T, by), dim3(256), 0, ctx->stream, s, p));
        B2_LAUNCHED(ctx);
    }
    if (p.n_chunks > 0) B2_CHECK(b2_memory_chunk_launch(ctx, s, p));
    if (p.n_chunks == 0 || p.B > 1) {
        const int k4 = (s.dim + 31) / 32;
        auto k = s.bonus ? (k4 <= 1 ? memory_scan_kernel<T, 1, true> : k4 <= 2 ? memory_scan_kernel<T, 2, true> : k4 <= 4 ? memory_scan_kernel<T, 4, true> : memory_scan_kernel<T, 8, true>)
                         : (k4 <= 1 ? memory_scan_kernel<T, 1, false> : k4 <= 2 ? memory_scan_kernel<T, 2, false> : k4 <= 4 ? memory_scan_kernel<T, 4, false> : memory_scan_kernel<T, 8, false>);
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3((s.vdim + SC_P - 1) / SC_P, s.heads, p.B), dim3(128), 0, ctx->stream, s, p));
        B2_LAUNCHED(ctx);
    }
    return B2_OK;
}

}  // namespace

int32_t b2_memory_launch(b2_ctx* ctx, bool f32, const MemorySpec& s, const MemoryParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_REQUIRE(s.dim <= 256, B2_ERR_UNSUPPORTED, "memory: key sizes up to 256");
    B2_REQUIRE(!(s.conv > 0 && s.rot.dims > 0), B2_ERR_UNSUPPORTED, "memory: a convolution and a rotation together");
    B2_REQUIRE(s.conv > 0 || s.shift > 0 || (!s.unit && !s.delta && s.decay == MemDecay::Fixed), B2_ERR_UNSUPPORTED,
               "memory: unit vectors, a delta rule or learned decays without a convolution or a token shift");
    B2_REQUIRE(s.shift == 0 || (s.conv == 0 && s.rot.dims == 0 && !s.unit && !s.delta && s.decay == MemDecay::PerChannel && s.decay_map == DecayMap::Exp && s.kv_heads == s.heads),
               B2_ERR_UNSUPPORTED, "memory: a token shift goes with plain queries and keys and a decay per channel");
    B2_REQUIRE(!s.bonus || (!s.delta && s.decay == MemDecay::PerChannel), B2_ERR_UNSUPPORTED, "memory: a bonus goes with decays per channel, without the delta rule");
    return f32 ? launch_memory<float>(ctx, s, p) : launch_memory<uint16_t>(ctx, s, p);
}
int32_t b2_token_shift_launch(b2_ctx* ctx, bool f32, const ShiftParams& p) {
    if (p.T <= 0) return B2_OK;
    const bool vec = p.width % 4 == 0 && p.ld_h % 4 == 0 && p.ldo % 4 == 0;
    const int bx = (p.ldo + (vec ? 1023 : 255)) / (vec ? 1024 : 256), want = 8 * ctx->sm_count / bx + 1;  // blocks along the tokens
    const int run = p.T > want ? (p.T + want - 1) / want : 1;
    auto k = vec ? (f32 ? token_shift_kernel<float, 4> : token_shift_kernel<uint16_t, 4>) : (f32 ? token_shift_kernel<float, 1> : token_shift_kernel<uint16_t, 1>);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3(bx, (p.T + run - 1) / run), dim3(256), 0, ctx->stream, p, run));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_branch_out_launch(b2_ctx* ctx, bool f32, const BranchOutParams& p) {
    if (p.T <= 0) return B2_OK;
    if (!p.o && !p.up && p.att_cols == p.ldo) return B2_OK;  // nothing to add, no padding
    const bool narrow = p.o && p.vdim <= 64 && p.vdim % 4 == 0 && p.ld_gate % 4 == 0 && ((uintptr_t)p.gate & (f32 ? 15 : 7)) == 0 && p.m_off % 4 == 0;
    const int pairs = narrow ? (p.T <= 2 * ctx->sm_count ? (p.heads + 1) / 2 : 8) : 0;  // (many tokens: fewer, longer warps)
    const int units = (p.o ? (pairs > 0 ? pairs : p.heads) : 0) + (p.up ? (p.ff + 255) / 256 : 0) + 1;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? branch_out_kernel<float> : branch_out_kernel<uint16_t>, dim3(p.T, (units + 7) / 8), dim3(256), 0, ctx->stream, p, pairs));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
