// Mamba-2 mixer between its two projections: short causal convolution with silu, selective state-space recurrence with
// one decay per head, gate and grouped RMS norm.
//
// Recurrent state of a sequence (f32, one slot per block-table row of the pool):
//   S     [heads][vdim][state]
//   conv  [channels][taps - 1]   the last inputs of the convolution, oldest first
// A sequence that starts in this step (nothing cached) starts from zero, whatever its slot held before.
//
// Per token and head:  d = softplus(dt + bias),  S <- exp(-exp(A_log) d) S + d x B^T,  y = S C + D x   (all f32).
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

template <typename T>
__global__ void __launch_bounds__(256) conv_silu_kernel(const Mamba2Spec s, const SsmParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int t = blockIdx.y, ch = blockIdx.x * 256 + threadIdx.x, C = s.channels(), taps = s.conv;
    if (ch >= C) return;
    const int b = p.token_seq[t], start = p.cu_seqlens[b], i = t - start;
    const int before = p.context_lens[b] - (p.cu_seqlens[b + 1] - start);  // tokens the state has seen
    const T* u = reinterpret_cast<const T*>(p.zx) + s.inner() + ch;
    const float* cs = p.state + (size_t)p.seq_slot[b] * p.slot_stride + (size_t)s.heads * s.vdim * s.state + (size_t)ch * (taps - 1);
    float v = p.conv_b[ch];
    for (int j = 0; j < taps; j++) {
        const int k = i - (taps - 1) + j;  // token of this step, or (negative) a kept one
        const float in = k >= 0 ? Elt<T>::ld(u + (size_t)(start + k) * p.ld) : (before > 0 ? cs[k + taps - 1] : 0.f);
        v = fmaf(p.conv_w[(size_t)ch * taps + j], in, v);
    }
    Elt<T>::st(reinterpret_cast<T*>(p.xbc) + (size_t)t * p.ld_xbc + ch, silu_f32(v));
}

// The recurrence, token after token.  Block = (16 value rows of one head, sequence); thread = (value row, one eighth of
// the state in float4 pieces).  Tokens pass through shared memory 16 at a time.
constexpr int SC_P = 16, SC_T = 16;
template <typename T, int K4>
__global__ void __launch_bounds__(128) scan_kernel(const Mamba2Spec s, const SsmParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    constexpr int NP = K4 * 32;  // padded state size
    __shared__ __align__(16) float Bs[SC_T][NP], Cs[SC_T][NP];
    __shared__ float xs[SC_T][SC_P], da[SC_T], dd[SC_T];
    const int h = blockIdx.y, b = blockIdx.z, p0 = blockIdx.x * SC_P;
    const int P = s.vdim, N = s.state, inner = s.inner(), taps = s.conv, grp = h / (s.heads / s.groups);
    const int tid = threadIdx.x, pr = tid >> 3, ln = tid & 7;
    const int start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start, before = p.context_lens[b] - n;
    if (n <= 0) return;
    float* slot = p.state + (size_t)p.seq_slot[b] * p.slot_stride;
    const bool live = p0 + pr < P;
    float* S = slot + ((size_t)h * P + p0 + pr) * N;
    float st[K4][4];
#pragma unroll
    for (int k = 0; k < K4; k++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int i = k * 32 + ln * 4 + e;
            st[k][e] = (before > 0 && live && i < N) ? S[i] : 0.f;
        }
    const T* zx = reinterpret_cast<const T*>(p.zx);
    const T* xbc = reinterpret_cast<const T*>(p.xbc);
    const float A = expf(p.A_log[h]), bias = p.dt_bias[h], D = p.D[h];
    for (int t0 = 0; t0 < n; t0 += SC_T) {
        const int cnt = min(SC_T, n - t0);
        __syncthreads();
        for (int i = tid; i < cnt * NP; i += 128) {
            const int t = i / NP, c = i - t * NP;
            const T* r = xbc + (size_t)(start + t0 + t) * p.ld_xbc + inner + grp * N;
            Bs[t][c] = c < N ? Elt<T>::ld(r + c) : 0.f;
            Cs[t][c] = c < N ? Elt<T>::ld(r + s.groups * N + c) : 0.f;
        }
        for (int i = tid; i < cnt * SC_P; i += 128) {
            const int t = i / SC_P, c = i - t * SC_P;
            xs[t][c] = p0 + c < P ? Elt<T>::ld(xbc + (size_t)(start + t0 + t) * p.ld_xbc + h * P + p0 + c) : 0.f;
        }
        if (tid < cnt) {
            const float d = softplus_f32(Elt<T>::ld(zx + (size_t)(start + t0 + tid) * p.ld + 2 * inner + 2 * s.groups * N + h) + bias);
            dd[tid] = d;
            da[tid] = expf(-A * d);
        }
        __syncthreads();
        for (int t = 0; t < cnt; t++) {
            const float x = xs[t][pr], a = da[t], dx = dd[t] * x;
            float y = 0.f;
#pragma unroll
            for (int k = 0; k < K4; k++) {
                const float4 B = *reinterpret_cast<const float4*>(&Bs[t][k * 32 + ln * 4]), C = *reinterpret_cast<const float4*>(&Cs[t][k * 32 + ln * 4]);
                st[k][0] = fmaf(B.x, dx, a * st[k][0]), y = fmaf(C.x, st[k][0], y);
                st[k][1] = fmaf(B.y, dx, a * st[k][1]), y = fmaf(C.y, st[k][1], y);
                st[k][2] = fmaf(B.z, dx, a * st[k][2]), y = fmaf(C.z, st[k][2], y);
                st[k][3] = fmaf(B.w, dx, a * st[k][3]), y = fmaf(C.w, st[k][3], y);
            }
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
            if (ln == 0 && live) p.y[(size_t)(start + t0 + t) * inner + h * P + p0 + pr] = fmaf(D, x, y);
        }
    }
    if (live) {
#pragma unroll
        for (int k = 0; k < K4; k++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = k * 32 + ln * 4 + e;
                if (i < N) S[i] = st[k][e];
            }
    }
    // the convolution's kept inputs: the block's own x channels, and the group's B and C channels once per group
    float* conv = slot + (size_t)s.heads * P * N;
    auto keep = [&](int ch) {
        float* c = conv + (size_t)ch * (taps - 1);
        const T* u = zx + inner + ch;
        for (int j = 0; j < taps - 1; j++) {  // ascending: a shift reads places it has not overwritten yet
            const int k = n - (taps - 1) + j;
            c[j] = k >= 0 ? Elt<T>::ld(u + (size_t)(start + k) * p.ld) : (before > 0 ? c[j + n] : 0.f);
        }
    };
    for (int c = tid; c < SC_P && p0 + c < P; c += 128) keep(h * P + p0 + c);
    if (blockIdx.x == 0 && h % (s.heads / s.groups) == 0)
        for (int c = tid; c < N; c += 128) {
            keep(inner + grp * N + c);
            keep(inner + s.groups * N + grp * N + c);
        }
}

// out = norm over equal parts of (y * silu(z)), times w; zero up to the padded width
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const Mamba2Spec s, const SsmParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    __shared__ float red[33];
    const int t = blockIdx.x, g = blockIdx.y, inner = s.inner(), part = inner / s.norm_groups, c0 = g * part;
    const T* z = reinterpret_cast<const T*>(p.zx) + (size_t)t * p.ld;
    float* y = p.y + (size_t)t * inner;
    float ss = 0.f;
    for (int i = c0 + threadIdx.x; i < c0 + part; i += blockDim.x) {
        const float v = y[i] * silu_f32(Elt<T>::ld(z + i));
        y[i] = v;  // read back by the same thread below
        ss += v * v;
    }
    ss = elt_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)part + p.eps);
    T* o = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo;
    for (int i = c0 + threadIdx.x; i < c0 + part; i += blockDim.x) Elt<T>::st(o + i, y[i] * inv * p.norm[i]);
    if (g == s.norm_groups - 1)
        for (int i = inner + threadIdx.x; i < p.ldo; i += blockDim.x) Elt<T>::st(o + i, 0.f);
}

template <typename T>
int32_t launch_ssm(b2_ctx* ctx, const Mamba2Spec& s, const SsmParams& p) {
    B2_REQUIRE(p.T <= 65535, B2_ERR_UNSUPPORTED, "mamba2: too many tokens in one step");
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, conv_silu_kernel<T>, dim3((s.channels() + 255) / 256, p.T), dim3(256), 0, ctx->stream, s, p));
    B2_LAUNCHED(ctx);
    const dim3 grid((s.vdim + SC_P - 1) / SC_P, s.heads, p.B);
    const int k4 = (s.state + 31) / 32;
    auto k = k4 <= 1 ? scan_kernel<T, 1> : k4 <= 2 ? scan_kernel<T, 2> : k4 <= 4 ? scan_kernel<T, 4> : scan_kernel<T, 8>;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, grid, dim3(128), 0, ctx->stream, s, p));
    B2_LAUNCHED(ctx);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gated_norm_kernel<T>, dim3(p.T, s.norm_groups), dim3(256), 0, ctx->stream, s, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}

}  // namespace

int32_t b2_ssm_launch(b2_ctx* ctx, bool f32, const Mamba2Spec& s, const SsmParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_REQUIRE(s.state <= 256, B2_ERR_UNSUPPORTED, "mamba2: state sizes up to 256");
    return f32 ? launch_ssm<float>(ctx, s, p) : launch_ssm<uint16_t>(ctx, s, p);
}
