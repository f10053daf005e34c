// Mamba-2 mixer between its two projections: short causal convolution with silu, selective state-space recurrence with
// one decay per head, gate and grouped RMS norm.
//
// Recurrent state of a sequence (f32, one slot per block-table row of the pool):
//   S     [heads][vdim][state]
//   conv  [taps - 1][channels]   the last inputs of the convolution, oldest first
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
    const float* cs = p.state + (size_t)p.seq_slot[b] * p.slot_stride + (size_t)s.heads * s.vdim * s.state + ch;
    float v = p.conv_b[ch];
    for (int j = 0; j < taps; j++) {
        const int k = i - (taps - 1) + j;  // token of this step, or (negative) a kept one
        const float in = k >= 0 ? Elt<T>::ld(u + (size_t)(start + k) * p.ld) : (before > 0 ? cs[(size_t)(k + taps - 1) * C] : 0.f);
        v = fmaf(p.conv_w[(size_t)j * C + ch], in, v);
    }
    Elt<T>::st(reinterpret_cast<T*>(p.xbc) + (size_t)t * p.ld_xbc + ch, silu_f32(v));
}

// The same for eight channels and a run of tokens per thread (sizes and offsets that allow 16-byte accesses): weights stay in
// registers, the window slides while the tokens belong to one sequence.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_silu8_kernel(const Mamba2Spec s, const SsmParams p, int run) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int ch = (blockIdx.x * 128 + threadIdx.x) * 8, C = s.channels();
    if (ch >= C) return;
    float w[TAPS][8], bias[8], win[TAPS][8];
    Elt<float>::ld8(p.conv_b + ch, bias);
#pragma unroll
    for (int j = 0; j < TAPS; j++) Elt<float>::ld8(p.conv_w + (size_t)j * C + ch, w[j]);
    const T* u = reinterpret_cast<const T*>(p.zx) + s.inner() + ch;
    int cur = -1;
    const int t_end = min((int)(blockIdx.y + 1) * run, p.T);
    float next[8];  // the input of the token after this one is on its way
    Elt<T>::ld8(u + (size_t)(blockIdx.y * run) * p.ld, next);
#pragma unroll 4
    for (int t = blockIdx.y * run; t < t_end; t++) {
        const int b = p.token_seq[t];
        if (b != cur) {  // the inputs before this token: of this step, or the kept ones
            cur = b;
            const int start = p.cu_seqlens[b], before = p.context_lens[b] - (p.cu_seqlens[b + 1] - start);
            const float* cs = p.state + (size_t)p.seq_slot[b] * p.slot_stride + (size_t)s.heads * s.vdim * s.state + ch;
#pragma unroll
            for (int j = 1; j < TAPS; j++) {
                const int k = t - start - TAPS + j;
                if (k >= 0) {
                    Elt<T>::ld8(u + (size_t)(start + k) * p.ld, win[j]);
                } else {
#pragma unroll
                    for (int e = 0; e < 8; e++) win[j][e] = before > 0 ? cs[(size_t)(k + TAPS - 1) * C + e] : 0.f;
                }
            }
        }
#pragma unroll
        for (int j = 0; j + 1 < TAPS; j++)
#pragma unroll
            for (int e = 0; e < 8; e++) win[j][e] = win[j + 1][e];
#pragma unroll
        for (int e = 0; e < 8; e++) win[TAPS - 1][e] = next[e];
        if (t + 1 < t_end) Elt<T>::ld8(u + (size_t)(t + 1) * p.ld, next);
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; e++) {
            v[e] = bias[e];
#pragma unroll
            for (int j = 0; j < TAPS; j++) v[e] = fmaf(w[j][e], win[j][e], v[e]);
            v[e] = silu_for<T>(v[e]);
        }
        Elt<T>::st8(reinterpret_cast<T*>(p.xbc) + (size_t)t * p.ld_xbc + ch, v);
    }
}

// The convolution's kept inputs after `n` tokens: the block's own x channels (value rows p0.. of head h) and, once per
// group, its B and C channels.
template <typename T>
__device__ __forceinline__ void keep_conv_inputs(const Mamba2Spec& s, const SsmParams& p, float* slot, int start, int n, int before, int h, int p0, int rows,
                                                 bool first_block) {
    const int P = s.vdim, N = s.state, inner = s.inner(), taps = s.conv, per = s.heads / s.groups, grp = h / per, C = s.channels();
    float* conv = slot + (size_t)s.heads * P * N;
    auto keep = [&](int ch) {
        float* c = conv + ch;
        const T* u = reinterpret_cast<const T*>(p.zx) + inner + ch;
        for (int j = 0; j < taps - 1; j++) {  // ascending: a shift reads places it has not overwritten yet
            const int k = n - (taps - 1) + j;
            c[(size_t)j * C] = k >= 0 ? Elt<T>::ld(u + (size_t)(start + k) * p.ld) : (before > 0 ? c[(size_t)(j + n) * C] : 0.f);
        }
    };
    for (int c = threadIdx.x; c < rows && p0 + c < P; c += blockDim.x) keep(h * P + p0 + c);
    if (first_block && h % per == 0)
        for (int c = threadIdx.x; c < N; c += blockDim.x) {
            keep(inner + grp * N + c);
            keep(inner + s.groups * N + grp * N + c);
        }
}

// The recurrence, token after token.  Block = (16 value rows of one head, sequence); thread = (value row, one eighth of
// the state in float4 pieces).  Tokens pass through shared memory 16 at a time.
constexpr int SC_P = 16, SC_T = 16;
constexpr int kChunkMin = 9;  // shortest portion that the chunked form takes
template <typename T, int K4>
__global__ void __launch_bounds__(128) scan_kernel(const Mamba2Spec s, const SsmParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    constexpr int NP = K4 * 32;  // padded state size
    __shared__ __align__(16) float Bs[SC_T][NP], Cs[SC_T][NP];
    __shared__ float xs[SC_T][SC_P], da[SC_T], dd[SC_T];
    const int h = blockIdx.y, b = blockIdx.z, p0 = blockIdx.x * SC_P;
    const int P = s.vdim, N = s.state, inner = s.inner(), grp = h / (s.heads / s.groups);
    const int tid = threadIdx.x, pr = tid >> 3, ln = tid & 7;
    const int start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start, before = p.context_lens[b] - n;
    if (n <= 0 || (p.chunked && n >= kChunkMin)) return;
    float* slot = p.state + (size_t)p.seq_slot[b] * p.slot_stride;
    const bool live = p0 + pr < P;
    float* S = slot + ((size_t)h * P + p0 + pr) * N;
    float st[K4][4];
    const bool vec = N % 4 == 0;  // the state's rows are 16-byte aligned then
#pragma unroll
    for (int k = 0; k < K4; k++) {
        const int i0 = k * 32 + ln * 4;
        const bool ok = before > 0 && live && i0 < N;
        if (vec) {
            const float4 v = ok ? *reinterpret_cast<const float4*>(S + i0) : make_float4(0.f, 0.f, 0.f, 0.f);
            st[k][0] = v.x, st[k][1] = v.y, st[k][2] = v.z, st[k][3] = v.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++) st[k][e] = ok && i0 + e < N ? S[i0 + e] : 0.f;
        }
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
        for (int k = 0; k < K4; k++) {
            const int i0 = k * 32 + ln * 4;
            if (vec && i0 < N) {
                *reinterpret_cast<float4*>(S + i0) = make_float4(st[k][0], st[k][1], st[k][2], st[k][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (i0 + e < N) S[i0 + e] = st[k][e];
            }
        }
    }
    keep_conv_inputs<T>(s, p, slot, start, n, before, h, p0, SC_P, blockIdx.x == 0);
}

// ---- prompts in the serving format: the recurrence 64 tokens at a time on tensor cores ------------------------------
// With c_t the running sum of -exp(A_log) d over a chunk and S0 the state before it,
//     y_t = exp(c_t) C_t S0 + sum_{s <= t} (C_t . B_s) exp(c_t - c_s) d_s x_s + D x_t
//     S   = exp(c_end) S0 + sum_s B_s (exp(c_end - c_s) d_s x_s)^T
// B, C and x are bf16 (the convolution's outputs) and enter the products as they are; every factor that is f32 by
// nature -- the state, the decays, the step sizes and what they multiply -- enters as a bf16 head plus a bf16 remainder,
// and all sums are f32.  The state stays in f32 registers from chunk to chunk.
//
// Block = (64 value rows of one head, sequence), 16 warps.  First the weights (C_t . B_s) exp(c_t - c_s) d_s of the chunk, a
// 16 x 16 tile per warp up to the diagonal, into shared memory; then y, a warp per 16 tokens x 16 value rows; then the
// state, a warp per 16 state rows x 32 value rows.  The next chunk's x, B and C arrive by cp.async meanwhile.
constexpr int CH_T = 64, CH_P = 64, CH_N = 128, CH_THREADS = 512;  // tokens, value rows, largest state
constexpr int CH_LN = CH_N + 8, CH_LP = CH_P + 8, CH_LM = CH_T + 8;  // row strides in shared memory (conflict-free ldmatrix)
struct ChunkSmem {
    static constexpr int kIn = (2 * CH_T * CH_LN + CH_T * CH_LP) * 2;  // C | B | x of one chunk
    static constexpr int kXw = 2 * CH_T * CH_LP * 2, kM = 2 * CH_T * CH_LM * 2, kS = 2 * CH_N * CH_LP * 2;
    static constexpr int kBytes = 2 * kIn + kXw + kM + kS + 2 * 4 * CH_T * 4;
};

__global__ void __launch_bounds__(CH_THREADS, 1) chunk_scan_kernel(const Mamba2Spec s, const SsmParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int h = blockIdx.y, b = blockIdx.z, p0 = blockIdx.x * CH_P;
    const int start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start, before = p.context_lens[b] - n;
    if (n < kChunkMin) return;  // the token-by-token kernel's
    extern __shared__ __align__(16) uint8_t smem[];
    const int P = s.vdim, N = s.state, inner = s.inner(), grp = h / (s.heads / s.groups);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, lr = lane & 7, g4 = lane >> 2, t4 = lane & 3;
    const int KN = (N + 15) / 16;
    uint8_t* const in0 = smem;
    uint16_t* xw = reinterpret_cast<uint16_t*>(smem + 2 * ChunkSmem::kIn);  // head, remainder [token][value row]
    uint16_t* sm = reinterpret_cast<uint16_t*>(smem + 2 * ChunkSmem::kIn + ChunkSmem::kXw);  // weights, head, remainder [token][earlier token]
    uint16_t* sh = reinterpret_cast<uint16_t*>(smem + 2 * ChunkSmem::kIn + ChunkSmem::kXw + ChunkSmem::kM);  // head, remainder [state row][value row]
    float* steps = reinterpret_cast<float*>(smem + 2 * ChunkSmem::kIn + ChunkSmem::kXw + ChunkSmem::kM + ChunkSmem::kS);  // two chunks' step sizes and decays
    const uint16_t* zx = reinterpret_cast<const uint16_t*>(p.zx);
    const uint16_t* xbc = reinterpret_cast<const uint16_t*>(p.xbc) + (size_t)start * p.ld_xbc;
    const float A = expf(p.A_log[h]), bias = p.dt_bias[h], D = p.D[h];
    const bool vec = P % 8 == 0 && N % 8 == 0 && inner % 8 == 0;
    // x, B, C of chunk c into buffer c & 1; rows past the portion and columns past the sizes are zero
    auto load = [&](int c) {
        uint16_t* dC = reinterpret_cast<uint16_t*>(in0 + (c & 1) * ChunkSmem::kIn);
        uint16_t *dB = dC + CH_T * CH_LN, *dx = dB + CH_T * CH_LN;
        const int t0 = c * CH_T, cB = inner + grp * N, cC = cB + s.groups * N, cx = h * P + p0;
        if (vec) {
            for (int i = tid; i < CH_T * (CH_N / 8); i += CH_THREADS) {
                const int t = i / (CH_N / 8), k = (i % (CH_N / 8)) * 8;
                const bool ok = t0 + t < n && k < N;
                const uint16_t* r = xbc + (size_t)(ok ? t0 + t : 0) * p.ld_xbc;
                cp_async16_zfill(smem_u32(dC + t * CH_LN + k), r + (ok ? cC + k : 0), ok);
                cp_async16_zfill(smem_u32(dB + t * CH_LN + k), r + (ok ? cB + k : 0), ok);
            }
            for (int i = tid; i < CH_T * (CH_P / 8); i += CH_THREADS) {
                const int t = i / (CH_P / 8), k = (i % (CH_P / 8)) * 8;
                const bool ok = t0 + t < n && p0 + k < P;
                cp_async16_zfill(smem_u32(dx + t * CH_LP + k), xbc + (size_t)(ok ? t0 + t : 0) * p.ld_xbc + (ok ? cx + k : 0), ok);
            }
        } else {
            for (int i = tid; i < CH_T * CH_N; i += CH_THREADS) {
                const int t = i / CH_N, k = i % CH_N;
                const bool ok = t0 + t < n && k < N;
                dC[t * CH_LN + k] = ok ? xbc[(size_t)(t0 + t) * p.ld_xbc + cC + k] : 0;
                dB[t * CH_LN + k] = ok ? xbc[(size_t)(t0 + t) * p.ld_xbc + cB + k] : 0;
            }
            for (int i = tid; i < CH_T * CH_P; i += CH_THREADS) {
                const int t = i / CH_P, k = i % CH_P;
                dx[t * CH_LP + k] = t0 + t < n && p0 + k < P ? xbc[(size_t)(t0 + t) * p.ld_xbc + cx + k] : 0;
            }
        }
    };
    // state of this warp: rows sr + g4 (+ 8), value rows sp + 8 j + 2 t4 (+ 1)
    const int sr = (warp >> 1) * 16, sp = (warp & 1) * 32;
    float S[4][4];
    float* slot = p.state + (size_t)p.seq_slot[b] * p.slot_stride;
    float* Sg = slot + ((size_t)h * P + p0) * N;
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = sr + g4 + (e >> 1) * 8, q = sp + j * 8 + 2 * t4 + (e & 1);
            S[j][e] = before > 0 && r < N && p0 + q < P ? Sg[(size_t)q * N + r] : 0.f;
        }
    const int mt = warp >> 2, jt = warp & 3;  // tokens mt * 16..; earlier tokens jt * 16.. (weights), value rows jt * 16.. (y)
    const int ta = mt * 16 + g4, tb = ta + 8;
    const int chunks = (n + CH_T - 1) / CH_T;
    // Step sizes and decays of a chunk, two tokens per lane of warp 3 (whose tile of the weights is above the diagonal): the raw
    // values are fetched when the chunk before it begins and turned into factors when that warp is done with its part.
    float raw[2] = {0.f, 0.f};
    auto fetch_steps = [&](int c) {
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int t = c * CH_T + 2 * lane + i;
            raw[i] = t < n ? bf2f(zx[(size_t)(start + t) * p.ld + 2 * inner + 2 * s.groups * N + h]) : 0.f;
        }
    };
    auto make_steps = [&](int c) {
        float* dts = steps + (c & 1) * 4 * CH_T;
        float d[2], run = 0.f;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            d[i] = c * CH_T + 2 * lane + i < n ? softplus_f32(raw[i] + bias) : 0.f;
            run += -A * d[i];
        }
        float incl = run;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += u;
        }
        const float end = __shfl_sync(0xffffffffu, incl, 31);
        float at = incl - run;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int t = 2 * lane + i;
            at += -A * d[i];
            dts[t] = d[i];
            dts[CH_T + t] = at;
            dts[2 * CH_T + t] = expf(at);
            dts[3 * CH_T + t] = expf(end - at) * d[i];
        }
    };
    load(0);
    cp_async_commit();
    if (warp == 3) {
        fetch_steps(0);
        make_steps(0);
    }
    for (int c = 0; c < chunks; c++) {
        if (warp == 3 && c + 1 < chunks) fetch_steps(c + 1);
        const int t0 = c * CH_T, cnt = min(CH_T, n - t0);
        const float *dts = steps + (c & 1) * 4 * CH_T, *cum = dts + CH_T, *ecum = cum + CH_T, *wend = ecum + CH_T;
        // the state before this chunk, as operand of C S0
#pragma unroll
        for (int j = 0; j < 4; j++)
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int at = (sr + g4 + half * 8) * CH_LP + sp + j * 8 + 2 * t4;
                const uint32_t hi = pack_bf2(S[j][2 * half], S[j][2 * half + 1]);
                *reinterpret_cast<uint32_t*>(sh + at) = hi;
                *reinterpret_cast<uint32_t*>(sh + CH_N * CH_LP + at) = pack_bf2(S[j][2 * half] - bflo(hi), S[j][2 * half + 1] - bfhi(hi));
            }
        if (c + 1 < chunks) load(c + 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const uint16_t* sC = reinterpret_cast<const uint16_t*>(in0 + (c & 1) * ChunkSmem::kIn);
        const uint16_t *sB = sC + CH_T * CH_LN, *sx = sB + CH_T * CH_LN;
        for (int i = tid; i < CH_T * CH_P / 2; i += CH_THREADS) {  // what the tokens add to the state: exp(c_end - c_s) d_s x_s
            const int t = i / (CH_P / 2), at = t * CH_LP + (i % (CH_P / 2)) * 2;
            const uint32_t x2 = *reinterpret_cast<const uint32_t*>(sx + at);
            const float a0 = bflo(x2) * wend[t], a1 = bfhi(x2) * wend[t];
            const uint32_t hi = pack_bf2(a0, a1);
            *reinterpret_cast<uint32_t*>(xw + at) = hi;
            *reinterpret_cast<uint32_t*>(xw + CH_T * CH_LP + at) = pack_bf2(a0 - bflo(hi), a1 - bfhi(hi));
        }
        const uint32_t aC = smem_u32(sC + (mt * 16 + lr + (mi & 1) * 8) * CH_LN + (mi >> 1) * 8);
        if (jt <= mt) {  // weights of 16 tokens on 16 earlier ones
            float m[2][4];
#pragma unroll
            for (int half = 0; half < 2; half++) m[half][0] = m[half][1] = m[half][2] = m[half][3] = 0.f;
            const uint32_t bB = smem_u32(sB + (jt * 16 + lr + (mi >> 1) * 8) * CH_LN + (mi & 1) * 8);
            for (int k = 0; k < KN; k++) {
                uint32_t af[4], v0[2], v1[2];
                ldmatrix_x4(af[0], af[1], af[2], af[3], aC + k * 32);
                ldmatrix_x4(v0[0], v0[1], v1[0], v1[1], bB + k * 32);
                mma_bf16_16816(m[0], af, v0);
                mma_bf16_16816(m[1], af, v1);
            }
            const float ca = cum[ta], cb = cum[tb];
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int s0 = jt * 16 + half * 8 + 2 * t4;
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int si = s0 + (e & 1);
                    m[half][e] = si <= (e < 2 ? ta : tb) ? m[half][e] * __expf((e < 2 ? ca : cb) - cum[si]) * dts[si] : 0.f;
                }
#pragma unroll
                for (int row = 0; row < 2; row++) {
                    const int at = (row ? tb : ta) * CH_LM + s0;
                    const uint32_t hi = pack_bf2(m[half][2 * row], m[half][2 * row + 1]);
                    *reinterpret_cast<uint32_t*>(sm + at) = hi;
                    *reinterpret_cast<uint32_t*>(sm + CH_T * CH_LM + at) = pack_bf2(m[half][2 * row] - bflo(hi), m[half][2 * row + 1] - bfhi(hi));
                }
            }
        }
        // ---- y of this warp: first C S0 (needs nothing of the other warps' weights)
        float y[2][4];
        y[0][0] = y[0][1] = y[0][2] = y[0][3] = y[1][0] = y[1][1] = y[1][2] = y[1][3] = 0.f;
        const uint32_t bS = smem_u32(sh + (lr + (mi & 1) * 8) * CH_LP + jt * 16 + (mi >> 1) * 8);
        for (int k = 0; k < KN; k++) {
            uint32_t af[4];
            ldmatrix_x4(af[0], af[1], af[2], af[3], aC + k * 32);
#pragma unroll
            for (int part = 0; part < 2; part++) {
                uint32_t v0[2], v1[2];
                ldmatrix_x4_trans(v0[0], v0[1], v1[0], v1[1], bS + (part * CH_N * CH_LP + k * 16 * CH_LP) * 2);
                mma_bf16_16816(y[0], af, v0);
                mma_bf16_16816(y[1], af, v1);
            }
        }
        const float ea = ecum[ta], eb = ecum[tb];
#pragma unroll
        for (int q = 0; q < 2; q++) y[q][0] *= ea, y[q][1] *= ea, y[q][2] *= eb, y[q][3] *= eb;
        if (warp == 3 && c + 1 < chunks) make_steps(c + 1);
        __syncthreads();  // the weights and the state's increments are complete
        const uint32_t aM = smem_u32(sm + (mt * 16 + lr + (mi & 1) * 8) * CH_LM + (mi >> 1) * 8);
        const uint32_t bX = smem_u32(sx + (lr + (mi & 1) * 8) * CH_LP + jt * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int k = 0; k < CH_T / 16; k++)
            if (k <= mt) {
                uint32_t hi[4], lo[4], v0[2], v1[2];
                ldmatrix_x4(hi[0], hi[1], hi[2], hi[3], aM + k * 32);
                ldmatrix_x4(lo[0], lo[1], lo[2], lo[3], aM + CH_T * CH_LM * 2 + k * 32);
                ldmatrix_x4_trans(v0[0], v0[1], v1[0], v1[1], bX + k * 16 * CH_LP * 2);
                mma_bf16_16816(y[0], hi, v0);
                mma_bf16_16816(y[1], hi, v1);
                mma_bf16_16816(y[0], lo, v0);
                mma_bf16_16816(y[1], lo, v1);
            }
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int t = half ? tb : ta, q = jt * 16 + j * 8 + 2 * t4;
                if (t >= cnt) continue;
                const uint32_t x2 = *reinterpret_cast<const uint32_t*>(sx + t * CH_LP + q);
                const float y0 = fmaf(D, bflo(x2), y[j][2 * half]), y1 = fmaf(D, bfhi(x2), y[j][2 * half + 1]);
                float* o = p.y + (size_t)(start + t0 + t) * inner + h * P + p0 + q;
                if (vec && p0 + q < P) {
                    *reinterpret_cast<float2*>(o) = make_float2(y0, y1);
                } else {
                    if (p0 + q < P) o[0] = y0;
                    if (p0 + q + 1 < P) o[1] = y1;
                }
            }
        // ---- state of this warp
        if (sr < N) {
            const float dec = ecum[CH_T - 1];
#pragma unroll
            for (int j = 0; j < 4; j++) S[j][0] *= dec, S[j][1] *= dec, S[j][2] *= dec, S[j][3] *= dec;
            const uint32_t aB = smem_u32(sB + (lr + (mi >> 1) * 8) * CH_LN + sr + (mi & 1) * 8);
            const uint32_t bW = smem_u32(xw + (lr + (mi & 1) * 8) * CH_LP + sp + (mi >> 1) * 8);
#pragma unroll
            for (int k = 0; k < CH_T / 16; k++) {
                uint32_t af[4];
                ldmatrix_x4_trans(af[0], af[1], af[2], af[3], aB + k * 16 * CH_LN * 2);
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int part = 0; part < 2; part++) {
                        uint32_t v0[2], v1[2];
                        ldmatrix_x4_trans(v0[0], v0[1], v1[0], v1[1], bW + (part * CH_T * CH_LP + k * 16 * CH_LP + j * 16) * 2);
                        mma_bf16_16816(S[2 * j], af, v0);
                        mma_bf16_16816(S[2 * j + 1], af, v1);
                    }
            }
        }
        __syncthreads();  // this chunk's buffers may be written again
    }
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = sr + g4 + (e >> 1) * 8, q = sp + j * 8 + 2 * t4 + (e & 1);
            if (r < N && p0 + q < P) Sg[(size_t)q * N + r] = S[j][e];
        }
    keep_conv_inputs<uint16_t>(s, p, slot, start, n, before, h, p0, CH_P, blockIdx.x == 0);
}

// out = norm over equal parts of (y * silu(z)), times w; zero up to the padded width
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const Mamba2Spec s, const SsmParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    __shared__ float red[33];
    const int t = blockIdx.x, g = blockIdx.y, inner = s.inner(), part = inner / s.norm_groups, c0 = g * part;
    const T* z = reinterpret_cast<const T*>(p.zx) + (size_t)t * p.ld;
    const float* y = p.y + (size_t)t * inner;
    float ss = 0.f;
    constexpr int KEEP = 4;  // chunks of four values a thread keeps between the passes (parts up to 4096 wide)
    const bool vec = part % 4 == 0 && inner % 4 == 0 && part <= KEEP * 4 * 256;
    float4 kept[KEEP];
    if (vec) {
#pragma unroll
        for (int k = 0; k < KEEP; k++) {
            const int i = c0 + (k * 256 + threadIdx.x) * 4;
            if (i >= c0 + part) break;
            float4 v = *reinterpret_cast<const float4*>(y + i);
            float zz[4];
            Elt<T>::ld4(z + i, zz);
            v.x *= silu_f32(zz[0]), v.y *= silu_f32(zz[1]), v.z *= silu_f32(zz[2]), v.w *= silu_f32(zz[3]);
            kept[k] = v;
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int i = c0 + threadIdx.x; i < c0 + part; i += blockDim.x) {
            const float v = y[i] * silu_f32(Elt<T>::ld(z + i));
            ss += v * v;
        }
    }
    ss = elt_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)part + p.eps);
    T* o = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo;
    if (vec) {
#pragma unroll
        for (int k = 0; k < KEEP; k++) {
            const int i = c0 + (k * 256 + threadIdx.x) * 4;
            if (i >= c0 + part) break;
            const float4 w = *reinterpret_cast<const float4*>(p.norm + i), v = kept[k];
            const float r[4] = {v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w};
            Elt<T>::st4(o + i, r);
        }
    } else {
        for (int i = c0 + threadIdx.x; i < c0 + part; i += blockDim.x) Elt<T>::st(o + i, y[i] * silu_f32(Elt<T>::ld(z + i)) * inv * p.norm[i]);
    }
    if (g == s.norm_groups - 1)
        for (int i = inner + threadIdx.x; i < p.ldo; i += blockDim.x) Elt<T>::st(o + i, 0.f);
}

template <typename T>
int32_t launch_ssm(b2_ctx* ctx, const Mamba2Spec& s, const SsmParams& p) {
    B2_REQUIRE(p.T <= 65535, B2_ERR_UNSUPPORTED, "mamba2: too many tokens in one step");
    if (s.channels() % 8 == 0 && s.inner() % 8 == 0 && s.conv >= 2 && s.conv <= 4) {
        const int bx = (s.channels() / 8 + 127) / 128, want = 12 * ctx->sm_count / bx + 1;  // blocks along the tokens
        const int run = p.T > want ? (p.T + want - 1) / want : 1;
        const dim3 cgrid(bx, (p.T + run - 1) / run);
        auto ck = s.conv == 2 ? conv_silu8_kernel<T, 2> : s.conv == 3 ? conv_silu8_kernel<T, 3> : conv_silu8_kernel<T, 4>;
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, ck, cgrid, dim3(128), 0, ctx->stream, s, p, run));
    } else {
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, conv_silu_kernel<T>, dim3((s.channels() + 255) / 256, p.T), dim3(256), 0, ctx->stream, s, p));
    }
    B2_LAUNCHED(ctx);
    const dim3 grid((s.vdim + SC_P - 1) / SC_P, s.heads, p.B);
    const int k4 = (s.state + 31) / 32;
    SsmParams q = p;
    q.chunked = sizeof(T) == 2 && s.state <= CH_N && p.T >= p.B - 1 + kChunkMin;  // some sequence may bring enough tokens
    if (q.chunked) {
        B2_SMEM_ONCE(ctx, chunk_scan_kernel, ChunkSmem::kBytes);
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, chunk_scan_kernel, dim3((s.vdim + CH_P - 1) / CH_P, s.heads, p.B), dim3(CH_THREADS), (size_t)ChunkSmem::kBytes,
                              ctx->stream, s, q));
        B2_LAUNCHED(ctx);
    }
    auto k = k4 <= 1 ? scan_kernel<T, 1> : k4 <= 2 ? scan_kernel<T, 2> : k4 <= 4 ? scan_kernel<T, 4> : scan_kernel<T, 8>;
    if (!q.chunked || p.B > 1) {
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, grid, dim3(128), 0, ctx->stream, s, q));
        B2_LAUNCHED(ctx);
    }
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
