// Linear memories over a prompt, 64 tokens at a time on tensor cores (serving format).
//
// With G_t the running sum of the decays' logarithms over a chunk (per key channel, or one number per head) and S0 the state
// before it,
//     (I + A) U = beta (V - Kf S0)      A_ts = beta_t k_t . (e^(G_t - G_s) k_s), s < t        Kf_t = e^(G_t) k_t
//     O = Qf S0 + P U                   P_ts = q_t . (e^(G_t - G_s) k_s), s <= t              Qf_t = e^(G_t) q_t
//     S = e^(G_end) S0 + Kb^T U         Kb_s = e^(G_end - G_s) k_s
// (a memory without the delta rule has U = V).  What does not depend on the state -- P, the inverse of I + A times beta, and
// the three scaled operands -- is made for all chunks of all heads at once by memory_factor_kernel; memory_chunk_kernel then
// walks the chunks of a head in order.
//
// Every operand that is f32 by nature enters the products as a bf16 head plus a bf16 remainder (the product of the two
// remainders is dropped), all sums are f32, and the state stays in f32 registers from chunk to chunk.
#include "memory.cuh"
#include "tc5.cuh"

namespace {

constexpr int C = kMemoryChunk, VB = 32;  // tokens per chunk; value columns per block of the walk
constexpr float kLog2e = 1.4426950408889634f;

// A chunk of one head in memory: tiles of bf16, rows of tokens, in the order and swizzle of the walk's shared memory.
template <int DK>
struct Record {
    static constexpr int kOp = C * DK * 2, kMat = C * C * 2;  // an operand tile, a weight tile
    static constexpr int Kf = 0, Qf = 2 * kOp, T = 4 * kOp, P = T + 2 * kMat, Kb = P + 2 * kMat, kBytes = Kb + 2 * kOp;  // head, then remainder
};
// byte of the 16-byte piece that holds column `col` of row `row`; rows of 128 bytes or a multiple
__device__ __forceinline__ uint32_t at_wide(int row, int piece, int row_bytes) { return (uint32_t)(row * row_bytes + ((piece ^ (row & 7)) << 4)); }
// ... rows of 64 bytes
__device__ __forceinline__ uint32_t at_narrow(int row, int piece) { return (uint32_t)(row * 64 + ((piece ^ ((row >> 1) & 3)) << 4)); }

struct Split {  // two f32 as bf16 pairs: head and remainder
    uint32_t hi, lo;
};
__device__ __forceinline__ Split split2(float a, float b) {
    Split s;
    s.hi = pack_bf2(a, b);
    s.lo = pack_bf2(a - bflo(s.hi), b - bfhi(s.hi));
    return s;
}
// d += (ah + al) (bh + bl) without al bl
__device__ __forceinline__ void mma3(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[2], const uint32_t (&bl)[2]) {
    mma_bf16_16816(d, ah, bh);
    mma_bf16_16816(d, ah, bl);
    mma_bf16_16816(d, al, bh);
}

// ---- factors ---------------------------------------------------------------------------------------------------------
constexpr int F_WARPS = 10, F_THREADS = F_WARPS * 32;  // a warp per 16 x 16 tile of P and A up to the diagonal
constexpr float kMaxSpread = 80.f;  // log2 units: largest decay inside 16 tokens whose inverse is used as a factor
template <int DK, bool CHANNEL>
struct FactorSmem {
    static constexpr int LD = DK + 4, LM = C + 4;
    static constexpr int K = 0, G = K + C * LD * 4, M = G + (CHANNEL ? C * LD * 4 : C * 4), Y = M + C * LM * 4, BETA = Y + 3 * 16 * 17 * 4, kBytes = BETA + C * 4;
};

template <int DK, bool CHANNEL>
__global__ void __launch_bounds__(F_THREADS) memory_factor_kernel(const MemorySpec s, const MemoryParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    using L = FactorSmem<DK, CHANNEL>;
    using R = Record<DK>;
    constexpr int LD = L::LD, LM = L::LM;
    extern __shared__ __align__(16) uint8_t smem[];
    float* ks = reinterpret_cast<float*>(smem + L::K);    // [C][LD] keys
    float* gs = reinterpret_cast<float*>(smem + L::G);    // [C][LD] or [C]: running sums of the decays' logarithms (base 2)
    float* M = reinterpret_cast<float*>(smem + L::M);     // [C][LM]: A below the diagonal, the transposed inverse above it
    float* Y = reinterpret_cast<float*>(smem + L::Y);     // [3][16][17]
    float* betas = reinterpret_cast<float*>(smem + L::BETA);
    __shared__ int wide[4];                               // 16-token blocks whose decays do not allow inverse factors
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
    const int chunk = blockIdx.x, h = blockIdx.y, D = s.dim, Q = s.q_cols(), kh = h / (s.heads / s.kv_heads);
    int b = -1;  // the last chunked portion that starts at or before this chunk (starts rise with the index)
    for (int i = lane; i < p.B; i += 32)
        if (p.chunk_off[i] >= 0 && p.chunk_off[i] <= chunk) b = i;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) b = max(b, __shfl_xor_sync(0xffffffffu, b, o));
    if (b < 0) return;
    const int n = p.cu_seqlens[b + 1] - p.cu_seqlens[b], t0 = (chunk - p.chunk_off[b]) * C, cnt = min(C, n - t0);
    if (cnt <= 0) return;
    const size_t tok0 = (size_t)p.cu_seqlens[b] + t0;
    uint8_t* rec = reinterpret_cast<uint8_t*>(p.chunk) + ((size_t)chunk * s.heads + h) * R::kBytes;
    const float* q = p.q + tok0 * Q + kh * D;

    if (tid < 4) wide[tid] = 0;
    for (int i = tid; i < C * DK; i += F_THREADS) {
        const int t = i / DK, d = i % DK;
        const bool ok = t < cnt && d < D;
        ks[t * LD + d] = ok ? p.k[(tok0 + t) * Q + kh * D + d] : 0.f;
        if constexpr (CHANNEL) gs[t * LD + d] = ok ? p.lg[(tok0 + t) * s.decays() + h * D + d] * kLog2e : 0.f;
    }
    if (!CHANNEL && tid < C) gs[tid] = tid < cnt ? (s.decay == MemDecay::Fixed ? p.log_decay[h] : p.lg[(tok0 + tid) * s.heads + h]) * kLog2e : 0.f;
    if (tid < C) betas[tid] = s.delta && tid < cnt ? p.beta[(tok0 + tid) * s.heads + h] : 0.f;
    __syncthreads();
    if constexpr (CHANNEL) {
        if (tid < DK) {
            float run = 0.f;
            for (int i = 0; i < 4; i++) {
                const float ref = run;
#pragma unroll
                for (int t = 0; t < 16; t++) {
                    run += gs[(16 * i + t) * LD + tid];
                    gs[(16 * i + t) * LD + tid] = run;
                }
                if (ref - run > kMaxSpread) atomicOr(&wide[i], 1);
            }
        }
    } else if (tid < 32) {
        float a = gs[2 * tid], c = gs[2 * tid + 1], sum = a + c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, sum, o);
            if (tid >= o) sum += u;
        }
        gs[2 * tid] = sum - c;
        gs[2 * tid + 1] = sum;
    }
    __syncthreads();

    // ---- P and A, a 16 x 16 tile (tokens 16 i .., earlier tokens 16 j ..) per warp
    {
        int i = 0, j = warp;
        while (j > i) j -= ++i;
        float a[2][4], pr[2][4];
#pragma unroll
        for (int half = 0; half < 2; half++)
#pragma unroll
            for (int e = 0; e < 4; e++) a[half][e] = pr[half][e] = 0.f;
        const int ta = 16 * i + g4, tb = ta + 8;
        if (CHANNEL && i == j && wide[i]) {
            // strong decays inside the block: every exponent from its difference, lanes over the channels
#pragma unroll 1
            for (int t = 16 * i; t < min(16 * i + 16, cnt); t++)
#pragma unroll 1
                for (int u = 16 * i; u <= t; u++) {
                    float sa = 0.f, sp = 0.f;
                    for (int d = lane; d < DK; d += 32) {
                        const float w = fast_exp2(gs[t * LD + d] - gs[u * LD + d]) * ks[u * LD + d];
                        sa = fmaf(w, ks[t * LD + d], sa);
                        sp = fmaf(w, d < D ? q[(size_t)t * Q + d] : 0.f, sp);
                    }
                    sa = elt_warp_sum(sa);
                    sp = elt_warp_sum(sp);
#pragma unroll
                    for (int half = 0; half < 2; half++)
#pragma unroll
                        for (int e = 0; e < 4; e++)
                            if (t == (e < 2 ? ta : tb) && u == 16 * i + half * 8 + 2 * t4 + (e & 1)) a[half][e] = sa, pr[half][e] = sp;
                }
        } else {
            const float* ref = gs + (16 * i - 1) * LD;  // the sums before the block's first token
#pragma unroll 2
            for (int k = 0; k < DK / 16; k++) {
                uint32_t kh_[4], kl_[4], qh_[4], ql_[4];
                float r[4];  // reference at columns d0, d0 + 1, d0 + 8, d0 + 9
                const int d0 = k * 16 + 2 * t4;
                if constexpr (CHANNEL) {
#pragma unroll
                    for (int e = 0; e < 4; e++) r[e] = i > 0 ? ref[d0 + (e >> 1) * 8 + (e & 1)] : 0.f;
                }
#pragma unroll
                for (int e = 0; e < 4; e++) {  // fragment e: row (e & 1), columns (e >> 1)
                    const int t = (e & 1) ? tb : ta, d = d0 + (e >> 1) * 8;
                    const float2 kv = *reinterpret_cast<const float2*>(ks + t * LD + d);
                    const float q0 = t < cnt && d < D ? q[(size_t)t * Q + d] : 0.f, q1 = t < cnt && d + 1 < D ? q[(size_t)t * Q + d + 1] : 0.f;
                    float w0 = 1.f, w1 = 1.f;
                    if constexpr (CHANNEL) {
                        const float2 gv = *reinterpret_cast<const float2*>(gs + t * LD + d);
                        w0 = fast_exp2(gv.x - r[(e >> 1) * 2]), w1 = fast_exp2(gv.y - r[(e >> 1) * 2 + 1]);
                    }
                    const Split sk = split2(kv.x * w0, kv.y * w1), sq = split2(q0 * w0, q1 * w1);
                    kh_[e] = sk.hi, kl_[e] = sk.lo, qh_[e] = sq.hi, ql_[e] = sq.lo;
                }
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    const int u = 16 * j + half * 8 + g4;
                    uint32_t bh[2], bl[2];
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const int d = d0 + e * 8;
                        const float2 kv = *reinterpret_cast<const float2*>(ks + u * LD + d);
                        float w0 = 1.f, w1 = 1.f;
                        if constexpr (CHANNEL) {
                            const float2 gv = *reinterpret_cast<const float2*>(gs + u * LD + d);
                            w0 = fast_exp2(r[e * 2] - gv.x), w1 = fast_exp2(r[e * 2 + 1] - gv.y);
                        }
                        const Split sk = split2(kv.x * w0, kv.y * w1);
                        bh[e] = sk.hi, bl[e] = sk.lo;
                    }
                    if (s.delta) mma3(a[half], kh_, kl_, bh, bl);
                    mma3(pr[half], qh_, ql_, bh, bl);
                }
            }
        }
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int u0 = 16 * j + half * 8 + 2 * t4;
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int t = e < 2 ? ta : tb, u = u0 + (e & 1);
                if constexpr (!CHANNEL) {
                    const float w = u <= t ? fast_exp2(gs[t] - gs[u]) : 0.f;
                    a[half][e] *= w;
                    pr[half][e] *= w;
                }
                if (u > t) pr[half][e] = 0.f;
                if (s.delta && u < t) M[t * LM + u] = a[half][e] * betas[t];
            }
#pragma unroll
            for (int row = 0; row < 2; row++) {
                const Split sp = split2(pr[half][2 * row], pr[half][2 * row + 1]);
                const uint32_t o = at_wide(row ? tb : ta, u0 >> 3, 128) + (u0 & 7) * 2;
                *reinterpret_cast<uint32_t*>(rec + R::P + o) = sp.hi;
                *reinterpret_cast<uint32_t*>(rec + R::P + R::kMat + o) = sp.lo;
            }
        }
    }
    // ---- the scaled operands, eight columns at a time
    const int last = cnt - 1;
    for (int i = tid; i < C * (DK / 8); i += F_THREADS) {
        const int t = i / (DK / 8), x = i % (DK / 8);
        float kf[8], qf[8], kb[8];
#pragma unroll
        for (int e = 0; e < 8; e++) {
            const int d = x * 8 + e;
            const float g = CHANNEL ? gs[t * LD + d] : gs[t], ge = CHANNEL ? gs[last * LD + d] : gs[last], k = ks[t * LD + d];
            const float f = fast_exp2(g);
            kf[e] = k * f;
            kb[e] = t < cnt ? k * fast_exp2(ge - g) : 0.f;
            qf[e] = t < cnt && d < D ? q[(size_t)t * Q + d] * f : 0.f;
        }
        const uint32_t o = at_wide(t, x, DK * 2);
        auto store = [&](int tile, const float (&v)[8]) {
            Split w[4];
#pragma unroll
            for (int e = 0; e < 4; e++) w[e] = split2(v[2 * e], v[2 * e + 1]);
            *reinterpret_cast<uint4*>(rec + tile + o) = make_uint4(w[0].hi, w[1].hi, w[2].hi, w[3].hi);
            *reinterpret_cast<uint4*>(rec + tile + R::kOp + o) = make_uint4(w[0].lo, w[1].lo, w[2].lo, w[3].lo);
        };
        if (s.delta) store(R::Kf, kf);
        store(R::Qf, qf);
        store(R::Kb, kb);
    }
    // the chunk's whole decay, over the first token's entry (which only this block reads)
    if constexpr (CHANNEL) {
        if (tid < D) p.lg[tok0 * s.decays() + h * D + tid] = fast_exp2(gs[last * LD + tid]);
    } else if (s.decay == MemDecay::PerHead && tid == 0) {
        p.lg[tok0 * s.heads + h] = fast_exp2(gs[last]);
    }
    if (!s.delta) return;
    // ---- inverse of the unit lower triangular I + A: diagonal blocks, then block diagonals outwards
    //      T_ij = -T_ii sum_{j <= k < i} A_ik T_kj.  T_ts is kept at M[s][t], its unit diagonal implied.
    __syncthreads();
    if (tid < C) {
        const int base = tid & ~15, c = tid & 15;
        float x[16];
#pragma unroll
        for (int t = 0; t < 16; t++) {
            float acc = 0.f;
#pragma unroll
            for (int u = 0; u < t; u++) acc = fmaf(M[(base + t) * LM + base + u], x[u], acc);
            x[t] = t == c ? 1.f : (t > c ? -acc : 0.f);
        }
        __syncwarp();
#pragma unroll
        for (int t = 0; t < 16; t++)
            if (t > c) M[(base + c) * LM + base + t] = x[t];
    }
    __syncthreads();
    auto inv = [&](int bi, int bj, int t, int u) {  // T of block (bi, bj) at (t, u)
        if (bi == bj && t <= u) return t == u ? 1.f : 0.f;
        return M[(16 * bj + u) * LM + 16 * bi + t];
    };
#pragma unroll 1
    for (int dist = 1; dist < 4; dist++) {
        const int pairs = 4 - dist;
        for (int e = tid; e < pairs * 256; e += F_THREADS) {
            const int j = e >> 8, i = j + dist, t = (e >> 4) & 15, u = e & 15;
            float acc = 0.f;
            for (int k = j; k < i; k++)
#pragma unroll
                for (int x = 0; x < 16; x++) acc = fmaf(M[(16 * i + t) * LM + 16 * k + x], inv(k, j, x, u), acc);
            Y[(j * 16 + t) * 17 + u] = acc;
        }
        __syncthreads();
        for (int e = tid; e < pairs * 256; e += F_THREADS) {
            const int j = e >> 8, i = j + dist, t = e & 15, u = (e >> 4) & 15;
            float acc = 0.f;
#pragma unroll
            for (int x = 0; x < 16; x++) acc = fmaf(inv(i, i, t, x), Y[(j * 16 + x) * 17 + u], acc);
            M[(16 * j + u) * LM + 16 * i + t] = -acc;
        }
        __syncthreads();
    }
    for (int e = tid; e < C * C / 2; e += F_THREADS) {  // times beta, pairs of columns up to the diagonal blocks
        const int t = e / (C / 2), u = (e % (C / 2)) * 2;
        if ((u >> 4) > (t >> 4)) continue;
        auto val = [&](int c) { return t < cnt && c <= t ? (c == t ? 1.f : M[c * LM + t]) * betas[c] : 0.f; };
        const Split sp = split2(val(u), val(u + 1));
        const uint32_t o = at_wide(t, u >> 3, 128) + (u & 7) * 2;
        *reinterpret_cast<uint32_t*>(rec + R::T + o) = sp.hi;
        *reinterpret_cast<uint32_t*>(rec + R::T + R::kMat + o) = sp.lo;
    }
}

// ---- the walk --------------------------------------------------------------------------------------------------------
// Block = (32 value columns of one head, sequence), eight warps.  Per chunk: Kf S0 and Qf S0 (a warp per 16 tokens x 16
// columns), U from them, then O and the state (a warp per 16 state rows x 32 columns, or x 16 for keys up to 64).  The next
// chunk's tiles arrive by bulk copies: Kf and Qf into the other of two buffers, the rest as soon as its place is free.
constexpr int W_THREADS = 256;
template <int DK>
struct WalkSmem {
    using R = Record<DK>;
    static constexpr int kKQ = 4 * R::kOp, kS = DK * VB * 2, kU = C * VB * 2;
    static constexpr int KQ = 0, T = 2 * kKQ, P = T + 2 * R::kMat, Kb = P + 2 * R::kMat, S = Kb + 2 * R::kOp, RU = S + 2 * kS, U = RU + 2 * kU, BAR = U + 2 * kU, kBytes = BAR + 64;
};

template <int DK, bool DELTA>
__global__ void __launch_bounds__(W_THREADS, 1) memory_chunk_kernel(const MemorySpec s, const MemoryParams p, int* err) {
    using namespace tc5;
    using L = WalkSmem<DK>;
    using R = Record<DK>;
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    extern __shared__ __align__(128) uint8_t smem[];
    const int h = blockIdx.y, b = blockIdx.z, p0 = blockIdx.x * VB;
    const int start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start, before = p.context_lens[b] - n;
    if (n < kMemoryChunkMin) return;  // the token-by-token kernel's
    const int D = s.dim, P = s.vdim, V = s.heads * P, chunks = (n + C - 1) / C;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
    const uint32_t base = smem_u32(smem), bar = base + L::BAR;
    // barriers: Kf | Qf of either buffer, T, P | Kb
    const uint32_t f_kq[2] = {bar, bar + 8}, f_t = bar + 16, f_pk = bar + 24;
    const uint8_t* rec0 = reinterpret_cast<const uint8_t*>(p.chunk) + ((size_t)p.chunk_off[b] * s.heads + h) * R::kBytes;
    const size_t rec_step = (size_t)s.heads * R::kBytes;
    if (tid == 0) {
        for (int i = 0; i < 4; i++) mbar_init(bar + 8 * i, 1);
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    auto load_kq = [&](int c) {
        const uint32_t dst = base + L::KQ + (c & 1) * L::kKQ;
        const uint8_t* src = rec0 + c * rec_step;
        mbar_expect_tx(f_kq[c & 1], DELTA ? 4 * R::kOp : 2 * R::kOp);
        if (DELTA) bulk_load(dst, src + R::Kf, 2 * R::kOp, f_kq[c & 1]);
        bulk_load(dst + 2 * R::kOp, src + R::Qf, 2 * R::kOp, f_kq[c & 1]);
    };
    auto load_t = [&](int c) {
        mbar_expect_tx(f_t, 2 * R::kMat);
        bulk_load(base + L::T, rec0 + c * rec_step + R::T, 2 * R::kMat, f_t);
    };
    auto load_pk = [&](int c) {
        mbar_expect_tx(f_pk, 2 * R::kMat + 2 * R::kOp);
        bulk_load(base + L::P, rec0 + c * rec_step + R::P, 2 * R::kMat + 2 * R::kOp, f_pk);  // P and Kb lie side by side in both places
    };
    static_assert(L::Kb == L::P + 2 * R::kMat && R::Kb == R::P + 2 * R::kMat, "one copy for P and Kb");
    // state of this warp: rows sr + g4 (+ 8), columns sc + 8 j + 2 t4 (+ 1)
    constexpr int NT = DK == 128 ? 4 : 2;
    const int sr = (DK == 128 ? warp : warp >> 1) * 16, sc = DK == 128 ? 0 : (warp & 1) * 16;
    float* Sg = p.state + (size_t)p.seq_slot[b] * p.slot_stride + ((size_t)h * P + p0) * D;
    float S[NT][4];
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = sr + g4 + (e >> 1) * 8, q = sc + j * 8 + 2 * t4 + (e & 1);
            S[j][e] = before > 0 && r < D && p0 + q < P ? Sg[(size_t)q * D + r] : 0.f;
        }
    auto put = [&](int off, int lo_off, int row, int col, float a, float c) {  // two neighbours of a 32-column tile
        const Split sp = split2(a, c);
        const uint32_t o = at_narrow(row, col >> 3) + (col & 7) * 2;
        *reinterpret_cast<uint32_t*>(smem + off + o) = sp.hi;
        *reinterpret_cast<uint32_t*>(smem + off + lo_off + o) = sp.lo;
    };
    auto put_state = [&]() {
#pragma unroll
        for (int j = 0; j < NT; j++) {
            put(L::S, L::kS, sr + g4, sc + j * 8 + 2 * t4, S[j][0], S[j][1]);
            put(L::S, L::kS, sr + g4 + 8, sc + j * 8 + 2 * t4, S[j][2], S[j][3]);
        }
    };
    put_state();
    __syncthreads();
    if (tid == 0) {
        load_kq(0);
        if (DELTA) load_t(0);
        load_pk(0);
    }
    const int mt = warp >> 1, nc = (warp & 1) * 16;  // tokens mt * 16 .., columns nc ..
    const int ta = mt * 16 + g4, tb = ta + 8;
    // values at this thread's places of the token tiles: rows ta, tb, columns nc + 8 j + 2 t4 (+ 1)
    const uint16_t* vg = reinterpret_cast<const uint16_t*>(p.v) + (size_t)start * p.ld_v + h * P + p0;
    const bool pair = P % 2 == 0 && p.ld_v % 2 == 0 && ((uintptr_t)p.v & 3) == 0;
    uint32_t vv[2][2];
    auto fetch_v = [&](int c) {
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int row = 0; row < 2; row++) {
                const int t = c * C + (row ? tb : ta), q = nc + j * 8 + 2 * t4;
                const uint16_t* x = vg + (size_t)t * p.ld_v + q;
                uint32_t r = 0;
                if (t < n && p0 + q < P) r = pair ? *reinterpret_cast<const uint32_t*>(x) : (uint32_t)x[0] | (p0 + q + 1 < P ? (uint32_t)x[1] << 16 : 0u);
                vv[j][row] = r;
            }
    };
    // the chunk's decay at this thread's state rows
    float dec[2];
    auto fetch_decay = [&](int c) {
        const size_t tok = (size_t)start + c * C;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int r = sr + g4 + i * 8;
            dec[i] = s.decay == MemDecay::PerChannel ? (r < D ? p.lg[tok * s.decays() + h * D + r] : 0.f)
                     : s.decay == MemDecay::PerHead ? p.lg[tok * s.heads + h] : exp2f(p.log_decay[h] * kLog2e * (float)min(C, n - c * C));
        }
    };
    // fragments: A from tiles with rows of tokens, B (transposed) from 32-column tiles; `kt`: 16 tokens or keys of the sum
    auto frag_a = [&](uint32_t tile, int row_bytes, int row0, int piece0, uint32_t (&f)[4]) {
        ldmatrix_x4(f[0], f[1], f[2], f[3], base + tile + at_wide(row0 + lr + (mi & 1) * 8, piece0 + (mi >> 1), row_bytes));
    };
    auto frag_b = [&](uint32_t tile, int row0, int piece0, uint32_t (&f0)[2], uint32_t (&f1)[2]) {
        ldmatrix_x4_trans(f0[0], f0[1], f1[0], f1[1], base + tile + at_narrow(row0 + lr + (mi & 1) * 8, piece0 + (mi >> 1)));
    };
    fetch_v(0);
    bool alive = true;
    for (int c = 0; c < chunks; c++) {
        const uint32_t ph = (uint32_t)c & 1u, kq = L::KQ + ph * L::kKQ;
        if (tid == 0 && c + 1 < chunks) load_kq(c + 1);  // (its buffer was last read before the previous chunk's barriers)
        fetch_decay(c);
        alive = mbar_wait(f_kq[ph], (uint32_t)(c >> 1) & 1u) && alive;
        // ---- what the state before the chunk answers
        float ak[2][4], o[2][4];
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) ak[j][e] = o[j][e] = 0.f;
#pragma unroll
        for (int k = 0; k < DK / 16; k++) {
            uint32_t ah[4], al[4], bh0[2], bh1[2], bl0[2], bl1[2];
            frag_b(L::S, k * 16, nc >> 3, bh0, bh1);
            frag_b(L::S + L::kS, k * 16, nc >> 3, bl0, bl1);
            if constexpr (DELTA) {
                frag_a(kq, DK * 2, mt * 16, 2 * k, ah);
                frag_a(kq + R::kOp, DK * 2, mt * 16, 2 * k, al);
                mma3(ak[0], ah, al, bh0, bl0);
                mma3(ak[1], ah, al, bh1, bl1);
            }
            frag_a(kq + 2 * R::kOp, DK * 2, mt * 16, 2 * k, ah);
            frag_a(kq + 3 * R::kOp, DK * 2, mt * 16, 2 * k, al);
            mma3(o[0], ah, al, bh0, bl0);
            mma3(o[1], ah, al, bh1, bl1);
        }
        // ---- U
        if constexpr (DELTA) {
#pragma unroll
            for (int j = 0; j < 2; j++) {
                put(L::RU, L::kU, ta, nc + j * 8 + 2 * t4, bflo(vv[j][0]) - ak[j][0], bfhi(vv[j][0]) - ak[j][1]);
                put(L::RU, L::kU, tb, nc + j * 8 + 2 * t4, bflo(vv[j][1]) - ak[j][2], bfhi(vv[j][1]) - ak[j][3]);
            }
            if (c + 1 < chunks) fetch_v(c + 1);
            alive = mbar_wait(f_t, ph) && alive;
            __syncthreads();
            float u[2][4];
#pragma unroll
            for (int j = 0; j < 2; j++) u[j][0] = u[j][1] = u[j][2] = u[j][3] = 0.f;
#pragma unroll
            for (int k = 0; k < C / 16; k++)
                if (k <= mt) {
                    uint32_t ah[4], al[4], bh0[2], bh1[2], bl0[2], bl1[2];
                    frag_a(L::T, 128, mt * 16, 2 * k, ah);
                    frag_a(L::T + R::kMat, 128, mt * 16, 2 * k, al);
                    frag_b(L::RU, k * 16, nc >> 3, bh0, bh1);
                    frag_b(L::RU + L::kU, k * 16, nc >> 3, bl0, bl1);
                    mma3(u[0], ah, al, bh0, bl0);
                    mma3(u[1], ah, al, bh1, bl1);
                }
#pragma unroll
            for (int j = 0; j < 2; j++) {
                put(L::U, L::kU, ta, nc + j * 8 + 2 * t4, u[j][0], u[j][1]);
                put(L::U, L::kU, tb, nc + j * 8 + 2 * t4, u[j][2], u[j][3]);
            }
        } else {  // the values themselves, bf16
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int row = 0; row < 2; row++) {
                    const int q = nc + j * 8 + 2 * t4;
                    *reinterpret_cast<uint32_t*>(smem + L::U + at_narrow(row ? tb : ta, q >> 3) + (q & 7) * 2) = vv[j][row];
                }
            if (c + 1 < chunks) fetch_v(c + 1);
        }
        alive = mbar_wait(f_pk, ph) && alive;
        alive = __syncthreads_and(alive);
        if (!alive) break;
        if (DELTA && tid == 0 && c + 1 < chunks) load_t(c + 1);
        // ---- O
#pragma unroll
        for (int k = 0; k < C / 16; k++)
            if (k <= mt) {
                uint32_t ah[4], al[4], bh0[2], bh1[2], bl0[2], bl1[2];
                frag_a(L::P, 128, mt * 16, 2 * k, ah);
                frag_a(L::P + R::kMat, 128, mt * 16, 2 * k, al);
                frag_b(L::U, k * 16, nc >> 3, bh0, bh1);
                if constexpr (DELTA) {
                    frag_b(L::U + L::kU, k * 16, nc >> 3, bl0, bl1);
                    mma3(o[0], ah, al, bh0, bl0);
                    mma3(o[1], ah, al, bh1, bl1);
                } else {
                    mma_bf16_16816(o[0], ah, bh0);
                    mma_bf16_16816(o[0], al, bh0);
                    mma_bf16_16816(o[1], ah, bh1);
                    mma_bf16_16816(o[1], al, bh1);
                }
            }
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int row = 0; row < 2; row++) {
                const int t = c * C + (row ? tb : ta), q = nc + j * 8 + 2 * t4;
                if (t >= n) continue;
                float* x = p.o + (size_t)(start + t) * V + h * P + p0 + q;
                if (P % 2 == 0 && p0 + q < P) {
                    *reinterpret_cast<float2*>(x) = make_float2(o[j][2 * row], o[j][2 * row + 1]);
                } else {
                    if (p0 + q < P) x[0] = o[j][2 * row];
                    if (p0 + q + 1 < P) x[1] = o[j][2 * row + 1];
                }
            }
        // ---- the state
#pragma unroll
        for (int j = 0; j < NT; j++) S[j][0] *= dec[0], S[j][1] *= dec[0], S[j][2] *= dec[1], S[j][3] *= dec[1];
#pragma unroll
        for (int k = 0; k < C / 16; k++) {
            // Kb^T: rows of keys from rows of tokens
            uint32_t ah[4], al[4];
            const uint32_t x = at_wide(k * 16 + lr + (mi >> 1) * 8, (sr >> 3) + (mi & 1), DK * 2);
            ldmatrix_x4_trans(ah[0], ah[1], ah[2], ah[3], base + L::Kb + x);
            ldmatrix_x4_trans(al[0], al[1], al[2], al[3], base + L::Kb + R::kOp + x);
#pragma unroll
            for (int j = 0; j < NT / 2; j++) {
                uint32_t bh0[2], bh1[2], bl0[2], bl1[2];
                frag_b(L::U, k * 16, (sc >> 3) + 2 * j, bh0, bh1);
                if constexpr (DELTA) {
                    frag_b(L::U + L::kU, k * 16, (sc >> 3) + 2 * j, bl0, bl1);
                    mma3(S[2 * j], ah, al, bh0, bl0);
                    mma3(S[2 * j + 1], ah, al, bh1, bl1);
                } else {
                    mma_bf16_16816(S[2 * j], ah, bh0);
                    mma_bf16_16816(S[2 * j], al, bh0);
                    mma_bf16_16816(S[2 * j + 1], ah, bh1);
                    mma_bf16_16816(S[2 * j + 1], al, bh1);
                }
            }
        }
        put_state();
        __syncthreads();
        if (tid == 0 && c + 1 < chunks) load_pk(c + 1);
    }
    if (!alive) {  // a copy did not arrive in time: report, and give what is in flight another chance to land
        if (tid == 0) {
            atomicExch(err, 19);
            for (int i = 0; i < 4; i++) mbar_wait(bar + 8 * i, 0), mbar_wait(bar + 8 * i, 1);
        }
        return;
    }
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = sr + g4 + (e >> 1) * 8, q = sc + j * 8 + 2 * t4 + (e & 1);
            if (r < D && p0 + q < P) Sg[(size_t)q * D + r] = S[j][e];
        }
    memory_keep_inputs<uint16_t>(s, p, b, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
}

template <int DK, bool CHANNEL>
int32_t launch_factors(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p) {
    constexpr int kBytes = FactorSmem<DK, CHANNEL>::kBytes;
    B2_SMEM_ONCE(ctx, (memory_factor_kernel<DK, CHANNEL>), kBytes);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, memory_factor_kernel<DK, CHANNEL>, dim3(p.n_chunks, s.heads), dim3(F_THREADS), (size_t)kBytes, ctx->stream, s, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
template <int DK>
int32_t launch(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p) {
    if (s.decay == MemDecay::PerChannel)
        B2_CHECK((launch_factors<DK, true>(ctx, s, p)));
    else
        B2_CHECK((launch_factors<DK, false>(ctx, s, p)));
    constexpr int kBytes = WalkSmem<DK>::kBytes;
    B2_SMEM_ONCE(ctx, (memory_chunk_kernel<DK, true>), kBytes);
    B2_SMEM_ONCE(ctx, (memory_chunk_kernel<DK, false>), kBytes);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, s.delta ? memory_chunk_kernel<DK, true> : memory_chunk_kernel<DK, false>, dim3((s.vdim + VB - 1) / VB, s.heads, p.B),
                          dim3(W_THREADS), (size_t)kBytes, ctx->stream, s, p, ctx->dev_err));
    B2_LAUNCHED(ctx);
    return B2_OK;
}

}  // namespace

bool b2_memory_chunk_eligible(const MemorySpec& s) { return s.dim <= 128; }
size_t b2_memory_chunk_bytes(const MemorySpec& s) { return (size_t)s.heads * (s.dim <= 64 ? Record<64>::kBytes : Record<128>::kBytes); }
int32_t b2_memory_chunk_launch(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p) {
    if (p.n_chunks <= 0) return B2_OK;
    return s.dim <= 64 ? launch<64>(ctx, s, p) : launch<128>(ctx, s, p);
}
