// Linear memories over a prompt, 64 tokens at a time on tensor cores (serving format).
//
// With G_t the running sum of the decays' logarithms over a chunk (per key channel, or one number per head) and S0 the state
// before it,
//     (I + A) U = beta (V - Kf S0)      A_ts = beta_t k_t . (e^(G_t - G_s) k_s), s < t        Kf_t = e^(G_t) k_t
//     O = Qf S0 + P U                   P_ts = q_t . (e^(G_t - G_s) k_s), s <= t              Qf_t = e^(G_t) q_t
//     S = e^(G_end) S0 + Kb^T U         Kb_s = e^(G_end - G_s) k_s
// (a memory without the delta rule has U = V; with a bonus b the read-out of token t comes before its decay and write: e^(G_{t-1})
// in place of e^(G_t) in Qf and P, and P_tt = q_t . (b k_t)).  What does not depend on the state -- P, the inverse of I + A times beta, and
// the three scaled operands -- is made for all chunks of all heads at once by memory_factor_kernel; memory_chunk_kernel then
// walks the chunks of a head in order.
//
// Every operand that is f32 by nature enters the products as a bf16 head plus a bf16 remainder (the product of the two
// remainders is dropped), all sums are f32, and the state stays in f32 registers from chunk to chunk.
#include <type_traits>

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
// Decays per channel: with a reference m_i for each 16-token block i, the exponent of token t of block i and an earlier token s
// of block j splits into
//     G_t - G_s = (G_t - m_i) + (m_i - m_j) + (m_j - G_s)
// The outer two belong to one token each, the middle one is a number per channel and pair of blocks.  The reference is the sum
// in the block's middle: for decays up to 2^-40 in eight tokens the outer factors stay inside 2^+-40, so that a middle one
// which underflows belongs to a product below 2^-46.  A channel that decays faster takes the sums at the block's borders
// (before it on the left, at its end on the right: no factor above one); in the block's own tile, where neither works, it is
// left out of the product and added with every exponent taken from its difference.
constexpr int F_WARPS = 10, F_THREADS = F_WARPS * 32;  // a warp per 16 x 16 tile of P and A up to the diagonal
constexpr float kMaxSpread = 40.f;  // log2 units
template <int DK, bool CHANNEL>
struct FactorSmem {
    static constexpr int LD = DK + 4, LM = C + 4, kOp = C * DK * 2;
    // left operands (k, q; head and remainder), then the right one in f32, whose place A and its inverse take later
    static constexpr int LK = 0, LQ = 2 * kOp, G = 4 * kOp, kG = CHANNEL ? C * LD * 4 : 0, kM = C * LM * 4;
    static constexpr int M = G, Y = G + (kG > kM ? kG : kM), REF = Y + 3 * 16 * 17 * 4, BETA = REF + (CHANNEL ? 9 * DK * 4 : C * 4), kBytes = BETA + C * 4;
};

// BONUS: queries and keys are bf16, straight from the projections.
template <int DK, bool CHANNEL, bool BONUS>
__global__ void __launch_bounds__(F_THREADS, 2) memory_factor_kernel(const MemorySpec s, const MemoryParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    using L = FactorSmem<DK, CHANNEL>;
    using R = Record<DK>;
    constexpr int LD = L::LD, LM = L::LM;
    extern __shared__ __align__(16) uint8_t smem[];
    float* gs = reinterpret_cast<float*>(smem + L::G);      // CHANNEL: [C][LD] running sums (base 2), then k e^(m_j - G_s)
    float* M = reinterpret_cast<float*>(smem + L::M);       // [C][LM]: A below the diagonal, the transposed inverse above it
    float* Y = reinterpret_cast<float*>(smem + L::Y);       // [3][16][17]
    float* ref = reinterpret_cast<float*>(smem + L::REF);   // CHANNEL: [4][DK] left and [4][DK] right references, [DK] the end; else [C] running sums
    float* betas = reinterpret_cast<float*>(smem + L::BETA);
    __shared__ uint32_t fast[4][DK / 32];                   // per block: channels with strong decays
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
    const int chunk = blockIdx.x, h = blockIdx.y, D = s.dim, Q = s.q_cols(), kh = h / (s.heads / s.kv_heads);
    int b = -1;  // the last chunked portion that starts at or before this chunk (starts rise with the index)
    for (int i = lane; i < p.B; i += 32)
        if (p.chunk_off[i] >= 0 && p.chunk_off[i] <= chunk) b = i;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) b = max(b, __shfl_xor_sync(0xffffffffu, b, o));
    if (b < 0) return;
    const int n = p.cu_seqlens[b + 1] - p.cu_seqlens[b], t0 = (chunk - p.chunk_off[b]) * C, cnt = min(C, n - t0), last = cnt - 1;
    if (cnt <= 0) return;
    const size_t tok0 = (size_t)p.cu_seqlens[b] + t0;
    uint8_t* rec = reinterpret_cast<uint8_t*>(p.chunk) + ((size_t)chunk * s.heads + h) * R::kBytes;
    using E = typename std::conditional<BONUS, uint16_t, float>::type;
    const E *q, *k;
    size_t ldq = Q;
    if constexpr (BONUS) {
        ldq = p.ld;
        q = reinterpret_cast<const uint16_t*>(p.in) + tok0 * ldq + p.c_off + kh * D;
        k = q + Q;
    } else {
        q = p.q + tok0 * Q + kh * D;
        k = p.k + tok0 * Q + kh * D;
    }
    const float* lg = CHANNEL ? p.lg + tok0 * s.decays() + h * D : nullptr;

    if (tid < 4 * (DK / 32)) fast[tid / (DK / 32)][tid % (DK / 32)] = 0;
    if (tid < C) betas[tid] = s.delta && tid < cnt ? p.beta[(tok0 + tid) * s.heads + h] : 0.f;
    __syncthreads();
    if constexpr (CHANNEL) {  // a thread per channel and half of the chunk; the second half is raised by the first one's end
        constexpr int H = C / 2;
        const int d = tid % DK, half = tid / DK;
        if (half < 2) {
            float run = 0.f, x[16];
#pragma unroll
            for (int i = 0; i < H / 16; i++) {
#pragma unroll
                for (int t = 0; t < 16; t++) {
                    const int tok = half * H + 16 * i + t;
                    x[t] = tok < cnt && d < D ? lg[(size_t)tok * s.decays() + d] : 0.f;
                }
                const float before = run;
                float mid = run;
#pragma unroll
                for (int t = 0; t < 16; t++) {
                    run = fmaf(x[t], kLog2e, run);
                    gs[(half * H + 16 * i + t) * LD + d] = run;
                    if (t == 7) mid = run;
                }
                const bool strong = before - mid > kMaxSpread || mid - run > kMaxSpread;
                ref[(half * 2 + i) * DK + d] = strong ? before : mid;
                ref[(4 + half * 2 + i) * DK + d] = strong ? run : mid;
                if (strong) atomicOr(&fast[half * 2 + i][d >> 5], 1u << (d & 31));
            }
            if (half == 0) ref[8 * DK + d] = run;
        }
        __syncthreads();
        if (half == 1) {
            const float first = ref[8 * DK + d];
#pragma unroll
            for (int i = 2; i < 4; i++) {
                ref[i * DK + d] += first;
                ref[(4 + i) * DK + d] += first;
            }
#pragma unroll 8
            for (int t = H; t < C; t++) gs[t * LD + d] += first;
            ref[8 * DK + d] = gs[(C - 1) * LD + d];
        }
    } else if (tid < 32) {
        auto at = [&](int t) { return t < cnt ? (s.decay == MemDecay::Fixed ? p.log_decay[h] : p.lg[(tok0 + t) * s.heads + h]) * kLog2e : 0.f; };
        const float x = at(2 * tid), y = at(2 * tid + 1);
        float sum = x + y;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, sum, o);
            if (tid >= o) sum += u;
        }
        ref[2 * tid] = sum - y;
        ref[2 * tid + 1] = sum;
    }
    __syncthreads();

    // ---- one pass over the chunk, eight columns at a time: the tiles' operands and the walk's
    const bool vec = D % 4 == 0 && Q % 4 == 0 && (!BONUS || (p.ld % 4 == 0 && p.c_off % 4 == 0));
    for (int i = tid; i < C * (DK / 8); i += F_THREADS) {
        const int t = i / (DK / 8), x = i % (DK / 8), blk = t >> 4;
        float kv[8], qv[8], left[8], right[8], a[8];
#pragma unroll
        for (int e = 0; e < 8; e += 4) {
            const int d = x * 8 + e;
            if (vec) {
                float k4[4] = {0.f, 0.f, 0.f, 0.f}, q4[4] = {0.f, 0.f, 0.f, 0.f};
                if (t < cnt && d < D) {
                    Elt<E>::ld4(k + t * ldq + d, k4);
                    Elt<E>::ld4(q + t * ldq + d, q4);
                }
#pragma unroll
                for (int f = 0; f < 4; f++) kv[e + f] = k4[f], qv[e + f] = q4[f];
            } else {
#pragma unroll
                for (int f = 0; f < 4; f++) {
                    const bool ok = t < cnt && d + f < D;
                    kv[e + f] = ok ? Elt<E>::ld(k + t * ldq + d + f) : 0.f;
                    qv[e + f] = ok ? Elt<E>::ld(q + t * ldq + d + f) : 0.f;
                }
            }
        }
        const uint32_t o = at_wide(t, x, DK * 2);
        auto store = [&](uint8_t* base, const float (&v)[8]) {
            Split w[4];
#pragma unroll
            for (int e = 0; e < 4; e++) w[e] = split2(v[2 * e], v[2 * e + 1]);
            *reinterpret_cast<uint4*>(base + o) = make_uint4(w[0].hi, w[1].hi, w[2].hi, w[3].hi);
            *reinterpret_cast<uint4*>(base + R::kOp + o) = make_uint4(w[0].lo, w[1].lo, w[2].lo, w[3].lo);
        };
        if constexpr (CHANNEL) {
            float r0[8], tail[8];  // e^(m_i), e^(G_end - m_i)
            float own[8];          // bonus: the token's own decay, which its read-out does not see
#pragma unroll
            for (int e = 0; e < 8; e++) own[e] = BONUS && t < cnt && x * 8 + e < D ? lg[(size_t)t * s.decays() + x * 8 + e] * kLog2e : 0.f;
#pragma unroll
            for (int e = 0; e < 8; e++) {
                const int d = x * 8 + e;
                const float r = ref[blk * DK + d], m = ref[(4 + blk) * DK + d], g = gs[t * LD + d];
                left[e] = fast_exp2(g - own[e] - r);
                right[e] = kv[e] * fast_exp2(m - g);
                r0[e] = fast_exp2(r);
                tail[e] = fast_exp2(ref[8 * DK + d] - m);
                gs[t * LD + d] = right[e];
            }
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] = kv[e] * left[e];
            if (!BONUS && s.delta) {
                store(smem + L::LK, a);
#pragma unroll
                for (int e = 0; e < 8; e++) a[e] *= r0[e];
                store(rec + R::Kf, a);
            }
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] = qv[e] * left[e];
            store(smem + L::LQ, a);
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] *= r0[e];
            store(rec + R::Qf, a);
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] = right[e] * tail[e];
            store(rec + R::Kb, a);
        } else {
            const float f = fast_exp2(ref[t]), w = fast_exp2(ref[last] - ref[min(t, last)]);
            store(smem + L::LK, kv);
            store(smem + L::LQ, qv);
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] = kv[e] * f;
            if (!BONUS && s.delta) store(rec + R::Kf, a);
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] = qv[e] * f;
            store(rec + R::Qf, a);
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] = kv[e] * w;
            store(rec + R::Kb, a);
        }
    }
    if constexpr (BONUS) {  // the diagonal of P, in the place of the step sizes
        for (int t = warp; t < C; t += F_WARPS) {
            float v = 0.f;
            if (t < cnt)
                for (int d = lane; d < D; d += 32) v = fmaf(Elt<E>::ld(q + t * ldq + d) * p.bonus[(size_t)h * D + d], Elt<E>::ld(k + t * ldq + d), v);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (lane == 0) betas[t] = v;
        }
    }
    __syncthreads();

    // ---- P and A, a 16 x 16 tile (tokens 16 i .., earlier tokens 16 j ..) per warp
    int i = 0, j = warp;
    while (j > i) j -= ++i;
    float a[2][4], pr[2][4];
#pragma unroll
    for (int half = 0; half < 2; half++)
#pragma unroll
        for (int e = 0; e < 4; e++) a[half][e] = pr[half][e] = 0.f;
    const int ta = 16 * i + g4, tb = ta + 8;
    {
        const uint32_t base = smem_u32(smem);
#pragma unroll 2
        for (int kk = 0; kk < DK / 16; kk++) {
            uint32_t ah[4], al[4], qh[4], ql[4], bh[2][2], bl[2][2];
            const uint32_t at = at_wide(16 * i + lr + (mi & 1) * 8, 2 * kk + (mi >> 1), DK * 2);
            if (!BONUS && s.delta) {
                ldmatrix_x4(ah[0], ah[1], ah[2], ah[3], base + L::LK + at);
                ldmatrix_x4(al[0], al[1], al[2], al[3], base + L::LK + R::kOp + at);
            }
            ldmatrix_x4(qh[0], qh[1], qh[2], qh[3], base + L::LQ + at);
            ldmatrix_x4(ql[0], ql[1], ql[2], ql[3], base + L::LQ + R::kOp + at);
            if constexpr (CHANNEL) {
                const int d0 = kk * 16 + 2 * t4;
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int d = d0 + e * 8;
                    const float2 r = *reinterpret_cast<const float2*>(ref + i * DK + d), en = *reinterpret_cast<const float2*>(ref + (4 + j) * DK + d);
                    // (inside a block the references differ for the strong channels only)
                    const float f0 = i == j ? (r.x == en.x ? 1.f : 0.f) : fast_exp2(r.x - en.x), f1 = i == j ? (r.y == en.y ? 1.f : 0.f) : fast_exp2(r.y - en.y);
#pragma unroll
                    for (int half = 0; half < 2; half++) {
                        const float2 v = *reinterpret_cast<const float2*>(gs + (16 * j + half * 8 + g4) * LD + d);
                        const Split sp = split2(v.x * f0, v.y * f1);
                        bh[half][e] = sp.hi, bl[half][e] = sp.lo;
                    }
                }
            } else {
                const uint32_t bt = at_wide(16 * j + lr + (mi >> 1) * 8, 2 * kk + (mi & 1), DK * 2);
                ldmatrix_x4(bh[0][0], bh[0][1], bh[1][0], bh[1][1], base + L::LK + bt);
                ldmatrix_x4(bl[0][0], bl[0][1], bl[1][0], bl[1][1], base + L::LK + R::kOp + bt);
            }
#pragma unroll
            for (int half = 0; half < 2; half++) {
                if (!BONUS && s.delta) mma3(a[half], ah, al, bh[half], bl[half]);
                mma3(pr[half], qh, ql, bh[half], bl[half]);
            }
        }
    }
    if (CHANNEL && i == j) {
#pragma unroll 1
        for (int word = 0; word < DK / 32; word++)
            for (uint32_t m = fast[i][word]; m; m &= m - 1) {
                const int d = word * 32 + __ffs(m) - 1, tok = 16 * i + (lane & 15);  // a lane per token
                const bool ok = tok < cnt && d < D;
                float g = ok ? lg[(size_t)tok * s.decays() + d] * kLog2e : 0.f;
                const float kv = ok ? Elt<E>::ld(k + tok * ldq + d) : 0.f, qv = ok ? Elt<E>::ld(q + tok * ldq + d) : 0.f;
#pragma unroll
                for (int o = 1; o < 16; o <<= 1) {
                    const float x = __shfl_up_sync(0xffffffffu, g, o, 16);
                    if ((lane & 15) >= o) g += x;
                }
                float gt[2], kt[2], qt[2];
                const float before = BONUS ? __shfl_up_sync(0xffffffffu, g, 1, 16) : 0.f;  // (the first token's is not used)
#pragma unroll
                for (int x = 0; x < 2; x++) {
                    gt[x] = __shfl_sync(0xffffffffu, BONUS ? before : g, g4 + 8 * x);
                    kt[x] = __shfl_sync(0xffffffffu, kv, g4 + 8 * x);
                    qt[x] = __shfl_sync(0xffffffffu, qv, g4 + 8 * x);
                }
#pragma unroll
                for (int half = 0; half < 2; half++)
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        const int u = half * 8 + 2 * t4 + c;
                        const float gu = __shfl_sync(0xffffffffu, g, u), ku = __shfl_sync(0xffffffffu, kv, u);
#pragma unroll
                        for (int x = 0; x < 2; x++)
                            if (BONUS ? u < g4 + 8 * x : u <= g4 + 8 * x) {
                                const float w = fast_exp2(gt[x] - gu) * ku;
                                a[half][2 * x + c] = fmaf(w, kt[x], a[half][2 * x + c]);
                                pr[half][2 * x + c] = fmaf(w, qt[x], pr[half][2 * x + c]);
                            }
                    }
            }
    }
    __syncthreads();  // the right operand's place becomes A's
#pragma unroll
    for (int half = 0; half < 2; half++) {
        const int u0 = 16 * j + half * 8 + 2 * t4;
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int t = e < 2 ? ta : tb, u = u0 + (e & 1);
            if constexpr (!CHANNEL) {
                const float w = u <= t ? fast_exp2(ref[t] - ref[u]) : 0.f;
                a[half][e] *= w;
                pr[half][e] *= w;
            }
            if (u > t) pr[half][e] = 0.f;
            if (CHANNEL && BONUS && u == t) pr[half][e] = betas[t];
            if (!BONUS && s.delta && u < t) M[t * LM + u] = a[half][e] * betas[t];
        }
#pragma unroll
        for (int row = 0; row < 2; row++) {
            const Split sp = split2(pr[half][2 * row], pr[half][2 * row + 1]);
            const uint32_t o = at_wide(row ? tb : ta, u0 >> 3, 128) + (u0 & 7) * 2;
            *reinterpret_cast<uint32_t*>(rec + R::P + o) = sp.hi;
            *reinterpret_cast<uint32_t*>(rec + R::P + R::kMat + o) = sp.lo;
        }
    }
    // the chunk's whole decay, over the first token's entry (which only this block reads)
    if constexpr (CHANNEL) {
        if (tid < D) p.lg[tok0 * s.decays() + h * D + tid] = fast_exp2(ref[8 * DK + tid]);
    } else if (s.decay == MemDecay::PerHead && tid == 0) {
        p.lg[tok0 * s.heads + h] = fast_exp2(ref[last]);
    }
    if (BONUS || !s.delta) return;
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
            for (int m = j; m < i; m++)
#pragma unroll
                for (int x = 0; x < 16; x++) acc = fmaf(M[(16 * i + t) * LM + 16 * m + x], inv(m, j, x, u), acc);
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
// Block = (32 value columns of one head, sequence).  Per chunk, eight warps (16 tokens x 16 columns each) form Kf S0 and from
// it U, while eight others form Qf S0; then those add P U and store O, and every warp updates its 16 x 16 part of the state.
// The next chunk's tiles arrive by bulk copies: Kf and Qf into the other of two buffers, the rest as soon as its place is free.
constexpr int W_THREADS = 512, W_HALF = 256;
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
    // state of this warp: rows sr + g4 (+ 8), columns sc + 8 j + 2 t4 (+ 1); with keys up to 64 half of the warps have none
    constexpr int NT = 2;
    const int sr = (warp >> 1) * 16, sc = (warp & 1) * 16;
    const bool has_state = sr < DK;
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
        if (!has_state) return;
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
    const bool reads = warp >= 8;                             // this warp forms O, not U
    const int mt = (warp >> 1) & 3, nc = (warp & 1) * 16;     // tokens mt * 16 .., columns nc ..
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
    // heads' and remainders' products in accumulators of their own: shorter chains
    struct Acc {
        float d[2][4], e[2][4];
        __device__ __forceinline__ void clear() {
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int i = 0; i < 4; i++) d[j][i] = e[j][i] = 0.f;
        }
        __device__ __forceinline__ void add(const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh0)[2], const uint32_t (&bh1)[2],
                                            const uint32_t (&bl0)[2], const uint32_t (&bl1)[2]) {
            mma_bf16_16816(d[0], ah, bh0);
            mma_bf16_16816(d[1], ah, bh1);
            mma_bf16_16816(e[0], ah, bl0);
            mma_bf16_16816(e[1], ah, bl1);
            mma_bf16_16816(e[0], al, bh0);
            mma_bf16_16816(e[1], al, bh1);
        }
        __device__ __forceinline__ void add(const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&b0)[2], const uint32_t (&b1)[2]) {
            mma_bf16_16816(d[0], ah, b0);
            mma_bf16_16816(d[1], ah, b1);
            mma_bf16_16816(e[0], al, b0);
            mma_bf16_16816(e[1], al, b1);
        }
        __device__ __forceinline__ float at(int j, int i) const { return d[j][i] + e[j][i]; }
    };
    if (!reads) fetch_v(0);
    bool alive = true;
    for (int c = 0; c < chunks; c++) {
        const uint32_t ph = (uint32_t)c & 1u, kq = L::KQ + ph * L::kKQ;
        if (tid == 0 && c + 1 < chunks) load_kq(c + 1);  // (its buffer was last read before the previous chunk's barriers)
        if (has_state) fetch_decay(c);
        alive = mbar_wait(ph ? f_kq[1] : f_kq[0], (uint32_t)(c >> 1) & 1u) && alive;
        Acc o;
        // ---- what the state before the chunk answers to the keys, or to the queries
        if (DELTA || reads) {
            const uint32_t op = kq + (reads ? 2 * R::kOp : 0);
            o.clear();
#pragma unroll
            for (int k = 0; k < DK / 16; k++) {
                uint32_t ah[4], al[4], bh0[2], bh1[2], bl0[2], bl1[2];
                frag_b(L::S, k * 16, nc >> 3, bh0, bh1);
                frag_b(L::S + L::kS, k * 16, nc >> 3, bl0, bl1);
                frag_a(op, DK * 2, mt * 16, 2 * k, ah);
                frag_a(op + R::kOp, DK * 2, mt * 16, 2 * k, al);
                o.add(ah, al, bh0, bh1, bl0, bl1);
            }
        }
        // ---- U
        if (!reads) {
            if constexpr (DELTA) {
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    put(L::RU, L::kU, ta, nc + j * 8 + 2 * t4, bflo(vv[j][0]) - o.at(j, 0), bfhi(vv[j][0]) - o.at(j, 1));
                    put(L::RU, L::kU, tb, nc + j * 8 + 2 * t4, bflo(vv[j][1]) - o.at(j, 2), bfhi(vv[j][1]) - o.at(j, 3));
                }
                if (c + 1 < chunks) fetch_v(c + 1);
                alive = mbar_wait(f_t, ph) && alive;
                asm volatile("bar.sync 1, %0;\n" ::"n"(W_HALF) : "memory");
                o.clear();
#pragma unroll
                for (int k = 0; k < C / 16; k++)
                    if (k <= mt) {
                        uint32_t ah[4], al[4], bh0[2], bh1[2], bl0[2], bl1[2];
                        frag_a(L::T, 128, mt * 16, 2 * k, ah);
                        frag_a(L::T + R::kMat, 128, mt * 16, 2 * k, al);
                        frag_b(L::RU, k * 16, nc >> 3, bh0, bh1);
                        frag_b(L::RU + L::kU, k * 16, nc >> 3, bl0, bl1);
                        o.add(ah, al, bh0, bh1, bl0, bl1);
                    }
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    put(L::U, L::kU, ta, nc + j * 8 + 2 * t4, o.at(j, 0), o.at(j, 1));
                    put(L::U, L::kU, tb, nc + j * 8 + 2 * t4, o.at(j, 2), o.at(j, 3));
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
        }
        alive = mbar_wait(f_pk, ph) && alive;
        alive = __syncthreads_and(alive);
        if (!alive) break;
        if (DELTA && tid == 0 && c + 1 < chunks) load_t(c + 1);
        // ---- the state
        if (has_state) {
            Acc u;
            u.clear();
#pragma unroll
            for (int j = 0; j < NT; j++) u.d[j][0] = S[j][0] * dec[0], u.d[j][1] = S[j][1] * dec[0], u.d[j][2] = S[j][2] * dec[1], u.d[j][3] = S[j][3] * dec[1];
#pragma unroll
            for (int k = 0; k < C / 16; k++) {
                // Kb^T: rows of keys from rows of tokens
                uint32_t ah[4], al[4], bh0[2], bh1[2], bl0[2], bl1[2];
                const uint32_t x = at_wide(k * 16 + lr + (mi >> 1) * 8, (sr >> 3) + (mi & 1), DK * 2);
                ldmatrix_x4_trans(ah[0], ah[1], ah[2], ah[3], base + L::Kb + x);
                ldmatrix_x4_trans(al[0], al[1], al[2], al[3], base + L::Kb + R::kOp + x);
                frag_b(L::U, k * 16, sc >> 3, bh0, bh1);
                if constexpr (DELTA) {
                    frag_b(L::U + L::kU, k * 16, sc >> 3, bl0, bl1);
                    u.add(ah, al, bh0, bh1, bl0, bl1);
                } else {
                    u.add(ah, al, bh0, bh1);
                }
            }
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int i = 0; i < 4; i++) S[j][i] = u.at(j, i);
            put_state();
        }
        // ---- O
        if (reads) {
#pragma unroll
            for (int k = 0; k < C / 16; k++)
                if (k <= mt) {
                    uint32_t ah[4], al[4], bh0[2], bh1[2], bl0[2], bl1[2];
                    frag_a(L::P, 128, mt * 16, 2 * k, ah);
                    frag_a(L::P + R::kMat, 128, mt * 16, 2 * k, al);
                    frag_b(L::U, k * 16, nc >> 3, bh0, bh1);
                    if constexpr (DELTA) {
                        frag_b(L::U + L::kU, k * 16, nc >> 3, bl0, bl1);
                        o.add(ah, al, bh0, bh1, bl0, bl1);
                    } else {
                        o.add(ah, al, bh0, bh1);
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
                        *reinterpret_cast<float2*>(x) = make_float2(o.at(j, 2 * row), o.at(j, 2 * row + 1));
                    } else {
                        if (p0 + q < P) x[0] = o.at(j, 2 * row);
                        if (p0 + q + 1 < P) x[1] = o.at(j, 2 * row + 1);
                    }
                }
        }
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
            if (has_state && r < D && p0 + q < P) Sg[(size_t)q * D + r] = S[j][e];
        }
    memory_keep_inputs<uint16_t>(s, p, b, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
}

template <int DK, bool CHANNEL, bool BONUS>
int32_t launch_factors(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p) {
    constexpr int kBytes = FactorSmem<DK, CHANNEL>::kBytes;
    B2_SMEM_ONCE(ctx, (memory_factor_kernel<DK, CHANNEL, BONUS>), kBytes);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, memory_factor_kernel<DK, CHANNEL, BONUS>, dim3(p.n_chunks, s.heads), dim3(F_THREADS), (size_t)kBytes, ctx->stream, s, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
template <int DK>
int32_t launch(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p) {
    if (s.bonus)
        B2_CHECK((launch_factors<DK, true, true>(ctx, s, p)));
    else if (s.decay == MemDecay::PerChannel)
        B2_CHECK((launch_factors<DK, true, false>(ctx, s, p)));
    else
        B2_CHECK((launch_factors<DK, false, false>(ctx, s, p)));
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
