// Prefill attention of latent-attention layers on the 5th-generation tensor cores (tcgen05 + TMEM).
//
// A prompt portion of more than a token sees every context row many times, so here the up-projections are NOT absorbed:
// the latents of each prefilling sequence's whole context are gathered from their pages and expanded once per layer
// (one dense product) into per-head keys and values, and the attention runs on those:
//   S = q_plain . k_plain(head) + q_rotated . k_rotated(shared),   O = P V(head)
// with the plain and the rotated part of a head padded to 64-wide blocks and V to one or two such blocks.
//
// CTA = (128-query tile of one sequence's portion, one head), flash attention over 128-key tiles:
//   warp 8      one thread: the Q tile, then per key tile the 64-wide K blocks (plain blocks from the expanded buffer,
//               rotated blocks from the buffer all heads share), two stages
//   warp 9      one thread: the V blocks, two stages
//   warp 10     one thread issues tcgen05.mma: S = Q K^T into one of two TMEM buffers; O += P V with P read from TMEM as
//               the A operand (bf16 head, then bf16 remainder) and V as an MN-major operand
//   warps 0-7   softmax, thread = (query row, half of the key tile); P goes over the scores it came from; the running
//               maximum is raised only when a tile exceeds it by 2^8; every wait bounded
// Keys past a sequence's context lie in the next sequence's rows (or in zeros): finite, and masked.
#include "elt.cuh"
#include "layer_kernels.h"
#include "tc5.cuh"

namespace {

using namespace tc5;

constexpr int QT = 128, KT = 128;
constexpr int kSoftmaxWarps = 8, kKWarp = 8, kVWarp = 9, kMmaWarp = 10, kThreads = 352;
constexpr int BLOCK_BYTES = 128 * 128;  // 128 rows x 64 bf16, 128-byte swizzle
constexpr float kRescaleThreshold = 8.0f;  // log2 units
// reference point of a row that sees nothing of the first tile (under a mask): its weights are zero until a tile raises it
constexpr float kNoKeyYet = -1e30f;

// f32 accumulate, bf16 x bf16, M = 128; bit 16 set = B is MN-major
constexpr uint32_t idesc(int n, bool b_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(128 >> 4) << 24) | (b_mn ? (1u << 16) : 0u);
}

template <int DKB, int VDB>
struct Layout {  // shared memory of a CTA
    static constexpr int NS = 2;  // K / V stages
    static constexpr int Q = 0, K = DKB * BLOCK_BYTES, V = K + NS * DKB * BLOCK_BYTES, BAR = V + NS * VDB * BLOCK_BYTES, X = BAR + 256, BYTES = X + 2048;
};

template <int DKB, int VDB>
__global__ void __launch_bounds__(kThreads, 1)
    latent_prefill_tc_kernel(const LatentPrefillParams p, const MaskSpec mask, int* err, const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                             const __grid_constant__ CUtensorMap map_r) {
    using L = Layout<DKB, VDB>;
    constexpr int NS = L::NS;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int w = blockIdx.x;
    if (w >= *p.n_work) return;
    const uint32_t base = smem_u32(smem_raw);
    if (base & 1023u) {  // the swizzled operand layouts need this alignment; every thread sees the same value
        if (threadIdx.x == 0) atomicExch(err, 7);
        return;
    }
    const uint32_t bar = base + L::BAR;
    const uint32_t q_full = bar;
    auto k_full = [&](int s) { return bar + 8u * (1 + s); };
    auto k_empty = [&](int s) { return bar + 8u * (3 + s); };
    auto v_full = [&](int s) { return bar + 8u * (5 + s); };
    auto v_empty = [&](int s) { return bar + 8u * (7 + s); };
    auto s_ready = [&](int s) { return bar + 8u * (9 + s); };
    auto p_ready = [&](int s) { return bar + 8u * (11 + s); };   // all softmax warps have written P over S buffer s
    auto x_ready = [&](int s) { return bar + 8u * (13 + s); };   // both softmax groups have published their maxima
    auto pv_done = [&](int s) { return bar + 8u * (15 + s); };   // P V of a tile of this parity has completed
    const uint32_t l_ready = bar + 8u * 17, slot_addr = bar + 8u * 18;
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem_raw + L::BAR + 8 * 18);

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int head = blockIdx.y;
    const int b = p.pf_seq[w], q_start = p.pf_qstart[w];
    const int tok0 = p.cu_seqlens[b], qn = p.cu_seqlens[b + 1] - tok0;
    const int ctx = p.context_lens[b], ctx_before = ctx - qn, kv0 = p.kv_off[b];
    const int rows = min(QT, qn - q_start);
    // under a mask the walk starts at the tile of the first query's first visible key; tile numbers count from there
    const int kv_lo = mask.first(ctx_before);  // the gathered rows start with this key
    const int first_tile = (mask.first(ctx_before + q_start) - kv_lo) / KT, key0 = kv_lo + first_tile * KT;
    const int n_tiles = (ctx_before + q_start + rows - 1 - key0) / KT + 1;

    if (tid == 0) {
        mbar_init(q_full, 1);
        for (int s = 0; s < NS; s++) {
            mbar_init(k_full(s), 1);
            mbar_init(k_empty(s), 1);
            mbar_init(v_full(s), 1);
            mbar_init(v_empty(s), 1);
            mbar_init(s_ready(s), 1);
            mbar_init(p_ready(s), kSoftmaxWarps);
            mbar_init(x_ready(s), kSoftmaxWarps);
            mbar_init(pv_done(s), 1);
        }
        mbar_init(l_ready, kSoftmaxWarps);
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == kMmaWarp) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(slot_addr), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t tmem_o = tmem_base + 256u;
    bool alive = true;

    if (warp == kKWarp) {
        if (lane == 0) {
            mbar_expect_tx(q_full, (uint32_t)DKB * BLOCK_BYTES);
            for (int i = 0; i < DKB; i++) tma_load_2d(base + L::Q + i * BLOCK_BYTES, &map_q, (head * DKB + i) * 64, tok0 + q_start, q_full);
            int st = 0;
            uint32_t par = 0;
            for (int j = 0; j < n_tiles; j++) {
                if (!mbar_wait(k_empty(st), par ^ 1u)) {
                    alive = false;
                    break;
                }
                mbar_expect_tx(k_full(st), (uint32_t)DKB * BLOCK_BYTES);
                const uint32_t dst = base + L::K + (uint32_t)st * DKB * BLOCK_BYTES;
                const int row = kv0 + (first_tile + j) * KT;
                for (int i = 0; i < DKB; i++)
                    if (i < p.plain_blocks)
                        tma_load_2d(dst + i * BLOCK_BYTES, &map_kv, (head * p.plain_blocks + i) * 64, row, k_full(st));
                    else
                        tma_load_2d(dst + i * BLOCK_BYTES, &map_r, (i - p.plain_blocks) * 64, row, k_full(st));
                if (++st == NS) st = 0, par ^= 1u;
            }
            if (!alive) atomicExch(err, 2);
        }
        __syncwarp();
    } else if (warp == kVWarp) {
        if (lane == 0) {
            int st = 0;
            uint32_t par = 0;
            for (int j = 0; j < n_tiles; j++) {
                if (!mbar_wait(v_empty(st), par ^ 1u)) {
                    alive = false;
                    break;
                }
                mbar_expect_tx(v_full(st), (uint32_t)VDB * BLOCK_BYTES);
                for (int i = 0; i < VDB; i++)
                    tma_load_2d(base + L::V + (uint32_t)(st * VDB + i) * BLOCK_BYTES, &map_kv, p.v_col0 + (head * VDB + i) * 64, kv0 + (first_tile + j) * KT, v_full(st));
                if (++st == NS) st = 0, par ^= 1u;
            }
            if (!alive) atomicExch(err, 2);
        }
        __syncwarp();
    } else if (warp == kMmaWarp) {
        if (lane == 0) {
            constexpr uint32_t kQK = idesc(128, false), kPV = idesc(VDB * 64, true);
            const uint64_t dq0 = desc_kmajor(base + L::Q), dk0 = desc_kmajor(base + L::K), dv0 = desc_mnmajor(base + L::V, BLOCK_BYTES);
            auto issue_qk = [&](int j, int kst) {  // S[j & 1] = Q K_j^T
                const uint64_t dk = dk0 + (uint64_t)((uint32_t)kst * DKB * (BLOCK_BYTES >> 4));
                const uint32_t ts = tmem_base + (uint32_t)(j & 1) * 128u;
#pragma unroll
                for (int k = 0; k < DKB * 4; k++) {
                    const uint64_t off = (uint64_t)((uint32_t)(k >> 2) * (BLOCK_BYTES >> 4) + (uint32_t)(k & 3) * 2);
                    tc_mma(ts, dq0 + off, dk + off, kQK, k > 0 ? 1u : 0u);
                }
                tc_commit(s_ready(j & 1));
                tc_commit(k_empty(kst));
            };
            alive = mbar_wait(q_full, 0);
            for (int j = 0; j < 2 && j < n_tiles && alive; j++) {
                alive = mbar_wait(k_full(j), 0);
                if (alive) {
                    tc_fence_after();
                    issue_qk(j, j);
                }
            }
            for (int j = 0; j < n_tiles && alive; j++) {  // with two stages, stage and parity follow from the tile number
                const int sb = j & 1;
                const uint32_t ph = (uint32_t)(j >> 1) & 1u;
                alive = mbar_wait(v_full(sb), ph) && mbar_wait(p_ready(sb), ph);
                if (!alive) break;
                tc_fence_after();
                const uint64_t dvs = dv0 + (uint64_t)((uint32_t)sb * VDB * (BLOCK_BYTES >> 4));
                const uint32_t tP = tmem_base + (uint32_t)sb * 128u;
#pragma unroll
                for (int k = 0; k < KT / 16; k++) {
                    // keys 0-63 of the tile: head in columns 0-31 of the buffer, remainder in 32-63; keys 64-127: 64-95, 96-127
                    const uint32_t ta = tP + (uint32_t)(k >> 2) * 64u + (uint32_t)(k & 3) * 8u;
                    // 16 keys of a V block (128 keys x 64 values; the next 64 values are a block further)
                    const uint64_t dv = dvs + (uint64_t)((uint32_t)k * (2048u >> 4));
                    tc_mma_ts(tmem_o, ta, dv, kPV, (j > 0 || k > 0) ? 1u : 0u);
                    tc_mma_ts(tmem_o, ta + 32u, dv, kPV, 1u);
                }
                tc_commit(pv_done(sb));
                tc_commit(v_empty(sb));
                if (j + 2 < n_tiles) {  // S(j+2) goes over P(j): issued after the MMAs above, which complete first
                    alive = mbar_wait(k_full(sb), ph ^ 1u);
                    if (!alive) break;
                    tc_fence_after();
                    issue_qk(j + 2, sb);
                }
            }
            if (!alive) atomicExch(err, 3);
        }
        __syncwarp();
    } else {
        // ---------------- softmax: thread = (query row = TMEM lane, half of the key tile) ----------------
        // warps 0-3 take keys 0-63 of every tile, warps 4-7 keys 64-127 (a warp reaches the TMEM lanes
        // 32 * (warp % 4) ..); the two threads of a row agree on the row maximum through shared memory
        const int wg = warp >> 2, r = tid & 127;
        const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
        const bool row_ok = r < rows;
        // last key this row may see; rows past the chunk see the whole context (their result is dropped)
        const int kvis = row_ok ? min(ctx_before + q_start + r, ctx - 1) : ctx - 1;
        const int klow = mask.first(kvis);  // first key it may see
        float m_run = -INFINITY, l_run = 0.f;  // l_run: this thread's half of the row sum
        volatile float* xb = reinterpret_cast<volatile float*>(smem_raw + L::X);  // [2 tiles in flight][2 groups][128 rows]
        for (int j = 0; j < n_tiles && alive; j++) {
            const int st = j & 1;
            const uint32_t s_addr = tmem_base + lane_addr + (uint32_t)st * 128u + (uint32_t)wg * 64u;
            if (!__all_sync(0xffffffffu, mbar_wait(s_ready(st), (uint32_t)(j >> 1) & 1u))) {
                alive = false;
                break;
            }
            tc_fence_after();
            const int key_base = key0 + j * KT + wg * 64;
            const bool need_mask = key_base + 63 > kvis || key_base < klow;
            // this thread's 64 scores (log2 domain, masked), their maximum, then the maximum of the whole row
            uint32_t v0[32], v1[32];
            tc_ld32_nowait(s_addr, v0);
            tc_ld32_nowait(s_addr + 32u, v1);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
            // raw scores: the scale is positive, so the maximum can be taken first and scaled once, and the
            // exponent below is one fused multiply-add per score.  Masking (tiles on an edge only) writes -inf.
            if (need_mask) {
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    if (key_base + i > kvis || key_base + i < klow) v0[i] = 0xff800000u;
                    if (key_base + 32 + i > kvis || key_base + 32 + i < klow) v1[i] = 0xff800000u;
                }
            }
            float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
                mx0 = fmaxf(mx0, __uint_as_float(v0[i]));
                mx1 = fmaxf(mx1, __uint_as_float(v0[i + 1]));
                mx2 = fmaxf(mx2, __uint_as_float(v1[i]));
                mx3 = fmaxf(mx3, __uint_as_float(v1[i + 1]));
            }
            float mx = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * p.scale_log2;
            xb[(st * 2 + wg) * 128 + r] = mx;
            __syncwarp();
            if (lane == 0) mbar_arrive(x_ready(st));  // (release: the maxima above are visible to whoever sees the phase complete)
            if (!__all_sync(0xffffffffu, mbar_wait(x_ready(st), (uint32_t)(j >> 1) & 1u))) {
                alive = false;
                break;
            }
            mx = fmaxf(mx, xb[(st * 2 + (wg ^ 1)) * 128 + r]);
            // raise the reference point only when this tile exceeds it by more than the threshold
            float alpha = 1.f;
            bool rescale = false;
            if (j == 0) {
                m_run = fmaxf(mx, kNoKeyYet);
            } else if (mx > m_run + kRescaleThreshold) {
                alpha = exp2f(m_run - mx);
                m_run = mx;
                rescale = true;
            }
            if (__any_sync(0xffffffffu, rescale)) {  // this group rescales its half of the values
                // O belongs to the previous tile's P V until it has completed (P V of this tile cannot have been
                // issued yet: it waits for this warp's arrival below)
                if (!__all_sync(0xffffffffu, mbar_wait(pv_done((j - 1) & 1), (uint32_t)((j - 1) >> 1) & 1u))) {
                    alive = false;
                    break;
                }
                tc_fence_after();
#pragma unroll 1
                for (int c = 0; c < VDB; c++) {
                    const uint32_t o_addr = tmem_o + lane_addr + (uint32_t)wg * (VDB * 32u) + (uint32_t)c * 32u;
                    uint32_t v[32];
                    tc_ld32(o_addr, v);
#pragma unroll
                    for (int i = 0; i < 32; i++) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
                    tc_st32(o_addr, v);
                }
            }
            l_run *= alpha;
            // P = exp2(scale * s - m), row sum; bf16 head and remainder as pairs of consecutive keys, over the scores'
            // own columns.  The head is the upper 16 bits of the f32 (truncated, not rounded: the remainder carries what
            // is cut off, and truncating the remainder leaves a relative error below 2^-15), so the split costs integer
            // and add instructions only -- conversions share the exp2 unit's narrow issue rate.
            // Columns of this thread's 64: head of keys 0-31 in 0-15, of keys 32-63 in 16-31, remainders in 32-47 and
            // 48-63 (a column holds two consecutive keys); the first half is on its way while the second is computed.
            const float neg_m = -m_run, sc = p.scale_log2;
            float l0 = 0.f, l1 = 0.f;
            {
                uint32_t hi[16], lo[16];
#pragma unroll
                for (int i = 0; i < 16; i++) {
                    const float a0 = fast_exp2(fmaf(__uint_as_float(v0[2 * i]), sc, neg_m)), a1 = fast_exp2(fmaf(__uint_as_float(v0[2 * i + 1]), sc, neg_m));
                    l0 += a0;
                    l1 += a1;
                    const uint32_t u0 = __float_as_uint(a0), u1 = __float_as_uint(a1);
                    hi[i] = __byte_perm(u0, u1, 0x7632);
                    lo[i] = __byte_perm(__float_as_uint(a0 - __uint_as_float(u0 & 0xffff0000u)), __float_as_uint(a1 - __uint_as_float(u1 & 0xffff0000u)), 0x7632);
                }
                tc_st16_nowait(s_addr, hi);
                tc_st16_nowait(s_addr + 32u, lo);
            }
            {
                uint32_t hi[16], lo[16];
#pragma unroll
                for (int i = 0; i < 16; i++) {
                    const float a0 = fast_exp2(fmaf(__uint_as_float(v1[2 * i]), sc, neg_m)), a1 = fast_exp2(fmaf(__uint_as_float(v1[2 * i + 1]), sc, neg_m));
                    l0 += a0;
                    l1 += a1;
                    const uint32_t u0 = __float_as_uint(a0), u1 = __float_as_uint(a1);
                    hi[i] = __byte_perm(u0, u1, 0x7632);
                    lo[i] = __byte_perm(__float_as_uint(a0 - __uint_as_float(u0 & 0xffff0000u)), __float_as_uint(a1 - __uint_as_float(u1 & 0xffff0000u)), 0x7632);
                }
                tc_st16_nowait(s_addr + 16u, hi);
                tc_st16_nowait(s_addr + 48u, lo);
            }
            l_run += l0 + l1;
            asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_ready(st));
        }
        // ---------------- output: O / l, each group its half of the values ----------------
        if (alive && !__all_sync(0xffffffffu, mbar_wait(pv_done((n_tiles - 1) & 1), (uint32_t)((n_tiles - 1) >> 1) & 1u))) alive = false;
        // the row sum is the two halves' sums (slot of the tile parity that is not in use any more)
        if (alive) {
            const int slot = n_tiles & 1;
            xb[(slot * 2 + wg) * 128 + r] = l_run;
            __syncwarp();
            if (lane == 0) mbar_arrive(l_ready);
            if (!__all_sync(0xffffffffu, mbar_wait(l_ready, 0))) alive = false;
            l_run += xb[(slot * 2 + (wg ^ 1)) * 128 + r];
        }
        if (alive) {
            tc_fence_after();
            const float inv = 1.0f / l_run;
            uint16_t* dst = reinterpret_cast<uint16_t*>(p.out) + (size_t)(tok0 + q_start + (row_ok ? r : 0)) * p.ldo + (size_t)head * p.vdim;
            const bool vec = p.vdim % 8 == 0;  // rows are 16-byte aligned then (ldo is a multiple of 64)
#pragma unroll 1
            for (int c = 0; c < VDB; c++) {
                uint32_t v[32];
                const int c0 = wg * (VDB * 32) + c * 32;
                tc_ld32(tmem_o + lane_addr + (uint32_t)c0, v);
#pragma unroll
                for (int g = 0; g < 4; g++) {
                    const int col = c0 + g * 8;
                    if (!row_ok) {
                        // nothing to store; the warp stays together for the next load
                    } else if (vec && col < p.vdim) {
                        uint4 o4;
                        o4.x = pack_bf2(__uint_as_float(v[g * 8 + 0]) * inv, __uint_as_float(v[g * 8 + 1]) * inv);
                        o4.y = pack_bf2(__uint_as_float(v[g * 8 + 2]) * inv, __uint_as_float(v[g * 8 + 3]) * inv);
                        o4.z = pack_bf2(__uint_as_float(v[g * 8 + 4]) * inv, __uint_as_float(v[g * 8 + 5]) * inv);
                        o4.w = pack_bf2(__uint_as_float(v[g * 8 + 6]) * inv, __uint_as_float(v[g * 8 + 7]) * inv);
                        *reinterpret_cast<uint4*>(dst + col) = o4;
                    } else if (!vec) {
#pragma unroll
                        for (int i = 0; i < 8; i++)
                            if (col + i < p.vdim) dst[col + i] = f2bf(__uint_as_float(v[g * 8 + i]) * inv);
                    }
                }
                __syncwarp();
            }
        } else if (lane == 0) {
            atomicExch(err, 4);
        }
    }

    tc_fence_before();
    __syncthreads();
    if (warp == kMmaWarp) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem_base), "r"(512) : "memory");
    }
}

// Context rows of the prefilling sequences, gathered from their pages: latents [rows, ld_lat] (zero beyond kv_rank) and
// rotated key parts [rows, rot_pad] (zero beyond rot_dim).  Under a mask a sequence's rows start with the first key that its
// portion's first token sees.  One warp per row.
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentAttnSpec a, const LatentGatherParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= p.rows) return;
    int best = -1;  // the last prefilling sequence that starts at or before this row (starts rise with the index)
    for (int i = lane; i < p.B; i += 32)
        if (p.kv_off[i] >= 0 && p.kv_off[i] <= row) best = i;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) best = max(best, __shfl_xor_sync(0xffffffffu, best, o));
    int key = 0;
    if (best >= 0) key = row - p.kv_off[best] + a.mask.first(p.context_lens[best] - (p.cu_seqlens[best + 1] - p.cu_seqlens[best]));
    const int W = a.row_pad(), R = a.kv_rank;
    const bool ok = best >= 0 && key < p.context_lens[best];
    const uint16_t* src = reinterpret_cast<const uint16_t*>(p.cache);
    if (ok) src += ((size_t)p.block_tables[(size_t)p.seq_slot[best] * p.max_blocks + key / p.page_size] * p.page_size + key % p.page_size) * W;
    uint16_t* lat = reinterpret_cast<uint16_t*>(p.lat) + (size_t)row * p.ld_lat;
    uint16_t* kr = reinterpret_cast<uint16_t*>(p.rot) + (size_t)row * p.rot_pad;
    if (R % 8 == 0) {
        for (int i = lane * 8; i < p.ld_lat; i += 256)
            *reinterpret_cast<uint4*>(lat + i) = ok && i < R ? *reinterpret_cast<const uint4*>(src + i) : make_uint4(0, 0, 0, 0);
    } else {
        for (int i = lane; i < p.ld_lat; i += 32) lat[i] = ok && i < R ? src[i] : 0;
    }
    for (int i = lane; i < p.rot_pad; i += 32) kr[i] = ok && i < a.rot_dim ? src[R + i] : 0;
}

template <int DKB, int VDB>
int32_t launch(b2_ctx* ctx, const LatentAttnSpec& a, const LatentPrefillParams& p, int grid_work, const CUtensorMap& mq, const CUtensorMap& mkv, const CUtensorMap& mr) {
    constexpr int kBytes = Layout<DKB, VDB>::BYTES;
    B2_SMEM_ONCE(ctx, (latent_prefill_tc_kernel<DKB, VDB>), kBytes);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, latent_prefill_tc_kernel<DKB, VDB>, dim3(grid_work, a.heads), dim3(kThreads), (size_t)kBytes, ctx->stream, p, a.mask,
                          ctx->dev_err, mq, mkv, mr));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int blocks64(int n) { return (n + 63) / 64; }

}  // namespace

bool b2_latent_prefill_eligible(const LatentAttnSpec& a) {
    const int dk = blocks64(a.dim) + blocks64(a.rot_dim);
    return dk <= 3 && blocks64(a.vdim) <= 2 && a.scale > 0.f;
}
int32_t b2_latent_gather_launch(b2_ctx* ctx, const LatentAttnSpec& a, const LatentGatherParams& p) {
    if (p.rows <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, latent_gather_kernel, dim3((p.rows + 7) / 8), dim3(256), 0, ctx->stream, a, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
// The work list must have been built with 128-query tiles; q, kv and rot have at least 128 rows each (a load box is never
// taller than its tensor).
int32_t b2_latent_prefill_launch(b2_ctx* ctx, const LatentAttnSpec& a, const LatentPrefillParams& p, int grid_work) {
    if (grid_work <= 0) return B2_OK;
    B2_REQUIRE(p.q_rows >= QT && p.kv_rows >= KT, B2_ERR_MSG, "latent prefill: operand buffers need at least 128 rows");
    const int dk = p.plain_blocks + blocks64(a.rot_dim), vd = blocks64(a.vdim);
    CUtensorMap mq, mkv, mr;
    B2_CHECK(get_map(ctx, p.q, (uint64_t)p.q_rows, (uint64_t)a.heads * dk * 64, (uint64_t)a.heads * dk * 64, QT, &mq));
    B2_CHECK(get_map(ctx, p.kv, (uint64_t)p.kv_rows, (uint64_t)p.ld_kv, (uint64_t)p.ld_kv, KT, &mkv));
    if (a.rot_dim > 0)
        B2_CHECK(get_map(ctx, p.rot, (uint64_t)p.kv_rows, (uint64_t)blocks64(a.rot_dim) * 64, (uint64_t)blocks64(a.rot_dim) * 64, KT, &mr));
    else
        mr = mkv;  // never read
    if (dk == 1 && vd == 1) return launch<1, 1>(ctx, a, p, grid_work, mq, mkv, mr);
    if (dk == 1 && vd == 2) return launch<1, 2>(ctx, a, p, grid_work, mq, mkv, mr);
    if (dk == 2 && vd == 1) return launch<2, 1>(ctx, a, p, grid_work, mq, mkv, mr);
    if (dk == 2 && vd == 2) return launch<2, 2>(ctx, a, p, grid_work, mq, mkv, mr);
    if (dk == 3 && vd == 1) return launch<3, 1>(ctx, a, p, grid_work, mq, mkv, mr);
    if (dk == 3 && vd == 2) return launch<3, 2>(ctx, a, p, grid_work, mq, mkv, mr);
    return b2_fail(B2_ERR_UNSUPPORTED, "latent prefill: head sizes outside the kernel's tiles");
}
