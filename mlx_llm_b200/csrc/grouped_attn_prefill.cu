// Grouped-query attention of the layered models for portions of more than one token, on the 5th-generation tensor cores
// (tcgen05 + TMEM, bf16), straight from the pages.
//
// CTA = (128-query tile of one sequence's portion, one head), flash attention over 128-key tiles.  Key and value heads have
// one to three 64-wide blocks each; the load box of a head's last block reads zeros past the head's row.
//   warp 8      the Q tile, then the keys' boxes (16 keys x 64 values, a box per lane, located through the block table)
//   warp 9      the values' boxes; two stages each
//   warp 10     one thread issues tcgen05.mma: S = Q K^T into one of two TMEM buffers; O += P V with P read from TMEM as
//               the A operand (bf16 head, then bf16 remainder) and V as an MN-major operand
//   warps 0-7   softmax, thread = (query row, half of the key tile): cap, mask, maximum (shared with the row's other thread),
//               exponentials, P over the scores it came from; the running maximum is raised only when a tile exceeds it by
//               2^8; the sink enters the row sum at the end; every wait bounded
// Two maps (differential attention): a key tile is two steps, one per map, on the S buffer, the K stage and the O accumulator of that map,
// both with the same V stage; the difference, its norm and the head's gate happen on the way out.
// Under a mask the tiles are those of the kept first keys, then those from the first query's first visible key on.
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
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float capped(float s, float a, float c) { return c - __fdividef(2.f * c, 1.f + fast_exp2(fminf(s * a, 126.f))); }

// f32 accumulate, bf16 x bf16, M = 128; bit 16 set = B is MN-major
constexpr uint32_t idesc(int n, bool b_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(128 >> 4) << 24) | (b_mn ? (1u << 16) : 0u);
}

template <int DKB, int VDB, int MAPS>
struct Layout {  // shared memory of a CTA
    static constexpr int NS = 2;  // K / V stages
    static constexpr int Q = 0, K = MAPS * DKB * BLOCK_BYTES, V = K + NS * DKB * BLOCK_BYTES, BAR = V + NS * VDB * BLOCK_BYTES, X = BAR + 256;
    // maxima [2 steps in flight][2 groups][128 rows]; two maps: row sums [2 maps][2 groups][128] and sums of squares [2 groups][128]
    static constexpr int BYTES = X + (MAPS == 2 ? 5120 : 2048);
};

template <int DKB, int VDB, bool CAP, int MAPS>
__global__ void __launch_bounds__(kThreads, 1)
    gqa_prefill_kernel(const GroupedAttnSpec a, const GqaAttnParams p, int* err, const __grid_constant__ CUtensorMap map_q,
                       const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v) {
    using L = Layout<DKB, VDB, MAPS>;
    constexpr int NS = L::NS;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    pdl_wait();
    const int w = *p.n_pf_work - 1 - (int)blockIdx.x;  // the longest contexts first
    if (w < 0) return;
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
    const int head = blockIdx.y, kvh = head / a.group(), KR = a.k_row();  // (a step s = tile * MAPS + map)
    const float score_scale = CAP ? 2.f * a.scale / a.softcap * kLog2e : a.scale * kLog2e, cap = a.softcap * kLog2e;
    const int b = p.pf_seq[w], q_start = p.pf_qstart[w];
    const int tok0 = p.cu_seqlens[b], qn = p.cu_seqlens[b + 1] - tok0;
    const int ctx = p.context_lens[b], ctx_before = ctx - qn;
    const int rows = min(QT, qn - q_start);
    // tiles in the order they are taken: kept keys, then from the first query's first visible key on
    const int first_pos = ctx_before + q_start, first_tile = a.mask.first(first_pos) / KT, kept = a.mask.kept_tiles(first_pos, KT), keep = a.mask.keep;
    const int n_tiles = kept + (first_pos + rows - 1) / KT - first_tile + 1, n_steps = n_tiles * MAPS;
    auto tile_key = [&](int j) { return (j < kept ? j : j - kept + first_tile) * KT; };  // first key of the j-th

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
    // only now: a dependent product allocates tensor memory before it waits for this grid, so every CTA must have its own by then
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t tmem_o = tmem_base + 256u;
    bool alive = true;

    if (warp == kKWarp || warp == kVWarp) {
        // a box of 16 keys x 64 values per lane, found through the block table; boxes past the context repeat its first page
        const bool is_k = warp == kKWarp;
        const int blocks = is_k ? DKB : VDB, sub = lane & 7, blk = lane >> 3, ps = p.page_size, per = is_k ? MAPS : 1;  // stages per tile
        const int32_t* bt = p.block_tables + (size_t)p.seq_slot[b] * p.max_blocks;
        auto row_of = [&](int i) {
            const int j = i / per, key = tile_key(j) + sub * 16, kk = key < ctx ? key : 0;
            return ((bt[kk / ps] * a.kv_heads + kvh) * per + (i - j * per)) * ps + kk % ps;
        };
        if (is_k && lane == 0) {
            mbar_expect_tx(q_full, (uint32_t)MAPS * DKB * BLOCK_BYTES);
            for (int i = 0; i < MAPS * DKB; i++)
                tma_load_2d(base + L::Q + i * BLOCK_BYTES, &map_q, (head * MAPS + i / DKB) * KR + i % DKB * 64, tok0 + q_start, q_full);
        }
        __syncwarp();
        int st = 0, next = row_of(0);
        uint32_t par = 0;
        for (int j = 0; j < n_tiles * per; j++) {
            const int row = next;
            next = row_of(j + 1);
            const uint32_t full = is_k ? k_full(st) : v_full(st);
            if (!__all_sync(0xffffffffu, mbar_wait(is_k ? k_empty(st) : v_empty(st), par ^ 1u))) {
                alive = false;
                break;
            }
            if (lane == 0) mbar_expect_tx(full, (uint32_t)blocks * BLOCK_BYTES);
            __syncwarp();
            if (blk < blocks)
                tma_load_2d(base + (is_k ? L::K + (uint32_t)(st * DKB + blk) * BLOCK_BYTES : L::V + (uint32_t)(st * VDB + blk) * BLOCK_BYTES) + sub * 2048,
                            is_k ? &map_k : &map_v, blk * 64, row, full);
            if (++st == NS) st = 0, par ^= 1u;
        }
        if (!alive && lane == 0) atomicExch(err, 2);
        __syncwarp();
    } else if (warp == kMmaWarp) {
        if (lane == 0) {
            constexpr uint32_t kQK = idesc(128, false), kPV = idesc(VDB * 64, true);
            const uint64_t dq0 = desc_kmajor(base + L::Q), dk0 = desc_kmajor(base + L::K), dv0 = desc_mnmajor(base + L::V, BLOCK_BYTES);
            auto issue_qk = [&](int j, int kst) {  // S[j & 1] = Q K_j^T of step j
                const uint64_t dk = dk0 + (uint64_t)((uint32_t)kst * DKB * (BLOCK_BYTES >> 4));
                const uint64_t dq = MAPS == 2 ? dq0 + (uint64_t)((uint32_t)(j & 1) * DKB * (BLOCK_BYTES >> 4)) : dq0;
                const uint32_t ts = tmem_base + (uint32_t)(j & 1) * 128u;
#pragma unroll
                for (int k = 0; k < DKB * 4; k++) {
                    const uint64_t off = (uint64_t)((uint32_t)(k >> 2) * (BLOCK_BYTES >> 4) + (uint32_t)(k & 3) * 2);
                    tc_mma(ts, dq + off, dk + off, kQK, k > 0 ? 1u : 0u);
                }
                tc_commit(s_ready(j & 1));
                tc_commit(k_empty(kst));
            };
            alive = mbar_wait(q_full, 0);
            for (int j = 0; j < 2 && j < n_steps && alive; j++) {
                alive = mbar_wait(k_full(j), 0);
                if (alive) {
                    tc_fence_after();
                    issue_qk(j, j);
                }
            }
            for (int j = 0; j < n_steps && alive; j++) {  // with two stages, stage and parity follow from the step's (values: the tile's) number
                const int sb = j & 1, vt = j / MAPS, vb = vt & 1;
                const uint32_t ph = (uint32_t)(j >> 1) & 1u;
                alive = mbar_wait(v_full(vb), (uint32_t)(vt >> 1) & 1u) && mbar_wait(p_ready(sb), ph);
                if (!alive) break;
                tc_fence_after();
                const uint64_t dvs = dv0 + (uint64_t)((uint32_t)vb * VDB * (BLOCK_BYTES >> 4));
                const uint32_t tP = tmem_base + (uint32_t)sb * 128u, tO = MAPS == 2 ? tmem_o + (uint32_t)sb * (VDB * 64u) : tmem_o;
#pragma unroll
                for (int k = 0; k < KT / 16; k++) {
                    // keys 0-63 of the tile: head in columns 0-31 of the buffer, remainder in 32-63; keys 64-127: 64-95, 96-127
                    const uint32_t ta = tP + (uint32_t)(k >> 2) * 64u + (uint32_t)(k & 3) * 8u;
                    // 16 keys of a V block (128 keys x 64 values; the next 64 values are a block further)
                    const uint64_t dv = dvs + (uint64_t)((uint32_t)k * (2048u >> 4));
                    tc_mma_ts(tO, ta, dv, kPV, (vt > 0 || k > 0) ? 1u : 0u);
                    tc_mma_ts(tO, ta + 32u, dv, kPV, 1u);
                }
                tc_commit(pv_done(sb));
                if (MAPS == 1 || sb == 1) tc_commit(v_empty(vb));  // (behind the tile's last map)
                if (j + 2 < n_steps) {  // S(j+2) goes over P(j): issued after the MMAs above, which complete first
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
        const int klow = a.mask.first(kvis);  // first key it may see
        const float sc = CAP ? 1.f : score_scale;
        float m_run = -INFINITY, l_run = 0.f;  // l_run: this thread's half of the row sum
        float m_other = -INFINITY, l_other = 0.f;  // two maps: the same of the other map, whose turn the next step is
        volatile float* xb = reinterpret_cast<volatile float*>(smem_raw + L::X);  // [2 steps in flight][2 groups][128 rows]
        for (int j = 0; j < n_steps && alive; j++) {
            const int st = j & 1;
            const uint32_t s_addr = tmem_base + lane_addr + (uint32_t)st * 128u + (uint32_t)wg * 64u;
            if (!__all_sync(0xffffffffu, mbar_wait(s_ready(st), (uint32_t)(j >> 1) & 1u))) {
                alive = false;
                break;
            }
            tc_fence_after();
            const int key_base = tile_key(j / MAPS) + wg * 64;
            const bool need_mask = key_base + 63 > kvis || key_base < klow;
            // this thread's 64 scores (log2 domain, masked), their maximum, then the maximum of the whole row
            uint32_t v0[32], v1[32];
            tc_ld32_nowait(s_addr, v0);
            tc_ld32_nowait(s_addr + 32u, v1);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
            // Capped scores are mapped here: c tanh(scale s / c) in units of log2, tanh(z) = 1 - 2 / (1 + e^(2z)), whose
            // absolute error (which is what a score's error counts by) stays at a few units of f32.  Otherwise they stay raw:
            // the scale is positive, so the maximum can be taken first and scaled once, and the exponent below is one
            // fused multiply-add per score.  Masking (tiles on an edge only) writes -inf.
            if constexpr (CAP) {
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    v0[i] = __float_as_uint(capped(__uint_as_float(v0[i]), score_scale, cap));
                    v1[i] = __float_as_uint(capped(__uint_as_float(v1[i]), score_scale, cap));
                }
            }
            if (need_mask) {
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    const int k0 = key_base + i, k1 = k0 + 32;
                    if (k0 > kvis || (k0 < klow && k0 >= keep)) v0[i] = 0xff800000u;
                    if (k1 > kvis || (k1 < klow && k1 >= keep)) v1[i] = 0xff800000u;
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
            float mx = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * sc;
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
            if (j < MAPS) {
                m_run = fmaxf(mx, kNoKeyYet);
            } else if (mx > m_run + kRescaleThreshold) {
                alpha = exp2f(m_run - mx);
                m_run = mx;
                rescale = true;
            }
            if (__any_sync(0xffffffffu, rescale)) {  // this group rescales its half of the values
                // O belongs to this map's previous P V until it has completed (P V of this step cannot have been
                // issued yet: it waits for this warp's arrival below)
                if (!__all_sync(0xffffffffu, mbar_wait(pv_done((j - MAPS) & 1), (uint32_t)((j - MAPS) >> 1) & 1u))) {
                    alive = false;
                    break;
                }
                tc_fence_after();
#pragma unroll 1
                for (int c = 0; c < VDB; c++) {
                    const uint32_t o_addr = tmem_o + (MAPS == 2 ? (uint32_t)st * (VDB * 64u) : 0u) + lane_addr + (uint32_t)wg * (VDB * 32u) + (uint32_t)c * 32u;
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
            const float neg_m = -m_run;
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
            if constexpr (MAPS == 2) {
                const float m_next = m_other, l_next = l_other;
                m_other = m_run, l_other = l_run;
                m_run = m_next, l_run = l_next;
            }
        }
        // ---------------- output: O / l, each group its half of the values ----------------
        if (alive && !__all_sync(0xffffffffu, mbar_wait(pv_done((n_steps - 1) & 1), (uint32_t)((n_steps - 1) >> 1) & 1u))) alive = false;
        // the row sum is the two halves' sums (slot of the tile parity that is not in use any more)
        if (MAPS == 2 && alive) {  // (an even number of steps: `run` is the first map's again; its last P V ended ahead of the second one's)
            volatile float *xl = xb + 512, *xs = xb + 1024;  // [2 maps][2 groups][128], [2 groups][128]
            xl[wg * 128 + r] = l_run;
            xl[(2 + wg) * 128 + r] = l_other;
            __syncwarp();
            if (lane == 0) mbar_arrive(l_ready);
            alive = __all_sync(0xffffffffu, mbar_wait(l_ready, 0));
            if (alive) {
                tc_fence_after();
                const float f1 = 1.f / (l_run + xl[(wg ^ 1) * 128 + r]), f2 = p.lambda / (l_other + xl[(2 + (wg ^ 1)) * 128 + r]);
                const uint32_t o1 = tmem_o + lane_addr + (uint32_t)wg * (VDB * 32u), o2 = o1 + VDB * 64u;
                float ss = 0.f;
#pragma unroll 1
                for (int c = 0; c < VDB; c++) {  // difference of the maps, back to the first one's place
                    uint32_t v[32], u[32];
                    tc_ld32_nowait(o1 + (uint32_t)c * 32u, v);
                    tc_ld32_nowait(o2 + (uint32_t)c * 32u, u);
                    asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 32; i++) {
                        const float d = __uint_as_float(v[i]) * f1 - __uint_as_float(u[i]) * f2;
                        ss += d * d;
                        v[i] = __float_as_uint(d);
                    }
                    tc_st32(o1 + (uint32_t)c * 32u, v);
                }
                xs[wg * 128 + r] = ss;
                __syncwarp();
                if (lane == 0) mbar_arrive(l_ready);
                alive = __all_sync(0xffffffffu, mbar_wait(l_ready, 1));
                ss += xs[(wg ^ 1) * 128 + r];
                l_run = sqrtf(ss / (float)a.vdim + p.eps) / (1.f - a.diff);
            }
        } else if (alive) {
            const int slot = n_tiles & 1;
            xb[(slot * 2 + wg) * 128 + r] = l_run;
            __syncwarp();
            if (lane == 0) mbar_arrive(l_ready);
            if (!__all_sync(0xffffffffu, mbar_wait(l_ready, 0))) alive = false;
            l_run += xb[(slot * 2 + (wg ^ 1)) * 128 + r];
        }
        if (alive) {
            tc_fence_after();
            if (a.sink) l_run += fast_exp2(-m_run);
            const float gate = a.head_gate && row_ok ? sigmoid_f32(bf2f(reinterpret_cast<const uint16_t*>(p.gate)[(size_t)(tok0 + q_start + r) * p.ld_gate + head])) : 1.f;
            const float inv = gate * p.out_scale / l_run;
            const int vdim = a.vdim;
            uint16_t* dst = reinterpret_cast<uint16_t*>(p.out) + (size_t)(tok0 + q_start + (row_ok ? r : 0)) * p.ldo + (size_t)head * vdim;
            const bool vec = vdim % 8 == 0;  // rows are 16-byte aligned then (ldo is a multiple of 64)
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
                    } else if (vec && col < vdim) {
                        uint4 o4;
                        o4.x = pack_bf2(__uint_as_float(v[g * 8 + 0]) * inv, __uint_as_float(v[g * 8 + 1]) * inv);
                        o4.y = pack_bf2(__uint_as_float(v[g * 8 + 2]) * inv, __uint_as_float(v[g * 8 + 3]) * inv);
                        o4.z = pack_bf2(__uint_as_float(v[g * 8 + 4]) * inv, __uint_as_float(v[g * 8 + 5]) * inv);
                        o4.w = pack_bf2(__uint_as_float(v[g * 8 + 6]) * inv, __uint_as_float(v[g * 8 + 7]) * inv);
                        *reinterpret_cast<uint4*>(dst + col) = o4;
                    } else if (!vec) {
#pragma unroll
                        for (int i = 0; i < 8; i++)
                            if (col + i < vdim) dst[col + i] = f2bf(__uint_as_float(v[g * 8 + i]) * inv);
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

template <int DKB, int VDB, int MAPS = 1>
int32_t launch(b2_ctx* ctx, const GroupedAttnSpec& a, const GqaAttnParams& p, int grid_work, const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv) {
    constexpr int kBytes = Layout<DKB, VDB, MAPS>::BYTES;
    auto k = gqa_prefill_kernel<DKB, VDB, false, MAPS>;
    B2_SMEM_ONCE(ctx, (gqa_prefill_kernel<DKB, VDB, false, MAPS>), kBytes);
    if constexpr (MAPS == 1) {
        B2_SMEM_ONCE(ctx, (gqa_prefill_kernel<DKB, VDB, true, MAPS>), kBytes);
        if (a.softcap > 0.f) k = gqa_prefill_kernel<DKB, VDB, true, MAPS>;
    }
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, dim3(grid_work, a.heads), dim3(kThreads), (size_t)kBytes, ctx->stream, a, p, ctx->dev_err, mq, mk, mv));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int blocks64(int n) { return (n + 63) / 64; }

}  // namespace

bool b2_gqa_prefill_eligible(const GroupedAttnSpec& a) {
    const int dk = blocks64(a.k_row()), vd = blocks64(a.v_row());
    if (a.maps == 2) return dk <= 2 && vd <= 2 && a.scale > 0.f && a.softcap == 0.f && !a.sink;
    return dk <= 3 && vd <= 3 && dk + vd < 6 && (a.scale > 0.f || a.softcap > 0.f);
}
// The work list must have been built with 128-query tiles; q has at least 128 rows (a load box is never taller than its tensor).
int32_t b2_gqa_prefill_launch(b2_ctx* ctx, const GroupedAttnSpec& a, const GqaAttnParams& p, int grid_work) {
    if (grid_work <= 0) return B2_OK;
    B2_REQUIRE(p.q_rows >= QT && p.page_size % 16 == 0, B2_ERR_MSG, "grouped attention: needs 128 query rows and pages of whole 16-key boxes");
    const uint64_t rows = (uint64_t)p.max_pages * a.kv_heads * p.page_size, q_cols = (uint64_t)a.q_heads() * a.k_row();
    B2_REQUIRE(rows * a.maps < (1ull << 31), B2_ERR_UNSUPPORTED, "grouped attention: the page pool is too large");
    CUtensorMap mq, mk, mv;
    B2_CHECK(get_map(ctx, p.q, (uint64_t)p.q_rows, q_cols, q_cols, QT, &mq));
    B2_CHECK(get_map(ctx, p.k_cache, rows * a.maps, (uint64_t)a.k_row(), (uint64_t)a.k_row(), 16, &mk));
    B2_CHECK(get_map(ctx, p.v_cache, rows, (uint64_t)a.v_row(), (uint64_t)a.v_row(), 16, &mv));
    const int blocks = blocks64(a.k_row()) * 4 + blocks64(a.v_row());
    if (a.maps == 2) {
        switch (blocks) {
            case 5: return launch<1, 1, 2>(ctx, a, p, grid_work, mq, mk, mv);
            case 6: return launch<1, 2, 2>(ctx, a, p, grid_work, mq, mk, mv);
            case 9: return launch<2, 1, 2>(ctx, a, p, grid_work, mq, mk, mv);
            case 10: return launch<2, 2, 2>(ctx, a, p, grid_work, mq, mk, mv);
        }
    }
    switch (blocks) {
        case 5: return launch<1, 1>(ctx, a, p, grid_work, mq, mk, mv);
        case 6: return launch<1, 2>(ctx, a, p, grid_work, mq, mk, mv);
        case 7: return launch<1, 3>(ctx, a, p, grid_work, mq, mk, mv);
        case 9: return launch<2, 1>(ctx, a, p, grid_work, mq, mk, mv);
        case 10: return launch<2, 2>(ctx, a, p, grid_work, mq, mk, mv);
        case 11: return launch<2, 3>(ctx, a, p, grid_work, mq, mk, mv);
        case 13: return launch<3, 1>(ctx, a, p, grid_work, mq, mk, mv);
        case 14: return launch<3, 2>(ctx, a, p, grid_work, mq, mk, mv);
    }
    return b2_fail(B2_ERR_UNSUPPORTED, "grouped attention: head sizes outside the kernel's tiles");
}
