// Grouped-query attention of the layered models, one query token per row, over the paged cache in place (bf16).
//
// Byte streaming like the flat decoders' kernel (paged_attn_decode.cu), for key and value heads of any size up to 256 (in
// 16-wide steps), any number of query heads per key head (blocks of eight), capped scores and a sink; with two maps (differential
// attention) a head's two queries are two of the eight columns, each of which meets its own map's keys:
//   CTA   (chunk of one row's keys, up to eight query heads of one key / value head)
//   warp  every 4th tile of 16 keys, its own three-stage cp.async ring, no CTA-wide barrier in the loop
//   mma   S^T = K Q^T with the keys on M and the heads on N, then O^T += V^T P^T; P enters as bf16 head and remainder
// Under a mask the tiles are those of the kept first keys, then those from the tile of the row's first visible key on, and every row
// has the same number of work items.
// Warps are merged in shared memory; the CTA of a (row, head block) that finishes last adds the chunks up, in chunk order.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

constexpr int kWarps = 4, kStages = 3, kHeads = 8, kMergeBatch = 256;
constexpr unsigned kFull = 0xffffffffu;
constexpr float kLog2e = 1.4426950408889634f;
// floats of shared memory that merging the warps, and then the chunks, takes
constexpr int fin_floats(int v_row) {
    const int merge = kWarps * v_row * 8 + 2 * kWarps * 8, chunks = 2 * kMergeBatch * 8 + 16;
    return merge > chunks ? merge : chunks;
}

// Score in units of log2: scale * s, capped as c tanh(scale * s / c) with tanh(z) = 1 - 2 / (1 + e^(2z)), whose absolute
// error (which is what a score's error counts by) stays at a few units of f32.
struct ScoreMap {
    bool cap;
    float a, c;  // no cap: s * a.  cap: c - 2 c / (1 + 2^(s * a))
    __device__ __forceinline__ explicit ScoreMap(const GroupedAttnSpec& sp) {
        cap = sp.softcap > 0.f;
        c = sp.softcap * kLog2e;
        a = cap ? 2.f * sp.scale / sp.softcap * kLog2e : sp.scale * kLog2e;
    }
    __device__ __forceinline__ float operator()(float s) const { return cap ? c - __fdividef(2.f * c, 1.f + fast_exp2(fminf(s * a, 126.f))) : s * a; }
};

// NB: 16-wide steps of the larger of the two rows (keys of all maps side by side, values), rounded up; EXACT: both have exactly that many.
template <int NB, bool EXACT, int MAPS>
__global__ void __launch_bounds__(kWarps * 32) gqa_decode_kernel(const GroupedAttnSpec a, const GqaAttnParams p, bool listed) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    extern __shared__ __align__(128) uint8_t smem[];
    __shared__ int s_last;
    pdl_wait();
    const int item = blockIdx.x, group = a.group() * MAPS, subs = (group + kHeads - 1) / kHeads, kvh = blockIdx.y / subs, h0 = kvh * group + (blockIdx.y % subs) * kHeads;
    const int QH = a.heads * MAPS, heads = min(kHeads, kvh * group + group - h0);  // heads from here on: queries, one per map
    const int MR = EXACT ? NB * 16 / MAPS : a.k_row(), KR = MR * MAPS, VR = EXACT ? NB * 16 : a.v_row();
    int row, chunk = 0, w0 = item, ctx, qrow, slot;  // entry of the list, its chunk, first work item of the row
    if (listed) {
        if (p.row_chunks > 0) {
            row = item / p.row_chunks;
            chunk = item - row * p.row_chunks;
            w0 = item - chunk;
        } else {
            if (item >= *p.n_dec_work) return;
            row = p.work_seq[item];
            chunk = p.work_chunk[item];
            w0 = p.work_off[row];
        }
        ctx = p.dec_ctx[row];
        qrow = p.dec_qrow[row];
        slot = p.dec_slot[row];
    } else {
        row = qrow = item;
        ctx = p.positions[row] + 1;
        slot = p.seq_slot[p.token_seq[row]];
    }
    const int lo = a.mask.first(ctx - 1), tile_lo = lo / 16, keep = a.mask.keep, kept = a.mask.kept_tiles(ctx - 1, 16);  // first visible key, its tile
    const int tiles_total = (ctx + 15) / 16 - tile_lo + kept, chunk_tiles = listed ? p.chunk_tiles : tiles_total, n_chunks = (tiles_total + chunk_tiles - 1) / chunk_tiles;
    if (chunk >= n_chunks) return;
    const int tile0 = chunk * chunk_tiles, n_tiles = min(chunk_tiles, tiles_total - tile0);
    auto first_key = [&](int i) { return (i < kept ? i : i - kept + tile_lo) * 16; };  // of the row's i-th tile
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int kd = KR / 16, vd = VR / 16;                              // 16-wide steps
    const int krow = (KR + 63) / 64 * 128, vrow = (VR + 63) / 64 * 128;  // bytes per row in shared memory, whole swizzle groups
    const int stage = 16 * (krow + vrow);
    const ScoreMap map(a);

    // Q^T as the B operand: thread (g, t) holds Q[head g][16 k + 2t, +1] and [.. + 8, + 9]
    uint32_t qf[NB][2];
    {
        const uint16_t* qh = reinterpret_cast<const uint16_t*>(p.q) + ((size_t)qrow * QH + h0 + min(g, heads - 1)) * MR;
#pragma unroll
        for (int k = 0; k < NB; k++) {
            const int map0 = MAPS == 2 && (g & 1) ? MR / 16 : 0;  // its map's first step
            const bool ok = g < heads && k >= map0 && k < map0 + MR / 16;
            qf[k][0] = ok ? *reinterpret_cast<const uint32_t*>(qh + (k - map0) * 16 + 2 * t) : 0u;
            qf[k][1] = ok ? *reinterpret_cast<const uint32_t*>(qh + (k - map0) * 16 + 2 * t + 8) : 0u;
        }
    }
    const int n_my = n_tiles > warp ? (n_tiles - warp + kWarps - 1) / kWarps : 0;
    const int32_t* bt = p.block_tables + (size_t)slot * p.max_blocks;
    const uint32_t wsm = smem_u32(smem) + warp * (kStages * stage);
    auto page_row = [&](int i) {  // cache row of this warp's i-th tile (page * page_size + offset) of one head; past the end: the last tile's
        const int key = first_key(tile0 + warp + min(i, max(n_my - 1, 0)) * kWarps), k = key < ctx ? key : 0;
        return make_int2(bt[k / p.page_size], k % p.page_size);
    };
    const int kr0 = lane / (MR / 8), kx0 = lane - kr0 * (MR / 8), vr0 = lane / (VR / 8), vx0 = lane - vr0 * (VR / 8);
    int2 next = page_row(0);  // looked up one tile ahead
    auto issue = [&](int i) {
        const int2 at = next;
        next = page_row(i + 1);
        const uint32_t dst = wsm + (i % kStages) * stage;
        const uint8_t* ks = reinterpret_cast<const uint8_t*>(p.k_cache) + (((size_t)at.x * a.kv_heads + kvh) * MAPS * p.page_size + at.y) * MR * 2;
        const uint8_t* vs = reinterpret_cast<const uint8_t*>(p.v_cache) + (((size_t)at.x * a.kv_heads + kvh) * p.page_size + at.y) * VR * 2;
        auto copy = [&](uint32_t to, int row_bytes, int x0, const uint8_t* from, int pieces, int r, int x) {  // 16-byte pieces of 16 rows, from piece x0 on
            const int dr = 32 / pieces, dx = 32 - dr * pieces;
            for (int c = lane; c < 16 * pieces; c += 32) {
                cp_async16(to + r * row_bytes + (((x0 + x) ^ (r & 7)) << 4), from + (size_t)c * 16);
                r += dr;
                x += dx;
                if (x >= pieces) x -= pieces, r++;
            }
        };
#pragma unroll
        for (int m = 0; m < MAPS; m++) copy(dst, krow, m * (MR / 8), ks + (size_t)m * p.page_size * MR * 2, MR / 8, kr0, kx0);
        copy(dst + 16 * krow, vrow, 0, vs, VR / 8, vr0, vx0);
    };
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f, o[NB][4];
#pragma unroll
    for (int i = 0; i < NB; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
    for (int i = 0; i < kStages - 1; i++) {
        if (i < n_my) issue(i);
        cp_async_commit();
    }
    const int mi = lane >> 3, lr = lane & 7;
    for (int i = 0; i < n_my; i++) {
        if (i + kStages - 1 < n_my) issue(i + kStages - 1);
        cp_async_commit();
        cp_async_wait<kStages - 1>();
        __syncwarp();
        const uint32_t kb = wsm + (i % kStages) * stage, vb = kb + 16 * krow;
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        {
            const int r = lr + (mi & 1) * 8;
#pragma unroll
            for (int k = 0; k < NB; k++)
                if (EXACT || k < kd) {
                    uint32_t f[4];
                    ldmatrix_x4(f[0], f[1], f[2], f[3], kb + r * krow + (((2 * k + (mi >> 1)) ^ (r & 7)) << 4));
                    mma_bf16_16816(s, f, qf[k]);
                }
        }
        const int key0 = first_key(tile0 + warp + i * kWarps);
#pragma unroll
        for (int j = 0; j < 4; j++) s[j] = map(s[j]);
        if (key0 + 16 > ctx) {
            if (key0 + g >= ctx) s[0] = s[1] = -INFINITY;
            if (key0 + g + 8 >= ctx) s[2] = s[3] = -INFINITY;
        }
        if (key0 < lo) {  // (the tile holds lo or a kept key: something stays visible)
            if (key0 + g < lo && key0 + g >= keep) s[0] = s[1] = -INFINITY;
            if (key0 + g + 8 < lo && key0 + g + 8 >= keep) s[2] = s[3] = -INFINITY;
        }
        float mx0 = fmaxf(s[0], s[2]), mx1 = fmaxf(s[1], s[3]);
#pragma unroll
        for (int sh = 4; sh <= 16; sh <<= 1) {
            mx0 = fmaxf(mx0, __shfl_xor_sync(kFull, mx0, sh));
            mx1 = fmaxf(mx1, __shfl_xor_sync(kFull, mx1, sh));
        }
        const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1), a0 = fast_exp2(m0 - mn0), a1 = fast_exp2(m1 - mn1);
        const float p0 = fast_exp2(s[0] - mn0), p1 = fast_exp2(s[1] - mn1), p2 = fast_exp2(s[2] - mn0), p3 = fast_exp2(s[3] - mn1);
        l0 = l0 * a0 + p0 + p2;
        l1 = l1 * a1 + p1 + p3;
        m0 = mn0;
        m1 = mn1;
#pragma unroll
        for (int q = 0; q < NB; q++) o[q][0] *= a0, o[q][1] *= a1, o[q][2] *= a0, o[q][3] *= a1;
        uint32_t pb[2], pl[2];
        {
            const uint32_t h01 = pack_bf2(p0, p1), h23 = pack_bf2(p2, p3);
            pb[0] = movmatrix_trans(h01);
            pb[1] = movmatrix_trans(h23);
            pl[0] = movmatrix_trans(pack_bf2(p0 - bflo(h01), p1 - bfhi(h01)));
            pl[1] = movmatrix_trans(pack_bf2(p2 - bflo(h23), p3 - bfhi(h23)));
        }
        {
            const int r = lr + (mi >> 1) * 8;
#pragma unroll
            for (int q = 0; q < NB; q++)
                if (EXACT || q < vd) {
                    uint32_t f[4];
                    ldmatrix_x4_trans(f[0], f[1], f[2], f[3], vb + r * vrow + (((2 * q + (mi & 1)) ^ (r & 7)) << 4));
                    mma_bf16_16816(o[q], f, pb);
                    mma_bf16_16816(o[q], f, pl);
                }
        }
        __syncwarp();
    }
#pragma unroll
    for (int sh = 4; sh <= 16; sh <<= 1) {
        l0 += __shfl_xor_sync(kFull, l0, sh);
        l1 += __shfl_xor_sync(kFull, l1, sh);
    }
    cp_async_wait<0>();
    __syncthreads();
    // the warps' results through shared memory (the rings are free now)
    float* so = reinterpret_cast<float*>(smem);  // [kWarps][VR][8]
    float* sm_m = so + kWarps * VR * 8;          // [kWarps][8]
    float* sm_l = sm_m + kWarps * 8;
#pragma unroll
    for (int q = 0; q < NB; q++)
        if (EXACT || q < vd) {
            float* base = so + ((size_t)warp * VR + 16 * q + g) * 8 + 2 * t;
            base[0] = o[q][0];
            base[1] = o[q][1];
            base[64] = o[q][2];  // value g + 8
            base[65] = o[q][3];
        }
    if (g == 0) {
        sm_m[warp * 8 + 2 * t] = m0;
        sm_m[warp * 8 + 2 * t + 1] = m1;
        sm_l[warp * 8 + 2 * t] = l0;
        sm_l[warp * 8 + 2 * t + 1] = l1;
    }
    __syncthreads();
    uint16_t* out = reinterpret_cast<uint16_t*>(p.out) + (size_t)qrow * p.ldo + h0 / MAPS * a.vdim;
    float* fin = reinterpret_cast<float*>(smem) + fin_floats(VR);  // [8][VR] two maps: their results
    // a head's output from its two maps: difference, norm, gate; a warp per head
    auto finish = [&]() {
        __syncthreads();
        for (int h = warp; h < heads / 2; h += kWarps) {
            const float *a1 = fin + 2 * h * VR, *a2 = a1 + VR;
            float ss = 0.f;
            for (int d = lane; d < a.vdim; d += 32) {
                const float v = a1[d] - p.lambda * a2[d];
                ss += v * v;
            }
            float f = (1.f - a.diff) / sqrtf(elt_warp_sum(ss) / (float)a.vdim + p.eps) * p.out_scale;
            if (a.head_gate) f *= sigmoid_f32(bf2f(reinterpret_cast<const uint16_t*>(p.gate)[(size_t)qrow * p.ld_gate + h0 / 2 + h]));
            for (int d = lane; d < a.vdim; d += 32) out[h * a.vdim + d] = f2bf((a1[d] - p.lambda * a2[d]) * f);
        }
    };
    for (int e = threadIdx.x; e < heads * VR; e += kWarps * 32) {
        const int h = e / VR, d = e - h * VR;
        float M = -INFINITY, L = 0.f, O = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; w++) M = fmaxf(M, sm_m[w * 8 + h]);
#pragma unroll
        for (int w = 0; w < kWarps; w++) {
            const float f = fast_exp2(sm_m[w * 8 + h] - M);
            L += sm_l[w * 8 + h] * f;
            O += so[((size_t)w * VR + d) * 8 + h] * f;
        }
        if (n_chunks == 1) {
            if (a.sink) L += fast_exp2(-M);
            if constexpr (MAPS == 2)
                fin[e] = O / L;
            else if (d < a.vdim)
                out[h * a.vdim + d] = f2bf(O / L * p.out_scale);
        } else {
            const size_t at = (size_t)item * QH + h0 + h;
            p.part_o[at * VR + d] = O;
            if (d == 0) *reinterpret_cast<float2*>(p.part_ml + at * 2) = make_float2(M, L);
        }
    }
    if (n_chunks == 1) {
        if constexpr (MAPS == 2) finish();
        return;
    }
    // No CTA waits for another; the counter returns to zero for the next launch.
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        int* counter = p.counters + (size_t)row * gridDim.y + blockIdx.y;
        s_last = atomicAdd(counter, 1) == n_chunks - 1;
        if (s_last) *counter = 0;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    // out = sum_c O_c 2^(m_c - M) / (sum_c l_c 2^(m_c - M) + sink), the sums in chunk order
    float* f_c = reinterpret_cast<float*>(smem);  // [kMergeBatch][8] maxima, then weights
    float* l_c = f_c + kMergeBatch * 8;           // [kMergeBatch][8]
    float* s_M = l_c + kMergeBatch * 8;           // [8]
    float* s_L = s_M + 8;                         // [8]
    auto ml = [&](int c, int h) { return __ldcg(reinterpret_cast<const float2*>(p.part_ml + ((size_t)(w0 + c) * QH + h0 + h) * 2)); };
    if (threadIdx.x < 32) {  // four lanes per head
        const int h = threadIdx.x >> 2;
        float M = -INFINITY;
        if (h < heads)
            for (int c = threadIdx.x & 3; c < n_chunks; c += 4) M = fmaxf(M, ml(c, h).x);
        M = fmaxf(M, __shfl_xor_sync(kFull, M, 1));
        M = fmaxf(M, __shfl_xor_sync(kFull, M, 2));
        if ((threadIdx.x & 3) == 0) {
            s_M[h] = M;
            s_L[h] = a.sink && h < heads ? fast_exp2(-M) : 0.f;
        }
    }
    constexpr int PER = kHeads * NB * 16 / (kWarps * 32);
    float acc[PER];
#pragma unroll
    for (int k = 0; k < PER; k++) acc[k] = 0.f;
    for (int c0 = 0; c0 < n_chunks; c0 += kMergeBatch) {
        const int nb = min(kMergeBatch, n_chunks - c0);
        __syncthreads();
        for (int i = threadIdx.x; i < nb * heads; i += kWarps * 32) {
            const int c = i / heads, h = i - c * heads;
            const float2 v = ml(c0 + c, h);
            f_c[c * 8 + h] = fast_exp2(v.x - s_M[h]);
            l_c[c * 8 + h] = v.y;
        }
        __syncthreads();
        if (threadIdx.x < heads) {
            float L = s_L[threadIdx.x];
            for (int c = 0; c < nb; c++) L = fmaf(l_c[c * 8 + threadIdx.x], f_c[c * 8 + threadIdx.x], L);
            s_L[threadIdx.x] = L;
        }
        for (int c = 0; c < nb; c += 8) {
#pragma unroll
            for (int k = 0; k < PER; k++) {
                const int e = threadIdx.x + k * kWarps * 32;
                if (e >= heads * VR) break;
                const int h = e / VR;
                const float* src = p.part_o + ((size_t)(w0 + c0 + c) * QH + h0) * VR + e;
                float v[8];
#pragma unroll
                for (int j = 0; j < 8; j++) v[j] = c + j < nb ? __ldcg(src + (size_t)j * QH * VR) : 0.f;
#pragma unroll
                for (int j = 0; j < 8; j++)
                    if (c + j < nb) acc[k] = fmaf(v[j], f_c[(c + j) * 8 + h], acc[k]);
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < PER; k++) {
        const int e = threadIdx.x + k * kWarps * 32;
        if (e >= heads * VR) break;
        const int h = e / VR, d = e - h * VR;
        if constexpr (MAPS == 2)
            fin[e] = acc[k] / s_L[h];
        else if (d < a.vdim)
            out[h * a.vdim + d] = f2bf(acc[k] / s_L[h] * p.out_scale);
    }
    if constexpr (MAPS == 2) finish();
}

int smem_bytes(const GroupedAttnSpec& a) {
    const int krow = (a.k_row() * a.maps + 63) / 64 * 128, vrow = (a.v_row() + 63) / 64 * 128;
    const int ring = kWarps * kStages * 16 * (krow + vrow), rest = (fin_floats(a.v_row()) + (a.maps == 2 ? 8 * a.v_row() : 0)) * 4;
    return ring > rest ? ring : rest;
}
template <int NB, bool EXACT, int MAPS = 1>
int32_t launch(b2_ctx* ctx, const GroupedAttnSpec& a, const GqaAttnParams& p, int items) {
    B2_SMEM_ONCE(ctx, (gqa_decode_kernel<NB, EXACT, MAPS>), kWarps * kStages * 16 * 2 * 512);
    const dim3 grid(items > 0 ? items : p.T, b2_gqa_head_blocks(a));
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gqa_decode_kernel<NB, EXACT, MAPS>, grid, dim3(kWarps * 32), (size_t)smem_bytes(a), ctx->stream, a, p, items > 0));
    B2_LAUNCHED(ctx);
    return B2_OK;
}

}  // namespace

bool b2_gqa_decode_eligible(const GroupedAttnSpec& a) { return a.k_row() * a.maps <= 256 && a.v_row() <= 256; }
int b2_gqa_head_blocks(const GroupedAttnSpec& a) { return a.kv_heads * ((a.group() * a.maps + kHeads - 1) / kHeads); }
int32_t b2_gqa_decode_launch(b2_ctx* ctx, const GroupedAttnSpec& a, const GqaAttnParams& p, int items) {
    if (p.T <= 0) return B2_OK;
    B2_REQUIRE(p.page_size % 16 == 0, B2_ERR_UNSUPPORTED, "grouped attention: pages of whole 16-key tiles");
    const int k_row = a.k_row() * a.maps, nb = (k_row > a.v_row() ? k_row : a.v_row()) / 16;
    if (a.maps == 2) {
        B2_REQUIRE(!a.sink, B2_ERR_UNSUPPORTED, "grouped attention: a sink beside two maps");
        if (k_row == a.v_row() && nb == 8) return launch<8, true, 2>(ctx, a, p, items);
        return nb <= 8 ? launch<8, false, 2>(ctx, a, p, items) : launch<16, false, 2>(ctx, a, p, items);
    }
    if (a.k_row() == a.v_row() && nb == 4) return launch<4, true>(ctx, a, p, items);
    if (a.k_row() == a.v_row() && nb == 8) return launch<8, true>(ctx, a, p, items);
    if (nb <= 8) return launch<8, false>(ctx, a, p, items);
    return launch<16, false>(ctx, a, p, items);
}
