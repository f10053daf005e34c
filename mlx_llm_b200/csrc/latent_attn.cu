// Attention over a shared low-rank latent (one latent vector and one rotated key part per token, shared by all heads).
//
// The keys' and values' up-projections are absorbed into the query and the output: with k_h = Wk_h c and v_h = Wv_h c,
//     q_h . k_h = (Wk_h^T q_h) . c        sum_j p_j v_hj = Wv_h (sum_j p_j c_j)
// so attention runs over the cached rows [c | rotated key] themselves, as one key/value head shared by every query head.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

// Block = (token, eight heads): a warp per head copies the plain part of the query and rotates the rest; the blocks of the
// first eight heads also norm the latent, rotate the shared key part and write the cache row.
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentAttnSpec a, const LatentPrepParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    __shared__ float red[33];
    const int t = blockIdx.x, R = a.kv_rank, rot = a.rot_dim, dims = a.rot.dims, half = dims / 2, W = a.row_pad();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y * 8 + warp;
    const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld;
    const float* ct = p.cos_t + (size_t)p.positions[t] * half;
    const float* st = p.sin_t + (size_t)p.positions[t] * half;
    auto turned = [&](const T* v, int d) -> float {  // element d of the rotated vector v
        const float x = Elt<T>::ld(v + d);
        if (d >= dims) return x;
        const float c = ct[d >> 1], s = st[d >> 1], o = Elt<T>::ld(v + (d ^ 1));
        return (d & 1) ? x * c + o * s : x * c - o * s;
    };
    if (h < a.heads) {
        const T* qh = row + h * (a.dim + rot);
        T* qo = reinterpret_cast<T*>(p.q) + ((size_t)t * a.heads + h) * (p.plain_pad + p.rot_pad);
        T* ql = reinterpret_cast<T*>(p.q_lat) + ((size_t)t * a.heads + h) * W + R;
        if ((a.dim + rot) % 8 == 0 && a.dim % 8 == 0) {
            for (int i = lane * 8; i < p.plain_pad; i += 256) {
                float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                if (i < a.dim) Elt<T>::ld8(qh + i, v);
                Elt<T>::st8(qo + i, v);
            }
        } else {
            for (int i = lane; i < p.plain_pad; i += 32) Elt<T>::st(qo + i, i < a.dim ? Elt<T>::ld(qh + i) : 0.f);
        }
        for (int i = lane; i < max(p.rot_pad, W - R); i += 32) {
            const float v = i < rot ? turned(qh + a.dim, i) : 0.f;
            if (i < p.rot_pad) Elt<T>::st(qo + p.plain_pad + i, v);
            if (i < W - R) Elt<T>::st(ql + i, v);
        }
    }
    if (blockIdx.y > 0) return;
    const T* lat = row + a.heads * (a.dim + rot);
    const int slot = p.slot_mapping[t];
    float ss = 0.f;
    for (int i = threadIdx.x; i < R; i += 256) {
        const float v = Elt<T>::ld(lat + i);
        ss += v * v;
    }
    ss = elt_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)R + p.eps);
    if (slot < 0) return;
    T* crow = reinterpret_cast<T*>(p.cache) + (size_t)slot * W;
    for (int i = threadIdx.x; i < W; i += 256)
        Elt<T>::st(crow + i, i < R ? Elt<T>::ld(lat + i) * inv * p.c_norm[i] : (i < R + rot ? turned(lat + R, i - R) : 0.f));
}

// Plain form: one block per (token, head), 128 keys at a time with an online softmax, everything f32.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_simple_kernel(const LatentAttnSpec a, const LatentAttnParams p) {
    pdl_wait();
    extern __shared__ float sm[];  // q [W] | acc [R] | p [128]
    __shared__ float red[33];
    const int t = p.row_idx ? p.row_idx[blockIdx.x] : blockIdx.x, h = blockIdx.y, W = a.row_pad(), R = a.kv_rank;
    float *q = sm, *acc = sm + W, *pr = acc + R;
    const int n = p.positions[t] + 1;
    const int32_t* bt = p.block_tables + (size_t)p.seq_slot[p.token_seq[t]] * p.max_blocks;
    const T* cache = reinterpret_cast<const T*>(p.cache);
    const T* qr = reinterpret_cast<const T*>(p.q_lat) + ((size_t)t * a.heads + h) * W;
    for (int i = threadIdx.x; i < W; i += 128) q[i] = Elt<T>::ld(qr + i);
    for (int i = threadIdx.x; i < R; i += 128) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    __syncthreads();
    for (int j0 = 0; j0 < n; j0 += 128) {
        const int j = j0 + threadIdx.x, cnt = min(128, n - j0);
        float s = -INFINITY;
        if (j < n) {
            const T* k = cache + ((size_t)bt[j / p.page_size] * p.page_size + j % p.page_size) * W;
            float d = 0.f;
            for (int i = 0; i < W; i += 8) {
                float v[8];
                Elt<T>::ld8(k + i, v);
#pragma unroll
                for (int e = 0; e < 8; e++) d = fmaf(q[i + e], v[e], d);
            }
            s = d * a.scale;
        }
        float mx = elt_warp_max(s);
        __syncthreads();
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])), m);
        const float alpha = expf(m - mx), e = j < n ? expf(s - mx) : 0.f;
        pr[threadIdx.x] = e;
        l = l * alpha + elt_block_sum(e, red);
        m = mx;
        for (int i = threadIdx.x; i < R; i += 128) {
            float v = acc[i] * alpha;
            for (int jj = 0; jj < cnt; jj++) {
                const int key = j0 + jj;
                v = fmaf(pr[jj], Elt<T>::ld(cache + ((size_t)bt[key / p.page_size] * p.page_size + key % p.page_size) * W + i), v);
            }
            acc[i] = v;
        }
        __syncthreads();
    }
    T* o = reinterpret_cast<T*>(p.o_lat) + ((size_t)t * a.heads + h) * p.o_pad;
    for (int i = threadIdx.x; i < p.o_pad; i += 128) Elt<T>::st(o + i, i < R ? acc[i] / l : 0.f);
}

// ---- decode: tensor cores, keys split over CTAs ---------------------------------------------------------------------
// One cached row serves every head, so the heads are the rows of the matrix products:
//   S [heads x keys] = Q [heads x W] . K^T,   O [heads x R] += P [heads x keys] . K[:, :R]
// CTA = (one chunk of one sequence's keys, up to MT * 16 heads), 8 warps, 64 keys per tile, double-buffered cp.async.
// Scores and weights are f32; the weights enter the second product as their bf16 head plus bf16 remainder.  For the
// second product the warps split the R columns (16-column tiles w, w + 8, ...).  With more than one chunk a sequence's
// partial results (f32) are added in chunk order by a second kernel: one block per (sequence, head), so that the sums of a
// long context spread over the machine.
constexpr int DK_KEYS = 64, DK_NJ = 4;  // keys per tile; 16-column tiles per warp (R up to 512)
constexpr int kDecodeMaxRank = DK_NJ * 8 * 16;
constexpr int PS = DK_KEYS + 8;         // row stride of the weights in shared memory

template <int MT>
struct DecodeSmem {
    static constexpr int H = MT * 16;
    static __host__ __device__ int qk_bytes(int W) { return (H + 2 * DK_KEYS) * (W + 8) * 2; }
    static __host__ __device__ int bytes(int W) { return qk_bytes(W) + 2 * H * PS * 2 + (8 * H * 2 + 3 * H) * 4; }
};

template <int MT>
__global__ void __launch_bounds__(256, 1) latent_decode_kernel(const LatentAttnSpec a, const LatentDecodeParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    constexpr int H = MT * 16, KW = MT == 2 ? 4 : 8, NK = 8 / KW;  // key groups of a tile, 8-key tiles per warp
    extern __shared__ __align__(16) uint8_t smem[];
    const int W = a.row_pad(), R = a.kv_rank, LD = W + 8;
    const uint32_t sQ = smem_u32(smem), sK = sQ + H * LD * 2;
    uint8_t* tail = smem + DecodeSmem<MT>::qk_bytes(W);
    uint16_t *ph = reinterpret_cast<uint16_t*>(tail), *pl = ph + H * PS;
    float *wmax = reinterpret_cast<float*>(pl + H * PS), *wsum = wmax + 8 * H, *rowm = wsum + 8 * H, *rowl = rowm + 2 * H;
    const uint32_t sPh = smem_u32(ph), sPl = smem_u32(pl);

    const int item = blockIdx.x, h0 = blockIdx.y * H;
    int sd, chunk, n_chunks, part0;  // row of the list, its chunk, chunks of the row, first partial slot of the row
    if (p.work_seq) {
        if (item >= *p.n_work) return;
        sd = p.work_seq[item];
        chunk = p.work_chunk[item];
        part0 = p.work_off[sd];
    } else {  // every row has the same number of work items
        sd = item / p.max_chunks;
        chunk = item - sd * p.max_chunks;
        part0 = sd * p.max_chunks;
    }
    const int ctx = p.ctx ? p.ctx[sd] : p.positions[sd] + 1, qrow = p.qrow ? p.qrow[sd] : sd;
    const int slot = p.slot ? p.slot[sd] : p.seq_slot[p.token_seq[sd]];
    const int chunk_keys = p.chunk_tiles * 16;
    n_chunks = (ctx + chunk_keys - 1) / chunk_keys;
    if (chunk >= n_chunks) return;
    const int k_lo = chunk * chunk_keys, k_hi = min(ctx, k_lo + chunk_keys);
    const int n_tiles = (k_hi - k_lo + DK_KEYS - 1) / DK_KEYS;
    const int32_t* bt = p.block_tables + (size_t)slot * p.max_blocks;
    const uint16_t* cache = reinterpret_cast<const uint16_t*>(p.cache);
    const uint16_t* q = reinterpret_cast<const uint16_t*>(p.q_lat) + (size_t)qrow * a.heads * W;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, lr = lane & 7;

    for (int r = warp; r < H; r += 8) {
        const bool ok = h0 + r < a.heads;
        for (int c = lane; c < W / 8; c += 32) cp_async16_zfill(sQ + (r * LD + c * 8) * 2, q + (size_t)(ok ? h0 + r : 0) * W + c * 8, ok);
    }
    // cache row of key (tile j, row warp + 8 * lane) in lanes 0-7, looked up a tile ahead; -1 past the chunk
    auto rows_of = [&](int j) {
        const int key = k_lo + j * DK_KEYS + warp + 8 * (lane & 7);
        return key < k_hi ? bt[key / p.page_size] * p.page_size + key % p.page_size : -1;
    };
    int row_next = rows_of(0);
    auto load = [&](int j) {
        const uint32_t dst = sK + (j & 1) * DK_KEYS * LD * 2;
        const int mine = row_next;
        row_next = rows_of(j + 1);
#pragma unroll
        for (int i = 0; i < DK_KEYS / 8; i++) {
            const int row = __shfl_sync(0xffffffffu, mine, i);
            const uint16_t* src = cache + (size_t)max(row, 0) * W;
            const uint32_t d = dst + (warp + 8 * i) * LD * 2;
            for (int c = lane; c < W / 8; c += 32) cp_async16_zfill(d + c * 16, src + c * 8, row >= 0);
        }
    };
    load(0);
    cp_async_commit();
    if (tid < H) {
        rowm[tid] = -INFINITY;
        rowl[tid] = 0.f;
    }
    float acc[MT][DK_NJ * 2][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int n = 0; n < DK_NJ * 2; n++) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
    const int mw = MT == 2 ? (warp & 1) : 0, kw = MT == 2 ? (warp >> 1) : warp;
    const int KS = W / 16, CT = (R + 15) / 16;
    const int row_a = mw * 16 + (lane >> 2), row_b = row_a + 8;
    for (int j = 0; j < n_tiles; j++) {
        if (j + 1 < n_tiles) load(j + 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const uint32_t kb = sK + (j & 1) * DK_KEYS * LD * 2;
        // ---- scores of this warp: 16 heads x NK * 8 keys
        float s[NK][4];
#pragma unroll
        for (int n = 0; n < NK; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
        const uint32_t qa = sQ + ((mw * 16 + lr + (mi & 1) * 8) * LD + (mi >> 1) * 8) * 2;
        if (NK == 2) {
            const uint32_t ka = kb + ((kw * 16 + lr + (mi >> 1) * 8) * LD + (mi & 1) * 8) * 2;
#pragma unroll 4
            for (int k = 0; k < KS; k++) {
                uint32_t af[4], b0[2], b1[2];
                ldmatrix_x4(af[0], af[1], af[2], af[3], qa + k * 32);
                ldmatrix_x4(b0[0], b0[1], b1[0], b1[1], ka + k * 32);
                mma_bf16_16816(s[0], af, b0);
                mma_bf16_16816(s[NK - 1], af, b1);
            }
        } else {
            const uint32_t ka = kb + ((kw * 8 + lr) * LD + (mi & 1) * 8) * 2;
#pragma unroll 4
            for (int k = 0; k < KS; k++) {
                uint32_t af[4], b0[2];
                ldmatrix_x4(af[0], af[1], af[2], af[3], qa + k * 32);
                ldmatrix_x2(b0[0], b0[1], ka + k * 32);
                mma_bf16_16816(s[0], af, b0);
            }
        }
        float m0 = -INFINITY, m1 = -INFINITY;
#pragma unroll
        for (int n = 0; n < NK; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int key = k_lo + j * DK_KEYS + kw * NK * 8 + n * 8 + 2 * (lane & 3) + (e & 1);
                s[n][e] = key < k_hi ? s[n][e] * p.scale_log2 : -INFINITY;
                if (e < 2)
                    m0 = fmaxf(m0, s[n][e]);
                else
                    m1 = fmaxf(m1, s[n][e]);
            }
#pragma unroll
        for (int o = 1; o < 4; o <<= 1) {
            m0 = fmaxf(m0, __shfl_xor_sync(0xffffffffu, m0, o));
            m1 = fmaxf(m1, __shfl_xor_sync(0xffffffffu, m1, o));
        }
        if ((lane & 3) == 0) {
            wmax[kw * H + row_a] = m0;
            wmax[kw * H + row_b] = m1;
        }
        __syncthreads();
        // ---- weights: the tile's row maximum over all warps, then exp2; the first tile always has a visible key
        const float *old_m = rowm + (j & 1) * H, *cur_m;
        float* new_m = rowm + ((j & 1) ^ 1) * H;
        m0 = old_m[row_a];
        m1 = old_m[row_b];
#pragma unroll
        for (int w = 0; w < KW; w++) {
            m0 = fmaxf(m0, wmax[w * H + row_a]);
            m1 = fmaxf(m1, wmax[w * H + row_b]);
        }
        float l0 = 0.f, l1 = 0.f;
#pragma unroll
        for (int n = 0; n < NK; n++) {
            const float e0 = exp2f(s[n][0] - m0), e1 = exp2f(s[n][1] - m0), e2 = exp2f(s[n][2] - m1), e3 = exp2f(s[n][3] - m1);
            l0 += e0 + e1;
            l1 += e2 + e3;
            const int col = kw * NK * 8 + n * 8 + 2 * (lane & 3);
            const uint32_t ha = pack_bf2(e0, e1), hb = pack_bf2(e2, e3);
            *reinterpret_cast<uint32_t*>(ph + row_a * PS + col) = ha;
            *reinterpret_cast<uint32_t*>(ph + row_b * PS + col) = hb;
            *reinterpret_cast<uint32_t*>(pl + row_a * PS + col) = pack_bf2(e0 - bflo(ha), e1 - bfhi(ha));
            *reinterpret_cast<uint32_t*>(pl + row_b * PS + col) = pack_bf2(e2 - bflo(hb), e3 - bfhi(hb));
        }
#pragma unroll
        for (int o = 1; o < 4; o <<= 1) {
            l0 += __shfl_xor_sync(0xffffffffu, l0, o);
            l1 += __shfl_xor_sync(0xffffffffu, l1, o);
        }
        if ((lane & 3) == 0) {
            wsum[kw * H + row_a] = l0;
            wsum[kw * H + row_b] = l1;
            if (kw == 0) {
                new_m[row_a] = m0;
                new_m[row_b] = m1;
            }
        }
        __syncthreads();
        // ---- O = alpha O + P K[:, :R]
        cur_m = new_m;
        if (tid < H) {
            float l = rowl[tid] * exp2f(old_m[tid] - cur_m[tid]);
#pragma unroll
            for (int w = 0; w < KW; w++) l += wsum[w * H + tid];
            rowl[tid] = l;
        }
#pragma unroll
        for (int m = 0; m < MT; m++) {
            const int ra = m * 16 + (lane >> 2);
            const float a0 = exp2f(old_m[ra] - cur_m[ra]), a1 = exp2f(old_m[ra + 8] - cur_m[ra + 8]);
            if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
                for (int n = 0; n < DK_NJ * 2; n++) acc[m][n][0] *= a0, acc[m][n][1] *= a0, acc[m][n][2] *= a1, acc[m][n][3] *= a1;
            }
        }
#pragma unroll
        for (int k = 0; k < DK_KEYS / 16; k++) {
            uint32_t fh[MT][4], fl[MT][4];
#pragma unroll
            for (int m = 0; m < MT; m++) {
                const uint32_t off = ((m * 16 + lr + (mi & 1) * 8) * PS + k * 16 + (mi >> 1) * 8) * 2;
                ldmatrix_x4(fh[m][0], fh[m][1], fh[m][2], fh[m][3], sPh + off);
                ldmatrix_x4(fl[m][0], fl[m][1], fl[m][2], fl[m][3], sPl + off);
            }
#pragma unroll
            for (int c = 0; c < DK_NJ; c++) {
                const int ct = warp + c * 8;
                if (ct < CT) {
                    uint32_t v0[2], v1[2];
                    ldmatrix_x4_trans(v0[0], v0[1], v1[0], v1[1], kb + ((k * 16 + lr + (mi & 1) * 8) * LD + ct * 16 + (mi >> 1) * 8) * 2);
#pragma unroll
                    for (int m = 0; m < MT; m++) {
                        mma_bf16_16816(acc[m][2 * c], fh[m], v0);
                        mma_bf16_16816(acc[m][2 * c + 1], fh[m], v1);
                        mma_bf16_16816(acc[m][2 * c], fl[m], v0);
                        mma_bf16_16816(acc[m][2 * c + 1], fl[m], v1);
                    }
                }
            }
        }
        __syncthreads();  // the tile's buffer, the weights and the row statistics may be overwritten
    }
    const float* fin_m = rowm + (n_tiles & 1) * H;
    uint16_t* out = reinterpret_cast<uint16_t*>(p.o_lat) + (size_t)qrow * a.heads * p.o_pad;
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int r = m * 16 + (lane >> 2) + half * 8, h = h0 + r;
            if (h >= a.heads) continue;
            const float inv = 1.0f / rowl[r];
#pragma unroll
            for (int c = 0; c < DK_NJ * 2; c++) {
                const int col = (warp + (c >> 1) * 8) * 16 + (c & 1) * 8 + 2 * (lane & 3);
                if ((warp + (c >> 1) * 8) >= CT) continue;
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    if (col + e >= R) continue;
                    const float v = acc[m][c][half * 2 + e];
                    if (n_chunks == 1)
                        out[(size_t)h * p.o_pad + col + e] = f2bf(v * inv);
                    else
                        p.part_o[((size_t)(part0 + chunk) * a.heads + h) * R + col + e] = v;
                }
            }
            if (n_chunks > 1 && warp == 0 && (lane & 3) == 0) {
                p.part_ml[((size_t)(part0 + chunk) * a.heads + h) * 2] = fin_m[r];
                p.part_ml[((size_t)(part0 + chunk) * a.heads + h) * 2 + 1] = rowl[r];
            }
        }
    if (R < p.o_pad && chunk == 0)  // the padding the value projection reads
        for (int r = warp; r < H && h0 + r < a.heads; r += 8)
            for (int col = R + lane; col < p.o_pad; col += 32) out[(size_t)(h0 + r) * p.o_pad + col] = 0;
}

constexpr int kMergeTile = 128;
// Sum of a row's chunks: out = sum_c 2^(m_c - M) O_c / sum_c 2^(m_c - M) l_c, M the largest m_c, chunks in order.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentAttnSpec a, const LatentDecodeParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int sd = blockIdx.x, h = blockIdx.y, R = a.kv_rank, chunk_keys = p.chunk_tiles * 16;
    const int n = (p.ctx[sd] + chunk_keys - 1) / chunk_keys;
    if (n <= 1) return;
    const size_t at0 = (size_t)p.work_off[sd] * a.heads + h;
    __shared__ float w[kMergeTile], sum[kMergeTile];  // maxima, then weights, of up to kMergeTile chunks; row sums
    float M = -INFINITY;
    for (int c = threadIdx.x; c < n; c += 128) M = fmaxf(M, p.part_ml[(at0 + (size_t)c * a.heads) * 2]);
    M = elt_warp_max(M);
    __shared__ float red[4];
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = M;
    __syncthreads();
    M = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    float acc[DK_NJ] = {0.f, 0.f, 0.f, 0.f}, L = 0.f;  // columns threadIdx.x + 128 i (R up to 512)
    for (int c0 = 0; c0 < n; c0 += kMergeTile) {
        const int cnt = min(kMergeTile, n - c0);
        __syncthreads();
        for (int c = threadIdx.x; c < cnt; c += 128) {
            const float2 ml = *reinterpret_cast<const float2*>(&p.part_ml[(at0 + (size_t)(c0 + c) * a.heads) * 2]);
            w[c] = exp2f(ml.x - M);
            sum[c] = ml.y;
        }
        __syncthreads();
#pragma unroll 4
        for (int c = 0; c < cnt; c++) {
            const float* o = p.part_o + (at0 + (size_t)(c0 + c) * a.heads) * R;
            L = fmaf(w[c], sum[c], L);
#pragma unroll
            for (int i = 0; i < DK_NJ; i++) {
                const int col = threadIdx.x + i * 128;
                if (col < R) acc[i] = fmaf(w[c], o[col], acc[i]);
            }
        }
    }
    const float inv = 1.0f / L;
    uint16_t* out = reinterpret_cast<uint16_t*>(p.o_lat) + ((size_t)p.qrow[sd] * a.heads + h) * p.o_pad;
#pragma unroll
    for (int i = 0; i < DK_NJ; i++) {
        const int col = threadIdx.x + i * 128;
        if (col < R) out[col] = f2bf(acc[i] * inv);
    }
}

}  // namespace

bool b2_latent_decode_eligible(const LatentAttnSpec& a) {
    return a.kv_rank <= kDecodeMaxRank && (a.heads > 16 ? DecodeSmem<2>::bytes(a.row_pad()) : DecodeSmem<1>::bytes(a.row_pad())) <= 226 * 1024;
}
int32_t b2_latent_decode_launch(b2_ctx* ctx, const LatentAttnSpec& a, const LatentDecodeParams& p, int items, int rows) {
    if (items <= 0) return B2_OK;
    const dim3 grid(items, a.heads > 16 ? (a.heads + 31) / 32 : 1);
    if (a.heads > 16) {
        B2_SMEM_ONCE(ctx, latent_decode_kernel<2>, 226 * 1024);
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, latent_decode_kernel<2>, grid, dim3(256), (size_t)DecodeSmem<2>::bytes(a.row_pad()), ctx->stream, a, p));
    } else {
        B2_SMEM_ONCE(ctx, latent_decode_kernel<1>, 226 * 1024);
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, latent_decode_kernel<1>, grid, dim3(256), (size_t)DecodeSmem<1>::bytes(a.row_pad()), ctx->stream, a, p));
    }
    B2_LAUNCHED(ctx);
    if (items > rows) {  // some row has more than one chunk
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, latent_merge_kernel, dim3(rows, a.heads), dim3(128), 0, ctx->stream, a, p));
        B2_LAUNCHED(ctx);
    }
    return B2_OK;
}

int32_t b2_latent_prep_launch(b2_ctx* ctx, bool f32, const LatentAttnSpec& a, const LatentPrepParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? latent_prep_kernel<float> : latent_prep_kernel<uint16_t>, dim3(p.T, (a.heads + 7) / 8), dim3(256), 0, ctx->stream, a, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_latent_attn_simple_launch(b2_ctx* ctx, bool f32, const LatentAttnSpec& a, const LatentAttnParams& p) {
    if (p.T <= 0) return B2_OK;
    const size_t smem = (size_t)(a.row_pad() + a.kv_rank + 128) * 4;
    B2_REQUIRE(smem <= 46 * 1024, B2_ERR_UNSUPPORTED, "latent attention: the latent is too wide");
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, f32 ? latent_attn_simple_kernel<float> : latent_attn_simple_kernel<uint16_t>, dim3(p.T, a.heads), dim3(128), smem,
                          ctx->stream, a, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
