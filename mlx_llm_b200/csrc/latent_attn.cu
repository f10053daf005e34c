// Attention over a shared low-rank latent (one latent vector and one rotated key part per token, shared by all heads).
//
// The keys' and values' up-projections are absorbed into the query and the output: with k_h = Wk_h c and v_h = Wv_h c,
//     q_h . k_h = (Wk_h^T q_h) . c        sum_j p_j v_hj = Wv_h (sum_j p_j c_j)
// so attention runs over the cached rows [c | rotated key] themselves, as one key/value head shared by every query head.
#include "elt.cuh"
#include "layer_kernels.h"
#include "tc5.cuh"

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
// CTA = (one chunk of one sequence's keys, up to MT * 16 heads), 16 warps, 64 keys per tile.  Tiles arrive by TMA, a box of 16
// keys x 64 values per copy located through the block table, into two 128-byte-swizzled buffers; a seventeenth warp
// issues them.  Scores: warp = 16 heads x 8 MT keys x every other 64-wide block of W; the two halves of W are added through shared
// memory, after which a warp owns 16 heads x 8 keys.  Scores and weights are f32; the weights enter the second product as
// their bf16 head plus bf16 remainder, the warps splitting the R columns (16-column tiles w, w + 16).  Keys past the chunk
// are other tokens' rows (finite) and get weight zero.  With more than one chunk a sequence's partial results (f32) are
// added in chunk order by a second kernel: one block per (sequence, head), so that long contexts spread over the machine.
constexpr int DK_KEYS = 64, DK_WARPS = 16, DK_NJ = 2;  // keys per tile; 16-column tiles per warp (R up to 512)
constexpr int kDecodeMaxRank = DK_NJ * DK_WARPS * 16;
constexpr int PS = DK_KEYS + 8;                        // row stride of the weights in shared memory
constexpr int DK_BLOCK = DK_KEYS * 128;                // 64 keys x 64 values

template <int MT>
struct DecodeSmem {
    static constexpr int H = MT * 16, kQBlock = H * 128;
    static __host__ __device__ int blocks(int W) { return (W + 63) / 64; }
    static __host__ __device__ int q_off(int W) { return 2 * blocks(W) * DK_BLOCK; }
    static __host__ __device__ int p_off(int W) { return q_off(W) + blocks(W) * kQBlock; }
    static __host__ __device__ int bytes(int W) { return p_off(W) + 2 * H * PS * 2 + DK_WARPS * 32 * 4 * 4 + (2 * 8 * H + 3 * H) * 4 + 32; }
};

// barrier of the sixteen computing warps
__device__ __forceinline__ void dk_sync() { asm volatile("bar.sync 1, %0;\n" ::"n"(DK_WARPS * 32) : "memory"); }

template <int MT>
__global__ void __launch_bounds__(DK_WARPS * 32 + 32, 1)
    latent_decode_kernel(const LatentAttnSpec a, const LatentDecodeParams p, int* err, const __grid_constant__ CUtensorMap map) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    using L = DecodeSmem<MT>;
    constexpr int H = L::H;
    extern __shared__ __align__(1024) uint8_t smem[];
    const int W = a.row_pad(), R = a.kv_rank, NB = L::blocks(W);
    const uint32_t base = smem_u32(smem);
    if (base & 1023u) {  // the swizzled layout needs this alignment; every thread sees the same value
        if (threadIdx.x == 0) atomicExch(err, 7);
        return;
    }
    const uint32_t sQ = base + L::q_off(W);
    uint16_t *ph = reinterpret_cast<uint16_t*>(smem + L::p_off(W)), *pl = ph + H * PS;
    float *xch = reinterpret_cast<float*>(pl + H * PS), *wmax = xch + DK_WARPS * 32 * 4, *wsum = wmax + 8 * H, *rowm = wsum + 8 * H, *rowl = rowm + 2 * H;
    const uint32_t full0 = smem_u32(rowl + H);
    const uint32_t sPh = smem_u32(ph), sPl = smem_u32(pl);

    const int item = blockIdx.x, h0 = blockIdx.y * H;
    int sd, chunk, part0;  // row of the list, its chunk, first partial slot of the row
    if (p.work_seq) {
        if (item >= *p.n_work) return;
        sd = p.work_seq[item];
        chunk = p.work_chunk[item];
        part0 = p.work_off[sd];
    } else {  // one work item per row
        sd = item;
        chunk = 0;
        part0 = item;
    }
    const int ctx = p.ctx ? p.ctx[sd] : p.positions[sd] + 1, qrow = p.qrow ? p.qrow[sd] : sd;
    const int slot = p.slot ? p.slot[sd] : p.seq_slot[p.token_seq[sd]];
    const int chunk_keys = p.chunk_tiles * 16;
    const int n_chunks = (ctx + chunk_keys - 1) / chunk_keys;
    if (chunk >= n_chunks) return;
    const int k_lo = chunk * chunk_keys, k_hi = min(ctx, k_lo + chunk_keys);
    const int n_tiles = (k_hi - k_lo + DK_KEYS - 1) / DK_KEYS;
    const int32_t* bt = p.block_tables + (size_t)slot * p.max_blocks;
    const uint16_t* q = reinterpret_cast<const uint16_t*>(p.q_lat) + (size_t)qrow * a.heads * W;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, lr = lane & 7;

    const uint32_t empty0 = full0 + 16;
    if (tid == 0) {
        for (int i = 0; i < 2; i++) {
            tc5::mbar_init(full0 + 8 * i, 1);
            tc5::mbar_init(empty0 + 8 * i, DK_WARPS);
        }
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (tid < H) {
        rowm[tid] = -INFINITY;
        rowl[tid] = 0.f;
    }
    __syncthreads();
    if (warp == DK_WARPS) {
        // tile j: four boxes of 16 keys per 64-value block, spread over the lanes; page rows looked up a tile ahead
        const int sub = lane & 3;
        auto row_of = [&](int j) {  // a box past the chunk repeats the chunk's first page: any finite rows will do
            const int key = k_lo + j * DK_KEYS + sub * 16, kk = key < k_hi ? key : k_lo;
            return bt[kk / p.page_size] * p.page_size + kk % p.page_size;
        };
        int next = row_of(0);
        for (int j = 0; j < n_tiles; j++) {
            const int row = next, st = j & 1;
            next = row_of(j + 1);
            if (!__all_sync(0xffffffffu, tc5::mbar_wait(empty0 + 8 * st, ((uint32_t)(j >> 1) & 1u) ^ 1u))) {
                if (lane == 0) atomicExch(err, 16);
                return;
            }
            if (lane == 0) tc5::mbar_expect_tx(full0 + 8 * st, (uint32_t)NB * DK_BLOCK);
            __syncwarp();
            for (int i = lane >> 2; i < NB; i += 8) tc5::tma_load_2d(base + (st * NB + i) * DK_BLOCK + sub * 2048, &map, i * 64, row, full0 + 8 * st);
        }
        return;
    }
    // queries: [64-value block][head][64 values], swizzled like the keys
    for (int r = warp; r < H; r += DK_WARPS) {
        const bool ok = h0 + r < a.heads;
        for (int c = lane; c < NB * 8; c += 32) {
            const bool in = ok && c * 8 < W;
            cp_async16_zfill(sQ + (c >> 3) * L::kQBlock + r * 128 + (((c & 7) ^ (r & 7)) << 4), q + (in ? (size_t)(h0 + r) * W + c * 8 : 0), in);
        }
    }
    cp_async_commit();
    cp_async_wait<0>();
    dk_sync();

    float acc[MT][DK_NJ * 2][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int n = 0; n < DK_NJ * 2; n++) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
    // scores: heads mw * 16.., keys kw * 8 MT.., blocks ks, ks + 2, ...
    const int ks = warp & 1, mw = MT == 2 ? (warp >> 1) & 1 : 0, kw = MT == 2 ? warp >> 2 : warp >> 1;
    const int own = MT == 2 ? kw * 2 + ks : kw;  // the 8 keys this warp turns into weights (MT 1: even warps only)
    const bool owner = MT == 2 || ks == 0;
    const int CT = (R + 15) / 16;
    const int row_a = mw * 16 + (lane >> 2), row_b = row_a + 8;
    const uint32_t qa = sQ + (mw * 16 + lr + (mi & 1) * 8) * 128;
    const uint32_t k_row = MT == 2 ? (uint32_t)(kw * 16 + lr + (mi >> 1) * 8) * 128 : (uint32_t)(kw * 8 + lr) * 128;
    uint32_t offa[4], offb[4];
#pragma unroll
    for (int i = 0; i < 4; i++) {
        offa[i] = (uint32_t)(((2 * i + (mi >> 1)) ^ lr) << 4);
        offb[i] = (uint32_t)(((2 * i + (mi & 1)) ^ lr) << 4);
    }
    bool alive = true;
    for (int j = 0; j < n_tiles; j++) {
        alive = alive && tc5::mbar_wait(full0 + (j & 1) * 8, (uint32_t)(j >> 1) & 1u);
        const uint32_t kb = base + (j & 1) * NB * DK_BLOCK;
        float s[MT][4];
#pragma unroll
        for (int n = 0; n < MT; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
        for (int blk = ks; blk < NB; blk += 2) {
            const uint32_t qb = qa + blk * L::kQBlock, kk = kb + k_row + blk * DK_BLOCK;
#pragma unroll
            for (int i = 0; i < 4; i++) {
                uint32_t af[4];
                ldmatrix_x4(af[0], af[1], af[2], af[3], qb + offa[i]);
                if (MT == 2) {
                    uint32_t b0[2], b1[2];
                    ldmatrix_x4(b0[0], b0[1], b1[0], b1[1], kk + offb[i]);
                    mma_bf16_16816(s[0], af, b0);
                    mma_bf16_16816(s[MT - 1], af, b1);
                } else {
                    uint32_t b0[2];
                    ldmatrix_x2(b0[0], b0[1], kk + offb[i]);
                    mma_bf16_16816(s[0], af, b0);
                }
            }
        }
        // hand over what the other half's warp owns, take what this one owns
        if (MT == 2)
            *reinterpret_cast<float4*>(xch + (warp * 32 + lane) * 4) = ks ? make_float4(s[0][0], s[0][1], s[0][2], s[0][3])
                                                                          : make_float4(s[MT - 1][0], s[MT - 1][1], s[MT - 1][2], s[MT - 1][3]);
        else if (ks)
            *reinterpret_cast<float4*>(xch + (warp * 32 + lane) * 4) = make_float4(s[0][0], s[0][1], s[0][2], s[0][3]);
        dk_sync();
        float v[4], m0 = -INFINITY, m1 = -INFINITY;
        if (owner) {
            const float4 o = *reinterpret_cast<const float4*>(xch + ((warp ^ 1) * 32 + lane) * 4);
            const float* mine = MT == 2 && ks ? s[MT - 1] : s[0];
            v[0] = mine[0] + o.x, v[1] = mine[1] + o.y, v[2] = mine[2] + o.z, v[3] = mine[3] + o.w;
            const int key = k_lo + j * DK_KEYS + own * 8 + 2 * (lane & 3);
            const bool ok0 = key < k_hi, ok1 = key + 1 < k_hi;
            v[0] = ok0 ? v[0] * p.scale_log2 : -INFINITY, v[1] = ok1 ? v[1] * p.scale_log2 : -INFINITY;
            v[2] = ok0 ? v[2] * p.scale_log2 : -INFINITY, v[3] = ok1 ? v[3] * p.scale_log2 : -INFINITY;
            m0 = fmaxf(v[0], v[1]);
            m1 = fmaxf(v[2], v[3]);
#pragma unroll
            for (int o2 = 1; o2 < 4; o2 <<= 1) {
                m0 = fmaxf(m0, __shfl_xor_sync(0xffffffffu, m0, o2));
                m1 = fmaxf(m1, __shfl_xor_sync(0xffffffffu, m1, o2));
            }
            if ((lane & 3) == 0) {
                wmax[own * H + row_a] = m0;
                wmax[own * H + row_b] = m1;
            }
        }
        dk_sync();
        // weights: the row maximum over the tile and the tiles before, then exp2 (a chunk's first key is visible)
        const float* old_m = rowm + (j & 1) * H;
        float* new_m = rowm + ((j & 1) ^ 1) * H;
        if (owner) {
            m0 = old_m[row_a];
            m1 = old_m[row_b];
#pragma unroll
            for (int w = 0; w < 8; w++) {
                m0 = fmaxf(m0, wmax[w * H + row_a]);
                m1 = fmaxf(m1, wmax[w * H + row_b]);
            }
            const float e0 = fast_exp2(v[0] - m0), e1 = fast_exp2(v[1] - m0), e2 = fast_exp2(v[2] - m1), e3 = fast_exp2(v[3] - m1);
            float l0 = e0 + e1, l1 = e2 + e3;
            const int col = own * 8 + 2 * (lane & 3);
            const uint32_t ha = pack_bf2(e0, e1), hb = pack_bf2(e2, e3);
            *reinterpret_cast<uint32_t*>(ph + row_a * PS + col) = ha;
            *reinterpret_cast<uint32_t*>(ph + row_b * PS + col) = hb;
            *reinterpret_cast<uint32_t*>(pl + row_a * PS + col) = pack_bf2(e0 - bflo(ha), e1 - bfhi(ha));
            *reinterpret_cast<uint32_t*>(pl + row_b * PS + col) = pack_bf2(e2 - bflo(hb), e3 - bfhi(hb));
#pragma unroll
            for (int o2 = 1; o2 < 4; o2 <<= 1) {
                l0 += __shfl_xor_sync(0xffffffffu, l0, o2);
                l1 += __shfl_xor_sync(0xffffffffu, l1, o2);
            }
            if ((lane & 3) == 0) {
                wsum[own * H + row_a] = l0;
                wsum[own * H + row_b] = l1;
                if (own == 0) {
                    new_m[row_a] = m0;
                    new_m[row_b] = m1;
                }
            }
        }
        dk_sync();
        // O = alpha O + P K[:, :R]
        if (tid < H) {
            float l = rowl[tid] * fast_exp2(old_m[tid] - new_m[tid]);
#pragma unroll
            for (int w = 0; w < 8; w++) l += wsum[w * H + tid];
            rowl[tid] = l;
        }
#pragma unroll
        for (int m = 0; m < MT; m++) {
            const int ra = m * 16 + (lane >> 2);
            const float a0 = fast_exp2(old_m[ra] - new_m[ra]), a1 = fast_exp2(old_m[ra + 8] - new_m[ra + 8]);
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
                const int ct = warp + c * DK_WARPS;  // values ct * 16 ..: block ct / 4, 16-byte chunks (ct % 4) * 2, + 1
                if (ct < CT) {
                    uint32_t v0[2], v1[2];
                    ldmatrix_x4_trans(v0[0], v0[1], v1[0], v1[1],
                                      kb + (ct >> 2) * DK_BLOCK + (k * 16 + lr + (mi & 1) * 8) * 128 + ((((ct & 3) * 2 + (mi >> 1)) ^ lr) << 4));
#pragma unroll
                    for (int m = 0; m < MT; m++) mma_bf16_16816(acc[m][2 * c], fh[m], v0), mma_bf16_16816(acc[m][2 * c + 1], fh[m], v1);
#pragma unroll
                    for (int m = 0; m < MT; m++) mma_bf16_16816(acc[m][2 * c], fl[m], v0), mma_bf16_16816(acc[m][2 * c + 1], fl[m], v1);
                }
            }
        }
        __syncwarp();
        if (lane == 0) tc5::mbar_arrive(empty0 + 8 * (j & 1));  // (behind the warp's last read of the tile)
        dk_sync();  // the weights and the row statistics may be overwritten
    }
    if (!alive && lane == 0) atomicExch(err, 15);
    const float* fin_m = rowm + (n_tiles & 1) * H;
    uint16_t* out = reinterpret_cast<uint16_t*>(p.o_lat) + (size_t)qrow * a.heads * p.o_pad;
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int r = m * 16 + (lane >> 2) + half * 8, h = h0 + r;
            if (h >= a.heads) continue;
            const float inv = 1.0f / rowl[r];
            uint16_t* orow = out + (size_t)h * p.o_pad;
            float* prow = p.part_o + ((size_t)(part0 + chunk) * a.heads + h) * R;
#pragma unroll
            for (int c = 0; c < DK_NJ * 2; c++) {
                const int ct = warp + (c >> 1) * DK_WARPS, col = ct * 16 + (c & 1) * 8 + 2 * (lane & 3);
                if (ct >= CT || col >= R) continue;
                const float v0 = acc[m][c][half * 2], v1 = acc[m][c][half * 2 + 1];
                if (n_chunks == 1) {  // columns up to o_pad may be written: those past R are zero weights' inputs, cleared below
                    *reinterpret_cast<uint32_t*>(orow + col) = pack_bf2(v0 * inv, col + 1 < R ? v1 * inv : 0.f);
                } else if (R % 2 == 0) {
                    *reinterpret_cast<float2*>(prow + col) = make_float2(v0, v1);
                } else {
                    prow[col] = v0;
                    if (col + 1 < R) prow[col + 1] = v1;
                }
            }
            if (n_chunks > 1 && warp == 0 && (lane & 3) == 0) {
                p.part_ml[((size_t)(part0 + chunk) * a.heads + h) * 2] = fin_m[r];
                p.part_ml[((size_t)(part0 + chunk) * a.heads + h) * 2 + 1] = rowl[r];
            }
        }
    if (R < p.o_pad && chunk == 0)  // the padding the value projection reads
        for (int r = warp; r < H && h0 + r < a.heads; r += DK_WARPS)
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
    float acc[4] = {0.f, 0.f, 0.f, 0.f}, L = 0.f;  // columns threadIdx.x + 128 i (R up to 512)
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
            for (int i = 0; i < 4; i++) {
                const int col = threadIdx.x + i * 128;
                if (col < R) acc[i] = fmaf(w[c], o[col], acc[i]);
            }
        }
    }
    const float inv = 1.0f / L;
    uint16_t* out = reinterpret_cast<uint16_t*>(p.o_lat) + ((size_t)p.qrow[sd] * a.heads + h) * p.o_pad;
#pragma unroll
    for (int i = 0; i < 4; i++) {
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
    CUtensorMap map;
    B2_CHECK(tc5::get_map(ctx, p.cache, (uint64_t)p.cache_rows, (uint64_t)a.row_pad(), (uint64_t)a.row_pad(), 16, &map));
    B2_SMEM_ONCE(ctx, latent_decode_kernel<1>, 226 * 1024);
    B2_SMEM_ONCE(ctx, latent_decode_kernel<2>, 226 * 1024);
    const int smem = a.heads > 16 ? DecodeSmem<2>::bytes(a.row_pad()) : DecodeSmem<1>::bytes(a.row_pad());
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, a.heads > 16 ? latent_decode_kernel<2> : latent_decode_kernel<1>, grid, dim3(DK_WARPS * 32 + 32), (size_t)smem, ctx->stream, a,
                          p, ctx->dev_err, map));
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
