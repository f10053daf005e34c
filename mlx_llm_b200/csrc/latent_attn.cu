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
    const int n = p.positions[t] + 1, lo = a.mask.first(p.positions[t]);
    const int32_t* bt = p.block_tables + (size_t)p.seq_slot[p.token_seq[t]] * p.max_blocks;
    const T* cache = reinterpret_cast<const T*>(p.cache);
    const T* qr = reinterpret_cast<const T*>(p.q_lat) + ((size_t)t * a.heads + h) * W;
    for (int i = threadIdx.x; i < W; i += 128) q[i] = Elt<T>::ld(qr + i);
    for (int i = threadIdx.x; i < R; i += 128) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    __syncthreads();
    for (int j0 = lo; j0 < n; j0 += 128) {
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

// ---- decode: tcgen05, keys split over CTAs -----------------------------------------------------------------------------
// One cached row serves every head, so the heads are rows of one product and columns of the other:
//   S [heads x keys] = Q [heads x W] . K^T,   O^T [R x heads] += K[:, :R]^T [R x keys] . P^T [keys x heads]
// CTA = (one chunk of one sequence's keys, up to NH heads), 48 keys per tile, three tiles in shared memory (two for very wide
// rows): a tile stays from its first load to the end of its second product, and the deeper ring is what keeps loads going:
//   warp 1           TMA: boxes of 16 keys x 64 values located through the block table, 128-byte swizzle
//   warps 2, 3       one thread each issues tcgen05.mma: S, a few 64-value blocks of a tile at a time as they arrive, into one
//                    of the TMEM buffers; O^T of a tile when its P is complete, which frees its place.  The tile is the
//                    K-major B operand of the first product and, transposed, the MN-major A operand of the second;
//                    Q has fewer than the 128 rows the first product computes: the rows past NH are whatever follows in shared
//                    memory and end in TMEM lanes nobody reads
//   warps 0 4 8      softmax (these warps reach TMEM lanes 0-31): thread = (head, 16 keys); P goes to shared memory, K-major,
//                    as bf16 head and bf16 remainder (2 NH columns of the second product: an MMA costs the same at 32 and at 64)
//   warps 16-19      follow the row maxima and rescale O^T in TMEM when one rises by more than 2^8 (lazily: the division by
//                    the row sum makes the result independent of the reference point); epilogue, thread = latent value
// Scores and weights are f32.  Keys past the chunk are other tokens' rows (finite) and get weight zero.  Every wait is
// bounded.  With more than one chunk a sequence's partial results (f32) are added in chunk order by a second kernel: one block
// per (sequence, head), so that long contexts spread over the machine.
constexpr int DK_KEYS = 48, DK_BLOCK = DK_KEYS * 128;  // keys per tile; bytes of 48 keys x 64 values
constexpr int DK_SOFT = DK_KEYS / 16, DK_WALK = (DK_SOFT + 4) * 32;  // softmax warps; threads that walk the tiles together
constexpr int kDecodeMaxRank = 512, kDecodeThreads = 640, kDecodeMaxSmem = 226 * 1024;
constexpr int DK_GB = 3, DK_NG = 4;                    // 64-value blocks per arrival barrier; barriers per tile (W up to 768)
constexpr float kDecodeRescale = 8.0f;                 // log2 units

template <int NH>
struct DecodeSmem {
    static constexpr int kQBlock = NH * 128, kP = NH * 128;  // one 64-value block of Q; one operand of P
    static __host__ __device__ int blocks(int W) { return (W + 63) / 64; }
    static __host__ __device__ int q_off(int W, int ns) { return ns * blocks(W) * DK_BLOCK; }
    static __host__ __device__ int p_off(int W, int ns) { return q_off(W, ns) + blocks(W) * kQBlock; }
    // behind P (a head and a remainder per tile): barriers, maxima and sums, then room for the rows past NH of the last Q block
    static __host__ __device__ int x_off(int W, int ns) { return p_off(W, ns) + ns * 2 * kP; }
    static __host__ __device__ int bytes(int W, int ns) {
        const int used = x_off(W, ns) + 256 + 3 * DK_SOFT * 32 * 4, reach = p_off(W, ns) - kQBlock + 128 * 128;
        return used > reach ? used : reach;
    }
    static int stages(int W) { return bytes(W, 3) <= kDecodeMaxSmem ? 3 : bytes(W, 2) <= kDecodeMaxSmem ? 2 : 0; }
};

template <int NH>
__global__ void __launch_bounds__(kDecodeThreads, 1)
    latent_decode_kernel(const LatentAttnSpec a, const LatentDecodeParams p, int* err, const __grid_constant__ CUtensorMap map) {
    using namespace tc5;
    using L = DecodeSmem<NH>;
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    extern __shared__ __align__(1024) uint8_t smem[];
    const int W = a.row_pad(), R = a.kv_rank, NB = L::blocks(W), NG = (NB + DK_GB - 1) / DK_GB, MB = (R + 127) / 128, NS = p.stages;
    const uint32_t base = smem_u32(smem);
    if (base & 1023u) {  // the swizzled layouts need this alignment; every thread sees the same value
        if (threadIdx.x == 0) atomicExch(err, 7);
        return;
    }
    const uint32_t sQ = base + L::q_off(W, NS), sP = base + L::p_off(W, NS), bar = base + L::x_off(W, NS);
    auto empty = [&](int s) { return bar + 8u * s; };
    auto s_ready = [&](int s) { return bar + 8u * (3 + s); };
    auto p_ready = [&](int s) { return bar + 8u * (6 + s); };
    auto pv_done = [&](int s) { return bar + 8u * (9 + s); };
    auto o_ready = [&](int s) { return bar + 8u * (12 + s); };
    const uint32_t slot_addr = bar + 8u * 15;
    auto full = [&](int s, int g) { return bar + 8u * (16 + s * DK_NG + g); };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + L::x_off(W, NS) + 8 * 15);
    float* xm = reinterpret_cast<float*>(smem + L::x_off(W, NS) + 256);  // [2 tiles][softmax warps][32 heads] maxima
    float* xl = xm + 2 * DK_SOFT * 32;                                   // [softmax warps][32 heads] row sums

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int i = 0; i < NS; i++) {
            for (int g = 0; g < DK_NG; g++) mbar_init(full(i, g), 1);
            mbar_init(empty(i), 1);
            mbar_init(s_ready(i), 1);
            mbar_init(p_ready(i), DK_SOFT);
            mbar_init(pv_done(i), 1);
            mbar_init(o_ready(i), 4);
        }
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    pdl_wait();  // (the barriers above may be set up while earlier kernels finish)
    const int item = blockIdx.x, h0 = blockIdx.y * NH;
    int sd, chunk, part0;  // row of the list, its chunk, first partial slot of the row
    if (p.row_chunks > 0) {
        sd = item / p.row_chunks;
        chunk = item - sd * p.row_chunks;
        part0 = item - chunk;
    } else if (p.work_seq) {
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
    const int k_first = a.mask.first(ctx - 1), k_base = k_first / 16 * 16;  // first visible key, its box: the chunks start there
    const int n_chunks = (ctx - k_base + chunk_keys - 1) / chunk_keys;
    if (chunk >= n_chunks) return;
    const int k_lo = k_base + chunk * chunk_keys, k_hi = min(ctx, k_lo + chunk_keys);
    const int n_tiles = (k_hi - k_lo + DK_KEYS - 1) / DK_KEYS;

    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(slot_addr), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    {  // queries: [64-value block][head][64 values], swizzled like the keys
        const uint16_t* q = reinterpret_cast<const uint16_t*>(p.q_lat) + (size_t)qrow * a.heads * W;
        for (int r = warp; r < NH; r += kDecodeThreads / 32) {
            const bool ok = h0 + r < a.heads;
            for (int c = lane; c < NB * 8; c += 32) {
                const bool in = ok && c * 8 < W;
                cp_async16_zfill(sQ + (c >> 3) * L::kQBlock + r * 128 + (((c & 7) ^ (r & 7)) << 4), q + (in ? (size_t)(h0 + r) * W + c * 8 : 0), in);
            }
        }
        cp_async_commit();
        cp_async_wait<0>();
        fence_proxy_async();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot, tmem_o = tmem + 192u;
    bool alive = true;

    if (warp == 1) {
        const int32_t* bt = p.block_tables + (size_t)slot * p.max_blocks;
        const int sub = lane % DK_SOFT, first = lane / DK_SOFT;
        auto row_of = [&](int j) {  // a box past the chunk repeats the chunk's first page: any finite rows will do
            const int key = k_lo + j * DK_KEYS + sub * 16, kk = key < k_hi ? key : k_lo;
            return bt[kk / p.page_size] * p.page_size + kk % p.page_size;
        };
        int next = row_of(0), st = 0;
        uint32_t ph = 0;
        for (int j = 0; j < n_tiles; j++) {
            const int row = next;
            next = row_of(j + 1);
            if (!__all_sync(0xffffffffu, mbar_wait(empty(st), ph ^ 1u))) {
                if (lane == 0) atomicExch(err, 16);
                break;
            }
            if (lane < NG) mbar_expect_tx(full(st, lane), (uint32_t)min(DK_GB, NB - lane * DK_GB) * DK_BLOCK);
            __syncwarp();
            if (first < 32 / DK_SOFT)
                for (int i = first; i < NB; i += 32 / DK_SOFT) tma_load_2d(base + (st * NB + i) * DK_BLOCK + sub * 2048, &map, i * 64, row, full(st, i / DK_GB));
            if (++st == NS) st = 0, ph ^= 1u;
        }
        __syncwarp();
    } else if (warp == 2) {
        if (lane == 0) {
            constexpr uint32_t kQK = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(DK_KEYS >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
            int st = 0;
            uint32_t ph = 0;
            for (int j = 0; j < n_tiles && alive; j++) {
                for (int g = 0; g < NG; g++) {
                    alive = mbar_wait(full(st, g), ph);
                    if (!alive) break;
                    tc_fence_after();
                    for (int b = g * DK_GB; b < min(NB, (g + 1) * DK_GB); b++) {
                        const uint64_t dq = desc_kmajor(sQ + b * L::kQBlock), dk = desc_kmajor(base + (st * NB + b) * DK_BLOCK);
#pragma unroll
                        for (int i = 0; i < 4; i++) tc_mma(tmem + (uint32_t)st * 64u, dq + 2 * i, dk + 2 * i, kQK, (b > 0 || i > 0) ? 1u : 0u);
                    }
                }
                if (alive) tc_commit(s_ready(st));
                if (++st == NS) st = 0, ph ^= 1u;
            }
            if (!alive) atomicExch(err, 17);
        }
        __syncwarp();
    } else if (warp == 3) {
        if (lane == 0) {
            constexpr uint32_t kPV = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 15) | ((uint32_t)(2 * NH >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
            int st = 0;
            uint32_t ph = 0;
            for (int j = 0; j < n_tiles && alive; j++) {
                // (P exists, so S of this tile has been computed: its stage may be freed when these products are done)
                alive = mbar_wait(p_ready(st), ph) && mbar_wait(o_ready(st), ph);
                if (!alive) break;
                tc_fence_after();
                const uint64_t dp = desc_kmajor(sP + st * 2 * L::kP);
                for (int m = 0; m < MB; m++) {
                    // 128 latent values = two 64-wide blocks DK_BLOCK apart (LBO); 16 keys per step, 2 KB further each
                    const uint64_t dv = desc_mnmajor(base + (st * NB + 2 * m) * DK_BLOCK, DK_BLOCK);
#pragma unroll
                    for (int k = 0; k < DK_KEYS / 16; k++)
                        tc_mma(tmem_o + (uint32_t)(m * 2 * NH), dv + (uint64_t)(k * (2048 >> 4)), dp + 2 * k, kPV, (j > 0 || k > 0) ? 1u : 0u);
                }
                tc_commit(pv_done(st));
                tc_commit(empty(st));
                if (++st == NS) st = 0, ph ^= 1u;
            }
            if (!alive) atomicExch(err, 18);
        }
        __syncwarp();
    } else if (warp >= 16 || ((warp & 3) == 0 && warp < 4 * DK_SOFT)) {
        // softmax warps and O^T warps walk the tiles together: one barrier per tile, behind the tile's row maxima
        const bool soft = warp < 16;
        const int q = warp >> 2;  // softmax: keys q * 16 .. of the tile
        const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
        const bool real = lane < NH && h0 + lane < a.heads;
        float m_run = -INFINITY, l = 0.f;
        int st = 0, prev = 0;  // stage of this tile, of the one before
        uint32_t ph = 0, prev_ph = 0;
        for (int j = 0; j < n_tiles; j++) {
            float* mx = xm + (j & 1) * DK_SOFT * 32;
            uint32_t v[16];
            if (soft) {
                alive = __all_sync(0xffffffffu, alive && mbar_wait(s_ready(st), ph));
                tc_fence_after();
                tc_ld16(tmem + (uint32_t)st * 64u + (uint32_t)q * 16u, v);
                const int key0 = k_lo + j * DK_KEYS + q * 16;
                float m = -INFINITY;
#pragma unroll
                for (int i = 0; i < 16; i++) {
                    const float s = !real ? 0.f : key0 + i < k_hi && key0 + i >= k_first ? __uint_as_float(v[i]) * p.scale_log2 : -INFINITY;
                    v[i] = __float_as_uint(s);
                    m = fmaxf(m, s);
                }
                mx[q * 32 + lane] = m;
            }
            asm volatile("bar.sync 1, %0;\n" ::"n"(DK_WALK) : "memory");
            // every warp follows the reference points by itself (lane = head), from the same numbers
            float m = mx[lane];
#pragma unroll
            for (int w = 1; w < DK_SOFT; w++) m = fmaxf(m, mx[w * 32 + lane]);
            float alpha = 1.f;
            if (j == 0) {
                m_run = m;  // a chunk's first box has a visible key
            } else if (m > m_run + kDecodeRescale) {
                alpha = fast_exp2(m_run - m);
                m_run = m;
            }
            if (soft) {
                l *= alpha;
                uint32_t hi[8], lo[8];
#pragma unroll
                for (int i = 0; i < 8; i++) {
                    const float e0 = fast_exp2(__uint_as_float(v[2 * i]) - m_run), e1 = fast_exp2(__uint_as_float(v[2 * i + 1]) - m_run);
                    l += e0 + e1;
                    hi[i] = pack_bf2(e0, e1);
                    lo[i] = pack_bf2(e0 - bflo(hi[i]), e1 - bfhi(hi[i]));
                }
                if (lane < NH) {
                    uint8_t* dst = smem + L::p_off(W, NS) + st * 2 * L::kP + lane * 128;
#pragma unroll
                    for (int i = 0; i < 2; i++) {
                        const int at = ((2 * q + i) ^ (lane & 7)) << 4;
                        *reinterpret_cast<uint4*>(dst + at) = make_uint4(hi[4 * i], hi[4 * i + 1], hi[4 * i + 2], hi[4 * i + 3]);
                        *reinterpret_cast<uint4*>(dst + L::kP + at) = make_uint4(lo[4 * i], lo[4 * i + 1], lo[4 * i + 2], lo[4 * i + 3]);
                    }
                }
                fence_proxy_async();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(p_ready(st));
            } else {
                if (__any_sync(0xffffffffu, alpha != 1.f)) {
                    // P V of the tile before must be complete (that of the tile before it is: its stage has been loaded again)
                    alive = __all_sync(0xffffffffu, alive && mbar_wait(pv_done(prev), prev_ph));
                    tc_fence_after();
                    for (int c = 0; c < MB * 2 * NH; c += 16) {
                        uint32_t o[16];
                        tc_ld16(tmem_o + lane_addr + (uint32_t)c, o);
#pragma unroll
                        for (int i = 0; i < 16; i++) o[i] = __float_as_uint(__uint_as_float(o[i]) * __shfl_sync(0xffffffffu, alpha, (c + i) % NH));
                        tc_st16(tmem_o + lane_addr + (uint32_t)c, o);
                    }
                }
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(o_ready(st));
            }
            prev = st, prev_ph = ph;
            if (++st == NS) st = 0, ph ^= 1u;
        }
        if (soft) xl[q * 32 + lane] = l;
        asm volatile("bar.sync 1, %0;\n" ::"n"(DK_WALK) : "memory");
        if (!soft) {
            alive = __all_sync(0xffffffffu, alive && mbar_wait(pv_done(prev), prev_ph));
            tc_fence_after();
            l = xl[lane];
#pragma unroll
            for (int w = 1; w < DK_SOFT; w++) l += xl[w * 32 + lane];
            const float inv = 1.0f / l;
            uint16_t* out = reinterpret_cast<uint16_t*>(p.o_lat) + ((size_t)qrow * a.heads + h0) * p.o_pad;
            const size_t slot0 = (size_t)(part0 + chunk) * a.heads + h0;
            const int heads = min(NH, a.heads - h0);
            for (int m = 0; m < MB; m++) {
                const int d = m * 128 + (warp & 3) * 32 + lane;  // this thread's latent value
#pragma unroll
                for (int c = 0; c < NH; c += 16) {
                    uint32_t o[16], o_lo[16];
                    tc_ld16(tmem_o + lane_addr + (uint32_t)(m * 2 * NH + c), o);
                    tc_ld16(tmem_o + lane_addr + (uint32_t)(m * 2 * NH + NH + c), o_lo);
#pragma unroll
                    for (int i = 0; i < 16; i++) {
                        const float w = __shfl_sync(0xffffffffu, inv, c + i);
                        o[i] = __float_as_uint(__uint_as_float(o[i]) + __uint_as_float(o_lo[i]));
                        if (c + i < heads && d < R) {
                            if (n_chunks == 1)
                                out[(size_t)(c + i) * p.o_pad + d] = f2bf(__uint_as_float(o[i]) * w);
                            else
                                p.part_o[(slot0 + c + i) * R + d] = __uint_as_float(o[i]);
                        }
                    }
                }
            }
            if (n_chunks > 1 && warp == 16 && lane < heads) {
                p.part_ml[(slot0 + lane) * 2] = m_run;
                p.part_ml[(slot0 + lane) * 2 + 1] = l;
            }
            if (R < p.o_pad && chunk == 0)  // the padding the value projection reads
                for (int r = warp & 3; r < heads; r += 4)
                    for (int col = R + lane; col < p.o_pad; col += 32) out[(size_t)r * p.o_pad + col] = 0;
        }
        if (!alive && lane == 0) atomicExch(err, 15);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 2) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(512) : "memory");
}

constexpr int kMergeTile = 128;
// Sum of a row's chunks: out = sum_c 2^(m_c - M) O_c / sum_c 2^(m_c - M) l_c, M the largest m_c, chunks in order.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentAttnSpec a, const LatentDecodeParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const int sd = blockIdx.x, h = blockIdx.y, R = a.kv_rank, chunk_keys = p.chunk_tiles * 16;
    const int n = (p.ctx[sd] - a.mask.first(p.ctx[sd] - 1) / 16 * 16 + chunk_keys - 1) / chunk_keys;
    if (n <= 1) return;
    const size_t at0 = (size_t)(p.row_chunks > 0 ? sd * p.row_chunks : p.work_off[sd]) * a.heads + h;
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
#pragma unroll 8
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

static int decode_stages(const LatentAttnSpec& a) { return a.heads > 16 ? DecodeSmem<32>::stages(a.row_pad()) : DecodeSmem<16>::stages(a.row_pad()); }
int b2_latent_decode_tile() { return DK_KEYS; }
bool b2_latent_decode_eligible(const LatentAttnSpec& a) {
    return a.kv_rank <= kDecodeMaxRank && a.row_pad() <= DK_NG * DK_GB * 64 && decode_stages(a) > 0;
}
int32_t b2_latent_decode_launch(b2_ctx* ctx, const LatentAttnSpec& a, LatentDecodeParams p, int items, int rows) {
    if (items <= 0) return B2_OK;
    p.stages = decode_stages(a);
    const dim3 grid(items, a.heads > 16 ? (a.heads + 31) / 32 : 1);
    CUtensorMap map;
    B2_CHECK(tc5::get_map(ctx, p.cache, (uint64_t)p.cache_rows, (uint64_t)a.row_pad(), (uint64_t)a.row_pad(), 16, &map));
    B2_SMEM_ONCE(ctx, latent_decode_kernel<16>, kDecodeMaxSmem);
    B2_SMEM_ONCE(ctx, latent_decode_kernel<32>, kDecodeMaxSmem);
    const int smem = a.heads > 16 ? DecodeSmem<32>::bytes(a.row_pad(), p.stages) : DecodeSmem<16>::bytes(a.row_pad(), p.stages);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, a.heads > 16 ? latent_decode_kernel<32> : latent_decode_kernel<16>, grid, dim3(kDecodeThreads), (size_t)smem, ctx->stream, a,
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
