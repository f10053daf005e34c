// One matrix product per group: out_g[r, n] = sum_k x_g[r, k] * w_g[n, k].
//
// Two uses: the experts of a routed feed-forward (groups own consecutive runs of sorted rows, given by a device-side
// offset table) and per-head projections (every group has the same rows, at a column offset of x and out).
//
// Three kernels: tcgen05 with TMA operands when the groups have rows enough and their rows are consecutive, an mma.sync tile
// kernel with a deep cp.async ring otherwise (16-row tiles stream the weights of small groups), CUDA cores in f32.
#include "layer_kernels.h"
#include "tc5.cuh"

namespace {

constexpr int BN = 64, BK = 64, kThreads = 128;

// Work item -> (group, first row, rows).  With an offset table the row tiles of all groups are numbered one after the
// other; `tile` beyond the last one yields rows = 0.
template <int BM>
__device__ __forceinline__ void find_tile(const GroupedGemmParams& p, int tile, int& g, int& r0, int& rows) {
    if (!p.offsets) {
        const int per = (p.M + BM - 1) / BM;
        g = tile / per;
        r0 = (tile - g * per) * BM;
        rows = min(BM, p.M - r0);
        return;
    }
    g = 0, r0 = 0, rows = 0;
    int left = tile;
    for (int i = 0; i < p.G; i++) {
        const int a = p.offsets[i], n = p.offsets[i + 1] - a, tiles = (n + BM - 1) / BM;
        if (left < tiles) {
            g = i;
            r0 = a + left * BM;
            rows = min(BM, a + n - r0);
            return;
        }
        left -= tiles;
    }
}

// bf16 tile kernel: BM rows x 64 outputs, 4 warps, mma.sync with f32 accumulation, cp.async ring of ST stages.
template <int BM, int ST, bool F32OUT>
__global__ void __launch_bounds__(kThreads) grouped_tile_kernel(const GroupedGemmParams p) {
    constexpr int MT = BM / 16;  // each warp: all BM rows x 16 outputs
    constexpr int A_BYTES = BM * BK * 2, B_BYTES = BN * BK * 2;
    extern __shared__ __align__(128) uint8_t smem[];
    const uint32_t sA = smem_u32(smem), sB = sA + ST * A_BYTES;
    pdl_wait();
    int g, r0, rows;
    find_tile<BM>(p, blockIdx.y, g, r0, rows);
    if (rows <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, n0 = blockIdx.x * BN;
    const bool tail = p.tail_n > 0 && g == p.G - 1;
    if (tail && n0 >= p.tail_n) return;
    const int n_out = tail ? p.tail_n : p.n_out;
    const uint16_t* x = reinterpret_cast<const uint16_t*>(p.x) + (size_t)g * p.x_gstride;
    const uint16_t* w = reinterpret_cast<const uint16_t*>(p.w) + (size_t)g * p.N * p.K;
    float acc[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < 2; j++) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
    auto load = [&](int kt, int st) {
        for (int c = tid; c < BM * 8; c += kThreads) {
            const int r = c >> 3, cc = c & 7;
            const bool ok = r < rows;
            const int row = r0 + (ok ? r : 0);
            const int src = p.row_idx ? p.row_idx[row] : row;
            cp_async16_zfill(sA + st * A_BYTES + r * 128 + ((cc ^ (r & 7)) << 4), x + (size_t)src * p.ldx + kt * BK + cc * 8, ok);
        }
#pragma unroll
        for (int c = tid; c < BN * 8; c += kThreads) {
            const int r = c >> 3, cc = c & 7;
            cp_async16(sB + st * B_BYTES + r * 128 + ((cc ^ (r & 7)) << 4), w + (size_t)(n0 + r) * p.K + kt * BK + cc * 8);
        }
    };
    const int KT = p.K / BK, mi = lane >> 3, lr = lane & 7;
#pragma unroll
    for (int i = 0; i < ST - 1; i++) {
        if (i < KT) load(i, i);
        cp_async_commit();
    }
    int st = 0;
    for (int kt = 0; kt < KT; kt++) {
        cp_async_wait<ST - 2>();
        __syncthreads();  // slab kt has arrived, and the stage of slab kt - 1 is free
        if (kt + ST - 1 < KT) load(kt + ST - 1, st == 0 ? ST - 1 : st - 1);
        cp_async_commit();
        const uint32_t a_base = sA + st * A_BYTES, b_base = sB + st * B_BYTES;
        if (++st == ST) st = 0;
#pragma unroll
        for (int ks = 0; ks < BK / 16; ks++) {
            uint32_t bf[2][2];
            {
                const int r = warp * 16 + lr + (mi >> 1) * 8, ch = 2 * ks + (mi & 1);
                ldmatrix_x4(bf[0][0], bf[0][1], bf[1][0], bf[1][1], b_base + r * 128 + ((ch ^ (r & 7)) << 4));
            }
#pragma unroll
            for (int mt = 0; mt < MT; mt++) {
                const int r = mt * 16 + lr + (mi & 1) * 8, ch = 2 * ks + (mi >> 1);
                uint32_t af[4];
                ldmatrix_x4(af[0], af[1], af[2], af[3], a_base + r * 128 + ((ch ^ (r & 7)) << 4));
                mma_bf16_16816(acc[mt][0], af, bf[0]);
                mma_bf16_16816(acc[mt][1], af, bf[1]);
            }
        }
    }
#pragma unroll
    for (int mt = 0; mt < MT; mt++)
#pragma unroll
        for (int nt = 0; nt < 2; nt++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = mt * 16 + (lane >> 2) + (e >> 1) * 8, n = n0 + warp * 16 + nt * 8 + 2 * (lane & 3) + (e & 1);
                if (r >= rows || n >= n_out) continue;
                const int orow = p.map_out ? p.row_idx[r0 + r] : r0 + r;
                if (tail) {
                    p.tail_out[(size_t)orow * p.tail_n + n] = acc[mt][nt][e];
                    continue;
                }
                const size_t o = (size_t)g * p.out_gstride + (size_t)orow * p.ldo + n;
                if (F32OUT)
                    reinterpret_cast<float*>(p.out)[o] = acc[mt][nt][e];
                else
                    reinterpret_cast<uint16_t*>(p.out)[o] = f2bf(acc[mt][nt][e]);
            }
}

// f32: 8 rows x 32 outputs per block, partial sums per 32 inputs
__global__ void __launch_bounds__(256) grouped_f32_kernel(const GroupedGemmParams p) {
    __shared__ float xs[8][33], ws[32][33];
    pdl_wait();
    int g, r0, rows;
    find_tile<8>(p, blockIdx.y, g, r0, rows);
    if (rows <= 0) return;
    const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5, n0 = blockIdx.x * 32;
    const float* x = reinterpret_cast<const float*>(p.x) + (size_t)g * p.x_gstride;
    const float* w = reinterpret_cast<const float*>(p.w) + (size_t)g * p.N * p.K;
    const int row = r0 + (ty < rows ? ty : 0), src = p.row_idx ? p.row_idx[row] : row;
    float acc = 0.f;
    for (int k0 = 0; k0 < p.K; k0 += 32) {  // K and N are multiples of 64
        xs[ty][tx] = x[(size_t)src * p.ldx + k0 + tx];
#pragma unroll
        for (int i = 0; i < 4; i++) ws[ty * 4 + i][tx] = w[(size_t)(n0 + ty * 4 + i) * p.K + k0 + tx];
        __syncthreads();
        float part = 0.f;
#pragma unroll
        for (int d = 0; d < 32; d++) part = fmaf(xs[ty][d], ws[tx][d], part);
        acc += part;
        __syncthreads();
    }
    if (ty < rows && n0 + tx < p.n_out) reinterpret_cast<float*>(p.out)[(size_t)g * p.out_gstride + (size_t)(p.map_out ? src : r0 + ty) * p.ldo + n0 + tx] = acc;
}

// upper bound of the number of row tiles (what the grid must cover)
int tile_bound(const GroupedGemmParams& p, int bm) {
    if (!p.offsets) return p.G * ((p.M + bm - 1) / bm);
    return (p.M + bm - 1) / bm + (p.M < p.G ? p.M : p.G);
}

template <int BM, int ST>
int32_t launch_tile(b2_ctx* ctx, const GroupedGemmParams& p) {
    constexpr int smem = ST * (BM + BN) * BK * 2;
    const dim3 grid(p.N / BN, tile_bound(p, BM));
    auto k = p.out_f32 ? grouped_tile_kernel<BM, ST, true> : grouped_tile_kernel<BM, ST, false>;
    B2_SMEM_ONCE(ctx, (grouped_tile_kernel<BM, ST, true>), smem);
    B2_SMEM_ONCE(ctx, (grouped_tile_kernel<BM, ST, false>), smem);
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, k, grid, dim3(kThreads), (size_t)smem, ctx->stream, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}

// ---- tcgen05: 128 rows x 256 outputs per tile, persistent CTAs -----------------------------------------------------
//   warp 0   one thread: TMA loads of 64-wide K slabs (128 rows of x, 256 rows of w), ring of four stages
//   warp 1   one thread: tcgen05.mma (M 128, N 256) into one of two accumulators (all 512 TMEM columns)
//   warps 4-7  epilogue of the tile before: thread = row; overlaps the next tile's products
// Tiles of a group are numbered with the row tile fastest, so that CTAs next to one another share the weights.  Rows past a
// group's last one belong to the next group (or to nobody) and are not stored.  Every wait is bounded.
constexpr int TC_M = 128, TC_N = 256, TC_ST = 4, TC_G = 1024;
constexpr int TC_A = TC_M * 128, TC_B = TC_N * 128, TC_STAGE = TC_A + TC_B;
constexpr int TC_BAR = TC_ST * TC_STAGE, TC_PREFIX = TC_BAR + 256, TC_SMEM = TC_PREFIX + (TC_G + 1) * 4;

struct TcTile {
    int g, r0, rows, n0;
};
__device__ __forceinline__ TcTile tc_tile(const GroupedGemmParams& p, const int* prefix, int nt, int tile) {
    int lo = 0, hi = p.G - 1;  // the group whose tiles (prefix x column tiles) contain this one
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (prefix[mid] * nt <= tile)
            lo = mid;
        else
            hi = mid - 1;
    }
    TcTile t;
    t.g = lo;
    const int in = tile - prefix[lo] * nt, mt = prefix[lo + 1] - prefix[lo];
    t.n0 = (in / mt) * TC_N;
    const int m = in - (in / mt) * mt;
    const int a = p.offsets ? p.offsets[lo] : 0, cnt = p.offsets ? p.offsets[lo + 1] - a : p.M;
    t.r0 = a + m * TC_M;
    t.rows = min(TC_M, cnt - m * TC_M);
    return t;
}

template <bool F32OUT>
__global__ void __launch_bounds__(256, 1)
    grouped_tc_kernel(const GroupedGemmParams p, int* err, const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w) {
    using namespace tc5;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const uint32_t base = smem_u32(smem_raw);
    if (base & 1023u) {
        if (threadIdx.x == 0) atomicExch(err, 7);
        return;
    }
    const uint32_t bar = base + TC_BAR;
    auto full = [&](int s) { return bar + 8u * s; };
    auto empty = [&](int s) { return bar + 8u * (TC_ST + s); };
    auto acc_full = [&](int a) { return bar + 8u * (2 * TC_ST + a); };
    auto acc_empty = [&](int a) { return bar + 8u * (2 * TC_ST + 2 + a); };
    const uint32_t slot_addr = bar + 8u * (2 * TC_ST + 4);
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem_raw + TC_BAR + 8 * (2 * TC_ST + 4));
    int* prefix = reinterpret_cast<int*>(smem_raw + TC_PREFIX);  // row tiles of the groups before each one
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int s = 0; s < TC_ST; s++) {
            mbar_init(full(s), 1);
            mbar_init(empty(s), 1);
        }
        for (int a = 0; a < 2; a++) {
            mbar_init(acc_full(a), 1);
            mbar_init(acc_empty(a), 4);
        }
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(slot_addr), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    if (warp == 3) {
        int run = 0;
        for (int g0 = 0; g0 < p.G; g0 += 32) {
            const int g = g0 + lane;
            const int cnt = g < p.G ? (p.offsets ? p.offsets[g + 1] - p.offsets[g] : p.M) : 0;
            int incl = (cnt + TC_M - 1) / TC_M;
            const int own = incl;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int u = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += u;
            }
            if (g < p.G) prefix[g] = run + incl - own;
            run += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (lane == 0) prefix[p.G] = run;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const int nt = (p.N + TC_N - 1) / TC_N, KT = p.K / 64, total = prefix[p.G] * nt;
    bool alive = true;
    if (warp == 0) {
        if (lane == 0) {
            int st = 0;
            uint32_t par = 0;
            for (int tile = blockIdx.x; tile < total && alive; tile += gridDim.x) {
                const TcTile t = tc_tile(p, prefix, nt, tile);
                const int xc = (int)(t.g * p.x_gstride), wr = t.g * p.N + t.n0;
                for (int k = 0; k < KT; k++) {
                    if (!mbar_wait(empty(st), par ^ 1u)) {
                        alive = false;
                        break;
                    }
                    const uint32_t dst = base + (uint32_t)st * TC_STAGE;
                    mbar_expect_tx(full(st), TC_STAGE);
                    tma_load_2d(dst, &map_x, xc + k * 64, t.r0, full(st));
                    tma_load_2d(dst + TC_A, &map_w, k * 64, wr, full(st));
                    if (++st == TC_ST) st = 0, par ^= 1u;
                }
            }
            if (!alive) atomicExch(err, 12);
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TC_N >> 3) << 17) | ((uint32_t)(TC_M >> 4) << 24);
            const uint64_t da0 = desc_kmajor(base), db0 = desc_kmajor(base + TC_A);
            int st = 0, it = 0;
            uint32_t par = 0;
            for (int tile = blockIdx.x; tile < total && alive; tile += gridDim.x, it++) {
                const int a = it & 1;
                if (!mbar_wait(acc_empty(a), ((uint32_t)(it >> 1) & 1u) ^ 1u)) {
                    alive = false;
                    break;
                }
                tc_fence_after();
                for (int k = 0; k < KT; k++) {
                    if (!mbar_wait(full(st), par)) {
                        alive = false;
                        break;
                    }
                    tc_fence_after();
                    const uint64_t off = (uint64_t)((uint32_t)st * (TC_STAGE >> 4));
#pragma unroll
                    for (int i = 0; i < 4; i++) tc_mma(tmem + (uint32_t)a * TC_N, da0 + off + 2 * i, db0 + off + 2 * i, kIdesc, (k > 0 || i > 0) ? 1u : 0u);
                    tc_commit(empty(st));
                    if (++st == TC_ST) st = 0, par ^= 1u;
                }
                if (alive) tc_commit(acc_full(a));
            }
            if (!alive) atomicExch(err, 13);
        }
        __syncwarp();
    } else if (warp >= 4) {
        const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
        const int r = (warp & 3) * 32 + lane;
        int it = 0;
        for (int tile = blockIdx.x; tile < total; tile += gridDim.x, it++) {
            const int a = it & 1;
            const TcTile t = tc_tile(p, prefix, nt, tile);
            if (!__all_sync(0xffffffffu, mbar_wait(acc_full(a), (uint32_t)(it >> 1) & 1u))) {
                alive = false;
                break;
            }
            tc_fence_after();
            const int cols = min(TC_N, p.n_out - t.n0);  // may be negative: a tile of padding
            const size_t o = (size_t)t.g * p.out_gstride + (size_t)(t.r0 + (r < t.rows ? r : 0)) * p.ldo + t.n0;
#pragma unroll 1
            for (int c = 0; c < cols; c += 32) {
                uint32_t v[32];
                tc_ld32(tmem + lane_addr + (uint32_t)(a * TC_N + c), v);
                if (r >= t.rows) {
                    // nothing to store; the warp stays together for the next load
                } else if (F32OUT) {
                    float* d = reinterpret_cast<float*>(p.out) + o + c;
                    if (c + 32 <= cols && p.vec_out) {
#pragma unroll
                        for (int i = 0; i < 32; i += 4) *reinterpret_cast<uint4*>(d + i) = make_uint4(v[i], v[i + 1], v[i + 2], v[i + 3]);
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; i++)
                            if (c + i < cols) d[i] = __uint_as_float(v[i]);
                    }
                } else {
                    uint16_t* d = reinterpret_cast<uint16_t*>(p.out) + o + c;
                    if (c + 32 <= cols && p.vec_out) {
#pragma unroll
                        for (int i = 0; i < 32; i += 8) {
                            uint4 u;
                            u.x = pack_bf2(__uint_as_float(v[i]), __uint_as_float(v[i + 1]));
                            u.y = pack_bf2(__uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
                            u.z = pack_bf2(__uint_as_float(v[i + 4]), __uint_as_float(v[i + 5]));
                            u.w = pack_bf2(__uint_as_float(v[i + 6]), __uint_as_float(v[i + 7]));
                            *reinterpret_cast<uint4*>(d + i) = u;
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; i++)
                            if (c + i < cols) d[i] = f2bf(__uint_as_float(v[i]));
                    }
                }
                __syncwarp();
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(acc_empty(a));
        }
        if (!alive && lane == 0) atomicExch(err, 14);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 2) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(512) : "memory");
}

int32_t launch_tc(b2_ctx* ctx, GroupedGemmParams p) {
    const int bytes = p.out_f32 ? 4 : 2;
    p.vec_out = ((uintptr_t)p.out & 15) == 0 && (p.ldo * bytes) % 16 == 0 && (p.out_gstride * bytes) % 16 == 0;
    CUtensorMap mx, mw;
    const uint64_t cols = p.offsets ? (uint64_t)p.K : (uint64_t)p.ldx;
    B2_CHECK(tc5::get_map(ctx, p.x, (uint64_t)p.x_rows, cols, (uint64_t)p.ldx, TC_M, &mx));
    const uint64_t w_rows = (uint64_t)p.G * p.N;
    B2_CHECK(tc5::get_map(ctx, p.w, w_rows, (uint64_t)p.K, (uint64_t)p.K, TC_N, &mw));
    B2_SMEM_ONCE(ctx, grouped_tc_kernel<true>, TC_SMEM);
    B2_SMEM_ONCE(ctx, grouped_tc_kernel<false>, TC_SMEM);
    int tiles = tile_bound(p, TC_M) * ((p.N + TC_N - 1) / TC_N);
    if (tiles > ctx->sm_count) tiles = ctx->sm_count;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, p.out_f32 ? grouped_tc_kernel<true> : grouped_tc_kernel<false>, dim3(tiles), dim3(256), (size_t)TC_SMEM, ctx->stream,
                          p, ctx->dev_err, mx, mw));
    B2_LAUNCHED(ctx);
    return B2_OK;
}

}  // namespace

bool b2_grouped_gemm_wants_rows(const b2_ctx* ctx, int M, bool sorted, int G, int N) {
    return ctx->use_tc && (sorted ? M / G : M) > 16 && G <= TC_G && (int64_t)G * N >= TC_N;
}
int32_t b2_grouped_gemm_launch(b2_ctx* ctx, bool f32, const GroupedGemmParams& p) {
    if (p.M <= 0) return B2_OK;
    B2_REQUIRE(p.N % 64 == 0 && p.K % 64 == 0 && p.n_out <= p.N, B2_ERR_UNSUPPORTED, "grouped gemm: N and K must be padded to multiples of 64");
    ctx->gemm_flops += 2.0 * p.M * (p.offsets ? 1 : p.G) * (double)p.N * p.K;
    ctx->gemm_weight_bytes += (double)p.N * p.K * 2 * p.G;
    B2_REQUIRE(p.tail_n == 0 || (!f32 && p.stream && !p.offsets), B2_ERR_UNSUPPORTED, "grouped gemm: a shorter last group");
    if (f32) {
        const int bound = tile_bound(p, 8);
        B2_REQUIRE(bound <= 65535, B2_ERR_UNSUPPORTED, "grouped gemm: too many rows for one step of the f32 path");
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, grouped_f32_kernel, dim3(p.N / 32, bound), dim3(256), 0, ctx->stream, p));
        B2_LAUNCHED(ctx);
        return B2_OK;
    }
    B2_REQUIRE(p.ldx % 8 == 0 && p.x_gstride % 8 == 0 && ((uintptr_t)p.x & 15) == 0, B2_ERR_UNSUPPORTED, "grouped gemm: rows must be 16-byte aligned");
    const int per_group = p.offsets ? p.M / p.G : p.M;
    if (!p.stream && !p.row_idx && p.x_rows >= TC_M && b2_grouped_gemm_wants_rows(ctx, p.M, p.offsets != nullptr, p.G, p.N)) return launch_tc(ctx, p);
    if (per_group <= 16) return launch_tile<16, 6>(ctx, p);
    if (p.stream && per_group <= 32) return launch_tile<32, 6>(ctx, p);
    return launch_tile<64, 4>(ctx, p);
}
