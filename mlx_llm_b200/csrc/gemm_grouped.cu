// One matrix product per group: out_g[r, n] = sum_k x_g[r, k] * w_g[n, k].
//
// Two uses: the experts of a routed feed-forward (groups own consecutive runs of sorted rows, given by a device-side
// offset table) and per-head projections (every group has the same rows, at a column offset of x and out).
#include "common.cuh"
#include "layer_kernels.h"

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

// bf16 tile kernel: BM rows x 64 outputs, 4 warps, mma.sync with f32 accumulation, cp.async double buffering.
template <int BM, bool F32OUT>
__global__ void __launch_bounds__(kThreads) grouped_tile_kernel(const GroupedGemmParams p) {
    constexpr int MT = BM / 16;  // each warp: all BM rows x 16 outputs
    constexpr int A_BYTES = BM * BK * 2, B_BYTES = BN * BK * 2;
    extern __shared__ __align__(128) uint8_t smem[];
    const uint32_t sA = smem_u32(smem), sB = sA + 2 * A_BYTES;
    pdl_wait();
    int g, r0, rows;
    find_tile<BM>(p, blockIdx.y, g, r0, rows);
    if (rows <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, n0 = blockIdx.x * BN;
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
    load(0, 0);
    cp_async_commit();
    for (int kt = 0; kt < KT; kt++) {
        if (kt + 1 < KT) load(kt + 1, (kt + 1) & 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const uint32_t a_base = sA + (kt & 1) * A_BYTES, b_base = sB + (kt & 1) * B_BYTES;
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
        __syncthreads();
    }
#pragma unroll
    for (int mt = 0; mt < MT; mt++)
#pragma unroll
        for (int nt = 0; nt < 2; nt++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = mt * 16 + (lane >> 2) + (e >> 1) * 8, n = n0 + warp * 16 + nt * 8 + 2 * (lane & 3) + (e & 1);
                if (r >= rows || n >= p.n_out) continue;
                const int orow = p.map_out ? p.row_idx[r0 + r] : r0 + r;
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

template <int BM>
int32_t launch_tile(b2_ctx* ctx, const GroupedGemmParams& p) {
    const int smem = 2 * (BM + BN) * BK * 2;
    const dim3 grid(p.N / BN, tile_bound(p, BM));
    if (p.out_f32)
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, grouped_tile_kernel<BM, true>, grid, dim3(kThreads), smem, ctx->stream, p));
    else
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, grouped_tile_kernel<BM, false>, grid, dim3(kThreads), smem, ctx->stream, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}

}  // namespace

int32_t b2_grouped_gemm_launch(b2_ctx* ctx, bool f32, const GroupedGemmParams& p) {
    if (p.M <= 0) return B2_OK;
    B2_REQUIRE(p.N % 64 == 0 && p.K % 64 == 0 && p.n_out <= p.N, B2_ERR_UNSUPPORTED, "grouped gemm: N and K must be padded to multiples of 64");
    ctx->gemm_flops += 2.0 * p.M * (p.offsets ? 1 : p.G) * (double)p.N * p.K;
    ctx->gemm_weight_bytes += (double)p.N * p.K * 2 * p.G;
    if (f32) {
        const int bound = tile_bound(p, 8);
        B2_REQUIRE(bound <= 65535, B2_ERR_UNSUPPORTED, "grouped gemm: too many rows for one step of the f32 path");
        B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, grouped_f32_kernel, dim3(p.N / 32, bound), dim3(256), 0, ctx->stream, p));
        B2_LAUNCHED(ctx);
        return B2_OK;
    }
    B2_REQUIRE(p.ldx % 8 == 0 && p.x_gstride % 8 == 0 && ((uintptr_t)p.x & 15) == 0, B2_ERR_UNSUPPORTED, "grouped gemm: rows must be 16-byte aligned");
    const int per_group = p.offsets ? p.M / p.G : p.M;
    if (per_group <= 16) return launch_tile<16>(ctx, p);
    return launch_tile<64>(ctx, p);
}
