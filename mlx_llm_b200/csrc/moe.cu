// Routing of a mixture of experts: sigmoid scores, the best `top` experts of every token, and the sorted order in which
// the grouped projections walk the (token, choice) pairs.
//
// One launch: every warp routes tokens and counts its choices; the block that finishes last turns the counts into
// offsets and places the pairs.  The place of a pair inside its expert's run depends on timing, its result does not:
// rows of a grouped product are independent.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

constexpr int kMaxThreads = 1024, kMaxExperts = 1024;

__global__ void __launch_bounds__(kMaxThreads) route_kernel(const RouteParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    extern __shared__ float sc[];  // [warps][experts]: logits of the token, -inf once taken
    __shared__ int cursor[kMaxExperts];
    __shared__ bool last;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5, E = p.experts;
    float* s = sc + (size_t)warp * E;
    for (int t = blockIdx.x * warps + warp; t < p.T; t += gridDim.x * warps) {
        for (int e = lane; e < E; e += 32) s[e] = p.logits[(size_t)t * p.ld + e];
        __syncwarp();
        for (int k = 0; k < p.top; k++) {  // the sigmoid rises with the logit: choose by logit, ties to the lower index
            float best = -INFINITY;
            int bi = 0x7fffffff;
            for (int e = lane; e < E; e += 32)
                if (s[e] > best) best = s[e], bi = e;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
                if (ov > best || (ov == best && oi < bi)) best = ov, bi = oi;
            }
            if (bi >= E) bi = 0;  // not-a-number logits only
            if (lane == 0) {
                p.expert[(size_t)t * p.top + k] = bi;
                p.weight[(size_t)t * p.top + k] = sigmoid_f32(best);
                s[bi] = -INFINITY;
                atomicAdd(&p.counters[bi], 1);
            }
            __syncwarp();
        }
    }
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) last = atomicAdd(&p.counters[E], 1) == (int)gridDim.x - 1;
    __syncthreads();
    if (!last) return;
    __threadfence();
    if (warp == 0) {  // exclusive prefix sum of the counts, 32 experts at a time
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int n = e0 + lane < E ? __ldcg(&p.counters[e0 + lane]) : 0;
            int incl = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int u = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += u;
            }
            if (e0 + lane < E) {
                cursor[e0 + lane] = base + incl - n;
                p.offsets[e0 + lane] = base + incl - n;
            }
            base += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (lane == 0) p.offsets[E] = base;
    }
    __syncthreads();
    for (int e = threadIdx.x; e <= E; e += blockDim.x) p.counters[e] = 0;  // ready for the next launch
    for (int i = threadIdx.x; i < p.T * p.top; i += blockDim.x) {
        const int e = __ldcg(&p.expert[i]), at = atomicAdd(&cursor[e], 1);
        p.pos[i] = at;
        p.src[at] = i / p.top;
        p.row_w[at] = __ldcg(&p.weight[i]);
    }
}

__global__ void __launch_bounds__(128) gather_rows_kernel(const uint16_t* __restrict__ x, const int32_t* __restrict__ src, int cols, int ld,
                                                          uint16_t* __restrict__ out) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    const uint16_t* s = x + (size_t)src[blockIdx.x] * ld;
    uint16_t* o = out + (size_t)blockIdx.x * ld;
    for (int i = threadIdx.x * 8; i < cols; i += 128 * 8) *reinterpret_cast<uint4*>(o + i) = *reinterpret_cast<const uint4*>(s + i);
}

}  // namespace

int32_t b2_gather_rows_launch(b2_ctx* ctx, const uint16_t* x, const int32_t* src, int n, int cols, int ld, uint16_t* out) {
    if (n <= 0) return B2_OK;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, gather_rows_kernel, dim3(n), dim3(128), 0, ctx->stream, x, src, cols, ld, out));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
int32_t b2_route_launch(b2_ctx* ctx, const RouteParams& p) {
    if (p.T <= 0) return B2_OK;
    B2_REQUIRE(p.experts <= kMaxExperts, B2_ERR_UNSUPPORTED, "routing: at most 1024 experts");
    const int warps = p.T <= 8 || p.experts > 256 ? 8 : 32;
    int grid = (p.T + warps - 1) / warps;
    if (grid > ctx->sm_count) grid = ctx->sm_count;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, route_kernel, dim3(grid), dim3(warps * 32), (size_t)warps * p.experts * 4, ctx->stream, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
