// Routing of a mixture of experts: scores (sigmoid, or softmax with a correction of the choice), the best `top` experts of every
// token, and the sorted order in which the grouped projections walk the (token, choice) pairs.  Identity experts are counted
// apart: their pairs have no place in that order.
//
// One launch: every warp routes tokens and counts its choices; the block that finishes last (a single block: the block itself,
// which counts in shared memory) turns the counts into offsets and places the pairs.  The place of a pair inside its expert's run depends on timing, its result does not:
// rows of a grouped product are independent.
#include "elt.cuh"
#include "layer_kernels.h"

namespace {

constexpr int kMaxThreads = 1024, kMaxExperts = 1024;

__global__ void __launch_bounds__(kMaxThreads) route_kernel(const RouteParams p) {
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    pdl_wait();
    extern __shared__ float sc[];  // [warps][outputs]: logits (Sigmoid) or choice scores (Softmax) of the token, -inf once taken
    __shared__ int cursor[kMaxExperts], own[kMaxExperts];
    const bool one = gridDim.x == 1;
    if (one)
        for (int e = threadIdx.x; e < p.experts; e += blockDim.x) own[e] = 0;
    __syncthreads();
    __shared__ bool last;
    __shared__ int total;  // pairs that have a place
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5, E = p.experts, N = E + p.identity;
    const bool soft = p.score == RouteScore::Softmax;
    float* s = sc + (size_t)warp * N;
    for (int t = blockIdx.x * warps + warp; t < p.T; t += gridDim.x * warps) {
        const float* z = p.logits + (size_t)t * p.ld;
        float top_z = -INFINITY, inv = 0.f, sum = 0.f, passed = 0.f;  // (sum, passed: lane 0)
        for (int e = lane; e < N; e += 32) s[e] = z[e], top_z = fmaxf(top_z, s[e]);
        if (soft) {
            top_z = elt_warp_max(top_z);
            float total = 0.f;
            for (int e = lane; e < N; e += 32) total += expf(s[e] - top_z);
            inv = 1.0f / elt_warp_sum(total);
            for (int e = lane; e < N; e += 32) s[e] = expf(s[e] - top_z) * inv + p.correction[e];
        }
        __syncwarp();
        for (int k = 0; k < p.top; k++) {  // the sigmoid rises with the logit: choose by logit; ties to the lower index
            float best = -INFINITY;
            int bi = 0x7fffffff;
            for (int e = lane; e < N; e += 32)
                if (s[e] > best) best = s[e], bi = e;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
                if (ov > best || (ov == best && oi < bi)) best = ov, bi = oi;
            }
            if (bi >= N) bi = 0;  // not-a-number logits only
            if (lane == 0) {
                const float w = soft ? expf(z[bi] - top_z) * inv : sigmoid_f32(best);
                p.expert[(size_t)t * p.top + k] = bi;
                p.weight[(size_t)t * p.top + k] = w;
                s[bi] = -INFINITY;
                sum += w;
                if (bi < E)
                    atomicAdd(one ? &own[bi] : &p.counters[bi], 1);
                else
                    passed += w;
            }
            __syncwarp();
        }
        if (soft) {  // (each lane scales what lane 0 wrote)
            const float f = p.scale / (__shfl_sync(0xffffffffu, sum, 0) + 1e-20f);
            for (int k = lane; k < p.top; k += 32) p.weight[(size_t)t * p.top + k] *= f;
            if (lane == 0 && p.identity) p.pass[t] = passed * f;
        }
        if (p.shared && lane == 0) p.shared_w[t] = sigmoid_f32(z[N]);
        __syncwarp();
    }
    if (!one) {
        __threadfence();
        __syncthreads();
        if (threadIdx.x == 0) last = atomicAdd(&p.counters[E], 1) == (int)gridDim.x - 1;
        __syncthreads();
        if (!last) return;
        __threadfence();
    } else {
        __syncthreads();
    }
    if (warp == 0) {  // exclusive prefix sum of the counts, 32 experts at a time
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int n = e0 + lane < E ? (one ? own[e0 + lane] : __ldcg(&p.counters[e0 + lane])) : 0;
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
        if (lane == 0) p.offsets[E] = total = base;
    }
    __syncthreads();
    for (int e = threadIdx.x; !one && e <= E; e += blockDim.x) p.counters[e] = 0;  // ready for the next launch
    const int per = p.top + (p.shared ? 1 : 0);
    for (int i = threadIdx.x; i < p.T * p.top; i += blockDim.x) {
        const int e = __ldcg(&p.expert[i]), t = i / p.top;
        if (e < E) {
            const int at = atomicAdd(&cursor[e], 1);
            p.pos[i + t * (per - p.top)] = at;
            p.src[at] = t;
            p.row_w[at] = __ldcg(&p.weight[i]);
        } else {
            p.pos[i + t * (per - p.top)] = -1;
        }
    }
    if (p.shared)
        for (int t = threadIdx.x; t < p.T; t += blockDim.x) p.pos[t * per + p.top] = p.T * p.top + t;
    for (int at = total + threadIdx.x; at < p.T * p.top; at += blockDim.x) p.src[at] = 0, p.row_w[at] = 0.f;  // (a gather reads every place)
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
    const int outputs = p.experts + p.identity;
    B2_REQUIRE(outputs <= 2 * kMaxExperts && (p.identity == 0 || p.score == RouteScore::Softmax), B2_ERR_UNSUPPORTED, "routing: identity experts");
    const int warps = p.T <= 8 || outputs > 256 ? (outputs > kMaxExperts ? 4 : 8) : 32;
    int grid = (p.T + warps - 1) / warps;
    if (grid > ctx->sm_count) grid = ctx->sm_count;
    B2_CUDA(b2_launch_pdl(ctx->pdl_consumers, route_kernel, dim3(grid), dim3(warps * 32), (size_t)warps * outputs * 4, ctx->stream, p));
    B2_LAUNCHED(ctx);
    return B2_OK;
}
