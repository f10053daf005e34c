// Storage element of the layered models' activations and weights: bf16 bits (uint16_t) or float.  Kernels that serve
// both number formats are templates over it; arithmetic is f32 in either.
#pragma once
#include "common.cuh"

template <typename T>
struct Elt;
template <>
struct Elt<uint16_t> {
    static __device__ __forceinline__ float ld(const uint16_t* p) { return bf2f(*p); }
    static __device__ __forceinline__ void st(uint16_t* p, float v) { *p = f2bf(v); }
    static __device__ __forceinline__ void ld8(const uint16_t* p, float (&v)[8]) {  // 16-byte aligned
        const uint4 u = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; i++) v[2 * i] = bflo(w[i]), v[2 * i + 1] = bfhi(w[i]);
    }
    static __device__ __forceinline__ void ld4(const uint16_t* p, float (&v)[4]) {  // 8-byte aligned
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        v[0] = bflo(u.x), v[1] = bfhi(u.x), v[2] = bflo(u.y), v[3] = bfhi(u.y);
    }
    static __device__ __forceinline__ void st4(uint16_t* p, const float (&v)[4]) {
        *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]));
    }
    static __device__ __forceinline__ void st8(uint16_t* p, const float (&v)[8]) {
        *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]), pack_bf2(v[4], v[5]), pack_bf2(v[6], v[7]));
    }
};
template <>
struct Elt<float> {
    static __device__ __forceinline__ float ld(const float* p) { return *p; }
    static __device__ __forceinline__ void st(float* p, float v) { *p = v; }
    static __device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
    }
    static __device__ __forceinline__ void ld4(const float* p, float (&v)[4]) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w;
    }
    static __device__ __forceinline__ void st4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    static __device__ __forceinline__ void st8(float* p, const float (&v)[8]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
};
__device__ __forceinline__ float elt_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float elt_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
// Sum over the block (blockDim.x a multiple of 32); `red` holds 33 floats.  Every thread gets the result.
__device__ __forceinline__ float elt_block_sum(float v, float* red) {
    v = elt_warp_sum(v);
    __syncthreads();  // the previous use of `red` is over
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    if (threadIdx.x < 32) {
        float s = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.f;
        s = elt_warp_sum(s);
        if (threadIdx.x == 0) red[32] = s;
    }
    __syncthreads();
    return red[32];
}
__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x * sigmoid_f32(x); }
// ... with the fast exponential and division where the result is rounded to bf16 anyway
template <typename T>
__device__ __forceinline__ float silu_for(float x) {
    return sizeof(T) == 2 ? __fdividef(x, 1.0f + __expf(-x)) : silu_f32(x);
}
