// Shared by the memory kernels: inputs kept between steps (the convolution's last ones, or the token shift's last row).
#pragma once
#include "elt.cuh"
#include "layer_kernels.h"

// Leaves the last taps - 1 inputs of sequence b's convolution, or the last row of the normed stream, in its record.  The `blocks`
// blocks that work on the sequence share the channels.
template <typename T>
__device__ __forceinline__ void memory_keep_inputs(const MemorySpec& s, const MemoryParams& p, int b, int block, int blocks) {
    if (s.shift > 0) {
        const T* h = reinterpret_cast<const T*>(p.h) + (size_t)(p.cu_seqlens[b + 1] - 1) * p.ld_h;
        float* kept = p.state + (size_t)p.seq_slot[b] * p.slot_stride + s.state_floats();
        for (int i = block * (int)blockDim.x + (int)threadIdx.x; i < s.shift; i += blocks * (int)blockDim.x) kept[i] = Elt<T>::ld(h + i);
    }
    const int keep = s.keep(), C = s.channels(), start = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - start, before = p.context_lens[b] - n;
    if (keep == 0) return;
    for (int ch = block * (int)blockDim.x + (int)threadIdx.x; ch < C; ch += blocks * (int)blockDim.x) {
        float* c = p.state + (size_t)p.seq_slot[b] * p.slot_stride + s.state_floats() + ch;
        const T* u = reinterpret_cast<const T*>(p.in) + p.c_off + ch;
        for (int j = 0; j < keep; j++) {  // ascending: a shift reads places it has not overwritten yet
            const int k = n - keep + j;
            c[(size_t)j * C] = k >= 0 ? Elt<T>::ld(u + (size_t)(start + k) * p.ld) : (before > 0 ? c[(size_t)(j + n) * C] : 0.f);
        }
    }
}
