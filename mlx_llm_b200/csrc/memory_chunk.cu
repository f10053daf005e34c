#include "layer_kernels.h"
#include "common.cuh"
bool b2_memory_chunk_eligible(const MemorySpec&) { return false; }
size_t b2_memory_chunk_bytes(const MemorySpec&, size_t) { return 0; }
int32_t b2_memory_chunk_launch(b2_ctx*, const MemorySpec&, const MemoryParams&) { return 0; }
