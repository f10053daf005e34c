#include "layer_kernels.h"
#include "common.cuh"
bool b2_gqa_decode_eligible(const GroupedAttnSpec&) { return false; }
int b2_gqa_head_blocks(const GroupedAttnSpec& a) { return a.kv_heads * ((a.group() + 7) / 8); }
int32_t b2_gqa_decode_launch(b2_ctx*, const GroupedAttnSpec&, const GqaAttnParams&, int) { return 0; }
