#include "layer_kernels.h"
#include "common.cuh"
bool b2_gqa_prefill_eligible(const GroupedAttnSpec&) { return false; }
int32_t b2_gqa_prefill_launch(b2_ctx*, const GroupedAttnSpec&, const GqaAttnParams&, int) { return 0; }
