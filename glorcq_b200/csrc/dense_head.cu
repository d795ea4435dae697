// Output projection of the unquantized decoders: bfloat16 weights, float logits times a constant (see lm_head.cuh).
#include "../../include/glorcq_b200_dense.h"
#include "lm_head.cuh"

using namespace glq;

extern "C" size_t glq_dense_head_workspace_bytes(void) { return lm_workspace_bytes(); }

extern "C" int glq_dense_head(const void* x, int64_t ldx, const void* W, int B, int V, int H, float scale, float* logits, int64_t ldl,
                              int64_t* argmax_out, void* workspace, size_t workspace_bytes, int32_t* counter, void* stream) {
    return lm_head_launch<true>(x, ldx, W, B, V, H, scale, logits, ldl, argmax_out, workspace, workspace_bytes, counter, stream);
}
