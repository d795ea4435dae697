// Output projection of the quantized decoders: fp16 weights and logits (see lm_head.cuh).
#include "lm_head.cuh"

using namespace glq;

extern "C" size_t glq_lm_head_workspace_bytes(void) { return lm_workspace_bytes(); }

extern "C" int glq_lm_head(const void* x, int64_t ldx, const void* W, int B, int V, int H, void* logits, int64_t ldl,
                           int64_t* argmax_out, void* workspace, size_t workspace_bytes, int32_t* counter,
                           void* stream) {
    return lm_head_launch<false>(x, ldx, W, B, V, H, 1.f, logits, ldl, argmax_out, workspace, workspace_bytes, counter, stream);
}
