// The variant of the weight-streaming projection with rotation, capped logits, clamped gated activations and shared gates (see gemv_kernel.cuh).
#include "gemv_kernel.cuh"

namespace hm {

cudaError_t launch_gemv_bf16_turn(const GemvArgs& a, int M, cudaStream_t st, bool pdl) { return launch_rows<2>(a, M, st, pdl); }

}  // namespace hm
