// The extended variant of the weight-streaming projection (see gemv_kernel.cuh).
#include "gemv_kernel.cuh"

namespace hm {

cudaError_t launch_gemv_bf16_ext(const GemvArgs& a, int M, cudaStream_t st, bool pdl) { return launch_rows<1>(a, M, st, pdl); }

}  // namespace hm
