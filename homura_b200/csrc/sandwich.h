// Residual sums between layer norms (sandwich.cu): what a sublayer gives back is normed and joins the residual, whose own norm is what
// the next projection reads.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "common.cuh"

namespace hm {

constexpr int SANDWICH_MAX_WIDTH = 16384;

struct SandwichArgs {
    float* x;                // [M][W] residual: x += LN(y) * w
    const float* y;          // [M][ldy], or null: nothing joins
    int ldy;
    // two results side by side, W apart: y is half the sum of their RMS norms with these weights
    const float *left_w, *right_w;  // or null
    const float* w;          // [W]
    const float* next_w;     // [W] or null: LN(x) * next_w
    float eps;
    int M, W;
    float* normed;           // [M][W], or, when xp is given, the activation image of the next tensor-core projection
    unsigned char* xp;
    int xp_mpad;
};
cudaError_t launch_sandwich(const SandwichArgs& a, cudaStream_t st, bool pdl);

}  // namespace hm
