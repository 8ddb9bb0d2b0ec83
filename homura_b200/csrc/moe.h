// Residual sums with normalised sublayer results, routers, and mixtures of experts (moe.cu).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "common.cuh"
#include "model_spec.h"

namespace hm {

// Where a router puts its choice.
struct RouteOut {
    int32_t* ids;       // [M][top] chosen experts, -1 for identity ones
    float* weights;     // [M][top]
    float* identity;    // [M] sum of the weights of the chosen identity experts
    float* dense;       // [M][experts] weight of every expert, 0 where it is not chosen; or null
    uint32_t* mask;     // [M][ceil(experts / 32)] with dense: one bit per chosen expert
};

// How a router chooses: `top` of n_out = experts + identity ones (the last) by score + correction; weights are the scores times scale.
struct RouteSpec {
    const float* correction; // [n_out] or null
    int experts, n_out, top;
    float scale;
    RouteOut out;
};

// x += mult * RMSnorm(y) * w, and then, optionally, the router over the new x.
struct PostNormArgs {
    const float* y;          // [M][W] what the sublayer gave back; with parts > 1 the sum of so many, part_stride apart
    int parts;
    size_t part_stride;
    const float* identity;   // [M] or null: y + identity * x instead of y
    float* x;                // [M][W] residual
    int M, W;
    const float* w;
    float mult, eps;
    unsigned char* xp;       // optional: the new x as the activation image of the next tensor-core projection
    int xp_mpad;
    // router
    const uint16_t* router;  // [n_out][W] bf16, or null
    const float* correction; // [n_out]
    int experts, n_out, top; // n_out = experts + identity ones (the last)
    RouteOut out;
};
cudaError_t launch_post_norm(const PostNormArgs& a, int sm_count, cudaStream_t st, bool pdl);

// Experts' weights as tensor-core tile images (gemm_tc.h), one after the other: gate and up interleaved 64 + 64 per block of 128
// rows over W, down [W] over ff; ff padded to 64.
struct ExpertWeights {
    const uint16_t *gu, *down;
    int n, W, ff, top;       // n experts
    float limit;
    int act;                 // GluAct
};
__host__ __device__ __forceinline__ int expert_blocks(int ff) { return (ff + 63) / 64; }
size_t expert_gu_elems(int W, int ff);
size_t expert_down_elems(int W, int ff);

// Few rows: every (row, chosen expert) pair reads its own weights.  act: [M * top][ff padded], already times the routing weight.
cudaError_t launch_expert_gate_up(const ExpertWeights& e, const float* x, int M, const RouteOut& r, float* act, cudaStream_t st, bool pdl);
// y = resid (or nothing) + the sum over the chosen experts; y may be resid.
cudaError_t launch_expert_down(const ExpertWeights& e, const float* act, int M, const RouteOut& r, const float* resid, float* y, cudaStream_t st, bool pdl);

// act(gate) * up of the kinds of gated feed-forwards (GluAct).
__device__ __forceinline__ float glu(int act, float gate, float up, float limit) {
    if (act == GLU_SILU) return gate / (1.0f + expf(-gate)) * up;
    if (act == GLU_GELU) return 0.5f * gate * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * gate * gate, gate, gate))) * up;
    return clamped_glu(gate, up, limit);
}

}  // namespace hm
