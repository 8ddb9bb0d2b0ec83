// Gated linear attention: per head a state S [dim x vdim] in f32 that every token of a sequence first shrinks, row by row, and then
// joins,  S <- diag(alpha) S + k v^T,  o = S^T q.  A CTA of 256 threads keeps a head's state in registers while it walks through a
// run's tokens (gla.cuh); between passes the state lives in the order of those registers.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "gqa_attn.h"

namespace hm {

constexpr int GLA_THREADS = 256;

// How a head's state is dealt out: `lanes` threads share a column, each with `rows` of its padded rows; a CTA holds `cols` columns at
// a time and goes through `slices` of them.
struct GlaShape {
    int rows = 0, lanes = 1, cols = 0, slices = 0;
    __host__ __device__ int padded_dim() const { return rows * lanes; }
    __host__ __device__ size_t state_floats() const { return (size_t)slices * rows * GLA_THREADS; }  // per head
};
bool gla_shape(int dim, int vdim, GlaShape* out);  // false: the sizes are not covered

struct GlaArgs {
    GlaShape shape;
    int heads, dim, vdim, rank;
    // columns of the layer's input projection [M][ld]: queries, keys [heads * dim], values, output gate [heads * vdim], decay latent [rank]
    const float* raw;
    int ld, q_off, k_off, v_off, g_off, a_off;
    float q_scale;
    const float* up;         // decay: [heads][rank][dim], and
    const float* bias;       // [heads * dim]: alpha = sigmoid(up . latent + bias)^inv_tau
    float inv_tau;
    const float* norm_w;     // [vdim]: every head's result is RMS-normed, times the silu of the gate
    float eps, out_scale;
    float* state;            // [sequence][heads][state_floats], sequences seq_stride floats apart; position 0 starts from zero
    size_t seq_stride;
    const int32_t *row_pos, *row_seq;
    int M;
    GqaRuns runs;
    int longest_run;
    int early;               // every row is its own sequence and the state was complete before the launch in front began
    float* out;              // [M][ld_out] from out_off on, or, when xp is given, the activation image of the next projection
    int ld_out, out_off;
    unsigned char* xp;
    int xp_mpad;
    int step;                // tokens staged at a time (gla_smem fills it in)
};
size_t gla_smem(GlaArgs* a);  // dynamic shared memory of a CTA

}  // namespace hm
