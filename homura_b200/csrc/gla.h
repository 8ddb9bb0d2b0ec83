// Gated linear attention: per head a state S [dim x vdim] in f32 that every token of a sequence first shrinks, row by row, and then
// joins,  S <- diag(alpha) S + k v^T,  o = S^T q.  In passes over runs of tokens the CTAs of a cluster share a head's columns and keep
// them in registers while they walk through a run; in passes of single tokens a head's state goes through a CTA's shared memory
// (gla.cuh).  Between passes the state lies column by column in memory, whatever the shape of the launches.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "gqa_attn.h"

namespace hm {

constexpr int GLA_THREADS = 256;

// How a launch deals out a head's state: `cluster` CTAs take `share` columns each and go through them in `slices` of `cols`; `lanes`
// threads share a column, each with `rows` of its rows.
struct GlaShape {
    int cluster, share, slices, cols, lanes, rows;
};
constexpr int GLA_MAX_CLUSTER = 8;
constexpr int GLA_UP_SMEM = 8192;        // floats of a head's decay projection that are staged ahead of the dependency
constexpr int GLA_TOKEN_DIM = 256;       // single tokens: largest key size, and bytes of a head's state, that go through shared memory
constexpr int GLA_TOKEN_BYTES = 96 * 1024;
// heads: (run, head) pairs of the launch.
GlaShape gla_shape(int dim, int vdim, int heads, int sm_count);
__host__ __device__ __forceinline__ int gla_pad(int dim) { return (dim + 3) & ~3; }
__host__ __device__ __forceinline__ size_t gla_state_floats(int dim, int vdim) { return (size_t)vdim * gla_pad(dim); }  // per head
constexpr int GLA_MAX_DIM = 1024, GLA_MAX_VDIM = 512;

struct GlaArgs {
    GlaShape shape;          // filled in by the launcher, like step
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
    float* state;            // [sequence][heads][vdim][gla_pad(dim)], sequences seq_stride floats apart; position 0 starts from zero
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
    int step;                // tokens staged at a time
    int* err_flag;
};

}  // namespace hm
