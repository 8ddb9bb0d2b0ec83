// Everything between a layer's input projection and its attention, as one launch (side.cu): queries, keys and values on their way to
// the cache, latents likewise, gated linear attention, the activations of a dense or shared feed-forward, the router's choice.
#pragma once
#include "gla.h"
#include "gqa_attn.h"
#include "latent_attn.h"
#include "moe.h"

namespace hm {

struct LatentSide {
    LatentPool pool;
    const float* c;          // [M][ld] latent and rotated key part
    const float* w;
    int rot_pairs;
    const double* turns;
    int neighbours;          // rotated pairs are (2 i, 2 i + 1)
    // queries' latent, with q_xp: RMS-normed into the activation image of its up-projection
    const float* cq;
    int q_rank;
    const float* q_w;
    unsigned char* q_xp;
};

struct MlpSide {
    // gated activations: act(gate) * up (* sigmoid of a per-row logit) for ff elements, rounded up to eight
    int ff;                  // 0: none
    int act;                 // GluAct
    const float *gate, *up;  // [M][ld]
    const float* row_gate;   // [M][ld], first column, or null
    float* out;              // [M][ld_out] from out_off on, or, when xp is given, the image of the next projection
    int ld_out, out_off;
    unsigned char* xp;
    // router
    const float* logits;     // [M][ld], or null
    RouteSpec route;
    // the layer's normalised input, for experts that read it row by row
    const float* x;          // [M][W]
    int W;
    const float* w;
    float* normed;           // or null
};

// What the gated delta rule reads besides queries, keys and values: factors out of two latents per row, [rank] x [rank][columns].
//   alpha = exp(neg_rate[head] * softplus(up_a . a + bias))    per head and key channel
//   gate  = up_g . g                                            per head and value channel (before its sigmoid)
struct LowRankSide {
    const float *a, *g;      // [M][ld] latents
    int rank_a, rank_g;
    const float *up_a, *bias, *neg_rate;
    const float* up_g;
    int heads, dim, vdim;
    float *alpha, *gate;     // [M][heads * dim], [M][heads * vdim]
};

struct SideArgs {
    int M, ld, xp_mpad;
    float eps;
    const int32_t *row_pos, *row_seq;
    int has_post, has_latent, has_gla, has_post2, has_low;
    GqaPostArgs post, post2;  // post2: rows for a recurrence (recur.h)
    LowRankSide low;
    LatentSide latent;
    GlaArgs gla;
    MlpSide mlp;
    // blocks of the parts, in launch order (filled in by the launcher)
    int n_gla, n_post, n_latent, n_act, n_route, n_normed, n_post2, n_low;
};
cudaError_t launch_side(const SideArgs& a, int sm_count, cudaStream_t st, bool pdl);

// Sums the parts of a sublayer's result into the residual and packs its RMS norm (weight w, null: nothing is packed) as the activation image of the next projection.
struct SumNormArgs {
    float* x;                // [M][W]
    const float* y;          // parts results, part_stride apart
    int parts;
    size_t part_stride;
    int M, W;
    const float* w;
    float eps;
    unsigned char* xp;
    int xp_mpad;
};
cudaError_t launch_sum_norm(const SumNormArgs& a, cudaStream_t st, bool pdl);

}  // namespace hm
