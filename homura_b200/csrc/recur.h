// Recurrences of linear attention over prepared rows: per head a state S [dim x vdim] in f32, one token after the other,
//   retention    S <- decay S + k v^T                                             (a fixed decay per head)
//   delta rule   S <- diag(alpha) S;  S <- S + k (beta (v - S^T k))^T             (a decay per key channel)
// and o = S^T q.  In passes over runs of tokens a cluster of CTAs shares a head's columns and keeps them in registers while it walks through
// a run; in passes of single tokens a head's state goes through a CTA's shared memory.  Between passes the state lies column by column
// in memory, as that of gla.h.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "gla.h"
#include "model_spec.h"

namespace hm {

struct RecurArgs {
    GlaShape shape;          // filled in by the launcher, like step
    int kind;                // LinearKind: LIN_RETENTION or LIN_DELTA
    int heads, kv_heads;     // head h reads query / key head h / (heads / kv_heads)
    int dim, vdim;
    const float *q, *k, *v;  // rows [M][ldq] of query heads head_ld apart, keys alike, [M][ldv] of values
    int ldq, ldk, ldv, head_ld;
    float q_scale;
    const float* decay;      // LIN_RETENTION: [heads]
    const float* alpha;      // LIN_DELTA: [M][heads * dim]
    const float* beta;       // LIN_DELTA: [M][ld_beta], before the sigmoid
    int ld_beta;
    const float* gate;       // [M][ld_gate]: every head's result is RMS-normed, times the silu (retention) or the sigmoid (delta rule) of this
    int ld_gate;
    const float* norm_w;     // [vdim] or null
    float eps;
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
cudaError_t launch_recur(const RecurArgs& a, int sm_count, cudaStream_t st, bool pdl);

}  // namespace hm
