// Grouped-query attention over a paged cache for head sizes of any kind: `dim` elements per query and key, `vdim` per value,
// an optional learned bias by distance, rows of several sequences in one launch (gqa_attn.cu).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "common.cuh"

namespace hm {

constexpr int GQA_PAGE = 64;       // tokens per page
constexpr int GQA_MAX_ROWS = 64;   // rows of one launch

// One layer's pools.  A page holds, per key/value head, its tokens in chunks of eight elements, [pad / 8][64 tokens][8] (pad = the
// size rounded up to 16, the tail zero): one contiguous block per head, whose 8x8 matrices for ldmatrix are 128 contiguous bytes.
struct GqaPool {
    void *k, *v;
    const int32_t* page_table;  // [sequences][max_pages]
    int max_pages;
    int kv_heads, dim, vdim;
    int bf16;
};
__host__ __device__ __forceinline__ int gqa_pad(int d) { return (d + 15) & ~15; }
__host__ __device__ __forceinline__ size_t gqa_page_elems(int kv_heads, int d) { return (size_t)kv_heads * GQA_PAGE * gqa_pad(d); }
__host__ __device__ __forceinline__ int gqa_tile_off(int t, int d) { return ((d >> 3) * GQA_PAGE + t) * 8 + (d & 7); }

// Rows as runs: consecutive positions of one sequence.
struct GqaRuns {
    int n = 0;                            // 0: every row is a run
    uint8_t row[GQA_MAX_ROWS + 1];        // first row of every run; row[n] = rows of the pass
    uint16_t tile[GQA_MAX_ROWS + 1];      // first tile of every run (filled in by the attention's launcher)
    // The run of row m: [first, end).
    __host__ __device__ __forceinline__ void find(int m, int& first, int& end) const {
        if (n == 0) {
            first = m;
            end = m + 1;
            return;
        }
        int lo = 0, hi = n;
        while (hi - lo > 1) {
            const int mid = (lo + hi) / 2;
            if (row[mid] <= m) lo = mid;
            else hi = mid;
        }
        first = row[lo];
        end = row[lo + 1];
    }
};

__host__ __device__ __forceinline__ int conv_slots(int taps) { return taps > 1 ? GQA_MAX_ROWS + taps - 1 : 0; }

// What happens to a projection's queries, keys and values before the attention: a short convolution, norms, rotation, temperature,
// blended values; keys and values go to their page slots, queries to q_out.
struct GqaPostArgs {
    GqaPool pool;
    const float* raw;        // [M][ld]: queries | keys | values
    int ld, M, heads;
    int qk_norm;             // QkNorm
    const float *q_norm, *k_norm;
    float eps;
    float q_scale;           // times the score scale (and log2 e: weights are powers of two)
    float temp_coef;
    int temp_every;          // 0: no temperature
    float* v_first;          // [M][kv_heads * vdim] or null: values of the layer that the others blend in
    const float* v_lambda;   // null: this layer keeps its values in v_first
    const int32_t *row_pos, *row_seq;
    float* q_out;            // [M][heads * dim]
    // Causal convolution over time of every channel (queries | keys | values), taps > 0: the inputs of the last taps - 1 tokens of a
    // sequence are kept in conv_state, position p in slot p % conv_slots(taps).  The ring is longer than a pass's rows, so that the slots
    // in front of a run are never written by the launch that reads them.
    int taps;
    const float* conv_w;     // [channels][taps], the last one meets the token itself
    float* conv_state;       // [sequence][conv_slots(taps)][channels], sequences conv_stride floats apart
    size_t conv_stride;
    GqaRuns runs;            // with taps > 1
    // rotation of the first rot_dims elements of queries and keys: pair (i, i + rot_dims / 2) makes turns[i] turns per position
    int rot_dims;
    const double* turns;
    // what only some designs have (the post kernels' third variant)
    int rot_neighbours;      // pairs are (2 i, 2 i + 1)
    int conv_silu;           // convolved values pass through the silu
    int tied_values;         // no values in `raw`: a key as it is before its rotation is its value
    int v_heads;             // with k_out: heads of values
    const float* head_scale; // [heads] or null: queries times this
    float *k_out, *v_out;    // rows [M][kv_heads * dim] and [M][v_heads * vdim] instead of page slots
    bool varied() const { return rot_neighbours || conv_silu || tied_values || head_scale || k_out; }
};
cudaError_t launch_gqa_post(const GqaPostArgs& a, cudaStream_t st, bool pdl);

struct GqaAttnArgs {
    GqaPool pool;
    const float* q;          // [M][heads * dim], scaled
    int M, heads;
    const int32_t *row_pos, *row_seq;  // a row sees the positions up to its own
    const float* bias;       // [heads][reach + 1] by distance (the last one for all beyond), times log2 e; or null
    int reach;
    int window, keep_first;  // window > 0: a row at position p sees the positions above p - window and those below keep_first
    int chunk;               // > 0: a row at position p sees the positions from p / chunk * chunk on
    const float* talk;       // [heads][heads] or null: the scores that the softmax gets are this matrix times the heads' scores
    const float* sink;       // [heads] or null: one more score in the denominator (not scaled, as it is in the softmax)
    const float* gate;       // results are multiplied by the sigmoid of gate [M][ld_gate] (per element, or per head)
    int ld_gate, gate_kind;  // OutGate
    float out_scale;         // and by this (0: not)
    int ld_out, out_off;     // row stride and first element of the results in `out` or the image (ld_out 0: heads * vdim)
    GqaRuns runs;            // rows and heads of a run share a CTA
    int longest_run, longest;  // rows of the longest run, tokens of the longest context
    int early;               // every row is its own sequence and the pages in front of its newest token were complete before the launch in front began
    int max_cluster;
    float* out;              // [M][heads * vdim], or, when xp is given, the activation image of the next tensor-core projection
    unsigned char* xp;
    int xp_mpad;
    int* err_flag;
    int nsplit;              // CTAs that share a tile's context; 0: as many as suit the launch
    // filled in by the launcher
    int tiles, tiles_per_row, stages;
};
cudaError_t launch_gqa_attn(const GqaAttnArgs& a, int sm_count, cudaStream_t st, bool pdl);
// Whether heads that mix their scores fit the kernels (all heads of a row share a CTA).
bool gqa_talk_fits(int heads, int dim, int vdim);
// Positions [0, len) of a sequence as f32 [kv_heads][len][dim] and [kv_heads][len][vdim].
cudaError_t launch_gqa_read(const GqaPool& pool, int seq, int len, float* k, float* v, cudaStream_t st);

}  // namespace hm
