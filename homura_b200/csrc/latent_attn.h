// Attention over a paged cache of latents: one vector of `rank` elements per token serves as key and value of every head
// (latent_attn.cu).  The caller has multiplied the queries with the up-projection of the keys and multiplies the result with
// that of the values, so that only latents are read per token.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "common.cuh"

namespace hm {

constexpr int LATENT_PAGE = 64;  // tokens per page

// One layer's pool.  f32 pages: rows [64][rank].  bf16 pages: [rank_pad / 64][64 tokens][64] with the 16-byte pieces of a
// token's 128-byte row XOR-ed by token & 7 (rank_pad = rank rounded up to 64, the tail zero): every 8 KB block is the
// shared-memory image of a tensor-core operand.
struct LatentPool {
    void* pages;
    const int32_t* page_table;  // [sequences][max_pages]
    int max_pages;
    int rank;
    int bf16;
};
__host__ __device__ __forceinline__ int latent_rank_pad(int rank) { return (rank + 63) & ~63; }
__host__ __device__ __forceinline__ size_t latent_page_elems(int rank, int bf16) { return (size_t)LATENT_PAGE * (bf16 ? latent_rank_pad(rank) : rank); }
__host__ __device__ __forceinline__ size_t latent_page_off(int t, int r, int rank, int bf16) {
    return bf16 ? (size_t)(r >> 6) * (LATENT_PAGE * 64) + (size_t)t * 64 + ((((r & 63) >> 3) ^ (t & 7)) << 3) + (r & 7) : (size_t)t * rank + r;
}

struct LatentAttnArgs {
    LatentPool pool;
    const float* q;          // [M][ldq]: query of (row, head) at head * rank
    int ldq;
    int M, heads;
    const int32_t* row_pos;  // a row sees positions <= its own
    const int32_t* row_seq;
    float scale;
    int window;              // > 0: a row at position p sees the positions above p - window only
    int rows_per_tile;       // latent_rows_per_tile: rows of one run (consecutive positions of a sequence) that may share a CTA
    int tiles;               // with rows_per_tile > 1 (at most 64 rows then): tiles the rows fall into, 0: not known
    int unmerged;            // leave the splits in part_acc / part_ml (the caller's next kernel combines them)
    int early;               // every row is its own sequence and the pages in front of its newest token were complete before the launch in front began
    int nsplit;
    float* part_acc;         // [M][heads][nsplit][rank], with nsplit > 1
    float* part_ml;          // [M][heads][nsplit][2]: running maximum (of base-2 exponents) and sum
    float* out;              // [M][ldo]: result of (row, head) at head * rank; or, when xp is given,
    int ldo;
    unsigned char* xp;       // activation images of a grouped tensor-core projection, one per head, xp_bytes apart
    int xp_mpad;
    size_t xp_bytes;
    int* err_flag;
};

// c rows [M][ldc] -> RMSNorm over rank with weight w -> the page slot of every row's position.
cudaError_t launch_latent_write(const LatentPool& pool, const float* c, int ldc, int M, const float* w, float eps, const int32_t* row_pos, const int32_t* row_seq, cudaStream_t st, bool pdl);
// Positions [0, len) of a sequence as f32 rows.
cudaError_t launch_latent_read(const LatentPool& pool, int seq, int len, float* out, cudaStream_t st);

// Largest (row, head) pair count a tensor-core CTA takes for this rank; 0: the kernel does not cover it (or the pages are f32).
int latent_tc_pairs(int rank, int bf16);
// Rows of a run that share a CTA, in a pass whose longest run has so many rows and whose longest context so many tokens.
int latent_rows_per_tile(int longest_run, int longest, int heads, int rank, int bf16);
// Splits of the longest context (in tokens) so that a pass of so many tiles fills the SMs; at most max_split.
int latent_pick_nsplit(int tiles, int rows_per_tile, int heads, int rank, int bf16, int longest, int sm_count, int max_split, bool free_merge);
cudaError_t launch_latent_attn(const LatentAttnArgs& a, cudaStream_t st, bool pdl, int* launches);

}  // namespace hm
