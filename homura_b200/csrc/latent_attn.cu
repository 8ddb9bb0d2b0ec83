// Attention over latents (see latent_attn.h).
//
//   latent_write_kernel      RMSNorm of the new latents and their page slots
//   latent_attn_kernel       CUDA cores, f32 or bf16 pages, any rank up to 1024: exact f32 arithmetic
//   latent_attn_tc_kernel    bf16 pages on the 5th-generation tensor cores, prompts and decoding alike
//   latent_merge_kernel      combines the splits of long contexts
//
// Tensor-core kernel.  The token axis is the MMA's M in both contractions, so that one copy of a tile of latents in shared
// memory serves as keys and values and nothing is transposed in memory:
//   scores  S^T [128 tokens x pairs] = C [128 x rank]   (K-major A, the tile as stored)  * Q^T
//   result  O^T [rank x pairs]      += C^T [rank x 128] (MN-major A, the same bytes)     * P^T
// The MMA's N holds the (row, head) pairs of the CTA three times: queries and weights stay f32 in effect, split into three
// bf16 terms (exact to 2^-24), and the three column groups are added when an accumulator is read back.  Rows of a prompt
// that follow one another share a CTA (each masks the tokens behind its own position); a decoded token is a tile of one row.
// Warp 0 copies pages into a ring of 128-element slices, warp 1 issues the MMAs, warps 2-9 turn scores into weights.  The
// reference maximum of a pair moves only when a score exceeds it by more than 2^8 (the weights then still fit), so the
// accumulators are almost never rescaled.
#include "latent_attn.h"

#include "latent_post.cuh"
#include "launch_attrs.h"
#include "mbarrier.cuh"

namespace hm {
namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float latent_load(const void* page, size_t off, int bf16) {
    return bf16 ? bf16_bits_to_f32(reinterpret_cast<const uint16_t*>(page)[off]) : reinterpret_cast<const float*>(page)[off];
}

__global__ void __launch_bounds__(128) latent_write_kernel(const LatentPool pool, const float* __restrict__ c, int ldc, const float* __restrict__ w, float eps, const int32_t* __restrict__ row_pos, const int32_t* __restrict__ row_seq) {
    __shared__ float part[4];
    pdl_launch_dependents();
    pdl_wait();
    latent_write_row<128, false>(pool, c, ldc, blockIdx.x, w, eps, row_pos, row_seq, 0, nullptr, part);
}

__global__ void latent_read_kernel(const LatentPool pool, int seq, int len, float* out) {
    const size_t total = (size_t)len * pool.rank;
    for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const int t = (int)(i / pool.rank), r = (int)(i % pool.rank);
        const size_t page = (size_t)pool.page_table[(size_t)seq * pool.max_pages + t / LATENT_PAGE] * latent_page_elems(pool.rank, pool.bf16);
        out[i] = latent_load(pool.pages, page + latent_page_off(t % LATENT_PAGE, r, pool.rank, pool.bf16), pool.bf16);
    }
}

__device__ __forceinline__ void put_result(const LatentAttnArgs& a, int m, int h, int r, float v) {
    if (a.xp) tc_xpack_store(a.xp + (size_t)h * a.xp_bytes, a.xp_mpad, m, r, v);
    else a.out[(size_t)m * a.ldo + (size_t)h * a.pool.rank + r] = v;
}

// ---- CUDA cores: a CTA takes one row, eight heads and one split ---------------------------------
constexpr int CC_HEADS = 8, CC_TOK = 32;

__host__ __device__ __forceinline__ int cc_stride(int rank) { return (((rank + 3) / 4) | 1) * 4; }  // an odd number of 16-byte pieces: no bank conflicts across tokens

template <int NC>
__global__ void __launch_bounds__(256) latent_attn_kernel(const LatentAttnArgs a) {
    extern __shared__ __align__(16) float cc_smem[];
    const int R = a.pool.rank, LD = cc_stride(R), R4 = (R + 3) / 4 * 4;
    float* qs = cc_smem;                    // [8][LD]
    float* cs = qs + CC_HEADS * LD;         // [32][LD]
    __shared__ __align__(16) float ps[CC_TOK][CC_HEADS];
    __shared__ float s_scale[CC_HEADS], s_l[CC_HEADS];
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x, h0 = blockIdx.y * CC_HEADS, split = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nh = min(CC_HEADS, a.heads - h0);
    const int len = a.row_pos[m] + 1, from = a.window > 0 ? max(0, len - a.window) : 0, first = from / CC_TOK;
    const int tiles = (len + CC_TOK - 1) / CC_TOK, per = (tiles - first + a.nsplit - 1) / a.nsplit;
    const int t0 = first + split * per, t1 = min(tiles, t0 + per);
    for (int i = tid; i < CC_HEADS * LD; i += 256) {
        const int h = i / LD, r = i % LD;
        qs[i] = h < nh && r < R ? ld_cg_f32(a.q + (size_t)m * a.ldq + (size_t)(h0 + h) * R + r) : 0.f;
    }
    float acc[NC][CC_HEADS];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int h = 0; h < CC_HEADS; ++h) acc[c][h] = 0.f;
    float mx = -INFINITY, l = 0.f;  // of head `warp`, the same in all lanes
    const int32_t* table = a.pool.page_table + (size_t)a.row_seq[m] * a.pool.max_pages;
    for (int t = t0; t < t1; ++t) {
        __syncthreads();
        const int tok0 = t * CC_TOK;
        const size_t page = (size_t)table[tok0 / LATENT_PAGE] * latent_page_elems(R, a.pool.bf16);
        for (int i = tid; i < CC_TOK * R4; i += 256) {
            const int tk = i / R4, r = i % R4;
            cs[tk * LD + r] = tok0 + tk < len && r < R ? latent_load(a.pool.pages, page + latent_page_off((tok0 + tk) % LATENT_PAGE, r, R, a.pool.bf16), a.pool.bf16) : 0.f;
        }
        __syncthreads();
        {
            float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
            const float4* q4 = reinterpret_cast<const float4*>(qs + warp * LD);
            const float4* c4 = reinterpret_cast<const float4*>(cs + lane * LD);
            for (int i = 0; i < R4 / 4; ++i) {
                const float4 q = q4[i], c = c4[i];
                s0 = fmaf(q.x, c.x, s0); s1 = fmaf(q.y, c.y, s1); s2 = fmaf(q.z, c.z, s2); s3 = fmaf(q.w, c.w, s3);
            }
            const float s = tok0 + lane < len && tok0 + lane >= from ? ((s0 + s1) + (s2 + s3)) * a.scale * LOG2E : -INFINITY;
            const float nm = fmaxf(mx, warp_max(s));  // finite: a tile holds at least one visible token
            const float p = exp2f(s - nm), f = exp2f(mx - nm);
            l = l * f + warp_sum(p);
            mx = nm;
            ps[lane][warp] = p;
            if (lane == 0) s_scale[warp] = f;
        }
        __syncthreads();
        float f[CC_HEADS];
#pragma unroll
        for (int h = 0; h < CC_HEADS; ++h) f[h] = s_scale[h];
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int h = 0; h < CC_HEADS; ++h) acc[c][h] *= f[h];
        for (int tk = 0; tk < CC_TOK; ++tk) {
            const float4 p0 = *reinterpret_cast<const float4*>(&ps[tk][0]), p1 = *reinterpret_cast<const float4*>(&ps[tk][4]);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const int r = tid + c * 256;
                const float v = r < R ? cs[tk * LD + r] : 0.f;
                acc[c][0] = fmaf(p0.x, v, acc[c][0]); acc[c][1] = fmaf(p0.y, v, acc[c][1]); acc[c][2] = fmaf(p0.z, v, acc[c][2]); acc[c][3] = fmaf(p0.w, v, acc[c][3]);
                acc[c][4] = fmaf(p1.x, v, acc[c][4]); acc[c][5] = fmaf(p1.y, v, acc[c][5]); acc[c][6] = fmaf(p1.z, v, acc[c][6]); acc[c][7] = fmaf(p1.w, v, acc[c][7]);
            }
        }
    }
    if (lane == 0) {
        s_l[warp] = l;
        if (a.nsplit > 1 && warp < nh) {
            float* ml = a.part_ml + (((size_t)m * a.heads + h0 + warp) * a.nsplit + split) * 2;
            ml[0] = mx;
            ml[1] = l;
        }
    }
    __syncthreads();
#pragma unroll
    for (int h = 0; h < CC_HEADS; ++h) {
        if (h >= nh) break;
        const float inv = 1.0f / s_l[h];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const int r = tid + c * 256;
            if (r >= R) continue;
            if (a.nsplit == 1) put_result(a, m, h0 + h, r, acc[c][h] * inv);
            else if (t1 > t0) a.part_acc[(((size_t)m * a.heads + h0 + h) * a.nsplit + split) * R + r] = acc[c][h];
        }
    }
}

__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentAttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x, h = blockIdx.y, r = blockIdx.z * 128 + threadIdx.x, R = a.pool.rank;
    const size_t base = ((size_t)m * a.heads + h) * a.nsplit;
    __shared__ float w[256];
    for (int s = threadIdx.x; s < a.nsplit; s += 128) w[s] = ld_cg_f32(a.part_ml + (base + s) * 2);
    __syncthreads();
    float mx = -INFINITY;
    for (int s = 0; s < a.nsplit; ++s) mx = fmaxf(mx, w[s]);
    __syncthreads();
    for (int s = threadIdx.x; s < a.nsplit; s += 128) w[s] = exp2f(w[s] - mx);  // a split that saw nothing: 0
    __syncthreads();
    if (r >= R) return;
    float acc = 0.f, l = 0.f;
#pragma unroll 8
    for (int s = 0; s < a.nsplit; ++s) {
        const float f = w[s];
        if (f > 0.f) {
            l = fmaf(f, ld_cg_f32(a.part_ml + (base + s) * 2 + 1), l);
            acc = fmaf(f, ld_cg_f32(a.part_acc + (base + s) * R + r), acc);
        }
    }
    put_result(a, m, h, r, acc / l);
}

// ---- tensor cores -----------------------------------------------------------------------------
constexpr int TCL_SWARPS = 8, TCL_STHREADS = 32 * TCL_SWARPS, TCL_THREADS = 64 + TCL_STHREADS, TCL_TERMS = 3;  // SWARPS: score warps, two per quarter of the tensor memory's lanes
constexpr int TCL_PAIR_SMEM = 113 * 1024 - 2048;  // dynamic shared memory with which two CTAs share an SM (2 KB static and 1 KB of the system's each)
constexpr int TCL_MAXSTG = 12, TCL_MAXPAIRS = 64;
constexpr float TCL_SLACK = 8.f;  // base-2 exponent by which a score may exceed the reference maximum

// Shared-memory operand descriptors, 128-byte swizzle, version 1.  K-major: groups of 8 rows 1024 B apart.  MN-major: pieces of
// 64 elements along MN `lbo` bytes apart, groups of 8 along K 1024 B apart.  Only the lower word depends on the address: the
// issuing thread steps through a tile by adding to it.
__device__ __forceinline__ uint32_t desc_lo(uint32_t addr, uint32_t lbo) { return ((addr >> 4) & 0x3FFF) | ((lbo >> 4) << 16); }
constexpr uint32_t DESC_HI = (1024u >> 4) | (1u << 14) | (2u << 29);
// f32 accumulator, bf16 operands; A transposed (MN-major) on request
__device__ __forceinline__ uint32_t idesc_bf16(int m, int n, int a_mn) { return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)a_mn << 15) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24); }
__device__ __forceinline__ void mma_bf16(uint32_t d, uint32_t a_lo, uint32_t b_lo, uint32_t idesc, bool accumulate) {
    asm volatile("{ .reg .pred p; .reg .b64 da, db; setp.ne.b32 p, %5, 0; mov.b64 da, {%1, %4}; mov.b64 db, {%2, %4};\n"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p; }" ::"r"(d), "r"(a_lo), "r"(b_lo), "r"(idesc), "n"(DESC_HI), "r"((uint32_t)accumulate) : "memory");
}
__device__ __forceinline__ void mma_commit(uint64_t* bar) { asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(s32(bar)) : "memory"); }
__device__ __forceinline__ void tmem_ld16(uint32_t addr, uint32_t (&r)[16]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(addr));
}
__device__ __forceinline__ void tmem_ld8(uint32_t addr, uint32_t (&r)[8]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(addr));
}
__device__ __forceinline__ void tmem_st16(uint32_t addr, const uint32_t (&r)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
                 "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
                 : "memory");
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void fence_async_smem() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }
__device__ __forceinline__ uint32_t elect_lane() {
    uint32_t p;
    asm volatile("{ .reg .pred P; .reg .b32 r; elect.sync r|P, 0xffffffff; selp.u32 %0, 1, 0, P; }" : "=r"(p));
    return p;
}
// barrier of the score warps with an OR over their predicates
__device__ __forceinline__ bool wbar_or(bool v) {
    __syncwarp();
    uint32_t r;
    asm volatile("{ .reg .pred p, q; setp.ne.u32 p, %1, 0; bar.red.or.pred q, 1, 256, p; selp.u32 %0, 1, 0, q; }" : "=r"(r) : "r"((uint32_t)v) : "memory");
    return r != 0;
}
struct TclGeom {
    int tok;       // tokens per tile: 128, or 64 for latents so wide that two tiles of 128 do not fit the ring
    int np;        // pairs, padded to 16
    int n;         // MMA N = 3 * np
    int nb;        // 128-element slices of a latent
    int kbs;       // 64-element blocks of a latent
    int stages;
    int look;      // scores of the next tile are issued before the weights of this one are ready (two score accumulators)
    int cols;      // TMEM columns, a power of two
    int pad;       // bytes by which the ring's second tile moves up to the end of the first, whose last slice is half full (rings of two tiles)
    int q_bytes, p_bytes, s_bytes;
    size_t smem;
    __host__ __device__ int slice() const { return 2 * tok * 128; }  // bytes of 128 elements of a tile's tokens: two K-major halves
};

bool tcl_geom_tok(int tok, int rank, int pairs, TclGeom* g) {
    g->tok = tok;
    g->np = (pairs + 15) / 16 * 16;
    if (g->np < 16 || g->np > TCL_MAXPAIRS) return false;
    g->n = TCL_TERMS * g->np;
    g->kbs = latent_rank_pad(rank) / 64;
    g->nb = (g->kbs + 1) / 2;
    g->q_bytes = g->kbs * g->n * 128;
    g->p_bytes = 2 * (tok / 64) * g->n * 128;  // the weights of two tiles
    g->s_bytes = g->np * (tok + 32) * 4;  // scores, and every lane's share of the sums
    const int fixed = g->q_bytes + g->p_bytes + g->s_bytes + 1024;
    g->stages = (222 * 1024 - fixed) / g->slice();
    if (g->stages > TCL_MAXSTG) g->stages = TCL_MAXSTG;
    g->pad = 0;
    if ((g->kbs & 1) && g->stages == 2 * g->nb - 1 && 2 * g->nb <= TCL_MAXSTG && g->kbs * g->slice() + fixed <= 222 * 1024) {
        g->stages = 2 * g->nb;
        g->pad = g->slice() / 2;
    }
    if (g->stages < (g->nb > 2 ? g->nb : 2)) return false;  // the values of a tile are needed after its scores: the ring holds a whole tile
    g->look = g->stages >= 2 * g->nb && (g->nb + 2) * g->n <= 512 ? 1 : 0;
    const int need = (g->nb + 1 + g->look) * g->n;
    if (need > 512) return false;
    g->cols = 32;
    while (g->cols < need) g->cols *= 2;
    // two CTAs per SM where their tensor memory and a ring of two tiles and a slice allow it
    const int pair = (TCL_PAIR_SMEM - fixed) / g->slice();
    if (g->look && g->pad == 0 && g->cols <= 256 && pair >= 2 * g->nb) g->stages = pair < TCL_MAXSTG ? pair : TCL_MAXSTG;
    g->smem = (size_t)fixed + (size_t)g->stages * g->slice() - g->pad;
    return true;
}
bool tcl_geom(int rank, int pairs, TclGeom* g) {
    if (tcl_geom_tok(128, rank, pairs, g) && g->look) return true;
    if (tcl_geom_tok(64, rank, pairs, g) && g->look) return true;
    return tcl_geom_tok(128, rank, pairs, g) || tcl_geom_tok(64, rank, pairs, g);
}

struct TclShared {
    uint64_t full[TCL_MAXSTG], empty[TCL_MAXSTG], s_full[2], p_full, pv_done[2], q_full;
    uint32_t tmem;
    volatile int abort_flag;
    float ref[TCL_MAXPAIRS], sum[TCL_MAXPAIRS], alpha[TCL_MAXPAIRS];
    int pos[TCL_MAXPAIRS];  // last visible position of the pair's row; -1: padding
    int row[TCL_MAXPAIRS], head[TCL_MAXPAIRS];
};

template <int TOK>
__global__ void __launch_bounds__(TCL_THREADS, 2) latent_attn_tc_kernel(const LatentAttnArgs a, const TclGeom g, int heads_per_cta) {
    extern __shared__ __align__(1024) unsigned char tcl_smem[];
    __shared__ TclShared sh;
    constexpr int SLICE = 2 * TOK * 128, PAGES = TOK / LATENT_PAGE, SLD = TOK, TPL = TOK / 32;  // bytes, pages per tile, score row, tokens per lane
    unsigned char* ring = tcl_smem + ((1024u - (s32(tcl_smem) & 1023u)) & 1023u);
    auto stage_at = [&](int s) { return (uint32_t)s * SLICE - (s >= g.nb ? (uint32_t)g.pad : 0u); };  // bytes from the ring's front
    unsigned char* qs = ring + stage_at(g.stages);         // [kbs][n][128 B]
    unsigned char* pb = qs + g.q_bytes;                    // [2][TOK / 64][n][128 B]
    float* sc = reinterpret_cast<float*>(pb + g.p_bytes);  // [np][SLD]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h0 = blockIdx.y * heads_per_cta, split = blockIdx.z;
    const int nh = min(heads_per_cta, a.heads - h0), R = a.pool.rank;
    // The pass's rows cut into tiles: a tile starts at every multiple of rows_per_tile and wherever a run starts.  Every warp
    // finds this CTA's tile, the blockIdx.x-th, on its own (the rows of a pass never change within it).
    int m0 = blockIdx.x, rows = 1;
    if (a.rows_per_tile > 1) {
        uint64_t starts = 0;
        for (int i = 0; i < a.M; i += 32) {
            const int m = i + lane;
            const bool st = m < a.M && (m % a.rows_per_tile == 0 || a.row_seq[m - 1] != a.row_seq[m] || a.row_pos[m - 1] + 1 != a.row_pos[m]);
            starts |= (uint64_t)__ballot_sync(0xffffffffu, st) << i;
        }
        if (a.M < 64) starts |= (uint64_t)1 << a.M;  // end mark
        for (int i = 0; i < (int)blockIdx.x && starts; ++i) starts &= starts - 1;
        m0 = starts ? __ffsll((long long)starts) - 1 : a.M;
        if (m0 >= a.M) return;  // fewer tiles than CTAs
        const uint64_t after = starts & (starts - 1);
        rows = (after ? __ffsll((long long)after) - 1 : a.M) - m0;
    }
    const int seq = a.row_seq[m0], pos0 = a.row_pos[m0];
    const int pairs = rows * nh;  // pair p: row p / nh, head p % nh
    const int from = a.window > 0 ? max(0, pos0 - a.window + 1) : 0;  // first position that the tile's first row sees
    const int len = pos0 + rows, tiles = (len + TOK - 1) / TOK, per = (tiles - from / TOK + a.nsplit - 1) / a.nsplit;
    const int t0 = from / TOK + split * per, nt = min(tiles, t0 + per) - t0;
    if (nt <= 0) {  // only with nsplit > 1
        pdl_launch_dependents();
        pdl_wait();  // the launch in front may still be reading this buffer
        for (int p = tid; p < pairs; p += TCL_THREADS) {
            float* ml = a.part_ml + (((size_t)(m0 + p / nh) * a.heads + h0 + p % nh) * a.nsplit + split) * 2;
            ml[0] = -INFINITY;
            ml[1] = 0.f;
        }
        return;
    }
    if (tid == 0) {
        for (int s = 0; s < g.stages; ++s) {
            mb_init(&sh.full[s], 1);
            mb_init(&sh.empty[s], 1);
        }
        mb_init(&sh.s_full[0], 1);
        mb_init(&sh.s_full[1], 1);
        mb_init(&sh.p_full, TCL_STHREADS);
        mb_init(&sh.pv_done[0], 1);
        mb_init(&sh.pv_done[1], 1);
        mb_init(&sh.q_full, TCL_STHREADS);
        sh.abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    for (int p = tid; p < g.np; p += TCL_THREADS) {
        sh.pos[p] = p < pairs ? pos0 + p / nh : -1;
        sh.row[p] = m0 + p / nh;
        sh.head[p] = h0 + p % nh;
        sh.ref[p] = -INFINITY;
    }
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(s32(&sh.tmem)), "r"(g.cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sh.tmem, tmem_o = tmem + (uint32_t)((1 + g.look) * g.n);
    pdl_launch_dependents();

    if (warp == 0) {
        if (lane == 0) {
            const int32_t* table = a.pool.page_table + (size_t)seq * a.pool.max_pages;
            const int npages = (len + LATENT_PAGE - 1) / LATENT_PAGE;
            const int settled = a.early ? pos0 / LATENT_PAGE : 0;  // pages in front of the one that gets this step's latent
            constexpr uint32_t piece = LATENT_PAGE * 128;
            const unsigned char* pool = reinterpret_cast<const unsigned char*>(a.pool.pages);
            // a tile's last page may lie behind the context: the last one of the context stands in (masked, but finite)
            auto page_of = [&](int t, int i) { return table[min(PAGES * t + i, npages - 1)]; };
            int next[PAGES];
#pragma unroll
            for (int i = 0; i < PAGES; ++i) next[i] = page_of(t0, i);
            int s = 0, it = 0;
            uint32_t phase = 1;  // of the stage's empty barrier; its first round needs no wait
            bool ok = true, waited = false;
            for (int t = 0; t < nt && ok; ++t) {
                int cur[PAGES];
#pragma unroll
                for (int i = 0; i < PAGES; ++i) cur[i] = next[i];
                if (t + 1 < nt)
#pragma unroll
                    for (int i = 0; i < PAGES; ++i) next[i] = page_of(t0 + t + 1, i);
                if (!waited && PAGES * (t0 + t + 1) > settled) {
                    pdl_wait();
                    waited = true;
                }
                for (int b = 0; b < g.nb; ++b, ++it) {
                    if (it >= g.stages && !mb_wait(&sh.empty[s], phase, a.err_flag, &sh.abort_flag)) { ok = false; break; }
                    const int halves = min(2, g.kbs - 2 * b);
                    mb_expect_tx(&sh.full[s], (uint32_t)halves * PAGES * piece);
                    for (int hf = 0; hf < halves; ++hf)
#pragma unroll
                        for (int i = 0; i < PAGES; ++i)
                            bulk_copy(ring + stage_at(s) + hf * (SLICE / 2) + i * piece, pool + ((size_t)cur[i] * g.kbs + 2 * b + hf) * piece, piece, &sh.full[s]);
                    if (++s == g.stages) {
                        s = 0;
                        phase ^= 1;
                    }
                }
            }
            if (!waited) pdl_wait();
        }
    } else if (warp == 1) {
        // The whole warp runs this in step, so that the addresses and stage counters live in uniform registers; one elected lane
        // issues (a lane that runs alone takes twice as long per MMA).
        const uint32_t lead = elect_lane();
        const uint32_t base = __shfl_sync(0xffffffffu, tmem, 0), base_o = base + (uint32_t)((1 + g.look) * g.n);
        const uint32_t id_s = idesc_bf16(TOK, g.n, 0), id_o = idesc_bf16(128, g.n, 1);
        const uint32_t qlo = desc_lo(s32(qs), 16), plo = desc_lo(s32(pb), 16), klo = desc_lo(s32(ring), 16), vlo = desc_lo(s32(ring), SLICE / 2);
        const uint32_t row_block = (uint32_t)g.n * 128 / 16;  // one 64-element block of Q or P, in descriptor units
        auto ready = [&](uint64_t* bar, uint32_t parity) { return __any_sync(0xffffffffu, mb_test(bar, parity)) != 0; };
        bool ok = __any_sync(0xffffffffu, mb_wait(&sh.q_full, 0, a.err_flag, &sh.abort_flag)) != 0;
        int ks_stage = 0, pv_stage = 0, ks_slice = 0, ks_tile = 0;
        uint32_t ks_phase = 0, q = qlo;
        for (int t = 0; t < nt && ok; ++t) {
            // Whatever is ready first: a slice of this tile (of the next one too, with two score accumulators) or this tile's
            // weights, whose product frees the ring for the tile after next.
            const int upto = g.look ? min(nt, t + 2) : t + 1;
            bool pv = false;
            unsigned long long spins = 0;
            while (!pv) {
                if (ks_tile > t && ready(&sh.p_full, t & 1)) {
                    tc_fence_after();
                    uint32_t d = base_o;
                    const uint32_t p = plo + (uint32_t)(t & 1) * (TOK / 64) * row_block;
                    for (int b = 0; b < g.nb; ++b, d += g.n) {
                        const uint32_t v = vlo + stage_at(pv_stage) / 16;
                        if (lead) {
#pragma unroll
                            for (int ks = 0; ks < TOK / 16; ++ks) mma_bf16(d, v + ks * 128, p + (ks >> 2) * row_block + (ks & 3) * 2, id_o, t > 0 || ks > 0);
                            mma_commit(&sh.empty[pv_stage]);
                        }
                        __syncwarp();
                        if (++pv_stage == g.stages) pv_stage = 0;
                    }
                    if (lead) mma_commit(&sh.pv_done[t & 1]);
                    __syncwarp();
                    pv = true;
                } else if (ks_tile < upto && ready(&sh.full[ks_stage], ks_phase)) {
                    // scores of one slice; the last slice of a tile publishes the tile's scores
                    tc_fence_after();
                    const uint32_t d = base + (g.look ? (uint32_t)((ks_tile & 1) * g.n) : 0u), k = klo + stage_at(ks_stage) / 16;
                    const bool two = 2 * ks_slice + 1 < g.kbs;
                    if (lead) {
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks) mma_bf16(d, k + ks * 2, q + ks * 2, id_s, ks_slice > 0 || ks > 0);
                        if (two)
#pragma unroll
                            for (int ks = 0; ks < 4; ++ks) mma_bf16(d, k + SLICE / 2 / 16 + ks * 2, q + row_block + ks * 2, id_s, true);
                    }
                    __syncwarp();
                    q += two ? 2 * row_block : row_block;
                    if (++ks_stage == g.stages) {
                        ks_stage = 0;
                        ks_phase ^= 1;
                    }
                    if (++ks_slice == g.nb) {
                        if (lead) mma_commit(&sh.s_full[ks_tile & 1]);
                        __syncwarp();
                        ks_slice = 0;
                        ++ks_tile;
                        q = qlo;
                    }
                    spins = 0;
                } else if (__any_sync(0xffffffffu, sh.abort_flag != 0) || ++spins > MB_SPIN_LIMIT) {
                    if (lane == 0 && !sh.abort_flag && a.err_flag) atomicExch(a.err_flag, 2);
                    sh.abort_flag = 1;
                    ok = false;
                    break;
                }
            }
        }
    } else {
        const int wt = tid - 64, ww = wt >> 5, half = ww >> 2;  // half: which eight of every 16 accumulator columns this warp reads
        const int lane_base = (warp & 3) * 32;  // the quarter of the TMEM lanes this warp may touch
        const uint32_t lane_addr = (uint32_t)lane_base << 16;
        // the token of a score accumulator's lane: M = 128 fills all lanes, M = 64 the first 16 of every quarter
        const bool has_tok = TOK == 128 || lane < 16;
        const int my_tok = TOK == 128 ? lane_base + lane : (warp & 3) * 16 + lane;
        float* ls = sc + (size_t)g.np * SLD;  // [np][32]: every lane's share of the pairs' sums
        for (int i = wt; i < g.np * 32; i += TCL_STHREADS) ls[i] = 0.f;
        pdl_wait();
        // queries: f32 rows -> three bf16 terms, K-major rows term * np + pair, 16-byte pieces XOR-ed by row & 7; four pieces of a
        // thread are requested before the first is used
        const int pieces = g.kbs * 8, items = g.np * pieces;
        const bool vec = ((R | a.ldq) & 3) == 0 && (reinterpret_cast<uintptr_t>(a.q) & 15) == 0;
        for (int base = wt; base < items; base += 4 * TCL_STHREADS) {
            float v[4][8];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int i = base + u * TCL_STHREADS, p = i / pieces, r = (i % pieces) * 8;
                const bool ok = i < items && p < pairs;
                const float* src = a.q + (ok ? (size_t)sh.row[p] * a.ldq + (size_t)sh.head[p] * R + r : 0);
                if (vec) {
                    const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
                    const float4 x = ok && r + 4 <= R ? ld_cg_f32x4(src) : z, y = ok && r + 8 <= R ? ld_cg_f32x4(src + 4) : z;
                    v[u][0] = x.x; v[u][1] = x.y; v[u][2] = x.z; v[u][3] = x.w; v[u][4] = y.x; v[u][5] = y.y; v[u][6] = y.z; v[u][7] = y.w;
                } else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) v[u][e] = ok && r + e < R ? ld_cg_f32(src + e) : 0.f;
                }
            }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int i = base + u * TCL_STHREADS;
                if (i < items) tc_xpack_store8(qs, g.np, i / pieces, (i % pieces) * 8, v[u]);  // the image layout of the projections' activations: [block][term][np][64]
            }
        }
        fence_async_smem();
        mb_arrive(&sh.q_full);
        const float scale2 = a.scale * LOG2E;
        bool bad = false;
        for (int t = 0; t < nt; ++t) {
            bad = !mb_wait(&sh.s_full[t & 1], (t >> 1) & 1, a.err_flag, &sh.abort_flag);
            __syncwarp();
            tc_fence_after();
            const uint32_t s_addr = tmem + lane_addr + (g.look ? (uint32_t)((t & 1) * g.n) : 0u);
            for (int c0 = half * 8; c0 < g.np; c0 += 16) {
                uint32_t r[TCL_TERMS][8];
#pragma unroll
                for (int k = 0; k < TCL_TERMS; ++k) tmem_ld8(s_addr + k * g.np + c0, r[k]);
                tmem_ld_wait();
                if (has_tok)
#pragma unroll
                    for (int j = 0; j < 8; ++j) sc[(c0 + j) * SLD + my_tok] = ((__uint_as_float(r[2][j]) + __uint_as_float(r[1][j])) + __uint_as_float(r[0][j])) * scale2;
                __syncwarp();
            }
            tc_fence_before();
            // this tile's weights go where those of two tiles ago were: their product must be done
            bad |= t > 1 && !mb_wait(&sh.pv_done[t & 1], ((t >> 1) - 1) & 1, a.err_flag, &sh.abort_flag);
            if (wbar_or(bad)) { bad = true; break; }
            unsigned char* pt = pb + (size_t)(t & 1) * (TOK / 64) * g.n * 128;
            const int tok = (t0 + t) * TOK + lane * TPL;
            const bool whole = (t0 + t + 1) * TOK - 1 <= pos0 && (a.window == 0 || (t0 + t) * TOK > len - 1 - a.window);  // every row sees every token of the tile
            bool moved = false;
            for (int c0 = 0; c0 < g.np; c0 += 16) {
                // two pairs per warp side by side
                float s[2][TPL], ref[2];
                bool grow = t == 0;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int p = c0 + ww + 8 * j;
                    if (TPL == 4) {
                        const float4 v = *reinterpret_cast<const float4*>(sc + p * SLD + lane * 4);
                        s[j][0] = v.x; s[j][1] = v.y; s[j][TPL - 2] = v.z; s[j][TPL - 1] = v.w;
                    } else {
                        const float2 v = *reinterpret_cast<const float2*>(sc + p * SLD + lane * 2);
                        s[j][0] = v.x; s[j][1] = v.y;
                    }
                    ref[j] = sh.ref[p];
                    if (!whole) {
                        const int last = sh.pos[p], before = a.window > 0 ? last - a.window : -1;
#pragma unroll
                        for (int e = 0; e < TPL; ++e)
                            if (tok + e > last || tok + e <= before) s[j][e] = -INFINITY;
                    }
#pragma unroll
                    for (int e = 0; e < TPL; ++e) grow |= s[j][e] > ref[j] + TCL_SLACK;
                }
                float al[2] = {1.f, 1.f};
                const bool any = __any_sync(0xffffffffu, grow);
                if (any) {
                    float mx[2];
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mx[j] = s[j][0];
#pragma unroll
                        for (int e = 1; e < TPL; ++e) mx[j] = fmaxf(mx[j], s[j][e]);
                    }
#pragma unroll
                    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                        for (int j = 0; j < 2; ++j) mx[j] = fmaxf(mx[j], __shfl_xor_sync(0xffffffffu, mx[j], o));
#pragma unroll
                    for (int j = 0; j < 2; ++j)
                        if (mx[j] > (t == 0 ? ref[j] : ref[j] + TCL_SLACK)) {
                            if (t > 0) al[j] = exp2f(ref[j] - mx[j]);
                            ref[j] = mx[j];
                            moved |= t > 0;
                        }
                }
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int p = c0 + ww + 8 * j;
                    float w[TPL], sum = 0.f;
#pragma unroll
                    for (int e = 0; e < TPL; ++e) {
                        w[e] = s[j][e] == -INFINITY ? 0.f : exp2f(s[j][e] - ref[j]);
                        sum += w[e];
                    }
                    ls[p * 32 + lane] = ls[p * 32 + lane] * al[j] + sum;
                    uint32_t q[TCL_TERMS][TPL / 2];
#pragma unroll
                    for (int e = 0; e < TPL / 2; ++e) bf16x2_split3(w[2 * e], w[2 * e + 1], q[0][e], q[1][e], q[2][e]);
                    // this lane's tokens of row term * np + p: 64-token block, 16-byte piece XOR-ed by row & 7, place in the piece
                    const int tk = lane * TPL;
                    unsigned char* blk = pt + (size_t)(tk >> 6) * g.n * 128 + (tk & 7) * 2;
#pragma unroll
                    for (int k = 0; k < TCL_TERMS; ++k) {
                        const int row = k * g.np + p;
                        unsigned char* dst = blk + (size_t)row * 128 + ((((tk & 63) >> 3) ^ (row & 7)) << 4);
                        if (TPL == 4) *reinterpret_cast<uint2*>(dst) = make_uint2(q[k][0], q[k][TPL / 2 - 1]);
                        else *reinterpret_cast<uint32_t*>(dst) = q[k][0];
                    }
                }
                __syncwarp();
                if (any && lane == 0)
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        sh.ref[c0 + ww + 8 * j] = ref[j];
                        sh.alpha[c0 + ww + 8 * j] = al[j];
                    }
                else if (lane == 0)
#pragma unroll
                    for (int j = 0; j < 2; ++j) sh.alpha[c0 + ww + 8 * j] = 1.f;
                __syncwarp();
            }
            if (wbar_or(moved)) {
                // the accumulators are rescaled once the tile in front has been added
                bad = !mb_wait(&sh.pv_done[(t - 1) & 1], ((t - 1) >> 1) & 1, a.err_flag, &sh.abort_flag);
                if (wbar_or(bad)) { bad = true; break; }
                tc_fence_after();
                for (int b = half; b < g.nb; b += 2)
                    for (int c0 = 0; c0 < g.n; c0 += 16) {
                        uint32_t r[16];
                        const uint32_t addr = tmem_o + lane_addr + (uint32_t)(b * g.n + c0);
                        tmem_ld16(addr, r);
                        tmem_ld_wait();
#pragma unroll
                        for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * sh.alpha[(c0 + j) % g.np]);
                        tmem_st16(addr, r);
                    }
                tmem_st_wait();
            }
            tc_fence_before();
            fence_async_smem();
            mb_arrive(&sh.p_full);
        }
        if (!bad) {
            for (int p = ww; p < g.np; p += TCL_SWARPS) {
                const float sum = warp_sum(ls[p * 32 + lane]);
                if (lane == 0) sh.sum[p] = a.nsplit == 1 ? 1.0f / sum : sum;
            }
            bad = !mb_wait(&sh.pv_done[(nt - 1) & 1], ((nt - 1) >> 1) & 1, a.err_flag, &sh.abort_flag);
        }
        if (!wbar_or(bad)) {
            tc_fence_after();
            if (a.nsplit > 1)
                for (int p = wt; p < pairs; p += TCL_STHREADS) {
                    float* ml = a.part_ml + (((size_t)sh.row[p] * a.heads + sh.head[p]) * a.nsplit + split) * 2;
                    ml[0] = sh.ref[p];
                    ml[1] = sh.sum[p];
                }
            for (int b = 0; b < g.nb; ++b) {
                const int r0 = b * 128 + lane_base + lane;
                for (int c0 = half * 8; c0 < g.np; c0 += 16) {
                    uint32_t r[TCL_TERMS][8];
#pragma unroll
                    for (int k = 0; k < TCL_TERMS; ++k) tmem_ld8(tmem_o + lane_addr + (uint32_t)(b * g.n + k * g.np + c0), r[k]);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 8; ++j) {
                        const int p = c0 + j;
                        if (p < pairs && r0 < R) {
                            const float v = (__uint_as_float(r[2][j]) + __uint_as_float(r[1][j])) + __uint_as_float(r[0][j]);
                            if (a.nsplit == 1) put_result(a, sh.row[p], sh.head[p], r0, v * sh.sum[p]);
                            else a.part_acc[(((size_t)sh.row[p] * a.heads + sh.head[p]) * a.nsplit + split) * R + r0] = v;
                        }
                    }
                    __syncwarp();
                }
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(g.cols) : "memory");
}

template <typename... KArgs, typename... Args>
cudaError_t launch(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, bool pdl, Args... args) {
    cudaError_t e = ensure_dyn_smem(kern, smem);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kern, KArgs(args)...);
}

// heads per CTA: all of them when they fit one tile, else equal shares of at most the tile's pairs
int tcl_heads(int heads, int max_pairs) {
    const int groups = (heads + max_pairs - 1) / max_pairs;
    return (heads + groups - 1) / groups;
}

}  // namespace

int latent_tc_pairs(int rank, int bf16) {
    if (!bf16) return 0;
    TclGeom g;
    for (int p = TCL_MAXPAIRS; p >= 16; p -= 16)
        if (tcl_geom(rank, p, &g)) return p;
    return 0;
}

// Rows share a CTA where that costs no MMA columns (16 pairs), and up to 32 pairs where the contexts are long enough for the
// re-read latents to matter more than the CTAs that are lost (measured: 64 pairs are slower at every length).
int latent_rows_per_tile(int longest_run, int longest, int heads, int rank, int bf16) {
    int mp = latent_tc_pairs(rank, bf16);
    if (mp == 0 || longest_run < 2) return 1;
    const int hpc = tcl_heads(heads, mp), fill = longest >= 4096 ? 32 : 16;
    if (mp > fill) mp = fill;
    int r = mp / hpc;
    if (r > longest_run) r = longest_run;
    return r < 1 ? 1 : r;
}

int latent_pick_nsplit(int tiles, int rows_per_tile, int heads, int rank, int bf16, int longest, int sm_count, int max_split, bool free_merge) {
    const int mp = latent_tc_pairs(rank, bf16);
    const int hpc = mp ? tcl_heads(heads, mp) : CC_HEADS, ctas = tiles * ((heads + hpc - 1) / hpc);
    TclGeom g;
    const bool tc = mp > 0 && tcl_geom(rank, rows_per_tile * hpc, &g);
    const int tok = tc ? g.tok : CC_TOK, most = (longest + tok - 1) / tok;
    const int slots = tc && g.smem <= TCL_PAIR_SMEM && g.cols <= 256 ? 2 * sm_count : sm_count;  // CTAs resident at once
    int s = slots / (ctas > 0 ? ctas : 1);
    if (s > most) s = most;
    if (s > max_split) s = max_split;
    if (s > 256) s = 256;
    if (tc && most < 4 && !free_merge) s = 1;  // the merge launch costs as much as three tiles
    return s < 1 ? 1 : s;
}

cudaError_t launch_latent_write(const LatentPool& pool, const float* c, int ldc, int M, const float* w, float eps, const int32_t* row_pos, const int32_t* row_seq, cudaStream_t st, bool pdl) {
    return launch(latent_write_kernel, dim3(M), dim3(128), 0, st, pdl, pool, c, ldc, w, eps, row_pos, row_seq);
}

cudaError_t launch_latent_read(const LatentPool& pool, int seq, int len, float* out, cudaStream_t st) {
    const size_t n = ((size_t)len * pool.rank + 255) / 256;
    latent_read_kernel<<<(unsigned)(n < 1 ? 1 : n > 2048 ? 2048 : n), 256, 0, st>>>(pool, seq, len, out);
    return cudaGetLastError();
}

cudaError_t launch_latent_attn(const LatentAttnArgs& a_in, cudaStream_t st, bool pdl, int* launches) {
    LatentAttnArgs a = a_in;
    const int R = a.pool.rank, mp = latent_tc_pairs(R, a.pool.bf16);
    if (R < 1 || a.M < 1 || (mp > 0 && a.rows_per_tile > 1 && a.M > 64) || a.tiles < 0 || a.tiles > a.M || a.heads < 1 || a.nsplit < 1 || a.nsplit > 256) return cudaErrorInvalidValue;
    cudaError_t e;
    if (mp > 0) {
        const int hpc = tcl_heads(a.heads, mp);
        TclGeom g;
        if (a.rows_per_tile < 1) a.rows_per_tile = 1;
        if (a.rows_per_tile == 1) a.tiles = a.M;
        if (!tcl_geom(R, a.rows_per_tile * hpc, &g)) return cudaErrorInvalidValue;
        const dim3 grid(a.tiles > 0 ? a.tiles : a.M, (a.heads + hpc - 1) / hpc, a.nsplit);
        e = g.tok == 128 ? launch(latent_attn_tc_kernel<128>, grid, dim3(TCL_THREADS), g.smem, st, pdl, a, g, hpc) : launch(latent_attn_tc_kernel<64>, grid, dim3(TCL_THREADS), g.smem, st, pdl, a, g, hpc);
    } else {
        const size_t smem = (size_t)(CC_HEADS + CC_TOK) * cc_stride(R) * 4;
        const dim3 grid(a.M, (a.heads + CC_HEADS - 1) / CC_HEADS, a.nsplit);
        if (R <= 256) e = launch(latent_attn_kernel<1>, grid, dim3(256), smem, st, pdl, a);
        else if (R <= 512) e = launch(latent_attn_kernel<2>, grid, dim3(256), smem, st, pdl, a);
        else if (R <= 1024) e = launch(latent_attn_kernel<4>, grid, dim3(256), smem, st, pdl, a);
        else return cudaErrorInvalidValue;
    }
    if (e != cudaSuccess) return e;
    ++*launches;
    if (a.nsplit > 1 && !a.unmerged) {
        e = launch(latent_merge_kernel, dim3(a.M, a.heads, (R + 127) / 128), dim3(128), 0, st, pdl, a);
        if (e == cudaSuccess) ++*launches;
    }
    return e;
}

}  // namespace hm
