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
// Warp 0 copies pages into a ring of 128-element slices, warp 1 issues the MMAs, warps 2-5 turn scores into weights.  The
// reference maximum of a pair moves only when a score exceeds it by more than 2^8 (the weights then still fit), so the
// accumulators are almost never rescaled.
#include "latent_attn.h"

#include "launch_attrs.h"
#include "mbarrier.cuh"

namespace hm {
namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float latent_load(const void* page, size_t off, int bf16) {
    return bf16 ? bf16_bits_to_f32(reinterpret_cast<const uint16_t*>(page)[off]) : reinterpret_cast<const float*>(page)[off];
}

__global__ void __launch_bounds__(128) latent_write_kernel(const LatentPool pool, const float* __restrict__ c, int ldc, const float* __restrict__ w, float eps, const int32_t* __restrict__ row_pos, const int32_t* __restrict__ row_seq) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x, tid = threadIdx.x, lane = tid & 31, R = pool.rank;
    const float* x = c + (size_t)m * ldc;
    float s = 0.f;
    for (int i = tid; i < R; i += 128) {
        const float v = ld_cg_f32(x + i);
        s = fmaf(v, v, s);
    }
    __shared__ float sw[4];
    s = warp_sum(s);
    if (lane == 0) sw[tid >> 5] = s;
    __syncthreads();
    const float inv = 1.0f / sqrtf((sw[0] + sw[1] + sw[2] + sw[3]) / (float)R + eps);
    const int pos = row_pos[m];
    const size_t page = (size_t)pool.page_table[(size_t)row_seq[m] * pool.max_pages + pos / LATENT_PAGE] * latent_page_elems(R, pool.bf16);
    for (int i = tid; i < R; i += 128) {
        const float v = (ld_cg_f32(x + i) * inv) * __ldg(w + i);
        const size_t off = page + latent_page_off(pos % LATENT_PAGE, i, R, pool.bf16);
        if (pool.bf16) reinterpret_cast<uint16_t*>(pool.pages)[off] = f32_to_bf16_rne(v);
        else reinterpret_cast<float*>(pool.pages)[off] = v;
    }
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
    const int len = a.row_pos[m] + 1, tiles = (len + CC_TOK - 1) / CC_TOK, per = (tiles + a.nsplit - 1) / a.nsplit;
    const int t0 = split * per, t1 = min(tiles, t0 + per);
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
            const float s = tok0 + lane < len ? ((s0 + s1) + (s2 + s3)) * a.scale * LOG2E : -INFINITY;
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
constexpr int TCL_THREADS = 192, TCL_TOK = 128, TCL_TERMS = 3, TCL_SLICE = 2 * TCL_TOK * 128;  // a slice: 128 elements of 128 tokens, two K-major halves of 16 KB
constexpr int TCL_MAXSTG = 8, TCL_MAXPAIRS = 64;
constexpr float TCL_SLACK = 8.f;  // base-2 exponent by which a score may exceed the reference maximum

// Shared-memory operand descriptors, 128-byte swizzle, version 1.  K-major: groups of 8 rows 1024 B apart.  MN-major: pieces of
// 64 elements along MN `lbo` bytes apart, groups of 8 along K 1024 B apart.
__device__ __forceinline__ uint64_t desc_sw128(uint32_t addr, uint32_t lbo) {
    return (uint64_t)((addr >> 4) & 0x3FFF) | ((uint64_t)(lbo >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}
// f32 accumulator, bf16 operands, M = 128; A transposed (MN-major) on request
__device__ __forceinline__ uint32_t idesc_bf16(int n, int a_mn) { return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)a_mn << 15) | ((uint32_t)(n >> 3) << 17) | (8u << 24); }
__device__ __forceinline__ void mma_bf16(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
    asm volatile("{ .reg .pred p; setp.ne.b32 p, %4, 0;\n"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }" ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate) : "memory");
}
__device__ __forceinline__ void mma_commit(uint64_t* bar) { asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(s32(bar)) : "memory"); }
__device__ __forceinline__ void tmem_ld16(uint32_t addr, uint32_t (&r)[16]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
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
// barrier of the four weight warps with an OR over their predicates
__device__ __forceinline__ bool wbar_or(bool v) {
    __syncwarp();
    uint32_t r;
    asm volatile("{ .reg .pred p, q; setp.ne.u32 p, %1, 0; bar.red.or.pred q, 1, 128, p; selp.u32 %0, 1, 0, q; }" : "=r"(r) : "r"((uint32_t)v) : "memory");
    return r != 0;
}
__device__ __forceinline__ void split3(float x, uint16_t& h, uint16_t& m, uint16_t& l) {
    h = f32_to_bf16_rne(x);
    const float r = x - bf16_bits_to_f32(h);
    m = f32_to_bf16_rne(r);
    l = f32_to_bf16_rne(r - bf16_bits_to_f32(m));
}

struct TclGeom {
    int np;        // pairs, padded to 16
    int n;         // MMA N = 3 * np
    int nb;        // 128-element slices of a latent
    int kbs;       // 64-element blocks of a latent
    int stages;
    int look;      // scores of the next tile are issued before the weights of this one are ready (two score accumulators)
    int cols;      // TMEM columns, a power of two
    int q_bytes, p_bytes, s_bytes;
    size_t smem;
};

bool tcl_geom(int rank, int pairs, TclGeom* g) {
    g->np = (pairs + 15) / 16 * 16;
    if (g->np < 16 || g->np > TCL_MAXPAIRS) return false;
    g->n = TCL_TERMS * g->np;
    g->kbs = latent_rank_pad(rank) / 64;
    g->nb = (g->kbs + 1) / 2;
    g->q_bytes = g->kbs * g->n * 128;
    g->p_bytes = 2 * g->n * 128;
    g->s_bytes = g->np * (TCL_TOK + 4) * 4;
    const int room = 224 * 1024 - (g->q_bytes + g->p_bytes + g->s_bytes + 1024);
    g->stages = room / TCL_SLICE;
    if (g->stages > TCL_MAXSTG) g->stages = TCL_MAXSTG;
    if (g->stages < (g->nb > 2 ? g->nb : 2)) return false;  // the values of a tile are needed after its scores: the ring holds a whole tile
    g->look = g->stages >= 2 * g->nb && (g->nb + 2) * g->n <= 512 ? 1 : 0;
    const int need = (g->nb + 1 + g->look) * g->n;
    if (need > 512) return false;
    g->cols = 32;
    while (g->cols < need) g->cols *= 2;
    g->smem = (size_t)g->q_bytes + g->p_bytes + g->s_bytes + (size_t)g->stages * TCL_SLICE + 1024;
    return true;
}

struct TclShared {
    uint64_t full[TCL_MAXSTG], empty[TCL_MAXSTG], s_full[2], p_full, pv_done, q_full;
    uint32_t tmem;
    volatile int abort_flag;
    float ref[TCL_MAXPAIRS], sum[TCL_MAXPAIRS], alpha[TCL_MAXPAIRS];
    int pos[TCL_MAXPAIRS];  // last visible position of the pair's row; -1: padding
};

__global__ void __launch_bounds__(TCL_THREADS, 1) latent_attn_tc_kernel(const LatentAttnArgs a, const TclGeom g, int heads_per_cta) {
    extern __shared__ __align__(1024) unsigned char tcl_smem[];
    __shared__ TclShared sh;
    unsigned char* ring = tcl_smem + ((1024u - (s32(tcl_smem) & 1023u)) & 1023u);
    unsigned char* qs = ring + (size_t)g.stages * TCL_SLICE;  // [kbs][n][128 B]
    unsigned char* pb = qs + g.q_bytes;                       // [2][n][128 B]
    float* sc = reinterpret_cast<float*>(pb + g.p_bytes);     // [np][132]
    constexpr int SLD = TCL_TOK + 4;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h0 = blockIdx.y * heads_per_cta, split = blockIdx.z;
    const int nh = min(heads_per_cta, a.heads - h0), R = a.pool.rank;
    // The pass's rows cut into tiles: a tile starts at every multiple of rows_per_tile and wherever a run starts.  Every warp
    // finds this CTA's tile, the blockIdx.x-th, on its own (the rows of a pass never change within it).
    uint64_t starts = 0;
    for (int i = 0; i < a.M; i += 32) {
        const int m = i + lane;
        const bool st = m < a.M && (m % a.rows_per_tile == 0 || a.row_seq[m - 1] != a.row_seq[m] || a.row_pos[m - 1] + 1 != a.row_pos[m]);
        starts |= (uint64_t)__ballot_sync(0xffffffffu, st) << i;
    }
    if (a.M < 64) starts |= (uint64_t)1 << a.M;  // end mark
    for (int i = 0; i < (int)blockIdx.x && starts; ++i) starts &= starts - 1;
    const int m0 = starts ? __ffsll((long long)starts) - 1 : a.M;
    if (m0 >= a.M) return;  // fewer tiles than CTAs
    const uint64_t after = starts & (starts - 1);
    const int rows = (after ? __ffsll((long long)after) - 1 : a.M) - m0;
    const int seq = a.row_seq[m0], pos0 = a.row_pos[m0];
    const int pairs = rows * nh;  // pair p: row p / nh, head p % nh
    const int len = pos0 + rows, tiles = (len + TCL_TOK - 1) / TCL_TOK, per = (tiles + a.nsplit - 1) / a.nsplit;
    const int t0 = split * per, nt = min(tiles, t0 + per) - t0;
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
        mb_init(&sh.p_full, 128);
        mb_init(&sh.pv_done, 1);
        mb_init(&sh.q_full, 128);
        sh.abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    for (int p = tid; p < g.np; p += TCL_THREADS) {
        sh.pos[p] = p < pairs ? pos0 + p / nh : -1;
        sh.ref[p] = -INFINITY;
        sh.sum[p] = 0.f;
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
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            const int32_t* table = a.pool.page_table + (size_t)seq * a.pool.max_pages;
            const int npages = (len + LATENT_PAGE - 1) / LATENT_PAGE;
            const uint32_t piece = LATENT_PAGE * 128;
            const unsigned char* pool = reinterpret_cast<const unsigned char*>(a.pool.pages);
            // a tile's second page may lie behind the context: its first page stands in (masked, but finite)
            auto page_of = [&](int t, int i) { return table[min(2 * t + i, npages - 1)]; };
            int pg0 = page_of(t0, 0), pg1 = page_of(t0, 1);
            int it = 0;
            bool ok = true;
            for (int t = 0; t < nt && ok; ++t) {
                const int c0 = pg0, c1 = pg1;
                if (t + 1 < nt) {
                    pg0 = page_of(t0 + t + 1, 0);
                    pg1 = page_of(t0 + t + 1, 1);
                }
                for (int b = 0; b < g.nb; ++b, ++it) {
                    const int s = it % g.stages;
                    if (it >= g.stages && !mb_wait(&sh.empty[s], ((it / g.stages) & 1) ^ 1, a.err_flag, &sh.abort_flag)) { ok = false; break; }
                    const int halves = min(2, g.kbs - 2 * b);
                    mb_expect_tx(&sh.full[s], (uint32_t)halves * 2 * piece);
                    for (int hf = 0; hf < halves; ++hf) {
                        unsigned char* dst = ring + (size_t)s * TCL_SLICE + hf * (TCL_SLICE / 2);
                        const size_t kb = (size_t)(2 * b + hf);
                        bulk_copy(dst, pool + ((size_t)c0 * g.kbs + kb) * piece, piece, &sh.full[s]);
                        bulk_copy(dst + piece, pool + ((size_t)c1 * g.kbs + kb) * piece, piece, &sh.full[s]);
                    }
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t id_s = idesc_bf16(g.n, 0), id_o = idesc_bf16(g.n, 1);
            const uint32_t q0 = s32(qs), p0 = s32(pb), r0 = s32(ring);
            bool ok = mb_wait(&sh.q_full, 0, a.err_flag, &sh.abort_flag);
            tc_fence_after();
            auto scores = [&](int t) {
                const uint32_t d = tmem + (g.look ? (uint32_t)((t & 1) * g.n) : 0u);
                for (int b = 0; b < g.nb; ++b) {
                    const int it = t * g.nb + b, s = it % g.stages;
                    if (!mb_wait(&sh.full[s], (it / g.stages) & 1, a.err_flag, &sh.abort_flag)) return false;
                    tc_fence_after();
                    const int halves = min(2, g.kbs - 2 * b);
                    for (int hf = 0; hf < halves; ++hf)
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks)
                            mma_bf16(d, desc_sw128(r0 + s * TCL_SLICE + hf * (TCL_SLICE / 2) + ks * 32, 16), desc_sw128(q0 + (2 * b + hf) * g.n * 128 + ks * 32, 16), id_s, (b | hf | ks) ? 1u : 0u);
                }
                mma_commit(&sh.s_full[t & 1]);
                return true;
            };
            if (ok && g.look) ok = scores(0);
            for (int t = 0; t < nt && ok; ++t) {
                if (!g.look) ok = scores(t);
                else if (t + 1 < nt) ok = scores(t + 1);
                if (!ok || !mb_wait(&sh.p_full, t & 1, a.err_flag, &sh.abort_flag)) break;
                tc_fence_after();
                for (int b = 0; b < g.nb; ++b) {
                    const int s = (t * g.nb + b) % g.stages;
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks)
                        mma_bf16(tmem_o + b * g.n, desc_sw128(r0 + s * TCL_SLICE + ks * 2048, TCL_SLICE / 2), desc_sw128(p0 + (ks >> 2) * g.n * 128 + (ks & 3) * 32, 16), id_o, (t | ks) ? 1u : 0u);
                    mma_commit(&sh.empty[s]);
                }
                mma_commit(&sh.pv_done);
            }
        }
    } else {
        const int wt = tid - 64, ww = wt >> 5;
        const int lane_base = (warp & 3) * 32;  // the quarter of the TMEM lanes this warp may touch
        const uint32_t lane_addr = (uint32_t)lane_base << 16;
        // queries: f32 rows -> three bf16 terms, K-major rows term * np + pair, 16-byte pieces XOR-ed by row & 7
        for (int i = wt; i < g.np * g.kbs * 8; i += 128) {
            const int p = i / (g.kbs * 8), c = i % (g.kbs * 8), r = c * 8;
            float v[8];
            const float* src = a.q + (size_t)(m0 + p / nh) * a.ldq + (size_t)(h0 + p % nh) * R + r;
            const bool vec = p < pairs && r + 8 <= R && (reinterpret_cast<uintptr_t>(src) & 15) == 0;
            if (vec) {
                const float4 x = ld_cg_f32x4(src), y = ld_cg_f32x4(src + 4);
                v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = p < pairs && r + e < R ? ld_cg_f32(src + e) : 0.f;
            }
            tc_xpack_store8(qs, g.np, p, r, v);  // the image layout of the projections' activations: [block][term][np][64]
        }
        fence_async_smem();
        mb_arrive(&sh.q_full);
        const float scale2 = a.scale * LOG2E;
        bool bad = false;
        for (int t = 0; t < nt; ++t) {
            bad = !mb_wait(&sh.s_full[t & 1], (t >> 1) & 1, a.err_flag, &sh.abort_flag);
            if (wbar_or(bad)) { bad = true; break; }
            tc_fence_after();
            const uint32_t s_addr = tmem + lane_addr + (g.look ? (uint32_t)((t & 1) * g.n) : 0u);
            for (int c0 = 0; c0 < g.np; c0 += 16) {
                uint32_t r[TCL_TERMS][16];
#pragma unroll
                for (int k = 0; k < TCL_TERMS; ++k) tmem_ld16(s_addr + k * g.np + c0, r[k]);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 16; ++j) sc[(c0 + j) * SLD + lane_base + lane] = (__uint_as_float(r[2][j]) + __uint_as_float(r[1][j])) + __uint_as_float(r[0][j]);
            }
            tc_fence_before();
            // the weights of the tile in front must have been consumed before theirs are overwritten (and before O is rescaled)
            bad = t > 0 && !mb_wait(&sh.pv_done, (t - 1) & 1, a.err_flag, &sh.abort_flag);
            if (wbar_or(bad)) { bad = true; break; }
            tc_fence_after();
            const int tok = (t0 + t) * TCL_TOK + lane * 4;
            bool moved = false;
            for (int p = ww; p < g.np; p += 4) {
                const float4 s4 = *reinterpret_cast<const float4*>(sc + p * SLD + lane * 4);
                const int last = sh.pos[p];
                float s[4] = {s4.x, s4.y, s4.z, s4.w}, mx = -INFINITY;
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s[e] = tok + e <= last ? s[e] * scale2 : -INFINITY;
                    mx = fmaxf(mx, s[e]);
                }
                mx = warp_max(mx);
                float ref = sh.ref[p], al = 1.f;
                if (mx > (t == 0 ? ref : ref + TCL_SLACK)) {
                    al = t == 0 ? 1.f : exp2f(ref - mx);
                    ref = mx;
                }
                float sum = 0.f;
                uint16_t w[TCL_TERMS][4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float v = s[e] == -INFINITY ? 0.f : exp2f(s[e] - ref);
                    sum += v;
                    split3(v, w[0][e], w[1][e], w[2][e]);
                }
                sum = warp_sum(sum);
                __syncwarp();
                if (lane == 0) {
                    sh.ref[p] = ref;
                    sh.sum[p] = sh.sum[p] * al + sum;
                    sh.alpha[p] = al;
                }
                moved |= al != 1.f;
                // tokens lane*4 .. +3 of row term * np + p: block lane / 16, 16-byte piece (lane % 16) / 2, half of it
                unsigned char* blk = pb + (size_t)(lane >> 4) * g.n * 128;
#pragma unroll
                for (int k = 0; k < TCL_TERMS; ++k) {
                    const int row = k * g.np + p;
                    *reinterpret_cast<uint2*>(blk + (size_t)row * 128 + ((((lane & 15) >> 1) ^ (row & 7)) << 4) + (lane & 1) * 8) =
                        make_uint2((uint32_t)w[k][0] | ((uint32_t)w[k][1] << 16), (uint32_t)w[k][2] | ((uint32_t)w[k][3] << 16));
                }
            }
            if (wbar_or(moved)) {
                for (int b = 0; b < g.nb; ++b)
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
        if (!bad) bad = !mb_wait(&sh.pv_done, (nt - 1) & 1, a.err_flag, &sh.abort_flag);
        if (!wbar_or(bad)) {
            tc_fence_after();
            if (a.nsplit > 1)
                for (int p = wt; p < pairs; p += 128) {
                    float* ml = a.part_ml + (((size_t)(m0 + p / nh) * a.heads + h0 + p % nh) * a.nsplit + split) * 2;
                    ml[0] = sh.ref[p];
                    ml[1] = sh.sum[p];
                }
            for (int b = 0; b < g.nb; ++b) {
                const int r0 = b * 128 + lane_base + lane;
                for (int c0 = 0; c0 < g.np; c0 += 16) {
                    uint32_t r[TCL_TERMS][16];
#pragma unroll
                    for (int k = 0; k < TCL_TERMS; ++k) tmem_ld16(tmem_o + lane_addr + (uint32_t)(b * g.n + k * g.np + c0), r[k]);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        const int p = c0 + j;
                        if (p < pairs && r0 < R) {
                            const float v = (__uint_as_float(r[2][j]) + __uint_as_float(r[1][j])) + __uint_as_float(r[0][j]);
                            const int m = m0 + p / nh, h = h0 + p % nh;
                            if (a.nsplit == 1) put_result(a, m, h, r0, v / sh.sum[p]);
                            else a.part_acc[(((size_t)m * a.heads + h) * a.nsplit + split) * R + r0] = v;
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

int latent_rows_per_tile(int M, int heads, int rank, int bf16) {
    const int mp = latent_tc_pairs(rank, bf16);
    if (mp == 0 || M < 2) return 1;
    const int r = mp / tcl_heads(heads, mp);
    return r < 1 ? 1 : r;
}

int latent_pick_nsplit(int tiles, int heads, int rank, int bf16, int longest, int sm_count, int max_split) {
    const int mp = latent_tc_pairs(rank, bf16);
    const int hg = mp ? (heads + tcl_heads(heads, mp) - 1) / tcl_heads(heads, mp) : (heads + CC_HEADS - 1) / CC_HEADS;
    const int ctas = tiles * hg;
    const int tok = mp ? TCL_TOK : CC_TOK;
    int s = sm_count / (ctas > 0 ? ctas : 1);
    const int most = (longest + tok - 1) / tok;
    if (s > most) s = most;
    if (s > max_split) s = max_split;
    if (s > 256) s = 256;
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
    if (R < 1 || a.M < 1 || (mp > 0 && a.M > 64) || a.tiles < 0 || a.tiles > a.M || a.heads < 1 || a.nsplit < 1 || a.nsplit > 256) return cudaErrorInvalidValue;
    cudaError_t e;
    if (mp > 0) {
        const int hpc = tcl_heads(a.heads, mp);
        a.rows_per_tile = latent_rows_per_tile(a.M, a.heads, R, a.pool.bf16);
        TclGeom g;
        const int rows = a.rows_per_tile < a.M ? a.rows_per_tile : a.M;
        if (!tcl_geom(R, rows * hpc, &g)) return cudaErrorInvalidValue;
        e = launch(latent_attn_tc_kernel, dim3(a.tiles > 0 ? a.tiles : a.M, (a.heads + hpc - 1) / hpc, a.nsplit), dim3(TCL_THREADS), g.smem, st, pdl, a, g, hpc);
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
    if (a.nsplit > 1) {
        e = launch(latent_merge_kernel, dim3(a.M, a.heads, (R + 127) / 128), dim3(128), 0, st, pdl, a);
        if (e == cudaSuccess) ++*launches;
    }
    return e;
}

}  // namespace hm
