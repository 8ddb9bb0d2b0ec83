// Grouped-query attention for listed designs.
//
//   gqa_post_kernel        norms, temperature and blending of a projection's queries, keys and values; page slots
//   gqa_attn_kernel        CUDA cores, f32 or bf16 pages, any head size
//   gqa_attn_mma_kernel    bf16 pages on warp-level MMAs, prompts and decoding alike
//   talk_attn_mma_kernel   the same where the heads mix their scores (gqa_talk.cuh)
//
// MMA kernel.  A CTA serves a tile of (row, query head) pairs of one key/value head: the heads of a decoded token, or the heads of
// several rows of a prompt that follow one another, so that a page is read once for all of them.  Pages come through a ring of
// bulk copies (one contiguous block of keys and one of values per page and head).  Every warp takes units of 16 tokens:
//   scores^T [16 tokens x pairs] = K [16 x dim]      . Q^T        (K chunks through ldmatrix)
//   out^T    [vdim x pairs]     += V^T [vdim x 16]   . P^T        (V chunks through ldmatrix, transposed)
// Queries and weights are three bf16 terms each (exact to 2^-24), so that the products are f32 x bf16 ones.  The warps of a CTA add
// their results up in shared memory; the CTAs of a cluster share the context of a tile and send one another their pairs' results by
// asynchronous stores.
#include "gqa_attn.h"

#include <algorithm>
#include <map>
#include <mutex>
#include <tuple>

#include "gqa_post.cuh"
#include "launch_attrs.h"
#include "mbarrier.cuh"
#include "model_spec.h"

namespace hm {
namespace {

constexpr int ATT_WARPS = 8;
constexpr int A_THREADS = 256;
constexpr int B_THREADS = ATT_WARPS * 32 + 32;
constexpr int MAX_STAGES = 8;
constexpr int MAX_CLUSTER = 16;

// ---- after the projection ------------------------------------------------------------------------
template <int X>
__global__ void __launch_bounds__(POST_WARPS * 32) gqa_post_kernel(const GqaPostArgs a) {
    extern __shared__ __align__(16) float post_sm[];
    pdl_launch_dependents();
    gqa_post_block<X>(a, blockIdx.x, blockIdx.y, post_sm);
}

__global__ void gqa_read_kernel(const GqaPool pool, int seq, int len, float* __restrict__ k, float* __restrict__ v) {
    const int D = pool.dim + pool.vdim;
    const size_t total = (size_t)pool.kv_heads * len * D;
    for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const int e = (int)(i % D), t = (int)(i / D % len), g = (int)(i / D / len);
        const bool is_k = e < pool.dim;
        const int d = is_k ? e : e - pool.dim, n = is_k ? pool.dim : pool.vdim;
        const size_t off = (size_t)pool.page_table[(size_t)seq * pool.max_pages + t / GQA_PAGE] * gqa_page_elems(pool.kv_heads, n) + (size_t)g * GQA_PAGE * gqa_pad(n) + gqa_tile_off(t % GQA_PAGE, d);
        const void* src = is_k ? pool.k : pool.v;
        (is_k ? k : v)[((size_t)g * len + t) * n + d] = pool.bf16 ? bf16_bits_to_f32(reinterpret_cast<const uint16_t*>(src)[off]) : reinterpret_cast<const float*>(src)[off];
    }
}

// ---- common to both attention kernels --------------------------------------------------------------
// X: the variant with windows, sinks, gates and results that share their rows with others'.
template <bool X>
__device__ __forceinline__ void store_piece(const GqaAttnArgs& a, int m, int head, int d0, float (&v)[8]) {
    const int vdim = a.pool.vdim, e0 = head * vdim + d0, off = X ? a.out_off : 0, k0 = off + e0, ld = X ? a.ld_out : a.heads * vdim;
    if (X && a.gate_kind != GATE_NONE) {
        const float* g = a.gate + (size_t)m * a.ld_gate;
        if (a.gate_kind == GATE_ELEM && d0 + 8 <= vdim && (reinterpret_cast<uintptr_t>(g + e0) & 15) == 0) {
            const float4 x = ld_cg_f32x4(g + e0), y = ld_cg_f32x4(g + e0 + 4);
            const float z[8] = {x.x, x.y, x.z, x.w, y.x, y.y, y.z, y.w};
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= 1.0f / (1.0f + expf(-z[i]));
        } else {
            const float all = a.gate_kind == GATE_HEAD ? 1.0f / (1.0f + expf(-ld_cg_f32(g + head))) : 1.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= a.gate_kind == GATE_HEAD ? all : d0 + i < vdim ? 1.0f / (1.0f + expf(-ld_cg_f32(g + e0 + i))) : 0.f;
        }
    }
    if (X && a.out_scale != 0.f)
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] *= a.out_scale;
    if (a.xp && ((vdim | off) & 7) == 0) {
        tc_xpack_store8(a.xp, a.xp_mpad, m, k0, v);
        return;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        if (d0 + i >= vdim) break;
        if (a.xp) tc_xpack_store(a.xp, a.xp_mpad, m, k0 + i, v[i]);
        else a.out[(size_t)m * ld + k0 + i] = v[i];
    }
}

// The sink's share of a denominator whose weights are relative to 2^mx.
template <bool X>
__device__ __forceinline__ float sink_weight(const GqaAttnArgs& a, int head, float mx) { return X && a.sink ? exp2f(fmaf(__ldg(a.sink + head), 1.4426950408889634f, -mx)) : 0.f; }

// Pages that rows at positions [lo, hi] see: those of the first tokens, then those of the window.  Page number i of the list is
// pages_skip(i): i itself in front of the gap, i + gap behind it.
struct PageList {
    int n, head, gap;
    __device__ __forceinline__ int page(int i) const { return i < head ? i : i + gap; }
};
// First position that a row at `pos` sees behind the kept ones.
__device__ __forceinline__ int first_visible(const GqaAttnArgs& a, int pos) { return a.chunk > 0 ? pos - pos % a.chunk : a.window > 0 ? max(0, pos - a.window + 1) : 0; }

template <bool X>
__device__ __forceinline__ PageList visible_pages(const GqaAttnArgs& a, int lo, int hi) {
    const int all = hi / GQA_PAGE + 1;
    PageList l{all, all, 0};
    if (X && (a.window > 0 || a.chunk > 0)) {
        const int from = first_visible(a, lo) / GQA_PAGE;  // first page of the window
        l.head = min((a.keep_first + GQA_PAGE - 1) / GQA_PAGE, from);
        l.gap = from - l.head;
        l.n = all - l.gap;
    }
    return l;
}

// Results of a CTA's pairs in its shared memory: o [pairs][ldo] (not yet divided), ml [pairs][2] (maximum as a base-2 exponent, sum).
// Splits are the CTAs of a cluster; every one of them combines and stores a share of the elements.  wts: [nsplit][pairs].
template <bool X, typename RowHead>
__device__ __forceinline__ void combine_and_store(const GqaAttnArgs& a, const float* o, int ldo, const float* ml, float* wts, int pairs, RowHead row_head) {
    const int tid = threadIdx.x, nt = blockDim.x, ns = a.nsplit;
    const int rank = ns > 1 ? (int)cluster_ctarank() : 0;
    if (ns > 1) cluster_sync_all();
    else __syncthreads();
    for (int p = tid; p < pairs; p += nt) {
        int sm_row = 0, sm_head = 0;
        if (X) row_head(p, sm_row, sm_head);
        if (ns == 1) {
            wts[p] = 1.0f / (ml[2 * p + 1] + sink_weight<X>(a, sm_head, ml[2 * p]));
            continue;
        }
        float mr[MAX_CLUSTER], lr[MAX_CLUSTER], mx = -INFINITY, l = 0.f;
#pragma unroll
        for (int r = 0; r < MAX_CLUSTER; ++r)
            if (r < ns) {
                mr[r] = ld_dsmem_f32(dsmem_addr(ml + 2 * p, (uint32_t)r));
                lr[r] = ld_dsmem_f32(dsmem_addr(ml + 2 * p + 1, (uint32_t)r));
            }
#pragma unroll
        for (int r = 0; r < MAX_CLUSTER; ++r)
            if (r < ns) mx = fmaxf(mx, mr[r]);
#pragma unroll
        for (int r = 0; r < MAX_CLUSTER; ++r)
            if (r < ns) {
                mr[r] = mr[r] == -INFINITY ? 0.f : exp2f(mr[r] - mx);
                l = fmaf(mr[r], lr[r], l);
            }
        l += sink_weight<X>(a, sm_head, mx);
#pragma unroll
        for (int r = 0; r < MAX_CLUSTER; ++r)
            if (r < ns) wts[r * pairs + p] = mr[r] / l;
    }
    __syncthreads();
    const int np = gqa_pad(a.pool.vdim) / 8;
    for (int i = rank * nt + tid; i < pairs * np; i += ns * nt) {
        const int p = i / np, d0 = (i - p * np) * 8;
        float v[8];
        if (ns == 1) {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = o[p * ldo + d0 + e] * wts[p];
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = 0.f;
#pragma unroll 4
            for (int r = 0; r < ns; ++r) {
                const float w = wts[r * pairs + p];
                const float4 x = ld_dsmem_f32x4(dsmem_addr(o + p * ldo + d0, (uint32_t)r)), y = ld_dsmem_f32x4(dsmem_addr(o + p * ldo + d0 + 4, (uint32_t)r));
                v[0] = fmaf(w, x.x, v[0]); v[1] = fmaf(w, x.y, v[1]); v[2] = fmaf(w, x.z, v[2]); v[3] = fmaf(w, x.w, v[3]);
                v[4] = fmaf(w, y.x, v[4]); v[5] = fmaf(w, y.y, v[5]); v[6] = fmaf(w, y.z, v[6]); v[7] = fmaf(w, y.w, v[7]);
            }
        }
        int m, head;
        row_head(p, m, head);
        if (d0 < a.pool.vdim) store_piece<X>(a, m, head, d0, v);
    }
    if (ns > 1) cluster_sync_all();  // nobody leaves while a peer reads its shared memory
}

// ---- CUDA cores ------------------------------------------------------------------------------------
// One CTA = one row, key/value head and split; TALK: all heads of a row and split.
template <bool BF16, bool X, bool TALK>
__global__ void __launch_bounds__(A_THREADS) gqa_attn_kernel(const GqaAttnArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int gq = a.heads / a.pool.kv_heads, g = TALK ? a.heads : gq, kvh = blockIdx.y, m = blockIdx.z, split = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int dim = a.pool.dim, vdim = a.pool.vdim, dp = gqa_pad(dim), vp = gqa_pad(vdim), ldo = vp + 4;
    float* q_s = sm;                  // [g][dp]
    float* o_s = q_s + g * dp;        // [g][ldo]
    float* p_s = o_s + g * ldo;       // [g][64]
    float* ml = p_s + g * GQA_PAGE;   // [g][2]
    float* corr = ml + 2 * g;         // [g]
    float* wts = corr + g;            // [nsplit][g]
    float* raw = TALK ? wts + a.nsplit * g : nullptr;  // [g][64] scores before they are mixed
    pdl_launch_dependents();
    pdl_wait();
    const int pos = a.row_pos[m], len = pos + 1, from = X ? first_visible(a, pos) : 0;
    auto seen = [&](int tok) { return !X || tok >= from || tok < a.keep_first; };
    const PageList list = visible_pages<X>(a, pos, pos);
    const int pps = (list.n + a.nsplit - 1) / a.nsplit, p0 = split * pps, p1 = min(list.n, p0 + pps);
    const int32_t* pt = a.pool.page_table + (size_t)a.row_seq[m] * a.pool.max_pages;
    for (int i = tid; i < g * dp; i += A_THREADS) {
        const int j = i / dp, d = i - j * dp;
        q_s[i] = d < dim ? ld_cg_f32(a.q + (size_t)m * a.heads * dim + (size_t)(kvh * g + j) * dim + d) : 0.f;
    }
    for (int i = tid; i < g * ldo; i += A_THREADS) o_s[i] = 0.f;
    for (int i = tid; i < g; i += A_THREADS) {
        ml[2 * i] = -INFINITY;
        ml[2 * i + 1] = 0.f;
    }
    __syncthreads();
    for (int pi = p0; pi < p1; ++pi) {
        const int p = list.page(pi);
        const size_t kb0 = (size_t)pt[p] * gqa_page_elems(a.pool.kv_heads, dim) + (size_t)kvh * GQA_PAGE * dp;
        const size_t vb0 = (size_t)pt[p] * gqa_page_elems(a.pool.kv_heads, vdim) + (size_t)kvh * GQA_PAGE * vp;
        const int nt = min(GQA_PAGE, len - p * GQA_PAGE);
        for (int i = tid; i < g * GQA_PAGE; i += A_THREADS) {
            const int j = i / GQA_PAGE, t = i % GQA_PAGE;
            float s = TALK ? 0.f : -INFINITY;
            if (t < nt && seen(p * GQA_PAGE + t)) {
                const float* q = q_s + j * dp;
                const size_t kb = TALK ? kb0 + (size_t)(j / gq) * GQA_PAGE * dp : kb0;
                s = 0.f;
                for (int c = 0; c < dp / 8; ++c) {
                    float k[8];
                    if (BF16) {
                        const uint4 u = __ldcg(reinterpret_cast<const uint4*>(reinterpret_cast<const uint16_t*>(a.pool.k) + kb + (size_t)(c * GQA_PAGE + t) * 8));
                        k[0] = bf16_lo(u.x); k[1] = bf16_hi(u.x); k[2] = bf16_lo(u.y); k[3] = bf16_hi(u.y);
                        k[4] = bf16_lo(u.z); k[5] = bf16_hi(u.z); k[6] = bf16_lo(u.w); k[7] = bf16_hi(u.w);
                    } else {
                        const float4* src = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(a.pool.k) + kb + (size_t)(c * GQA_PAGE + t) * 8);
                        const float4 x = __ldcg(src), y = __ldcg(src + 1);
                        k[0] = x.x; k[1] = x.y; k[2] = x.z; k[3] = x.w; k[4] = y.x; k[5] = y.y; k[6] = y.z; k[7] = y.w;
                    }
#pragma unroll
                    for (int e = 0; e < 8; ++e) s = fmaf(q[c * 8 + e], k[e], s);
                }
                if (a.bias) s += __ldg(a.bias + (size_t)(kvh * g + j) * (a.reach + 1) + min(pos - (p * GQA_PAGE + t), a.reach));
            }
            (TALK ? raw : p_s)[i] = s;
        }
        __syncthreads();
        if constexpr (TALK) {
            for (int i = tid; i < g * GQA_PAGE; i += A_THREADS) {
                const int j = i / GQA_PAGE, t = i % GQA_PAGE;
                const float* w = a.talk + (size_t)j * g;
                float s = 0.f;
                for (int e = 0; e < g; ++e) s = fmaf(__ldg(w + e), raw[e * GQA_PAGE + t], s);
                p_s[i] = t < nt && seen(p * GQA_PAGE + t) ? s : -INFINITY;
            }
            __syncthreads();
        }
        for (int j = warp; j < g; j += A_THREADS / 32) {
            const float s0 = p_s[j * GQA_PAGE + lane], s1 = p_s[j * GQA_PAGE + 32 + lane];
            const float old = ml[2 * j], mx = fmaxf(old, warp_max(fmaxf(s0, s1)));  // a page of the list has a token that is seen
            const float e0 = exp2f(s0 - mx), e1 = exp2f(s1 - mx), f = exp2f(old - mx);
            p_s[j * GQA_PAGE + lane] = e0;
            p_s[j * GQA_PAGE + 32 + lane] = e1;
            const float l = warp_sum(e0 + e1);
            __syncwarp();
            if (lane == 0) {
                ml[2 * j] = mx;
                ml[2 * j + 1] = fmaf(ml[2 * j + 1], f, l);
                corr[j] = f;
            }
        }
        __syncthreads();
        for (int i = tid; i < g * vdim; i += A_THREADS) {
            const int j = i / vdim, d = i - j * vdim;
            const size_t vb = TALK ? vb0 + (size_t)(j / gq) * GQA_PAGE * vp : vb0;
            float s = 0.f;
#pragma unroll 4
            for (int t = 0; t < nt; ++t) {
                const size_t off = vb + gqa_tile_off(t, d);
                s = fmaf(p_s[j * GQA_PAGE + t], BF16 ? bf16_bits_to_f32(__ldcg(reinterpret_cast<const uint16_t*>(a.pool.v) + off)) : __ldcg(reinterpret_cast<const float*>(a.pool.v) + off), s);
            }
            o_s[j * ldo + d] = fmaf(o_s[j * ldo + d], corr[j], s);
        }
        __syncthreads();
    }
    combine_and_store<X>(a, o_s, ldo, ml, wts, g, [&](int p, int& row, int& head) {
        row = m;
        head = kvh * g + p;
    });
}

// ---- warp-level MMAs on bf16 pages ---------------------------------------------------------------------
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ uint32_t transpose8x8(uint32_t v) {
    uint32_t r;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
    return r;
}

__host__ __device__ inline size_t b_stage_bytes(int dp, int vp) { return (size_t)GQA_PAGE * (dp + vp) * 2; }
__host__ __device__ inline size_t b_query_bytes(int nt, int dp) { return (size_t)nt * (dp / 16) * 3 * 32 * 8; }
// the ring's memory takes the warps' results afterwards: maxima, sums and values
__host__ __device__ inline size_t b_merge_bytes(int nt, int vp) { return sizeof(float) * ATT_WARPS * nt * 8 * ((size_t)2 + vp + 4); }
// what a CTA receives: from every split, its share of the pairs (values, maximum, sum)
__host__ __device__ inline size_t b_recv_bytes(int nt, int vp, int nsplit) { return sizeof(float) * (size_t)nsplit * ((nt * 8 + nsplit - 1) / nsplit) * (vp + 4); }

// VT: tiles of 16 value elements (at most), NT: tiles of eight pairs.
template <int VT, int NT, bool X>
__global__ void __launch_bounds__(B_THREADS, NT == 1 && VT <= 8 ? 2 : 1) gqa_attn_mma_kernel(const GqaAttnArgs a, size_t ring_bytes) {
    constexpr int P = NT * 8;
    extern __shared__ __align__(128) unsigned char dyn[];
    const int g = a.heads / a.pool.kv_heads, kvh = blockIdx.y, split = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int dim = a.pool.dim, vdim = a.pool.vdim, dp = gqa_pad(dim), vp = gqa_pad(vdim), kt_n = dp / 16, vt_n = vp / 16, ldo = vp + 4;
    const int NST = a.stages;
    const uint32_t k_bytes = (uint32_t)(GQA_PAGE * dp * 2), v_bytes = (uint32_t)(GQA_PAGE * vp * 2), stage = k_bytes + v_bytes;
    unsigned char* ring = dyn;
    uint2* qf = reinterpret_cast<uint2*>(dyn + ring_bytes);                                 // [NT][kt_n][3][32]
    float* recv = reinterpret_cast<float*>(dyn + ring_bytes + b_query_bytes(NT, dp));       // [nsplit][pairs of this CTA][vp + 4]
    int32_t* pt_s = reinterpret_cast<int32_t*>(dyn + ring_bytes + b_query_bytes(NT, dp) + b_recv_bytes(NT, vp, a.nsplit));  // this CTA's pages
    __shared__ uint64_t full[MAX_STAGES], empty[MAX_STAGES], s_rbar;
    __shared__ volatile int s_abort;
    __shared__ int s_pos[P], s_bias[P], s_from[X ? P : 1];  // position of the pair's row (-1: no such pair), first element of its bias row, first position it sees

    // this tile's pairs: run, first pair, rows
    int row0, rows, pair0;
    if (a.runs.n == 0) {
        row0 = blockIdx.z / a.tiles_per_row;
        rows = 1;
        pair0 = (blockIdx.z - row0 * a.tiles_per_row) * P;
    } else {
        int r = 0;
        while (r + 1 < a.runs.n && a.runs.tile[r + 1] <= blockIdx.z) ++r;
        row0 = a.runs.row[r];
        rows = a.runs.row[r + 1] - row0;
        pair0 = (blockIdx.z - a.runs.tile[r]) * P;
    }
    const int pairs = min(P, rows * g - pair0);
    // the splits of a tile share its pairs: pair p is combined and stored by split p % ns
    const int ns = a.nsplit, rank = ns > 1 ? (int)cluster_ctarank() : 0, own = pairs > rank ? (pairs - rank + ns - 1) / ns : 0, own_most = (P + ns - 1) / ns;
    if (tid == 0) {
        for (int s = 0; s < NST; ++s) {
            mb_init(&full[s], 1);
            mb_init(&empty[s], 4);
        }
        mb_init(&s_rbar, 1);
        s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        if (ns > 1 && own > 0) mb_expect_tx(&s_rbar, (uint32_t)((ns - 1) * own * (vp + 2) * 4));
    }
    pdl_launch_dependents();
    if (ns > 1) {
        cluster_arrive_release();
        cluster_wait_acquire();
    }
    if (!a.early) pdl_wait();
    const int row_hi = row0 + (pair0 + pairs - 1) / g;
    const int seq = a.row_seq[row0], len = a.row_pos[row_hi] + 1;
    const PageList list = visible_pages<X>(a, X && (a.window > 0 || a.chunk > 0) ? a.row_pos[row0 + pair0 / g] : 0, len - 1);
    auto page_at = [&](int i) { return X ? list.page(i) : i; };
    const int pps = (list.n + a.nsplit - 1) / a.nsplit;
    const int p0 = split * pps, np = max(0, min(list.n, p0 + pps) - p0);
    const int32_t* pt = a.pool.page_table + (size_t)seq * a.pool.max_pages;
    for (int i = tid; i < np; i += B_THREADS) pt_s[i] = pt[page_at(p0 + i)];
    if (tid < P) {
        const int pr = pair0 + tid;
        s_pos[tid] = tid < pairs ? a.row_pos[row0 + pr / g] : -1;
        if (X) s_from[tid] = tid < pairs ? first_visible(a, s_pos[tid]) : 0;
        s_bias[tid] = (kvh * g + (tid < pairs ? pr % g : 0)) * (a.reach + 1);
    }
    __syncthreads();
    const unsigned char *kpool = reinterpret_cast<const unsigned char*>(a.pool.k), *vpool = reinterpret_cast<const unsigned char*>(a.pool.v);
    auto fetch = [&](int i, int s) {
        const size_t tile = (size_t)pt_s[i] * a.pool.kv_heads + kvh;
        unsigned char* dst = ring + (size_t)s * stage;
        mb_expect_tx(&full[s], stage);
        bulk_copy(dst, kpool + tile * k_bytes, k_bytes, &full[s]);
        bulk_copy(dst + k_bytes, vpool + tile * v_bytes, v_bytes, &full[s]);
    };
    int n_pre = 0;
    if (a.early) {
        if (tid == ATT_WARPS * 32)
            for (; n_pre < np && n_pre < NST && page_at(p0 + n_pre) < (len - 1) / GQA_PAGE; ++n_pre) fetch(n_pre, n_pre);
        pdl_wait();
    }
    if (warp == ATT_WARPS) {
        if (lane == 0)
            for (int i = n_pre; i < np; ++i) {
                const int s = i % NST;
                if (i >= NST && !mb_wait(&empty[s], ((i / NST) & 1u) ^ 1u, a.err_flag, &s_abort)) break;
                fetch(i, s);
            }
    } else {
        // B fragments of the queries: lane (pair = lane / 4, i = lane % 4) holds elements 2i, 2i + 1 and 2i + 8, 2i + 9 of every 16
        const bool even = (dim & 1) == 0;  // rows of queries are then 8-byte aligned
#pragma unroll 4
        for (int i = tid; i < NT * kt_n * 32; i += ATT_WARPS * 32) {
            const int ln = i & 31, kt = (i >> 5) % kt_n, nt = (i >> 5) / kt_n, p = nt * 8 + (ln >> 2), d0 = kt * 16 + (ln & 3) * 2;
            float2 x = make_float2(0.f, 0.f), y = x;
            if (p < pairs) {
                const float* q = a.q + (size_t)(s_pos[p] - s_pos[0] + row0 + pair0 / g) * a.heads * dim + (size_t)(kvh * g + (pair0 + p) % g) * dim;
                auto at = [&](int d) {
                    if (even) return d < dim ? __ldcg(reinterpret_cast<const float2*>(q + d)) : make_float2(0.f, 0.f);
                    return make_float2(d < dim ? __ldcg(q + d) : 0.f, d + 1 < dim ? __ldcg(q + d + 1) : 0.f);
                };
                x = at(d0);
                y = at(d0 + 8);
            }
            uint32_t lo[3], hi[3];
            bf16x2_split3(x.x, x.y, lo[0], lo[1], lo[2]);
            bf16x2_split3(y.x, y.y, hi[0], hi[1], hi[2]);
#pragma unroll
            for (int t3 = 0; t3 < 3; ++t3) qf[((nt * kt_n + kt) * 3 + t3) * 32 + ln] = make_uint2(lo[t3], hi[t3]);
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
    }

    const int gid = lane >> 2, tig = lane & 3;
    float tm[NT][2], tl[NT][2], to[NT][VT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
        tm[nt][0] = tm[nt][1] = -INFINITY;
        tl[nt][0] = tl[nt][1] = 0.f;
#pragma unroll
        for (int mt = 0; mt < VT; ++mt) to[nt][mt][0] = to[nt][mt][1] = to[nt][mt][2] = to[nt][mt][3] = 0.f;
    }
    if (warp < ATT_WARPS) {
        const int u = warp & 3, mj = lane >> 3, mr = lane & 7;
        int pos[NT][2], brow[NT][2], from[NT][2];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int hh = 0; hh < 2; ++hh) {
                pos[nt][hh] = s_pos[nt * 8 + 2 * tig + hh];
                brow[nt][hh] = s_bias[nt * 8 + 2 * tig + hh];
                from[nt][hh] = X ? s_from[nt * 8 + 2 * tig + hh] : 0;
            }
        const uint32_t k_lane = (uint32_t)(((mj >> 1) * GQA_PAGE + u * 16 + (mj & 1) * 8 + mr) * 16), v_lane = (uint32_t)(((mj & 1) * GQA_PAGE + u * 16 + (mj >> 1) * 8 + mr) * 16);
        // pages alternate between the two groups of four warps; the stage count is even, so a stage is always the same group's
        for (int i = warp >> 2; i < np; i += 2) {
            const int s = i % NST;
            if (!__all_sync(0xffffffffu, mb_wait(&full[s], (i / NST) & 1u, a.err_flag, &s_abort))) break;
            const int tok = page_at(p0 + i) * GQA_PAGE + u * 16;
            if (tok < len) {
                const uint32_t kb = s32(ring + (size_t)s * stage) + k_lane, vb = s32(ring + (size_t)s * stage + k_bytes) + v_lane;
                constexpr int CH = NT == 1 ? 3 : 1;  // a lone tile of pairs: one accumulator per term, or its MMAs would wait for one another
                float sc[NT][CH][4];
#pragma unroll
                for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                    for (int c = 0; c < CH; ++c) sc[nt][c][0] = sc[nt][c][1] = sc[nt][c][2] = sc[nt][c][3] = 0.f;
#pragma unroll 2
                for (int kt = 0; kt < kt_n; ++kt) {
                    uint32_t ka[4];
                    ldsm4(ka, kb + (uint32_t)kt * (2 * GQA_PAGE * 16));
#pragma unroll
                    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                        for (int t3 = 0; t3 < 3; ++t3) {
                            const uint2 b = qf[((nt * kt_n + kt) * 3 + t3) * 32 + lane];
                            mma16816(sc[nt][t3 % CH], ka, b.x, b.y);
                        }
                }
                uint32_t pb[NT][3][2];
                const int t0 = tok + gid, t1 = t0 + 8;
#pragma unroll
                for (int nt = 0; nt < NT; ++nt) {
                    float pr[4], corr[2];
#pragma unroll
                    for (int c = CH - 1; c > 0; --c)  // small terms first
#pragma unroll
                        for (int e = 0; e < 4; ++e) sc[nt][c - 1][e] += sc[nt][c][e];
#pragma unroll
                    for (int hh = 0; hh < 2; ++hh) {
                        const int n0 = pos[nt][hh] - t0, n1 = pos[nt][hh] - t1;
                        float s0 = sc[nt][0][hh], s1 = sc[nt][0][2 + hh];
                        if (a.bias) {
                            s0 += __ldg(a.bias + brow[nt][hh] + min(max(n0, 0), a.reach));
                            s1 += __ldg(a.bias + brow[nt][hh] + min(max(n1, 0), a.reach));
                        }
                        s0 = n0 >= 0 && (!X || t0 >= from[nt][hh] || t0 < a.keep_first) ? s0 : -INFINITY;
                        s1 = n1 >= 0 && (!X || t1 >= from[nt][hh] || t1 < a.keep_first) ? s1 : -INFINITY;
                        float mx = fmaxf(s0, s1);
#pragma unroll
                        for (int o = 4; o < 32; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
                        mx = fmaxf(tm[nt][hh], mx);
                        const float ref = mx == -INFINITY ? 0.f : mx;  // no token of this pair yet
                        const float e0 = exp2f(s0 - ref), e1 = exp2f(s1 - ref);
                        corr[hh] = exp2f(tm[nt][hh] - ref);
                        tl[nt][hh] = fmaf(tl[nt][hh], corr[hh], e0 + e1);  // this lane's tokens
                        tm[nt][hh] = mx;
                        pr[hh] = e0;
                        pr[2 + hh] = e1;
                    }
                    uint32_t lo[3], hi[3];
                    bf16x2_split3(pr[0], pr[1], lo[0], lo[1], lo[2]);
                    bf16x2_split3(pr[2], pr[3], hi[0], hi[1], hi[2]);
#pragma unroll
                    for (int t3 = 0; t3 < 3; ++t3) {
                        pb[nt][t3][0] = transpose8x8(lo[t3]);
                        pb[nt][t3][1] = transpose8x8(hi[t3]);
                    }
                    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
                        for (int mt = 0; mt < VT; ++mt) {
                            to[nt][mt][0] *= corr[0];
                            to[nt][mt][1] *= corr[1];
                            to[nt][mt][2] *= corr[0];
                            to[nt][mt][3] *= corr[1];
                        }
                    }
                }
#pragma unroll
                for (int mt = 0; mt < VT; ++mt) {
                    if (mt < vt_n) {
                        uint32_t va[4];
                        ldsm4_trans(va, vb + (uint32_t)mt * (2 * GQA_PAGE * 16));
#pragma unroll
                        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                            for (int t3 = 0; t3 < 3; ++t3) mma16816(to[nt][mt], va, pb[nt][t3][0], pb[nt][t3][1]);
                    }
                }
            }
            __syncwarp();
            if (lane == 0) mb_arrive(&empty[s]);
        }
    }
    __syncthreads();  // every page consumed: the ring becomes scratch
    float* wm = reinterpret_cast<float*>(ring);  // [ATT_WARPS][P]
    float* wl = wm + ATT_WARPS * P;
    float* buf = wl + ATT_WARPS * P;             // [ATT_WARPS][P][ldo]
    if (warp < ATT_WARPS) {
        float* b = buf + (size_t)warp * P * ldo;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
#pragma unroll
            for (int hh = 0; hh < 2; ++hh)
#pragma unroll
                for (int o = 4; o < 32; o <<= 1) tl[nt][hh] += __shfl_xor_sync(0xffffffffu, tl[nt][hh], o);
            if (gid == 0) {
#pragma unroll
                for (int hh = 0; hh < 2; ++hh) {
                    wm[warp * P + nt * 8 + 2 * tig + hh] = tm[nt][hh];
                    wl[warp * P + nt * 8 + 2 * tig + hh] = tl[nt][hh];
                }
            }
#pragma unroll
            for (int mt = 0; mt < VT; ++mt)
                if (mt < vt_n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) b[(nt * 8 + 2 * tig + (e & 1)) * ldo + mt * 16 + gid + (e >> 1) * 8] = to[nt][mt][e];
        }
    }
    __syncthreads();
    // the warps' results added up, four values a thread, and sent to the split that owns the pair
    for (int i = tid; i < pairs * (vp / 4); i += B_THREADS) {
        const int p = i / (vp / 4), d = (i - p * (vp / 4)) * 4;
        float f[ATT_WARPS], mx = -INFINITY, l = 0.f;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int w = 0; w < ATT_WARPS; ++w) {
            f[w] = wm[w * P + p];
            mx = fmaxf(mx, f[w]);
        }
#pragma unroll
        for (int w = 0; w < ATT_WARPS; ++w) {
            f[w] = f[w] == -INFINITY ? 0.f : exp2f(f[w] - mx);
            const float4 x = *reinterpret_cast<const float4*>(buf + (size_t)(w * P + p) * ldo + d);
            v.x = fmaf(f[w], x.x, v.x); v.y = fmaf(f[w], x.y, v.y); v.z = fmaf(f[w], x.z, v.z); v.w = fmaf(f[w], x.w, v.w);
            l = fmaf(f[w], wl[w * P + p], l);
        }
        const uint32_t owner = (uint32_t)(p % ns);
        float* slot = recv + (size_t)(rank * own_most + p / ns) * (vp + 4);
        if ((int)owner == rank) {
            *reinterpret_cast<float4*>(slot + d) = v;
            if (d == 0) {
                slot[vp] = mx;
                slot[vp + 1] = l;
            }
        } else {
            const uint32_t bar = dsmem_addr(&s_rbar, owner);
            st_async_f32x4(dsmem_addr(slot + d, owner), v, bar);
            if (d == 0) st_async_f32x2(dsmem_addr(slot + vp, owner), mx, l, bar);
        }
    }
    if (own == 0) return;
    __syncthreads();
    if (ns > 1 && !mb_wait_cluster(&s_rbar, 0, a.err_flag, &s_abort)) return;  // bounded
    for (int i = tid; i < own * (vp / 8); i += B_THREADS) {
        const int k = i / (vp / 8), d0 = (i - k * (vp / 8)) * 8, p = k * ns + rank;
        float v[8], mx = -INFINITY, l = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = 0.f;
        for (int r = 0; r < ns; ++r) mx = fmaxf(mx, recv[(size_t)(r * own_most + k) * (vp + 4) + vp]);
#pragma unroll 4
        for (int r = 0; r < ns; ++r) {
            const float* slot = recv + (size_t)(r * own_most + k) * (vp + 4);
            const float f = slot[vp] == -INFINITY ? 0.f : exp2f(slot[vp] - mx);
            const float4 x = *reinterpret_cast<const float4*>(slot + d0), y = *reinterpret_cast<const float4*>(slot + d0 + 4);
            l = fmaf(f, slot[vp + 1], l);
            v[0] = fmaf(f, x.x, v[0]); v[1] = fmaf(f, x.y, v[1]); v[2] = fmaf(f, x.z, v[2]); v[3] = fmaf(f, x.w, v[3]);
            v[4] = fmaf(f, y.x, v[4]); v[5] = fmaf(f, y.y, v[5]); v[6] = fmaf(f, y.z, v[6]); v[7] = fmaf(f, y.w, v[7]);
        }
        const float inv = 1.0f / (l + sink_weight<X>(a, kvh * g + (pair0 + p) % g, mx));
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= inv;
        if (d0 < vdim) store_piece<X>(a, row0 + (pair0 + p) / g, kvh * g + (pair0 + p) % g, d0, v);
    }
}

template <typename... KArgs, typename... Args>
cudaError_t launch_clustered(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, int cluster, cudaStream_t st, bool pdl, Args... args) {
    cudaError_t e = ensure_dyn_smem(kern, smem);
    if (e == cudaSuccess && cluster > 8) e = ensure_nonportable_clusters(kern);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    int n = 0;
    if (pdl) {
        at[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        at[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    if (cluster > 1) {
        at[n].id = cudaLaunchAttributeClusterDimension;
        at[n].val.clusterDim.x = (unsigned)cluster;
        at[n].val.clusterDim.y = 1;
        at[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = at;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, kern, KArgs(args)...);
}

// Clusters of a kernel that the current device holds at the same time (asked once per shape).
template <typename... KArgs>
int clusters_at_once(void (*kern)(KArgs...), int cluster, int threads, size_t smem) {
    static std::mutex mu;
    static std::map<std::tuple<const void*, int, int, size_t>, int> known;
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess) return 0;
    const auto key = std::make_tuple(reinterpret_cast<const void*>(kern), dev, cluster, smem);
    std::lock_guard<std::mutex> lk(mu);
    const auto it = known.find(key);
    if (it != known.end()) return it->second;
    int n = 0;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)cluster);
    cfg.blockDim = dim3((unsigned)threads);
    cfg.dynamicSmemBytes = smem;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = (unsigned)cluster;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    cfg.attrs = at;
    cfg.numAttrs = 1;
    if (ensure_dyn_smem(kern, smem) != cudaSuccess || (cluster > 8 && ensure_nonportable_clusters(kern) != cudaSuccess) || cudaOccupancyMaxActiveClusters(&n, kern, &cfg) != cudaSuccess) {
        cudaGetLastError();
        n = 0;
    }
    return known[key] = n;
}

// Pages that a tile of so many (row, head) pairs can see.
int most_pages(const GqaAttnArgs& a, int pairs) {
    const int all = (a.longest + GQA_PAGE - 1) / GQA_PAGE;
    if (a.window == 0 && a.chunk == 0) return all;
    const int rows = std::min(a.longest_run, (pairs + a.heads / a.pool.kv_heads - 1) / (a.heads / a.pool.kv_heads) + 1);
    const long seen = (a.keep_first + GQA_PAGE - 1) / GQA_PAGE + ((long)(a.chunk > 0 ? a.chunk : a.window) + rows - 2) / GQA_PAGE + 2;
    return (int)std::min<long>(all, seen);
}

template <int VT, int NT, bool X>
cudaError_t launch_mma(GqaAttnArgs a, int sm_count, cudaStream_t st, bool pdl) {
    constexpr int P = NT * 8;
    const int g = a.heads / a.pool.kv_heads, dp = gqa_pad(a.pool.dim), vp = gqa_pad(a.pool.vdim);
    a.tiles_per_row = (g + P - 1) / P;
    if (a.runs.n == 0) {
        a.tiles = a.M * a.tiles_per_row;
    } else {
        a.tiles = 0;
        for (int r = 0; r < a.runs.n; ++r) {
            a.runs.tile[r] = (uint16_t)a.tiles;
            a.tiles += ((a.runs.row[r + 1] - a.runs.row[r]) * g + P - 1) / P;
        }
        a.runs.tile[a.runs.n] = (uint16_t)a.tiles;
    }
    const int pages = most_pages(a, P), pairs = a.tiles * a.pool.kv_heads;
    constexpr int PER_SM = NT == 1 && VT <= 8 ? 2 : 1;
    const size_t stage = b_stage_bytes(dp, vp);
    size_t ring = 0, fixed = 0;
    auto shape = [&](int nsplit) {  // ring and shared memory of a launch with so many splits
        const int ppc = (pages + nsplit - 1) / nsplit;
        fixed = b_query_bytes(NT, dp) + b_recv_bytes(NT, vp, nsplit) + 4 * (size_t)ppc + 128;
        // CTAs that have an SM to themselves take a deep ring
        const size_t budget = (PER_SM == 2 && (long)pairs * nsplit > sm_count ? 110 : 220) * 1024;
        int stages = MAX_STAGES;
        while (stages > 2 && (stages * stage + fixed > budget || stages - 2 >= ppc)) stages -= 2;
        a.stages = stages;
        ring = (std::max(stages * stage, b_merge_bytes(NT, vp)) + 127) / 128 * 128;
    };
    if (a.nsplit < 1) {
        // as many splits as run at once; clusters of more than eight CTAs are hard to place: only for long contexts
        a.nsplit = std::max(1, std::min({PER_SM * sm_count / pairs, a.max_cluster, pages > 128 ? MAX_CLUSTER : 8, pages}));
        for (; a.nsplit > 1; --a.nsplit) {
            shape(a.nsplit);
            if (ring + fixed <= 226 * 1024 && clusters_at_once(gqa_attn_mma_kernel<VT, NT, X>, a.nsplit, B_THREADS, ring + fixed) >= pairs) break;
        }
    }
    shape(a.nsplit);
    if (ring + fixed > 226 * 1024) return cudaErrorInvalidValue;
    return launch_clustered(gqa_attn_mma_kernel<VT, NT, X>, dim3((unsigned)a.nsplit, (unsigned)a.pool.kv_heads, (unsigned)a.tiles), dim3(B_THREADS), ring + fixed, a.nsplit, st, pdl, a, ring);
}

template <int VT, bool X>
cudaError_t launch_mma_n(const GqaAttnArgs& a, int sm_count, cudaStream_t st, bool pdl) {
    const int pairs = a.longest_run * (a.heads / a.pool.kv_heads);
    if (pairs <= 8) return launch_mma<VT, 1, X>(a, sm_count, st, pdl);
    if (pairs <= 16 || VT > 4) return launch_mma<VT, 2, X>(a, sm_count, st, pdl);  // four tiles of wide values do not fit the registers
    return launch_mma<VT, VT <= 4 ? 4 : 2, X>(a, sm_count, st, pdl);
}

#include "gqa_talk.cuh"

}  // namespace

cudaError_t launch_gqa_post(const GqaPostArgs& a, cudaStream_t st, bool pdl) {
    const dim3 grid((unsigned)a.M, (unsigned)gqa_post_blocks(a)), block(POST_WARPS * 32);
    if (a.varied()) return launch_clustered(gqa_post_kernel<2>, grid, block, gqa_post_smem(a), 1, st, pdl, a);
    return gqa_post_buf(a) > 0 ? launch_clustered(gqa_post_kernel<1>, grid, block, gqa_post_smem(a), 1, st, pdl, a) : launch_clustered(gqa_post_kernel<0>, grid, block, 0, 1, st, pdl, a);
}

cudaError_t launch_gqa_attn(const GqaAttnArgs& a_in, int sm_count, cudaStream_t st, bool pdl) {
    GqaAttnArgs a = a_in;
    if (a.M < 1 || a.M > GQA_MAX_ROWS || a.nsplit > MAX_CLUSTER || a.heads % a.pool.kv_heads != 0) return cudaErrorInvalidValue;
    if (!a.bias) a.reach = 0;
    const bool x = a.window > 0 || a.chunk > 0 || a.talk || a.sink || a.gate_kind != GATE_NONE || a.out_scale != 0.f || a.ld_out != 0;
    if (a.ld_out == 0) a.ld_out = a.heads * a.pool.vdim;
    const int g = a.heads / a.pool.kv_heads, dp = gqa_pad(a.pool.dim), vp = gqa_pad(a.pool.vdim);
    if (a.runs.n == 0) a.longest_run = 1;
    if (a.talk) {
        if (a.bias) return cudaErrorInvalidValue;
        return launch_talk(a, sm_count, st, pdl);
    }
    const long ppc_most = most_pages(a, 32);
    if (a.pool.bf16 && vp <= 256 && dp <= 256 && ppc_most <= 8192) {
        if (vp <= 64) return x ? launch_mma_n<4, true>(a, sm_count, st, pdl) : launch_mma_n<4, false>(a, sm_count, st, pdl);
        if (vp <= 128) return x ? launch_mma_n<8, true>(a, sm_count, st, pdl) : launch_mma_n<8, false>(a, sm_count, st, pdl);
        return x ? launch_mma_n<16, true>(a, sm_count, st, pdl) : launch_mma_n<16, false>(a, sm_count, st, pdl);
    }
    const int pages = most_pages(a, 1);
    if (a.nsplit < 1) a.nsplit = std::max(1, std::min({4 * sm_count / (a.M * a.pool.kv_heads), a.max_cluster, MAX_CLUSTER, pages}));
    const size_t smem = sizeof(float) * (size_t)g * (dp + vp + 4 + GQA_PAGE + 3 + a.nsplit);
    const dim3 grid((unsigned)a.nsplit, (unsigned)a.pool.kv_heads, (unsigned)a.M);
    auto go = [&](auto kern) { return launch_clustered(kern, grid, dim3(A_THREADS), smem, a.nsplit, st, pdl, a); };
    if (x) return a.pool.bf16 ? go(gqa_attn_kernel<true, true, false>) : go(gqa_attn_kernel<false, true, false>);
    return a.pool.bf16 ? go(gqa_attn_kernel<true, false, false>) : go(gqa_attn_kernel<false, false, false>);
}

bool gqa_talk_fits(int heads, int dim, int vdim) { return talk_plain_smem(heads, gqa_pad(dim), gqa_pad(vdim), MAX_CLUSTER) <= 226 * 1024; }

cudaError_t launch_gqa_read(const GqaPool& pool, int seq, int len, float* k, float* v, cudaStream_t st) {
    const size_t total = (size_t)pool.kv_heads * len * (pool.dim + pool.vdim);
    gqa_read_kernel<<<(unsigned)std::min<size_t>((total + 255) / 256, 4096), 256, 0, st>>>(pool, seq, len, k, v);
    return cudaGetLastError();
}

}  // namespace hm
