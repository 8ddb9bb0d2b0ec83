// See side.h.  Blocks take their parts in order of weight: the recurrences first, then heads, latents, activations, routers; the variant for
// recurrences that are a launch of their own: factors, heads, latents.
#include "side.h"

#include <algorithm>

#include "gemm_tc.h"
#include "gla.cuh"
#include "gqa_post.cuh"
#include "latent_post.cuh"
#include "launch_attrs.h"
#include "route.cuh"

namespace hm {
namespace {

constexpr int THREADS = 256, WARPS = THREADS / 32;
static_assert(THREADS == GLA_THREADS && WARPS == POST_WARPS, "one block size for all parts");

__device__ __forceinline__ float block_sum(float v, float* part) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) s += part[i];
    return s;
}

__device__ __forceinline__ int act_blocks(int ff) { return ((ff + 7) / 8 + THREADS - 1) / THREADS; }

__device__ __forceinline__ void act_block(const SideArgs& a, int b) {
    const MlpSide& f = a.mlp;
    const int per = act_blocks(f.ff), m = b / per, c = ((b - m * per) * THREADS + threadIdx.x) * 8;
    if (c >= f.ff) return;
    const size_t row = (size_t)m * a.ld;
    const float4 g0 = ld_cg_f32x4(f.gate + row + c), g1 = ld_cg_f32x4(f.gate + row + c + 4), u0 = ld_cg_f32x4(f.up + row + c), u1 = ld_cg_f32x4(f.up + row + c + 4);
    const float rg = f.row_gate ? 1.0f / (1.0f + expf(-ld_cg_f32(f.row_gate + row))) : 1.f;
    const float g[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w}, u[8] = {u0.x, u0.y, u0.z, u0.w, u1.x, u1.y, u1.z, u1.w};
    float v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = glu(f.act, g[e], u[e], 0.f) * rg;
    if (f.xp) {
        tc_xpack_store8(f.xp, a.xp_mpad, m, f.out_off + c, v);
    } else {
        float* o = f.out + (size_t)m * f.ld_out + f.out_off + c;
        reinterpret_cast<float4*>(o)[0] = make_float4(v[0], v[1], v[2], v[3]);
        reinterpret_cast<float4*>(o)[1] = make_float4(v[4], v[5], v[6], v[7]);
    }
}

// One warp chooses, the others leave; z: 2 * n_out floats.
__device__ __forceinline__ void route_block(const SideArgs& a, int m, float* z) {
    const MlpSide& f = a.mlp;
    if (f.route.out.dense)
        for (int i = threadIdx.x; i < f.route.experts; i += THREADS) f.route.out.dense[(size_t)m * f.route.experts + i] = 0.f;
    for (int i = threadIdx.x; i < f.route.n_out; i += THREADS) z[i] = ld_cg_f32(f.logits + (size_t)m * a.ld + i);
    __syncthreads();
    if (threadIdx.x < 32) choose_experts(f.route, m, z, z + f.route.n_out);
}

__device__ __forceinline__ void normed_block(const SideArgs& a, int m, float* part) {
    const MlpSide& f = a.mlp;
    const float* x = f.x + (size_t)m * f.W;
    float s = 0.f;
#pragma unroll 4
    for (int i = threadIdx.x; i < f.W; i += THREADS) {
        const float v = ld_cg_f32(x + i);
        s = fmaf(v, v, s);
    }
    const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)f.W + a.eps);
#pragma unroll 4
    for (int i = threadIdx.x; i < f.W; i += THREADS) f.normed[(size_t)m * f.W + i] = (ld_cg_f32(x + i) * inv) * __ldg(f.w + i);
}

// The queries' latent of row m, RMS-normed and packed.
__device__ __forceinline__ void query_latent_block(const SideArgs& a, int m, float* part) {
    const LatentSide& l = a.latent;
    const float* x = l.cq + (size_t)m * a.ld;
    float s = 0.f;
    for (int i = threadIdx.x; i < l.q_rank; i += THREADS) {
        const float v = ld_cg_f32(x + i);
        s = fmaf(v, v, s);
    }
    const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)l.q_rank + a.eps);
    for (int c = threadIdx.x * 8; c < (l.q_rank + 63) / 64 * 64; c += THREADS * 8) {
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = c + e < l.q_rank ? (ld_cg_f32(x + c + e) * inv) * __ldg(l.q_w + c + e) : 0.f;
        tc_xpack_store8(l.q_xp, a.xp_mpad, m, c, v);
    }
}

// LR_ROWS rows and 32 columns of one of the two factors (LowRankSide); the warps share the rank.
constexpr int LR_ROWS = 8, LR_AHEAD = 16;
__device__ __forceinline__ int low_rank_blocks(const LowRankSide& l) { return (l.heads * l.dim + 31) / 32 + (l.heads * l.vdim + 31) / 32; }

__device__ __forceinline__ void low_rank_block(const SideArgs& a, int b, float* sm) {
    const LowRankSide& l = a.low;
    const int per = low_rank_blocks(l), na = (l.heads * l.dim + 31) / 32, tile = b / per, cb = b - tile * per, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const bool is_a = cb < na;
    const int N = l.heads * (is_a ? l.dim : l.vdim), col = (is_a ? cb : cb - na) * 32 + lane, rank = is_a ? l.rank_a : l.rank_g, m0 = tile * LR_ROWS, rows = min(LR_ROWS, a.M - m0);
    const float* up = (is_a ? l.up_a : l.up_g) + col;
    const float* lat = is_a ? l.a : l.g;
    const bool on = col < N;
    float w[LR_AHEAD];  // weights do not depend on the launch in front
#pragma unroll
    for (int i = 0; i < LR_AHEAD; ++i) {
        const int r = warp + i * WARPS;
        w[i] = on && r < rank ? __ldg(up + (size_t)r * N) : 0.f;
    }
    const float bias = is_a && on ? __ldg(l.bias + col) : 0.f, rate = is_a && on ? __ldg(l.neg_rate + col / l.dim) : 0.f;
    pdl_wait();
    float* red = sm + LR_ROWS * rank;  // [WARPS][LR_ROWS][32]
    for (int i = threadIdx.x; i < rows * rank; i += THREADS) {
        const int t = i / rank;
        sm[i] = ld_cg_f32(lat + (size_t)(m0 + t) * a.ld + (i - t * rank));
    }
    __syncthreads();
    float acc[LR_ROWS];
#pragma unroll
    for (int t = 0; t < LR_ROWS; ++t) acc[t] = 0.f;
    for (int r0 = 0; r0 < rank; r0 += LR_AHEAD * WARPS) {
#pragma unroll
        for (int i = 0; i < LR_AHEAD; ++i) {
            const int r = r0 + warp + i * WARPS;
            if (r < rank) {
#pragma unroll
                for (int t = 0; t < LR_ROWS; ++t)
                    if (t < rows) acc[t] = fmaf(w[i], sm[t * rank + r], acc[t]);
            }
        }
#pragma unroll
        for (int i = 0; i < LR_AHEAD; ++i) {
            const int r = r0 + (LR_AHEAD + i) * WARPS + warp;
            w[i] = on && r < rank ? __ldg(up + (size_t)r * N) : 0.f;
        }
    }
#pragma unroll
    for (int t = 0; t < LR_ROWS; ++t) red[(warp * LR_ROWS + t) * 32 + lane] = acc[t];
    __syncthreads();
    if (warp >= rows || !on) return;
    float z = 0.f;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) z += red[(i * LR_ROWS + warp) * 32 + lane];
    if (is_a) {
        z += bias;
        l.alpha[(size_t)(m0 + warp) * N + col] = expf(rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
    } else {
        l.gate[(size_t)(m0 + warp) * N + col] = z;
    }
}

// RD: state rows per thread of the linear attention, 0: there is none, -1: single tokens, states in shared memory, -2: rows are
// prepared for a recurrence, and whatever GqaPostArgs::varied() names
template <int RD>
__global__ void __launch_bounds__(THREADS, RD > 32 ? 1 : RD > 0 ? 2 : 3) side_kernel(const __grid_constant__ SideArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float part[WARPS];
    pdl_launch_dependents();
    int b = blockIdx.x;
    if constexpr (RD == -2) {
        if (b < a.n_low) {
            low_rank_block(a, b, sm);
            return;
        }
        b -= a.n_low;
        if (b < a.n_post2) {
            const int per = gqa_post_blocks(a.post2);
            gqa_post_block<2>(a.post2, b / per, b % per, sm);
            return;
        }
        b -= a.n_post2;
        if (b < a.n_post) {
            const int per = gqa_post_blocks(a.post);
            gqa_post_block<2>(a.post, b / per, b % per, sm);
            return;
        }
        b -= a.n_post;
        pdl_wait();
        if (b < a.n_latent) latent_write_row<THREADS, true>(a.latent.pool, a.latent.c, a.ld, b, a.latent.w, a.eps, a.row_pos, a.row_seq, a.latent.rot_pairs, a.latent.turns, part, a.latent.neighbours != 0);
        return;
    }
    if constexpr (RD != 0) {
        if (b < a.n_gla) {
            if constexpr (RD > 0) gla_block<RD>(a.gla, b, sm);
            else gla_token_block(a.gla, b, sm, part);
            return;
        }
        b -= a.n_gla;
    }
    if (b < a.n_post) {
        const int per = gqa_post_blocks(a.post);
        gqa_post_block<1>(a.post, b / per, b % per, sm);
        return;
    }
    b -= a.n_post;
    pdl_wait();
    if (b < a.n_latent) {
        if (b < a.M) latent_write_row<THREADS, true>(a.latent.pool, a.latent.c, a.ld, b, a.latent.w, a.eps, a.row_pos, a.row_seq, a.latent.rot_pairs, a.latent.turns, part);
        else query_latent_block(a, b - a.M, part);
        return;
    }
    b -= a.n_latent;
    if (b < a.n_act) {
        act_block(a, b);
        return;
    }
    b -= a.n_act;
    if (b < a.n_route) {
        route_block(a, b, sm);
        return;
    }
    b -= a.n_route;
    if (b < a.n_normed) normed_block(a, b, part);  // (the rest fills the last cluster)
}

__global__ void __launch_bounds__(THREADS) sum_norm_kernel(const SumNormArgs a) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float part[WARPS];
    const int m = blockIdx.x, tid = threadIdx.x, Wp = (a.W + 63) / 64 * 64;
    pdl_launch_dependents();
    pdl_wait();
    if (m >= a.M) {  // rows that pad the image
        if (a.w)
            for (int c = tid * 8; c < Wp; c += THREADS * 8) {
                const float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                tc_xpack_store8(a.xp, a.xp_mpad, m, c, v);
            }
        return;
    }
    float* x = a.x + (size_t)m * a.W;
    const float* y = a.y + (size_t)m * a.W;
    float s = 0.f;
    if ((a.W & 3) == 0) {
        for (int i = tid; i < a.W / 4; i += THREADS) {
            float4 v = ld_cg_f32x4(x + 4 * (size_t)i);
            for (int p = 0; p < a.parts; ++p) {
                const float4 t = ld_cg_f32x4(y + p * a.part_stride + 4 * (size_t)i);
                v = make_float4(v.x + t.x, v.y + t.y, v.z + t.z, v.w + t.w);
            }
            s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
            reinterpret_cast<float4*>(xs)[i] = v;
            if (a.parts) reinterpret_cast<float4*>(x)[i] = v;
        }
    } else {
        for (int i = tid; i < a.W; i += THREADS) {
            float v = ld_cg_f32(x + i);
            for (int p = 0; p < a.parts; ++p) v += ld_cg_f32(y + p * a.part_stride + i);
            s = fmaf(v, v, s);
            xs[i] = v;
            if (a.parts) x[i] = v;
        }
    }
    if (!a.w) return;
    const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)a.W + a.eps);  // (its barrier publishes the row as well)
    for (int c = tid * 8; c < Wp; c += THREADS * 8) {
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = c + e < a.W ? (xs[c + e] * inv) * __ldg(a.w + c + e) : 0.f;
        tc_xpack_store8(a.xp, a.xp_mpad, m, c, v);
    }
}

template <typename K, typename A>
cudaError_t launch(K kern, unsigned blocks, size_t smem, int cluster, cudaStream_t st, bool pdl, const A& args) {
    const cudaError_t e = ensure_dyn_smem(kern, smem);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(blocks);
    cfg.blockDim = dim3(THREADS);
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
        at[n].val.clusterDim.y = at[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = at;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, kern, args);
}

}  // namespace

GlaShape gla_shape(int dim, int vdim, int heads, int sm_count) {
    GlaShape s{};
    // a head's columns are spread over CTAs until they fill the SMs, as long as every thread has rows, and over enough of them that a
    // thread holds at most 32 rows
    s.cluster = 1;
    auto share = [&](int cluster) { return ((vdim + cluster - 1) / cluster + 7) / 8 * 8; };
    while (s.cluster < GLA_MAX_CLUSTER && vdim / (2 * s.cluster) >= 8 &&
           ((2 * s.cluster * heads <= sm_count && GLA_THREADS / share(2 * s.cluster) * 4 <= gla_pad(dim)) || (size_t)gla_pad(dim) * vdim / s.cluster > 32 * GLA_THREADS))
        s.cluster *= 2;
    s.share = share(s.cluster);
    s.cols = 8;
    while (s.cols < s.share && s.cols < GLA_THREADS) s.cols *= 2;
    for (; s.cols > 8; s.cols /= 2)
        if (GLA_THREADS / s.cols * 64 >= dim) break;
    s.lanes = GLA_THREADS / s.cols;
    s.rows = 4;
    while (s.rows * s.lanes < dim) s.rows *= 2;
    s.slices = (s.share + s.cols - 1) / s.cols;
    return s;
}

cudaError_t launch_side(const SideArgs& a_in, int sm_count, cudaStream_t st, bool pdl) {
    SideArgs a = a_in;
    if (a.M < 1 || a.M > GQA_MAX_ROWS) return cudaErrorInvalidValue;
    const int runs = a.gla.runs.n ? a.gla.runs.n : a.M;
    size_t smem = 0;
    a.n_gla = a.n_post = a.n_latent = a.n_act = a.n_route = a.n_normed = a.n_post2 = a.n_low = 0;
    int cluster = 1, kind = 0;
    if (a.has_gla) {
        GlaArgs& g = a.gla;
        if (g.dim > GLA_MAX_DIM || g.vdim > GLA_MAX_VDIM) return cudaErrorInvalidValue;
        const int rows = g.runs.n ? g.longest_run : 1;
        if (rows == 1 && g.dim <= GLA_TOKEN_DIM && gla_state_floats(g.dim, g.vdim) * 4 <= GLA_TOKEN_BYTES) {
            kind = -1;
            a.n_gla = a.M * g.heads;
            smem = (size_t)gla_token_smem(g).total * 4;
        } else {
            g.shape = gla_shape(g.dim, g.vdim, runs * g.heads, sm_count);
            kind = g.shape.rows;
            cluster = g.shape.cluster;
            a.n_gla = runs * g.heads * cluster;
            for (g.step = rows; g.step > 1 && (size_t)gla_smem(g, rows).total * 4 > 110 * 1024; g.step = (g.step + 1) / 2) {
            }
            smem = (size_t)gla_smem(g, rows).total * 4;
        }
    }
    if (a.has_post) {
        a.n_post = a.M * gqa_post_blocks(a.post);
        smem = std::max(smem, gqa_post_smem(a.post));
    }
    if (a.has_post2 || a.has_low || (a.has_post && a.post.varied()) || (a.has_latent && a.latent.neighbours)) {
        if (a.has_gla || a.mlp.ff || a.mlp.logits || a.mlp.normed || (a.has_latent && a.latent.q_xp)) return cudaErrorInvalidValue;
        kind = -2;
    }
    if (a.has_post2) {
        a.n_post2 = a.M * gqa_post_blocks(a.post2);
        smem = std::max(smem, gqa_post_smem(a.post2));
    }
    if (a.has_low) {
        const LowRankSide& l = a.low;
        a.n_low = (a.M + LR_ROWS - 1) / LR_ROWS * ((l.heads * l.dim + 31) / 32 + (l.heads * l.vdim + 31) / 32);
        smem = std::max(smem, sizeof(float) * LR_ROWS * ((size_t)std::max(l.rank_a, l.rank_g) + WARPS * 32));
    }
    if (a.has_latent) a.n_latent = a.M * (a.latent.q_xp ? 2 : 1);
    if (a.mlp.ff) a.n_act = a.M * (((a.mlp.ff + 7) / 8 + THREADS - 1) / THREADS);
    if (a.mlp.logits) {
        a.n_route = a.M;
        smem = std::max(smem, 2 * sizeof(float) * (size_t)a.mlp.route.n_out);
    }
    if (a.mlp.normed) a.n_normed = a.M;
    const unsigned blocks = (unsigned)((a.n_gla + a.n_post + a.n_latent + a.n_act + a.n_route + a.n_normed + a.n_post2 + a.n_low + cluster - 1) / cluster * cluster);
    switch (kind) {
        case -2: return launch(side_kernel<-2>, blocks, smem, cluster, st, pdl, a);
        case -1: return launch(side_kernel<-1>, blocks, smem, cluster, st, pdl, a);
        case 4: return launch(side_kernel<4>, blocks, smem, cluster, st, pdl, a);
        case 0: return launch(side_kernel<0>, blocks, smem, cluster, st, pdl, a);
        case 8: return launch(side_kernel<8>, blocks, smem, cluster, st, pdl, a);
        case 16: return launch(side_kernel<16>, blocks, smem, cluster, st, pdl, a);
        case 32: return launch(side_kernel<32>, blocks, smem, cluster, st, pdl, a);
        case 64: return launch(side_kernel<64>, blocks, smem, cluster, st, pdl, a);
        default: return cudaErrorInvalidValue;
    }
}

cudaError_t launch_sum_norm(const SumNormArgs& a, cudaStream_t st, bool pdl) {
    if (!a.w && !a.parts) return cudaSuccess;
    return launch(sum_norm_kernel, (unsigned)(a.w ? tc_mpad(a.M) : a.M), sizeof(float) * (size_t)((a.W + 7) / 8 * 8), 1, st, pdl, a);
}

}  // namespace hm
