// Residual sums with normalised sublayer results, routers, mixtures of experts.
//
//   post_norm_kernel       x += mult * RMSnorm(y) * w; router logits, softmax and choice over the new x.  A row is a cluster of CTAs,
//                          which share the router's outputs.
//   expert_gate_up_kernel  one (row, chosen expert) pair and 16 activations per CTA
//   expert_down_kernel     one row and 8 outputs per CTA, over all chosen experts of the row
// The two expert kernels serve passes of few rows; larger passes multiply every used expert with all rows on the tensor cores
// (gemm_tc.cu).  Both read the same tile images of the weights.
#include "moe.h"

#include <algorithm>

#include "gemm_tc.h"
#include "launch_attrs.h"
#include "route.cuh"

namespace hm {
namespace {

constexpr int THREADS = 256, WARPS = THREADS / 32;
constexpr int TILE = 128 * 64;  // elements of a tile image: 128 rows of 64 k, 16-byte pieces XOR-ed by row & 7
constexpr int GU_ROWS = 16, DOWN_ROWS = 8;
constexpr int REG4 = 2;         // 16-byte pieces of a residual row that a thread of the post-norm keeps in registers

__device__ __forceinline__ float block_sum(float v, float* part) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) s += part[i];
    return s;
}
__device__ __forceinline__ float dot8(const uint4& w, const float4& x, const float4& y, float s) {
    s = fmaf(bf16_lo(w.x), x.x, s);
    s = fmaf(bf16_hi(w.x), x.y, s);
    s = fmaf(bf16_lo(w.y), x.z, s);
    s = fmaf(bf16_hi(w.y), x.w, s);
    s = fmaf(bf16_lo(w.z), y.x, s);
    s = fmaf(bf16_hi(w.z), y.y, s);
    s = fmaf(bf16_lo(w.w), y.z, s);
    return fmaf(bf16_hi(w.w), y.w, s);
}

__global__ void __launch_bounds__(THREADS) post_norm_kernel(const PostNormArgs a, int cluster) {
    extern __shared__ __align__(16) float sm[];
    const int Wp = (a.W + 7) & ~7;
    float *xs = sm, *ys = xs + Wp, *z = ys + Wp, *choice = z + a.n_out;
    __shared__ float part[WARPS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, m = blockIdx.x / cluster, rank = blockIdx.x - m * cluster;
    pdl_launch_dependents();
    // weights do not depend on the launch in front: norm weights, and the first router row of the warp
    const bool regs = (a.W & 7) == 0 && a.W <= 4 * REG4 * THREADS;
    float4 w4[REG4];
    uint4 r4[REG4 * 4];
    const int first = rank * WARPS + warp;
    if (regs) {
#pragma unroll
        for (int k = 0; k < REG4; ++k)
            if (tid + k * THREADS < a.W / 4) w4[k] = __ldg(reinterpret_cast<const float4*>(a.w) + tid + k * THREADS);
        if (a.router && first < a.n_out) {
            const uint4* wr = reinterpret_cast<const uint4*>(a.router + (size_t)first * a.W);
#pragma unroll
            for (int k = 0; k < REG4 * 4; ++k) r4[k] = lane + k * 32 < a.W / 8 ? __ldg(wr + lane + k * 32) : make_uint4(0, 0, 0, 0);
        }
    }
    if (cluster > 1) {  // every CTA of the cluster has started before the first one stores into rank 0
        cluster_arrive_release();
        cluster_wait_acquire();
    }
    pdl_wait();
    const float idw = a.identity ? ld_cg_f32(a.identity + m) : 0.f;
    const float *x = a.x + (size_t)m * a.W, *y = a.y + (size_t)m * a.W;
    float ss = 0.f;
    if (regs) {
        float4 x4[REG4], y4[REG4];
#pragma unroll
        for (int k = 0; k < REG4; ++k) {
            const int i = tid + k * THREADS;
            x4[k] = y4[k] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < a.W / 4) {
                x4[k] = ld_cg_f32x4(x + 4 * (size_t)i);
                y4[k] = ld_cg_f32x4(y + 4 * (size_t)i);
            }
        }
        for (int p = 1; p < a.parts; ++p)
#pragma unroll
            for (int k = 0; k < REG4; ++k)
                if (tid + k * THREADS < a.W / 4) {
                    const float4 t = ld_cg_f32x4(y + p * a.part_stride + 4 * (size_t)(tid + k * THREADS));
                    y4[k] = make_float4(y4[k].x + t.x, y4[k].y + t.y, y4[k].z + t.z, y4[k].w + t.w);
                }
#pragma unroll
        for (int k = 0; k < REG4; ++k) {
            y4[k] = make_float4(fmaf(idw, x4[k].x, y4[k].x), fmaf(idw, x4[k].y, y4[k].y), fmaf(idw, x4[k].z, y4[k].z), fmaf(idw, x4[k].w, y4[k].w));
            ss = fmaf(y4[k].x, y4[k].x, fmaf(y4[k].y, y4[k].y, fmaf(y4[k].z, y4[k].z, fmaf(y4[k].w, y4[k].w, ss))));
        }
        const float inv = 1.0f / sqrtf(block_sum(ss, part) / (float)a.W + a.eps);
#pragma unroll
        for (int k = 0; k < REG4; ++k)
            if (tid + k * THREADS < a.W / 4)
                reinterpret_cast<float4*>(xs)[tid + k * THREADS] = make_float4(fmaf(a.mult, (y4[k].x * inv) * w4[k].x, x4[k].x), fmaf(a.mult, (y4[k].y * inv) * w4[k].y, x4[k].y),
                                                                              fmaf(a.mult, (y4[k].z * inv) * w4[k].z, x4[k].z), fmaf(a.mult, (y4[k].w * inv) * w4[k].w, x4[k].w));
    } else {
        for (int i = tid; i < a.W; i += THREADS) {
            const float xv = ld_cg_f32(x + i);
            float yv = ld_cg_f32(y + i);
            for (int p = 1; p < a.parts; ++p) yv += ld_cg_f32(y + p * a.part_stride + i);
            yv = fmaf(idw, xv, yv);
            xs[i] = xv;
            ys[i] = yv;
            ss = fmaf(yv, yv, ss);
        }
        const float inv = 1.0f / sqrtf(block_sum(ss, part) / (float)a.W + a.eps);
        for (int i = tid; i < Wp; i += THREADS) xs[i] = i < a.W ? fmaf(a.mult, (ys[i] * inv) * __ldg(a.w + i), xs[i]) : 0.f;
    }
    __syncthreads();
    if (a.router) {
        for (int r = first; r < a.n_out; r += cluster * WARPS) {
            const uint16_t* wr = a.router + (size_t)r * a.W;
            float s = 0.f;
            if (regs && r == first) {
#pragma unroll
                for (int k = 0; k < REG4 * 4; ++k)
                    if (lane + k * 32 < a.W / 8) s = dot8(r4[k], reinterpret_cast<const float4*>(xs)[2 * (lane + k * 32)], reinterpret_cast<const float4*>(xs)[2 * (lane + k * 32) + 1], s);
            } else if ((a.W & 7) == 0) {
#pragma unroll 4
                for (int c = lane; c < a.W / 8; c += 32)
                    s = dot8(__ldg(reinterpret_cast<const uint4*>(wr) + c), reinterpret_cast<const float4*>(xs)[2 * c], reinterpret_cast<const float4*>(xs)[2 * c + 1], s);
            } else {
                for (int i = lane; i < a.W; i += 32) s = fmaf(bf16_bits_to_f32(__ldg(wr + i)), xs[i], s);
            }
            s = warp_sum(s);
            if (lane == 0) {
                if (rank == 0) z[r] = s;
                else st_dsmem_f32(dsmem_addr(z + r, 0u), s);
            }
        }
        if (rank == 0 && a.out.dense)
            for (int i = tid; i < a.experts; i += THREADS) a.out.dense[(size_t)m * a.experts + i] = 0.f;
    }
    // the residual is stored when every CTA of the row has read it
    if (cluster > 1) cluster_sync_all();
    else __syncthreads();
    if (a.router && rank == 0 && warp == 0) choose_experts(RouteSpec{a.correction, a.experts, a.n_out, a.top, 1.f, a.out}, m, z, choice);
    const int c_n = a.xp ? (a.W + 63) / 64 * 8 : Wp / 8;
    for (int c = rank * THREADS + tid; c < c_n; c += cluster * THREADS) {
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = c < Wp / 8 ? xs[c * 8 + e] : 0.f;
        if (a.xp) tc_xpack_store8(a.xp, a.xp_mpad, m, c * 8, v);
        float* o = a.x + (size_t)m * a.W + c * 8;
        if ((a.W & 7) == 0) {
            if (c < a.W / 8) {
                reinterpret_cast<float4*>(o)[0] = make_float4(v[0], v[1], v[2], v[3]);
                reinterpret_cast<float4*>(o)[1] = make_float4(v[4], v[5], v[6], v[7]);
            }
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (c * 8 + e < a.W) o[e] = v[e];
        }
    }
}

// ---- experts, a pair at a time -----------------------------------------------------------------------
// A warp reads rows of 128 bytes (64 k) with eight lanes each; a lane's 16-byte piece p of row R holds the k's of piece p ^ (R & 7).
__global__ void __launch_bounds__(THREADS) expert_gate_up_kernel(const ExpertWeights w, const float* __restrict__ x, const int32_t* __restrict__ ids, const float* __restrict__ weights, float* __restrict__ act) {
    extern __shared__ __align__(16) float xs[];  // [W padded to 64]
    __shared__ float red[WARPS][2 * GU_ROWS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, pair = blockIdx.y, m = pair / w.top;
    const int blocks = expert_blocks(w.ff), blk = blockIdx.x / (64 / GU_ROWS), sub = blockIdx.x % (64 / GU_ROWS), kbs = (w.W + 63) / 64;
    pdl_wait();
    pdl_launch_dependents();  // not earlier: the launch behind relies on the router's choice from its start
    const int e = __ldcg(ids + pair);
    if (e < 0 || e >= w.n) return;
    const float rw = ld_cg_f32(weights + pair);
    const uint16_t* base = w.gu + ((size_t)e * blocks + blk) * kbs * TILE;
    const int r8 = lane >> 3, p = lane & 7;
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    // loads j = 0..3: gate rows sub * 16 + 4 j + r8; j = 4..7: up rows
    const uint16_t* src[2] = {base + (size_t)(sub * GU_ROWS + r8) * 64 + p * 8, base + (size_t)(64 + sub * GU_ROWS + r8) * 64 + p * 8};
    uint4 v[8], next[8];
    auto fetch = [&](int kb, uint4 (&t)[8]) {
#pragma unroll
        for (int j = 0; j < 8; ++j) t[j] = ld_stream_u4(src[j >> 2] + (size_t)kb * TILE + (size_t)(j & 3) * 4 * 64);
    };
    if (warp < kbs) fetch(warp, next);
    stage_row<THREADS, false>(x + (size_t)m * w.W, xs, w.W, tid);
    for (int i = w.W + tid; i < kbs * 64; i += THREADS) xs[i] = 0.f;
    __syncthreads();
    for (int kb = warp; kb < kbs; kb += WARPS) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = next[j];
        if (kb + WARPS < kbs) fetch(kb + WARPS, next);
        float4 xa[2], xb[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const float* xk = xs + kb * 64 + (p ^ ((h * 4 + r8) & 7)) * 8;
            xa[h] = *reinterpret_cast<const float4*>(xk);
            xb[h] = *reinterpret_cast<const float4*>(xk + 4);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = dot8(v[j], xa[j & 1], xb[j & 1], acc[j]);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
#pragma unroll
        for (int o = 1; o < 8; o <<= 1) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], o);
        if (p == 0) red[warp][(j >> 2) * GU_ROWS + (j & 3) * 4 + r8] = acc[j];
    }
    __syncthreads();
    if (tid < GU_ROWS) {
        float g = 0.f, u = 0.f;
#pragma unroll
        for (int i = 0; i < WARPS; ++i) {
            g += red[i][tid];
            u += red[i][GU_ROWS + tid];
        }
        act[(size_t)pair * blocks * 64 + blk * 64 + sub * GU_ROWS + tid] = (w.act == GLU_CLAMPED ? clamped_glu(g, u, w.limit) : glu(w.act, g, u, w.limit)) * rw;
    }
}

// staged: the row's activations [top][ff padded] fit shared memory
__global__ void __launch_bounds__(THREADS) expert_down_kernel(const ExpertWeights w, const float* __restrict__ act, const int32_t* __restrict__ ids, const float* resid, float* y, int staged) {
    extern __shared__ __align__(16) float as[];
    __shared__ float red[WARPS][DOWN_ROWS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, m = blockIdx.y;
    const int blocks = expert_blocks(w.ff), nbs = (w.W + 127) / 128, nb = blockIdx.x / (128 / DOWN_ROWS), sub = blockIdx.x % (128 / DOWN_ROWS);
    const int units = w.top * blocks;
    const float* row = act + (size_t)m * units * 64;
    int* s_id = reinterpret_cast<int*>(as + (staged ? units * 64 : 0));
    pdl_launch_dependents();
    // the router's choice was complete before the gate / up projection let this launch start: weights are requested ahead of the wait,
    // the first ones into registers, the others into the L2
    for (int i = tid; i < w.top; i += THREADS) s_id[i] = __ldcg(ids + m * w.top + i);
    __syncthreads();
    const int r8 = lane >> 3, p = lane & 7;
    float acc[2] = {0.f, 0.f};
    const size_t sub_off = (size_t)sub * DOWN_ROWS * 64, row_off = (size_t)r8 * 64 + p * 8;
    auto tile = [&](int u) -> const uint16_t* {  // this CTA's rows of the u-th block of the chosen experts
        const int slot = u / blocks, e = u < units ? s_id[slot] : -1;
        return e < 0 || e >= w.n ? nullptr : w.down + (((size_t)e * nbs + nb) * blocks + (u - slot * blocks)) * TILE + sub_off;
    };
    constexpr int B = 4;  // blocks of a warp at a time
    uint4 v[B][2], next[B][2];
    const uint16_t *on[B], *next_on[B];
    auto fetch = [&](int u0, uint4 (&t)[B][2], const uint16_t* (&o)[B]) {
#pragma unroll
        for (int i = 0; i < B; ++i) {
            o[i] = tile(u0 + i * WARPS);
            if (o[i]) {
                t[i][0] = ld_stream_u4(o[i] + row_off);
                t[i][1] = ld_stream_u4(o[i] + row_off + 4 * 64);
            }
        }
    };
    fetch(warp, next, next_on);
    for (int u = B * WARPS + tid; u < units; u += THREADS)
        if (const uint16_t* t = tile(u)) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(t), "r"(DOWN_ROWS * 128) : "memory");
    pdl_wait();
    if (staged) stage_row<THREADS, false>(row, as, units * 64, tid);
    __syncthreads();
    for (int u0 = warp; u0 < units; u0 += B * WARPS) {
#pragma unroll
        for (int i = 0; i < B; ++i) {
            v[i][0] = next[i][0];
            v[i][1] = next[i][1];
            on[i] = next_on[i];
        }
        fetch(u0 + B * WARPS, next, next_on);
#pragma unroll
        for (int i = 0; i < B; ++i)
            if (on[i]) {
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int k = (u0 + i * WARPS) * 64 + (p ^ ((h * 4 + r8) & 7)) * 8;
                    const float4 q0 = staged ? *reinterpret_cast<const float4*>(as + k) : ld_cg_f32x4(row + k), q1 = staged ? *reinterpret_cast<const float4*>(as + k + 4) : ld_cg_f32x4(row + k + 4);
                    acc[h] = dot8(v[i][h], q0, q1, acc[h]);
                }
            }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
#pragma unroll
        for (int o = 1; o < 8; o <<= 1) acc[h] += __shfl_xor_sync(0xffffffffu, acc[h], o);
        if (p == 0) red[warp][h * 4 + r8] = acc[h];
    }
    __syncthreads();
    const int n = nb * 128 + sub * DOWN_ROWS + tid;
    if (tid < DOWN_ROWS && n < w.W) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < WARPS; ++i) s += red[i][tid];
        y[(size_t)m * w.W + n] = resid ? ld_cg_f32(resid + (size_t)m * w.W + n) + s : s;
    }
}

template <typename... KArgs, typename... Args>
cudaError_t launch(void (*kern)(KArgs...), dim3 grid, size_t smem, int cluster, cudaStream_t st, bool pdl, Args... args) {
    const cudaError_t e = ensure_dyn_smem(kern, smem);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
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
        at[n].val.clusterDim.y = 1;
        at[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = at;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, kern, KArgs(args)...);
}

}  // namespace

size_t expert_gu_elems(int W, int ff) { return (size_t)expert_blocks(ff) * ((W + 63) / 64) * TILE; }
size_t expert_down_elems(int W, int ff) { return (size_t)((W + 127) / 128) * expert_blocks(ff) * TILE; }

cudaError_t launch_post_norm(const PostNormArgs& a, int sm_count, cudaStream_t st, bool pdl) {
    int cluster = 1;
    if (a.router)
        while (cluster < 8 && 2 * cluster * a.M <= sm_count && cluster * WARPS < a.n_out) cluster *= 2;
    const size_t smem = sizeof(float) * (2 * (size_t)((a.W + 7) & ~7) + 2 * (size_t)(a.router ? a.n_out : 0));
    PostNormArgs b = a;
    if (!a.router) b.n_out = 0;
    return launch(post_norm_kernel, dim3((unsigned)(a.M * cluster)), smem, cluster, st, pdl, b, cluster);
}

cudaError_t launch_expert_gate_up(const ExpertWeights& e, const float* x, int M, const RouteOut& r, float* act, cudaStream_t st, bool pdl) {
    const size_t smem = sizeof(float) * (size_t)((e.W + 63) / 64) * 64;
    return launch(expert_gate_up_kernel, dim3((unsigned)(expert_blocks(e.ff) * (64 / GU_ROWS)), (unsigned)(M * e.top)), smem, 1, st, pdl, e, x, r.ids, r.weights, act);
}

cudaError_t launch_expert_down(const ExpertWeights& e, const float* act, int M, const RouteOut& r, const float* resid, float* y, cudaStream_t st, bool pdl) {
    const size_t rows = sizeof(float) * (size_t)e.top * expert_blocks(e.ff) * 64;
    const int staged = rows <= 128 * 1024;
    const size_t smem = (staged ? rows : 0) + sizeof(int) * e.top;
    return launch(expert_down_kernel, dim3((unsigned)((e.W + 127) / 128 * (128 / DOWN_ROWS)), (unsigned)M), smem, 1, st, pdl, e, act, r.ids, resid, y, staged);
}

}  // namespace hm
