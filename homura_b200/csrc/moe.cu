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

namespace hm {
namespace {

constexpr int THREADS = 256, WARPS = THREADS / 32;
constexpr int TILE = 128 * 64;  // elements of a tile image: 128 rows of 64 k, 16-byte pieces XOR-ed by row & 7
constexpr int GU_ROWS = 16, DOWN_ROWS = 8;

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

// softmax over the router's outputs, choice by score + correction (ties to the lower index), weights without it: one warp
__device__ __forceinline__ void choose(const PostNormArgs& a, int m, float* z, float* choice) {
    const int lane = threadIdx.x & 31;
    float mx = -INFINITY, l = 0.f;
    for (int r = lane; r < a.n_out; r += 32) mx = fmaxf(mx, z[r]);
    mx = warp_max(mx);
    for (int r = lane; r < a.n_out; r += 32) {
        const float e = expf(z[r] - mx);
        z[r] = e;
        l += e;
    }
    l = warp_sum(l);
    for (int r = lane; r < a.n_out; r += 32) {
        const float s = z[r] / l;
        z[r] = s;
        choice[r] = s + __ldg(a.correction + r);
    }
    __syncwarp();
    float ident = 0.f;
    for (int k = 0; k < a.top; ++k) {
        float bv = -INFINITY;
        int bi = a.n_out;
        for (int r = lane; r < a.n_out; r += 32)
            if (choice[r] > bv || bi == a.n_out) {
                bv = choice[r];
                bi = r;
            }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (oi < a.n_out && (bi == a.n_out || ov > bv || (ov == bv && oi < bi))) {
                bv = ov;
                bi = oi;
            }
        }
        const float s = z[bi];
        if (lane == 0) {
            choice[bi] = -INFINITY;
            const bool id = bi >= a.experts;
            a.out.ids[(size_t)m * a.top + k] = id ? -1 : bi;
            a.out.weights[(size_t)m * a.top + k] = s;
            if (id) ident += s;
            else if (a.out.dense) {
                a.out.dense[(size_t)m * a.experts + bi] = s;
                a.out.mask[(size_t)m * ((a.experts + 31) / 32) + bi / 32] |= 1u << (bi & 31);
            }
        }
        __syncwarp();
    }
    if (lane == 0) a.out.identity[m] = ident;
}

__global__ void __launch_bounds__(THREADS) post_norm_kernel(const PostNormArgs a, int cluster) {
    extern __shared__ __align__(16) float sm[];
    const int Wp = (a.W + 7) & ~7;
    float *xs = sm, *ys = xs + Wp, *z = ys + Wp, *choice = z + a.n_out;
    __shared__ float part[WARPS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, m = blockIdx.x / cluster, rank = blockIdx.x - m * cluster;
    pdl_launch_dependents();
    if (cluster > 1) {  // every CTA of the cluster has started before the first one stores into rank 0
        cluster_arrive_release();
        cluster_wait_acquire();
    }
    pdl_wait();
    const float idw = a.identity ? ld_cg_f32(a.identity + m) : 0.f;
    const float *x = a.x + (size_t)m * a.W, *y = a.y + (size_t)m * a.W;
    float ss = 0.f;
    if ((a.W & 3) == 0) {
#pragma unroll 2
        for (int i = tid; i < a.W / 4; i += THREADS) {
            const float4 xv = ld_cg_f32x4(x + 4 * (size_t)i);
            float4 yv = ld_cg_f32x4(y + 4 * (size_t)i);
            for (int p = 1; p < a.parts; ++p) {
                const float4 t = ld_cg_f32x4(y + p * a.part_stride + 4 * (size_t)i);
                yv = make_float4(yv.x + t.x, yv.y + t.y, yv.z + t.z, yv.w + t.w);
            }
            yv = make_float4(fmaf(idw, xv.x, yv.x), fmaf(idw, xv.y, yv.y), fmaf(idw, xv.z, yv.z), fmaf(idw, xv.w, yv.w));
            reinterpret_cast<float4*>(xs)[i] = xv;
            reinterpret_cast<float4*>(ys)[i] = yv;
            ss = fmaf(yv.x, yv.x, fmaf(yv.y, yv.y, fmaf(yv.z, yv.z, fmaf(yv.w, yv.w, ss))));
        }
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
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, part) / (float)a.W + a.eps);
    for (int i = tid; i < Wp; i += THREADS) xs[i] = i < a.W ? fmaf(a.mult, (ys[i] * inv) * __ldg(a.w + i), xs[i]) : 0.f;
    __syncthreads();
    if (a.router) {
        for (int r = rank * WARPS + warp; r < a.n_out; r += cluster * WARPS) {
            const uint16_t* wr = a.router + (size_t)r * a.W;
            float s = 0.f;
            if ((a.W & 7) == 0) {
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
        if (rank == 0 && a.out.dense) {
            for (int i = tid; i < a.experts; i += THREADS) a.out.dense[(size_t)m * a.experts + i] = 0.f;
            const int words = (a.experts + 31) / 32;
            for (int i = tid; i < words; i += THREADS) a.out.mask[(size_t)m * words + i] = 0u;
        }
    }
    // the residual is stored when every CTA of the row has read it
    if (cluster > 1) cluster_sync_all();
    else __syncthreads();
    if (a.router && rank == 0 && warp == 0) choose(a, m, z, choice);
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
    pdl_launch_dependents();
    pdl_wait();
    const int e = __ldcg(ids + pair);
    if (e < 0) return;
    stage_row<THREADS, false>(x + (size_t)m * w.W, xs, w.W, tid);
    for (int i = w.W + tid; i < kbs * 64; i += THREADS) xs[i] = 0.f;
    const float rw = ld_cg_f32(weights + pair);
    __syncthreads();
    const uint16_t* base = w.gu + ((size_t)e * blocks + blk) * kbs * TILE;
    const int r8 = lane >> 3, p = lane & 7;
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    // loads j = 0..3: gate rows sub * 16 + 4 j + r8; j = 4..7: up rows
    const uint16_t* src[2] = {base + (size_t)(sub * GU_ROWS + r8) * 64 + p * 8, base + (size_t)(64 + sub * GU_ROWS + r8) * 64 + p * 8};
#pragma unroll 2
    for (int kb = warp; kb < kbs; kb += WARPS) {
        uint4 v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = ld_stream_u4(src[j >> 2] + (size_t)kb * TILE + (size_t)(j & 3) * 4 * 64);
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
        act[(size_t)pair * blocks * 64 + blk * 64 + sub * GU_ROWS + tid] = clamped_glu(g, u, w.limit) * rw;
    }
}

// staged: the row's activations [top][ff padded] fit shared memory
__global__ void __launch_bounds__(THREADS) expert_down_kernel(const ExpertWeights w, const float* __restrict__ act, const int32_t* __restrict__ ids, float* __restrict__ y, int staged) {
    extern __shared__ __align__(16) float as[];
    __shared__ float red[WARPS][DOWN_ROWS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, m = blockIdx.y;
    const int blocks = expert_blocks(w.ff), nbs = (w.W + 127) / 128, nb = blockIdx.x / (128 / DOWN_ROWS), sub = blockIdx.x % (128 / DOWN_ROWS);
    const int units = w.top * blocks;
    const float* row = act + (size_t)m * units * 64;
    int* s_id = reinterpret_cast<int*>(as + (staged ? units * 64 : 0));
    pdl_launch_dependents();
    pdl_wait();
    for (int i = tid; i < w.top; i += THREADS) s_id[i] = __ldcg(ids + m * w.top + i);
    if (staged) stage_row<THREADS, false>(row, as, units * 64, tid);
    __syncthreads();
    const int r8 = lane >> 3, p = lane & 7;
    float acc[2] = {0.f, 0.f};
    const size_t row_off = (size_t)(sub * DOWN_ROWS + r8) * 64 + p * 8;
    for (int u0 = warp; u0 < units; u0 += 4 * WARPS) {
        uint4 v[4][2];
        bool on[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int u = u0 + i * WARPS, slot = u / blocks, e = u < units ? s_id[slot] : -1;
            on[i] = e >= 0;
            if (on[i]) {
                const uint16_t* t = w.down + (((size_t)e * nbs + nb) * blocks + (u - slot * blocks)) * TILE + row_off;
                v[i][0] = ld_stream_u4(t);
                v[i][1] = ld_stream_u4(t + 4 * 64);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
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
        y[(size_t)m * w.W + n] = s;
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

cudaError_t launch_expert_down(const ExpertWeights& e, const float* act, int M, const RouteOut& r, float* y, cudaStream_t st, bool pdl) {
    const size_t rows = sizeof(float) * (size_t)e.top * expert_blocks(e.ff) * 64;
    const int staged = rows <= 128 * 1024;
    const size_t smem = (staged ? rows : 0) + sizeof(int) * e.top;
    return launch(expert_down_kernel, dim3((unsigned)((e.W + 127) / 128 * (128 / DOWN_ROWS)), (unsigned)M), smem, 1, st, pdl, e, act, r.ids, y, staged);
}

}  // namespace hm
