// See recur.h.
#include "recur.h"

#include "launch_attrs.h"

namespace hm {
namespace {

// Shared memory of a CTA, in floats from the front.  rows: of the longest run.
struct RecurSmem {
    int q, k, alpha, v, beta, kq, sq, o, total;
};
__host__ __device__ __forceinline__ RecurSmem recur_smem(const RecurArgs& a, int rows) {
    RecurSmem s;
    const int DP = a.shape.rows * a.shape.lanes, kept = a.shape.slices > 1 ? rows : a.step;
    int at = 0;
    auto take = [&](int n) {
        const int first = at;
        at += (n + 3) & ~3;
        return first;
    };
    s.q = take(a.step * DP);
    s.k = take(a.step * DP);
    s.alpha = take(a.kind == LIN_DELTA ? a.step * DP : 0);
    s.v = take(a.step * a.shape.cols);
    s.beta = take(a.kind == LIN_DELTA ? a.step : 0);
    s.kq = take(a.kind == LIN_DELTA ? a.step : 0);
    s.sq = take(2 * a.shape.cluster * kept);
    s.o = take(kept * a.shape.share);
    s.total = at;
    return s;
}

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// RD: state rows of a thread.
template <int RD, int KIND>
__global__ void __launch_bounds__(GLA_THREADS, RD > 32 ? 1 : 2) recur_kernel(const __grid_constant__ RecurArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int CS = a.shape.cluster, LP = a.shape.lanes, CP = a.shape.cols, DP = RD * LP, D4 = DP / 4, dim = a.dim, vdim = a.vdim, slices = a.shape.slices, TR = a.step, share = a.shape.share;
    const int cta = blockIdx.x % CS, head = blockIdx.x / CS % a.heads, run = blockIdx.x / CS / a.heads, kvh = head / (a.heads / a.kv_heads);
    const int c_lo = min(vdim, cta * share), c_n = min(vdim, c_lo + share) - c_lo;  // this CTA's columns
    const int col = tid / LP, part = tid - col * LP;
    int first = run, end = run + 1;
    if (a.runs.n) {
        first = a.runs.row[run];
        end = a.runs.row[run + 1];
    }
    const int n = end - first, kept = slices > 1 ? n : TR;
    const RecurSmem lay = recur_smem(a, a.runs.n ? a.longest_run : 1);
    float *qs = sm + lay.q, *ks = sm + lay.k, *as = sm + lay.alpha, *vs = sm + lay.v, *bs = sm + lay.beta, *kq = sm + lay.kq, *os = sm + lay.o, *sq = sm + lay.sq;
    pdl_launch_dependents();
    const int seq = a.row_seq[first], pos = a.row_pos[first], ldd = gla_pad(dim);
    float* const state = a.state + (size_t)seq * a.seq_stride + (size_t)head * vdim * ldd;
    const float decay = KIND == LIN_RETENTION ? __ldg(a.decay + head) : 0.f;
    const bool vec = ((a.head_ld | a.ldq | a.ldk) & 3) == 0 && ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k)) & 15) == 0;
    const bool avec = (dim & 3) == 0;
    if (CS > 1) cluster_sync_all();  // nobody stores into a CTA that has not started
    bool waited = a.early == 0;
    if (waited) pdl_wait();
    int turn = 0;
    // norm, gate and store of rows r0 .. of the run, which `os` holds from its front on
    auto finish = [&](int r0, int rows) {
        __syncthreads();
        float* sums = sq + (turn++ & 1) * CS * kept;  // [CTA][rows]
        for (int t = warp; t < rows; t += GLA_THREADS / 32) {
            float s = 0.f;
            for (int c = lane; c < c_n; c += 32) s = fmaf(os[t * share + c], os[t * share + c], s);
            s = warp_sum(s);
            if (lane < CS) {
                if (CS > 1) st_dsmem_f32(dsmem_addr(sums + cta * kept + t, (uint32_t)lane), s);
                else sums[t] = s;
            }
        }
        if (CS > 1) cluster_sync_all();
        else __syncthreads();
        const bool pieces = a.xp && ((vdim | a.out_off | share) & 7) == 0;
        const int per = pieces ? c_n / 8 : c_n;
        for (int i = tid; i < rows * per; i += GLA_THREADS) {
            const int t = i / per, c = (i - t * per) * (pieces ? 8 : 1), m = first + r0 + t, k0 = a.out_off + head * vdim + c_lo + c;
            const float *g = a.gate + (size_t)m * a.ld_gate + (size_t)head * vdim + c_lo + c, *o = os + t * share + c;
            float s = 0.f;
            for (int r = 0; r < CS; ++r) s += sums[r * kept + t];
            const float f = 1.0f / sqrtf(s / (float)vdim + a.eps);
            auto value = [&](int e, float z) {
                const float w = a.norm_w ? __ldg(a.norm_w + c_lo + c + e) : 1.f, y = (o[e] * f) * w;
                return KIND == LIN_RETENTION ? y * (z * sigmoid(z)) : y * sigmoid(z);
            };
            if (pieces) {
                const float4 g0 = ld_cg_f32x4(g), g1 = ld_cg_f32x4(g + 4);
                const float gv[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
                float v[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = value(e, gv[e]);
                tc_xpack_store8(a.xp, a.xp_mpad, m, k0, v);
            } else {
                const float v = value(0, ld_cg_f32(g));
                if (a.xp) tc_xpack_store(a.xp, a.xp_mpad, m, k0, v);
                else a.out[(size_t)m * a.ld_out + k0] = v;
            }
        }
    };
    for (int sl = 0; sl < slices; ++sl) {
        const int c = sl * CP + col;
        const bool on = c < c_n;
        float4* const column = reinterpret_cast<float4*>(state + (size_t)(c_lo + (on ? c : 0)) * ldd) + part;
        float4 S[RD / 4];
#pragma unroll
        for (int j = 0; j < RD / 4; ++j) S[j] = on && pos > 0 && (j * LP + part) * 4 < dim ? __ldcg(column + j * LP) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (!waited) {
            pdl_wait();
            waited = true;
        }
        for (int t0 = 0; t0 < n; t0 += TR) {
            const int tr = min(TR, n - t0);
            __syncthreads();  // the tokens in front are done with
            const float *qr = a.q + (size_t)(first + t0) * a.ldq + (size_t)kvh * a.head_ld, *kr = a.k + (size_t)(first + t0) * a.ldk + (size_t)kvh * a.head_ld;
            const float* ar = KIND == LIN_DELTA ? a.alpha + ((size_t)(first + t0) * a.heads + head) * dim : nullptr;
            if (vec) {  // (elements behind a head's last one, up to a multiple of four, are zeros or masked here)
#pragma unroll 4
                for (int i = tid; i < tr * D4; i += GLA_THREADS) {
                    const int t = i / D4, d = (i - t * D4) * 4;
                    float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
                    if (d < dim) {
                        q = ld_cg_f32x4(qr + (size_t)t * a.ldq + d);
                        k = ld_cg_f32x4(kr + (size_t)t * a.ldk + d);
                    }
                    reinterpret_cast<float4*>(qs)[i] = make_float4(q.x * a.q_scale, q.y * a.q_scale, q.z * a.q_scale, q.w * a.q_scale);
                    reinterpret_cast<float4*>(ks)[i] = k;
                }
            } else {
                for (int i = tid; i < tr * DP; i += GLA_THREADS) {
                    const int t = i / DP, d = i - t * DP;
                    qs[i] = d < dim ? ld_cg_f32(qr + (size_t)t * a.ldq + d) * a.q_scale : 0.f;
                    ks[i] = d < dim ? ld_cg_f32(kr + (size_t)t * a.ldk + d) : 0.f;
                }
            }
            if constexpr (KIND == LIN_DELTA) {
                if (avec) {
#pragma unroll 4
                    for (int i = tid; i < tr * D4; i += GLA_THREADS) {
                        const int t = i / D4, d = (i - t * D4) * 4;
                        reinterpret_cast<float4*>(as)[i] = d < dim ? ld_cg_f32x4(ar + (size_t)t * a.heads * dim + d) : make_float4(0.f, 0.f, 0.f, 0.f);
                    }
                } else {
                    for (int i = tid; i < tr * DP; i += GLA_THREADS) {
                        const int t = i / DP, d = i - t * DP;
                        as[i] = d < dim ? ld_cg_f32(ar + (size_t)t * a.heads * dim + d) : 0.f;
                    }
                }
                for (int t = tid; t < tr; t += GLA_THREADS) bs[t] = sigmoid(ld_cg_f32(a.beta + (size_t)(first + t0 + t) * a.ld_beta + head));
            }
#pragma unroll 4
            for (int i = tid; i < tr * CP; i += GLA_THREADS) {
                const int t = i / CP, cc = sl * CP + i - t * CP;
                vs[i] = cc < c_n ? ld_cg_f32(a.v + (size_t)(first + t0 + t) * a.ldv + (size_t)head * vdim + c_lo + cc) : 0.f;
            }
            __syncthreads();
            if constexpr (KIND == LIN_DELTA) {  // k . q: what a token's own write adds to its result
                for (int t = warp; t < tr; t += GLA_THREADS / 32) {
                    float s = 0.f;
                    for (int d = lane; d < DP; d += 32) s = fmaf(ks[t * DP + d], qs[t * DP + d], s);
                    s = warp_sum(s);
                    if (lane == 0) kq[t] = s;
                }
                __syncthreads();
            }
            float* const orow = os + (size_t)(slices > 1 ? t0 : 0) * share + c;
            if constexpr (KIND == LIN_RETENTION) {
                auto step = [&](int t) -> float {  // this thread's share of o
                    const float v = vs[t * CP + col];
                    const float4 *q4 = reinterpret_cast<const float4*>(qs + t * DP) + part, *k4 = reinterpret_cast<const float4*>(ks + t * DP) + part;
                    float o0 = 0.f, o1 = 0.f;
#pragma unroll
                    for (int j = 0; j < RD / 4; ++j) {
                        const float4 k = k4[j * LP], q = q4[j * LP];
                        S[j].x = fmaf(S[j].x, decay, k.x * v);
                        S[j].y = fmaf(S[j].y, decay, k.y * v);
                        S[j].z = fmaf(S[j].z, decay, k.z * v);
                        S[j].w = fmaf(S[j].w, decay, k.w * v);
                        o0 = fmaf(S[j].x, q.x, fmaf(S[j].y, q.y, o0));
                        o1 = fmaf(S[j].z, q.z, fmaf(S[j].w, q.w, o1));
                    }
                    return o0 + o1;
                };
                int t = 0;
                constexpr int U = RD <= 16 ? 4 : 2;  // tokens whose sums over the lanes go side by side
                for (; t + U <= tr; t += U) {
                    float o[U];
#pragma unroll
                    for (int u = 0; u < U; ++u) o[u] = step(t + u);
                    for (int s = 1; s < LP; s <<= 1)
#pragma unroll
                        for (int u = 0; u < U; ++u) o[u] += __shfl_xor_sync(0xffffffffu, o[u], s);
                    if (part == 0 && on)
#pragma unroll
                        for (int u = 0; u < U; ++u) orow[(t + u) * share] = o[u];
                }
                for (; t < tr; ++t) {
                    float o = step(t);
                    for (int s = 1; s < LP; s <<= 1) o += __shfl_xor_sync(0xffffffffu, o, s);
                    if (part == 0 && on) orow[t * share] = o;
                }
            } else {
                for (int t = 0; t < tr; ++t) {
                    const float4 *q4 = reinterpret_cast<const float4*>(qs + t * DP) + part, *k4 = reinterpret_cast<const float4*>(ks + t * DP) + part, *a4 = reinterpret_cast<const float4*>(as + t * DP) + part;
                    // both sums over the shrunk state go through the lanes side by side: what it gives back for k, and for q
                    float sk0 = 0.f, sk1 = 0.f, sq0 = 0.f, sq1 = 0.f;
#pragma unroll
                    for (int j = 0; j < RD / 4; ++j) {
                        const float4 al = a4[j * LP], k = k4[j * LP], q = q4[j * LP];
                        S[j].x *= al.x; S[j].y *= al.y; S[j].z *= al.z; S[j].w *= al.w;
                        sk0 = fmaf(S[j].x, k.x, fmaf(S[j].y, k.y, sk0));
                        sk1 = fmaf(S[j].z, k.z, fmaf(S[j].w, k.w, sk1));
                        sq0 = fmaf(S[j].x, q.x, fmaf(S[j].y, q.y, sq0));
                        sq1 = fmaf(S[j].z, q.z, fmaf(S[j].w, q.w, sq1));
                    }
                    float sk = sk0 + sk1, so = sq0 + sq1;
                    for (int s = 1; s < LP; s <<= 1) {
                        sk += __shfl_xor_sync(0xffffffffu, sk, s);
                        so += __shfl_xor_sync(0xffffffffu, so, s);
                    }
                    const float u = bs[t] * (vs[t * CP + col] - sk);
#pragma unroll
                    for (int j = 0; j < RD / 4; ++j) {
                        const float4 k = k4[j * LP];
                        S[j].x = fmaf(k.x, u, S[j].x); S[j].y = fmaf(k.y, u, S[j].y); S[j].z = fmaf(k.z, u, S[j].z); S[j].w = fmaf(k.w, u, S[j].w);
                    }
                    if (part == 0 && on) orow[t * share] = fmaf(kq[t], u, so);
                }
            }
            if (slices == 1) finish(t0, tr);
        }
#pragma unroll
        for (int j = 0; j < RD / 4; ++j)
            if (on && (j * LP + part) * 4 < dim) __stcg(column + j * LP, S[j]);
    }
    if (slices > 1) finish(0, n);
}

template <int RD, int KIND>
cudaError_t launch(const RecurArgs& a, unsigned blocks, size_t smem, cudaStream_t st, bool pdl) {
    const cudaError_t e = ensure_dyn_smem(recur_kernel<RD, KIND>, smem);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(blocks);
    cfg.blockDim = dim3(GLA_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    int n = 0;
    if (pdl) {
        at[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        at[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    if (a.shape.cluster > 1) {
        at[n].id = cudaLaunchAttributeClusterDimension;
        at[n].val.clusterDim.x = (unsigned)a.shape.cluster;
        at[n].val.clusterDim.y = at[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = at;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, recur_kernel<RD, KIND>, a);
}

template <int KIND>
cudaError_t launch_kind(const RecurArgs& a, unsigned blocks, size_t smem, cudaStream_t st, bool pdl) {
    switch (a.shape.rows) {
        case 4: return launch<4, KIND>(a, blocks, smem, st, pdl);
        case 8: return launch<8, KIND>(a, blocks, smem, st, pdl);
        case 16: return launch<16, KIND>(a, blocks, smem, st, pdl);
        case 32: return launch<32, KIND>(a, blocks, smem, st, pdl);
        case 64: return launch<64, KIND>(a, blocks, smem, st, pdl);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

cudaError_t launch_recur(const RecurArgs& a_in, int sm_count, cudaStream_t st, bool pdl) {
    RecurArgs a = a_in;
    if (a.M < 1 || a.M > GQA_MAX_ROWS || a.dim > GLA_MAX_DIM || a.vdim > GLA_MAX_VDIM || a.heads % a.kv_heads != 0 || (a.kind != LIN_RETENTION && a.kind != LIN_DELTA)) return cudaErrorInvalidValue;
    const int runs = a.runs.n ? a.runs.n : a.M, rows = a.runs.n ? a.longest_run : 1;
    a.shape = gla_shape(a.dim, a.vdim, runs * a.heads, sm_count);
    for (a.step = rows; a.step > 1 && (size_t)recur_smem(a, rows).total * 4 > 110 * 1024; a.step = (a.step + 1) / 2) {
    }
    const size_t smem = (size_t)recur_smem(a, rows).total * 4;
    const unsigned blocks = (unsigned)(runs * a.heads * a.shape.cluster);
    return a.kind == LIN_DELTA ? launch_kind<LIN_DELTA>(a, blocks, smem, st, pdl) : launch_kind<LIN_RETENTION>(a, blocks, smem, st, pdl);
}

}  // namespace hm
