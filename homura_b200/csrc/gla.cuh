// Device side of gated linear attention (gla.h): one CTA = one head of one run.
#pragma once
#include "gla.h"

namespace hm {

constexpr int GLA_UP_SMEM = 8192;  // floats of a head's decay projection that are staged ahead of the dependency

// sigmoid(z)^t
__device__ __forceinline__ float gla_decay(float z, float t) { return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * t); }

template <int RD>
__device__ __forceinline__ void gla_block(const GlaArgs& a, int head, int run, float* sm) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int LP = a.shape.lanes, CP = a.shape.cols, DP = RD * LP, dim = a.dim, vdim = a.vdim, rank = a.rank, slices = a.shape.slices, TR = a.step;
    const int col = tid / LP, part = tid - col * LP;
    int first = run, end = run + 1;
    if (a.runs.n) {
        first = a.runs.row[run];
        end = a.runs.row[run + 1];
    }
    const int n = end - first, kept = slices > 1 ? n : TR;
    const bool staged_up = rank * dim <= GLA_UP_SMEM;
    float* ups = sm;                                   // [rank][dim]
    float* qs = ups + (staged_up ? (rank * dim + 3) / 4 * 4 : 0);  // [TR][DP]
    float* ks = qs + TR * DP;
    float* as = ks + TR * DP;
    float* vs = as + TR * DP;                          // [TR][CP]
    float* as1 = vs + TR * CP;                         // [TR][rank]
    float* os = as1 + TR * rank;                       // [kept][vdim]
    const float* up = a.up + (size_t)head * rank * dim;
    if (staged_up) {
        for (int i = tid; i < rank * dim; i += GLA_THREADS) ups[i] = __ldg(up + i);
        up = ups;
    }
    if (!a.early) pdl_wait();
    const int seq = a.row_seq[first], pos = a.row_pos[first];
    float4* const state = reinterpret_cast<float4*>(a.state + (size_t)seq * a.seq_stride + head * a.shape.state_floats());
    auto finish = [&](int r0, int rows) {  // norm, gate and store of rows r0 .. of the run, which `os` holds from its front on
        __syncthreads();
        for (int t = warp; t < rows; t += GLA_THREADS / 32) {
            const float* o = os + (size_t)t * vdim;
            const int m = first + r0 + t;
            const float* g = a.raw + (size_t)m * a.ld + a.g_off + (size_t)head * vdim;
            float s = 0.f;
            for (int c = lane; c < vdim; c += 32) s = fmaf(o[c], o[c], s);
            const float inv = 1.0f / sqrtf(warp_sum(s) / (float)vdim + a.eps);
            const int k0 = a.out_off + head * vdim;
            auto at = [&](int c) {
                const float z = ld_cg_f32(g + c);
                return ((o[c] * inv) * __ldg(a.norm_w + c)) * (z / (1.0f + expf(-z))) * a.out_scale;
            };
            if (a.xp && ((vdim | a.out_off) & 7) == 0) {
                for (int c = lane * 8; c < vdim; c += 256) {
                    float v[8];
#pragma unroll
                    for (int e = 0; e < 8; ++e) v[e] = at(c + e);
                    tc_xpack_store8(a.xp, a.xp_mpad, m, k0 + c, v);
                }
            } else {
                for (int c = lane; c < vdim; c += 32) {
                    if (a.xp) tc_xpack_store(a.xp, a.xp_mpad, m, k0 + c, at(c));
                    else a.out[(size_t)m * a.ld_out + k0 + c] = at(c);
                }
            }
        }
    };
    for (int sl = 0; sl < slices; ++sl) {
        float4 S[RD / 4];
#pragma unroll
        for (int j = 0; j < RD / 4; ++j) S[j] = pos > 0 ? __ldcg(state + (size_t)(sl * (RD / 4) + j) * GLA_THREADS + tid) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (a.early && sl == 0) pdl_wait();
        for (int t0 = 0; t0 < n; t0 += TR) {
            const int tr = min(TR, n - t0);
            __syncthreads();
            const float* raw = a.raw + (size_t)(first + t0) * a.ld;
            for (int i = tid; i < tr * rank; i += GLA_THREADS) {
                const int t = i / rank;
                as1[i] = ld_cg_f32(raw + (size_t)t * a.ld + a.a_off + (i - t * rank));
            }
            for (int i = tid; i < tr * DP; i += GLA_THREADS) {
                const int t = i / DP, d = i - t * DP;
                const float* row = raw + (size_t)t * a.ld + (size_t)head * dim + d;
                qs[i] = d < dim ? ld_cg_f32(row + a.q_off) * a.q_scale : 0.f;
                ks[i] = d < dim ? ld_cg_f32(row + a.k_off) : 0.f;
            }
            for (int i = tid; i < tr * CP; i += GLA_THREADS) {
                const int t = i / CP, c = sl * CP + i - t * CP;
                vs[i] = c < vdim ? ld_cg_f32(raw + (size_t)t * a.ld + a.v_off + (size_t)head * vdim + c) : 0.f;
            }
            __syncthreads();
            for (int i = tid; i < tr * DP; i += GLA_THREADS) {
                const int t = i / DP, d = i - t * DP;
                float v = 0.f;
                if (d < dim) {
                    float z = 0.f;
#pragma unroll 8
                    for (int r = 0; r < rank; ++r) z = fmaf(up[r * dim + d], as1[t * rank + r], z);
                    v = gla_decay(z + __ldg(a.bias + (size_t)head * dim + d), a.inv_tau);
                }
                as[i] = v;
            }
            __syncthreads();
            for (int t = 0; t < tr; ++t) {
                const float v = vs[t * CP + col];
                const float4 *q4 = reinterpret_cast<const float4*>(qs + t * DP) + part, *k4 = reinterpret_cast<const float4*>(ks + t * DP) + part, *a4 = reinterpret_cast<const float4*>(as + t * DP) + part;
                float o0 = 0.f, o1 = 0.f;
#pragma unroll
                for (int j = 0; j < RD / 4; ++j) {
                    const float4 al = a4[j * LP], k = k4[j * LP], q = q4[j * LP];
                    S[j].x = fmaf(S[j].x, al.x, k.x * v);
                    S[j].y = fmaf(S[j].y, al.y, k.y * v);
                    S[j].z = fmaf(S[j].z, al.z, k.z * v);
                    S[j].w = fmaf(S[j].w, al.w, k.w * v);
                    o0 = fmaf(S[j].x, q.x, fmaf(S[j].y, q.y, o0));
                    o1 = fmaf(S[j].z, q.z, fmaf(S[j].w, q.w, o1));
                }
                float o = o0 + o1;
                for (int s = 1; s < LP; s <<= 1) o += __shfl_xor_sync(0xffffffffu, o, s);
                const int c = sl * CP + col;
                if (part == 0 && c < vdim) os[(size_t)(slices > 1 ? t0 + t : t) * vdim + c] = o;
            }
            if (slices == 1) finish(t0, tr);
        }
#pragma unroll
        for (int j = 0; j < RD / 4; ++j) __stcg(state + (size_t)(sl * (RD / 4) + j) * GLA_THREADS + tid, S[j]);
    }
    if (slices > 1) finish(0, n);
    (void)kept;
}

}  // namespace hm
