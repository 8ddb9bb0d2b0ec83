// Device side of gated linear attention (gla.h).
//   gla_block        one cluster of CTAs = one head of one run of tokens, state in registers
//   gla_token_block  one CTA = one head of one token, state in shared memory
#pragma once
#include "gla.h"
#include "mbarrier.cuh"

namespace hm {

// sigmoid(z)^t
__device__ __forceinline__ float gla_decay(float z, float t) { return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * t); }
__device__ __forceinline__ float gla_silu(float z) { return z / (1.0f + expf(-z)); }

__device__ __forceinline__ void st_dsmem_f32x4(uint32_t addr, const float4& v) {
    asm volatile("st.shared::cluster.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(addr), "f"(v.x), "f"(v.y), "f"(v.z), "f"(v.w) : "memory");
}

// Shared memory of a CTA, in floats from the front.  rows: of the longest run.
struct GlaSmem {
    int up, q, k, alpha, v, lat, sq, o, total;
};
__host__ __device__ __forceinline__ GlaSmem gla_smem(const GlaArgs& a, int rows) {
    GlaSmem s;
    const int DP = a.shape.rows * a.shape.lanes, kept = a.shape.slices > 1 ? rows : a.step;
    int at = 0;
    auto take = [&](int n) {
        const int first = at;
        at += (n + 3) & ~3;
        return first;
    };
    s.up = take(a.rank * a.dim <= GLA_UP_SMEM ? a.rank * a.dim : 0);
    s.q = take(a.step * DP);
    s.k = take(a.step * DP);
    s.alpha = take(a.step * DP);
    s.v = take(a.step * a.shape.cols);
    s.lat = take(a.step * a.rank);
    s.sq = take(2 * a.shape.cluster * kept);
    s.o = take(kept * a.shape.share);
    s.total = at;
    return s;
}

// RD: state rows of a thread.
template <int RD>
__device__ __forceinline__ void gla_block(const GlaArgs& a, int block, float* sm) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int CS = a.shape.cluster, LP = a.shape.lanes, CP = a.shape.cols, DP = RD * LP, D4 = DP / 4, dim = a.dim, vdim = a.vdim, rank = a.rank, slices = a.shape.slices, TR = a.step, share = a.shape.share;
    const int cta = block % CS, head = block / CS % a.heads, run = block / CS / a.heads;
    const int c_lo = min(vdim, cta * share), c_n = min(vdim, c_lo + share) - c_lo;  // this CTA's columns
    const int col = tid / LP, part = tid - col * LP;
    int first = run, end = run + 1;
    if (a.runs.n) {
        first = a.runs.row[run];
        end = a.runs.row[run + 1];
    }
    const int n = end - first, kept = slices > 1 ? n : TR;
    const GlaSmem lay = gla_smem(a, a.runs.n ? a.longest_run : 1);
    float *qs = sm + lay.q, *ks = sm + lay.k, *as = sm + lay.alpha, *vs = sm + lay.v, *lat = sm + lay.lat, *os = sm + lay.o, *sq = sm + lay.sq;
    const float* up = a.up + (size_t)head * rank * dim;
    if (rank * dim <= GLA_UP_SMEM) {
        for (int i = tid; i < rank * dim; i += GLA_THREADS) sm[lay.up + i] = __ldg(up + i);
        up = sm + lay.up;
    }
    const int seq = a.row_seq[first], pos = a.row_pos[first], ldd = gla_pad(dim);
    pdl_wait();
    float* const state = a.state + (size_t)seq * a.seq_stride + (size_t)head * vdim * ldd;
    const bool vec = (dim & 3) == 0;  // queries and keys in 16-byte pieces
    int turn = 0;
    auto sync = [&]() {
        if (CS > 1) cluster_sync_all();
        else __syncthreads();
    };
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
        sync();
        const bool pieces = a.xp && ((vdim | a.out_off | share) & 7) == 0;
        const int per = pieces ? c_n / 8 : c_n;
        for (int i = tid; i < rows * per; i += GLA_THREADS) {
            const int t = i / per, c = (i - t * per) * (pieces ? 8 : 1), m = first + r0 + t, k0 = a.out_off + head * vdim + c_lo + c;
            const float *g = a.raw + (size_t)m * a.ld + a.g_off + (size_t)head * vdim + c_lo + c, *o = os + t * share + c, *w = a.norm_w + c_lo + c;
            float s = 0.f;
            for (int r = 0; r < CS; ++r) s += sums[r * kept + t];
            const float f = 1.0f / sqrtf(s / (float)vdim + a.eps);
            if (pieces) {
                const float4 g0 = ld_cg_f32x4(g), g1 = ld_cg_f32x4(g + 4);
                const float gv[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
                float v[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = ((o[e] * f) * __ldg(w + e)) * gla_silu(gv[e]) * a.out_scale;
                tc_xpack_store8(a.xp, a.xp_mpad, m, k0, v);
            } else {
                const float v = ((o[0] * f) * __ldg(w)) * gla_silu(ld_cg_f32(g)) * a.out_scale;
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
        for (int t0 = 0; t0 < n; t0 += TR) {
            const int tr = min(TR, n - t0);
            sync();  // the cluster's CTAs have started, and are done with the tokens in front
            const float* raw = a.raw + (size_t)(first + t0) * a.ld;
            if (vec) {
#pragma unroll 4
                for (int i = tid; i < tr * D4; i += GLA_THREADS) {
                    const int t = i / D4, d = (i - t * D4) * 4;
                    const float* row = raw + (size_t)t * a.ld + (size_t)head * dim + d;
                    float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
                    if (d < dim) {
                        q = ld_cg_f32x4(row + a.q_off);
                        k = ld_cg_f32x4(row + a.k_off);
                    }
                    reinterpret_cast<float4*>(qs)[i] = make_float4(q.x * a.q_scale, q.y * a.q_scale, q.z * a.q_scale, q.w * a.q_scale);
                    reinterpret_cast<float4*>(ks)[i] = k;
                }
            } else {
                for (int i = tid; i < tr * DP; i += GLA_THREADS) {
                    const int t = i / DP, d = i - t * DP;
                    const float* row = raw + (size_t)t * a.ld + (size_t)head * dim + d;
                    qs[i] = d < dim ? ld_cg_f32(row + a.q_off) * a.q_scale : 0.f;
                    ks[i] = d < dim ? ld_cg_f32(row + a.k_off) : 0.f;
                }
            }
#pragma unroll 4
            for (int i = tid; i < tr * CP; i += GLA_THREADS) {
                const int t = i / CP, cc = sl * CP + i - t * CP;
                vs[i] = cc < c_n ? ld_cg_f32(raw + (size_t)t * a.ld + a.v_off + (size_t)head * vdim + c_lo + cc) : 0.f;
            }
#pragma unroll 4
            for (int i = tid; i < tr * rank; i += GLA_THREADS) {
                const int t = i / rank;
                lat[i] = ld_cg_f32(raw + (size_t)t * a.ld + a.a_off + (i - t * rank));
            }
            __syncthreads();
            // decays of the tokens cta, cta + CS, ..., for every CTA of the cluster
            for (int i = tid; i < (tr - cta + CS - 1) / CS * D4; i += GLA_THREADS) {
                const int tt = i / D4, d = (i - tt * D4) * 4, t = cta + tt * CS;
                const float* l = lat + t * rank;
                float z[4] = {0.f, 0.f, 0.f, 0.f}, v[4];
                if (vec) {
                    if (d < dim)
#pragma unroll 4
                        for (int r = 0; r < rank; ++r) {
                            const float4 w = *reinterpret_cast<const float4*>(up + r * dim + d);
                            z[0] = fmaf(w.x, l[r], z[0]); z[1] = fmaf(w.y, l[r], z[1]); z[2] = fmaf(w.z, l[r], z[2]); z[3] = fmaf(w.w, l[r], z[3]);
                        }
                } else {
                    for (int r = 0; r < rank; ++r)
#pragma unroll
                        for (int e = 0; e < 4; ++e)
                            if (d + e < dim) z[e] = fmaf(up[r * dim + d + e], l[r], z[e]);
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) v[e] = d + e < dim ? gla_decay(z[e] + __ldg(a.bias + (size_t)head * dim + d + e), a.inv_tau) : 0.f;
                const float4 v4 = make_float4(v[0], v[1], v[2], v[3]);
                if (CS == 1) reinterpret_cast<float4*>(as)[t * D4 + d / 4] = v4;
                else
                    for (int r = 0; r < CS; ++r) st_dsmem_f32x4(dsmem_addr(as + t * DP + d, (uint32_t)r), v4);
            }
            sync();
            auto step = [&](int t) -> float {  // this thread's share of o
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
                return o0 + o1;
            };
            float* const orow = os + (size_t)(slices > 1 ? t0 : 0) * share + c;
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
            if (slices == 1) finish(t0, tr);
        }
#pragma unroll
        for (int j = 0; j < RD / 4; ++j)
            if (on && (j * LP + part) * 4 < dim) __stcg(column + j * LP, S[j]);
    }
    if (slices > 1) finish(0, n);
}

// ---- single tokens ---------------------------------------------------------------------------------
// The state arrives in shared memory by one bulk copy, in the captured decode step ahead of the dependency wait, and goes back from
// registers column by column.
struct GlaTokenSmem {
    int state, up, alpha, lat, v, gate, o, total;
};
__host__ __device__ __forceinline__ GlaTokenSmem gla_token_smem(const GlaArgs& a) {
    GlaTokenSmem s;
    int at = 0;
    auto take = [&](int n) {
        const int first = at;
        at += (n + 3) & ~3;
        return first;
    };
    s.state = take((int)gla_state_floats(a.dim, a.vdim));
    s.up = take(a.rank * a.dim <= GLA_UP_SMEM ? a.rank * a.dim : 0);
    s.alpha = take(gla_pad(a.dim));
    s.lat = take(a.rank);
    s.v = take(a.vdim);
    s.gate = take(a.vdim);
    s.o = take(a.vdim);
    s.total = at;
    return s;
}

__device__ __forceinline__ void gla_token_block(const GlaArgs& a, int block, float* sm, float* part) {
    constexpr int NJ = GLA_TOKEN_DIM / 128;  // 16-byte pieces of a column per lane
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int head = block % a.heads, m = block / a.heads, dim = a.dim, vdim = a.vdim, rank = a.rank, ldd = gla_pad(dim), ld4 = ldd / 4;
    const GlaTokenSmem lay = gla_token_smem(a);
    constexpr uint32_t CHUNK = 16384;
    __shared__ uint64_t landed[(GLA_TOKEN_BYTES + CHUNK - 1) / CHUNK], up_landed;  // a barrier per piece of the copy
    __shared__ volatile int s_abort;
    const uint32_t bytes = (uint32_t)(vdim * ldd * 4);
    const float* up = a.up + (size_t)head * rank * dim;
    const bool up_staged = rank * dim <= GLA_UP_SMEM, up_bulk = up_staged && (rank * dim & 3) == 0;
    if (tid == 0) {
        for (uint32_t i = 0; i * CHUNK < bytes; ++i) mb_init(&landed[i], 1);
        mb_init(&up_landed, 1);
        s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        if (up_bulk) {
            mb_expect_tx(&up_landed, (uint32_t)(rank * dim * 4));
            bulk_copy(sm + lay.up, up, (uint32_t)(rank * dim * 4), &up_landed);
        }
    }
    const int seq = a.row_seq[m], pos = a.row_pos[m];
    float* const state = a.state + (size_t)seq * a.seq_stride + (size_t)head * vdim * ldd;
    auto fetch = [&]() {
        for (uint32_t i = 0, o = 0; o < bytes; ++i, o += CHUNK) {
            mb_expect_tx(&landed[i], min(CHUNK, bytes - o));
            bulk_copy(reinterpret_cast<char*>(sm + lay.state) + o, reinterpret_cast<const char*>(state) + o, min(CHUNK, bytes - o), &landed[i]);
        }
    };
    if (tid == 0 && a.early && pos > 0) fetch();
    // weights of this thread's first decay and result
    const float bias0 = tid < dim ? __ldg(a.bias + (size_t)head * dim + tid) : 0.f, norm0 = tid < vdim ? __ldg(a.norm_w + tid) : 0.f;
    if (up_staged && !up_bulk)
        for (int i = tid; i < rank * dim; i += GLA_THREADS) sm[lay.up + i] = __ldg(up + i);
    if (up_staged) up = sm + lay.up;
    pdl_wait();
    if (tid == 0 && !a.early && pos > 0) fetch();
    const float* raw = a.raw + (size_t)m * a.ld;
    // everything of the row is requested before the first use
    const float lat0 = tid < rank ? ld_cg_f32(raw + a.a_off + tid) : 0.f, v0 = tid < vdim ? ld_cg_f32(raw + a.v_off + (size_t)head * vdim + tid) : 0.f, g0 = tid < vdim ? ld_cg_f32(raw + a.g_off + (size_t)head * vdim + tid) : 0.f;
    // lanes of a column: a power of two, so that several short columns share a warp
    const int LC = ld4 >= 32 ? 32 : 1 << (32 - __clz(ld4 - 1)), sub = lane / LC, piece = lane - sub * LC, CW = 32 / LC;
    float4 q[NJ], k[NJ], al[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        q[j] = k[j] = al[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        const int d = (j * 32 + piece) * 4;
        if (d >= dim) continue;
        const float *qr = raw + a.q_off + (size_t)head * dim + d, *kr = raw + a.k_off + (size_t)head * dim + d;
        if ((dim & 3) == 0) {
            q[j] = ld_cg_f32x4(qr);
            k[j] = ld_cg_f32x4(kr);
        } else {
            q[j] = make_float4(ld_cg_f32(qr), d + 1 < dim ? ld_cg_f32(qr + 1) : 0.f, d + 2 < dim ? ld_cg_f32(qr + 2) : 0.f, d + 3 < dim ? ld_cg_f32(qr + 3) : 0.f);
            k[j] = make_float4(ld_cg_f32(kr), d + 1 < dim ? ld_cg_f32(kr + 1) : 0.f, d + 2 < dim ? ld_cg_f32(kr + 2) : 0.f, d + 3 < dim ? ld_cg_f32(kr + 3) : 0.f);
        }
    }
    if (tid < rank) sm[lay.lat + tid] = lat0;
    if (tid < vdim) {
        sm[lay.v + tid] = v0;
        sm[lay.gate + tid] = g0;
    }
    for (int i = GLA_THREADS + tid; i < rank; i += GLA_THREADS) sm[lay.lat + i] = ld_cg_f32(raw + a.a_off + i);
    for (int i = GLA_THREADS + tid; i < vdim; i += GLA_THREADS) {
        sm[lay.v + i] = ld_cg_f32(raw + a.v_off + (size_t)head * vdim + i);
        sm[lay.gate + i] = ld_cg_f32(raw + a.g_off + (size_t)head * vdim + i);
    }
    __syncthreads();
    const bool up_ok = !up_bulk || mb_wait(&up_landed, 0, a.err_flag, &s_abort);  // bounded, like the waits below
    for (int d = tid; d < ldd; d += GLA_THREADS) {
        float v = 0.f;
        if (d < dim && up_ok) {
            float z = 0.f;
#pragma unroll 8
            for (int r = 0; r < rank; ++r) z = fmaf(up[r * dim + d], sm[lay.lat + r], z);
            v = gla_decay(z + (d == tid ? bias0 : __ldg(a.bias + (size_t)head * dim + d)), a.inv_tau);
        }
        sm[lay.alpha + d] = v;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        if (j * 32 + piece < ld4) al[j] = reinterpret_cast<const float4*>(sm + lay.alpha)[j * 32 + piece];
        q[j] = make_float4(q[j].x * a.q_scale, q[j].y * a.q_scale, q[j].z * a.q_scale, q[j].w * a.q_scale);
    }
    bool ok = true;
    uint32_t seen = 0;  // pieces that have landed
    const float4* tile = reinterpret_cast<const float4*>(sm + lay.state);
    constexpr int U = 4;  // columns whose sums go side by side
    for (int g = warp * U; g * CW < vdim; g += GLA_THREADS / 32 * U) {
        if (pos > 0)  // every piece is waited for, so that none is on its way when the CTA ends; the waits are bounded
            for (const uint32_t last = min(bytes, (uint32_t)((g + U) * CW * ldd * 4)); seen * CHUNK < last; ++seen) ok = mb_wait(&landed[seen], 0, a.err_flag, &s_abort) && ok;
        float o[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = (g + u) * CW + sub;
            o[u] = 0.f;
            if (c >= vdim) continue;
            const float v = sm[lay.v + c];
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const int p = j * 32 + piece;
                if (p >= ld4) continue;
                float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
                if (pos > 0 && ok) S = tile[c * ld4 + p];
                S.x = fmaf(S.x, al[j].x, k[j].x * v);
                S.y = fmaf(S.y, al[j].y, k[j].y * v);
                S.z = fmaf(S.z, al[j].z, k[j].z * v);
                S.w = fmaf(S.w, al[j].w, k[j].w * v);
                __stcg(reinterpret_cast<float4*>(state) + (size_t)c * ld4 + p, S);
                o[u] += fmaf(S.x, q[j].x, S.y * q[j].y) + fmaf(S.z, q[j].z, S.w * q[j].w);
            }
        }
        for (int s = 1; s < LC; s <<= 1)
#pragma unroll
            for (int u = 0; u < U; ++u) o[u] += __shfl_xor_sync(0xffffffffu, o[u], s);
        if (piece == 0)
#pragma unroll
            for (int u = 0; u < U; ++u)
                if ((g + u) * CW + sub < vdim) sm[lay.o + (g + u) * CW + sub] = o[u];
    }
    __syncthreads();
    float s = 0.f;
    for (int c = tid; c < vdim; c += GLA_THREADS) s = fmaf(sm[lay.o + c], sm[lay.o + c], s);
    s = warp_sum(s);
    if (lane == 0) part[warp] = s;
    for (int c = tid; c < vdim; c += GLA_THREADS) sm[lay.v + c] = c == tid ? norm0 : __ldg(a.norm_w + c);  // the values have been used
    __syncthreads();
    s = 0.f;
#pragma unroll
    for (int w = 0; w < GLA_THREADS / 32; ++w) s += part[w];
    const float f = 1.0f / sqrtf(s / (float)vdim + a.eps);
    const int k0 = a.out_off + head * vdim;
    auto value = [&](int c, float w) { return ((sm[lay.o + c] * f) * w) * gla_silu(sm[lay.gate + c]) * a.out_scale; };
    if (a.xp && ((vdim | a.out_off) & 7) == 0) {
        for (int c = tid * 8; c < vdim; c += GLA_THREADS * 8) {
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = value(c + e, sm[lay.v + c + e]);
            tc_xpack_store8(a.xp, a.xp_mpad, m, k0 + c, v);
        }
    } else {
        for (int c = tid; c < vdim; c += GLA_THREADS) {
            const float v = value(c, sm[lay.v + c]);
            if (a.xp) tc_xpack_store(a.xp, a.xp_mpad, m, k0 + c, v);
            else a.out[(size_t)m * a.ld_out + k0 + c] = v;
        }
    }
}

}  // namespace hm
