// See recur.h.
#include "recur.h"

#include "launch_attrs.h"
#include "mbarrier.cuh"

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
#pragma unroll 4
                for (int t = warp; t < tr; t += GLA_THREADS / 32) {
                    float s = 0.f;
                    for (int d = lane * 4; d < DP; d += 128) {
                        const float4 x = *reinterpret_cast<const float4*>(ks + t * DP + d), y = *reinterpret_cast<const float4*>(qs + t * DP + d);
                        s = fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, s))));
                    }
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
                // with few rows a thread requests the next token's before this one's sums go through the lanes
                constexpr bool AHEAD = RD <= 8;
                float4 nq[AHEAD ? RD / 4 : 1], nk[AHEAD ? RD / 4 : 1], na[AHEAD ? RD / 4 : 1];
                auto request = [&](int t) {
                    if constexpr (AHEAD) {
#pragma unroll
                        for (int j = 0; j < RD / 4; ++j) {
                            na[j] = (reinterpret_cast<const float4*>(as + t * DP) + part)[j * LP];
                            nk[j] = (reinterpret_cast<const float4*>(ks + t * DP) + part)[j * LP];
                            nq[j] = (reinterpret_cast<const float4*>(qs + t * DP) + part)[j * LP];
                        }
                    }
                };
                request(0);
                for (int t = 0; t < tr; ++t) {
                    const float4 *q4 = reinterpret_cast<const float4*>(qs + t * DP) + part, *k4 = reinterpret_cast<const float4*>(ks + t * DP) + part, *a4 = reinterpret_cast<const float4*>(as + t * DP) + part;
                    const float v = vs[t * CP + col], beta = bs[t], own = kq[t];
                    float4 kt[AHEAD ? RD / 4 : 1];
                    // both sums over the shrunk state go through the lanes side by side: what it gives back for k, and for q
                    float sk0 = 0.f, sk1 = 0.f, sq0 = 0.f, sq1 = 0.f;
#pragma unroll
                    for (int j = 0; j < RD / 4; ++j) {
                        const float4 al = AHEAD ? na[AHEAD ? j : 0] : a4[j * LP], k = AHEAD ? nk[AHEAD ? j : 0] : k4[j * LP], q = AHEAD ? nq[AHEAD ? j : 0] : q4[j * LP];
                        if (AHEAD) kt[AHEAD ? j : 0] = k;
                        S[j].x *= al.x; S[j].y *= al.y; S[j].z *= al.z; S[j].w *= al.w;
                        sk0 = fmaf(S[j].x, k.x, fmaf(S[j].y, k.y, sk0));
                        sk1 = fmaf(S[j].z, k.z, fmaf(S[j].w, k.w, sk1));
                        sq0 = fmaf(S[j].x, q.x, fmaf(S[j].y, q.y, sq0));
                        sq1 = fmaf(S[j].z, q.z, fmaf(S[j].w, q.w, sq1));
                    }
                    request(min(t + 1, tr - 1));
                    float sk = sk0 + sk1, so = sq0 + sq1;
#pragma unroll
                    for (int s = 1; s < 32; s <<= 1)
                        if (s < LP) {
                            sk += __shfl_xor_sync(0xffffffffu, sk, s);
                            so += __shfl_xor_sync(0xffffffffu, so, s);
                        }
                    const float u = beta * (v - sk);
#pragma unroll
                    for (int j = 0; j < RD / 4; ++j) {
                        const float4 k = AHEAD ? kt[AHEAD ? j : 0] : k4[j * LP];
                        S[j].x = fmaf(k.x, u, S[j].x); S[j].y = fmaf(k.y, u, S[j].y); S[j].z = fmaf(k.z, u, S[j].z); S[j].w = fmaf(k.w, u, S[j].w);
                    }
                    if (part == 0 && on) orow[t * share] = fmaf(own, u, so);
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

// ---- single tokens ---------------------------------------------------------------------------------
// A CTA per (sequence, head).  The state arrives in shared memory by bulk copies, in the captured decode step ahead of the dependency
// wait; a warp takes whole columns, lanes along the key dimension, and stores them from registers as their piece has landed.
struct RecurTokenSmem {
    int state, v, gate, o, total;
};
__host__ __device__ __forceinline__ RecurTokenSmem recur_token_smem(const RecurArgs& a) {
    const int vp = (a.vdim + 3) & ~3, st = (int)gla_state_floats(a.dim, a.vdim);
    return RecurTokenSmem{0, st, st + vp, st + 2 * vp, st + 3 * vp};
}

template <int KIND>
__global__ void __launch_bounds__(GLA_THREADS, 3) recur_token_kernel(const __grid_constant__ RecurArgs a) {
    constexpr int NJ = GLA_TOKEN_DIM / 128, W = GLA_THREADS / 32;  // 16-byte pieces of a column per lane; warps
    constexpr uint32_t CHUNK = 16384;
    extern __shared__ __align__(16) float sm[];
    __shared__ uint64_t landed[(GLA_TOKEN_BYTES + CHUNK - 1) / CHUNK];  // a barrier per piece of the copy
    __shared__ volatile int s_abort;
    __shared__ float part[W];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int head = blockIdx.x % a.heads, m = blockIdx.x / a.heads, kvh = head / (a.heads / a.kv_heads), dim = a.dim, vdim = a.vdim, ldd = gla_pad(dim), ld4 = ldd / 4;
    const RecurTokenSmem lay = recur_token_smem(a);
    float *vs = sm + lay.v, *gs = sm + lay.gate, *os = sm + lay.o;
    const uint32_t bytes = (uint32_t)(vdim * ldd * 4);
    if (tid == 0) {
        for (uint32_t i = 0; i * CHUNK < bytes; ++i) mb_init(&landed[i], 1);
        s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    pdl_launch_dependents();
    const int seq = a.row_seq[m], pos = a.row_pos[m];
    float* const state = a.state + (size_t)seq * a.seq_stride + (size_t)head * vdim * ldd;
    auto fetch = [&]() {
        for (uint32_t i = 0, o = 0; o < bytes; ++i, o += CHUNK) {
            mb_expect_tx(&landed[i], min(CHUNK, bytes - o));
            bulk_copy(reinterpret_cast<char*>(sm + lay.state) + o, reinterpret_cast<const char*>(state) + o, min(CHUNK, bytes - o), &landed[i]);
        }
    };
    if (tid == 0 && a.early && pos > 0) fetch();
    const float decay = KIND == LIN_RETENTION ? __ldg(a.decay + head) : 0.f, norm0 = a.norm_w && tid < vdim ? __ldg(a.norm_w + tid) : 1.f;
    // lanes of a column: a power of two, so that several short columns share a warp
    const int LC = ld4 >= 32 ? 32 : 1 << (32 - __clz(ld4 - 1)), sub = lane / LC, piece = lane - sub * LC, CW = 32 / LC;
    pdl_wait();
    if (tid == 0 && !a.early && pos > 0) fetch();
    // everything of the row is requested before the first use
    const float v0 = tid < vdim ? ld_cg_f32(a.v + (size_t)m * a.ldv + (size_t)head * vdim + tid) : 0.f, g0 = tid < vdim ? ld_cg_f32(a.gate + (size_t)m * a.ld_gate + (size_t)head * vdim + tid) : 0.f;
    const float b0 = KIND == LIN_DELTA ? ld_cg_f32(a.beta + (size_t)m * a.ld_beta + head) : 0.f;
    const float *qr = a.q + (size_t)m * a.ldq + (size_t)kvh * a.head_ld, *kr = a.k + (size_t)m * a.ldk + (size_t)kvh * a.head_ld, *ar = KIND == LIN_DELTA ? a.alpha + ((size_t)m * a.heads + head) * dim : nullptr;
    auto load4 = [&](const float* row, int d) {
        if ((reinterpret_cast<uintptr_t>(row) & 15) == 0 && d + 4 <= dim) return ld_cg_f32x4(row + d);
        return make_float4(ld_cg_f32(row + d), d + 1 < dim ? ld_cg_f32(row + d + 1) : 0.f, d + 2 < dim ? ld_cg_f32(row + d + 2) : 0.f, d + 3 < dim ? ld_cg_f32(row + d + 3) : 0.f);
    };
    float4 q[NJ], k[NJ], al[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        q[j] = k[j] = al[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        const int d = (j * 32 + piece) * 4;
        if (d >= dim) continue;
        q[j] = load4(qr, d);
        k[j] = load4(kr, d);
        if (KIND == LIN_DELTA) al[j] = load4(ar, d);
    }
    if (tid < vdim) {
        vs[tid] = v0;
        gs[tid] = g0;
    }
    for (int i = GLA_THREADS + tid; i < vdim; i += GLA_THREADS) {
        vs[i] = ld_cg_f32(a.v + (size_t)m * a.ldv + (size_t)head * vdim + i);
        gs[i] = ld_cg_f32(a.gate + (size_t)m * a.ld_gate + (size_t)head * vdim + i);
    }
    float kq = 0.f;  // what the token's own write adds to its result
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        q[j] = make_float4(q[j].x * a.q_scale, q[j].y * a.q_scale, q[j].z * a.q_scale, q[j].w * a.q_scale);
        if (KIND == LIN_DELTA) kq += fmaf(q[j].x, k[j].x, q[j].y * k[j].y) + fmaf(q[j].z, k[j].z, q[j].w * k[j].w);
    }
    if (KIND == LIN_DELTA)
        for (int s = 1; s < LC; s <<= 1) kq += __shfl_xor_sync(0xffffffffu, kq, s);
    const float beta = KIND == LIN_DELTA ? sigmoid(b0) : 0.f;
    __syncthreads();
    bool ok = true;
    uint32_t seen = 0;  // pieces that have landed
    const float4* tile = reinterpret_cast<const float4*>(sm + lay.state);
    constexpr int U = KIND == LIN_DELTA ? 2 : 4;  // columns whose sums go side by side
    for (int g = warp * U; g * CW < vdim; g += W * U) {
        if (pos > 0)  // every piece is waited for, so that none is on its way when the CTA ends; the waits are bounded
            for (const uint32_t last = min(bytes, (uint32_t)((g + U) * CW * ldd * 4)); seen * CHUNK < last; ++seen) ok = mb_wait(&landed[seen], 0, a.err_flag, &s_abort) && ok;
        float4 S[U][NJ];
        float o[U], sk[U], v[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = (g + u) * CW + sub;
            o[u] = sk[u] = 0.f;
            v[u] = c < vdim ? vs[c] : 0.f;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const int p = j * 32 + piece;
                S[u][j] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c >= vdim || p >= ld4) continue;
                if (pos > 0 && ok) S[u][j] = tile[c * ld4 + p];
                float4& t = S[u][j];
                if (KIND == LIN_DELTA) {
                    t = make_float4(t.x * al[j].x, t.y * al[j].y, t.z * al[j].z, t.w * al[j].w);
                    sk[u] += fmaf(t.x, k[j].x, t.y * k[j].y) + fmaf(t.z, k[j].z, t.w * k[j].w);
                } else {
                    t = make_float4(fmaf(t.x, decay, k[j].x * v[u]), fmaf(t.y, decay, k[j].y * v[u]), fmaf(t.z, decay, k[j].z * v[u]), fmaf(t.w, decay, k[j].w * v[u]));
                    __stcg(reinterpret_cast<float4*>(state) + (size_t)c * ld4 + p, t);
                }
                o[u] += fmaf(t.x, q[j].x, t.y * q[j].y) + fmaf(t.z, q[j].z, t.w * q[j].w);
            }
        }
        for (int s = 1; s < LC; s <<= 1)
#pragma unroll
            for (int u = 0; u < U; ++u) {
                o[u] += __shfl_xor_sync(0xffffffffu, o[u], s);
                if (KIND == LIN_DELTA) sk[u] += __shfl_xor_sync(0xffffffffu, sk[u], s);
            }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = (g + u) * CW + sub;
            if (c >= vdim) continue;
            if (KIND == LIN_DELTA) {
                const float w = beta * (v[u] - sk[u]);
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const int p = j * 32 + piece;
                    if (p >= ld4) continue;
                    const float4 t = S[u][j];
                    __stcg(reinterpret_cast<float4*>(state) + (size_t)c * ld4 + p, make_float4(fmaf(k[j].x, w, t.x), fmaf(k[j].y, w, t.y), fmaf(k[j].z, w, t.z), fmaf(k[j].w, w, t.w)));
                }
                o[u] = fmaf(kq, w, o[u]);
            }
            if (piece == 0) os[c] = o[u];
        }
    }
    if (pos > 0)  // (a warp whose columns end before the last piece)
        for (; seen * CHUNK < bytes; ++seen) mb_wait(&landed[seen], 0, a.err_flag, &s_abort);
    __syncthreads();
    float s = 0.f;
    for (int c = tid; c < vdim; c += GLA_THREADS) s = fmaf(os[c], os[c], s);
    s = warp_sum(s);
    if (lane == 0) part[warp] = s;
    for (int c = tid; c < vdim; c += GLA_THREADS) vs[c] = c == tid ? norm0 : a.norm_w ? __ldg(a.norm_w + c) : 1.f;  // the values have been used
    __syncthreads();
    s = 0.f;
#pragma unroll
    for (int w = 0; w < W; ++w) s += part[w];
    const float f = 1.0f / sqrtf(s / (float)vdim + a.eps);
    const int k0 = a.out_off + head * vdim;
    auto value = [&](int c) {
        const float y = (os[c] * f) * vs[c], z = gs[c];
        return KIND == LIN_RETENTION ? y * (z * sigmoid(z)) : y * sigmoid(z);
    };
    if (a.xp && ((vdim | a.out_off) & 7) == 0) {
        for (int c = tid * 8; c < vdim; c += GLA_THREADS * 8) {
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = value(c + e);
            tc_xpack_store8(a.xp, a.xp_mpad, m, k0 + c, v);
        }
    } else {
        for (int c = tid; c < vdim; c += GLA_THREADS) {
            if (a.xp) tc_xpack_store(a.xp, a.xp_mpad, m, k0 + c, value(c));
            else a.out[(size_t)m * a.ld_out + k0 + c] = value(c);
        }
    }
}

template <typename K>
cudaError_t launch(K kern, const RecurArgs& a, unsigned blocks, size_t smem, int cluster, cudaStream_t st, bool pdl) {
    const cudaError_t e = ensure_dyn_smem(kern, smem);
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
    if (cluster > 1) {
        at[n].id = cudaLaunchAttributeClusterDimension;
        at[n].val.clusterDim.x = (unsigned)cluster;
        at[n].val.clusterDim.y = at[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = at;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, kern, a);
}

template <int KIND>
cudaError_t launch_kind(const RecurArgs& a, unsigned blocks, size_t smem, cudaStream_t st, bool pdl) {
    switch (a.shape.rows) {
        case 4: return launch(recur_kernel<4, KIND>, a, blocks, smem, a.shape.cluster, st, pdl);
        case 8: return launch(recur_kernel<8, KIND>, a, blocks, smem, a.shape.cluster, st, pdl);
        case 16: return launch(recur_kernel<16, KIND>, a, blocks, smem, a.shape.cluster, st, pdl);
        case 32: return launch(recur_kernel<32, KIND>, a, blocks, smem, a.shape.cluster, st, pdl);
        case 64: return launch(recur_kernel<64, KIND>, a, blocks, smem, a.shape.cluster, st, pdl);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

cudaError_t launch_recur(const RecurArgs& a_in, int sm_count, cudaStream_t st, bool pdl) {
    RecurArgs a = a_in;
    if (a.M < 1 || a.M > GQA_MAX_ROWS || a.dim > GLA_MAX_DIM || a.vdim > GLA_MAX_VDIM || a.heads % a.kv_heads != 0 || (a.kind != LIN_RETENTION && a.kind != LIN_DELTA)) return cudaErrorInvalidValue;
    const int runs = a.runs.n ? a.runs.n : a.M, rows = a.runs.n ? a.longest_run : 1;
    // (a few tokens: more CTAs per head are worth more than the earlier loads)
    if (rows == 1 && a.M * a.heads > sm_count && a.dim <= GLA_TOKEN_DIM && gla_state_floats(a.dim, a.vdim) * 4 <= GLA_TOKEN_BYTES) {
        const size_t smem = (size_t)recur_token_smem(a).total * 4;
        const unsigned blocks = (unsigned)(a.M * a.heads);
        return a.kind == LIN_DELTA ? launch(recur_token_kernel<LIN_DELTA>, a, blocks, smem, 1, st, pdl) : launch(recur_token_kernel<LIN_RETENTION>, a, blocks, smem, 1, st, pdl);
    }
    a.shape = gla_shape(a.dim, a.vdim, runs * a.heads, sm_count);
    for (a.step = rows; a.step > 1 && (size_t)recur_smem(a, rows).total * 4 > 110 * 1024; a.step = (a.step + 1) / 2) {
    }
    const size_t smem = (size_t)recur_smem(a, rows).total * 4;
    const unsigned blocks = (unsigned)(runs * a.heads * a.shape.cluster);
    return a.kind == LIN_DELTA ? launch_kind<LIN_DELTA>(a, blocks, smem, st, pdl) : launch_kind<LIN_RETENTION>(a, blocks, smem, st, pdl);
}

}  // namespace hm
