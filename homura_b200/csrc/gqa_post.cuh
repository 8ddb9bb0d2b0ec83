// What happens to the rows of a fused query / key / value projection before the attention (GqaPostArgs): one warp per row and head.
#pragma once
#include "gqa_attn.h"
#include "model_spec.h"

namespace hm {

constexpr int POST_WARPS = 8;

__host__ __device__ __forceinline__ int gqa_post_v_heads(const GqaPostArgs& a) { return a.tied_values ? 0 : a.k_out ? a.v_heads : a.pool.kv_heads; }
__host__ __device__ __forceinline__ int gqa_post_slots(const GqaPostArgs& a) { return a.heads + a.pool.kv_heads + gqa_post_v_heads(a); }
__host__ __device__ __forceinline__ int gqa_post_blocks(const GqaPostArgs& a) { return (gqa_post_slots(a) + POST_WARPS - 1) / POST_WARPS; }  // per row
// a head's elements per warp, kept only where they are needed twice
__host__ __device__ __forceinline__ int gqa_post_buf(const GqaPostArgs& a) { return a.taps > 0 || a.rot_dims > 0 || a.qk_norm >= QKN_UNIT || a.conv_silu || a.tied_values ? (a.pool.dim > a.pool.vdim ? a.pool.dim : a.pool.vdim) : 0; }
__host__ __device__ __forceinline__ size_t gqa_post_smem(const GqaPostArgs& a) { return sizeof(float) * POST_WARPS * (size_t)gqa_post_buf(a); }

// Rotates `half` pairs (buf[i], buf[i + half]), or neighbours, with the lanes of a warp.
__device__ __forceinline__ void rotate_pairs(float* buf, int half, const double* turns, int pos, int lane, bool neighbours = false) {
    for (int i = lane; i < half; i += 32) {
        float c, s;
        rotation_at(__ldg(turns + i), pos, c, s);
        const int a = neighbours ? 2 * i : i, b = neighbours ? 2 * i + 1 : i + half;
        const float u = buf[a], v = buf[b];
        buf[a] = fmaf(u, c, -v * s);
        buf[b] = fmaf(v, c, u * s);
    }
}

// X: 1 with convolution, rotation or norms behind it (the plain variant keeps no head in shared memory), 2 with everything that
// GqaPostArgs::varied() names as well.  Row m of one head slot ([heads] queries, [kv_heads] keys, [kv_heads] values).  part_q / part_k: sums of squares of the whole
// projections (QKN_ALL); first: the first row of m's run.
template <int X>
__device__ __forceinline__ void gqa_post_row(const GqaPostArgs& a, int m, int slot, int first, int pos, int seq, size_t page, float part_q, float part_k, float* buf) {
    const int lane = threadIdx.x & 31;
    const int G = a.pool.kv_heads, dim = a.pool.dim, vdim = a.pool.vdim, nq = a.heads * dim, nk = G * dim;
    const int t = pos % GQA_PAGE;
    const bool is_v = slot >= a.heads + G, is_q = slot < a.heads;
    const int h = is_v ? slot - a.heads - G : is_q ? slot : slot - a.heads, n = is_v ? vdim : dim;
    const int ch0 = (is_v ? nq + nk : is_q ? 0 : nq) + h * n;  // first channel
    const float* x = a.raw + (size_t)m * a.ld + ch0;
    const bool buffered = X && gqa_post_buf(a) > 0;
    const int VH = X == 2 ? gqa_post_v_heads(a) : G;
    auto put_page = [&](void* pool, size_t off, float v) {
        if (a.pool.bf16) reinterpret_cast<uint16_t*>(pool)[off] = f32_to_bf16_rne(v);
        else reinterpret_cast<float*>(pool)[off] = v;
    };
    if (buffered) {
        const float* state = a.taps > 1 ? a.conv_state + (size_t)seq * a.conv_stride + ch0 : nullptr;
        const int channels = nq + nk + VH * vdim, slots = conv_slots(a.taps);
        for (int d = lane; d < n; d += 32) {
            float v = ld_cg_f32(x + d);
            if (a.taps > 0) {
                const float* w = a.conv_w + (size_t)(ch0 + d) * a.taps;
                auto input = [&](int j) { return m - j >= first ? ld_cg_f32(x + d - (ptrdiff_t)j * a.ld) : ld_cg_f32(state + (size_t)((pos - j) % slots) * channels + d); };
                const int back = min(a.taps - 1, pos);
                float u[3] = {0.f, 0.f, 0.f};  // requested together
#pragma unroll
                for (int j = 1; j <= 3; ++j)
                    if (j <= back) u[j - 1] = input(j);
                v *= __ldg(w + a.taps - 1);
#pragma unroll
                for (int j = 1; j <= 3; ++j)
                    if (j <= back) v = fmaf(u[j - 1], __ldg(w + a.taps - 1 - j), v);
                for (int j = 4; j <= back; ++j) v = fmaf(input(j), __ldg(w + a.taps - 1 - j), v);
            }
            if (X == 2 && a.conv_silu) v = v / (1.0f + expf(-v));
            buf[d] = v;
            if (X == 2 && a.tied_values && !is_q) put_page(a.pool.v, page * gqa_page_elems(G, dim) + (size_t)h * GQA_PAGE * gqa_pad(dim) + gqa_tile_off(t, d), v);
        }
        __syncwarp();
    }
    auto at = [&](int d) { return buffered ? buf[d] : ld_cg_f32(x + d); };
    if (!is_v) {
        float inv = 1.f;
        if (a.qk_norm == QKN_ALL) {
            inv = 1.0f / sqrtf((is_q ? part_q : part_k) / (float)(is_q ? nq : nk) + a.eps);
        } else if (a.qk_norm == QKN_HEAD) {
            float s = 0.f;
#pragma unroll 4
            for (int d = lane; d < dim; d += 32) {
                const float v = at(d);
                s = fmaf(v, v, s);
            }
            inv = 1.0f / sqrtf(warp_sum(s) / (float)dim + a.eps);
        }
        const float* w = a.qk_norm == QKN_HEAD || a.qk_norm == QKN_ALL ? (is_q ? a.q_norm : a.k_norm) + (a.qk_norm == QKN_ALL ? (size_t)h * dim : 0) : nullptr;
        auto normed = [&](int d) { return w ? (at(d) * inv) * __ldg(w + d) : at(d); };
        float unit = 1.f;
        const bool turned = X && a.rot_dims > 0, after = X && (turned || a.qk_norm >= QKN_UNIT);
        if (after) {
            if (w)
                for (int d = lane; d < dim; d += 32) buf[d] = normed(d);
            __syncwarp();
            if (turned) rotate_pairs(buf, a.rot_dims / 2, a.turns, pos, lane, X == 2 && a.rot_neighbours);
            __syncwarp();
            if (a.qk_norm >= QKN_UNIT) {
                float s = 0.f;
                for (int d = lane; d < dim; d += 32) s = fmaf(buf[d], buf[d], s);
                s = warp_sum(s);
                unit = 1.0f / sqrtf((X == 2 && a.qk_norm == QKN_SUM ? s : s / (float)dim) + a.eps);
            }
        }
        auto value = [&](int d) { return after ? buf[d] * unit : normed(d); };
        if (is_q) {
            float f = 1.f;
            if (a.temp_every > 0) f = 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every) + 1.0f);
            if (X == 2 && a.head_scale) f = __ldg(a.head_scale + h);
            float* o = a.q_out + (size_t)m * nq + (size_t)h * dim;
            for (int d = lane; d < dim; d += 32) o[d] = (value(d) * f) * a.q_scale;
        } else if (X == 2 && a.k_out) {
            for (int d = lane; d < dim; d += 32) a.k_out[(size_t)m * nk + (size_t)h * dim + d] = value(d);
        } else {
            const size_t base = page * gqa_page_elems(G, dim) + (size_t)h * GQA_PAGE * gqa_pad(dim);
            for (int d = lane; d < dim; d += 32) put_page(a.pool.k, base + gqa_tile_off(t, d), value(d));
        }
    } else if (X == 2 && a.k_out) {
        for (int d = lane; d < vdim; d += 32) a.v_out[(size_t)m * VH * vdim + (size_t)h * vdim + d] = at(d);
    } else {
        float* kept = a.v_first ? a.v_first + (size_t)m * G * vdim + (size_t)h * vdim : nullptr;
        const float lam = kept && a.v_lambda ? __ldg(a.v_lambda) : 0.f;
        const size_t base = page * gqa_page_elems(G, vdim) + (size_t)h * GQA_PAGE * gqa_pad(vdim);
        for (int d = lane; d < vdim; d += 32) {
            float v = at(d);
            if (kept) {
                if (a.v_lambda) v = (1.0f - lam) * v + lam * ld_cg_f32(kept + d);
                else kept[d] = v;
            }
            put_page(a.pool.v, base + gqa_tile_off(t, d), v);
        }
    }
    __syncwarp();
}

// Row m and POST_WARPS head slots from blk * POST_WARPS on.
template <int X>
__device__ __forceinline__ void gqa_post_block(const GqaPostArgs& a, int m, int blk, float* smem) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int G = a.pool.kv_heads, dim = a.pool.dim, vdim = a.pool.vdim, nq = a.heads * dim, nk = G * dim;
    const int slot0 = blk * POST_WARPS, slot = slot0 + warp;
    __shared__ float s_part[2][POST_WARPS];
    // positions and pages do not depend on the launch in front
    auto page_of = [&](int seq, int pos) { return X == 2 && a.k_out ? (size_t)0 : (size_t)a.pool.page_table[(size_t)seq * a.pool.max_pages + pos / GQA_PAGE]; };
    const int pos = a.row_pos[m], seq = a.row_seq[m];
    const size_t page = page_of(seq, pos);
    pdl_wait();
    float sq = 0.f, sk = 0.f;
    if (a.qk_norm == QKN_ALL) {  // every CTA sums the squares of the part it needs
        const float* raw = a.raw + (size_t)m * a.ld;
        if (slot0 < a.heads)
#pragma unroll 4
            for (int i = tid; i < nq; i += POST_WARPS * 32) {
                const float v = ld_cg_f32(raw + i);
                sq = fmaf(v, v, sq);
            }
        if (slot0 < a.heads + G && slot0 + POST_WARPS > a.heads)
#pragma unroll 4
            for (int i = tid; i < nk; i += POST_WARPS * 32) {
                const float v = ld_cg_f32(raw + nq + i);
                sk = fmaf(v, v, sk);
            }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) {
            s_part[0][warp] = sq;
            s_part[1][warp] = sk;
        }
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int w = 0; w < POST_WARPS; ++w) {
            sq += s_part[0][w];
            sk += s_part[1][w];
        }
    }
    if (slot >= gqa_post_slots(a)) return;
    float* buf = X ? smem + warp * gqa_post_buf(a) : nullptr;
    if (!X || a.taps <= 1) {
        gqa_post_row<X>(a, m, slot, m, pos, seq, page, sq, sk, buf);
        return;
    }
    int first, end;
    a.runs.find(m, first, end);
    gqa_post_row<X>(a, m, slot, first, pos, seq, page, sq, sk, buf);
    if (m < end - (a.taps - 1)) return;
    // the inputs of a run's last rows are kept
    const bool is_v = slot >= a.heads + G, is_q = slot < a.heads;
    const int h = is_v ? slot - a.heads - G : is_q ? slot : slot - a.heads, n = is_v ? vdim : dim, ch0 = (is_v ? nq + nk : is_q ? 0 : nq) + h * n, channels = nq + nk + (X == 2 ? gqa_post_v_heads(a) : G) * vdim;
    float* kept = a.conv_state + (size_t)seq * a.conv_stride + (size_t)(pos % conv_slots(a.taps)) * channels + ch0;
#pragma unroll 4
    for (int d = lane; d < n; d += 32) kept[d] = ld_cg_f32(a.raw + (size_t)m * a.ld + ch0 + d);
}

}  // namespace hm
