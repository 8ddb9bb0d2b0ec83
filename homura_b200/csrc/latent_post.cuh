// What a token leaves in a cache of latents: the normalised latent and, optionally, a rotated key part behind it.
#pragma once
#include "gqa_post.cuh"
#include "latent_attn.h"

namespace hm {

// Row m of c [M][ldc]: rank - 2 * rot_pairs elements RMS-normed with weight w, then rot_pairs pairs (i, i + rot_pairs), or neighbours, rotated and
// cached side by side.  All NT threads of the block; part: a float per warp.
template <int NT, bool ROT>
__device__ __forceinline__ void latent_write_row(const LatentPool& pool, const float* __restrict__ c, int ldc, int m, const float* __restrict__ w, float eps, const int32_t* __restrict__ row_pos, const int32_t* __restrict__ row_seq, int rot_pairs,
                                                 const double* turns, float* part, bool neighbours = false) {
    const int tid = threadIdx.x, lane = tid & 31, R = pool.rank, N = ROT ? R - 2 * rot_pairs : R;
    const float* x = c + (size_t)m * ldc;
    float s = 0.f;
    for (int i = tid; i < N; i += NT) {
        const float v = ld_cg_f32(x + i);
        s = fmaf(v, v, s);
    }
    s = warp_sum(s);
    if (lane == 0) part[tid >> 5] = s;
    __syncthreads();
    s = 0.f;
#pragma unroll
    for (int i = 0; i < NT / 32; ++i) s += part[i];
    const float inv = 1.0f / sqrtf(s / (float)N + eps);
    const int pos = row_pos[m];
    const size_t page = (size_t)pool.page_table[(size_t)row_seq[m] * pool.max_pages + pos / LATENT_PAGE] * latent_page_elems(R, pool.bf16);
    auto put = [&](int i, float v) {
        const size_t off = page + latent_page_off(pos % LATENT_PAGE, i, R, pool.bf16);
        if (pool.bf16) reinterpret_cast<uint16_t*>(pool.pages)[off] = f32_to_bf16_rne(v);
        else reinterpret_cast<float*>(pool.pages)[off] = v;
    };
    for (int i = tid; i < N; i += NT) put(i, (ld_cg_f32(x + i) * inv) * __ldg(w + i));
    if constexpr (ROT) {
        for (int i = NT - 1 - tid; i < rot_pairs; i += NT) {
            float cs, sn;
            rotation_at(__ldg(turns + i), pos, cs, sn);
            const float u = ld_cg_f32(x + N + (neighbours ? 2 * i : i)), v = ld_cg_f32(x + N + (neighbours ? 2 * i + 1 : rot_pairs + i));
            put(N + 2 * i, fmaf(u, cs, -v * sn));
            put(N + 2 * i + 1, fmaf(v, cs, u * sn));
        }
    }
}

}  // namespace hm
