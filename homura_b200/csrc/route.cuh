// The choice of a router (one warp per row).
#pragma once
#include "common.cuh"
#include "moe.h"

namespace hm {

// Softmax over a row's n_out logits z (shared memory, replaced by the scores), choice by score + correction (ties to the lower index),
// weights without the correction, times `scale`.  choice: n_out words of scratch.
__device__ __forceinline__ void choose_experts(const RouteSpec& a, int m, float* z, float* choice) {
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
    uint32_t* key = reinterpret_cast<uint32_t*>(choice);  // unsigned integers in the order of the floats; 0: chosen already
    for (int r = lane; r < a.n_out; r += 32) {
        const float s = z[r] / l;
        z[r] = s * a.scale;
        const uint32_t u = __float_as_uint(a.correction ? s + __ldg(a.correction + r) : s);
        key[r] = u >> 31 ? ~u : u | 0x80000000u;
    }
    __syncwarp();
    float ident = 0.f;
    for (int k = 0; k < a.top; ++k) {
        uint32_t best = 0u, at = lane < a.n_out ? lane : 0xffffffffu;
        for (int r = lane; r < a.n_out; r += 32)
            if (key[r] > best) {
                best = key[r];
                at = r;
            }
        const uint32_t most = __reduce_max_sync(0xffffffffu, best);
        const int bi = (int)__reduce_min_sync(0xffffffffu, best == most ? at : 0xffffffffu);
        const float s = z[bi];
        __syncwarp();
        if (lane == 0) {
            key[bi] = 0u;
            const bool id = bi >= a.experts;
            a.out.ids[(size_t)m * a.top + k] = id ? -1 : bi;
            a.out.weights[(size_t)m * a.top + k] = s;
            if (id) ident += s;
            else if (a.out.dense) a.out.dense[(size_t)m * a.experts + bi] = s;
        }
        __syncwarp();
    }
    if (a.out.dense) {  // the chosen ones are those whose key is gone
        const int words = (a.experts + 31) / 32;
        for (int w = 0; w < words; ++w) {
            const int r = w * 32 + lane;
            const uint32_t bits = __ballot_sync(0xffffffffu, r < a.experts && key[r] == 0u);
            if (lane == 0) a.out.mask[(size_t)m * words + w] = bits;
        }
    }
    if (lane == 0 && a.out.identity) a.out.identity[m] = ident;
}

}  // namespace hm
