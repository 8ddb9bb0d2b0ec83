// See sandwich.h.  One CTA per row, the row in registers; means first, then the squared deviations from them.
#include "sandwich.h"

#include "gemm_tc.h"
#include "launch_attrs.h"

namespace hm {
namespace {

template <int T, int NV>
__global__ void __launch_bounds__(T) sandwich_kernel(const SandwichArgs a) {
    extern __shared__ __align__(16) float row[];
    __shared__ float part[6][T / 32];
    const int m = blockIdx.x, tid = threadIdx.x, W = a.W, Wp = (W + 63) / 64 * 64;
    pdl_launch_dependents();
    if (m >= a.M) {  // rows that pad the image
        pdl_wait();
        for (int c = tid * 8; c < Wp; c += T * 8) {
            const float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            tc_xpack_store8(a.xp, a.xp_mpad, m, c, v);
        }
        return;
    }
    int turn = 0;
    auto sum = [&](float v) {
        float* p = part[turn++];
        v = warp_sum(v);
        if ((tid & 31) == 0) p[tid >> 5] = v;
        __syncthreads();
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < T / 32; ++i) s += p[i];
        return s;
    };
    float v[NV], x[NV], w[NV], nw[NV];
    // weights do not depend on the launch in front
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = tid + k * T;
        w[k] = a.y && i < W ? __ldg(a.w + i) : 0.f;
        nw[k] = a.next_w && i < W ? __ldg(a.next_w + i) : 0.f;
    }
    pdl_wait();
    const float n = (float)W;
    float* xr = a.x + (size_t)m * W;
#pragma unroll
    for (int k = 0; k < NV; ++k) x[k] = tid + k * T < W ? ld_cg_f32(xr + tid + k * T) : 0.f;
    // deviations from the mean and 1 / their root mean square
    auto deviations = [&](float (&z)[NV]) {
        float s = 0.f, q = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) s += z[k];
        const float mean = sum(s) / n;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            z[k] = tid + k * T < W ? z[k] - mean : 0.f;
            q = fmaf(z[k], z[k], q);
        }
        return 1.0f / sqrtf(sum(q) / n + a.eps);
    };
    if (a.y) {
        const float* y = a.y + (size_t)m * a.ldy;
#pragma unroll
        for (int k = 0; k < NV; ++k) v[k] = tid + k * T < W ? ld_cg_f32(y + tid + k * T) : 0.f;
        if (a.left_w) {
            float r[NV], sl = 0.f, sr = 0.f;
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                r[k] = tid + k * T < W ? ld_cg_f32(y + W + tid + k * T) : 0.f;
                sl = fmaf(v[k], v[k], sl);
                sr = fmaf(r[k], r[k], sr);
            }
            const float fl = 1.0f / sqrtf(sum(sl) / n + a.eps), fr = 1.0f / sqrtf(sum(sr) / n + a.eps);
#pragma unroll
            for (int k = 0; k < NV; ++k)
                if (tid + k * T < W) v[k] = 0.5f * ((v[k] * fl) * __ldg(a.left_w + tid + k * T) + (r[k] * fr) * __ldg(a.right_w + tid + k * T));
        }
        const float f = deviations(v);
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            x[k] += (v[k] * f) * w[k];
            if (tid + k * T < W) xr[tid + k * T] = x[k];
        }
    }
    if (!a.next_w) return;
    const float f = deviations(x);
    if (!a.xp) {
#pragma unroll
        for (int k = 0; k < NV; ++k)
            if (tid + k * T < W) a.normed[(size_t)m * W + tid + k * T] = (x[k] * f) * nw[k];
        return;
    }
#pragma unroll
    for (int k = 0; k < NV; ++k)
        if (tid + k * T < Wp) row[tid + k * T] = (x[k] * f) * nw[k];
    for (int c = NV * T + tid; c < Wp; c += T) row[c] = 0.f;
    __syncthreads();
    for (int c = tid * 8; c < Wp; c += T * 8) {
        float o[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = row[c + e];
        tc_xpack_store8(a.xp, a.xp_mpad, m, c, o);
    }
}

template <int T, int NV>
cudaError_t launch(const SandwichArgs& a, cudaStream_t st, bool pdl) {
    const size_t smem = a.xp ? sizeof(float) * (size_t)((a.W + 63) / 64 * 64) : 0;
    const cudaError_t e = ensure_dyn_smem(sandwich_kernel<T, NV>, smem);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)(a.xp && a.next_w ? tc_mpad(a.M) : a.M));
    cfg.blockDim = dim3(T);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, sandwich_kernel<T, NV>, a);
}

}  // namespace

cudaError_t launch_sandwich(const SandwichArgs& a, cudaStream_t st, bool pdl) {
    if (a.M < 1 || a.W < 1 || a.W > SANDWICH_MAX_WIDTH) return cudaErrorInvalidValue;
    if (a.W <= 1024) return launch<256, 4>(a, st, pdl);
    if (a.W <= 2048) return launch<256, 8>(a, st, pdl);
    if (a.W <= 4096) return launch<512, 8>(a, st, pdl);
    if (a.W <= 8192) return launch<1024, 8>(a, st, pdl);
    return launch<1024, 16>(a, st, pdl);
}

}  // namespace hm
