// Shared by the engine's translation units.
#pragma once

#define HM_CUDA(call)                                      \
    do {                                                   \
        cudaError_t _e = (call);                           \
        if (_e != cudaSuccess) return cuda_fail(_e, #call); \
    } while (0)

namespace hm {
// kernel classes of profile_decode; the classes behind PC_COUNT exist in listed designs only
enum ProfClass { PC_EMBED = 0, PC_QKV, PC_ATTN, PC_O, PC_GATE_UP, PC_DOWN, PC_LM_HEAD, PC_SAMPLE, PC_COUNT, PC_LATENT = PC_COUNT, PC_KUP, PC_VUP, PC_KV_WRITE, PC_ROUTE, PC_NORM, PC_QUP, PC_RECUR, PC_COUNT_LISTED };
}  // namespace hm
