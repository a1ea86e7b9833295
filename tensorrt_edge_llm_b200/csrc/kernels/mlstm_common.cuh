// Launch parameters and gate functions shared by the mLSTM kernels (mlstm.cu, mlstm_tc5.cu).
#pragma once

#include <cuda_runtime.h>

namespace telb {

constexpr float kMlstmEps = 1e-6f;       // added to the normaliser

// Host mirror: ops/cuda.py (MlstmParams).
struct MlstmParams {
    const void* qkvg;          // [T, ld] packed projections: q [heads * dk] | k [heads * dk] | v [heads * dv] | g [heads * dv]
    const float* gates;        // [T, ldg] fp32: input-gate pre-activations [heads] | forget-gate pre-activations [heads] | ...
    float* state;              // [slots, heads, dk, dv] fp32
    float* norm_state;         // [slots, heads, dk + 1] fp32: n, then the running maximum m
    const float* norm_w;       // [heads * dv] fp32
    void* out;                 // [T, heads * dv]
    float* o32;                // [T, heads, dv] fp32 scratch (unused by the decode step)
    float* n_next;             // [sequences, heads, dk + 1] fp32 scratch: normalisers on their way to norm_state
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* slot_ids;
    int* status;
    int ld, ldg, heads, dk, dv, k_off, v_off, g_off, dv_real;
    float scale, cap, eps;
};

__device__ __forceinline__ float mlstm_input_gate(float x, float cap) { return cap * tanhf(x / cap); }
// log(sigmoid(z)) of the capped pre-activation, without cancellation for either sign
__device__ __forceinline__ float mlstm_forget_gate(float x, float cap) {
    const float z = cap * tanhf(x / cap);
    return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

}  // namespace telb
