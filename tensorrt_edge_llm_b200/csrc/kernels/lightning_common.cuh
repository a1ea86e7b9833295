// Launch parameters and the activation shared by the lightning attention kernels (lightning.cu, lightning_tc5.cu).
#pragma once

#include <cuda_runtime.h>

#include "tc5_common.cuh"

namespace telb {

// Host mirror: ops/cuda.py (LightningParams).
struct LightningParams {
    const void* rows;          // [T, ld] packed projections: q [heads * dk] | k [heads * dk] | v [heads * dv] | g [heads * dv]
    void* act;                 // [T, g_off]: silu of q | k | v (scratch of the chunk kernel)
    const float* powers;       // [heads, n_powers]: decay^0, decay^1, ...
    float* state;              // [slots, heads, dk, dv] fp32
    const float* norm_w;       // [heads * dv] fp32
    void* out;                 // [T, heads * dv]: read-outs times weight and gate
    float* sums;               // [T, heads * dv / 32]: squares of 32 read-outs each
    float* carry;              // [sequences, heads, segments, dk, dv] fp32 scratch: states in front of the segments (chunk kernel)
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* slot_ids;
    int* status;
    int ld, heads, dk, dv, k_off, v_off, g_off, n_powers, tokens, num_seqs, segments, seg_chunks;
};

// silu in the precision of the projection it belongs to
template <typename T>
__device__ __forceinline__ float lightning_silu(float x) {
    if constexpr (sizeof(T) == 4) return x / (1.f + expf(-x));
    else return Cvt<T>::to_f(Cvt<T>::from_f(__fdividef(x, 1.f + __expf(-x))));
}

// weight and sigmoid gate of a read-out
template <typename T>
__device__ __forceinline__ float lightning_gate(float o, float w, float g) {
    if constexpr (sizeof(T) == 4) return o * w / (1.f + expf(-g));
    else return __fdividef(o * w, 1.f + __expf(-g));
}

}  // namespace telb
