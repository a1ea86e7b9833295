// Steps of the softmax warps that several attention kernels share.
#pragma once

#include "tc5_common.cuh"

namespace telb {

// Maxima of N column values over the warp; lane l receives that of column l % N.
template <int N>
__device__ __forceinline__ float lat_column_max(const float (&s)[N], int lane) {
    float v[N];
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = s[i];
#pragma unroll
    for (int o = N / 2; o > 0; o >>= 1) {
        const bool hi = lane & o;
#pragma unroll
        for (int i = 0; i < o; ++i) v[i] = fmaxf(hi ? v[i + o] : v[i], __shfl_xor_sync(0xffffffffu, hi ? v[i] : v[i + o], o));
    }
    if constexpr (N == 16) v[0] = fmaxf(v[0], __shfl_xor_sync(0xffffffffu, v[0], 16));
    return v[0];
}

// Whether any of the 128 softmax threads says yes.
__device__ __forceinline__ bool lat_any(bool yes) {
    uint32_t r;
    asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.u32 q, %1, 0;\n\tbar.red.or.pred p, 1, 128, q;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                 : "=r"(r) : "r"(yes ? 1u : 0u) : "memory");
    return r != 0;
}

}  // namespace telb
