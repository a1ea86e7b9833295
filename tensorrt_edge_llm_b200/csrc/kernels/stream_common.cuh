// Row accesses shared by the kernels of the fp32 residual stream: four consecutive features at a time, as fp32 whatever the row holds.
#pragma once

#include "tc5_common.cuh"

namespace telb {

template <typename T>
__device__ __forceinline__ void get4(const T* p, float (&v)[4]) {
    if constexpr (sizeof(T) == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = Cvt<T>::to_f(e[i]);
    }
}
template <typename T>
__device__ __forceinline__ void put4(T* p, const float (&v)[4]) {
    if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        uint2 u;
        u.x = Cvt<T>::pack2(v[0], v[1]);
        u.y = Cvt<T>::pack2(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = u;
    }
}
__device__ __forceinline__ float post_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

}  // namespace telb
