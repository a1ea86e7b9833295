// What lies between the projections and the attention of layers whose heads mix their scores:
//
//   mixed_kv_write   keys and values of the step's rows go to the paged cache, values as (1 - share) v + share * first when the layer mixes
//                    them with another layer's; queries become wide.  Scores are linear in the queries, so Σ_g M[h,g] (q_g · k) is one
//                    product of the wide query [Σ_{g of KV head c} M[h,g] q_g]_c with the keys of all KV heads side by side.
//
// The sums are fp32.  16-bit wide queries leave as one value per feature, or (halves = 2) as a high and a low half, 2^-17 together.
#include <type_traits>

#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

// Host mirror: ops/cuda.py (MixedKvParams).
struct MixedKvParams {
    const void* rows;            // [T, ld]: q [hq * d] | k [hkv * d] | v [hkv * d] | ...
    const void* first;           // [T, ld_first] values of another layer, heads of d_first features (padded unlike d perhaps), or null
    void* q_out;                 // [T, hq, halves * hkv * d]
    void* kv;                    // [pages, 2, hkv, P, d]
    const float* mix;            // [hq, hq]
    const float* share;          // scalar
    const int* seq_ids;
    const int* q_start;
    const int* past_len;
    const int* page_table;
    long long ld, ld_first;
    int tokens, max_pages, page_size, hq, hkv, d, halves, d_first;
};

constexpr int kMixThreads = 256;

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&v)[8]) {
    alignas(16) T e[8];
#pragma unroll
    for (int i = 0; i < (int)(8 * sizeof(T) / 16); ++i) reinterpret_cast<uint4*>(e)[i] = reinterpret_cast<const uint4*>(p)[i];
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = Cvt<T>::to_f(e[i]);
}
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&v)[8]) {
    alignas(16) T e[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) e[i] = Cvt<T>::from_f(v[i]);
#pragma unroll
    for (int i = 0; i < (int)(8 * sizeof(T) / 16); ++i) reinterpret_cast<uint4*>(p)[i] = reinterpret_cast<const uint4*>(e)[i];
}

// One CTA per row.  An item is (part of the query heads, KV head, eight features); the threads behind the items only help with keys and values.
// GS: query heads per KV head kept in registers (0: any number, read again for every result).
template <typename T, int GS>
__global__ void __launch_bounds__(kMixThreads) mixed_kv_write_kernel(const __grid_constant__ MixedKvParams p) {
    pdl_prologue();
    const int tid = threadIdx.x, t = blockIdx.x, hq = p.hq, d = p.d, gs = GS > 0 ? GS : hq / p.hkv, vecs = d / 8, units = p.hkv * vecs;
    const int parts = min(hq, max(1, (int)blockDim.x / units)), per = (hq + parts - 1) / parts, wide = p.hkv * d;
    const T* row = reinterpret_cast<const T*>(p.rows) + (size_t)t * p.ld;
    T* out = reinterpret_cast<T*>(p.q_out) + (size_t)t * hq * wide * p.halves;
    for (int w = tid; w < units * parts; w += blockDim.x) {
        const int part = w / units, u = w - part * units, c = u / vecs, f = (u - c * vecs) * 8;
        const T* src = row + (size_t)c * gs * d + f;
        float q[GS > 0 ? GS : 1][8];
        if constexpr (GS > 0) {
#pragma unroll
            for (int i = 0; i < GS; ++i) load8(src + (size_t)i * d, q[i]);
        }
        const int h1 = min(hq, (part + 1) * per);
#pragma unroll 4
        for (int h = part * per; h < h1; ++h) {
            const float* m = p.mix + h * hq + c * gs;
            float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if constexpr (GS > 0) {
                alignas(16) float mm[GS];
                if constexpr (GS % 4 == 0) {             // hq and c * gs are multiples of 4 then
#pragma unroll
                    for (int i = 0; i < GS; i += 4) *reinterpret_cast<float4*>(mm + i) = __ldg(reinterpret_cast<const float4*>(m + i));
                } else {
#pragma unroll
                    for (int i = 0; i < GS; ++i) mm[i] = __ldg(m + i);
                }
#pragma unroll
                for (int i = 0; i < GS; ++i)
#pragma unroll
                    for (int k = 0; k < 8; ++k) v[k] = fmaf(mm[i], q[i][k], v[k]);
            } else {
                for (int i = 0; i < gs; ++i) {
                    load8(src + (size_t)i * d, q[0]);
#pragma unroll
                    for (int k = 0; k < 8; ++k) v[k] = fmaf(__ldg(m + i), q[0][k], v[k]);
                }
            }
            T* dst = out + (size_t)h * wide * p.halves + c * d + f;
            store8(dst, v);
            if constexpr (sizeof(T) == 2) {
                if (p.halves == 2) {
#pragma unroll
                    for (int k = 0; k < 8; ++k) v[k] -= Cvt<T>::to_f(Cvt<T>::from_f(v[k]));
                    store8(dst + wide, v);
                }
            }
        }
    }
    const int seq = p.seq_ids[t], slot = p.past_len[seq] + t - p.q_start[seq];
    const int page = p.page_table[(size_t)seq * p.max_pages + slot / p.page_size];
    if (page < 0) return;
    T* kv = reinterpret_cast<T*>(p.kv) + ((size_t)page * 2 * p.hkv * p.page_size + slot % p.page_size) * d;
    const float share = p.first ? *p.share : 0.f;
    for (int w = tid; w < 2 * units; w += blockDim.x) {                  // heads count through both planes
        const int c = w / vecs, f = (w - c * vecs) * 8;
        float v[8];
        load8(row + (size_t)hq * d + (size_t)w * 8, v);
        if (p.first && w >= units) {
            float o[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (f < p.d_first) load8(reinterpret_cast<const T*>(p.first) + (size_t)t * p.ld_first + (size_t)(c - p.hkv) * p.d_first + f, o);
#pragma unroll
            for (int k = 0; k < 8; ++k) v[k] = fmaf(share, o[k], (1.f - share) * v[k]);
        }
        store8(kv + (size_t)c * p.page_size * d + f, v);
    }
}

template <typename T>
static int launch_mixed_kv(const MixedKvParams& p, cudaStream_t stream) {
    const int units = p.hkv * p.d / 8;
    const int threads = 2 * units > kMixThreads ? kMixThreads : 2 * units < 64 ? 64 : (2 * units + 31) / 32 * 32;
#define TELB_MIX(GS_) TELB_LAUNCH("mixed_kv_write_kernel", (mixed_kv_write_kernel<T, GS_>), dim3(p.tokens), dim3(threads), 0, stream, p)
    switch (p.hq / p.hkv) {
        case 1: TELB_MIX(1); break;
        case 2: TELB_MIX(2); break;
        case 4: TELB_MIX(4); break;
        case 8: TELB_MIX(8); break;
        default: TELB_MIX(0);
    }
#undef TELB_MIX
    TELB_CHECK_LAUNCH("mixed_kv_write_kernel");
    return 0;
}

}  // namespace telb

using namespace telb;

// dtype: 1 bf16, 2 fp32 (of rows, first, q_out and the cache).
extern "C" int telb_mixed_kv_write(const MixedKvParams* pp, int dtype, cudaStream_t stream) {
    const MixedKvParams& p = *pp;
    if (p.tokens <= 0) return 0;
    if (p.hkv <= 0 || p.hq % p.hkv) return fail("telb_mixed_kv_write: query heads are a multiple of the KV heads");
    if (p.d % 8 || p.ld % 8 || p.ld_first % 8 || p.d_first % 8) return fail("telb_mixed_kv_write: heads and row pitches in multiples of 8");
    if (p.halves != 1 && (p.halves != 2 || dtype == 2)) return fail("telb_mixed_kv_write: one or (16-bit) two halves");
    if (p.first && !p.share) return fail("telb_mixed_kv_write: mixed values have a share");
    if (dtype == 2) return launch_mixed_kv<float>(p, stream);
    return launch_mixed_kv<__nv_bfloat16>(p, stream);
}
