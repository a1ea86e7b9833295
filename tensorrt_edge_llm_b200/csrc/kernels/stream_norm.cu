// The fp32 residual stream of parallel blocks.  A parallel layer normalises once, both sublayers read that row, and the stream
// advances by x += mult * (mixer + feed-forward).  One kernel does everything that lies between two layers:
//
//   source      x = table_mult * table[id] (first call) or the running fp32 stream
//   update      x += mult * (a + Σ_k w[t,k] · y[dst_row[t,k]])      a: mixer output, the sum: combine of the routed experts
//   step        x += step                                            one vector for all rows (start of a pass of a looped stack)
//   norm        h = x / sqrt(mean(x²) + eps) * (offset + weight)     written in the activation type for the next GEMMs, or
//               h = tanh(alpha x) * weight + bias                    with a scalar alpha: no statistics, no reduction
//
// so neither the combined expert output nor the sum of the two sublayers ever goes to memory, and the stream itself is read and
// written once per layer.  The stream, the norm and the weights stay fp32; `offset` 1 serves weights that are stored around zero.
#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

struct StreamParams {
    const int* ids;          // embedding source, or null
    const void* table;       // [vocab, width]
    int vocab;
    const float* x_in;       // [T, width] fp32 stream when ids is null
    const void* a;           // [T, width] or null
    const void* y;           // [rows_pad, ldy] expert outputs, or null
    const int* dst_row;      // [T, top_k]
    const float* topk_w;     // [T, top_k]
    int top_k, ldy;
    float mult;
    const float* step;       // [width] or null
    const float* weight;     // [width] or null (no norm)
    float offset, eps;
    const float* alpha;      // scalar: element-wise tanh norm, or null
    const float* bias;       // [width], with alpha
    float table_mult;
    float* x_out;            // [T, width]
    void* h;                 // [T, width] or null
    int width;
};

constexpr int kStreamThreads = 256;
constexpr int kStreamMaxTopK = 32;

// Four consecutive values of a row as fp32.
template <typename T>
__device__ __forceinline__ void load4(const T* p, float (&v)[4]) {
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

// One CTA per row; thread i owns features 4 i, 4 (i + 256), ... (kept in registers: E groups of four, width <= 1024 E).
template <typename T, int E>
__global__ void __launch_bounds__(kStreamThreads) stream_norm_kernel(const __grid_constant__ StreamParams p) {
    pdl_prologue();
    __shared__ float red[8];
    __shared__ int s_row[kStreamMaxTopK];
    __shared__ float s_w[kStreamMaxTopK];
    const size_t t = blockIdx.x;
    const int tid = threadIdx.x;
    if (p.y) {
        if (tid < p.top_k) {
            s_row[tid] = p.dst_row[t * p.top_k + tid];
            s_w[tid] = p.topk_w[t * p.top_k + tid];
        }
        __syncthreads();
    }
    float x[E][4];
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * kStreamThreads + tid) * 4;
        if (c >= p.width) break;
        if (p.ids) {
            const int id = min(max(p.ids[t], 0), p.vocab - 1);
            load4(reinterpret_cast<const T*>(p.table) + (size_t)id * p.width + c, x[e]);
#pragma unroll
            for (int i = 0; i < 4; ++i) x[e][i] *= p.table_mult;
        } else {
            load4(p.x_in + t * p.width + c, x[e]);
        }
        if (p.a || p.y) {
            float d[4] = {0.f, 0.f, 0.f, 0.f};
            if (p.a) load4(reinterpret_cast<const T*>(p.a) + t * p.width + c, d);
            if (p.y) {
                for (int k = 0; k < p.top_k; ++k) {
                    if (s_row[k] < 0) continue;
                    float v[4];
                    load4(reinterpret_cast<const T*>(p.y) + (size_t)s_row[k] * p.ldy + c, v);
#pragma unroll
                    for (int i = 0; i < 4; ++i) d[i] += s_w[k] * v[i];
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) x[e][i] += p.mult * d[i];
        }
        if (p.step) {
            float v[4];
            load4(p.step + c, v);
#pragma unroll
            for (int i = 0; i < 4; ++i) x[e][i] += v[i];
        }
        *reinterpret_cast<float4*>(p.x_out + t * p.width + c) = make_float4(x[e][0], x[e][1], x[e][2], x[e][3]);
#pragma unroll
        for (int i = 0; i < 4; ++i) ss += x[e][i] * x[e][i];
    }
    if (!p.h) return;
    float inv = 0.f, alpha = 0.f;
    if (p.alpha) {
        alpha = *p.alpha;
    } else {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if ((tid & 31) == 0) red[tid >> 5] = ss;
        __syncthreads();
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < kStreamThreads / 32; ++w) tot += red[w];
        inv = 1.f / sqrtf(tot / p.width + p.eps);
    }
    T* h = reinterpret_cast<T*>(p.h) + t * p.width;
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * kStreamThreads + tid) * 4;
        if (c >= p.width) break;
        float g[4];
        load4(p.weight + c, g);
        if (p.alpha) {
            float b[4];
            load4(p.bias + c, b);
#pragma unroll
            for (int i = 0; i < 4; ++i) g[i] = fmaf(tanhf(alpha * x[e][i]), g[i], b[i]);
        } else {
#pragma unroll
            for (int i = 0; i < 4; ++i) g[i] = x[e][i] * inv * (p.offset + g[i]);
        }
        if constexpr (sizeof(T) == 4) {
            *reinterpret_cast<float4*>(h + c) = make_float4(g[0], g[1], g[2], g[3]);
        } else {
            uint2 u;
            u.x = Cvt<T>::pack2(g[0], g[1]);
            u.y = Cvt<T>::pack2(g[2], g[3]);
            *reinterpret_cast<uint2*>(h + c) = u;
        }
    }
}

template <typename T>
static int launch_stream(const StreamParams& p, int tokens, cudaStream_t stream) {
    const int groups = (p.width + kStreamThreads * 4 - 1) / (kStreamThreads * 4);
#define TELB_STREAM(E_) TELB_LAUNCH("stream_norm_kernel", (stream_norm_kernel<T, E_>), dim3(tokens), dim3(kStreamThreads), 0, stream, p)
    if (groups <= 1) TELB_STREAM(1);
    else if (groups <= 2) TELB_STREAM(2);
    else if (groups <= 4) TELB_STREAM(4);
    else if (groups <= 8) TELB_STREAM(8);
    else TELB_STREAM(16);
#undef TELB_STREAM
    TELB_CHECK_LAUNCH("stream_norm_kernel");
    return 0;
}

}  // namespace telb

using namespace telb;

// dtype: 0 fp16, 1 bf16, 2 fp32 (of table, a, y and h; the stream, step and weight are fp32).
extern "C" int telb_stream_norm(const int* ids, const void* table, int vocab, const float* x_in, const void* a, const void* y, const int* dst_row,
                                const float* topk_w, int top_k, int ldy, float mult, const float* step, const float* weight, float offset,
                                float eps, const float* alpha, const float* bias, float table_mult, float* x_out, void* h, int tokens,
                                int width, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (width % 4 || width > 16 * 1024) return fail("telb_stream_norm: width must be a multiple of 4 and at most 16384");
    if (y && (top_k > kStreamMaxTopK || ldy % 4)) return fail("telb_stream_norm: top_k <= 32 and an expert row pitch that is a multiple of 4");
    if (!ids && !x_in) return fail("telb_stream_norm: ids or a stream is needed");
    if (alpha && weight && !bias) return fail("telb_stream_norm: the tanh norm has a bias");
    StreamParams p{ids, table, vocab, x_in, a, y, dst_row, topk_w, top_k, ldy, mult, step, weight, offset, eps, alpha, bias, table_mult, x_out, h, width};
    if (dtype == 2) return launch_stream<float>(p, tokens, stream);
    return dtype == 1 ? launch_stream<__nv_bfloat16>(p, tokens, stream) : launch_stream<__half>(p, tokens, stream);
}
