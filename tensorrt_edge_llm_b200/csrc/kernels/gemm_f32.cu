// True fp32 matrix product on the CUDA cores (no TF32): out[M,N] = x[M,K] · w[N,K]ᵀ (+ bias[N]), plain and grouped.
// The tensor cores of this part have no fp32 operand type, so models that run in 32 bits (numerics work, small models) use this
// kernel wherever a 16-bit model uses the tcgen05 GEMMs; it keeps their interface, the padded expert layout of the grouped form
// included.  64 x 64 tiles, 256 threads with 4 x 4 outputs each, 16-wide K steps staged in shared memory.
#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

constexpr int kF32Tile = 64;
constexpr int kF32K = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, float* __restrict__ out, const float* __restrict__ bias, int m, int n,
                int k, int ldo, const int* __restrict__ tile_expert, int max_tiles) {
    pdl_prologue();
    __shared__ float sx[kF32K][kF32Tile + 4], sw[kF32K][kF32Tile + 4];
    const int m0 = blockIdx.y * kF32Tile, n0 = blockIdx.x * kF32Tile;
    const float* wb = w;
    const float* bb = bias;
    int rows = m;
    if (tile_expert) {                                   // 128-row tiles, each of one expert (-1 = unused)
        const int tile = m0 >> 7;
        const int e = tile_expert[tile];
        if (e < 0) return;
        rows = (tile << 7) + tile_expert[max_tiles + tile];
        if (m0 >= rows) return;
        wb = w + (size_t)e * n * k;
        if (bias) bb = bias + (size_t)e * n;
    }
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < k; k0 += kF32K) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int kk = k0 + lc + i;
            sx[lc + i][lr] = (m0 + lr < rows && kk < k) ? x[(size_t)(m0 + lr) * k + kk] : 0.f;
            sw[lc + i][lr] = (n0 + lr < n && kk < k) ? wb[(size_t)(n0 + lr) * k + kk] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < kF32K; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = sx[kk][ty * 4 + i];
                b[i] = sw[kk][tx * 4 + i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = m0 + ty * 4 + i;
        if (r >= rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = n0 + tx * 4 + j;
            if (c < n) out[(size_t)r * ldo + c] = acc[i][j] + (bb ? bb[c] : 0.f);
        }
    }
}

// out[t, i] = act(in[t, i]) * in[t, inter + i] for the models whose products above feed it; act: gelu in tanh form, or relu.
__global__ void __launch_bounds__(256) glu_f32_kernel(const float* __restrict__ in, float* __restrict__ out, long long rows, int inter, int relu) {
    pdl_prologue();
    const long long n = rows * inter;
    for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) {
        const long long r = i / inter;
        const float x = in[r * 2 * inter + i - r * inter], u = in[r * 2 * inter + inter + i - r * inter];
        out[i] = (relu ? fmaxf(x, 0.f) : 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)))) * u;
    }
}

// Logit cap in place: x <- cap tanh(x / cap).
__global__ void __launch_bounds__(256) softcap_kernel(float* x, long long n, float cap) {
    pdl_prologue();
    for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) x[i] = cap * tanhf(x[i] / cap);
}

static unsigned grid_for(long long n) {
    const long long blocks = (n + 255) / 256;
    return (unsigned)(blocks < 148 * 16 ? blocks : 148 * 16);
}

}  // namespace telb

using namespace telb;

extern "C" int telb_glu_f32(const float* in, float* out, long long rows, int inter, int relu, cudaStream_t stream) {
    if (rows <= 0 || inter <= 0) return 0;
    TELB_LAUNCH("glu_f32_kernel", glu_f32_kernel, dim3(grid_for(rows * inter)), dim3(256), 0, stream, in, out, rows, inter, relu);
    TELB_CHECK_LAUNCH("glu_f32_kernel");
    return 0;
}

extern "C" int telb_softcap(float* x, long long n, float cap, cudaStream_t stream) {
    if (n <= 0) return 0;
    TELB_LAUNCH("softcap_kernel", softcap_kernel, dim3(grid_for(n)), dim3(256), 0, stream, x, n, cap);
    TELB_CHECK_LAUNCH("softcap_kernel");
    return 0;
}

extern "C" int telb_gemm_f32(const float* x, const float* w, float* out, int M, int N, int K, const float* bias, cudaStream_t stream) {
    if (M <= 0 || N <= 0 || K <= 0) return 0;
    const dim3 grid((N + kF32Tile - 1) / kF32Tile, (M + kF32Tile - 1) / kF32Tile);
    if (grid.y > 65535) return fail("telb_gemm_f32: too many rows");
    TELB_LAUNCH("gemm_f32_kernel", gemm_f32_kernel, grid, dim3(256), 0, stream, x, w, out, bias, M, N, K, N, (const int*)nullptr, 0);
    TELB_CHECK_LAUNCH("gemm_f32_kernel");
    return 0;
}

// The grouped form over the padded expert layout of telb_gemm_f16_grouped.
extern "C" int telb_gemm_f32_grouped(const float* x, const float* w, float* out, int rows_pad, int N, int K, const int* tile_expert,
                                     const float* bias, cudaStream_t stream) {
    if (rows_pad <= 0 || N <= 0 || K <= 0) return 0;
    if (rows_pad % 128) return fail("telb_gemm_f32_grouped: rows_pad must be a multiple of 128");
    const dim3 grid((N + kF32Tile - 1) / kF32Tile, rows_pad / kF32Tile);
    if (grid.y > 65535) return fail("telb_gemm_f32_grouped: too many rows");
    TELB_LAUNCH("gemm_f32_kernel", gemm_f32_kernel, grid, dim3(256), 0, stream, x, w, out, bias, rows_pad, N, K, N, tile_expert, rows_pad / 128);
    TELB_CHECK_LAUNCH("gemm_f32_kernel");
    return 0;
}
