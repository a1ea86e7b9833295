// Row kernels around attention layers whose cache or head geometry is their own:
//
//   latent_write     latent attention: RMS norm of the latent, interleaved rotation of the query and key parts, cache row
//   unit_kv_write    queries and keys over their root mean square, query temperature, cache rows
//   head_linear      one small matrix per head, y[t,h] = W[h] x[t,h]: carries queries into latent space and results out of it
//   latent_gather    cached latent rows of the step's sequences, back to back (input of the key / value expansion)
//
// Norms, rotation and sums are fp32; inputs and outputs have the activation type.
#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

template <typename T>
__device__ __forceinline__ T* cache_row(T* kv, const int* page_table, int max_pages, int page_size, int seq, int slot, int page_rows, int width) {
    const int page = page_table[(size_t)seq * max_pages + slot / page_size];
    return page < 0 ? nullptr : kv + ((size_t)page * page_rows + slot % page_size) * width;
}

// One CTA per row.  Columns: q [heads * kp] | q rotated [heads * rp] | latent [rank_pad] | key rotated [rp].
template <typename T>
__global__ void __launch_bounds__(128)
latent_write_kernel(T* rows, T* kv, const float* cos_sin, const float* norm_w, const int* positions, const int* seq_ids, const int* q_start,
                    const int* past_len, const int* page_table, int max_pages, int page_size, int heads, int kp, int rp, int rank_pad, int rank, int rot,
                    int table_ld, float eps) {
    pdl_prologue();
    __shared__ float red[4];
    const int t = blockIdx.x, tid = threadIdx.x;
    const size_t ld = (size_t)heads * (kp + rp) + rank_pad + rp;
    T* qr = rows + t * ld + (size_t)heads * kp;
    const T* c = qr + (size_t)heads * rp;
    const T* kr = c + rank_pad;
    const float* cs = cos_sin + (size_t)positions[t] * table_ld;
    const int half = rot / 2;
    for (int i = tid; i < heads * half; i += 128) {
        const int h = i / half, j = i - h * half;
        T* pair = qr + h * rp + 2 * j;
        const float u = Cvt<T>::to_f(pair[0]), v = Cvt<T>::to_f(pair[1]), co = cs[j], si = cs[half + j];
        pair[0] = Cvt<T>::from_f(u * co - v * si);
        pair[1] = Cvt<T>::from_f(v * co + u * si);
    }
    float ss = 0.f;
    for (int i = tid; i < rank_pad; i += 128) {
        const float x = Cvt<T>::to_f(c[i]);
        ss += x * x;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    const float inv = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / rank + eps);
    const int s = seq_ids[t];
    T* dst = cache_row(kv, page_table, max_pages, page_size, s, past_len[s] + t - q_start[s], page_size, rank_pad + rp);
    if (!dst) return;
    for (int i = tid; i < rank_pad; i += 128) dst[i] = Cvt<T>::from_f(Cvt<T>::to_f(c[i]) * inv * norm_w[i]);
    dst += rank_pad;
    for (int j = tid; j < rp / 2; j += 128) {
        float u = Cvt<T>::to_f(kr[2 * j]), v = Cvt<T>::to_f(kr[2 * j + 1]);
        if (j < half) {
            const float co = cs[j], si = cs[half + j], a = u * co - v * si;
            v = v * co + u * si;
            u = a;
        }
        dst[2 * j] = Cvt<T>::from_f(u);
        dst[2 * j + 1] = Cvt<T>::from_f(v);
    }
}

// One warp per (row, head) of packed q | k | v; d: padded head, real: features that count in the mean.
template <typename T>
__global__ void __launch_bounds__(128)
unit_kv_write_kernel(const T* qkv, T* q_out, T* kv, const float* temperature, const int* positions, const int* seq_ids, const int* q_start,
                     const int* past_len, const int* page_table, int max_pages, int page_size, int tokens, int hq, int hkv, int d, int real, float eps) {
    pdl_prologue();
    const int heads = hq + 2 * hkv, lane = threadIdx.x & 31;
    const long long wid = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (wid >= (long long)tokens * heads) return;
    const int t = (int)(wid / heads), h = (int)(wid - (long long)t * heads);
    const T* src = qkv + ((size_t)t * heads + h) * d;
    float f = 1.f;
    if (h < hq + hkv) {
        float ss = 0.f;
        for (int i = lane * 2; i < d; i += 64) {
            const float a = Cvt<T>::to_f(src[i]), b = Cvt<T>::to_f(src[i + 1]);
            ss += a * a + b * b;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        f = 1.f / sqrtf(ss / real + eps);
    }
    T* dst;
    if (h < hq) {
        f *= temperature[positions[t]];
        dst = q_out + ((size_t)t * hq + h) * d;
    } else {
        const int s = seq_ids[t], g = h - hq;             // planes keys | values: g counts through both
        dst = cache_row(kv, page_table, max_pages, page_size, s, past_len[s] + t - q_start[s], 2 * hkv * page_size, d);
        if (!dst) return;
        dst += (size_t)g * page_size * d;
    }
    for (int i = lane * 2; i < d; i += 64) {
        dst[i] = Cvt<T>::from_f(Cvt<T>::to_f(src[i]) * f);
        dst[i + 1] = Cvt<T>::from_f(Cvt<T>::to_f(src[i + 1]) * f);
    }
}

// y[t, h, 0..n) = W[h] x[t, h]; then `tail` values of x2[t, h] behind them.  Pitches in elements: ldx / ldy per row, hy per head of y;
// heads of x and x2 lie side by side.  64 x 64 tiles, 4 x 4 results per thread, fp32 sums.
template <typename T>
__global__ void __launch_bounds__(256)
head_linear_kernel(const T* x, const T* w, T* y, const T* x2, int tokens, int n, int k, int tail, int ldx, int ldx2, int ldy, int hy) {
    pdl_prologue();
    __shared__ float sx[32][68], sw[32][68];
    const int h = blockIdx.z, t0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    if (n0 >= n) {                                        // the last column of CTAs copies
        for (int i = threadIdx.x; i < 64 * tail; i += 256) {
            const int t = t0 + i / tail, c = i % tail;
            if (t < tokens) y[(size_t)t * ldy + (size_t)h * hy + n + c] = x2[(size_t)t * ldx2 + (size_t)h * tail + c];
        }
        return;
    }
    const T* wh = w + (size_t)h * n * k;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4, lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 8;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < k; k0 += 32) {                  // k is a multiple of 64, n too
        alignas(16) T a[8], b[8];
        constexpr int kV = 8 * sizeof(T) / 16;
        const bool in = t0 + lr < tokens;
#pragma unroll
        for (int v = 0; v < kV; ++v) {
            reinterpret_cast<uint4*>(a)[v] = in ? reinterpret_cast<const uint4*>(x + (size_t)(t0 + lr) * ldx + (size_t)h * k + k0 + lc)[v] : make_uint4(0, 0, 0, 0);
            reinterpret_cast<uint4*>(b)[v] = reinterpret_cast<const uint4*>(wh + (size_t)(n0 + lr) * k + k0 + lc)[v];
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            sx[lc + i][lr] = Cvt<T>::to_f(a[i]);
            sw[lc + i][lr] = Cvt<T>::to_f(b[i]);
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 32; ++kk) {
            const float4 av = *reinterpret_cast<const float4*>(&sx[kk][ty * 4]), bv = *reinterpret_cast<const float4*>(&sw[kk][tx * 4]);
            const float av4[4] = {av.x, av.y, av.z, av.w}, bv4[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av4[i], bv4[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= tokens) continue;
        T* dst = y + (size_t)t * ldy + (size_t)h * hy + n0 + tx * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) dst[j] = Cvt<T>::from_f(acc[i][j]);
    }
}

// Cached rows [0, past + q_len) of every sequence, sequence s from row out_start[s]; one warp per row, 16 bytes per lane and turn.
// Sequences with at most min_q rows in the step are left out.
__global__ void __launch_bounds__(128)
latent_gather_kernel(const uint4* kv, uint4* latent, uint4* rot, const int* out_start, const int* q_len, const int* past_len, const int* page_table, int max_pages,
                     int page_size, int rank16, int rot16, int min_q) {
    pdl_prologue();
    const int seq = blockIdx.y, lane = threadIdx.x & 31;
    const int ql = q_len[seq];
    if (ql <= min_q) return;
    const int total = past_len[seq] + ql;
    for (int r = blockIdx.x * 4 + (threadIdx.x >> 5); r < total; r += gridDim.x * 4) {
        const uint4* src = cache_row(kv, page_table, max_pages, page_size, seq, r, page_size, rank16 + rot16);
        const size_t o = (size_t)out_start[seq] + r;
        for (int i = lane; i < rank16 + rot16; i += 32) {
            const uint4 v = src ? src[i] : make_uint4(0, 0, 0, 0);
            if (i < rank16) latent[o * rank16 + i] = v;
            else rot[o * rot16 + i - rank16] = v;
        }
    }
}

}  // namespace telb

using namespace telb;

#define TELB_BY_TYPE(dtype, CALL)                                  \
    if ((dtype) == 2) { typedef float T; CALL; }                   \
    else if ((dtype) == 1) { typedef __nv_bfloat16 T; CALL; }      \
    else { typedef __half T; CALL; }

extern "C" int telb_latent_write(void* rows, void* kv_layer, const float* cos_sin, const float* norm_w, const int* positions, const int* seq_ids,
                                 const int* q_start, const int* past_len, const int* page_table, int tokens, int max_pages, int page_size, int heads, int kp,
                                 int rp, int rank_pad, int rank, int rot, int table_ld, float eps, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (rot % 2 || rot > rp || rank > rank_pad || rank <= 0) return fail("telb_latent_write: sizes");
    TELB_BY_TYPE(dtype, TELB_LAUNCH("latent_write_kernel", (latent_write_kernel<T>), dim3(tokens), dim3(128), 0, stream, (T*)rows, (T*)kv_layer, cos_sin, norm_w,
                                    positions, seq_ids, q_start, past_len, page_table, max_pages, page_size, heads, kp, rp, rank_pad, rank, rot, table_ld, eps))
    TELB_CHECK_LAUNCH("latent_write_kernel");
    return 0;
}

extern "C" int telb_unit_kv_write(const void* qkv, void* q_out, void* kv_layer, const float* temperature, const int* positions, const int* seq_ids,
                                  const int* q_start, const int* past_len, const int* page_table, int tokens, int max_pages, int page_size, int hq, int hkv,
                                  int d, int real, float eps, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (d % 64 || real <= 0 || real > d) return fail("telb_unit_kv_write: padded heads are multiples of 64");
    const long long warps = (long long)tokens * (hq + 2 * hkv);
    TELB_BY_TYPE(dtype, TELB_LAUNCH("unit_kv_write_kernel", (unit_kv_write_kernel<T>), dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, stream, (const T*)qkv, (T*)q_out,
                                    (T*)kv_layer, temperature, positions, seq_ids, q_start, past_len, page_table, max_pages, page_size, tokens, hq, hkv, d, real, eps))
    TELB_CHECK_LAUNCH("unit_kv_write_kernel");
    return 0;
}

extern "C" int telb_head_linear(const void* x, const void* w, void* y, const void* x2, int tokens, int heads, int n, int k, int tail, int ldx, int ldx2,
                                int ldy, int hy, int dtype, cudaStream_t stream) {
    if (tokens <= 0 || heads <= 0) return 0;
    if (n % 64 || k % 64 || ldx % 8) return fail("telb_head_linear: sizes must be multiples of 64 and the row pitch of 8");
    if (heads > 65535 || tokens > 65535 * 64) return fail("telb_head_linear: too many heads or rows");
    const dim3 grid(n / 64 + (tail > 0 ? 1 : 0), (tokens + 63) / 64, heads);
    TELB_BY_TYPE(dtype, TELB_LAUNCH("head_linear_kernel", (head_linear_kernel<T>), grid, dim3(256), 0, stream, (const T*)x, (const T*)w, (T*)y, (const T*)x2,
                                    tokens, n, k, tail, ldx, ldx2, ldy, hy))
    TELB_CHECK_LAUNCH("head_linear_kernel");
    return 0;
}

// rank, rot in bytes (multiples of 16).
extern "C" int telb_latent_gather(const void* kv_layer, void* latent, void* rot, const int* out_start, const int* q_len, const int* past_len, const int* page_table,
                                  int num_seqs, int max_total, int max_pages, int page_size, int rank_bytes, int rot_bytes, int min_q, cudaStream_t stream) {
    if (num_seqs <= 0 || max_total <= 0) return 0;
    if (rank_bytes % 16 || rot_bytes % 16 || num_seqs > 65535) return fail("telb_latent_gather: sizes");
    const int blocks = min((max_total + 3) / 4, 2048);
    TELB_LAUNCH("latent_gather_kernel", latent_gather_kernel, dim3(blocks, num_seqs), dim3(128), 0, stream, (const uint4*)kv_layer, (uint4*)latent, (uint4*)rot,
                out_start, q_len, past_len, page_table, max_pages, page_size, rank_bytes / 16, rot_bytes / 16, min_q);
    TELB_CHECK_LAUNCH("latent_gather_kernel");
    return 0;
}
