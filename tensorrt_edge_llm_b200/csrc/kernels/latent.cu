// Row kernels around attention layers whose cache or head geometry is their own:
//
//   latent_write     latent attention: RMS norm of the latent, interleaved rotation of the query and key parts, cache row
//   unit_kv_write    queries and keys over their root mean square, query temperature, cache rows
//   turned_kv_write  norms over whole query and key rows, interleaved rotation of queries, keys and values, cache rows
//   head_linear      one small matrix per head, y[t,h] = W[h] x[t,h]: carries queries into latent space and results out of it
//   latent_gather    cached latent rows of the step's sequences, back to back (input of the key / value expansion)
//
// Norms, rotation and sums are fp32; inputs and outputs have the activation type.
#include <type_traits>

#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

template <typename T>
__device__ __forceinline__ T* cache_row(T* kv, const int* page_table, int max_pages, int page_size, int seq, int slot, int page_rows, int width) {
    const int page = page_table[(size_t)seq * max_pages + slot / page_size];
    return page < 0 ? nullptr : kv + ((size_t)page * page_rows + slot % page_size) * width;
}

// Eight consecutive values, moved as 16-byte words.
template <typename T>
struct Eight {
    alignas(16) T e[8];
    __device__ __forceinline__ void load(const T* p) {
#pragma unroll
        for (int v = 0; v < (int)(8 * sizeof(T) / 16); ++v) reinterpret_cast<uint4*>(e)[v] = reinterpret_cast<const uint4*>(p)[v];
    }
    __device__ __forceinline__ void store(T* p) const {
#pragma unroll
        for (int v = 0; v < (int)(8 * sizeof(T) / 16); ++v) reinterpret_cast<uint4*>(p)[v] = reinterpret_cast<const uint4*>(e)[v];
    }
    // pairs j .. j + 3 of a head; those from `half` on pass
    __device__ __forceinline__ void turn(const float* cs, int j, int half) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            if (j + i >= half) break;
            const float u = Cvt<T>::to_f(e[2 * i]), v = Cvt<T>::to_f(e[2 * i + 1]), co = cs[j + i], si = cs[half + j + i];
            e[2 * i] = Cvt<T>::from_f(u * co - v * si);
            e[2 * i + 1] = Cvt<T>::from_f(v * co + u * si);
        }
    }
};

// Columns of a row: q [heads * kp] | q rotated [heads * rp] | latent [rank_pad] | key rotated [rp].  Two kinds of warps: one per row for
// the latent and the key part, and one per row and 1024 rotated query features.
template <typename T>
__global__ void __launch_bounds__(128)
latent_write_kernel(T* rows, T* kv, const float* cos_sin, const float* norm_w, const int* positions, const int* seq_ids, const int* q_start,
                    const int* past_len, const int* page_table, int max_pages, int page_size, int tokens, int heads, int kp, int rp, int rank_pad, int rank,
                    int rot, int table_ld, float eps, int parts) {
    pdl_prologue();
    const int lane = threadIdx.x & 31;
    const long long wid = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (wid >= (long long)tokens * parts) return;
    const int t = (int)(wid / parts), part = (int)(wid - (long long)t * parts);
    const size_t ld = (size_t)heads * (kp + rp) + rank_pad + rp;
    T* qr = rows + t * ld + (size_t)heads * kp;
    const float* cs = cos_sin + (size_t)positions[t] * table_ld;
    const int half = rot / 2;
    Eight<T> x;
    if (part > 0) {
        const int end = min(heads * rp, part * 1024);
        for (int i = (part - 1) * 1024 + lane * 8; i < end; i += 256) {
            const int j = i % rp / 2;
            if (j >= half) continue;                      // padding
            x.load(qr + i);
            x.turn(cs, j, half);
            x.store(qr + i);
        }
        return;
    }
    const T* c = qr + (size_t)heads * rp;
    float ss = 0.f;
    for (int i = lane * 8; i < rank_pad; i += 256) {
        x.load(c + i);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const float v = Cvt<T>::to_f(x.e[k]);
            ss = fmaf(v, v, ss);
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = 1.f / sqrtf(ss / rank + eps);
    const int s = seq_ids[t];
    T* dst = cache_row(kv, page_table, max_pages, page_size, s, past_len[s] + t - q_start[s], page_size, rank_pad + rp);
    if (!dst) return;
    for (int i = lane * 8; i < rank_pad; i += 256) {
        x.load(c + i);
#pragma unroll
        for (int k = 0; k < 8; ++k) x.e[k] = Cvt<T>::from_f(Cvt<T>::to_f(x.e[k]) * inv * norm_w[i + k]);
        x.store(dst + i);
    }
    for (int i = lane * 8; i < rp; i += 256) {
        x.load(c + rank_pad + i);
        x.turn(cs, i / 2, half);
        x.store(dst + rank_pad + i);
    }
}

// One CTA per row of packed q | k | v.  The norms divide by the real features of all heads together; every pair of a padded head turns
// by its own row of the table (features that do not rotate have angle zero).
struct TurnedKvParams {
    const void* rows;            // [T, ld]
    void* q_out;                 // [T, hq, d]
    void* kv;                    // [pages, 2, hkv, P, d]
    const float* key_table;      // [positions, d]: d / 2 cos | d / 2 sin
    const float* value_table;
    const float* q_norm;         // [hq * d]
    const float* k_norm;         // [hkv * d]
    const int* positions;
    const int* seq_ids;
    const int* q_start;
    const int* past_len;
    const int* page_table;
    int ld, tokens, max_pages, page_size, hq, hkv, d, real;
    float eps;
};

constexpr int kTurnThreads = 128;

template <typename T>
__global__ void __launch_bounds__(kTurnThreads) turned_kv_write_kernel(const __grid_constant__ TurnedKvParams p) {
    pdl_prologue();
    __shared__ float red[2][kTurnThreads / 32];
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const T* src = reinterpret_cast<const T*>(p.rows) + (size_t)t * p.ld;
    const int qn = p.hq * p.d, kn = p.hkv * p.d;
    float ss[2] = {0.f, 0.f};
    Eight<T> x;
    for (int c = tid * 8; c < qn + kn; c += kTurnThreads * 8) {
        x.load(src + c);
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float v = Cvt<T>::to_f(x.e[i]);
            s = fmaf(v, v, s);
        }
        ss[c < qn ? 0 : 1] += s;
    }
#pragma unroll
    for (int k = 0; k < 2; ++k) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss[k] += __shfl_xor_sync(0xffffffffu, ss[k], o);
        if (lane == 0) red[k][warp] = ss[k];
    }
    __syncthreads();
    float inv[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < kTurnThreads / 32; ++w) s += red[k][w];
        inv[k] = 1.f / sqrtf(s / ((k ? p.hkv : p.hq) * p.real) + p.eps);
    }
    const int seq = p.seq_ids[t], pos = p.positions[t], half = p.d / 2;
    T* dst = cache_row(reinterpret_cast<T*>(p.kv), p.page_table, p.max_pages, p.page_size, seq, p.past_len[seq] + t - p.q_start[seq], 2 * p.hkv * p.page_size, p.d);
    for (int c = tid * 8; c < qn + 2 * kn; c += kTurnThreads * 8) {
        const int kind = c < qn ? 0 : c < qn + kn ? 1 : 2, f = c % p.d;
        const float* cs = (kind == 2 ? p.value_table : p.key_table) + (size_t)pos * p.d + f / 2;
        const float4 co4 = *reinterpret_cast<const float4*>(cs), si4 = *reinterpret_cast<const float4*>(cs + half);
        const float co[4] = {co4.x, co4.y, co4.z, co4.w}, si[4] = {si4.x, si4.y, si4.z, si4.w};
        x.load(src + c);
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = Cvt<T>::to_f(x.e[i]);
        if (kind < 2) {
            const float* w = kind ? p.k_norm + c - qn : p.q_norm + c;
            const float4 w0 = *reinterpret_cast<const float4*>(w), w1 = *reinterpret_cast<const float4*>(w + 4);
            const float g[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= inv[kind] * g[i];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            x.e[2 * i] = Cvt<T>::from_f(v[2 * i] * co[i] - v[2 * i + 1] * si[i]);
            x.e[2 * i + 1] = Cvt<T>::from_f(v[2 * i + 1] * co[i] + v[2 * i] * si[i]);
        }
        if (kind == 0) x.store(reinterpret_cast<T*>(p.q_out) + (size_t)t * qn + c);
        else if (dst) x.store(dst + (size_t)((c - qn) / p.d) * p.page_size * p.d + f);      // planes keys | values: heads count through both
    }
}

// One warp per row and group of heads of packed q | k | v: a lane holds eight consecutive features, d / 8 lanes a head, so a warp takes
// 256 / d heads at once (wider heads in turns of 256 features).  d: padded head, real: features that count in the mean.
template <typename T>
__global__ void __launch_bounds__(128)
unit_kv_write_kernel(const T* qkv, T* q_out, T* kv, const float* temperature, const int* positions, const int* seq_ids, const int* q_start,
                     const int* past_len, const int* page_table, int max_pages, int page_size, int tokens, int hq, int hkv, int d, int real, float eps,
                     int lanes) {
    pdl_prologue();
    constexpr int kV = 8 * sizeof(T) / 16;
    const int heads = hq + 2 * hkv, lane = threadIdx.x & 31, per = 32 / lanes, groups = (heads + per - 1) / per;
    const long long wid = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (wid >= (long long)tokens * groups) return;
    const int t = (int)(wid / groups), h = (int)(wid - (long long)t * groups) * per + lane / lanes, li = lane % lanes;
    const bool live = h < heads;
    const T* src = qkv + ((size_t)t * heads + (live ? h : 0)) * d;
    float ss = 0.f;
    alignas(16) T e[8];
    for (int c = li * 8; c < d; c += lanes * 8) {
#pragma unroll
        for (int v = 0; v < kV; ++v) reinterpret_cast<uint4*>(e)[v] = reinterpret_cast<const uint4*>(src + c)[v];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float x = Cvt<T>::to_f(e[i]);
            ss = fmaf(x, x, ss);
        }
    }
    for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!live) return;
    float f = h < hq + hkv ? 1.f / sqrtf(ss / real + eps) : 1.f;
    T* dst;
    if (h < hq) {
        f *= temperature[positions[t]];
        dst = q_out + ((size_t)t * hq + h) * d;
    } else {
        const int s = seq_ids[t];                         // planes keys | values: h - hq counts through both
        dst = cache_row(kv, page_table, max_pages, page_size, s, past_len[s] + t - q_start[s], 2 * hkv * page_size, d);
        if (!dst) return;
        dst += (size_t)(h - hq) * page_size * d;
    }
    for (int c = li * 8; c < d; c += lanes * 8) {
        if (d > lanes * 8) {                              // several turns: read again
#pragma unroll
            for (int v = 0; v < kV; ++v) reinterpret_cast<uint4*>(e)[v] = reinterpret_cast<const uint4*>(src + c)[v];
        }
        if (h < hq + hkv) {
#pragma unroll
            for (int i = 0; i < 8; ++i) e[i] = Cvt<T>::from_f(Cvt<T>::to_f(e[i]) * f);
        }
#pragma unroll
        for (int v = 0; v < kV; ++v) reinterpret_cast<uint4*>(dst + c)[v] = reinterpret_cast<const uint4*>(e)[v];
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

// The same product for 16-bit rows on tcgen05: Yᵀ[64 outputs, 64 rows] = W[h] (A, K-major) · X[:, h]ᵀ (B, K-major).  A CTA keeps its 64 rows
// of one head's matrix in shared memory and walks the row tiles.  The upper half of the 128-row A tile is never loaded; what it holds only
// reaches accumulator rows that nobody reads.  Warps 0-1: results; warp 2: copies and MMA; warp 3: TMEM, tail columns.
template <typename T>
__global__ void __launch_bounds__(128)
head_linear_tc5_kernel(const __grid_constant__ CUtensorMap tma_w, const __grid_constant__ CUtensorMap tma_x, T* y, const T* x2, int tokens, int n, int kc, int tail,
                       int ldx2, int ldy, int hy, int* status) {
    constexpr bool kBf16 = std::is_same<T, __nv_bfloat16>::value;
    constexpr int kWChunk = 128 * 128, kXChunk = 64 * 128;
    extern __shared__ uint8_t hl_raw[];
    __shared__ uint64_t bar_w, bar_x, bar_d, bar_free;
    __shared__ uint32_t tmem_word, abort_word;
    uint8_t* s_w = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(hl_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* s_x = s_w + kc * kWChunk;
    volatile uint32_t* abort_flag = &abort_word;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, n0 = blockIdx.x * 64;
    const int tiles = (tokens + 63) / 64;
    if (threadIdx.x == 0) {
        mbar_init(&bar_w, 1);
        mbar_init(&bar_x, 1);
        mbar_init(&bar_d, 1);
        mbar_init(&bar_free, 64);
        abort_word = 0;
        mbar_fence_init();
    }
    __syncthreads();
    if (warp == 2 && lane == 0) {                         // the matrix does not depend on earlier kernels
        mbar_expect_tx(&bar_w, kc * 64 * 128);
        for (int c = 0; c < kc; ++c) tma_load_2d(s_w + c * kWChunk, &tma_w, &bar_w, c * 64, h * n + n0);
    }
    pdl_wait();                                           // before TMEM: a kernel that is still running may be about to allocate its own
    if (warp == 3) {
        tmem_alloc(&tmem_word, 64);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = tmem_word;
    pdl_launch_dependents();
    if (warp == 2) {
        if (lane == 0) {
            const uint32_t idesc = idesc_f16(128, 64, kBf16);
            bool ok = true;
            int it = 0;
            for (int t = blockIdx.z; t < tiles && ok; t += gridDim.z, ++it) {
                // the tile before has been read out: its product is complete and its accumulator free
                if (it > 0) ok = mbar_wait(&bar_free, (it - 1) & 1, abort_flag, status, kStatusProducerTimeout);
                if (!ok) break;
                tc_fence_after_sync();
                mbar_expect_tx(&bar_x, kc * kXChunk);
                for (int c = 0; c < kc; ++c) tma_load_3d(s_x + c * kXChunk, &tma_x, &bar_x, c * 64, h, t * 64);
                if (it == 0) ok = mbar_wait(&bar_w, 0, abort_flag, status, kStatusMmaTimeout);
                ok = ok && mbar_wait(&bar_x, it & 1, abort_flag, status, kStatusMmaTimeout);
                if (!ok) break;
                tc_fence_after_sync();
                for (int c = 0; c < kc; ++c) {
                    const uint64_t dw = smem_desc_sw128(s_w + c * kWChunk), dx = smem_desc_sw128(s_x + c * kXChunk);
#pragma unroll
                    for (int k = 0; k < 4; ++k) umma_f16(tmem, dw + 2 * k, dx + 2 * k, idesc, (c | k) ? 1u : 0u);
                }
                umma_commit(&bar_d);
            }
        }
    } else if (warp < 2) {
        const int r = warp * 32 + lane;
        int it = 0;
        for (int t = blockIdx.z; t < tiles; t += gridDim.z, ++it) {
            if (!mbar_wait(&bar_d, it & 1, abort_flag, status, kStatusEpilogueTimeout)) break;
            tc_fence_after_sync();
            uint32_t a[32], b[32];
            tmem_ld_x32(tmem + (static_cast<uint32_t>(warp * 32) << 16), a);
            tmem_ld_x32(tmem + (static_cast<uint32_t>(warp * 32) << 16) + 32, b);
            tmem_ld_wait();
            tc_fence_before_sync();
            mbar_arrive(&bar_free);
            T* dst = y + (size_t)t * 64 * ldy + (size_t)h * hy + n0 + r;
            const int cnt = min(64, tokens - t * 64);
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                if (i < cnt) dst[(size_t)i * ldy] = Cvt<T>::from_f(__uint_as_float(a[i]));
                if (i + 32 < cnt) dst[(size_t)(i + 32) * ldy] = Cvt<T>::from_f(__uint_as_float(b[i]));
            }
        }
    } else if (tail > 0 && n0 == 0) {
        const int v = tail / 8;                           // 16-byte pieces
        for (int t = blockIdx.z; t < tiles; t += gridDim.z)
            for (int i = lane; i < 64 * v; i += 32) {
                const int row = t * 64 + i / v, c = i % v * 8;
                if (row < tokens)
                    *reinterpret_cast<uint4*>(y + (size_t)row * ldy + (size_t)h * hy + n + c) =
                        *reinterpret_cast<const uint4*>(x2 + (size_t)row * ldx2 + (size_t)h * tail + c);
            }
    }
    if (*abort_flag) {
        const uint64_t t0 = global_timer_ns();
        while (global_timer_ns() - t0 < 200000ull) __nanosleep(1000);
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 3) {
        tc_fence_after_sync();
        tmem_dealloc(tmem, 64);
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
    if (rot % 2 || rot > rp || rp % 8 || kp % 8 || rank_pad % 8 || rank > rank_pad || rank <= 0) return fail("telb_latent_write: sizes");
    const int parts = 1 + (heads * rp + 1023) / 1024;
    const long long warps = (long long)tokens * parts;
    TELB_BY_TYPE(dtype, TELB_LAUNCH("latent_write_kernel", (latent_write_kernel<T>), dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, stream, (T*)rows, (T*)kv_layer,
                                    cos_sin, norm_w, positions, seq_ids, q_start, past_len, page_table, max_pages, page_size, tokens, heads, kp, rp, rank_pad, rank,
                                    rot, table_ld, eps, parts))
    TELB_CHECK_LAUNCH("latent_write_kernel");
    return 0;
}

extern "C" int telb_unit_kv_write(const void* qkv, void* q_out, void* kv_layer, const float* temperature, const int* positions, const int* seq_ids,
                                  const int* q_start, const int* past_len, const int* page_table, int tokens, int max_pages, int page_size, int hq, int hkv,
                                  int d, int real, float eps, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (d % 64 || real <= 0 || real > d) return fail("telb_unit_kv_write: padded heads are multiples of 64");
    const int lanes = d <= 64 ? 8 : d <= 128 ? 16 : 32;
    const long long warps = (long long)tokens * ((hq + 2 * hkv + 32 / lanes - 1) / (32 / lanes));
    TELB_BY_TYPE(dtype, TELB_LAUNCH("unit_kv_write_kernel", (unit_kv_write_kernel<T>), dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, stream, (const T*)qkv, (T*)q_out,
                                    (T*)kv_layer, temperature, positions, seq_ids, q_start, past_len, page_table, max_pages, page_size, tokens, hq, hkv, d, real, eps, lanes))
    TELB_CHECK_LAUNCH("unit_kv_write_kernel");
    return 0;
}

template <typename T>
static int launch_head_linear_tc5(const void* x, const void* w, void* y, const void* x2, int tokens, int heads, int n, int k, int tail, int ldx, int ldx2, int ldy,
                                  int hy, int* status, cudaStream_t stream) {
    const int kc = k / 64, smem = kc * (128 + 64) * 128 + 1024;
    static int configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(head_linear_tc5_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(head_linear_tc5)", e);
        configured = smem;
    }
    const CUtensorMapDataType dt = std::is_same<T, __nv_bfloat16>::value ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16;
    CUtensorMap mw, mx;
    if (make_tmap_2d(&mw, dt, 2, w, (uint64_t)heads * n, k, (uint64_t)k * 2, 64, 64, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    const uint64_t dims[3] = {(uint64_t)k, (uint64_t)heads, (uint64_t)tokens}, strides[2] = {(uint64_t)k * 2, (uint64_t)ldx * 2};
    const uint32_t box[3] = {64, 1, 64};
    if (make_tmap_nd(&mx, dt, 3, x, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    const int tiles = (tokens + 63) / 64, want = (2 * sm_count() + heads * (n / 64) - 1) / (heads * (n / 64));
    TELB_LAUNCH("head_linear_tc5_kernel", (head_linear_tc5_kernel<T>), dim3(n / 64, heads, tiles < want ? tiles : want), dim3(128), smem, stream, mw, mx, (T*)y,
                (const T*)x2, tokens, n, kc, tail, ldx2, ldy, hy, status);
    TELB_CHECK_LAUNCH("head_linear_tc5_kernel");
    return 0;
}

extern "C" int telb_head_linear(const void* x, const void* w, void* y, const void* x2, int tokens, int heads, int n, int k, int tail, int ldx, int ldx2,
                                int ldy, int hy, int dtype, int* status, cudaStream_t stream) {
    if (tokens <= 0 || heads <= 0) return 0;
    if (n % 64 || k % 64 || ldx % 8) return fail("telb_head_linear: sizes must be multiples of 64 and the row pitch of 8");
    if (heads > 65535 || tokens > 65535 * 64) return fail("telb_head_linear: too many heads or rows");
    if (dtype != 2 && k <= 576 && ldx2 % 8 == 0 && ldy % 8 == 0 && hy % 8 == 0 && tail % 8 == 0)
        return dtype == 1 ? launch_head_linear_tc5<__nv_bfloat16>(x, w, y, x2, tokens, heads, n, k, tail, ldx, ldx2, ldy, hy, status, stream)
                          : launch_head_linear_tc5<__half>(x, w, y, x2, tokens, heads, n, k, tail, ldx, ldx2, ldy, hy, status, stream);
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

// dtype: 0 fp16, 1 bf16, 2 fp32.  Heads are padded to multiples of 8, row pitches likewise.
extern "C" int telb_turned_kv_write(const TurnedKvParams* pp, int dtype, cudaStream_t stream) {
    const TurnedKvParams& p = *pp;
    if (p.tokens <= 0) return 0;
    if (p.d % 8 || p.ld % 8 || p.hq < 1 || p.hkv < 1) return fail("telb_turned_kv_write: head and row sizes are multiples of 8");
    const dim3 grid(p.tokens), block(kTurnThreads);
    if (dtype == 2) TELB_LAUNCH("turned_kv_write_kernel", (turned_kv_write_kernel<float>), grid, block, 0, stream, p);
    else if (dtype == 1) TELB_LAUNCH("turned_kv_write_kernel", (turned_kv_write_kernel<__nv_bfloat16>), grid, block, 0, stream, p);
    else TELB_LAUNCH("turned_kv_write_kernel", (turned_kv_write_kernel<__half>), grid, block, 0, stream, p);
    TELB_CHECK_LAUNCH("turned_kv_write_kernel");
    return 0;
}
