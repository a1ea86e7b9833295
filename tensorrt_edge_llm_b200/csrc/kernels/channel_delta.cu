// Delta-rule mixer with one decay per head and key channel, over the packed ragged step.  Per head (S: keys x values, fp32):
//
//   q, k, v <- silu(short causal convolution)            q, k <- x / sqrt(sum x² + 1e-6), q also times dim^-1/2
//   g = exp(-exp(a_log) · softplus(decay + bias))        beta = sigmoid(beta)
//   S <- diag(g) S;  u = beta (v - Sᵀ k);  S <- S + k uᵀ;  o = Sᵀ q
//   y = o / rms(o) · w · sigmoid(gate)
//
// Prompt portions run as four launches: `prep` (convolutions, norms as one scale per row and head, decays; parallel over tokens), `walk`
// (the recurrence, state in registers), `out` (head norm and gate) and `roll` (convolution history).  A step with one row per
// sequence runs `decode`: everything fused in one launch per layer when q / k heads are not shared, behind `prep` otherwise.
//
// The walk never leaves fp32.  A head's state is cut into column slices that do not talk to each other: a warp owns 4 · CPL columns,
// eight lanes share the rows of a column and hold RPL rows x CPL columns each, as packed row pairs (fma.rn.f32x2).  Because Sᵀk with
// the decayed state equals Sᵀ(g ∘ k) with the old one, the decay of S runs beside the reduction that u waits for.
#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

// Host mirror: ops/cuda.py (ChannelDeltaParams).
struct ChannelDeltaParams {
    const void* qkv;           // [T, channels] projections: q [kv_heads * dk] | k [kv_heads * dk] | v [heads * dv]
    const float* decay;        // [T, ld_decay] pre-activations [heads * dk]
    const void* gate;          // [T, ld_gate] pre-activations [heads * dv], fp32 when gate_f32
    const float* beta;         // [T, heads] pre-activations
    const void* conv_w;        // [channels, taps]
    const float* a_log;        // [heads]
    const float* decay_bias;   // [heads * dk]
    const float* norm_w;       // [dv]
    void* conv_state;          // [slots, channels, taps - 1], oldest first
    float* state;              // [slots, heads, dk, dv]
    void* mixed;               // [T, channels] scratch: convolved q | k | v
    float* row_scale;          // [T, 2, kv_heads] scratch: 1 / |q|, 1 / |k|
    float* g;                  // [T, heads * dk] scratch: decays
    float* b;                  // [T, heads] scratch: step sizes
    void* o;                   // [T, heads * dv] scratch: read-outs
    void* out;                 // [T, heads * dv]
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* slot_ids;
    const int* seq_ids;
    int tokens, num_seqs, heads, kv_heads, dk, dv, dk_real, dv_real, taps, channels, ld_decay, ld_gate, gate_f32;
    float eps;
};

constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float cd_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float cd_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float cd_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float cd_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// N consecutive values as fp32 (N · sizeof(T) bytes aligned to their own size, at most 16 at a time).
template <typename T, int N>
__device__ __forceinline__ void load_n(const T* p, float (&v)[N]) {
    constexpr int kBytes = N * (int)sizeof(T);
    alignas(16) T e[N];
    if constexpr (kBytes >= 16) {
#pragma unroll
        for (int i = 0; i < kBytes / 16; ++i) reinterpret_cast<uint4*>(e)[i] = reinterpret_cast<const uint4*>(p)[i];
    } else if constexpr (kBytes == 8) {
        *reinterpret_cast<uint2*>(e) = *reinterpret_cast<const uint2*>(p);
    } else if constexpr (kBytes == 4) {
        *reinterpret_cast<uint32_t*>(e) = *reinterpret_cast<const uint32_t*>(p);
    } else {
        e[0] = p[0];
    }
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = Cvt<T>::to_f(e[i]);
}
template <typename T, int N>
__device__ __forceinline__ void store_n(T* p, const T (&e)[N]) {
    constexpr int kBytes = N * (int)sizeof(T);
    if constexpr (kBytes >= 16) {
#pragma unroll
        for (int i = 0; i < kBytes / 16; ++i) reinterpret_cast<uint4*>(p)[i] = reinterpret_cast<const uint4*>(e)[i];
    } else if constexpr (kBytes == 8) {
        *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(e);
    } else if constexpr (kBytes == 4) {
        *reinterpret_cast<uint32_t*>(p) = *reinterpret_cast<const uint32_t*>(e);
    } else {
        p[0] = e[0];
    }
}

// ---- prep: convolution + silu + norm scales, decays, step sizes ------------------------------------------
constexpr int kPrepTokens = 8;       // rows per warp

// One head of q, k or v over rows t0 .. t1 - 1; a lane owns C consecutive channels.  W: window size, taps <= W.
template <typename T, int C, int W>
__device__ void prep_conv(const ChannelDeltaParams& p, int ch0, int t0, int t1, float* scale, int scale_ld) {
    const int lane = threadIdx.x & 31;
    const int ch = ch0 + lane * C;
    const T* x = reinterpret_cast<const T*>(p.qkv);
    const T* cw = reinterpret_cast<const T*>(p.conv_w);
    const T* cs = reinterpret_cast<const T*>(p.conv_state);
    const int hist = p.taps - 1;
    float w[W][C], win[W][C];
#pragma unroll
    for (int j = 0; j < W; ++j)
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int tap = j - (W - p.taps);
            w[j][c] = tap >= 0 ? Cvt<T>::to_f(cw[(size_t)(ch + c) * p.taps + tap]) : 0.f;
            win[j][c] = 0.f;
        }
    int prev_seq = -1;
    for (int t = t0; t < t1; ++t) {
        const int seq = p.seq_ids[t];
        const int i = t - p.q_start[seq];
        if (seq != prev_seq) {                            // fill the window: earlier rows of the portion, then the kept history
            prev_seq = seq;
            const bool fresh = p.past_len[seq] == 0;
            const size_t slot = (size_t)p.slot_ids[seq] * p.channels;
#pragma unroll
            for (int j = 0; j < W - 1; ++j) {
                const int back = W - 1 - j, r = i - back;
#pragma unroll
                for (int c = 0; c < C; ++c) win[j + 1][c] = 0.f;
                if (back > hist) continue;
                if (r >= 0) {
                    load_n<T, C>(x + (size_t)(t - back) * p.channels + ch, win[j + 1]);
                } else if (!fresh) {
#pragma unroll
                    for (int c = 0; c < C; ++c) win[j + 1][c] = Cvt<T>::to_f(cs[(slot + ch + c) * hist + hist + r]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < W - 1; ++j)
#pragma unroll
            for (int c = 0; c < C; ++c) win[j][c] = win[j + 1][c];
        load_n<T, C>(x + (size_t)t * p.channels + ch, win[W - 1]);
        T y[C];
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < C; ++c) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < W; ++j) acc = fmaf(w[j][c], win[j][c], acc);
            y[c] = Cvt<T>::from_f(cd_silu(acc));
            const float r = Cvt<T>::to_f(y[c]);
            ss += r * r;
        }
        store_n<T, C>(reinterpret_cast<T*>(p.mixed) + (size_t)t * p.channels + ch, y);
        if (scale) {
            ss = cd_warp_sum(ss);
            if (lane == 0) scale[(size_t)t * scale_ld] = 1.f / sqrtf(ss + kUnitEps);
        }
    }
}

template <int C>
__device__ void prep_decay(const ChannelDeltaParams& p, int h, int t0, int t1) {
    const int lane = threadIdx.x & 31, col = h * p.dk + lane * C;
    const float rate = -expf(p.a_log[h]);
    float bias[C];
    load_n<float, C>(p.decay_bias + col, bias);
    for (int t = t0; t < t1; ++t) {
        float z[C];
        load_n<float, C>(p.decay + (size_t)t * p.ld_decay + col, z);
#pragma unroll
        for (int c = 0; c < C; ++c) z[c] = expf(rate * cd_softplus(z[c] + bias[c]));
        store_n<float, C>(p.g + (size_t)t * p.heads * p.dk + col, z);
        if (lane == 0) p.b[(size_t)t * p.heads + h] = cd_sigmoid(p.beta[(size_t)t * p.heads + h]);
    }
}

#define TELB_BY_LANES(dim, CALL)        \
    switch ((dim) >> 5) {               \
        case 1: { constexpr int C = 1; CALL; break; } \
        case 2: { constexpr int C = 2; CALL; break; } \
        case 4: { constexpr int C = 4; CALL; break; } \
        default: { constexpr int C = 8; CALL; break; } \
    }

template <typename T, int W>
__global__ void __launch_bounds__(128) channel_delta_prep_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_prologue();
    const int unit = blockIdx.y;                          // q heads, k heads, v heads, decays
    const int t0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * kPrepTokens;
    if (t0 >= p.tokens) return;
    const int t1 = min(p.tokens, t0 + kPrepTokens);
    const int nk = p.kv_heads;
    if (unit < 2 * nk) {
        TELB_BY_LANES(p.dk, (prep_conv<T, C, W>(p, unit * p.dk, t0, t1, p.row_scale + unit, 2 * nk)))
    } else if (unit < 2 * nk + p.heads) {
        TELB_BY_LANES(p.dv, (prep_conv<T, C, W>(p, 2 * nk * p.dk + (unit - 2 * nk) * p.dv, t0, t1, nullptr, 0)))
    } else {
        TELB_BY_LANES(p.dk, (prep_decay<C>(p, unit - 2 * nk - p.heads, t0, t1)))
    }
}

// History of the convolutions after a portion: the last taps - 1 inputs.
template <typename T>
__global__ void __launch_bounds__(128) channel_delta_roll_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_prologue();
    const int seq = blockIdx.y, ch = blockIdx.x * 128 + threadIdx.x;
    const int ql = p.q_len[seq], hist = p.taps - 1;
    if (ch >= p.channels || ql <= 0) return;
    const T* x = reinterpret_cast<const T*>(p.qkv) + (size_t)p.q_start[seq] * p.channels + ch;
    T* cs = reinterpret_cast<T*>(p.conv_state) + ((size_t)p.slot_ids[seq] * p.channels + ch) * hist;
    const bool fresh = p.past_len[seq] == 0;
    for (int j = 0; j < hist; ++j) {                      // ascending: an old value is read before its place is written
        const int r = ql - hist + j;
        cs[j] = r >= 0 ? x[(size_t)r * p.channels] : (fresh ? Cvt<T>::from_f(0.f) : cs[j + ql]);
    }
}

// ---- walk ------------------------------------------------------------------------------------------------
typedef unsigned long long f2;                            // two fp32 values in one register pair
__device__ __forceinline__ f2 f2_pack(float a, float b) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float f2_sum(f2 v) {
    float a, b;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
    return a + b;
}
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async8(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Rows of lane group rl (of 8): blocks of BL = min(8, RPL) rows, block j at rows j · 8 BL + rl · BL.
template <int RPL>
struct WalkRows {
    static constexpr int BL = RPL < 8 ? RPL : 8;
    static __device__ __forceinline__ int row(int rl, int i) { return (i / BL) * (8 * BL) + rl * BL + i % BL; }
    // shared-memory place of fp32 granule m (rows 4 m .. 4 m + 3): granules that the eight groups read together lie side by side
    static __device__ __forceinline__ int granule(int m) { return BL == 8 ? ((m >> 4) * 2 + (m & 1)) * 8 + ((m & 15) >> 1) : m; }
};

template <typename T, int RPL>
__device__ __forceinline__ void walk_load(const T* s, int rl, f2 (&v)[RPL / 2]) {
    constexpr int BL = WalkRows<RPL>::BL;
#pragma unroll
    for (int j = 0; j < RPL / BL; ++j) {
        if constexpr (sizeof(T) == 4) {
#pragma unroll
            for (int h = 0; h < BL / 4; ++h) {
                const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(s + ((j * (BL / 4) + h) * 8 + rl) * 4);
                v[j * BL / 2 + h * 2] = u.x;
                v[j * BL / 2 + h * 2 + 1] = u.y;
            }
        } else {
            uint32_t u[BL / 2];
            if constexpr (BL == 8) *reinterpret_cast<uint4*>(u) = *reinterpret_cast<const uint4*>(s + j * 64 + rl * 8);
            else *reinterpret_cast<uint2*>(u) = *reinterpret_cast<const uint2*>(s + j * 32 + rl * 4);
#pragma unroll
            for (int i = 0; i < BL / 2; ++i) {
                if constexpr (std::is_same<T, __nv_bfloat16>::value) {
                    v[j * BL / 2 + i] = f2_pack(__uint_as_float(u[i] << 16), __uint_as_float(u[i] & 0xffff0000u));
                } else {
                    const float2 f = __half22float2(*reinterpret_cast<const __half2*>(&u[i]));
                    v[j * BL / 2 + i] = f2_pack(f.x, f.y);
                }
            }
        }
    }
}

// Sums of C column values over the eight lanes of a group; a lane receives the sum of column walk_col<C>(rl).
template <int C>
__device__ __forceinline__ int walk_col(int rl) { return C == 4 ? rl >> 1 : C == 2 ? rl >> 2 : 0; }
template <int C>
__device__ __forceinline__ float walk_reduce(float (&a)[C], int rl) {
    constexpr unsigned kAll = 0xffffffffu;
    if constexpr (C == 4) {
        const bool hi = rl & 4;
        const float s0 = __shfl_xor_sync(kAll, hi ? a[0] : a[2], 4), s1 = __shfl_xor_sync(kAll, hi ? a[1] : a[3], 4);
        const float b0 = (hi ? a[2] : a[0]) + s0, b1 = (hi ? a[3] : a[1]) + s1;
        const bool h2 = rl & 2;
        float v = (h2 ? b1 : b0) + __shfl_xor_sync(kAll, h2 ? b0 : b1, 2);
        return v + __shfl_xor_sync(kAll, v, 1);
    } else if constexpr (C == 2) {
        const bool hi = rl & 4;
        float v = (hi ? a[1] : a[0]) + __shfl_xor_sync(kAll, hi ? a[0] : a[1], 4);
        v += __shfl_xor_sync(kAll, v, 2);
        return v + __shfl_xor_sync(kAll, v, 1);
    } else {
        float v = a[0];
        v += __shfl_xor_sync(kAll, v, 4);
        v += __shfl_xor_sync(kAll, v, 2);
        return v + __shfl_xor_sync(kAll, v, 1);
    }
}

constexpr int kWalkTokens = 8;       // rows per stage
constexpr int kWalkStages = 3;

template <typename T>
__host__ __device__ inline int walk_row_bytes(int dk, int cols) { return dk * (2 * (int)sizeof(T) + 4) + ((cols * (int)sizeof(T) + 15) & ~15) + 16; }

// grid (column slices of a head, heads, sequences); blockDim = warps of one slice
template <typename T, int RPL, int CPL>
__global__ void __launch_bounds__(128) channel_delta_walk_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_prologue();
    constexpr int DK = RPL * 8;
    extern __shared__ __align__(16) uint8_t walk_smem[];
    const int seq = blockIdx.z, h = blockIdx.y;
    const int ql = p.q_len[seq];
    if (ql <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthr = blockDim.x;
    const int rl = lane & 7, cg = lane >> 3;
    const int cols = (nthr >> 5) * 4 * CPL;               // columns of this CTA
    const int col0 = blockIdx.x * cols;                   // within the head
    const int lcol = warp * 4 * CPL + cg * CPL;           // first column of this lane, within the CTA
    const int hk = h / (p.heads / p.kv_heads);
    const size_t r0 = p.q_start[seq];
    const int row_bytes = walk_row_bytes<T>(DK, cols), stage_bytes = row_bytes * kWalkTokens;
    const T* mixed = reinterpret_cast<const T*>(p.mixed);

    auto fetch = [&](int chunk) {
        const int first = chunk * kWalkTokens, n = min(kWalkTokens, ql - first);
        uint8_t* st = walk_smem + (chunk % kWalkStages) * stage_bytes;
        constexpr int kQ = DK * (int)sizeof(T) / 16, kG = DK / 4;
        const int kV = cols * (int)sizeof(T) / 8;
        const int per = 2 * kQ + kG + kV + 3;
        for (int idx = tid; idx < n * per; idx += nthr) {
            const int i = idx / per;
            int e = idx - i * per;
            uint8_t* row = st + i * row_bytes;
            const size_t t = r0 + first + i;
            const T* m = mixed + t * p.channels;
            if (e < 2 * kQ) {
                const int qk = e >= kQ;
                e -= qk * kQ;
                const int dst = sizeof(T) == 4 ? WalkRows<RPL>::granule(e) : e;
                cp_async16(row + qk * DK * (int)sizeof(T) + dst * 16, reinterpret_cast<const uint8_t*>(m + (qk * p.kv_heads + hk) * DK) + e * 16);
            } else if (e < 2 * kQ + kG) {
                e -= 2 * kQ;
                cp_async16(row + 2 * DK * (int)sizeof(T) + WalkRows<RPL>::granule(e) * 16, p.g + (t * p.heads + h) * DK + e * 4);
            } else if (e < 2 * kQ + kG + kV) {
                e -= 2 * kQ + kG;
                cp_async8(row + DK * (2 * (int)sizeof(T) + 4) + 16 + e * 8,
                          reinterpret_cast<const uint8_t*>(m + 2 * p.kv_heads * DK + h * p.dv + col0) + e * 8);
            } else {
                e -= 2 * kQ + kG + kV;
                const float* src = e == 2 ? p.b + t * p.heads + h : p.row_scale + t * 2 * p.kv_heads + e * p.kv_heads + hk;
                cp_async4(row + DK * (2 * (int)sizeof(T) + 4) + e * 4, src);
            }
        }
    };

    f2 S[RPL / 2][CPL];
    float* state = p.state + (((size_t)p.slot_ids[seq] * p.heads + h) * DK) * p.dv + col0 + lcol;
    if (p.past_len[seq] > 0) {
#pragma unroll
        for (int i = 0; i < RPL / 2; ++i) {
            float a[CPL], b[CPL];
            load_n<float, CPL>(state + (size_t)WalkRows<RPL>::row(rl, 2 * i) * p.dv, a);
            load_n<float, CPL>(state + (size_t)WalkRows<RPL>::row(rl, 2 * i + 1) * p.dv, b);
#pragma unroll
            for (int c = 0; c < CPL; ++c) S[i][c] = f2_pack(a[c], b[c]);
        }
    } else {
#pragma unroll
        for (int i = 0; i < RPL / 2; ++i)
#pragma unroll
            for (int c = 0; c < CPL; ++c) S[i][c] = 0ull;
    }

    const int chunks = (ql + kWalkTokens - 1) / kWalkTokens;
#pragma unroll
    for (int s = 0; s < kWalkStages - 1; ++s) {
        if (s < chunks) fetch(s);
        cp_async_commit();
    }
    const float q_scale = rsqrtf((float)p.dk_real);
    const int my_col = walk_col<CPL>(rl);
    const bool writer = CPL == 4 ? !(rl & 1) : CPL == 2 ? !(rl & 3) : rl == 0;
    T* out = reinterpret_cast<T*>(p.o) + r0 * p.heads * p.dv + (size_t)h * p.dv + col0 + lcol + my_col;
    for (int ch = 0; ch < chunks; ++ch) {
        cp_async_wait<kWalkStages - 2>();
        __syncthreads();
        if (ch + kWalkStages - 1 < chunks) fetch(ch + kWalkStages - 1);
        cp_async_commit();
        const uint8_t* st = walk_smem + (ch % kWalkStages) * stage_bytes;
        const int n = min(kWalkTokens, ql - ch * kWalkTokens);
        for (int i = 0; i < n; ++i) {
            const uint8_t* row = st + i * row_bytes;
            const float* sc = reinterpret_cast<const float*>(row + DK * (2 * (int)sizeof(T) + 4));
            f2 k[RPL / 2], g[RPL / 2];
            walk_load<T, RPL>(reinterpret_cast<const T*>(row) + DK, rl, k);
            walk_load<float, RPL>(reinterpret_cast<const float*>(row + 2 * DK * (int)sizeof(T)), rl, g);
            const float v = Cvt<T>::to_f(reinterpret_cast<const T*>(sc + 4)[lcol + my_col]);
            const float sk = sc[1], beta = sc[2];
            f2 acc[CPL];
            float a[CPL];
#pragma unroll
            for (int c = 0; c < CPL; ++c) acc[c] = 0ull;
#pragma unroll
            for (int r = 0; r < RPL / 2; ++r) {
                const f2 kg = f2_mul(k[r], g[r]);
#pragma unroll
                for (int c = 0; c < CPL; ++c) acc[c] = f2_fma(S[r][c], kg, acc[c]);
            }
#pragma unroll
            for (int c = 0; c < CPL; ++c) a[c] = f2_sum(acc[c]);
            const float sum = walk_reduce<CPL>(a, rl);
#pragma unroll
            for (int r = 0; r < RPL / 2; ++r)
#pragma unroll
                for (int c = 0; c < CPL; ++c) S[r][c] = f2_mul(S[r][c], g[r]);
            const float us = beta * (v - sk * sum) * sk;          // u times the norm scale of k
            f2 q[RPL / 2];
            walk_load<T, RPL>(reinterpret_cast<const T*>(row), rl, q);
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
                const float uc = __shfl_sync(0xffffffffu, us, (lane & 24) | (CPL == 4 ? c * 2 : CPL == 2 ? c * 4 : 0));
                const f2 u2 = f2_pack(uc, uc);
                acc[c] = 0ull;
#pragma unroll
                for (int r = 0; r < RPL / 2; ++r) {
                    S[r][c] = f2_fma(k[r], u2, S[r][c]);
                    acc[c] = f2_fma(S[r][c], q[r], acc[c]);
                }
            }
#pragma unroll
            for (int c = 0; c < CPL; ++c) a[c] = f2_sum(acc[c]);
            const float o = walk_reduce<CPL>(a, rl) * sc[0] * q_scale;
            if (writer) out[(size_t)(ch * kWalkTokens + i) * p.heads * p.dv] = Cvt<T>::from_f(o);
        }
    }
#pragma unroll
    for (int i = 0; i < RPL / 2; ++i) {
        float a[CPL], b[CPL];
#pragma unroll
        for (int c = 0; c < CPL; ++c) asm("mov.b64 {%0, %1}, %2;" : "=f"(a[c]), "=f"(b[c]) : "l"(S[i][c]));
        store_n<float, CPL>(state + (size_t)WalkRows<RPL>::row(rl, 2 * i) * p.dv, a);
        store_n<float, CPL>(state + (size_t)WalkRows<RPL>::row(rl, 2 * i + 1) * p.dv, b);
    }
}

// ---- out: head norm and gate, one warp per (row, head) ---------------------------------------------------
template <typename T, int C>
__device__ void delta_out(const ChannelDeltaParams& p, size_t t, int h) {
    const int lane = threadIdx.x & 31, col = h * p.dv + lane * C;
    float o[C], w[C], z[C];
    load_n<T, C>(reinterpret_cast<const T*>(p.o) + t * p.heads * p.dv + col, o);
    load_n<float, C>(p.norm_w + lane * C, w);
    if (p.gate_f32) load_n<float, C>(reinterpret_cast<const float*>(p.gate) + t * p.ld_gate + col, z);
    else load_n<T, C>(reinterpret_cast<const T*>(p.gate) + t * p.ld_gate + col, z);
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < C; ++c) ss += o[c] * o[c];
    const float inv = 1.f / sqrtf(cd_warp_sum(ss) / p.dv_real + p.eps);
    T y[C];
#pragma unroll
    for (int c = 0; c < C; ++c) y[c] = Cvt<T>::from_f(o[c] * inv * w[c] * cd_sigmoid(z[c]));
    store_n<T, C>(reinterpret_cast<T*>(p.out) + t * p.heads * p.dv + col, y);
}

template <typename T>
__global__ void __launch_bounds__(128) channel_delta_out_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_prologue();
    const long long wid = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (wid >= (long long)p.tokens * p.heads) return;
    const size_t t = wid / p.heads;
    const int h = (int)(wid - (long long)t * p.heads);
    TELB_BY_LANES(p.dv, (delta_out<T, C>(p, t, h)))
}

// ---- decode: one row per sequence, everything in one CTA per (head, sequence) -----------------------------
// Eight warps share the rows of S; a lane owns DV / 32 columns of its warp's DK / 8 rows, in registers from load to store.
// FUSED: q, k, v are convolved here (their heads are not shared); otherwise `prep` has run.
template <typename T, int DK, int DV, bool FUSED>
__global__ void __launch_bounds__(256) channel_delta_decode_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_prologue();
    constexpr int R = DK / 8, C = DV / 32;
    __shared__ float s_q[DK], s_k[DK], s_g[DK], s_v[DV], s_u[DV], s_a[8][DV], s_b[8][DV], s_red[8];
    const int seq = blockIdx.y, h = blockIdx.x;
    if (p.q_len[seq] <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const size_t t = p.q_start[seq], slot = p.slot_ids[seq];
    const bool fresh = p.past_len[seq] == 0;
    const int group = p.heads / p.kv_heads, hk = h / group, hist = p.taps - 1;
    float S[R][C];
    float* state = p.state + (((slot * p.heads + h) * DK) + warp * R) * DV + lane * C;
    if (!fresh) {
#pragma unroll
        for (int r = 0; r < R; ++r) load_n<float, C>(state + r * DV, S[r]);
    } else {
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int c = 0; c < C; ++c) S[r][c] = 0.f;
    }
    const T* x = reinterpret_cast<const T*>(FUSED ? p.qkv : p.mixed) + t * p.channels;
    const T* raw = reinterpret_cast<const T*>(p.qkv) + t * p.channels;
    for (int i = tid; i < 2 * DK + DV; i += 256) {
        const int ch = i < DK ? hk * DK + i : i < 2 * DK ? p.kv_heads * DK + hk * DK + i - DK : 2 * p.kv_heads * DK + h * DV + i - 2 * DK;
        T* cs = reinterpret_cast<T*>(p.conv_state) + (slot * p.channels + ch) * hist;
        float y = Cvt<T>::to_f(x[ch]);
        if constexpr (FUSED) {
            const T* cw = reinterpret_cast<const T*>(p.conv_w) + (size_t)ch * p.taps;
            float acc = 0.f;
            if (!fresh)
                for (int j = 0; j < hist; ++j) acc = fmaf(Cvt<T>::to_f(cw[j]), Cvt<T>::to_f(cs[j]), acc);
            acc = fmaf(Cvt<T>::to_f(cw[hist]), y, acc);
            y = Cvt<T>::to_f(Cvt<T>::from_f(cd_silu(acc)));
        }
        if (hist > 0 && (i >= 2 * DK || h % group == 0)) {             // this CTA keeps the history of the channel
            for (int j = 0; j + 1 < hist; ++j) cs[j] = fresh ? Cvt<T>::from_f(0.f) : cs[j + 1];
            cs[hist - 1] = raw[ch];
        }
        (i < DK ? s_q[i] : i < 2 * DK ? s_k[i - DK] : s_v[i - 2 * DK]) = y;
    }
    float beta;
    if constexpr (FUSED) {
        const float rate = -expf(p.a_log[h]);
        for (int i = tid; i < DK; i += 256) s_g[i] = expf(rate * cd_softplus(p.decay[t * p.ld_decay + h * DK + i] + p.decay_bias[h * DK + i]));
        beta = cd_sigmoid(p.beta[t * p.heads + h]);
    } else {
        for (int i = tid; i < DK; i += 256) s_g[i] = p.g[(t * p.heads + h) * DK + i];
        beta = p.b[t * p.heads + h];
    }
    __syncthreads();
    float qq = 0.f, kk = 0.f, qk = 0.f;                                 // every warp: |q|², |k|², q·k
    for (int i = lane; i < DK; i += 32) {
        const float a = s_q[i], b = s_k[i];
        qq = fmaf(a, a, qq);
        kk = fmaf(b, b, kk);
        qk = fmaf(a, b, qk);
    }
    qq = cd_warp_sum(qq);
    kk = cd_warp_sum(kk);
    qk = cd_warp_sum(qk);
    const float sk = 1.f / sqrtf(kk + kUnitEps), sq = 1.f / sqrtf(qq + kUnitEps) * rsqrtf((float)p.dk_real);
    float a[C], b[C];
#pragma unroll
    for (int c = 0; c < C; ++c) a[c] = b[c] = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = warp * R + r;
        const float g = s_g[row], kr = s_k[row], qr = s_q[row];
#pragma unroll
        for (int c = 0; c < C; ++c) {
            S[r][c] *= g;
            a[c] = fmaf(S[r][c], kr, a[c]);
            b[c] = fmaf(S[r][c], qr, b[c]);
        }
    }
#pragma unroll
    for (int c = 0; c < C; ++c) {
        s_a[warp][lane * C + c] = a[c];
        s_b[warp][lane * C + c] = b[c];
    }
    __syncthreads();
    float o = 0.f;
    if (tid < DV) {
        float sa = 0.f, sb = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            sa += s_a[w][tid];
            sb += s_b[w][tid];
        }
        const float us = beta * (s_v[tid] - sk * sa) * sk;
        s_u[tid] = us;
        o = sq * fmaf(us, qk, sb);                                      // (S + k uᵀ)ᵀ q without a second pass over S
    }
    const float ss = cd_warp_sum(o * o);
    if (lane == 0) s_red[warp] = ss;
    __syncthreads();
    float u[C];
#pragma unroll
    for (int c = 0; c < C; ++c) u[c] = s_u[lane * C + c];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const float kr = s_k[warp * R + r];
#pragma unroll
        for (int c = 0; c < C; ++c) S[r][c] = fmaf(kr, u[c], S[r][c]);
        store_n<float, C>(state + r * DV, S[r]);
    }
    if (tid < DV) {
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < (DV + 31) / 32; ++w) tot += s_red[w];
        const float inv = 1.f / sqrtf(tot / p.dv_real + p.eps);
        const size_t gi = t * p.ld_gate + h * DV + tid;
        const float z = p.gate_f32 ? reinterpret_cast<const float*>(p.gate)[gi] : Cvt<T>::to_f(reinterpret_cast<const T*>(p.gate)[gi]);
        reinterpret_cast<T*>(p.out)[(t * p.heads + h) * DV + tid] = Cvt<T>::from_f(o * inv * p.norm_w[tid] * cd_sigmoid(z));
    }
}

// ---- launchers ---------------------------------------------------------------------------------------------
template <typename T>
static int launch_prep(const ChannelDeltaParams& p, cudaStream_t stream) {
    const int warps = (p.tokens + kPrepTokens - 1) / kPrepTokens;
    const dim3 grid((warps + 3) / 4, 2 * p.kv_heads + 2 * p.heads);
    if (p.taps <= 4) TELB_LAUNCH("channel_delta_prep_kernel", (channel_delta_prep_kernel<T, 4>), grid, dim3(128), 0, stream, p);
    else TELB_LAUNCH("channel_delta_prep_kernel", (channel_delta_prep_kernel<T, 8>), grid, dim3(128), 0, stream, p);
    TELB_CHECK_LAUNCH("channel_delta_prep_kernel");
    return 0;
}

template <typename T, int RPL, int CPL>
static int launch_walk_as(const ChannelDeltaParams& p, int warps, cudaStream_t stream) {
    while (warps > 1 && p.dv % (warps * 4 * CPL)) warps >>= 1;
    const int cols = warps * 4 * CPL;
    const size_t smem = (size_t)walk_row_bytes<T>(RPL * 8, cols) * kWalkTokens * kWalkStages;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(channel_delta_walk_kernel<T, RPL, CPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(channel_delta_walk)", e);
    }
    TELB_LAUNCH("channel_delta_walk_kernel", (channel_delta_walk_kernel<T, RPL, CPL>), dim3(p.dv / cols, p.heads, p.num_seqs), dim3(warps * 32), smem,
                stream, p);
    TELB_CHECK_LAUNCH("channel_delta_walk_kernel");
    return 0;
}

template <typename T, int RPL>
static int launch_walk(const ChannelDeltaParams& p, cudaStream_t stream) {
    // few (sequence, head) pairs: narrow slices, one warp each, so that every scheduler has a chain of its own
    const long long columns = (long long)p.num_seqs * p.heads * p.dv;
    if (columns / 4 <= 4LL * sm_count()) return launch_walk_as<T, RPL, 1>(p, 1, stream);
    if (RPL > 16 || columns / 8 <= 4LL * sm_count()) return launch_walk_as<T, RPL, 2>(p, columns / 8 <= 4LL * sm_count() ? 1 : 4, stream);
    return launch_walk_as<T, RPL, (RPL > 16 ? 2 : 4)>(p, columns / 16 <= 4LL * sm_count() ? 1 : 2, stream);
}

template <typename T>
static int channel_delta_rows(const ChannelDeltaParams& p, cudaStream_t stream) {
    if (launch_prep<T>(p, stream)) return -1;
    int rc = 0;
    switch (p.dk) {
        case 32: rc = launch_walk<T, 4>(p, stream); break;
        case 64: rc = launch_walk<T, 8>(p, stream); break;
        case 128: rc = launch_walk<T, 16>(p, stream); break;
        default: rc = launch_walk<T, 32>(p, stream); break;
    }
    if (rc) return rc;
    const long long warps = (long long)p.tokens * p.heads;
    TELB_LAUNCH("channel_delta_out_kernel", (channel_delta_out_kernel<T>), dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, stream, p);
    TELB_CHECK_LAUNCH("channel_delta_out_kernel");
    if (p.taps > 1) {
        TELB_LAUNCH("channel_delta_roll_kernel", (channel_delta_roll_kernel<T>), dim3((p.channels + 127) / 128, p.num_seqs), dim3(128), 0, stream, p);
        TELB_CHECK_LAUNCH("channel_delta_roll_kernel");
    }
    return 0;
}

template <typename T, int DK, int DV>
static int launch_decode_step(const ChannelDeltaParams& p, cudaStream_t stream) {
    const dim3 grid(p.heads, p.num_seqs);
    if (p.heads == p.kv_heads) {
        TELB_LAUNCH("channel_delta_decode_kernel", (channel_delta_decode_kernel<T, DK, DV, true>), grid, dim3(256), 0, stream, p);
    } else {
        if (launch_prep<T>(p, stream)) return -1;
        TELB_LAUNCH("channel_delta_decode_kernel", (channel_delta_decode_kernel<T, DK, DV, false>), grid, dim3(256), 0, stream, p);
    }
    TELB_CHECK_LAUNCH("channel_delta_decode_kernel");
    return 0;
}

template <typename T, int DK>
static int decode_by_dv(const ChannelDeltaParams& p, cudaStream_t stream) {
    if (p.dv == 32) return launch_decode_step<T, DK, 32>(p, stream);
    if (p.dv == 64) return launch_decode_step<T, DK, 64>(p, stream);
    return launch_decode_step<T, DK, 128>(p, stream);
}

template <typename T>
static int channel_delta_step(const ChannelDeltaParams& p, cudaStream_t stream) {
    if (p.dk == 32) return decode_by_dv<T, 32>(p, stream);
    if (p.dk == 64) return decode_by_dv<T, 64>(p, stream);
    return decode_by_dv<T, 128>(p, stream);
}

}  // namespace telb

using namespace telb;

// dtype: 0 fp16, 1 bf16, 2 fp32 (of qkv, conv_w, conv_state, mixed, o, out and, unless gate_f32, gate).
// decode != 0: every sequence has at most one row and dk, dv <= 128.
extern "C" int telb_channel_delta(const ChannelDeltaParams* pp, int decode, int dtype, cudaStream_t stream) {
    const ChannelDeltaParams& p = *pp;
    if (p.tokens <= 0 || p.num_seqs <= 0) return 0;
    auto size_ok = [](int d) { return d == 32 || d == 64 || d == 128 || d == 256; };
    if (!size_ok(p.dk) || !size_ok(p.dv)) return fail("telb_channel_delta: padded head sizes are 32, 64, 128 or 256");
    if (p.taps < 1 || p.taps > 8) return fail("telb_channel_delta: convolutions have 1 to 8 taps");
    if (p.kv_heads <= 0 || p.heads % p.kv_heads) return fail("telb_channel_delta: heads must be a multiple of the q / k heads");
    if (p.num_seqs > 65535 || p.heads > 65535 / 4) return fail("telb_channel_delta: too many sequences or heads");
    if (decode) {
        if (p.dk > 128 || p.dv > 128) return fail("telb_channel_delta: the decode step covers heads up to 128");
        if (dtype == 2) return channel_delta_step<float>(p, stream);
        return dtype == 1 ? channel_delta_step<__nv_bfloat16>(p, stream) : channel_delta_step<__half>(p, stream);
    }
    if (dtype == 2) return channel_delta_rows<float>(p, stream);
    return dtype == 1 ? channel_delta_rows<__nv_bfloat16>(p, stream) : channel_delta_rows<__half>(p, stream);
}
