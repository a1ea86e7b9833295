// Delta-rule mixer with one decay per head and key channel (or one per head), over the packed ragged step.  Per head (S: keys x values, fp32):
//
//   q, k, v <- silu(short causal convolution)            q, k <- x / sqrt(sum x² + 1e-6), q also times dim^-1/2
//   g = exp(-exp(a_log) · softplus(decay + bias))        beta = sigmoid(beta)
//   S <- diag(g) S;  u = beta (v - Sᵀ k);  S <- S + k uᵀ;  o = Sᵀ q
//   y = o / rms(o) · w · sigmoid(gate)                   (or silu(gate))
//
// Prompt portions run as five launches: `prep` twice (values; q, k and decays: convolutions and norms, parallel over tokens), `walk` (the
// recurrence, state in registers), `out` (head norm and gate) and `roll` (convolution history).  A step with one row per sequence runs
// `decode`, everything in one launch (`roll` behind it when several heads share a q / k head).
//
// The walk takes four tokens at a time and never leaves fp32.  With S the state before a block, D_i = g_1 ∘ .. ∘ g_i and k, q normalised,
//
//   u_i = beta_i (v_i - Sᵀ(D_i ∘ k_i) - Σ_{j<i} m_ij u_j)        m_ij = Σ_c k_i k_j g_{j+1} .. g_i
//   o_i = Sᵀ(D_i ∘ q_i) + Σ_{j<=i} n_ij u_j                      n_ij = Σ_c q_i k_j g_{j+1} .. g_i
//   S  <- D_4 ∘ S + Σ_j (g_{j+1} .. g_4 ∘ k_j) u_jᵀ
//
// so the eight products with S do not wait for one another, and one reduction over lanes serves four tokens.  `prep` writes the three
// vectors per token, D_4 and the scalars, computed from products of decays only (no quotients).  With one decay per head the products leave
// the vectors: a block then is k_1 .. k_4, q_1 .. q_4 and scalars (D_i joins the products with S, g_{j+1} .. g_4 the steps u_j).  A head's state is cut into column slices that
// do not talk to each other: a warp owns 4 · CPL columns, eight lanes share the rows of a column and hold RPL rows x CPL columns each,
// as packed row pairs (fma.rn.f32x2).
#include <type_traits>

#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

// Host mirror: ops/cuda.py (ChannelDeltaParams).
struct ChannelDeltaParams {
    const void* qkv;           // [T, ld_qkv] projections: q [kv_heads * dk] | k [kv_heads * dk] | v [heads * dv]
    const float* decay;        // [T, ld_decay] pre-activations [heads * dk] (head_decay: [heads])
    const void* gate;          // [T, ld_gate] pre-activations [heads * dv], fp32 when gate_f32
    const float* beta;         // [T, ld_beta] pre-activations [heads]
    const void* conv_w;        // [channels, taps]
    const float* a_log;        // [heads]
    const float* decay_bias;   // [heads * dk]
    const float* norm_w;       // [dv]
    void* conv_state;          // [slots, channels, taps - 1], oldest first
    float* state;              // [slots, heads, dk, dv]
    float* blocks;             // [blocks, heads, 13 dk + 32] scratch (8 dk + 32 with head_decay): per block of four tokens the vectors and scalars of the walk
    void* v_blocks;            // [blocks, heads, dv, 4] scratch: convolved values
    void* o;                   // [T, heads * dv] scratch: read-outs
    void* out;                 // [T, ld_out]: heads * dv
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* slot_ids;
    const int* seq_ids;
    int* status;
    int tokens, num_seqs, heads, kv_heads, dk, dv, dk_real, dv_real, taps, channels, ld_decay, ld_gate, gate_f32;
    int ld_qkv, ld_beta, ld_out, head_decay, gate_silu;      // head_decay: decay [T, heads] and decay_bias [heads]; gate_silu: silu instead of a sigmoid
    float eps, mult;             // mult: factor of the outputs
};

constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float cd_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float cd_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float cd_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// Activations of 16-bit models use the hardware's exponential; their results are rounded to 16 bits, and the decays keep fp32 accuracy:
// the logarithm of 1 + e carries an absolute error of about 1e-7, no more than the rounding of the decay itself.
template <typename T>
__device__ __forceinline__ float cd_silu_as(float x) {
    if constexpr (sizeof(T) == 4) return cd_silu(x);
    else return __fdividef(x, 1.f + __expf(-x));
}
template <typename T>
__device__ __forceinline__ float cd_decay_as(float rate, float z) {
    if constexpr (sizeof(T) == 4) return expf(rate * cd_softplus(z));
    else return __expf(rate * (fmaxf(z, 0.f) + __logf(1.f + __expf(-fabsf(z)))));
}
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

// ---- prep ------------------------------------------------------------------------------------------------
constexpr int kBlk = 4;              // tokens of a block
constexpr int kPrepTokens = 16;      // rows whose blocks a warp takes
constexpr int kScalars = 32;         // m_21 m_31 m_32 m_41 m_42 m_43 | n_11 n_21 n_22 n_31 .. n_44 | beta_1 .. beta_4 | head decays: D_1 .. D_4 |
                                     // head decays: g_{j+1} .. g_4 for j = 1 .. 4; padded

// vectors of a block: D_i k_i, D_i q_i, k_j times the decays behind it, D_4; or k_i, q_i
template <bool HEAD>
struct BlockVectors {
    static constexpr int value = HEAD ? 8 : 13;
};
// First block of a sequence: blocks count from the start of its portion, and those of different sequences never meet.
__device__ __forceinline__ int first_block(int q_start, int seq) { return q_start / kBlk + seq; }

// fp32 granule m (rows 4 m .. 4 m + 3 of a head) in the order of the walk's lanes: granules that its eight row groups read together lie
// side by side.
__device__ __forceinline__ int walk_granule(int dk, int m) { return dk >= 64 ? ((m >> 4) * 2 + (m & 1)) * 8 + ((m & 15) >> 1) : m; }

// Taps of C channels from ch on, right-aligned in a window of W (taps <= W).
template <typename T, int C, int W>
__device__ __forceinline__ void load_taps(const ChannelDeltaParams& p, int ch, float (&w)[W][C]) {
    const T* cw = reinterpret_cast<const T*>(p.conv_w) + (size_t)ch * p.taps;
    if (p.taps == W) {                                    // C x W values in a row
        float all[C * W];
        load_n<T, C * W>(cw, all);
#pragma unroll
        for (int j = 0; j < W; ++j)
#pragma unroll
            for (int c = 0; c < C; ++c) w[j][c] = all[c * W + j];
        return;
    }
#pragma unroll
    for (int j = 0; j < W; ++j)
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int tap = j - (W - p.taps);
            w[j][c] = tap >= 0 ? Cvt<T>::to_f(cw[(size_t)c * p.taps + tap]) : 0.f;
        }
}

// Convolved and rounded rows i .. i + n - 1 of C channels from ch on (zero behind them).
template <typename T, int C, int W>
__device__ __forceinline__ void conv_block(const ChannelDeltaParams& p, const float (&w)[W][C], int ch, size_t t, int i, int n, const T* history, float (&y)[kBlk][C]) {
    const T* x = reinterpret_cast<const T*>(p.qkv) + ch;
    const int hist = p.taps - 1;
    float rows[W - 1 + kBlk][C];
    if (n == kBlk && i >= W - 1) {                        // inside the portion
#pragma unroll
        for (int j = 0; j < W - 1 + kBlk; ++j) load_n<T, C>(x + (t + j - (W - 1)) * p.ld_qkv, rows[j]);
    } else {
#pragma unroll
        for (int j = 0; j < W - 1 + kBlk; ++j) {
            const int d = j - (W - 1);                    // row relative to the block's first
#pragma unroll
            for (int c = 0; c < C; ++c) rows[j][c] = 0.f;
            if (d < n && i + d >= 0 && d >= -hist) {
                load_n<T, C>(x + (t + d) * p.ld_qkv, rows[j]);
            } else if (d < 0 && d >= -hist && history) {
#pragma unroll
                for (int c = 0; c < C; ++c) rows[j][c] = Cvt<T>::to_f(history[(size_t)(ch + c) * hist + hist + i + d]);
            }
        }
    }
#pragma unroll
    for (int b = 0; b < kBlk; ++b)
#pragma unroll
        for (int c = 0; c < C; ++c) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < W; ++j) acc = fmaf(w[j][c], rows[b + j][c], acc);
            y[b][c] = b < n ? Cvt<T>::to_f(Cvt<T>::from_f(cd_silu_as<T>(acc))) : 0.f;
        }
}

// Totals of 32 values over the warp; lane l receives that of value l.
__device__ __forceinline__ float total_of_lane(float (&v)[32], int lane) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool hi = lane & o;
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const float give = hi ? v[i] : v[i + o];
            v[i] = (hi ? v[i + o] : v[i]) + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
    return v[0];
}

// q, k and decays of one head and block; HEAD: one decay per head.
template <typename T, int C, int W, bool HEAD>
__device__ __forceinline__ void prep_head(const ChannelDeltaParams& p, const float (&wq)[W][C], const float (&wk)[W][C], const float (&bias)[C], float rate, int h,
                                          int seq, size_t t, int i, int n, const T* history) {
    constexpr int V = C < 4 ? C : 4;
    const int lane = threadIdx.x & 31, dk = p.dk, hk = h / (p.heads / p.kv_heads);
    float q[kBlk][C], k[kBlk][C], g[kBlk][C];
#pragma unroll
    for (int b = 0; b < kBlk; ++b) {
        if (b >= n) continue;
        if constexpr (HEAD) g[b][0] = p.decay[(t + b) * p.ld_decay + h];
        else load_n<float, C>(p.decay + (t + b) * p.ld_decay + h * dk + lane * C, g[b]);
    }
    conv_block<T, C, W>(p, wq, hk * dk + lane * C, t, i, n, history, q);
    conv_block<T, C, W>(p, wk, (p.kv_heads + hk) * dk + lane * C, t, i, n, history, k);
#pragma unroll
    for (int b = 0; b < kBlk; ++b)
#pragma unroll
        for (int c = 0; c < (HEAD ? 1 : C); ++c) g[b][c] = b < n ? cd_decay_as<T>(rate, g[b][c] + bias[c]) : 1.f;
    // values 0-5: m, 6-15: n, 16-19: |k|², 20-23: |q|²; ends[j]: k_j times the decays behind it
    float sums[32], ends[kBlk][C];
#pragma unroll
    for (int x = 0; x < 32; ++x) sums[x] = 0.f;
#pragma unroll
    for (int j = 0; j < kBlk; ++j)
#pragma unroll
        for (int c = 0; c < C; ++c) {
            float d = k[j][c];
            sums[16 + j] = fmaf(d, d, sums[16 + j]);
            sums[20 + j] = fmaf(q[j][c], q[j][c], sums[20 + j]);
            sums[6 + j * (j + 1) / 2 + j] = fmaf(q[j][c], d, sums[6 + j * (j + 1) / 2 + j]);
#pragma unroll
            for (int x = j + 1; x < kBlk; ++x) {
                if constexpr (!HEAD) d *= g[x][c];
                sums[x * (x - 1) / 2 + j] = fmaf(k[x][c], d, sums[x * (x - 1) / 2 + j]);
                sums[6 + x * (x + 1) / 2 + j] = fmaf(q[x][c], d, sums[6 + x * (x + 1) / 2 + j]);
            }
            ends[j][c] = d;
        }
    float total = total_of_lane(sums, lane);
    const float inv = 1.f / sqrtf(total + kUnitEps);      // of use on lanes 16-23
    float rk[kBlk], rq[kBlk];
#pragma unroll
    for (int b = 0; b < kBlk; ++b) {
        rk[b] = __shfl_sync(0xffffffffu, inv, 16 + b);
        rq[b] = __shfl_sync(0xffffffffu, inv, 20 + b) * rsqrtf((float)p.dk_real);
    }
    constexpr int kVecs = BlockVectors<HEAD>::value;
    float* out = p.blocks + ((size_t)(first_block(p.q_start[seq], seq) + i / kBlk) * p.heads + h) * (kVecs * dk + kScalars);
    // scalars: scale by the norms of their pair
    float f = 1.f;
#pragma unroll
    for (int j = 0; j < kBlk; ++j) {
        float between = 1.f;                              // g_{j+1} .. g_x (in the sums already with one decay per channel)
#pragma unroll
        for (int x = j; x < kBlk; ++x) {
            if (HEAD && x > j) between *= g[x][0];
            if (j < x && lane == x * (x - 1) / 2 + j) f = rk[x] * rk[j] * between;
            if (lane == 6 + x * (x + 1) / 2 + j) f = rq[x] * rk[j] * between;
        }
    }
    total *= f;
    if (lane >= 16) total = lane < 16 + n ? cd_sigmoid(p.beta[(t + lane - 16) * p.ld_beta + h]) : 0.f;
    if constexpr (HEAD) {
        float up = 1.f, behind = 1.f;
#pragma unroll
        for (int b = 0; b < kBlk; ++b) {
            up *= g[b][0];
            if (lane == 20 + b) total = up;
            if (lane == 24 + kBlk - 1 - b) total = behind;
            behind *= g[kBlk - 1 - b][0];
        }
    }
    out[kVecs * dk + lane] = total;
    if constexpr (HEAD) {
#pragma unroll
        for (int v = 0; v < C; v += V) {
            const int ch = lane * C + v, at = walk_granule(dk, ch >> 2) * 4 + (ch & 3);
#pragma unroll
            for (int b = 0; b < kBlk; ++b) {
                float x[V], y[V];
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    x[e] = k[b][v + e] * rk[b];
                    y[e] = q[b][v + e] * rq[b];
                }
                store_n<float, V>(out + b * dk + at, x);
                store_n<float, V>(out + (kBlk + b) * dk + at, y);
            }
        }
        return;
    }
    float d[C];
#pragma unroll
    for (int c = 0; c < C; ++c) d[c] = 1.f;
#pragma unroll
    for (int v = 0; v < C; v += V) {
        const int ch = lane * C + v, at = walk_granule(dk, ch >> 2) * 4 + (ch & 3);
#pragma unroll
        for (int b = 0; b < kBlk; ++b) {
            float x[V], y[V], z[V];
#pragma unroll
            for (int e = 0; e < V; ++e) {
                d[v + e] *= g[b][v + e];
                x[e] = d[v + e] * k[b][v + e] * rk[b];
                y[e] = d[v + e] * q[b][v + e] * rq[b];
                z[e] = ends[b][v + e] * rk[b];
            }
            store_n<float, V>(out + b * dk + at, x);
            store_n<float, V>(out + (kBlk + b) * dk + at, y);
            store_n<float, V>(out + (2 * kBlk + b) * dk + at, z);
        }
        float e4[V];
#pragma unroll
        for (int e = 0; e < V; ++e) e4[e] = d[v + e];
        store_n<float, V>(out + 3 * kBlk * dk + at, e4);
    }
}

template <typename T, int C, int W>
__device__ __forceinline__ void prep_values(const ChannelDeltaParams& p, const float (&w)[W][C], int h, int seq, size_t t, int i, int n, const T* history) {
    const int lane = threadIdx.x & 31;
    float y[kBlk][C];
    conv_block<T, C, W>(p, w, 2 * p.kv_heads * p.dk + h * p.dv + lane * C, t, i, n, history, y);
    T* out = reinterpret_cast<T*>(p.v_blocks) + (((size_t)(first_block(p.q_start[seq], seq) + i / kBlk) * p.heads + h) * p.dv + lane * C) * kBlk;
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const T e[kBlk] = {Cvt<T>::from_f(y[0][c]), Cvt<T>::from_f(y[1][c]), Cvt<T>::from_f(y[2][c]), Cvt<T>::from_f(y[3][c])};
        store_n<T, kBlk>(out + c * kBlk, e);
    }
}

#define TELB_BY_LANES(dim, CALL)        \
    switch ((dim) >> 5) {               \
        case 1: { constexpr int C = 1; CALL; break; } \
        case 2: { constexpr int C = 2; CALL; break; } \
        case 4: { constexpr int C = 4; CALL; break; } \
        default: { constexpr int C = 8; CALL; break; } \
    }

// The blocks that start in rows t0 .. t1 - 1.
template <typename T, int C, int W, bool VALUES, bool HEAD>
__device__ void prep_range(const ChannelDeltaParams& p, int h, int t0, int t1) {
    const int lane = threadIdx.x & 31, hk = h / (p.heads / p.kv_heads);
    float w0[W][C], w1[VALUES ? 1 : W][C], bias[C];
    float rate = 0.f;
    if constexpr (VALUES) {
        load_taps<T, C, W>(p, 2 * p.kv_heads * p.dk + h * p.dv + lane * C, w0);
    } else {
        load_taps<T, C, W>(p, hk * p.dk + lane * C, w0);
        load_taps<T, C, W>(p, (p.kv_heads + hk) * p.dk + lane * C, w1);
        if constexpr (HEAD) bias[0] = p.decay_bias[h];
        else load_n<float, C>(p.decay_bias + h * p.dk + lane * C, bias);
        rate = -expf(p.a_log[h]);
    }
    for (int t = t0; t < t1;) {
        const int seq = p.seq_ids[t], i = t - p.q_start[seq];
        if (i % kBlk) {
            t += min(kBlk - i % kBlk, p.q_len[seq] - i);
            continue;
        }
        const int n = min(kBlk, p.q_len[seq] - i);
        const T* history = p.past_len[seq] > 0 ? reinterpret_cast<const T*>(p.conv_state) + (size_t)p.slot_ids[seq] * p.channels * (p.taps - 1) : nullptr;
        if constexpr (VALUES) prep_values<T, C, W>(p, w0, h, seq, t, i, n, history);
        else prep_head<T, C, W, HEAD>(p, w0, w1, bias, rate, h, seq, t, i, n, history);
        t += n;
    }
}

// grid (row ranges, heads).  VALUES: the value heads, else q, k and decays.
template <typename T, int C, int W, bool VALUES, bool HEAD>
__global__ void __launch_bounds__(128) channel_delta_prep_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_prologue();
    const int t0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * kPrepTokens, t1 = min(p.tokens, t0 + kPrepTokens);
    prep_range<T, C, W, VALUES, HEAD>(p, blockIdx.y, t0, t1);
}

// History of the convolutions after a portion: the last taps - 1 inputs.
template <typename T>
__global__ void __launch_bounds__(128) channel_delta_roll_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_prologue();
    const int seq = blockIdx.y, ch = blockIdx.x * 128 + threadIdx.x;
    const int ql = p.q_len[seq], hist = p.taps - 1;
    if (ch >= p.channels || ql <= 0) return;
    const T* x = reinterpret_cast<const T*>(p.qkv) + (size_t)p.q_start[seq] * p.ld_qkv + ch;
    T* cs = reinterpret_cast<T*>(p.conv_state) + ((size_t)p.slot_ids[seq] * p.channels + ch) * hist;
    const bool fresh = p.past_len[seq] == 0;
    for (int j = 0; j < hist; ++j) {                      // ascending: an old value is read before its place is written
        const int r = ql - hist + j;
        cs[j] = r >= 0 ? x[(size_t)r * p.ld_qkv] : (fresh ? Cvt<T>::from_f(0.f) : cs[j + ql]);
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
// Rows of lane group rl (of 8): blocks of BL = min(8, RPL) rows, block j at rows j · 8 BL + rl · BL.
template <int RPL>
struct WalkRows {
    static constexpr int BL = RPL < 8 ? RPL : 8;
    static __device__ __forceinline__ int row(int rl, int i) { return (i / BL) * (8 * BL) + rl * BL + i % BL; }
};

// Totals over the eight lanes of a group of a[c][i] (products with k) and b[c][i] (with q), columns c of the lane, tokens i.  Even lanes
// receive the four k sums of column walk_col, odd lanes the four q sums.
template <int C>
__device__ __forceinline__ int walk_col(int rl) { return C == 4 ? rl >> 1 : C == 2 ? (rl >> 1) & 1 : 0; }
template <int C>
__device__ __forceinline__ void walk_reduce(const float (&a)[C][kBlk], const float (&b)[C][kBlk], int rl, float (&w)[kBlk]) {
    constexpr unsigned kAll = 0xffffffffu;
    float s[C][kBlk];
    const bool odd = rl & 1;
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
        for (int i = 0; i < kBlk; ++i) s[c][i] = (odd ? b[c][i] : a[c][i]) + __shfl_xor_sync(kAll, odd ? a[c][i] : b[c][i], 1);
    const bool h2 = rl & 2, h4 = rl & 4;
    if constexpr (C == 4) {
        float x[2][kBlk];
#pragma unroll
        for (int i = 0; i < kBlk; ++i) {
            x[0][i] = (h4 ? s[2][i] : s[0][i]) + __shfl_xor_sync(kAll, h4 ? s[0][i] : s[2][i], 4);
            x[1][i] = (h4 ? s[3][i] : s[1][i]) + __shfl_xor_sync(kAll, h4 ? s[1][i] : s[3][i], 4);
        }
#pragma unroll
        for (int i = 0; i < kBlk; ++i) w[i] = (h2 ? x[1][i] : x[0][i]) + __shfl_xor_sync(kAll, h2 ? x[0][i] : x[1][i], 2);
    } else {
#pragma unroll
        for (int i = 0; i < kBlk; ++i) {
            float x;
            if constexpr (C == 2) x = (h2 ? s[1][i] : s[0][i]) + __shfl_xor_sync(kAll, h2 ? s[0][i] : s[1][i], 2);
            else x = s[0][i] + __shfl_xor_sync(kAll, s[0][i], 2);
            w[i] = x + __shfl_xor_sync(kAll, x, 4);
        }
    }
}

constexpr int kWalkStages = 4;

// grid (column slices of a head, heads, sequences); blockDim = warps of one slice
template <typename T, int RPL, int CPL, bool HEAD>
__global__ void __launch_bounds__(128) channel_delta_walk_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_wait();                                           // dependents start at the end: a long kernel runs slower under waiting ones
    constexpr int DK = RPL * 8;
    constexpr unsigned kAll = 0xffffffffu;
    extern __shared__ __align__(16) uint8_t walk_smem[];
    __shared__ uint64_t full[kWalkStages];
    __shared__ uint32_t abort_word;
    volatile uint32_t* abort_flag = &abort_word;
    const int seq = blockIdx.z, h = blockIdx.y;
    const int ql = p.q_len[seq];
    if (ql <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int rl = lane & 7, cg = lane >> 3;
    const int cols = (blockDim.x >> 5) * 4 * CPL;         // columns of this CTA
    const int lcol = blockIdx.x * cols + warp * 4 * CPL + cg * CPL;      // first column of this lane, within the head
    const int r0 = p.q_start[seq], blk0 = first_block(r0, seq);
    const int chunks = (ql + kBlk - 1) / kBlk;
    constexpr int kVecs = BlockVectors<HEAD>::value, kFloats = kVecs * DK + kScalars;

    const int v_bytes = cols * kBlk * (int)sizeof(T), stage_bytes = kFloats * 4 + v_bytes;

    auto fetch = [&](int chunk) {
        uint64_t* bar = &full[chunk % kWalkStages];
        uint8_t* st = walk_smem + (chunk % kWalkStages) * stage_bytes;
        const size_t blk = (size_t)(blk0 + chunk) * p.heads + h;
        mbar_expect_tx(bar, stage_bytes);
        bulk_load(st, p.blocks + blk * kFloats, kFloats * 4, bar);
        bulk_load(st + kFloats * 4, reinterpret_cast<const T*>(p.v_blocks) + (blk * p.dv + blockIdx.x * cols) * kBlk, v_bytes, bar);
    };
    if (tid == 0) {
        for (int s = 0; s < kWalkStages; ++s) mbar_init(&full[s], 1);
        abort_word = 0;
        mbar_fence_init();
        for (int s = 0; s < kWalkStages && s < chunks; ++s) fetch(s);
    }

    f2 S[RPL / 2][CPL];
    float* state = p.state + (((size_t)p.slot_ids[seq] * p.heads + h) * DK) * p.dv + lcol;
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
    const int my_col = walk_col<CPL>(rl);
    const bool writer = (rl & 1) && (CPL == 4 || (CPL == 2 ? !(rl & 4) : rl == 1));      // one odd lane per column
    T* out = reinterpret_cast<T*>(p.o) + (size_t)r0 * p.heads * p.dv + (size_t)h * p.dv + lcol + my_col;
    __syncthreads();
    bool ok = true;
    for (int ch = 0; ch < chunks; ++ch) {
        ok = mbar_wait(&full[ch % kWalkStages], (ch / kWalkStages) & 1, abort_flag, p.status, kStatusEpilogueTimeout);
        if (!ok) break;
        const float* st = reinterpret_cast<const float*>(walk_smem + (ch % kWalkStages) * stage_bytes);
        // eight products with the state before the block: four rows of all vectors at a time, every product with a chain of its own
        float a[CPL][kBlk], b[CPL][kBlk];
        {
            f2 acc[2 * kBlk][CPL];
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                ulonglong2 x[2 * kBlk];
#pragma unroll
                for (int i = 0; i < 2 * kBlk; ++i) x[i] = *reinterpret_cast<const ulonglong2*>(st + i * DK + (j * 8 + rl) * 4);
#pragma unroll
                for (int i = 0; i < 2 * kBlk; ++i)
#pragma unroll
                    for (int c = 0; c < CPL; ++c) acc[i][c] = j == 0 ? f2_mul(S[0][c], x[i].x) : f2_fma(S[2 * j][c], x[i].x, acc[i][c]);
#pragma unroll
                for (int i = 0; i < 2 * kBlk; ++i)
#pragma unroll
                    for (int c = 0; c < CPL; ++c) acc[i][c] = f2_fma(S[2 * j + 1][c], x[i].y, acc[i][c]);
            }
#pragma unroll
            for (int c = 0; c < CPL; ++c)
#pragma unroll
                for (int i = 0; i < kBlk; ++i) {
                    a[c][i] = f2_sum(acc[i][c]);
                    b[c][i] = f2_sum(acc[kBlk + i][c]);
                }
        }
        float w[kBlk];
        walk_reduce<CPL>(a, b, rl, w);
        alignas(16) float sc[HEAD ? 28 : 20];
#pragma unroll
        for (int i = 0; i < (HEAD ? 7 : 5); ++i) reinterpret_cast<float4*>(sc)[i] = reinterpret_cast<const float4*>(st + kVecs * DK)[i];
        if constexpr (HEAD) {
#pragma unroll
            for (int i = 0; i < kBlk; ++i) w[i] *= sc[20 + i];
        }
        float v[kBlk];
        load_n<T, kBlk>(reinterpret_cast<const T*>(st + kFloats) + (lcol - (int)blockIdx.x * cols + my_col) * kBlk, v);
        float u[kBlk];                                    // even lanes
        u[0] = sc[16] * (v[0] - w[0]);
        u[1] = sc[17] * (v[1] - w[1] - sc[0] * u[0]);
        u[2] = sc[18] * (v[2] - w[2] - sc[1] * u[0] - sc[2] * u[1]);
        u[3] = sc[19] * (v[3] - w[3] - sc[3] * u[0] - sc[4] * u[1] - sc[5] * u[2]);
        float mine[kBlk];                                 // odd lanes: the steps of their column
#pragma unroll
        for (int i = 0; i < kBlk; ++i) mine[i] = __shfl_xor_sync(kAll, u[i], 1);
        f2 ub[CPL][kBlk];
#pragma unroll
        for (int c = 0; c < CPL; ++c)
#pragma unroll
            for (int i = 0; i < kBlk; ++i) {
                float x = CPL == 1 ? (rl & 1 ? mine[i] : u[i]) : __shfl_sync(kAll, u[i], (lane & 24) | (c * 2));
                if constexpr (HEAD) x *= sc[24 + i];
                ub[c][i] = f2_pack(x, x);
            }
        if (writer) {
            const int n = min(kBlk, ql - ch * kBlk);
            float o[kBlk];
            o[0] = w[0] + sc[6] * mine[0];
            o[1] = w[1] + sc[7] * mine[0] + sc[8] * mine[1];
            o[2] = w[2] + sc[9] * mine[0] + sc[10] * mine[1] + sc[11] * mine[2];
            o[3] = w[3] + sc[12] * mine[0] + sc[13] * mine[1] + sc[14] * mine[2] + sc[15] * mine[3];
#pragma unroll
            for (int i = 0; i < kBlk; ++i)
                if (i < n) out[(size_t)i * p.heads * p.dv] = Cvt<T>::from_f(o[i]);
        }
        out += (size_t)kBlk * p.heads * p.dv;
#pragma unroll
        for (int j = 0; j < RPL / 4; ++j) {
            ulonglong2 x[kBlk + 1];                       // D_4 is the vector behind the four (one number with head decays)
#pragma unroll
            for (int i = 0; i < (HEAD ? kBlk : kBlk + 1); ++i) x[i] = *reinterpret_cast<const ulonglong2*>(st + ((HEAD ? 0 : 2 * kBlk) + i) * DK + (j * 8 + rl) * 4);
            if constexpr (HEAD) x[kBlk].x = x[kBlk].y = f2_pack(sc[23], sc[23]);
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
                S[2 * j][c] = f2_mul(S[2 * j][c], x[kBlk].x);
                S[2 * j + 1][c] = f2_mul(S[2 * j + 1][c], x[kBlk].y);
            }
#pragma unroll
            for (int i = 0; i < kBlk; ++i)
#pragma unroll
                for (int c = 0; c < CPL; ++c) {
                    S[2 * j][c] = f2_fma(x[i].x, ub[c][i], S[2 * j][c]);
                    S[2 * j + 1][c] = f2_fma(x[i].y, ub[c][i], S[2 * j + 1][c]);
                }
        }
        if (ch + kWalkStages < chunks) {                  // every warp is done with the stage: refill it
            __syncthreads();
            if (tid == 0) fetch(ch + kWalkStages);
        }
    }
    pdl_launch_dependents();
    if (!ok) {                                            // a copy never arrived: leave the state alone, let what is in flight land
        const uint64_t t0 = global_timer_ns();
        while (global_timer_ns() - t0 < 200000ull) __nanosleep(1000);
        return;
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

// The walk for few (sequence, head) pairs and keys of 128 or 256: all 32 lanes share the rows of four columns (four rows, G granules each),
// so a vector costs one shared-memory read per warp and granule instead of four and the chain of a block is short.  The 32 products of
// a block (columns x (k, q) x tokens) are reduced so that lane 8 c + 4 a + i holds product a of column c and token i.
template <typename T, int G, bool HEAD>
__global__ void __launch_bounds__(128) channel_delta_walk_narrow_kernel(const __grid_constant__ ChannelDeltaParams p) {
    pdl_wait();
    constexpr int DK = G * 128, C = 4, kCols = 16;
    constexpr unsigned kAll = 0xffffffffu;
    constexpr int kVecs = BlockVectors<HEAD>::value, kFloats = kVecs * DK + kScalars, kVBytes = kCols * kBlk * (int)sizeof(T), kStage = kFloats * 4 + kVBytes;
    extern __shared__ __align__(16) uint8_t walk_smem[];
    __shared__ uint64_t full[kWalkStages];
    __shared__ uint32_t abort_word;
    volatile uint32_t* abort_flag = &abort_word;
    const int seq = blockIdx.z, h = blockIdx.y;
    const int ql = p.q_len[seq];
    if (ql <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int col0 = blockIdx.x * kCols + warp * C, c_own = lane >> 3, i_own = lane & 3;
    const int r0 = p.q_start[seq], blk0 = first_block(r0, seq), chunks = (ql + kBlk - 1) / kBlk;
    auto fetch = [&](int chunk) {
        uint64_t* bar = &full[chunk % kWalkStages];
        uint8_t* st = walk_smem + (chunk % kWalkStages) * kStage;
        const size_t blk = (size_t)(blk0 + chunk) * p.heads + h;
        mbar_expect_tx(bar, kStage);
        bulk_load(st, p.blocks + blk * kFloats, kFloats * 4, bar);
        bulk_load(st + kFloats * 4, reinterpret_cast<const T*>(p.v_blocks) + (blk * p.dv + blockIdx.x * kCols) * kBlk, kVBytes, bar);
    };
    if (tid == 0) {
        for (int s = 0; s < kWalkStages; ++s) mbar_init(&full[s], 1);
        abort_word = 0;
        mbar_fence_init();
        for (int s = 0; s < kWalkStages && s < chunks; ++s) fetch(s);
    }
    // granule at place x of a vector in lane order holds rows 4 m .. 4 m + 3 with m = place_granule(x)
    auto first_row = [&](int g) {
        const int x = lane + 32 * g, j = x >> 3;
        return 4 * ((j >> 1) * 16 + 2 * (x & 7) + (j & 1));
    };
    f2 S[2 * G][C];
    float* state = p.state + (((size_t)p.slot_ids[seq] * p.heads + h) * DK) * p.dv + col0;
    const bool fresh = p.past_len[seq] == 0;
#pragma unroll
    for (int r = 0; r < 2 * G; ++r) {
        float a[C] = {}, b[C] = {};
        if (!fresh) {
            const size_t row = first_row(r >> 1) + 2 * (r & 1);
            load_n<float, C>(state + row * p.dv, a);
            load_n<float, C>(state + (row + 1) * p.dv, b);
        }
#pragma unroll
        for (int c = 0; c < C; ++c) S[r][c] = f2_pack(a[c], b[c]);
    }
    T* out = reinterpret_cast<T*>(p.o) + ((size_t)r0 + i_own) * p.heads * p.dv + (size_t)h * p.dv + col0 + c_own;
    const int n_row = kVecs * DK + 6 + i_own * (i_own + 1) / 2;
    __syncthreads();
    bool ok = true;
    for (int ch = 0; ch < chunks; ++ch) {
        ok = mbar_wait(&full[ch % kWalkStages], (ch / kWalkStages) & 1, abort_flag, p.status, kStatusEpilogueTimeout);
        if (!ok) break;
        const float* st = reinterpret_cast<const float*>(walk_smem + (ch % kWalkStages) * kStage);
        f2 acc[2 * kBlk][C];
#pragma unroll
        for (int g = 0; g < G; ++g)
#pragma unroll
            for (int i = 0; i < 2 * kBlk; ++i) {
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(st + i * DK + (lane + 32 * g) * 4);
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    acc[i][c] = g == 0 ? f2_mul(S[0][c], x.x) : f2_fma(S[2 * g][c], x.x, acc[i][c]);
                    acc[i][c] = f2_fma(S[2 * g + 1][c], x.y, acc[i][c]);
                }
            }
        float sums[32];
#pragma unroll
        for (int c = 0; c < C; ++c)
#pragma unroll
            for (int i = 0; i < 2 * kBlk; ++i) sums[c * 8 + i] = f2_sum(acc[i][c]);
        float total = total_of_lane(sums, lane);
        if constexpr (HEAD) total *= st[kVecs * DK + 20 + i_own];
        float w[kBlk], v[kBlk], u[kBlk];
        load_n<T, kBlk>(reinterpret_cast<const T*>(st + kFloats) + (warp * C + c_own) * kBlk, v);
        alignas(16) float m[8], beta[kBlk], behind[kBlk];
        reinterpret_cast<float4*>(m)[0] = *reinterpret_cast<const float4*>(st + kVecs * DK);
        reinterpret_cast<float4*>(m)[1] = *reinterpret_cast<const float4*>(st + kVecs * DK + 4);
        *reinterpret_cast<float4*>(beta) = *reinterpret_cast<const float4*>(st + kVecs * DK + 16);
        if constexpr (HEAD) *reinterpret_cast<float4*>(behind) = *reinterpret_cast<const float4*>(st + kVecs * DK + 24);
        const float all = HEAD ? st[kVecs * DK + 23] : 1.f;
        float nr[kBlk];
#pragma unroll
        for (int j = 0; j < kBlk; ++j) nr[j] = j <= i_own ? st[n_row + j] : 0.f;
#pragma unroll
        for (int i = 0; i < kBlk; ++i) w[i] = __shfl_sync(kAll, total, (lane & 24) + i);
        u[0] = beta[0] * (v[0] - w[0]);
        u[1] = beta[1] * (v[1] - w[1] - m[0] * u[0]);
        u[2] = beta[2] * (v[2] - w[2] - m[1] * u[0] - m[2] * u[1]);
        u[3] = beta[3] * (v[3] - w[3] - m[3] * u[0] - m[4] * u[1] - m[5] * u[2]);
        if ((lane & 4) && i_own < ql - ch * kBlk)
            *out = Cvt<T>::from_f(total + nr[0] * u[0] + nr[1] * u[1] + (nr[2] * u[2] + nr[3] * u[3]));
        out += (size_t)kBlk * p.heads * p.dv;
        f2 ub[C][kBlk];
#pragma unroll
        for (int c = 0; c < C; ++c)
#pragma unroll
            for (int i = 0; i < kBlk; ++i) {
                float x = __shfl_sync(kAll, u[i], c * 8);
                if constexpr (HEAD) x *= behind[i];
                ub[c][i] = f2_pack(x, x);
            }
#pragma unroll
        for (int g = 0; g < G; ++g) {
            ulonglong2 x[kBlk + 1];
#pragma unroll
            for (int i = 0; i < (HEAD ? kBlk : kBlk + 1); ++i) x[i] = *reinterpret_cast<const ulonglong2*>(st + ((HEAD ? 0 : 2 * kBlk) + i) * DK + (lane + 32 * g) * 4);
            if constexpr (HEAD) x[kBlk].x = x[kBlk].y = f2_pack(all, all);
#pragma unroll
            for (int c = 0; c < C; ++c) {
                S[2 * g][c] = f2_mul(S[2 * g][c], x[kBlk].x);
                S[2 * g + 1][c] = f2_mul(S[2 * g + 1][c], x[kBlk].y);
            }
#pragma unroll
            for (int i = 0; i < kBlk; ++i)
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    S[2 * g][c] = f2_fma(x[i].x, ub[c][i], S[2 * g][c]);
                    S[2 * g + 1][c] = f2_fma(x[i].y, ub[c][i], S[2 * g + 1][c]);
                }
        }
        if (ch + kWalkStages < chunks) {                  // every warp is done with the stage: refill it
            __syncthreads();
            if (tid == 0) fetch(ch + kWalkStages);
        }
    }
    pdl_launch_dependents();
    if (!ok) {                                            // a copy never arrived: leave the state alone, let what is in flight land
        const uint64_t t0 = global_timer_ns();
        while (global_timer_ns() - t0 < 200000ull) __nanosleep(1000);
        return;
    }
#pragma unroll
    for (int r = 0; r < 2 * G; ++r) {
        float a[C], b[C];
#pragma unroll
        for (int c = 0; c < C; ++c) asm("mov.b64 {%0, %1}, %2;" : "=f"(a[c]), "=f"(b[c]) : "l"(S[r][c]));
        const size_t row = first_row(r >> 1) + 2 * (r & 1);
        store_n<float, C>(state + row * p.dv, a);
        store_n<float, C>(state + (row + 1) * p.dv, b);
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
    for (int c = 0; c < C; ++c) {
        const float s = sizeof(T) == 4 ? cd_sigmoid(z[c]) : __fdividef(1.f, 1.f + __expf(-z[c]));
        y[c] = Cvt<T>::from_f(o[c] * inv * w[c] * (p.gate_silu ? s * z[c] : s) * p.mult);
    }
    store_n<T, C>(reinterpret_cast<T*>(p.out) + t * p.ld_out + col, y);
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
// The convolution history is rolled here unless heads share q and k (they would read what another CTA rolls).
template <typename T, int DK, int DV>
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
    const T* x = reinterpret_cast<const T*>(p.qkv) + t * p.ld_qkv;
    for (int i = tid; i < 2 * DK + DV; i += 256) {
        const int ch = i < DK ? hk * DK + i : i < 2 * DK ? p.kv_heads * DK + hk * DK + i - DK : 2 * p.kv_heads * DK + h * DV + i - 2 * DK;
        T* cs = reinterpret_cast<T*>(p.conv_state) + (slot * p.channels + ch) * hist;
        const T* cw = reinterpret_cast<const T*>(p.conv_w) + (size_t)ch * p.taps;
        float acc = 0.f;
        if (!fresh)
            for (int j = 0; j < hist; ++j) acc = fmaf(Cvt<T>::to_f(cw[j]), Cvt<T>::to_f(cs[j]), acc);
        acc = fmaf(Cvt<T>::to_f(cw[hist]), Cvt<T>::to_f(x[ch]), acc);
        const float y = Cvt<T>::to_f(Cvt<T>::from_f(cd_silu_as<T>(acc)));
        if (hist > 0 && group == 1) {
            for (int j = 0; j + 1 < hist; ++j) cs[j] = fresh ? Cvt<T>::from_f(0.f) : cs[j + 1];
            cs[hist - 1] = x[ch];
        }
        (i < DK ? s_q[i] : i < 2 * DK ? s_k[i - DK] : s_v[i - 2 * DK]) = y;
    }
    const float rate = -expf(p.a_log[h]), beta = cd_sigmoid(p.beta[t * p.ld_beta + h]);
    for (int i = tid; i < DK; i += 256) {
        const int at = p.head_decay ? h : h * DK + i;
        s_g[i] = cd_decay_as<T>(rate, p.decay[t * p.ld_decay + at] + p.decay_bias[at]);
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
        reinterpret_cast<T*>(p.out)[t * p.ld_out + h * DV + tid] = Cvt<T>::from_f(o * inv * p.norm_w[tid] * cd_sigmoid(z) * (p.gate_silu ? z : 1.f) * p.mult);
    }
}

// ---- launchers ---------------------------------------------------------------------------------------------
template <typename T, bool HEAD>
static int launch_prep(const ChannelDeltaParams& p, cudaStream_t stream) {
    const int warps = (p.tokens + kPrepTokens - 1) / kPrepTokens;
    const dim3 grid((warps + 3) / 4, p.heads);
#define TELB_PREP(W_, VALUES_, HEAD_) \
    TELB_LAUNCH("channel_delta_prep_kernel", (channel_delta_prep_kernel<T, C, W_, VALUES_, HEAD_>), grid, dim3(128), 0, stream, p)
    if (p.taps <= 4) {
        TELB_BY_LANES(p.dv, TELB_PREP(4, true, false))
        TELB_BY_LANES(p.dk, TELB_PREP(4, false, HEAD))
    } else {
        TELB_BY_LANES(p.dv, TELB_PREP(8, true, false))
        TELB_BY_LANES(p.dk, TELB_PREP(8, false, HEAD))
    }
#undef TELB_PREP
    TELB_CHECK_LAUNCH("channel_delta_prep_kernel");
    return 0;
}

template <typename T>
static int launch_roll(const ChannelDeltaParams& p, cudaStream_t stream) {
    if (p.taps < 2) return 0;
    TELB_LAUNCH("channel_delta_roll_kernel", (channel_delta_roll_kernel<T>), dim3((p.channels + 127) / 128, p.num_seqs), dim3(128), 0, stream, p);
    TELB_CHECK_LAUNCH("channel_delta_roll_kernel");
    return 0;
}

template <typename T, int RPL, int CPL, bool HEAD>
static int launch_walk_as(const ChannelDeltaParams& p, cudaStream_t stream) {
    constexpr int warps = CPL == 1 ? 4 : 2, cols = warps * 4 * CPL;      // 16 or 32: divides every padded head
    constexpr int smem = ((BlockVectors<HEAD>::value * RPL * 8 + kScalars) * 4 + cols * kBlk * (int)sizeof(T)) * kWalkStages;
    if (smem > 48 * 1024) {
        static bool configured = false;
        if (!configured) {
            cudaError_t e = cudaFuncSetAttribute(channel_delta_walk_kernel<T, RPL, CPL, HEAD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
            if (e != cudaSuccess) return fail("cudaFuncSetAttribute(channel_delta_walk)", e);
            configured = true;
        }
    }
    TELB_LAUNCH_SERIAL("channel_delta_walk_kernel", (channel_delta_walk_kernel<T, RPL, CPL, HEAD>), dim3(p.dv / cols, p.heads, p.num_seqs), dim3(warps * 32), smem, stream, p);
    TELB_CHECK_LAUNCH("channel_delta_walk_kernel");
    return 0;
}

template <typename T, int G, bool HEAD>
static int launch_walk_narrow(const ChannelDeltaParams& p, cudaStream_t stream) {
    constexpr int smem = ((BlockVectors<HEAD>::value * G * 128 + kScalars) * 4 + 16 * kBlk * (int)sizeof(T)) * kWalkStages;
    if (smem > 48 * 1024) {
        static bool configured = false;
        if (!configured) {
            cudaError_t e = cudaFuncSetAttribute(channel_delta_walk_narrow_kernel<T, G, HEAD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
            if (e != cudaSuccess) return fail("cudaFuncSetAttribute(channel_delta_walk_narrow)", e);
            configured = true;
        }
    }
    TELB_LAUNCH_SERIAL("channel_delta_walk_narrow_kernel", (channel_delta_walk_narrow_kernel<T, G, HEAD>), dim3(p.dv / 16, p.heads, p.num_seqs), dim3(128), smem, stream, p);
    TELB_CHECK_LAUNCH("channel_delta_walk_narrow_kernel");
    return 0;
}

static int g_walk_cols = 0;          // columns per lane; 0 = by the number of columns

template <typename T, int RPL, bool HEAD>
static int launch_walk(const ChannelDeltaParams& p, cudaStream_t stream) {
    // few (sequence, head) pairs: narrow slices, so that every scheduler has a chain of its own; many: wide ones, which read less
    const long long columns = (long long)p.num_seqs * p.heads * p.dv;
    int cpl = columns / 4 <= 8LL * sm_count() ? 1 : RPL > 16 ? 2 : 4;
    if (g_walk_cols) cpl = g_walk_cols;
    if constexpr (RPL >= 16) {
        if (cpl == 1) return launch_walk_narrow<T, RPL / 16, HEAD>(p, stream);
    } else {
        if (cpl == 1) return launch_walk_as<T, RPL, 1, HEAD>(p, stream);
    }
    if (cpl == 2 || RPL > 16) return launch_walk_as<T, RPL, 2, HEAD>(p, stream);
    return launch_walk_as<T, RPL, (RPL > 16 ? 2 : 4), HEAD>(p, stream);
}

template <typename T, bool HEAD>
static int channel_delta_rows(const ChannelDeltaParams& p, cudaStream_t stream) {
    if (launch_prep<T, HEAD>(p, stream)) return -1;
    int rc = 0;
    switch (p.dk) {
        case 32: rc = launch_walk<T, 4, HEAD>(p, stream); break;
        case 64: rc = launch_walk<T, 8, HEAD>(p, stream); break;
        case 128: rc = launch_walk<T, 16, HEAD>(p, stream); break;
        default: rc = launch_walk<T, 32, HEAD>(p, stream); break;
    }
    if (rc) return rc;
    const long long warps = (long long)p.tokens * p.heads;
    TELB_LAUNCH("channel_delta_out_kernel", (channel_delta_out_kernel<T>), dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, stream, p);
    TELB_CHECK_LAUNCH("channel_delta_out_kernel");
    return launch_roll<T>(p, stream);
}

template <typename T, int DK, int DV>
static int launch_decode_step(const ChannelDeltaParams& p, cudaStream_t stream) {
    const dim3 grid(p.heads, p.num_seqs);
    TELB_LAUNCH("channel_delta_decode_kernel", (channel_delta_decode_kernel<T, DK, DV>), grid, dim3(256), 0, stream, p);
    TELB_CHECK_LAUNCH("channel_delta_decode_kernel");
    return p.heads == p.kv_heads ? 0 : launch_roll<T>(p, stream);
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

// Columns per lane of the walk: 1, 2 or 4; 0 picks by the number of columns.  Process-wide.
extern "C" int telb_set_delta_walk_columns(int n) {
    if (n != 0 && n != 1 && n != 2 && n != 4) return fail("telb_set_delta_walk_columns: 0, 1, 2 or 4");
    g_walk_cols = n;
    return 0;
}

// dtype: 0 fp16, 1 bf16, 2 fp32 (of qkv, conv_w, conv_state, v_blocks, o, out and, unless gate_f32, gate).
// decode != 0: every sequence has at most one row and dk, dv <= 128.
extern "C" int telb_channel_delta(const ChannelDeltaParams* pp, int decode, int dtype, cudaStream_t stream) {
    const ChannelDeltaParams& p = *pp;
    if (p.tokens <= 0 || p.num_seqs <= 0) return 0;
    auto size_ok = [](int d) { return d == 32 || d == 64 || d == 128 || d == 256; };
    if (!size_ok(p.dk) || !size_ok(p.dv)) return fail("telb_channel_delta: padded head sizes are 32, 64, 128 or 256");
    if (p.taps < 1 || p.taps > 8) return fail("telb_channel_delta: convolutions have 1 to 8 taps");
    if (p.kv_heads <= 0 || p.heads % p.kv_heads) return fail("telb_channel_delta: heads must be a multiple of the q / k heads");
    if (p.ld_qkv % 8 || p.ld_out % 8) return fail("telb_channel_delta: row pitches are multiples of 8");
    if (p.num_seqs > 65535 || p.heads > 65535) return fail("telb_channel_delta: too many sequences or heads");
    if (decode) {
        if (p.dk > 128 || p.dv > 128) return fail("telb_channel_delta: the decode step covers heads up to 128");
        if (dtype == 2) return channel_delta_step<float>(p, stream);
        return dtype == 1 ? channel_delta_step<__nv_bfloat16>(p, stream) : channel_delta_step<__half>(p, stream);
    }
    if (p.head_decay) {
        if (dtype == 0) return fail("telb_channel_delta: prompts with one decay per head are built for bf16 and fp32");
        return dtype == 2 ? channel_delta_rows<float, true>(p, stream) : channel_delta_rows<__nv_bfloat16, true>(p, stream);
    }
    if (dtype == 2) return channel_delta_rows<float, false>(p, stream);
    return dtype == 1 ? channel_delta_rows<__nv_bfloat16, false>(p, stream) : channel_delta_rows<__half, false>(p, stream);
}
