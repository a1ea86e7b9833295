// The fp32 residual stream of blocks with a norm in front of and behind every sublayer.  What lies between two sublayers:
//
//   source   x = table[id] or the running stream, plus the row of the token's position (first call)
//   update   d = y + Σ_k w[t,k] · e[dst_row[t,k]]            y: sublayer output, the sum: combine of the routed experts (either may be absent)
//            x += mult * d / rms(d) * post
//   norm     h = x / rms(x) * norm
//   shift    h_t += shift * (h_{t-1} - h_t)                  for a mixer: h_{t-1} of the row before in the sequence, its state row, or zero
//
// Stream, norms, shift and state are fp32; tables, y, e and the written h have the activation type.  One CTA walks a block of rows of one
// sequence.  A shifted block starts with the row before it: inside a portion that row is computed once more, the first row of a portion
// takes the state.  The CTA that reads a sequence's state also writes it (it computes the portion's last row for that), so no CTA reads
// what another one of its launch writes, and the rows x are never advanced in place.  Steps of
// many rows run a warp per block instead.
#include "host_utils.h"
#include "stream_common.cuh"

namespace telb {

// Host mirror: ops/cuda.py (StreamSandwichParams).
struct StreamSandwichParams {
    const int* ids;              // embedding source, or null
    const void* table;           // [vocab, width]
    const void* pos_table;       // [max_pos, width] or null
    const float* x_in;           // [T, width] when ids is null
    const void* y;               // [T, width] or null
    const void* e;               // [rows, lde] expert outputs or null
    const int* dst_row;          // [T, top_k]
    const float* topk_w;         // [T, top_k]
    const float* post;           // [width], with y or e
    const float* norm;           // [width] or null
    const float* shift;          // [width] or null
    float* state;                // [slots, width], with shift
    float* x_out;                // [T, width]
    void* h;                     // [T, width], with norm
    const int* positions;
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* slot_ids;
    const int* seq_ids;
    int vocab, max_pos, width, tokens, block_rows, top_k, lde;
    float mult, eps;
};

// How a row lies on threads: N threads hold E vectors of four features each, thread i features 4 (e N + i) .. + 3.  N = 32: a warp per row,
// several rows' blocks per CTA, widths of exactly 128 E (no guards, no barriers); else the whole CTA.
template <int N>
struct RowThreads {
    static constexpr bool kWarp = N == 32;
    static constexpr int kBlocks = kWarp ? 4 : 1;                    // row blocks of a CTA
    float* red;                                                      // [2][N / 32], used alternately: one barrier per sum
    int turn = 0;
    __device__ __forceinline__ int idx() const { return kWarp ? threadIdx.x & 31 : threadIdx.x; }
    __device__ __forceinline__ int block() const { return kWarp ? blockIdx.x * kBlocks + (threadIdx.x >> 5) : blockIdx.x; }
    __device__ __forceinline__ int col(int e) const { return (e * N + idx()) * 4; }
    __device__ __forceinline__ bool in(int e, int width) const { return kWarp || col(e) < width; }
    __device__ __forceinline__ float sum(float v) {
        v = post_warp_sum(v);
        if constexpr (kWarp) return v;
        float* buf = red + (turn & 1) * (N / 32);
        ++turn;
        if ((threadIdx.x & 31) == 0) buf[threadIdx.x >> 5] = v;
        __syncthreads();
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < N / 32; ++w) s += buf[w];
        return s;
    }
};

template <typename T>
__device__ __forceinline__ void raw4(const T* p, T (&v)[4]) {
    if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
    else *reinterpret_cast<uint2*>(v) = *reinterpret_cast<const uint2*>(p);
}

// A row as it lies in memory, so that fetching it waits for nothing: the stream and the sublayer's output, or the token's table row.
template <typename T, int E>
struct RowRaw {
    float x[E][4];
    alignas(16) T y[E][4];
};

template <typename T, int N, int E>
__device__ __forceinline__ void fetch_row(const StreamSandwichParams& p, const RowThreads<N>& th, int t, RowRaw<T, E>& r) {
    const T* y = reinterpret_cast<const T*>(p.y) + (size_t)t * p.width;
    if (p.ids) y = reinterpret_cast<const T*>(p.table) + (size_t)min(max(p.ids[t], 0), p.vocab - 1) * p.width;
    const float* x = p.x_in + (size_t)t * p.width;
    if (!p.ids) {
#pragma unroll
        for (int e = 0; e < E; ++e)
            if (th.in(e, p.width)) get4(x + th.col(e), r.x[e]);
    }
    if (p.ids || p.y) {
#pragma unroll
        for (int e = 0; e < E; ++e)
            if (th.in(e, p.width)) raw4(y + th.col(e), r.y[e]);
    }
}

// Advances the row in r.x (stored when `own`) and returns one over its root mean square.
template <typename T, int N, int E, bool EXPERTS>
__device__ __forceinline__ float advance_row(const StreamSandwichParams& p, RowThreads<N>& th, int t, bool own, RowRaw<T, E>& r) {
    if (p.ids) {
#pragma unroll
        for (int e = 0; e < E; ++e)
#pragma unroll
            for (int i = 0; i < 4; ++i) r.x[e][i] = th.in(e, p.width) ? Cvt<T>::to_f(r.y[e][i]) : 0.f;
    }
    if (!EXPERTS && p.pos_table) {
        const T* row = reinterpret_cast<const T*>(p.pos_table) + (size_t)min(max(p.positions[t], 0), p.max_pos - 1) * p.width;
#pragma unroll
        for (int e = 0; e < E; ++e)
            if (th.in(e, p.width)) raw4(row + th.col(e), r.y[e]);
#pragma unroll
        for (int e = 0; e < E; ++e)
#pragma unroll
            for (int i = 0; i < 4; ++i) r.x[e][i] += th.in(e, p.width) ? Cvt<T>::to_f(r.y[e][i]) : 0.f;
    } else if constexpr (EXPERTS) {
        float d[E][4];
#pragma unroll
        for (int e = 0; e < E; ++e)
#pragma unroll
            for (int i = 0; i < 4; ++i) d[e][i] = p.y && th.in(e, p.width) ? Cvt<T>::to_f(r.y[e][i]) : 0.f;
        for (int k0 = 0; k0 < p.top_k; k0 += 4) {                    // four expert rows in flight
            const T* src[4];
            float w[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int row = k0 + k < p.top_k ? p.dst_row[(size_t)t * p.top_k + k0 + k] : -1;
                w[k] = row < 0 ? 0.f : p.topk_w[(size_t)t * p.top_k + k0 + k];
                src[k] = reinterpret_cast<const T*>(p.e) + (size_t)max(row, 0) * p.lde;
            }
#pragma unroll
            for (int e = 0; e < E; ++e) {
                if (!th.in(e, p.width)) continue;
                alignas(16) T v[4][4];
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (w[k] != 0.f) raw4(src[k] + th.col(e), v[k]);
#pragma unroll
                for (int k = 0; k < 4; ++k)
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (w[k] != 0.f) d[e][i] = fmaf(w[k], Cvt<T>::to_f(v[k][i]), d[e][i]);
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < E; ++e)
#pragma unroll
            for (int i = 0; i < 4; ++i) ss = fmaf(d[e][i], d[e][i], ss);
        const float f = p.mult / sqrtf(th.sum(ss) / p.width + p.eps);
#pragma unroll
        for (int e = 0; e < E; ++e) {
            if (!th.in(e, p.width)) continue;
            float w[4];
            get4(p.post + th.col(e), w);
#pragma unroll
            for (int i = 0; i < 4; ++i) r.x[e][i] = fmaf(d[e][i] * f, w[i], r.x[e][i]);
        }
    } else if (p.y) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < E; ++e)
            if (th.in(e, p.width)) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float v = Cvt<T>::to_f(r.y[e][i]);
                    ss = fmaf(v, v, ss);
                }
            }
        const float f = p.mult / sqrtf(th.sum(ss) / p.width + p.eps);
#pragma unroll
        for (int e = 0; e < E; ++e) {
            if (!th.in(e, p.width)) continue;
            float w[4];
            get4(p.post + th.col(e), w);
#pragma unroll
            for (int i = 0; i < 4; ++i) r.x[e][i] = fmaf(Cvt<T>::to_f(r.y[e][i]) * f, w[i], r.x[e][i]);
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) {
        if (!th.in(e, p.width)) continue;
        if (own && p.x_out) put4(p.x_out + (size_t)t * p.width + th.col(e), r.x[e]);
#pragma unroll
        for (int i = 0; i < 4; ++i) ss = fmaf(r.x[e][i], r.x[e][i], ss);
    }
    return p.norm ? 1.f / sqrtf(th.sum(ss) / p.width + p.eps) : 0.f;
}

// Every block index takes the blocks that start in its range of block_rows rows (blocks count from the start of a sequence's portion).
template <typename T, int N, int E, bool SHIFT, bool EXPERTS>
__global__ void __launch_bounds__(N * RowThreads<N>::kBlocks) stream_sandwich_kernel(const __grid_constant__ StreamSandwichParams p) {
    pdl_prologue();
    __shared__ float red[2 * (N / 32)];
    RowThreads<N> th;
    th.red = red;
    RowRaw<T, E> r, next;
    constexpr bool kAhead = !RowThreads<N>::kWarp;                   // warps overlap one another instead
    const int lo = th.block() * p.block_rows, hi = min(p.tokens, lo + p.block_rows);
    T* h = reinterpret_cast<T*>(p.h);
    if (lo >= hi) return;                                            // whole rows of threads at once
    if constexpr (!SHIFT) {
        if (kAhead) fetch_row<T, N, E>(p, th, lo, next);
        for (int t = lo; t < hi; ++t) {
            if (kAhead) {
                r = next;
                if (t + 1 < hi) fetch_row<T, N, E>(p, th, t + 1, next);
            } else {
                fetch_row<T, N, E>(p, th, t, r);
            }
            const float inv = advance_row<T, N, E, EXPERTS>(p, th, t, true, r);
            if (!p.norm) continue;
#pragma unroll
            for (int e = 0; e < E; ++e) {
                if (!th.in(e, p.width)) continue;
                float w[4];
                get4(p.norm + th.col(e), w);
#pragma unroll
                for (int i = 0; i < 4; ++i) w[i] *= r.x[e][i] * inv;
                put4(h + (size_t)t * p.width + th.col(e), w);
            }
        }
    } else {
        float before[E][4];                                          // normed row in front of the current one
        auto keep = [&](float inv) {
#pragma unroll
            for (int e = 0; e < E; ++e) {
                if (!th.in(e, p.width)) continue;
                float w[4];
                get4(p.norm + th.col(e), w);
#pragma unroll
                for (int i = 0; i < 4; ++i) before[e][i] = r.x[e][i] * inv * w[i];
            }
        };
        for (int t = lo; t < hi;) {
            const int seq = p.seq_ids[t], t0 = p.q_start[seq], i0 = t - t0, ql = p.q_len[seq];
            if (i0 % p.block_rows) {                                 // inside a block that starts in an earlier range
                t += min(p.block_rows - i0 % p.block_rows, ql - i0);
                continue;
            }
            const int end = t + min(p.block_rows, ql - i0);
            float* state = p.state + (size_t)p.slot_ids[seq] * p.width;
            if (i0 > 0) {
                fetch_row<T, N, E>(p, th, t - 1, r);
                if (kAhead) fetch_row<T, N, E>(p, th, t, next);
                keep(advance_row<T, N, E, EXPERTS>(p, th, t - 1, false, r));
            } else {
                const bool fresh = p.past_len[seq] <= 0;
                if (kAhead) fetch_row<T, N, E>(p, th, t, next);
#pragma unroll
                for (int e = 0; e < E; ++e) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) before[e][i] = 0.f;
                    if (!fresh && th.in(e, p.width)) get4(state + th.col(e), before[e]);
                }
            }
            for (int u = t; u < end; ++u) {
                if (kAhead) {
                    r = next;
                    if (u + 1 < end) fetch_row<T, N, E>(p, th, u + 1, next);
                } else {
                    fetch_row<T, N, E>(p, th, u, r);
                }
                const float inv = advance_row<T, N, E, EXPERTS>(p, th, u, true, r);
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    if (!th.in(e, p.width)) continue;
                    float w[4], sh[4];
                    get4(p.norm + th.col(e), w);
                    get4(p.shift + th.col(e), sh);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float v = r.x[e][i] * inv * w[i];
                        w[i] = fmaf(before[e][i] - v, sh[i], v);
                        before[e][i] = v;
                    }
                    put4(h + (size_t)u * p.width + th.col(e), w);
                }
            }
            if (i0 == 0) {                                           // the state moves to the portion's last row
                if (end < t0 + ql) {
                    fetch_row<T, N, E>(p, th, t0 + ql - 1, r);
                    keep(advance_row<T, N, E, EXPERTS>(p, th, t0 + ql - 1, false, r));
                }
#pragma unroll
                for (int e = 0; e < E; ++e)
                    if (th.in(e, p.width)) put4(state + th.col(e), before[e]);
            }
            t = end;
        }
    }
}

template <typename T, int N, int E>
static int launch_sandwich(const StreamSandwichParams& p, cudaStream_t stream) {
    constexpr int kBlocks = RowThreads<N>::kBlocks;
    const int blocks = (p.tokens + p.block_rows - 1) / p.block_rows;
    const dim3 grid((blocks + kBlocks - 1) / kBlocks), threads(N * kBlocks);
#define TELB_SANDWICH(SHIFT_, EXPERTS_) TELB_LAUNCH("stream_sandwich_kernel", (stream_sandwich_kernel<T, N, E, SHIFT_, EXPERTS_>), grid, threads, 0, stream, p)
    if (p.shift && p.e) TELB_SANDWICH(true, true);
    else if (p.shift) TELB_SANDWICH(true, false);
    else if (p.e) TELB_SANDWICH(false, true);
    else TELB_SANDWICH(false, false);
#undef TELB_SANDWICH
    TELB_CHECK_LAUNCH("stream_sandwich_kernel");
    return 0;
}

template <typename T>
static int run_sandwich(const StreamSandwichParams& p, int warp_rows, cudaStream_t stream) {
    if (sizeof(T) == 2 && warp_rows > 0) {
        StreamSandwichParams w = p;
        w.block_rows = warp_rows;
        if (p.width == 1024) return launch_sandwich<T, 32, 8>(w, stream);
        if (p.width == 1536) return launch_sandwich<T, 32, 12>(w, stream);
        if (p.width == 2048) return launch_sandwich<T, 32, 16>(w, stream);
    }
    if (p.width <= 512) return launch_sandwich<T, 128, 1>(p, stream);
    if (p.width <= 1024) return launch_sandwich<T, 256, 1>(p, stream);
    if (p.width <= 2048) return launch_sandwich<T, 256, 2>(p, stream);
    if (p.width <= 4096) return launch_sandwich<T, 512, 2>(p, stream);
    return launch_sandwich<T, 1024, 4>(p, stream);
}

}  // namespace telb

using namespace telb;

// dtype: 1 bf16, 2 fp32 (of the tables, y, e and h).  warp_rows > 0: blocks of that many rows run on a warp each where the width allows.
extern "C" int telb_stream_sandwich(const StreamSandwichParams* pp, int warp_rows, int dtype, cudaStream_t stream) {
    const StreamSandwichParams& p = *pp;
    if (p.tokens <= 0) return 0;
    if (p.width % 4 || p.width > 16 * 1024) return fail("telb_stream_sandwich: width must be a multiple of 4 and at most 16384");
    if (!p.ids == !p.x_in) return fail("telb_stream_sandwich: either ids or a stream");
    if (p.block_rows < 1) return fail("telb_stream_sandwich: blocks of at least one row");
    if (p.ids && (p.y || p.e)) return fail("telb_stream_sandwich: a stream that starts from ids has no update");
    if (p.pos_table && (p.y || p.e)) return fail("telb_stream_sandwich: position rows join before the first update");
    if ((p.y || p.e) && !p.post) return fail("telb_stream_sandwich: an update has a weight");
    if (p.e && (!p.dst_row || !p.topk_w || p.lde % 4)) return fail("telb_stream_sandwich: expert rows come with their tables");
    if (p.pos_table && (!p.positions || p.max_pos < 1)) return fail("telb_stream_sandwich: position rows need positions");
    if (p.norm && !p.h) return fail("telb_stream_sandwich: a norm has an output");
    if (p.shift && (!p.norm || !p.state)) return fail("telb_stream_sandwich: a shift has a norm and a state");
    if (p.x_out && p.x_out == p.x_in) return fail("telb_stream_sandwich: rows are not advanced in place");
    return dtype == 2 ? run_sandwich<float>(p, warp_rows, stream) : run_sandwich<__nv_bfloat16>(p, warp_rows, stream);
}
