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
// what another one of its launch writes, and the rows x are never advanced in place.
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

// Sum over the CTA's N threads; `red` holds two turns of N / 32 warp sums, used alternately (one barrier per sum).
template <int N>
__device__ __forceinline__ float block_total(float v, float* red, int& turn) {
    v = post_warp_sum(v);
    float* buf = red + (turn & 1) * (N / 32);
    ++turn;
    if ((threadIdx.x & 31) == 0) buf[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < N / 32; ++w) s += buf[w];
    return s;
}

// What a row is made of, fetched ahead of the sums of the row before.
template <typename T, int E>
struct RowParts {
    float x[E][4], d[E][4];
};

template <typename T, int N, int E>
__device__ __forceinline__ void fetch_row(const StreamSandwichParams& p, int t, RowParts<T, E>& r) {
    const int id = p.ids ? min(max(p.ids[t], 0), p.vocab - 1) : 0;
    const int pos = p.pos_table ? min(max(p.positions[t], 0), p.max_pos - 1) : 0;
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + threadIdx.x) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) r.x[e][i] = r.d[e][i] = 0.f;
        if (c >= p.width) continue;
        if (p.ids) get4(reinterpret_cast<const T*>(p.table) + (size_t)id * p.width + c, r.x[e]);
        else get4(p.x_in + (size_t)t * p.width + c, r.x[e]);
        if (p.pos_table) {
            float v[4];
            get4(reinterpret_cast<const T*>(p.pos_table) + (size_t)pos * p.width + c, v);
#pragma unroll
            for (int i = 0; i < 4; ++i) r.x[e][i] += v[i];
        }
        if (p.y) get4(reinterpret_cast<const T*>(p.y) + (size_t)t * p.width + c, r.d[e]);
    }
    if (p.e) {
        for (int k = 0; k < p.top_k; ++k) {
            const int row = p.dst_row[(size_t)t * p.top_k + k];
            if (row < 0) continue;
            const float w = p.topk_w[(size_t)t * p.top_k + k];
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int c = (e * N + threadIdx.x) * 4;
                if (c >= p.width) break;
                float v[4];
                get4(reinterpret_cast<const T*>(p.e) + (size_t)row * p.lde + c, v);
#pragma unroll
                for (int i = 0; i < 4; ++i) r.d[e][i] = fmaf(w, v[i], r.d[e][i]);
            }
        }
    }
}

// Advances the row in place (stored when `own`) and leaves its norm, without the weight, in r.d.
template <typename T, int N, int E>
__device__ __forceinline__ void advance_row(const StreamSandwichParams& p, int t, bool own, RowParts<T, E>& r, const float (&post)[E][4], float* red, int& turn) {
    if (p.y || p.e) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < E; ++e)
#pragma unroll
            for (int i = 0; i < 4; ++i) ss = fmaf(r.d[e][i], r.d[e][i], ss);
        const float f = p.mult / sqrtf(block_total<N>(ss, red, turn) / p.width + p.eps);
#pragma unroll
        for (int e = 0; e < E; ++e)
#pragma unroll
            for (int i = 0; i < 4; ++i) r.x[e][i] = fmaf(r.d[e][i] * f, post[e][i], r.x[e][i]);
    }
    if (own && p.x_out) {
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int c = (e * N + threadIdx.x) * 4;
            if (c < p.width) put4(p.x_out + (size_t)t * p.width + c, r.x[e]);
        }
    }
    if (!p.norm) return;
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e)
#pragma unroll
        for (int i = 0; i < 4; ++i) ss = fmaf(r.x[e][i], r.x[e][i], ss);
    const float inv = 1.f / sqrtf(block_total<N>(ss, red, turn) / p.width + p.eps);
#pragma unroll
    for (int e = 0; e < E; ++e)
#pragma unroll
        for (int i = 0; i < 4; ++i) r.d[e][i] = r.x[e][i] * inv;
}

template <int N, int E>
__device__ __forceinline__ void load_weight(const float* w, int width, float (&v)[E][4]) {
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + threadIdx.x) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) v[e][i] = 0.f;
        if (w && c < width) get4(w + c, v[e]);
    }
}

// Every CTA takes the blocks that start in its range of block_rows rows (blocks count from the start of a sequence's portion).
template <typename T, int N, int E, bool SHIFT>
__global__ void __launch_bounds__(N) stream_sandwich_kernel(const __grid_constant__ StreamSandwichParams p) {
    pdl_prologue();
    __shared__ float red[2 * (N / 32)];
    const int tid = threadIdx.x;
    int turn = 0;
    float post[E][4], norm[E][4], shift[E][4];
    load_weight<N, E>(p.post, p.width, post);
    load_weight<N, E>(p.norm, p.width, norm);
    if constexpr (SHIFT) load_weight<N, E>(p.shift, p.width, shift);
    RowParts<T, E> r, next;
    const int lo = blockIdx.x * p.block_rows, hi = min(p.tokens, lo + p.block_rows);
    if constexpr (!SHIFT) {
        fetch_row<T, N, E>(p, lo, next);
        for (int t = lo; t < hi; ++t) {
            r = next;
            if (t + 1 < hi) fetch_row<T, N, E>(p, t + 1, next);
            advance_row<T, N, E>(p, t, true, r, post, red, turn);
            if (!p.norm) continue;
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int c = (e * N + tid) * 4;
                if (c >= p.width) break;
#pragma unroll
                for (int i = 0; i < 4; ++i) r.d[e][i] *= norm[e][i];
                put4(reinterpret_cast<T*>(p.h) + (size_t)t * p.width + c, r.d[e]);
            }
        }
    } else {
        float before[E][4];                               // normed row in front of the current one, with its weight
        auto keep = [&](const RowParts<T, E>& row) {
#pragma unroll
            for (int e = 0; e < E; ++e)
#pragma unroll
                for (int i = 0; i < 4; ++i) before[e][i] = row.d[e][i] * norm[e][i];
        };
        for (int t = lo; t < hi;) {
            const int seq = p.seq_ids[t], t0 = p.q_start[seq], i0 = t - t0, ql = p.q_len[seq];
            if (i0 % p.block_rows) {                      // inside a block that starts in an earlier range
                t += min(p.block_rows - i0 % p.block_rows, ql - i0);
                continue;
            }
            const int end = t + min(p.block_rows, ql - i0);
            float* state = p.state + (size_t)p.slot_ids[seq] * p.width;
            if (i0 > 0) {
                fetch_row<T, N, E>(p, t - 1, r);
                fetch_row<T, N, E>(p, t, next);
                advance_row<T, N, E>(p, t - 1, false, r, post, red, turn);
                keep(r);
            } else {
                fetch_row<T, N, E>(p, t, next);
                load_weight<N, E>(p.past_len[seq] > 0 ? state : nullptr, p.width, before);
            }
            for (int u = t; u < end; ++u) {
                r = next;
                if (u + 1 < end) fetch_row<T, N, E>(p, u + 1, next);
                advance_row<T, N, E>(p, u, true, r, post, red, turn);
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    const int c = (e * N + tid) * 4;
                    float v[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float h = r.d[e][i] * norm[e][i];
                        v[i] = fmaf(before[e][i] - h, shift[e][i], h);
                        before[e][i] = h;
                    }
                    if (c < p.width) put4(reinterpret_cast<T*>(p.h) + (size_t)u * p.width + c, v);
                }
            }
            if (i0 == 0) {                                // the state moves to the portion's last row
                if (end < t0 + ql) {
                    fetch_row<T, N, E>(p, t0 + ql - 1, r);
                    advance_row<T, N, E>(p, t0 + ql - 1, false, r, post, red, turn);
                    keep(r);
                }
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    const int c = (e * N + tid) * 4;
                    if (c < p.width) put4(state + c, before[e]);
                }
            }
            t = end;
        }
    }
}

template <typename T, int N, int E>
static int launch_sandwich(const StreamSandwichParams& p, cudaStream_t stream) {
    const dim3 grid((p.tokens + p.block_rows - 1) / p.block_rows);
    if (p.shift) TELB_LAUNCH("stream_sandwich_kernel", (stream_sandwich_kernel<T, N, E, true>), grid, dim3(N), 0, stream, p);
    else TELB_LAUNCH("stream_sandwich_kernel", (stream_sandwich_kernel<T, N, E, false>), grid, dim3(N), 0, stream, p);
    TELB_CHECK_LAUNCH("stream_sandwich_kernel");
    return 0;
}

template <typename T>
static int run_sandwich(const StreamSandwichParams& p, cudaStream_t stream) {
    if (p.width <= 512) return launch_sandwich<T, 128, 1>(p, stream);
    if (p.width <= 1024) return launch_sandwich<T, 256, 1>(p, stream);
    if (p.width <= 2048) return launch_sandwich<T, 256, 2>(p, stream);
    if (p.width <= 4096) return launch_sandwich<T, 512, 2>(p, stream);
    return launch_sandwich<T, 1024, 4>(p, stream);
}

}  // namespace telb

using namespace telb;

// dtype: 0 fp16, 1 bf16, 2 fp32 (of the tables, y, e and h).
extern "C" int telb_stream_sandwich(const StreamSandwichParams* pp, int dtype, cudaStream_t stream) {
    const StreamSandwichParams& p = *pp;
    if (p.tokens <= 0) return 0;
    if (p.width % 4 || p.width > 16 * 1024) return fail("telb_stream_sandwich: width must be a multiple of 4 and at most 16384");
    if (!p.ids == !p.x_in) return fail("telb_stream_sandwich: either ids or a stream");
    if (p.block_rows < 1) return fail("telb_stream_sandwich: blocks of at least one row");
    if ((p.y || p.e) && !p.post) return fail("telb_stream_sandwich: an update has a weight");
    if (p.e && (!p.dst_row || !p.topk_w || p.lde % 4)) return fail("telb_stream_sandwich: expert rows come with their tables");
    if (p.pos_table && (!p.positions || p.max_pos < 1)) return fail("telb_stream_sandwich: position rows need positions");
    if (p.norm && !p.h) return fail("telb_stream_sandwich: a norm has an output");
    if (p.shift && (!p.norm || !p.state)) return fail("telb_stream_sandwich: a shift has a norm and a state");
    if (p.x_out && p.x_out == p.x_in) return fail("telb_stream_sandwich: rows are not advanced in place");
    if (dtype == 2) return run_sandwich<float>(p, stream);
    return dtype == 1 ? run_sandwich<__nv_bfloat16>(p, stream) : run_sandwich<__half>(p, stream);
}
