// The fp32 residual stream of blocks that are normed behind their sublayers.  What lies between two sublayers:
//
//   source   x = table[id] + bigram[row(previous id, id)] (first call) or the running fp32 stream
//   update   x += y / rms(y) * w                       y: sublayer output; each of `groups` equal parts of a row has its own rms.  With
//                                                       `sums` the row is first divided by the rms of the row that was projected to y
//   output   h = x                                     for a feed-forward
//            h = x / rms(x) * w'                       same parts, for the head
//            h = x + Σ_j c[j] ∘ x_{t - taps + 1 + j}   causal convolution over time, for a mixer
//
// Stream, norms, convolution and its history are fp32; y, the tables and h have the activation type.
//
// post_row_kernel does all of it for one row per CTA (steps of many rows update the stream with one row per warp instead: post_warp_kernel),
// the convolution included when every sequence has one row (decoding: the rows in front
// are the history of its seat).  Longer portions take the convolution from the advanced stream in a second launch (post_conv_kernel):
// blocks of rows count from the start of a sequence's portion, only the first one needs the history row of the seat, and the CTA that owns
// it also writes the new history, so no CTA reads what another one of its launch writes.  The last token of a sequence is kept likewise.
#include "host_utils.h"
#include "stream_common.cuh"

namespace telb {

// Host mirror: ops/cuda.py (StreamPostParams).
struct StreamPostParams {
    const int* ids;              // embedding source, or null
    const void* table;           // [vocab, width]
    const void* bigram;          // [buckets + 1, width] or null
    int* last;                   // [slots]: last token of each sequence (with bigram)
    const float* x_in;           // [T, width] when ids is null
    const void* delta;           // [T, width] or null
    const float* weight;         // [width], with delta
    const float* sums;           // [T, n_sums]: sums of squares of the row behind delta, or null
    const float* conv;           // [taps, width] or null
    float* history;              // [slots, taps - 1, width], oldest first
    const float* out_norm;       // [width] or null
    float* x_out;                // [T, width]
    void* h;                     // [T, width]
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* slot_ids;
    const int* seq_ids;
    long long buckets, mul_prev, mul_cur;
    int vocab, width, groups, tokens, taps, block_rows, n_sums, sum_count;      // sum_count: features of that row
    float eps;
};

constexpr int kPostMaxGroups = 256;
constexpr int kPostMaxTaps = 8;

// One over the root mean square of the row that was projected to row `row` of delta (every warp computes it).
__device__ __forceinline__ float row_scale(const StreamPostParams& p, size_t row) {
    float s = 0.f;
    for (int i = threadIdx.x & 31; i < p.n_sums; i += 32) s += p.sums[row * p.n_sums + i];
    return 1.f / sqrtf(post_warp_sum(s) / p.sum_count + p.eps);
}

// Divide every part of R rows by its root mean square, in place.  Thread i of N holds features 4 (e N + i) .. + 3 of each row.  Parts that are
// multiples of 128 features: a warp's four-feature vectors lie in one part, so warp sums are enough (`red` alternates between two
// buffers, one barrier); other parts: sums of squares of four features (or single ones) go through shared memory.
template <int N, int E, int R>
__device__ __forceinline__ void norm_parts(const StreamPostParams& p, float (&d)[R][E][4], float* red, int turn) {
    constexpr int kWarps = N / 32, kSlots = E * kWarps;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int part = p.width / p.groups;
    if (part % 128 == 0) {
        float* buf = red + (turn & 1) * R * kSlots;
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const float s = post_warp_sum(d[r][e][0] * d[r][e][0] + d[r][e][1] * d[r][e][1] + d[r][e][2] * d[r][e][2] + d[r][e][3] * d[r][e][3]);
                if (lane == 0) buf[r * kSlots + e * kWarps + warp] = s;
            }
        __syncthreads();
        const int n = part / 128;
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int c = (e * N + tid) * 4;
            if (c >= p.width) break;
            const float* src = buf + c / part * n;
            float s[R];
#pragma unroll
            for (int r = 0; r < R; ++r) s[r] = 0.f;
            for (int i = 0; i < n; ++i)
#pragma unroll
                for (int r = 0; r < R; ++r) s[r] += src[r * kSlots + i];
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float inv = 1.f / sqrtf(s[r] / part + p.eps);
#pragma unroll
                for (int i = 0; i < 4; ++i) d[r][e][i] *= inv;
            }
        }
        return;
    }
    const int unit = part % 4 == 0 ? 4 : 1, per_row = p.width / unit, n = part / unit;
    float* sums = red + R * per_row;
    __syncthreads();                                      // the previous call's readers are done
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int c = (e * N + tid) * 4;
            if (c >= p.width) break;
            if (unit == 4) {
                red[r * per_row + c / 4] = d[r][e][0] * d[r][e][0] + d[r][e][1] * d[r][e][1] + d[r][e][2] * d[r][e][2] + d[r][e][3] * d[r][e][3];
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) red[r * per_row + c + i] = d[r][e][i] * d[r][e][i];
            }
        }
    __syncthreads();
    for (int k = warp; k < R * p.groups; k += kWarps) {
        const float* src = red + (k / p.groups) * per_row + (k % p.groups) * n;
        float s = 0.f;
        for (int i = lane; i < n; i += 32) s += src[i];
        s = post_warp_sum(s);
        if (lane == 0) sums[k] = 1.f / sqrtf(s / part + p.eps);
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int c = (e * N + tid) * 4;
            if (c >= p.width) break;
#pragma unroll
            for (int i = 0; i < 4; ++i) d[r][e][i] *= sums[r * p.groups + (c + i) / part];
        }
}

// One CTA per row.  IDS: the stream starts from token ids.  CONV: every sequence has at most one row, h is the convolved stream.
template <typename T, int N, int E, bool CONV, bool IDS>
__global__ void __launch_bounds__(N) post_row_kernel(const __grid_constant__ StreamPostParams p) {
    pdl_prologue();
    extern __shared__ float red[];
    const size_t row = (size_t)blockIdx.x * p.width;
    const int tid = threadIdx.x, t = blockIdx.x;
    float x[1][E][4], d[1][E][4], w[E][4], conv[E][4];
    int slot = 0;
    bool fresh = true;
    if (CONV || IDS) {
        const int seq = p.seq_ids[t];
        slot = p.slot_ids[seq];
        fresh = p.past_len[seq] <= 0;
    }
    float* hist = CONV ? p.history + (size_t)slot * (p.taps - 1) * p.width : nullptr;
    if constexpr (CONV) {                                 // what the convolution takes from the rows in front; the history moves up
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int c = (e * N + tid) * 4;
#pragma unroll
            for (int i = 0; i < 4; ++i) conv[e][i] = 0.f;
            if (c >= p.width) continue;
            float old[kPostMaxTaps - 1][4], tap[kPostMaxTaps - 1][4];
#pragma unroll
            for (int j = 0; j < kPostMaxTaps - 1; ++j) {
                if (j >= p.taps - 1) break;
                get4(p.conv + (size_t)j * p.width + c, tap[j]);
                if (fresh) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) old[j][i] = 0.f;
                } else {
                    get4(hist + (size_t)j * p.width + c, old[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < kPostMaxTaps - 1; ++j) {
                if (j >= p.taps - 1) break;
#pragma unroll
                for (int i = 0; i < 4; ++i) conv[e][i] = fmaf(tap[j][i], old[j][i], conv[e][i]);
                if (j > 0) put4(hist + (size_t)(j - 1) * p.width + c, old[j]);
            }
        }
    }
    int id = 0;
    long long pair = 0;
    if constexpr (IDS) {
        const int seq = p.seq_ids[t], t0 = p.q_start[seq];
        id = min(max(p.ids[t], 0), p.vocab - 1);
        if (p.bigram) {
            const int prev = t > t0 ? p.ids[t - 1] : fresh ? -1 : p.last[slot];
            pair = p.buckets;
            if (prev >= 0) {
                pair = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
                if (pair < 0) pair += p.buckets;
            }
            if (t == t0) {                                // the CTA that reads the last token also replaces it
                __syncthreads();
                if (tid == 0) p.last[slot] = p.ids[t0 + p.q_len[seq] - 1];
            }
        }
    }
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + tid) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) x[0][e][i] = d[0][e][i] = 0.f;
        if (c >= p.width) continue;
        if constexpr (IDS) {
            get4(reinterpret_cast<const T*>(p.table) + (size_t)id * p.width + c, x[0][e]);
            if (p.bigram) {
                float b[4];
                get4(reinterpret_cast<const T*>(p.bigram) + (size_t)pair * p.width + c, b);
#pragma unroll
                for (int i = 0; i < 4; ++i) x[0][e][i] += b[i];
            }
        } else {
            get4(p.x_in + row + c, x[0][e]);
            if (p.delta) {
                get4(reinterpret_cast<const T*>(p.delta) + row + c, d[0][e]);
                get4(p.weight + c, w[e]);
            }
        }
    }
    if constexpr (!IDS) {
        if (p.delta) {
            if (p.sums) {
                const float scale = row_scale(p, t);
#pragma unroll
                for (int e = 0; e < E; ++e)
#pragma unroll
                    for (int i = 0; i < 4; ++i) d[0][e][i] *= scale;
            }
            norm_parts<N, E, 1>(p, d, red, 0);
        }
    }
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + tid) * 4;
        if (c >= p.width) break;
        if (!IDS && p.delta) {
#pragma unroll
            for (int i = 0; i < 4; ++i) x[0][e][i] = fmaf(d[0][e][i], w[e][i], x[0][e][i]);
        }
        put4(p.x_out + row + c, x[0][e]);
        if constexpr (CONV) {
            float tap[4], y[4];
            get4(p.conv + (size_t)(p.taps - 1) * p.width + c, tap);
#pragma unroll
            for (int i = 0; i < 4; ++i) y[i] = x[0][e][i] + fmaf(tap[i], x[0][e][i], conv[e][i]);
            put4(reinterpret_cast<T*>(p.h) + row + c, y);
            if (p.taps > 1) put4(hist + (size_t)(p.taps - 2) * p.width + c, x[0][e]);
        } else if (p.h && !p.out_norm) {
            put4(reinterpret_cast<T*>(p.h) + row + c, x[0][e]);
        }
    }
    if (CONV || !p.out_norm) return;
    norm_parts<N, E, 1>(p, x, red, 1);
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + tid) * 4;
        if (c >= p.width) break;
        float g[4];
        get4(p.out_norm + c, g);
#pragma unroll
        for (int i = 0; i < 4; ++i) g[i] *= x[0][e][i];
        put4(reinterpret_cast<T*>(p.h) + row + c, g);
    }
}

// Many rows: one warp per row, x += norm(y) w, h = x.  Parts are multiples of 128 features, so a vector of a warp (four features per lane)
// lies in one part; E vectors of the row stay in registers.
constexpr int kPostWarps = 8;
template <typename T, int E>
__global__ void __launch_bounds__(kPostWarps * 32, 2) post_warp_kernel(const __grid_constant__ StreamPostParams p) {
    pdl_prologue();
    __shared__ float part_inv[kPostWarps][E];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * kPostWarps + warp;
    if (t >= p.tokens) return;
    const size_t row = (size_t)t * p.width + lane * 4;
    const int live = p.width / 128, n = live / p.groups;  // vectors of a row and of a part
    T raw[E][4];
    float x[E][4];
#pragma unroll
    for (int e = 0; e < E; ++e) {
        if (e >= live) break;
        const T* src = reinterpret_cast<const T*>(p.delta) + row + e * 128;
        if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(raw[e]) = *reinterpret_cast<const float4*>(src);
        else *reinterpret_cast<uint2*>(raw[e]) = *reinterpret_cast<const uint2*>(src);
        get4(p.x_in + row + e * 128, x[e]);
    }
    const float scale = p.sums ? row_scale(p, t) : 1.f;
#pragma unroll
    for (int e = 0; e < E; ++e) {
        if (e >= live) break;
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float v = Cvt<T>::to_f(raw[e][i]) * scale;
            s = fmaf(v, v, s);
        }
        s = post_warp_sum(s);
        if (lane == 0) part_inv[warp][e] = s;
    }
    __syncwarp();
    float inv = 0.f;
    if (lane < live) {
        for (int i = lane / n * n; i < lane / n * n + n; ++i) inv += part_inv[warp][i];
        inv = scale / sqrtf(inv / (n * 128) + p.eps);
    }
    __syncwarp();
    if (lane < live) part_inv[warp][lane] = inv;
    __syncwarp();
#pragma unroll
    for (int e = 0; e < E; ++e) {
        if (e >= live) break;
        const float f = part_inv[warp][e];
        float w[4];
        get4(p.weight + lane * 4 + e * 128, w);
#pragma unroll
        for (int i = 0; i < 4; ++i) x[e][i] = fmaf(Cvt<T>::to_f(raw[e][i]) * f, w[i], x[e][i]);
        put4(p.x_out + row + e * 128, x[e]);
        if (p.h) put4(reinterpret_cast<T*>(p.h) + row + e * 128, x[e]);
    }
}

// Convolution of the advanced stream (p.x_out) over blocks of rows; a thread walks four features down a block.  W: window of the taps
// (right-aligned), R: rows whose loads are in flight together.
constexpr int kConvThreads = 128;
template <typename T, int W>
__global__ void __launch_bounds__(kConvThreads) post_conv_kernel(const __grid_constant__ StreamPostParams p) {
    constexpr int R = 8;
    pdl_prologue();
    const int c = (blockIdx.y * kConvThreads + threadIdx.x) * 4, pad = W - p.taps, front = p.taps - 1;
    if (c >= p.width) return;
    float taps[W][4];
#pragma unroll
    for (int j = 0; j < W; ++j) {
#pragma unroll
        for (int i = 0; i < 4; ++i) taps[j][i] = 0.f;
        if (j >= pad) get4(p.conv + (size_t)(j - pad) * p.width + c, taps[j]);
    }
    const int lo = blockIdx.x * p.block_rows, hi = min(p.tokens, lo + p.block_rows);
    for (int t = lo; t < hi;) {
        const int seq = p.seq_ids[t], t0 = p.q_start[seq], i0 = t - t0, ql = p.q_len[seq];
        if (i0 % p.block_rows) {                          // inside a block that starts in an earlier range
            t += min(p.block_rows - i0 % p.block_rows, ql - i0);
            continue;
        }
        const int n = min(p.block_rows, ql - i0), slot = p.slot_ids[seq];
        const bool first = i0 == 0, fresh = p.past_len[seq] <= 0;
        const float* src = p.x_out + (size_t)t0 * p.width + c;
        T* dst = reinterpret_cast<T*>(p.h) + (size_t)t0 * p.width + c;
        float* state = p.history + (size_t)slot * front * p.width + c;
        // row of the portion, or of the history in front of it
        auto row_at = [&](int j, float (&v)[4]) {
            if (j >= 0) {
                get4(src + (size_t)j * p.width, v);
            } else if (!fresh && j >= -front) {
                get4(state + (size_t)(front + j) * p.width, v);
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) v[i] = 0.f;
            }
        };
        float rows[W - 1 + R][4];
#pragma unroll
        for (int j = 0; j < W - 1; ++j) row_at(i0 - (W - 1) + j, rows[j]);
        for (int j0 = i0; j0 < i0 + n; j0 += R) {
#pragma unroll
            for (int r = 0; r < R; ++r)
                if (j0 + r < i0 + n) get4(src + (size_t)(j0 + r) * p.width, rows[W - 1 + r]);
#pragma unroll
            for (int r = 0; r < R; ++r) {
                if (j0 + r >= i0 + n) break;
                float y[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    float s = 0.f;
#pragma unroll
                    for (int k = 0; k < W; ++k) s = fmaf(taps[k][i], rows[r + k][i], s);
                    y[i] = rows[r + W - 1][i] + s;
                }
                put4(dst + (size_t)(j0 + r) * p.width, y);
            }
#pragma unroll
            for (int j = 0; j < W - 1; ++j)
#pragma unroll
                for (int i = 0; i < 4; ++i) rows[j][i] = rows[j + R][i];
        }
        if (first) {                                      // new history: the last rows of the portion, behind it what is left of the old one
            float keep[W - 1][4];
#pragma unroll
            for (int j = 0; j < W - 1; ++j)
                if (j >= pad) row_at(ql - (W - 1) + j, keep[j]);
#pragma unroll
            for (int j = 0; j < W - 1; ++j)
                if (j >= pad) put4(state + (size_t)(j - pad) * p.width, keep[j]);
        }
        t += n;
    }
}

template <typename T, int N, int E>
static int launch_row(const StreamPostParams& p, bool conv, cudaStream_t stream) {
    const int part = p.width / p.groups;
    const size_t smem = (part % 128 == 0 ? (size_t)2 * E * (N / 32) : (size_t)(part % 4 == 0 ? p.width / 4 : p.width) + p.groups) * sizeof(float);
    if (smem > 48 * 1024) return fail("telb_stream_post: parts of this size are not built for rows this wide");
#define TELB_ROW(CONV_, IDS_) TELB_LAUNCH("post_row_kernel", (post_row_kernel<T, N, E, CONV_, IDS_>), dim3(p.tokens), dim3(N), smem, stream, p)
    if (conv && p.ids) TELB_ROW(true, true);
    else if (conv) TELB_ROW(true, false);
    else if (p.ids) TELB_ROW(false, true);
    else TELB_ROW(false, false);
#undef TELB_ROW
    TELB_CHECK_LAUNCH("post_row_kernel");
    return 0;
}

template <typename T, int E>
static int launch_warp(const StreamPostParams& p, cudaStream_t stream) {
    TELB_LAUNCH("post_warp_kernel", (post_warp_kernel<T, E>), dim3((p.tokens + kPostWarps - 1) / kPostWarps), dim3(kPostWarps * 32), 0, stream, p);
    TELB_CHECK_LAUNCH("post_warp_kernel");
    return 0;
}

template <typename T>
static int run_row(const StreamPostParams& p, bool conv, cudaStream_t stream) {
    if (p.tokens >= kPostWarps * sm_count() && p.delta && !conv && !p.out_norm && p.width / p.groups % 128 == 0 && p.width <= 4096) {
        if (p.width <= 1024) return launch_warp<T, 8>(p, stream);
        if (p.width <= 2048) return launch_warp<T, 16>(p, stream);
        return launch_warp<T, 32>(p, stream);
    }
    if (p.width <= 1024) return launch_row<T, 256, 1>(p, conv, stream);
    if (p.width <= 2048) return launch_row<T, 256, 2>(p, conv, stream);
    if (p.width <= 4096) return launch_row<T, 512, 2>(p, conv, stream);
    return launch_row<T, 1024, 4>(p, conv, stream);
}

template <typename T>
static int run_post(const StreamPostParams& p, int one_row, cudaStream_t stream) {
    if (!p.conv || one_row) return run_row<T>(p, p.conv != nullptr, stream);
    StreamPostParams first = p;
    first.h = nullptr;
    if (run_row<T>(first, false, stream)) return -1;
    const dim3 grid((p.tokens + p.block_rows - 1) / p.block_rows, (p.width / 4 + kConvThreads - 1) / kConvThreads);
    if (p.taps <= 4) TELB_LAUNCH("post_conv_kernel", (post_conv_kernel<T, 4>), grid, dim3(kConvThreads), 0, stream, p);
    else TELB_LAUNCH("post_conv_kernel", (post_conv_kernel<T, 8>), grid, dim3(kConvThreads), 0, stream, p);
    TELB_CHECK_LAUNCH("post_conv_kernel");
    return 0;
}

}  // namespace telb

using namespace telb;

// dtype: 1 bf16, 2 fp32 (of the tables, delta and h; the un-normed stream needs bf16's range).  one_row: every sequence has at most one row.
// Otherwise a convolution goes over blocks of p->block_rows rows (at least 8).
extern "C" int telb_stream_post(const StreamPostParams* pp, int one_row, int dtype, cudaStream_t stream) {
    const StreamPostParams& p = *pp;
    if (p.tokens <= 0) return 0;
    if (p.width % 4 || p.width > 16 * 1024) return fail("telb_stream_post: width must be a multiple of 4 and at most 16384");
    if (p.groups < 1 || p.groups > kPostMaxGroups || p.width % p.groups) return fail("telb_stream_post: 1 to 256 groups that divide the width");
    if (!p.ids == !p.x_in) return fail("telb_stream_post: either ids or a stream");
    if (p.delta && (!p.weight || p.ids)) return fail("telb_stream_post: an update has a weight and a stream to join");
    if (p.sums && (!p.delta || p.n_sums < 1 || p.sum_count < 1)) return fail("telb_stream_post: sums belong to an update");
    if (p.bigram && (!p.last || p.buckets < 1)) return fail("telb_stream_post: the bigram table needs buckets and last tokens");
    if (p.conv) {
        if (p.taps < 1 || p.taps > kPostMaxTaps) return fail("telb_stream_post: convolutions have 1 to 8 taps");
        if (p.taps > 1 && !p.history) return fail("telb_stream_post: the convolution keeps a history");
        if (!one_row && p.block_rows < kPostMaxTaps) return fail("telb_stream_post: blocks of at least 8 rows");
        if (p.out_norm) return fail("telb_stream_post: a convolution or a norm, not both");
    }
    return dtype == 2 ? run_post<float>(p, one_row, stream) : run_post<__nv_bfloat16>(p, one_row, stream);
}
