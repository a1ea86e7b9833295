// The fp32 residual stream of blocks that are normed behind their sublayers.  Everything that lies between two sublayers is one kernel:
//
//   source   x = table[id] + bigram[row(previous id, id)] (first call) or the running fp32 stream
//   update   x += y / rms(y) * w                       y: sublayer output; each of `groups` equal parts of a row has its own rms.  With
//                                                       `sums` the row is first divided by the rms of the row that was projected to y
//   output   h = x                                     for a feed-forward                                  (post_row_kernel)
//            h = x / rms(x) * w'                       same parts, for the head                            (post_row_kernel)
//            h = x + Σ_j c[j] ∘ x_{t - taps + 1 + j}   causal convolution over time, for a mixer           (post_conv_kernel)
//
// Stream, norms, convolution and its history are fp32; y, the tables and h have the activation type.
//
// The convolution looks at rows that other CTAs advance, so a CTA takes a block of rows and advances the taps - 1 rows in front of it
// once more (reads only).  Blocks count from the start of a sequence's portion: only the first block of a portion needs the history
// row of its seat, and the CTA that owns it also writes the new history (the last rows of the portion, advanced once more when they
// lie in another block), so no CTA reads what another one writes.  The same holds for the last token of the sequence.
#include "host_utils.h"
#include "tc5_common.cuh"

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

template <typename T>
__device__ __forceinline__ void get4(const T* p, float (&v)[4]) {
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
template <typename T>
__device__ __forceinline__ void put4(T* p, const float (&v)[4]) {
    if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        uint2 u;
        u.x = Cvt<T>::pack2(v[0], v[1]);
        u.y = Cvt<T>::pack2(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = u;
    }
}
__device__ __forceinline__ float post_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// One over the root mean square of the row that was projected to row `row` of delta (every warp computes it).
__device__ __forceinline__ float row_scale(const StreamPostParams& p, size_t row) {
    if (!p.sums) return 1.f;
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

// One CTA per row: x += norm(y) w, h = x or norm(x) w'.
template <typename T, int N, int E>
__global__ void __launch_bounds__(N) post_row_kernel(const __grid_constant__ StreamPostParams p) {
    pdl_prologue();
    extern __shared__ float red[];
    const size_t row = (size_t)blockIdx.x * p.width;
    const int tid = threadIdx.x;
    float x[1][E][4], d[1][E][4];
    const float scale = row_scale(p, blockIdx.x);
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + tid) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) x[0][e][i] = d[0][e][i] = 0.f;
        if (c >= p.width) continue;
        get4(p.x_in + row + c, x[0][e]);
        if (p.delta) get4(reinterpret_cast<const T*>(p.delta) + row + c, d[0][e]);
#pragma unroll
        for (int i = 0; i < 4; ++i) d[0][e][i] *= scale;
    }
    if (p.delta) norm_parts<N, E, 1>(p, d, red, 0);
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + tid) * 4;
        if (c >= p.width) break;
        if (p.delta) {
            float w[4];
            get4(p.weight + c, w);
#pragma unroll
            for (int i = 0; i < 4; ++i) x[0][e][i] = fmaf(d[0][e][i], w[i], x[0][e][i]);
        }
        put4(p.x_out + row + c, x[0][e]);
        if (!p.out_norm) put4(reinterpret_cast<T*>(p.h) + row + c, x[0][e]);
    }
    if (!p.out_norm) return;
    norm_parts<N, E, 1>(p, x, red, 1);
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + tid) * 4;
        if (c >= p.width) break;
        float w[4];
        get4(p.out_norm + c, w);
#pragma unroll
        for (int i = 0; i < 4; ++i) w[i] *= x[0][e][i];
        put4(reinterpret_cast<T*>(p.h) + row + c, w);
    }
}

// Blocks of rows with the convolution; W: window of the taps (right-aligned), R: rows at a time.
template <typename T, int N, int E, int W>
__global__ void __launch_bounds__(N) post_conv_kernel(const __grid_constant__ StreamPostParams p) {
    constexpr int R = 2;
    pdl_prologue();
    extern __shared__ float red[];
    const int tid = threadIdx.x, pad = W - p.taps, past_rows = p.taps - 1;
    float taps[W][E][4], nw[E][4];
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = (e * N + tid) * 4;
#pragma unroll
        for (int j = 0; j < W; ++j) {
#pragma unroll
            for (int i = 0; i < 4; ++i) taps[j][e][i] = 0.f;
            if (j >= pad && c < p.width) get4(p.conv + (size_t)(j - pad) * p.width + c, taps[j][e]);
        }
        if (p.delta && c < p.width) get4(p.weight + c, nw[e]);
    }
    int turn = 0;
    const int lo = blockIdx.x * p.block_rows, hi = min(p.tokens, lo + p.block_rows);
    for (int t = lo; t < hi;) {
        const int seq = p.seq_ids[t], t0 = p.q_start[seq], i0 = t - t0, ql = p.q_len[seq];
        if (i0 % p.block_rows) {                          // inside a block that starts in an earlier range
            t += min(p.block_rows - i0 % p.block_rows, ql - i0);
            continue;
        }
        const int n = min(p.block_rows, ql - i0), slot = p.slot_ids[seq];
        const bool first = i0 == 0, fresh = p.past_len[seq] <= 0;
        float* hist_row = p.history + (size_t)slot * past_rows * p.width;
        float hist[W - 1][E][4];                          // the rows in front, newest last
#pragma unroll
        for (int j = 0; j < W - 1; ++j)
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int c = (e * N + tid) * 4;
#pragma unroll
                for (int i = 0; i < 4; ++i) hist[j][e][i] = 0.f;
                if (first && !fresh && j >= pad && c < p.width) get4(hist_row + (size_t)(j - pad) * p.width + c, hist[j][e]);
            }
        // rows j0 .. j1 - 1 of the portion pass through, those from `emit` on are written: the block behind the rows in front of it, then,
        // for the history, the portion's last rows when they lie in another block
        for (int pass = 0; pass < (first && n < ql ? 2 : 1); ++pass) {
            const int j0 = pass ? ql - past_rows : first ? i0 : i0 - past_rows;
            const int j1 = pass ? ql : i0 + n, emit = pass ? ql : i0;
            for (int j = j0; j < j1; j += R) {
                float x[R][E][4], d[R][E][4];
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const bool live = j + r < j1;
                    const size_t row = (size_t)(t0 + j + r) * p.width;
                    const float scale = live ? row_scale(p, t0 + j + r) : 1.f;
                    int id = 0;
                    long long pair = 0;
                    if (p.ids && live) {
                        id = min(max(p.ids[t0 + j + r], 0), p.vocab - 1);
                        if (p.bigram) {
                            const int prev = j + r > 0 ? p.ids[t0 + j + r - 1] : fresh ? -1 : p.last[slot];
                            pair = p.buckets;
                            if (prev >= 0) {
                                pair = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
                                if (pair < 0) pair += p.buckets;
                            }
                        }
                    }
#pragma unroll
                    for (int e = 0; e < E; ++e) {
                        const int c = (e * N + tid) * 4;
#pragma unroll
                        for (int i = 0; i < 4; ++i) x[r][e][i] = d[r][e][i] = 0.f;
                        if (!live || c >= p.width) continue;
                        if (p.ids) {
                            get4(reinterpret_cast<const T*>(p.table) + (size_t)id * p.width + c, x[r][e]);
                            if (p.bigram) {
                                float b[4];
                                get4(reinterpret_cast<const T*>(p.bigram) + (size_t)pair * p.width + c, b);
#pragma unroll
                                for (int i = 0; i < 4; ++i) x[r][e][i] += b[i];
                            }
                        } else {
                            get4(p.x_in + row + c, x[r][e]);
                        }
                        if (p.delta) get4(reinterpret_cast<const T*>(p.delta) + row + c, d[r][e]);
#pragma unroll
                        for (int i = 0; i < 4; ++i) d[r][e][i] *= scale;
                    }
                }
                if (p.delta) norm_parts<N, E, R>(p, d, red, turn++);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    if (j + r >= j1) break;
                    const size_t row = (size_t)(t0 + j + r) * p.width;
                    const bool out = j + r >= emit;
#pragma unroll
                    for (int e = 0; e < E; ++e) {
                        const int c = (e * N + tid) * 4;
                        if (c >= p.width) break;
                        if (p.delta) {
#pragma unroll
                            for (int i = 0; i < 4; ++i) x[r][e][i] = fmaf(d[r][e][i], nw[e][i], x[r][e][i]);
                        }
                        if (out) {
                            put4(p.x_out + row + c, x[r][e]);
                            float y[4];
#pragma unroll
                            for (int i = 0; i < 4; ++i) {
                                float s = 0.f;
#pragma unroll
                                for (int k = 0; k < W - 1; ++k) s = fmaf(taps[k][e][i], hist[k][e][i], s);
                                y[i] = x[r][e][i] + fmaf(taps[W - 1][e][i], x[r][e][i], s);
                            }
                            put4(reinterpret_cast<T*>(p.h) + row + c, y);
                        }
#pragma unroll
                        for (int k = 0; k + 1 < W - 1; ++k)
#pragma unroll
                            for (int i = 0; i < 4; ++i) hist[k][e][i] = hist[k + 1][e][i];
#pragma unroll
                        for (int i = 0; i < 4; ++i) hist[W - 2][e][i] = x[r][e][i];
                    }
                }
            }
        }
        if (first) {
#pragma unroll
            for (int j = 0; j < W - 1; ++j)
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    const int c = (e * N + tid) * 4;
                    if (j >= pad && c < p.width) put4(hist_row + (size_t)(j - pad) * p.width + c, hist[j][e]);
                }
            if (p.ids && p.bigram) {
                __syncthreads();                          // everyone has read the old last token
                if (tid == 0) p.last[slot] = p.ids[t0 + ql - 1];
            }
        }
        t += n;
    }
}

template <int N, int E, int R>
static size_t post_smem(const StreamPostParams& p) {
    const int part = p.width / p.groups;
    if (part % 128 == 0) return (size_t)2 * R * E * (N / 32) * sizeof(float);
    return (size_t)R * ((part % 4 == 0 ? p.width / 4 : p.width) + p.groups) * sizeof(float);
}

template <typename T, int N, int E>
static int launch_row(const StreamPostParams& p, cudaStream_t stream) {
    const size_t smem = post_smem<N, E, 1>(p);
    if (smem > 48 * 1024) return fail("telb_stream_post: parts of this size are not built for rows this wide");
    TELB_LAUNCH("post_row_kernel", (post_row_kernel<T, N, E>), dim3(p.tokens), dim3(N), smem, stream, p);
    TELB_CHECK_LAUNCH("post_row_kernel");
    return 0;
}

template <typename T, int N, int E, int W>
static int launch_conv(const StreamPostParams& p, cudaStream_t stream) {
    const size_t smem = post_smem<N, E, 2>(p);
    if (smem > 48 * 1024) return fail("telb_stream_post: parts of this size are not built for rows this wide");
    TELB_LAUNCH("post_conv_kernel", (post_conv_kernel<T, N, E, W>), dim3((p.tokens + p.block_rows - 1) / p.block_rows), dim3(N), smem, stream, p);
    TELB_CHECK_LAUNCH("post_conv_kernel");
    return 0;
}

template <typename T>
static int run_post(const StreamPostParams& p, cudaStream_t stream) {
    if (!p.conv) {
        if (p.width <= 1024) return launch_row<T, 256, 1>(p, stream);
        if (p.width <= 2048) return launch_row<T, 256, 2>(p, stream);
        if (p.width <= 4096) return launch_row<T, 256, 4>(p, stream);
        return launch_row<T, 1024, 4>(p, stream);
    }
    if (p.taps <= 4) {
        if (p.width <= 1024) return launch_conv<T, 256, 1, 4>(p, stream);
        if (p.width <= 2048) return launch_conv<T, 256, 2, 4>(p, stream);
        if (p.width <= 4096) return launch_conv<T, 512, 2, 4>(p, stream);
        return launch_conv<T, 512, 4, 4>(p, stream);
    }
    if (p.width <= 1024) return launch_conv<T, 256, 1, 8>(p, stream);
    if (p.width <= 4096) return launch_conv<T, 512, 2, 8>(p, stream);
    return launch_conv<T, 512, 4, 8>(p, stream);
}

}  // namespace telb

using namespace telb;

// dtype: 1 bf16, 2 fp32 (of the tables, delta and h; the un-normed stream needs bf16's range).  With a convolution, p->block_rows is 1 (then every sequence has at most one
// row) or at least 8.
extern "C" int telb_stream_post(const StreamPostParams* pp, int dtype, cudaStream_t stream) {
    const StreamPostParams& p = *pp;
    if (p.tokens <= 0) return 0;
    if (p.width % 4 || p.width > 16 * 1024) return fail("telb_stream_post: width must be a multiple of 4 and at most 16384");
    if (p.groups < 1 || p.groups > kPostMaxGroups || p.width % p.groups) return fail("telb_stream_post: 1 to 256 groups that divide the width");
    if (!p.ids == !p.x_in) return fail("telb_stream_post: either ids or a stream");
    if (p.delta && !p.weight) return fail("telb_stream_post: the update has a weight");
    if (p.conv) {
        if (p.width > 8 * 1024) return fail("telb_stream_post: the convolution covers rows up to 8192 wide");
        if (p.taps < 1 || p.taps > kPostMaxTaps) return fail("telb_stream_post: convolutions have 1 to 8 taps");
        if (p.taps > 1 && !p.history) return fail("telb_stream_post: the convolution keeps a history");
        if (p.block_rows != 1 && p.block_rows < kPostMaxTaps) return fail("telb_stream_post: blocks of 1 or at least 8 rows");
        if (p.bigram && (!p.last || p.buckets < 1)) return fail("telb_stream_post: the bigram table needs buckets and last tokens");
        if (p.out_norm) return fail("telb_stream_post: a convolution or a norm, not both");
    } else if (p.ids) {
        return fail("telb_stream_post: token ids enter through the convolution form");
    }
    if (p.sums && (!p.delta || p.n_sums < 1 || p.sum_count < 1)) return fail("telb_stream_post: sums belong to an update");
    return dtype == 2 ? run_post<float>(p, stream) : run_post<__nv_bfloat16>(p, stream);
}
