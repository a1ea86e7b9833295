// Lightning attention on the ragged step ABI: linear attention whose state decays by a constant of its head, state rows addressed by slot.
//
//   q, k, v <- silu(q), silu(k), silu(v)
//   S = decay S + k vᵀ,   o = Sᵀ q                       per head; S starts at zero
//   y = o / rms(o) · w · σ(g)                            rms over all heads of a row together
//
// Projections arrive packed as [q | k | v | g] rows in the activation type; state and read-outs are fp32.  Heads may be padded at the end
// (zero projection rows).
//
// The kernels write u = o · w · σ(g) and the sums of squares of o.  The rms is one number per row, so it commutes with the output
// projection: whoever adds the projected row to the residual stream divides by it (stream_post.cu), and no pass over the heads of a
// row is needed here.
//
// Here: the walk over the rows of a sequence in order (any size, any type; state tile in shared memory), the decode step (one row per
// sequence) and the activation pass in front of the chunked tensor-core form (lightning_tc5.cu).
#include "host_utils.h"
#include "lightning_common.cuh"

namespace telb {

__device__ __forceinline__ float lightning_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

constexpr int kWalkCols = 64;          // value columns per CTA of the walk
constexpr int kWalkThreads = 256;

// One CTA per (sequence, head, 64 value columns): thread (column c, row group r) owns S[r, r + 4, ...][c].
template <typename T>
__global__ void __launch_bounds__(kWalkThreads) lightning_walk_kernel(const __grid_constant__ LightningParams p) {
    pdl_prologue();
    extern __shared__ float sm[];
    float* S = sm;                                   // [dk][64]
    float* sq = S + (size_t)p.dk * kWalkCols;        // [dk]
    float* sk = sq + p.dk;                           // [dk]
    float* part = sk + p.dk;                         // [4][64]
    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kWalkCols;
    const int ql = p.q_len[seq];
    if (ql <= 0) return;
    const int tid = threadIdx.x, c = tid & 63, rg = tid >> 6;
    float* gs = p.state + ((size_t)p.slot_ids[seq] * p.heads + h) * p.dk * p.dv + c0 + c;
    const bool fresh = p.past_len[seq] <= 0;
    const float decay = p.powers[(size_t)h * p.n_powers + 1];
    for (int r = rg; r < p.dk; r += 4) S[r * kWalkCols + c] = fresh ? 0.f : gs[(size_t)r * p.dv];
    for (int i = 0; i < ql; ++i) {
        const size_t t = (size_t)p.q_start[seq] + i;
        const T* row = reinterpret_cast<const T*>(p.rows) + t * p.ld;
        for (int r = tid; r < p.dk; r += kWalkThreads) {
            sq[r] = lightning_silu<T>(Cvt<T>::to_f(row[h * p.dk + r]));
            sk[r] = lightning_silu<T>(Cvt<T>::to_f(row[p.k_off + h * p.dk + r]));
        }
        const float v = lightning_silu<T>(Cvt<T>::to_f(row[p.v_off + h * p.dv + c0 + c]));
        __syncthreads();                             // q, k staged; `part` of the previous row is read
        float acc = 0.f;
        for (int r = rg; r < p.dk; r += 4) {
            const float s = fmaf(decay, S[r * kWalkCols + c], v * sk[r]);
            S[r * kWalkCols + c] = s;
            acc = fmaf(s, sq[r], acc);
        }
        part[rg * kWalkCols + c] = acc;
        __syncthreads();
        if (tid < kWalkCols) {
            const float o = (part[c] + part[64 + c]) + (part[128 + c] + part[192 + c]);
            const size_t col = (size_t)h * p.dv + c0 + c;
            reinterpret_cast<T*>(p.out)[t * p.heads * p.dv + col] = Cvt<T>::from_f(lightning_gate<T>(o, p.norm_w[col], Cvt<T>::to_f(row[p.g_off + col])));
            const float ss = lightning_warp_sum(o * o);
            if ((tid & 31) == 0) p.sums[(t * p.heads * p.dv + col) / 32] = ss;
        }
    }
    for (int r = rg; r < p.dk; r += 4) gs[(size_t)r * p.dv] = S[r * kWalkCols + c];
}

// Decode: one row per sequence, one CTA per (sequence, head, 128 value columns).  Warp w owns key rows w, w + 8, ...; a lane four columns of
// them, K rows in flight at a time.
constexpr int kStepThreads = 256;
template <typename T, int K>
__global__ void __launch_bounds__(kStepThreads, 2) lightning_step_kernel(const __grid_constant__ LightningParams p) {
    pdl_prologue();
    extern __shared__ float sm[];
    float* sq = sm;                                  // [dk]
    float* sk = sq + p.dk;                           // [dk]
    float* part = sk + p.dk;                         // [8][128]
    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * 128;
    if (p.q_len[seq] <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const size_t t = p.q_start[seq];
    const bool fresh = p.past_len[seq] <= 0;
    const T* row = reinterpret_cast<const T*>(p.rows) + t * p.ld;
    float* gs = p.state + ((size_t)p.slot_ids[seq] * p.heads + h) * p.dk * p.dv + c0 + lane * 4;
    float4 s[K];
    auto fetch = [&](int r0) {
#pragma unroll
        for (int i = 0; i < K; ++i) s[i] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(gs + (size_t)(r0 + i * 8) * p.dv);
    };
    fetch(warp);                                     // under the activations
    const float decay = p.powers[(size_t)h * p.n_powers + 1];
    for (int r = tid; r < p.dk; r += kStepThreads) {
        sq[r] = lightning_silu<T>(Cvt<T>::to_f(row[h * p.dk + r]));
        sk[r] = lightning_silu<T>(Cvt<T>::to_f(row[p.k_off + h * p.dk + r]));
    }
    float v[4], a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = lightning_silu<T>(Cvt<T>::to_f(row[p.v_off + h * p.dv + c0 + lane * 4 + i]));
    __syncthreads();
    for (int r0 = warp; r0 < p.dk; r0 += K * 8) {
        if (r0 != warp) fetch(r0);
#pragma unroll
        for (int i = 0; i < K; ++i) {
            const float k = sk[r0 + i * 8], q = sq[r0 + i * 8];
            s[i].x = fmaf(decay, s[i].x, v[0] * k);
            s[i].y = fmaf(decay, s[i].y, v[1] * k);
            s[i].z = fmaf(decay, s[i].z, v[2] * k);
            s[i].w = fmaf(decay, s[i].w, v[3] * k);
            *reinterpret_cast<float4*>(gs + (size_t)(r0 + i * 8) * p.dv) = s[i];
            a[0] = fmaf(s[i].x, q, a[0]);
            a[1] = fmaf(s[i].y, q, a[1]);
            a[2] = fmaf(s[i].z, q, a[2]);
            a[3] = fmaf(s[i].w, q, a[3]);
        }
    }
    *reinterpret_cast<float4*>(part + warp * 128 + lane * 4) = make_float4(a[0], a[1], a[2], a[3]);
    __syncthreads();
    if (tid < 128) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < kStepThreads / 32; ++w) o += part[w * 128 + tid];
        const size_t col = (size_t)h * p.dv + c0 + tid;
        reinterpret_cast<T*>(p.out)[t * p.heads * p.dv + col] = Cvt<T>::from_f(lightning_gate<T>(o, p.norm_w[col], Cvt<T>::to_f(row[p.g_off + col])));
        const float ss = lightning_warp_sum(o * o);
        if (lane == 0) p.sums[(t * p.heads * p.dv + col) / 32] = ss;
    }
}

// act = silu(q | k | v), rounded to the activation type: the operands of the chunk kernel's products.
template <typename T>
__global__ void __launch_bounds__(256) lightning_act_kernel(const __grid_constant__ LightningParams p) {
    pdl_prologue();
    const int per_row = p.g_off / 8;
    const long long n = (long long)p.tokens * per_row;
    for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) {
        const long long t = i / per_row;
        const int c = (int)(i - t * per_row) * 8;
        const uint4 u = *reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(p.rows) + t * p.ld + c);
        const T* e = reinterpret_cast<const T*>(&u);
        float f[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const float x = Cvt<T>::to_f(e[k]);
            f[k] = __fdividef(x, 1.f + __expf(-x));
        }
        uint4 r;
        r.x = Cvt<T>::pack2(f[0], f[1]);
        r.y = Cvt<T>::pack2(f[2], f[3]);
        r.z = Cvt<T>::pack2(f[4], f[5]);
        r.w = Cvt<T>::pack2(f[6], f[7]);
        *reinterpret_cast<uint4*>(reinterpret_cast<T*>(p.act) + t * p.g_off + c) = r;
    }
}

template <typename T>
static int run_walk(const LightningParams& p, cudaStream_t stream) {
    const size_t smem = ((size_t)p.dk * kWalkCols + 2 * p.dk + 4 * kWalkCols) * sizeof(float);
    static size_t configured = 48 * 1024;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(lightning_walk_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(lightning_walk)", e);
        configured = smem;
    }
    TELB_LAUNCH("lightning_walk_kernel", (lightning_walk_kernel<T>), dim3(p.num_seqs, p.heads, p.dv / kWalkCols), dim3(kWalkThreads), smem, stream, p);
    TELB_CHECK_LAUNCH("lightning_walk_kernel");
    return 0;
}

template <typename T>
static int run_step(const LightningParams& p, cudaStream_t stream) {
    const size_t smem = (2 * (size_t)p.dk + 8 * 128) * sizeof(float);
    const dim3 grid(p.num_seqs, p.heads, p.dv / 128);
    if (p.dk % 128 == 0) TELB_LAUNCH("lightning_step_kernel", (lightning_step_kernel<T, 16>), grid, dim3(kStepThreads), smem, stream, p);
    else TELB_LAUNCH("lightning_step_kernel", (lightning_step_kernel<T, 8>), grid, dim3(kStepThreads), smem, stream, p);
    TELB_CHECK_LAUNCH("lightning_step_kernel");
    return 0;
}

}  // namespace telb

using namespace telb;

static int check_sizes(const LightningParams* p) {
    if (p->dk % 64 || p->dv % 128 || p->dk > 512 || p->ld % 8) return fail("telb_lightning: key heads are multiples of 64 up to 512, value heads of 128, row pitches of 8");
    if (p->n_powers < 2 || p->heads > 65535) return fail("telb_lightning: the decays need their first power, and at most 65535 heads");
    return 0;
}

// Walk over every sequence's rows.  dtype: 1 bf16, 2 fp32 (un-normed rows need bf16's range).
extern "C" int telb_lightning_walk(const LightningParams* p, int dtype, cudaStream_t stream) {
    if (p->num_seqs <= 0 || p->tokens <= 0) return 0;
    if (check_sizes(p)) return -1;
    return dtype == 2 ? run_walk<float>(*p, stream) : run_walk<__nv_bfloat16>(*p, stream);
}

// Every sequence has at most one row (decode).
extern "C" int telb_lightning_step(const LightningParams* p, int dtype, cudaStream_t stream) {
    if (p->num_seqs <= 0 || p->tokens <= 0) return 0;
    if (check_sizes(p)) return -1;
    return dtype == 2 ? run_step<float>(*p, stream) : run_step<__nv_bfloat16>(*p, stream);
}

// p->act = silu(q | k | v), bf16.
extern "C" int telb_lightning_act(const LightningParams* p, cudaStream_t stream) {
    if (p->tokens <= 0) return 0;
    const long long blocks = ((long long)p->tokens * (p->g_off / 8) + 255) / 256;
    const dim3 grid((unsigned)(blocks < 148 * 32 ? blocks : 148 * 32));
    TELB_LAUNCH("lightning_act_kernel", (lightning_act_kernel<__nv_bfloat16>), grid, dim3(256), 0, stream, *p);
    TELB_CHECK_LAUNCH("lightning_act_kernel");
    return 0;
}
