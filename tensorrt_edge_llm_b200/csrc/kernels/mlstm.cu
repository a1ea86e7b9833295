// Matrix-memory LSTM (mLSTM) on the ragged step ABI: recurrence with an exponential input gate, a sigmoid forget gate and a
// running maximum, state rows addressed by slot id.  Per head, with log gates i and f:
//
//   m' = max(f + m, i),   S = e^{f+m-m'} S + e^{i-m'} k vᵀ,   n = e^{f+m-m'} n + e^{i-m'} k,   o = Sᵀ q / (max(|n·q|, e^{-m'}) + 1e-6)
//   i = cap · tanh(x_i / cap),   f = log σ(cap · tanh(x_f / cap));   S, n and m start at zero
//   y = o / rms(o) · w · σ(g)                                       (per head, then the output projection)
//
// Projections arrive packed as [q | k | v | g] rows in the activation type, gate pre-activations as fp32 columns; gates, state,
// stabiliser, normaliser and the head norm are fp32.  Heads may be padded at the end (zero projection rows): `dv_real` is the
// number of value features that the norm averages over.
//
// Here: the walk over the rows of a sequence in order (any size, any type; state tile in shared memory), the fused decode step
// (one row per sequence: gates, state update, read-out, head norm and output gate in one launch) and the head norm + gate.
// Long prompts in 16 bits take the chunked tensor-core form of mlstm_tc5.cu.
#include "host_utils.h"
#include "mlstm_common.cuh"
#include "tc5_common.cuh"

namespace telb {

constexpr int kScanCols = 64;          // value columns per CTA of the walk
constexpr int kScanThreads = 256;

// One CTA per (sequence, head, 64 value columns): thread (column c, row group r) owns S[r, r + 4, ...][c].
template <typename T>
__global__ void __launch_bounds__(kScanThreads) mlstm_scan_kernel(const __grid_constant__ MlstmParams p) {
    pdl_prologue();
    extern __shared__ float sm[];
    float* S = sm;                                   // [dk][64]
    float* sn = S + (size_t)p.dk * kScanCols;        // [dk]
    float* sq = sn + p.dk;                           // [dk]
    float* sk = sq + p.dk;                           // [dk]
    float* part = sk + p.dk;                         // [4][64]
    float* red = part + 4 * kScanCols;               // [8]
    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kScanCols;
    const int ql = p.q_len[seq];
    if (ql <= 0) return;
    const int tid = threadIdx.x, c = tid & 63, rg = tid >> 6, warp = tid >> 5, lane = tid & 31;
    const size_t slot = (size_t)p.slot_ids[seq] * p.heads + h;
    float* gs = p.state + slot * p.dk * p.dv;
    float* gn = p.norm_state + slot * (p.dk + 1);
    const bool fresh = p.past_len[seq] <= 0;
    for (int r = rg; r < p.dk; r += 4) S[r * kScanCols + c] = fresh ? 0.f : gs[(size_t)r * p.dv + c0 + c];
    for (int r = tid; r < p.dk; r += kScanThreads) sn[r] = fresh ? 0.f : gn[r];
    float m = fresh ? 0.f : gn[p.dk];
    for (int i = 0; i < ql; ++i) {
        const size_t t = (size_t)p.q_start[seq] + i;
        const T* row = reinterpret_cast<const T*>(p.qkvg) + t * p.ld;
        for (int r = tid; r < p.dk; r += kScanThreads) {
            sq[r] = Cvt<T>::to_f(row[h * p.dk + r]) * p.scale;
            sk[r] = Cvt<T>::to_f(row[p.k_off + h * p.dk + r]);
        }
        const float v = Cvt<T>::to_f(row[p.v_off + h * p.dv + c0 + c]);
        const float gi = mlstm_input_gate(p.gates[t * p.ldg + h], p.cap);
        const float gf = mlstm_forget_gate(p.gates[t * p.ldg + p.heads + h], p.cap);
        const float m_new = fmaxf(gf + m, gi);
        const float keep = expf(gf + m - m_new), add = expf(gi - m_new);
        m = m_new;
        __syncthreads();                             // q, k staged (also: the state tile on the first row)
        float acc = 0.f;
        const float av = add * v;
        for (int r = rg; r < p.dk; r += 4) {
            const float s = keep * S[r * kScanCols + c] + av * sk[r];
            S[r * kScanCols + c] = s;
            acc = fmaf(s, sq[r], acc);
        }
        part[rg * kScanCols + c] = acc;
        float qn = 0.f;
        for (int r = tid; r < p.dk; r += kScanThreads) {
            const float n = keep * sn[r] + add * sk[r];
            sn[r] = n;
            qn = fmaf(n, sq[r], qn);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) qn += __shfl_xor_sync(0xffffffffu, qn, o);
        if (lane == 0) red[warp] = qn;
        __syncthreads();
        if (tid < kScanCols) {
            float den = 0.f;
#pragma unroll
            for (int w = 0; w < kScanThreads / 32; ++w) den += red[w];
            const float num = part[c] + part[64 + c] + part[128 + c] + part[192 + c];
            p.o32[(t * p.heads + h) * p.dv + c0 + c] = num / (fmaxf(fabsf(den), expf(-m)) + kMlstmEps);
        }
        // the next row's staging only touches sq / sk, which nobody reads past the barrier above; `part` and `red` are rewritten
        // after the next row's first barrier
    }
    for (int r = rg; r < p.dk; r += 4) gs[(size_t)r * p.dv + c0 + c] = S[r * kScanCols + c];
    // every column tile read the old normaliser, so the new one waits in scratch until they are all done
    if (blockIdx.z == 0) {
        float* nn = p.n_next + ((size_t)seq * p.heads + h) * (p.dk + 1);
        for (int r = tid; r < p.dk; r += kScanThreads) nn[r] = sn[r];
        if (tid == 0) nn[p.dk] = m;
    }
}

// Decode: one row per sequence, one CTA per (sequence, head).  Threads stream the state in 16-byte pieces, read and write once;
// the head's output is reduced across row groups in shared memory, normalised, gated and stored in the activation type.
constexpr int kDecodeThreads = 256;
template <typename T>
__global__ void __launch_bounds__(kDecodeThreads) mlstm_decode_kernel(const __grid_constant__ MlstmParams p) {
    pdl_prologue();
    extern __shared__ float sm[];
    const int cols4 = p.dv >> 2;                     // 16-byte columns
    const int groups = kDecodeThreads / cols4;
    float* sq = sm;                                  // [dk]
    float* sk = sq + p.dk;                           // [dk]
    float* part = sk + p.dk;                         // [groups][dv]
    float* red = part + groups * p.dv;               // [16]
    const int seq = blockIdx.x, h = blockIdx.y;
    if (p.q_len[seq] <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const size_t t = p.q_start[seq];
    const size_t slot = (size_t)p.slot_ids[seq] * p.heads + h;
    float* gn = p.norm_state + slot * (p.dk + 1);
    const bool fresh = p.past_len[seq] <= 0;
    const T* row = reinterpret_cast<const T*>(p.qkvg) + t * p.ld;
    const float m = fresh ? 0.f : gn[p.dk];
    const float gi = mlstm_input_gate(p.gates[t * p.ldg + h], p.cap);
    const float gf = mlstm_forget_gate(p.gates[t * p.ldg + p.heads + h], p.cap);
    const float m_new = fmaxf(gf + m, gi);
    const float keep = expf(gf + m - m_new), add = expf(gi - m_new);
    __syncthreads();                                 // every thread has read m before it is replaced
    float qn = 0.f;
    for (int r = tid; r < p.dk; r += kDecodeThreads) {
        const float q = Cvt<T>::to_f(row[h * p.dk + r]) * p.scale;
        const float k = Cvt<T>::to_f(row[p.k_off + h * p.dk + r]);
        sq[r] = q;
        sk[r] = k;
        const float n = (fresh ? 0.f : keep * gn[r]) + add * k;
        gn[r] = n;
        qn = fmaf(n, q, qn);
    }
    if (tid == 0) gn[p.dk] = m_new;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) qn += __shfl_xor_sync(0xffffffffu, qn, o);
    if (lane == 0) red[warp] = qn;
    __syncthreads();
    float den = 0.f;
#pragma unroll
    for (int w = 0; w < kDecodeThreads / 32; ++w) den += red[w];
    const float inv = 1.f / (fmaxf(fabsf(den), expf(-m_new)) + kMlstmEps);
    const int c4 = tid % cols4, g = tid / cols4;
    if (g < groups) {
        float4* gs = reinterpret_cast<float4*>(p.state + slot * p.dk * p.dv) + c4;
        float v[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = add * Cvt<T>::to_f(row[p.v_off + h * p.dv + c4 * 4 + i]);
        float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
        for (int r = g; r < p.dk; r += groups) {
            float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : gs[(size_t)r * cols4];
            const float k = sk[r], q = sq[r];
            s.x = keep * s.x + v[0] * k;
            s.y = keep * s.y + v[1] * k;
            s.z = keep * s.z + v[2] * k;
            s.w = keep * s.w + v[3] * k;
            gs[(size_t)r * cols4] = s;
            a[0] = fmaf(s.x, q, a[0]);
            a[1] = fmaf(s.y, q, a[1]);
            a[2] = fmaf(s.z, q, a[2]);
            a[3] = fmaf(s.w, q, a[3]);
        }
        *reinterpret_cast<float4*>(part + g * p.dv + c4 * 4) = make_float4(a[0], a[1], a[2], a[3]);
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < p.dv; c += kDecodeThreads) {
        float o = 0.f;
        for (int i = 0; i < groups; ++i) o += part[i * p.dv + c];
        o *= inv;
        part[c] = o;                                 // column c of group 0: read by this thread only
        ss = fmaf(o, o, ss);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) red[8 + warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kDecodeThreads / 32; ++w) tot += red[8 + w];
    const float rn = 1.f / sqrtf(tot / p.dv_real + p.eps);
    T* out = reinterpret_cast<T*>(p.out) + (t * p.heads + h) * p.dv;
    for (int c = tid; c < p.dv; c += kDecodeThreads) {
        const float gate = Cvt<T>::to_f(row[p.g_off + h * p.dv + c]);
        out[c] = Cvt<T>::from_f(part[c] * rn * p.norm_w[h * p.dv + c] / (1.f + expf(-gate)));
    }
}

// Head norm and output gate of rows that the walk (or the chunk kernel with several value tiles) left in fp32: one warp per
// (token, head).  The first warps also move the new normalisers to their state rows.
template <typename T>
__global__ void __launch_bounds__(256) mlstm_gate_norm_kernel(const __grid_constant__ MlstmParams p, int tokens, int num_seqs) {
    pdl_prologue();
    const long long wid = (blockIdx.x * 256ll + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (wid >= (long long)tokens * p.heads) return;
    if (wid < (long long)num_seqs * p.heads) {
        const int seq = (int)(wid / p.heads), h = (int)(wid - (long long)seq * p.heads);
        if (p.q_len[seq] > 0) {
            const float* src = p.n_next + (size_t)wid * (p.dk + 1);
            float* dst = p.norm_state + ((size_t)p.slot_ids[seq] * p.heads + h) * (p.dk + 1);
            for (int r = lane; r <= p.dk; r += 32) dst[r] = src[r];
        }
    }
    const size_t t = wid / p.heads;
    const int h = (int)(wid - (long long)t * p.heads);
    const float* o = p.o32 + (size_t)wid * p.dv;
    const T* g = reinterpret_cast<const T*>(p.qkvg) + t * p.ld + p.g_off + h * p.dv;
    T* out = reinterpret_cast<T*>(p.out) + (size_t)wid * p.dv;
    float ss = 0.f;
    for (int c = lane * 4; c < p.dv; c += 128) {
        const float4 v = *reinterpret_cast<const float4*>(o + c);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    const float rn = 1.f / sqrtf(ss / p.dv_real + p.eps);
    for (int c = lane * 4; c < p.dv; c += 128) {
        const float4 v = *reinterpret_cast<const float4*>(o + c);
        const float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
            out[c + i] = Cvt<T>::from_f(e[i] * rn * p.norm_w[h * p.dv + c + i] / (1.f + expf(-Cvt<T>::to_f(g[c + i]))));
    }
}

template <typename T>
static int run_gate_norm(const MlstmParams& p, int num_seqs, int tokens, cudaStream_t stream) {
    const long long threads = (long long)tokens * p.heads * 32;
    TELB_LAUNCH("mlstm_gate_norm_kernel", (mlstm_gate_norm_kernel<T>), dim3((unsigned)((threads + 255) / 256)), dim3(256), 0, stream, p, tokens, num_seqs);
    TELB_CHECK_LAUNCH("mlstm_gate_norm_kernel");
    return 0;
}

template <typename T>
static int run_scan(const MlstmParams& p, int num_seqs, int tokens, cudaStream_t stream) {
    const size_t smem = ((size_t)p.dk * kScanCols + 3 * p.dk + 4 * kScanCols + 8) * sizeof(float);
    static size_t configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(mlstm_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(mlstm_scan)", e);
        configured = smem;
    }
    TELB_LAUNCH("mlstm_scan_kernel", (mlstm_scan_kernel<T>), dim3(num_seqs, p.heads, p.dv / kScanCols), dim3(kScanThreads), smem, stream, p);
    TELB_CHECK_LAUNCH("mlstm_scan_kernel");
    return run_gate_norm<T>(p, num_seqs, tokens, stream);
}

template <typename T>
static int run_decode(const MlstmParams& p, int num_seqs, cudaStream_t stream) {
    const int groups = kDecodeThreads / (p.dv / 4);
    const size_t smem = ((size_t)2 * p.dk + (size_t)groups * p.dv + 16) * sizeof(float);
    TELB_LAUNCH("mlstm_decode_kernel", (mlstm_decode_kernel<T>), dim3(num_seqs, p.heads), dim3(kDecodeThreads), smem, stream, p);
    TELB_CHECK_LAUNCH("mlstm_decode_kernel");
    return 0;
}

}  // namespace telb

using namespace telb;

static int check_params(const MlstmParams* p) {
    if (p->dk % 64 || p->dv % 64 || p->dk > 512) return fail("telb_mlstm: padded head sizes are multiples of 64, keys at most 512 wide");
    return 0;
}

// Walk over every sequence's rows, then head norm + output gate.  p->o32 [tokens, heads, dv] and p->n_next [seqs, heads, dk + 1] are
// scratch.  dtype: 0 fp16, 1 bf16, 2 fp32.
extern "C" int telb_mlstm_scan(const MlstmParams* p, int num_seqs, int tokens, int dtype, cudaStream_t stream) {
    if (num_seqs <= 0 || tokens <= 0) return 0;
    if (check_params(p)) return -1;
    if (dtype == 2) return run_scan<float>(*p, num_seqs, tokens, stream);
    return dtype == 1 ? run_scan<__nv_bfloat16>(*p, num_seqs, tokens, stream) : run_scan<__half>(*p, num_seqs, tokens, stream);
}

// Every sequence has one row (decode): the fused step.
extern "C" int telb_mlstm_decode(const MlstmParams* p, int num_seqs, int dtype, cudaStream_t stream) {
    if (num_seqs <= 0) return 0;
    if (check_params(p)) return -1;
    if (p->dv > 1024) return fail("telb_mlstm_decode: value heads at most 1024 wide");
    if (dtype == 2) return run_decode<float>(*p, num_seqs, stream);
    return dtype == 1 ? run_decode<__nv_bfloat16>(*p, num_seqs, stream) : run_decode<__half>(*p, num_seqs, stream);
}

// Head norm and output gate alone (after the chunk kernel left fp32 rows in p->o32 and normalisers in p->n_next).
extern "C" int telb_mlstm_gate_norm(const MlstmParams* p, int num_seqs, int tokens, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (dtype == 2) return run_gate_norm<float>(*p, num_seqs, tokens, stream);
    return dtype == 1 ? run_gate_norm<__nv_bfloat16>(*p, num_seqs, tokens, stream) : run_gate_norm<__half>(*p, num_seqs, tokens, stream);
}
