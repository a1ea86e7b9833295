// Paged grouped-query attention on the CUDA cores, for the element type and head sizes that the tcgen05 kernels do not take
// (fp32 caches, heads wider than 256).  Same tensors and masks as the tile kernel of attention_tc5_extra.cu: causal, sliding
// window, chunked (a row sees only keys of its own `chunk`-token block, counted from position 0) and sink logits.
//
// Latent rows (one plane, one row per token that serves as key and, with its first dv features, as value) are covered as well, and
// wide queries: a head's query spans the keys of all KV heads side by side, its scores lose slope * distance, its output is gated.
//
// One warp per (token, query head): 32 keys at a time, one key per lane for the scores, then one slice of the head per lane for
// the weighted values, with a running maximum.  Everything after the loads is fp32.
#include "host_utils.h"
#include "tc5_common.cuh"

namespace telb {

struct SimtAttnParams {
    const void* q;
    const void* kv;
    void* out;
    const int* q_start;
    const int* past_len;
    const int* seq_ids;
    const int* page_table;
    int tokens, max_pages, page_size, hq, hkv, d, window, chunk;
    int dv, planes;              // value features; 2 = key and value planes, 1 = values are the first dv features of the keys
    float scale;
    const float* sinks;
    const float* back;           // [positions, d] cos | sin: outputs turn back by their position, pairs of neighbours; or null
    float mult;                  // factor of the outputs, with back
    long long ld_out;            // row pitch of out
    int wide = 0;                // 1: queries span the keys of all KV heads, [T, hq, hkv * d]
    const float* slopes = nullptr;       // [hq]: scores lose slope * distance
    const void* gate = nullptr;          // [T, ld_gate]: outputs times its sigmoid, or null
    long long ld_gate = 0;
};

template <typename T, int E>                             // E: value features per lane, dv <= 32 E
__global__ void __launch_bounds__(128) attn_simt_kernel(const __grid_constant__ SimtAttnParams p) {
    pdl_prologue();
    extern __shared__ float s_q[];                       // [4 warps][features of a query]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long wid = (long long)blockIdx.x * 4 + warp;
    if (wid >= (long long)p.tokens * p.hq) return;
    const int t = (int)(wid / p.hq), h = (int)(wid - (long long)t * p.hq);
    const int kvh = h / (p.hq / p.hkv);
    const int seq = p.seq_ids[t];
    const int pos = p.past_len[seq] + (t - p.q_start[seq]);
    const int key_heads = p.wide ? p.hkv : 1, qd = key_heads * p.d;
    const T* q = reinterpret_cast<const T*>(p.q) + ((size_t)t * p.hq + h) * qd;
    float* sq = s_q + warp * qd;
    for (int i = lane; i < qd; i += 32) sq[i] = Cvt<T>::to_f(q[i]);
    __syncwarp();
    int lo = 0;
    if (p.window > 0) lo = max(lo, pos - p.window + 1);
    if (p.chunk > 0) lo = max(lo, pos / p.chunk * p.chunk);
    const T* kv = reinterpret_cast<const T*>(p.kv);
    const int* pages = p.page_table + (size_t)seq * p.max_pages;
    const size_t v_rows = p.planes == 2 ? (size_t)p.hkv * p.page_size : 0;
    float m = p.sinks ? p.sinks[h] : -INFINITY;
    float l = p.sinks ? 1.f : 0.f;
    float acc[E];
#pragma unroll
    for (int e = 0; e < E; ++e) acc[e] = 0.f;
    for (int j0 = lo; j0 <= pos; j0 += 32) {
        const int j = j0 + lane;
        const int page = j <= pos ? pages[j / p.page_size] : -1;
        const size_t krow = page < 0 ? 0 : (((size_t)page * p.planes) * p.hkv + kvh) * p.page_size + j % p.page_size;
        float s = -INFINITY;
        if (page >= 0) {
            const T* k = kv + (p.wide ? krow - (size_t)kvh * p.page_size : krow) * p.d;
            float dot = 0.f;
            for (int c = 0; c < key_heads; ++c, k += (size_t)p.page_size * p.d)
                for (int i = 0; i < p.d; ++i) dot = fmaf(sq[c * p.d + i], Cvt<T>::to_f(k[i]), dot);
            s = dot * p.scale;
            if (p.slopes) s = fmaf(p.slopes[h], (float)(j - pos), s);
        }
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m, mx);
        if (m_new == -INFINITY) continue;
        const float f = m == -INFINITY ? 0.f : expf(m - m_new);
        const float e_s = s == -INFINITY ? 0.f : expf(s - m_new);
        float sum = e_s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        l = l * f + sum;
        m = m_new;
#pragma unroll
        for (int e = 0; e < E; ++e) acc[e] *= f;
        const int cnt = min(32, pos - j0 + 1);
        for (int jj = 0; jj < cnt; ++jj) {
            const float w = __shfl_sync(0xffffffffu, e_s, jj);
            const unsigned long long row = __shfl_sync(0xffffffffu, (unsigned long long)krow, jj);
            const T* v = kv + ((size_t)row + v_rows) * p.d;
#pragma unroll
            for (int e = 0; e < E; ++e)
                if (e * 32 + lane < p.dv) acc[e] = fmaf(w, Cvt<T>::to_f(v[e * 32 + lane]), acc[e]);
        }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)h * p.dv;
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = e * 32 + lane;
        float o = acc[e] * inv;
        if (p.back) {                                        // uniform: the pair's other half sits on the next lane
            const float other = __shfl_xor_sync(0xffffffffu, o, 1);
            if (c < p.dv) {
                const float* cs = p.back + (size_t)pos * p.dv + c / 2;
                o = (o * cs[0] + ((lane & 1) ? -other : other) * cs[p.dv / 2]) * p.mult;
            }
        }
        if (p.gate && c < p.dv)
            o /= 1.f + expf(-Cvt<T>::to_f(reinterpret_cast<const T*>(p.gate)[(size_t)t * p.ld_gate + (size_t)h * p.dv + c]));
        if (c < p.dv) out[c] = Cvt<T>::from_f(o);
    }
}

template <typename T>
static int launch_simt(const SimtAttnParams& p, cudaStream_t stream) {
    const long long warps = (long long)p.tokens * p.hq;
    const dim3 grid((unsigned)((warps + 3) / 4));
    const size_t smem = (size_t)4 * p.d * (p.wide ? p.hkv : 1) * sizeof(float);
    if (smem > 200 * 1024) return fail("attn_simt_kernel: queries too wide");
#define TELB_SIMT(E_)                                                                                                                       \
    do {                                                                                                                                    \
        if (smem > 48 * 1024) {                                                                                                             \
            cudaError_t e = cudaFuncSetAttribute(attn_simt_kernel<T, E_>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);         \
            if (e != cudaSuccess) return fail("cudaFuncSetAttribute(attn_simt)", e);                                                        \
        }                                                                                                                                   \
        TELB_LAUNCH("attn_simt_kernel", (attn_simt_kernel<T, E_>), grid, dim3(128), smem, stream, p);                                       \
    } while (0)
    if (p.dv <= 64) TELB_SIMT(2);
    else if (p.dv <= 128) TELB_SIMT(4);
    else if (p.dv <= 256) TELB_SIMT(8);
    else if (p.dv <= 512) TELB_SIMT(16);
    else TELB_SIMT(32);
#undef TELB_SIMT
    TELB_CHECK_LAUNCH("attn_simt_kernel");
    return 0;
}

}  // namespace telb

using namespace telb;

extern "C" int telb_paged_attention_simt(const void* q, const void* kv_layer, void* out, const int* q_start, const int* past_len, const int* seq_ids,
                                         const int* page_table, int total_tokens, int max_pages, int page_size, int hq, int hkv, int d, float scale,
                                         int window, int chunk, const float* sinks, const float* back, float mult, long long ld_out, int dtype,
                                         cudaStream_t stream) {
    if (total_tokens <= 0) return 0;
    if (d > 1024) return fail("telb_paged_attention_simt: head_dim must be at most 1024");
    if (hkv <= 0 || hq % hkv) return fail("telb_paged_attention_simt: Hq must be a multiple of Hkv");
    SimtAttnParams p{q, kv_layer, out, q_start, past_len, seq_ids, page_table, total_tokens, max_pages, page_size, hq, hkv, d, window, chunk, d, 2, scale, sinks, back, mult, ld_out};
    if (dtype == 2) return launch_simt<float>(p, stream);
    return dtype == 1 ? launch_simt<__nv_bfloat16>(p, stream) : launch_simt<__half>(p, stream);
}

// Causal latent attention: q [T, Hq, row] against cached rows [pages, 1, 1, P, row]; out [T, Hq, dv], dv <= row.
extern "C" int telb_latent_attention_simt(const void* q, const void* kv_layer, void* out, const int* q_start, const int* past_len, const int* seq_ids,
                                          const int* page_table, int total_tokens, int max_pages, int page_size, int hq, int row, int dv, float scale,
                                          int dtype, cudaStream_t stream) {
    if (total_tokens <= 0) return 0;
    if (dv > 1024 || dv > row || row > 2048) return fail("telb_latent_attention_simt: at most 1024 latent features");
    SimtAttnParams p{q, kv_layer, out, q_start, past_len, seq_ids, page_table, total_tokens, max_pages, page_size, hq, 1, row, 0, 0, dv, 1, scale, nullptr, nullptr, 1.f, (long long)hq * dv};
    if (dtype == 2) return launch_simt<float>(p, stream);
    return dtype == 1 ? launch_simt<__nv_bfloat16>(p, stream) : launch_simt<__half>(p, stream);
}

// Wide queries q [T, Hq, Hkv * D] (scores mixed across heads), windowed; slopes [Hq]; gate [T, ld_gate] or null; out [T, Hq * D].  dtype: 1 bf16, 2 fp32.
extern "C" int telb_mixed_attention_simt(const void* q, const void* kv_layer, void* out, const int* q_start, const int* past_len, const int* seq_ids,
                                         const int* page_table, int total_tokens, int max_pages, int page_size, int hq, int hkv, int d, float scale, int window,
                                         const float* slopes, const void* gate, long long ld_gate, int dtype, cudaStream_t stream) {
    if (total_tokens <= 0) return 0;
    if (d > 1024) return fail("telb_mixed_attention_simt: head_dim must be at most 1024");
    if (hkv <= 0 || hq % hkv) return fail("telb_mixed_attention_simt: Hq must be a multiple of Hkv");
    SimtAttnParams p{q, kv_layer, out, q_start, past_len, seq_ids, page_table, total_tokens, max_pages, page_size, hq, hkv, d, window, 0, d, 2, scale, nullptr, nullptr, 1.f,
                     (long long)hq * d, 1, slopes, gate, ld_gate};
    if (dtype == 2) return launch_simt<float>(p, stream);
    return launch_simt<__nv_bfloat16>(p, stream);
}
