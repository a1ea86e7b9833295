// Chunked mLSTM prefill on 5th-generation tensor cores (recurrence: mlstm.cu).
//
// A sequence is cut into chunks of 128 tokens.  With F_l = Σ_{i≤l} f_i (log forget gates inside the chunk), u_s = i_s − F_s and
// B_l = max(m_prev, max_{s≤l} u_s), the running maximum is m_l = F_l + B_l and the chunk is five matrix products:
//   G      = Q Kᵀ                                       [128 x 128]
//   P[l,s] = G[l,s] · scale · e^{u_s − B_l}  (s ≤ l)
//   Y      = P V  +  e^{m_prev − B_l} · scale · (Q S_prev)
//   den_l  = max(|Σ_s P[l,s] + e^{m_prev − B_l} · scale · q_l·n_prev|, e^{−m_l}) + 1e-6
//   S      = e^{m_prev − B_end} S_prev + Kᵀ diag(e^{u_s − B_end}) V,   n likewise,   m = F_end + B_end
// F cancels out of every weight, so no exponent grows with the chunk.
//
// Q, K and V are 16-bit values as the projections left them.  What the recurrence adds to them stays fp32: the operands that carry
// decays, gates or state (P, S, the weighted V) enter the tensor cores as a high and a low 16-bit part whose sum holds the fp32
// value to 2^-17 (2^-22 with fp16), two accumulating products each; row sums, n, gates and the stabiliser are fp32 on the CUDA
// cores, and the master copy of the state is fp32 in TMEM.
//
// One CTA owns (sequence, head, 128 value features) and walks the chunks in order.  The state is kept transposed, Sᵀ[128 v, DK], so
// that its 128 value rows are the TMEM lanes for any key width DK in {64, 128}.  With a single value tile per head the epilogue also
// applies the head norm and the output gate and stores 16-bit rows; with more, fp32 rows go to scratch for mlstm_gate_norm.
//
// Shared memory (DK = 128: 160 KB): Q | later P_hi | later (wV)_lo [32 KB] · K [DK/64 x 16 KB] · V | later (wV)_hi [32 KB] ·
// Sᵀ_hi, Sᵀ_lo [2 x DK/64 x 16 KB] | later P_lo [32 KB], all 128-byte-swizzled rows.  TMEM: G / then P·V at [0,128), Q·S at
// [128,256), Sᵀ at [256, 256 + DK).  Rows past the end of a ragged sequence have weight zero and are not stored.  Every wait is bounded.
#include <type_traits>

#include "host_utils.h"
#include "mlstm_common.cuh"
#include "tc5_common.cuh"

namespace telb {

constexpr int kMlL = 128;              // chunk length
constexpr int kMlV = 128;              // value features per CTA
constexpr int kMlThreads = 192;

// Split eight fp32 values into high and low 16-bit halves of one swizzled 16-byte unit each.
template <typename T>
__device__ __forceinline__ void split8(const float (&x)[8], uint4& hi, uint4& lo) {
    float l[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) l[i] = x[i] - Cvt<T>::to_f(Cvt<T>::from_f(x[i]));
    hi.x = Cvt<T>::pack2(x[0], x[1]);
    hi.y = Cvt<T>::pack2(x[2], x[3]);
    hi.z = Cvt<T>::pack2(x[4], x[5]);
    hi.w = Cvt<T>::pack2(x[6], x[7]);
    lo.x = Cvt<T>::pack2(l[0], l[1]);
    lo.y = Cvt<T>::pack2(l[2], l[3]);
    lo.z = Cvt<T>::pack2(l[4], l[5]);
    lo.w = Cvt<T>::pack2(l[6], l[7]);
}

// All 128 compute threads meet and agree: true when every one of them passed `ok`.
__device__ __forceinline__ bool compute_barrier_and(bool ok) {
    uint32_t r;
    asm volatile(
        "{\n\t.reg .pred p, q;\n\tsetp.ne.b32 p, %1, 0;\n\tbarrier.cta.red.and.pred q, 1, 128, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
        : "=r"(r) : "r"(ok ? 1u : 0u) : "memory");
    return r != 0;
}

template <typename T, int DK, bool FUSED>
__global__ void __launch_bounds__(kMlThreads, 1)
mlstm_chunk_kernel(const __grid_constant__ CUtensorMap tma, const __grid_constant__ MlstmParams p) {
    constexpr bool kBf16 = std::is_same<T, __nv_bfloat16>::value;
    constexpr int kAtoms = DK / 64;                      // 64-wide column atoms of a key row
    constexpr float kLog2e = 1.4426950408889634f;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* sQ = smem;                                  // 32 KB (P_hi and (wV)_lo need all of it)
    uint8_t* sK = sQ + 32768;
    uint8_t* sV = sK + kAtoms * 16384;                   // 32 KB
    uint8_t* sS = sV + 32768;                            // Sᵀ_hi | Sᵀ_lo; P_lo overlays the first 32 KB
    float* sU = reinterpret_cast<float*>(sS + 2 * kAtoms * 16384);     // u_s (base 2)                  [128]
    float* sW = sU + kMlL;                               // e^{u_s − B_end}                              [128]
    float* sN = sW + kMlL;                               // normaliser n                                 [DK]
    float* sWarp = sN + DK;                              // per-warp totals of the scans                 [8]
    float* sEnd = sWarp + 8;                             // F_end, B_end
    uint64_t* bars = reinterpret_cast<uint64_t*>(sEnd + 8);
    uint64_t* full_bar = bars;        // inputs of the chunk have landed (TMA)
    uint64_t* g_bar = bars + 1;       // G and Q·S_prev are in TMEM
    uint64_t* p_full = bars + 2;      // P_hi, P_lo are in shared memory (128 arrivals)
    uint64_t* y_bar = bars + 3;       // P·V is in TMEM
    uint64_t* xs_full = bars + 4;     // (wV) is in shared memory, Sᵀ is decayed (128 arrivals)
    uint64_t* s_bar = bars + 5;       // the state update has completed
    uint64_t* s_ready = bars + 6;     // Sᵀ copies are in shared memory (128 arrivals)
    uint64_t* k_done = bars + 7;      // the normaliser update has read K (128 arrivals)
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
    volatile uint32_t* abort_flag = tmem_slot + 1;

    const int warp = threadIdx.x >> 5;
    const int lane = threadIdx.x & 31;
    const int tiles_v = p.dv / kMlV;
    const int vt = blockIdx.x % tiles_v;
    const int sh = blockIdx.x / tiles_v;
    const int seq = sh / p.heads, h = sh - seq * p.heads;

    if (threadIdx.x == 0) {
        mbar_init(full_bar, 1);
        mbar_init(g_bar, 1);
        mbar_init(p_full, 128);
        mbar_init(y_bar, 1);
        mbar_init(xs_full, 128);
        mbar_init(s_bar, 1);
        mbar_init(s_ready, 128);
        mbar_init(k_done, 128);
        *abort_flag = 0;
        mbar_fence_init();
        prefetch_tensormap(&tma);
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, 512);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    pdl_prologue();
    const uint32_t tmem_base = *tmem_slot;
    const int ql = p.q_len[seq];
    const int t_first = p.q_start[seq];
    const int nchunks = (ql + kMlL - 1) / kMlL;
    constexpr uint32_t kColG = 0, kColYI = 128, kColS = 256;

    if (warp == 0) {
        // ---------------- producer ----------------
        if (lane == 0) {
            for (int c = 0; c < nchunks; ++c) {
                // V and K are read by the previous chunk's state update, the Q region holds (wV)_lo until then
                if (c > 0 && !(mbar_wait(s_bar, (uint32_t)(c - 1) & 1u, abort_flag, p.status, kStatusProducerTimeout) &&
                               mbar_wait(k_done, (uint32_t)(c - 1) & 1u, abort_flag, p.status, kStatusProducerTimeout))) break;
                const int t0 = t_first + c * kMlL;
                mbar_expect_tx(full_bar, (2 * kAtoms + 2) * 16384);
#pragma unroll
                for (int a = 0; a < kAtoms; ++a) {
                    tma_load_2d(sQ + a * 16384, &tma, full_bar, h * DK + a * 64, t0);
                    tma_load_2d(sK + a * 16384, &tma, full_bar, p.k_off + h * DK + a * 64, t0);
                }
#pragma unroll
                for (int a = 0; a < 2; ++a) tma_load_2d(sV + a * 16384, &tma, full_bar, p.v_off + h * p.dv + vt * kMlV + a * 64, t0);
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            const uint32_t idesc_kk = idesc_f16(128, 128, kBf16);                   // K-major A, K-major B: Q Kᵀ and Q S
            const uint32_t idesc_y = idesc_f16(128, kMlV, kBf16, false, true);      // K-major A (P), MN-major B (V)
            const uint32_t idesc_s = idesc_f16(kMlV, DK, kBf16, true, true);        // MN-major A (Vᵀ), MN-major B (K)
            for (int c = 0; c < nchunks; ++c) {
                const uint32_t par = (uint32_t)c & 1u;
                if (!mbar_wait(full_bar, par, abort_flag, p.status, kStatusMmaTimeout)) break;
                if (!mbar_wait(s_ready, par, abort_flag, p.status, kStatusMmaTimeout)) break;     // completion c: copies of the state before chunk c
                tc_fence_after_sync();
                const uint64_t dQ = smem_desc_sw128(sQ), dK = smem_desc_sw128(sK);
                const uint64_t dS = smem_desc_sw128(sS);
#pragma unroll
                for (int k = 0; k < DK / 16; ++k) {
                    const uint64_t off = (uint64_t)((k >> 2) * 16384 >> 4) + 2 * (k & 3);
                    umma_f16(tmem_base + kColG, dQ + off, dK + off, idesc_kk, k > 0 ? 1u : 0u);
                }
#pragma unroll
                for (int part = 0; part < 2; ++part)
#pragma unroll
                    for (int k = 0; k < DK / 16; ++k) {
                        const uint64_t off = (uint64_t)((k >> 2) * 16384 >> 4) + 2 * (k & 3);
                        umma_f16(tmem_base + kColYI, dQ + off, dS + (uint64_t)(part * kAtoms * 16384 >> 4) + off, idesc_kk, part + k > 0 ? 1u : 0u);
                    }
                umma_commit(g_bar);
                if (!mbar_wait(p_full, par, abort_flag, p.status, kStatusMmaTimeout)) break;
                tc_fence_after_sync();
                const uint64_t dV = smem_desc_sw128_mn(sV, 16384, 1024);
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    const uint64_t dP = smem_desc_sw128(part == 0 ? sQ : sS);
#pragma unroll
                    for (int k = 0; k < 8; ++k) {
                        const uint64_t off = (uint64_t)((k >> 2) * 16384 >> 4) + 2 * (k & 3);
                        umma_f16(tmem_base + kColG, dP + off, dV + (uint64_t)(k * 2048 >> 4), idesc_y, part + k > 0 ? 1u : 0u);
                    }
                }
                umma_commit(y_bar);
                if (!mbar_wait(xs_full, par, abort_flag, p.status, kStatusMmaTimeout)) break;
                tc_fence_after_sync();
                const uint64_t dKn = smem_desc_sw128_mn(sK, 16384, 1024);
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    const uint64_t dVt = smem_desc_sw128_mn(part == 0 ? sV : sQ, 16384, 1024);
#pragma unroll
                    for (int k = 0; k < 8; ++k)
                        umma_f16(tmem_base + kColS, dVt + (uint64_t)(k * 2048 >> 4), dKn + (uint64_t)(k * 2048 >> 4), idesc_s, 1u);
                }
                umma_commit(s_bar);
            }
        }
    } else {
        // ---------------- compute threads: token row r of the chunk, value row r of the state ----------------
        const int quad = warp & 3;
        const int r = quad * 32 + lane;
        const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quad * 32) << 16);
        const uint32_t row_off = (r >> 3) * 1024 + (r & 7) * 128;
        const size_t slot = (size_t)p.slot_ids[seq] * p.heads + h;
        float* st = p.state + slot * DK * p.dv + vt * kMlV + r;          // column r of this tile, rows p.dv apart
        float* gn = p.norm_state + slot * (DK + 1);
        const bool fresh = p.past_len[seq] <= 0;
        // Every thread takes every named barrier of a chunk, also after a wait ran out (the work in between is skipped then), and the
        // threads leave the loop together: `ok` is uniform per warp after each wait and uniform per CTA at the head of a chunk.
        bool ok = nchunks > 0;
        auto wait = [&](uint64_t* bar, uint32_t parity) {
            const bool got = ok && mbar_wait(bar, parity, abort_flag, p.status, kStatusEpilogueTimeout);
            ok = __all_sync(0xffffffffu, got);
            if (ok) tc_fence_after_sync();
        };
        float m_prev = 0.f;                                              // base 2
        // row r of the transposed state: fp32 in TMEM, high / low halves in shared memory
        auto store_state = [&](int c8, const float (&v)[8]) {
            uint4 hi, lo;
            split8<T>(v, hi, lo);
            uint8_t* dst = sS + (c8 >> 3) * 16384 + row_off + (((c8 & 7) ^ (r & 7)) << 4);
            *reinterpret_cast<uint4*>(dst) = hi;
            *reinterpret_cast<uint4*>(dst + kAtoms * 16384) = lo;
        };
        if (ok) {
            if (!fresh) m_prev = gn[DK] * kLog2e;
            if (r < DK) sN[r] = fresh ? 0.f : gn[r];
#pragma unroll 1
            for (int c8 = 0; c8 < DK / 8; ++c8) {
                float v[8];
                uint32_t u[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    v[i] = fresh ? 0.f : st[(size_t)(c8 * 8 + i) * p.dv];
                    u[i] = __float_as_uint(v[i]);
                }
                tmem_st_x8(lane_addr + kColS + c8 * 8, u);
                store_state(c8, v);
            }
            tmem_st_wait();
            tc_fence_before_sync();
            fence_proxy_async_smem();
            mbar_arrive(s_ready);
        }
        // gate pre-activations are fetched one chunk ahead: nothing else covers their latency at the head of a chunk
        float raw_i = 0.f, raw_f = 0.f;
        auto fetch_gates = [&](int c) {
            if (c * kMlL + r < ql) {
                const float* g = p.gates + ((size_t)t_first + (size_t)c * kMlL + r) * p.ldg + h;
                raw_i = g[0];
                raw_f = g[p.heads];
            }
        };
        fetch_gates(0);
        for (int c = 0; c < nchunks; ++c) {
            const uint32_t par = (uint32_t)c & 1u;
            const int len = min(kMlL, ql - c * kMlL);
            const size_t t = (size_t)t_first + (size_t)c * kMlL + r;
            const bool valid = r < len;
            // ---- gates, cumulative log forget gate and running maximum (base 2) ----
            float f = 0.f, gi = -INFINITY;
            if (valid) {
                gi = mlstm_input_gate(raw_i, p.cap) * kLog2e;
                f = mlstm_forget_gate(raw_f, p.cap) * kLog2e;
            }
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float n = __shfl_up_sync(0xffffffffu, f, o);
                if (lane >= o) f += n;
            }
            ok = compute_barrier_and(ok);                  // the previous chunk's readers of sU / sW / sWarp / sEnd are done
            if (!ok) break;
            if (lane == 31) sWarp[quad] = f;
            named_barrier_sync(1, 128);
            for (int w = 0; w < quad; ++w) f += sWarp[w];
            const float u = gi - f;
            float b = u;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float n = __shfl_up_sync(0xffffffffu, b, o);
                if (lane >= o) b = fmaxf(b, n);
            }
            if (lane == 31) sWarp[4 + quad] = b;
            sU[r] = u;
            named_barrier_sync(1, 128);
            for (int w = 0; w < quad; ++w) b = fmaxf(b, sWarp[4 + w]);
            b = fmaxf(b, m_prev);
            if (r == kMlL - 1) {
                sEnd[0] = f;
                sEnd[1] = b;
            }
            named_barrier_sync(1, 128);
            const float f_end = sEnd[0], b_end = sEnd[1];
            const float wgt = exp2f(u - b_end);            // 0 for rows past the end
            sW[r] = wgt;
            const float carry = exp2f(m_prev - b) * p.scale;
            // ---- q · n_prev (needs the raw Q rows, before P replaces them) ----
            wait(full_bar, par);
            float den = 0.f;
            if (ok) {
#pragma unroll 4
                for (int c8 = 0; c8 < DK / 8; ++c8) {
                    const uint4 qu = *reinterpret_cast<const uint4*>(sQ + (c8 >> 3) * 16384 + row_off + (((c8 & 7) ^ (r & 7)) << 4));
                    const T* qe = reinterpret_cast<const T*>(&qu);
                    const float4 n0 = *reinterpret_cast<const float4*>(sN + c8 * 8), n1 = *reinterpret_cast<const float4*>(sN + c8 * 8 + 4);
                    const float nn[8] = {n0.x, n0.y, n0.z, n0.w, n1.x, n1.y, n1.z, n1.w};
#pragma unroll
                    for (int i = 0; i < 8; ++i) den = fmaf(Cvt<T>::to_f(qe[i]), nn[i], den);
                }
                den *= carry;
            }
            // ---- P = G ∘ weights: high half over Q, low half over the state copies ----
            wait(g_bar, par);
            if (ok) {
#pragma unroll 1
                for (int cc = 0; cc < 4; ++cc) {                // 32 chunk columns at a time
                    uint8_t* prow = sQ + (cc >> 1) * 16384 + row_off;
                    uint8_t* plow = sS + (cc >> 1) * 16384 + row_off;
                    if (cc * 32 > quad * 32 + 31) {             // wholly above the diagonal for this warp
#pragma unroll
                        for (int q = 0; q < 4; ++q) {
                            const int unit = ((((cc & 1) * 4 + q) ^ (r & 7)) << 4);
                            *reinterpret_cast<uint4*>(prow + unit) = make_uint4(0, 0, 0, 0);
                            *reinterpret_cast<uint4*>(plow + unit) = make_uint4(0, 0, 0, 0);
                        }
                        continue;
                    }
                    uint32_t gr[32];
                    tmem_ld_x32(lane_addr + kColG + cc * 32, gr);
                    tmem_ld_wait();
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        float e[8];
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            const int s = cc * 32 + q * 8 + i;
                            e[i] = s <= r ? __uint_as_float(gr[q * 8 + i]) * (p.scale * exp2f(sU[s] - b)) : 0.f;
                            den += e[i];
                        }
                        uint4 hi, lo;
                        split8<T>(e, hi, lo);
                        const int unit = ((((cc & 1) * 4 + q) ^ (r & 7)) << 4);
                        *reinterpret_cast<uint4*>(prow + unit) = hi;
                        *reinterpret_cast<uint4*>(plow + unit) = lo;
                    }
                }
                tc_fence_before_sync();
                fence_proxy_async_smem();
                mbar_arrive(p_full);
            }
            fetch_gates(c + 1);
            uint4 gate_row[FUSED ? kMlV / 8 : 1];          // output-gate row, fetched under the products
            if constexpr (FUSED) {
                const uint4* gp = reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(p.qkvg) + t * p.ld + p.g_off + h * p.dv);
#pragma unroll
                for (int i = 0; i < kMlV / 8; ++i) gate_row[i] = valid ? gp[i] : make_uint4(0, 0, 0, 0);
            }
            const float inv = 1.f / (fmaxf(fabsf(den), exp2f(-(f + b))) + kMlstmEps);
            // ---- Sᵀ ← e^{m_prev − B_end} Sᵀ (row r), under the P·V product ----
            if (ok) {
                const float dec = exp2f(m_prev - b_end);
#pragma unroll 1
                for (int c16 = 0; c16 < DK / 16; c16 += 2) {
                    uint32_t v[16], w[16];
                    tmem_ld_x16(lane_addr + kColS + c16 * 16, v);
                    tmem_ld_x16(lane_addr + kColS + c16 * 16 + 16, w);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        v[i] = __float_as_uint(__uint_as_float(v[i]) * dec);
                        w[i] = __float_as_uint(__uint_as_float(w[i]) * dec);
                    }
                    tmem_st_x16(lane_addr + kColS + c16 * 16, v);
                    tmem_st_x16(lane_addr + kColS + c16 * 16 + 16, w);
                }
                tmem_st_wait();
            }
            wait(y_bar, par);
            if (ok) {
                // ---- (wV): high half in place, low half over P_hi (row r is this thread's own) ----
#pragma unroll 4
                for (int c8 = 0; c8 < kMlV / 8; ++c8) {
                    const uint32_t off = (c8 >> 3) * 16384 + row_off + (((c8 & 7) ^ (r & 7)) << 4);
                    const uint4 vu = *reinterpret_cast<const uint4*>(sV + off);
                    const T* ve = reinterpret_cast<const T*>(&vu);
                    float x[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) x[i] = wgt == 0.f ? 0.f : Cvt<T>::to_f(ve[i]) * wgt;
                    uint4 hi, lo;
                    split8<T>(x, hi, lo);
                    *reinterpret_cast<uint4*>(sV + off) = hi;
                    *reinterpret_cast<uint4*>(sQ + off) = lo;
                }
                tc_fence_before_sync();
                fence_proxy_async_smem();
                mbar_arrive(xs_full);
                // ---- outputs, under the state update: (P V + carry · Q S) / den, then head norm and gate when the tile is the head ----
                const float inter = carry * inv;
                if constexpr (FUSED) {
                    float ss = 0.f;
#pragma unroll 1
                    for (int c32 = 0; c32 < kMlV / 32; ++c32) {
                        uint32_t ya[32], yi[32];
                        tmem_ld_x32(lane_addr + kColG + c32 * 32, ya);
                        tmem_ld_x32(lane_addr + kColYI + c32 * 32, yi);
                        tmem_ld_wait();
                        float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                        for (int i = 0; i < 32; ++i) {
                            const float o = __uint_as_float(ya[i]) * inv + __uint_as_float(yi[i]) * inter;
                            part[i & 3] = fmaf(o, o, part[i & 3]);
                        }
                        ss += (part[0] + part[1]) + (part[2] + part[3]);
                    }
                    const float rn = 1.f / sqrtf(ss / p.dv_real + p.eps);
                    const float* nw = p.norm_w + h * p.dv;
                    T* op = reinterpret_cast<T*>(p.out) + (t * p.heads + h) * p.dv;
#pragma unroll
                    for (int c16 = 0; c16 < kMlV / 16; ++c16) {
                        uint32_t ya[16], yi[16];
                        tmem_ld_x16(lane_addr + kColG + c16 * 16, ya);
                        tmem_ld_x16(lane_addr + kColYI + c16 * 16, yi);
                        tmem_ld_wait();
#pragma unroll
                        for (int q = 0; q < 2; ++q) {
                            const T* ge = reinterpret_cast<const T*>(&gate_row[c16 * 2 + q]);
                            const float4 w0 = *reinterpret_cast<const float4*>(nw + c16 * 16 + q * 8), w1 = *reinterpret_cast<const float4*>(nw + c16 * 16 + q * 8 + 4);
                            const float w8[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
                            float o[8];
#pragma unroll
                            for (int i = 0; i < 8; ++i)
                                o[i] = __fdividef((__uint_as_float(ya[q * 8 + i]) * inv + __uint_as_float(yi[q * 8 + i]) * inter) * rn * w8[i],
                                                  1.f + __expf(-Cvt<T>::to_f(ge[i])));
                            uint4 ou;
                            ou.x = Cvt<T>::pack2(o[0], o[1]);
                            ou.y = Cvt<T>::pack2(o[2], o[3]);
                            ou.z = Cvt<T>::pack2(o[4], o[5]);
                            ou.w = Cvt<T>::pack2(o[6], o[7]);
                            if (valid) *reinterpret_cast<uint4*>(op + c16 * 16 + q * 8) = ou;
                        }
                    }
                } else {
                    float* op = p.o32 + (t * p.heads + h) * p.dv + vt * kMlV;
#pragma unroll 1
                    for (int c8 = 0; c8 < kMlV / 8; ++c8) {
                        uint32_t ya[8], yi[8];
                        tmem_ld_x8(lane_addr + kColG + c8 * 8, ya);
                        tmem_ld_x8(lane_addr + kColYI + c8 * 8, yi);
                        tmem_ld_wait();
                        if (valid) {
                            float o[8];
#pragma unroll
                            for (int i = 0; i < 8; ++i) o[i] = __uint_as_float(ya[i]) * inv + __uint_as_float(yi[i]) * inter;
                            *reinterpret_cast<float4*>(op + c8 * 8) = make_float4(o[0], o[1], o[2], o[3]);
                            *reinterpret_cast<float4*>(op + c8 * 8 + 4) = make_float4(o[4], o[5], o[6], o[7]);
                        }
                    }
                }
            }
            // ---- n ← e^{m_prev − B_end} n + Σ_s w_s k_s: thread r owns key feature r ----
            named_barrier_sync(1, 128);                    // sW is complete; every row has read the old n
            if (ok && r < DK) {
                const uint8_t* kc = sK + (r >> 6) * 16384 + (r & 7) * 2;
                const int unit = (r & 63) >> 3;
                float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
                for (int s8 = 0; s8 < kMlL / 8; ++s8) {
                    const float4 w0 = *reinterpret_cast<const float4*>(sW + s8 * 8), w1 = *reinterpret_cast<const float4*>(sW + s8 * 8 + 4);
                    const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const T k = *reinterpret_cast<const T*>(kc + s8 * 1024 + i * 128 + ((unit ^ i) << 4));
                        acc[i] = w[i] == 0.f ? acc[i] : fmaf(w[i], Cvt<T>::to_f(k), acc[i]);
                    }
                }
                const float sum = ((acc[0] + acc[1]) + (acc[2] + acc[3])) + ((acc[4] + acc[5]) + (acc[6] + acc[7]));
                sN[r] = sN[r] * exp2f(m_prev - b_end) + sum;
            }
            if (ok) mbar_arrive(k_done);
            m_prev = f_end + b_end;
            // ---- new state: halves for the next chunk, fp32 to the pool after the last one ----
            wait(s_bar, par);
            if (!ok) continue;                             // leaves at the next barrier (or with the loop)
            const bool last = c == nchunks - 1;
#pragma unroll 4
            for (int c8 = 0; c8 < DK / 8; ++c8) {
                uint32_t u8[8];
                tmem_ld_x8(lane_addr + kColS + c8 * 8, u8);
                tmem_ld_wait();
                float v[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(u8[i]);
                if (last) {
#pragma unroll
                    for (int i = 0; i < 8; ++i) st[(size_t)(c8 * 8 + i) * p.dv] = v[i];
                } else {
                    store_state(c8, v);
                }
            }
            if (last) {
                // several value tiles read the old normaliser: the new one waits in scratch until they are all done
                float* dst = FUSED ? gn : p.n_next + ((size_t)seq * p.heads + h) * (DK + 1);
                if (vt == 0) {
                    if (r < DK) dst[r] = sN[r];
                    if (r == 0) dst[DK] = m_prev / kLog2e;
                }
            } else {
                tc_fence_before_sync();
                fence_proxy_async_smem();
                mbar_arrive(s_ready);
            }
        }
    }

    if (*abort_flag) {
        const uint64_t t0 = global_timer_ns();
        while (global_timer_ns() - t0 < 200000ull) __nanosleep(1000);
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after_sync();
        tmem_dealloc(tmem_base, 512);
    }
}

template <typename T, int DK, bool FUSED>
static int launch_chunk(const CUtensorMap& tma, const MlstmParams& p, int num_seqs, cudaStream_t stream) {
    constexpr int smem = 32768 + DK / 64 * 16384 + 32768 + DK / 64 * 32768 + (2 * kMlL + DK + 16) * 4 + 128 + 1024;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_kernel<T, DK, FUSED>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(mlstm_chunk)", e);
        configured = true;
    }
    TELB_LAUNCH("mlstm_chunk_kernel", (mlstm_chunk_kernel<T, DK, FUSED>), dim3(num_seqs * p.heads * (p.dv / kMlV)), dim3(kMlThreads), smem, stream, tma, p);
    TELB_CHECK_LAUNCH("mlstm_chunk_kernel");
    return 0;
}

template <typename T>
static int dispatch_chunk(const CUtensorMap& tma, const MlstmParams& p, int num_seqs, cudaStream_t stream) {
    const bool fused = p.dv == kMlV;
    if (p.dk == 64) return fused ? launch_chunk<T, 64, true>(tma, p, num_seqs, stream) : launch_chunk<T, 64, false>(tma, p, num_seqs, stream);
    return fused ? launch_chunk<T, 128, true>(tma, p, num_seqs, stream) : launch_chunk<T, 128, false>(tma, p, num_seqs, stream);
}

}  // namespace telb

using namespace telb;

extern "C" int telb_mlstm_gate_norm(const MlstmParams* p, int num_seqs, int tokens, int dtype, cudaStream_t stream);

// Chunked prefill (see the top of the file): key heads padded to 64 or 128, value heads to a multiple of 128, 16-bit types.
// p->o32 and p->n_next are used only when a head has more than one value tile.
extern "C" int telb_mlstm_chunk(const MlstmParams* p, int num_seqs, int tokens, int is_bf16, cudaStream_t stream) {
    if (num_seqs <= 0 || tokens <= 0) return 0;
    if ((p->dk != 64 && p->dk != 128) || p->dv % kMlV) return fail("telb_mlstm_chunk: key heads of 64 or 128 and value heads in multiples of 128 are the compiled shapes");
    if (p->ld % 8) return fail("telb_mlstm_chunk: the projection row pitch must be a multiple of 8");
    CUtensorMap tma;
    const CUtensorMapDataType dt = is_bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16;
    if (make_tmap_2d(&tma, dt, 2, p->qkvg, tokens, p->ld, (uint64_t)p->ld * 2, kMlL, 64, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    const int rc = is_bf16 ? dispatch_chunk<__nv_bfloat16>(tma, *p, num_seqs, stream) : dispatch_chunk<__half>(tma, *p, num_seqs, stream);
    if (rc) return rc;
    return p->dv == kMlV ? 0 : telb_mlstm_gate_norm(p, num_seqs, tokens, is_bf16 ? 1 : 0, stream);
}
