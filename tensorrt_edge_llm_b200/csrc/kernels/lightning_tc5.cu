// Chunked lightning attention on 5th-generation tensor cores (recurrence: lightning.cu; q, k, v arrive activated).
//
// A sequence is cut into chunks of 128 tokens.  With the decay λ of the head, the state S_prev in front of a chunk and n its live rows:
//   G      = Q Kᵀ                                        [128 x 128]
//   P[l,s] = G[l,s] · λ^{l-s}  (s ≤ l)
//   O      = P V + λ^{l+1} · (Q S_prev)
//   S      = λ^n S_prev + Kᵀ diag(λ^{n-1-s}) V
// Powers of λ come from a table (rounded once from double), so nothing is divided and nothing grows.
//
// Q, K and V are 16-bit values.  The operands that carry decays or state (P, S, the weighted V) enter the tensor cores as a high and a
// low 16-bit part whose sum holds the fp32 value to 2^-17, two accumulating products each; the master copy of the state is fp32 in
// registers.
//
// One CTA owns (sequence, head, 128 value features, segment of chunks) and walks its chunks in order.  The state is kept transposed,
// Sᵀ [128 v, DK]: thread (row r, quarter) of the sixteen compute warps holds a quarter of value row r, and serves a quarter of token row r
// elsewhere.
// Weighted V needs nothing but V, so the state update is issued before P is ready; the loads of the next chunk start when the last
// product of this one is done, and run under the state's bookkeeping, the outputs and their gates.
//
// Few (sequence, head) pairs: sequences are cut into segments that run side by side.  The same kernel first takes every segment but the
// last from a zero state (STATE_ONLY: K and V, no outputs), lightning_carry chains the ends with λ^rows, and the full pass starts every
// segment from its true state.
//
// Shared memory (DK = 128: 224 KB): K | V [32 KB] | weighted V hi, lo [2 x 32 KB] | Q, later P hi [32 KB] | Sᵀ hi, lo, the first 32 KB later
// P lo; all 128-byte-swizzled rows.  TMEM: G [0,128) · P V [128,256) · Q S [256,384) · state update [384, 384 + DK).  Rows past the end of a
// ragged sequence have weight zero and are not stored.  Every wait is bounded.
#include "host_utils.h"
#include "lightning_common.cuh"

namespace telb {

constexpr int kLtL = 128;              // chunk length
constexpr int kLtCompute = 512;        // sixteen compute warps
constexpr int kLtThreads = 64 + kLtCompute;

// Split eight fp32 values into high and low bf16 halves of one swizzled 16-byte unit each.  A packed pair is widened by shifts: conversions
// are the slow instructions here.
__device__ __forceinline__ void lightning_split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = Cvt<__nv_bfloat16>::pack2(a, b);
    lo = Cvt<__nv_bfloat16>::pack2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ void lightning_split8(const float (&x)[8], uint4& hi, uint4& lo) {
    lightning_split2(x[0], x[1], hi.x, lo.x);
    lightning_split2(x[2], x[3], hi.y, lo.y);
    lightning_split2(x[4], x[5], hi.z, lo.z);
    lightning_split2(x[6], x[7], hi.w, lo.w);
}

template <int DK, bool STATE_ONLY>
__global__ void __launch_bounds__(kLtThreads, 1)
lightning_chunk_kernel(const __grid_constant__ CUtensorMap tma, const __grid_constant__ LightningParams p) {
    using T = __nv_bfloat16;
    constexpr int kAtoms = DK / 64;                      // 64-wide column atoms of a key row
    pdl_wait();
    const int tiles_v = p.dv / 128;
    const int live_segs = STATE_ONLY ? p.segments - 1 : p.segments;
    const int seg = blockIdx.x % live_segs;
    const int rest = blockIdx.x / live_segs;
    const int vt = rest % tiles_v, sh = rest / tiles_v;
    const int seq = sh / p.heads, h = sh - seq * p.heads;
    const int seg_rows = p.segments > 1 ? p.seg_chunks * kLtL : 1 << 30;
    const int ql_all = p.q_len[seq], row0 = p.segments > 1 ? seg * seg_rows : 0;
    const int ql = min(ql_all - row0, seg_rows);         // rows of this segment
    const bool last_seg = row0 + ql >= ql_all;
    if (ql <= 0 || (STATE_ONLY && last_seg)) return;     // uniform per CTA, before any barrier / TMEM use
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* sK = smem;
    uint8_t* sV = sK + kAtoms * 16384;
    uint8_t* sW = sV + 32768;                            // weighted V: hi | lo
    uint8_t* sQ = sW + 65536;                            // 32 KB: P hi needs all of it
    uint8_t* sS = sQ + 32768;                            // Sᵀ hi | Sᵀ lo (at least 32 KB); P lo overlays the first 32 KB
    uint8_t* tail = STATE_ONLY ? sQ : sS + 2 * kAtoms * 16384;
    float* sPw = reinterpret_cast<float*>(tail);         // λ^0 .. λ^128
    float* sNw = sPw + 132;                              // norm weights of the tile's features
    float* sNear = sNw + 128;                            // λ^31 .. λ^0
    uint64_t* bars = reinterpret_cast<uint64_t*>(tail + 528 + 512 + 128);
    uint64_t* full_bar = bars;        // inputs of the chunk have landed (TMA)
    uint64_t* g_bar = bars + 1;       // G is in TMEM
    uint64_t* yi_bar = bars + 2;      // Q S_prev is in TMEM
    uint64_t* w_full = bars + 3;      // weighted V is in shared memory (512 arrivals)
    uint64_t* p_full = bars + 4;      // P hi, lo are in shared memory (512 arrivals)
    uint64_t* y_bar = bars + 5;       // every product of the chunk is done
    uint64_t* s_ready = bars + 6;     // state copies of the chunk written, TMEM of the chunk before it read (512 arrivals)
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
    volatile uint32_t* abort_flag = tmem_slot + 1;

    const int warp = threadIdx.x >> 5;
    const int lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        mbar_init(full_bar, 1);
        mbar_init(g_bar, 1);
        mbar_init(yi_bar, 1);
        mbar_init(w_full, kLtCompute);
        mbar_init(p_full, kLtCompute);
        mbar_init(y_bar, 1);
        mbar_init(s_ready, kLtCompute);
        *abort_flag = 0;
        mbar_fence_init();
        prefetch_tensormap(&tma);
    }
    for (int i = threadIdx.x; i <= kLtL; i += kLtThreads) sPw[i] = p.powers[(size_t)h * p.n_powers + i];
    if (threadIdx.x < 32) sNear[threadIdx.x] = p.powers[(size_t)h * p.n_powers + 31 - threadIdx.x];
    if (!STATE_ONLY && threadIdx.x < 128) sNw[threadIdx.x] = p.norm_w[(size_t)h * p.dv + vt * 128 + threadIdx.x];
    if (warp == 1) {
        tmem_alloc(tmem_slot, 512);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    pdl_launch_dependents();          // after the allocation: a dependent that allocates ahead of its own wait must not take the columns first
    const uint32_t tmem_base = *tmem_slot;
    const int t_first = p.q_start[seq] + row0;
    const int nchunks = (ql + kLtL - 1) / kLtL;
    constexpr uint32_t kColG = 0, kColY = 128, kColYI = 256, kColS = 384;

    if (warp == 0) {
        // ---------------- producer ----------------
        if (lane == 0) {
            for (int c = 0; c < nchunks; ++c) {
                if (c > 0 && !mbar_wait(y_bar, (uint32_t)(c - 1) & 1u, abort_flag, p.status, kStatusProducerTimeout)) break;
                const int t0 = t_first + c * kLtL;
                mbar_expect_tx(full_bar, ((STATE_ONLY ? 1 : 2) * kAtoms + 2) * 16384);
#pragma unroll
                for (int a = 0; a < kAtoms; ++a) {
                    if (!STATE_ONLY) tma_load_2d(sQ + a * 16384, &tma, full_bar, h * DK + a * 64, t0);
                    tma_load_2d(sK + a * 16384, &tma, full_bar, p.k_off + h * DK + a * 64, t0);
                }
#pragma unroll
                for (int a = 0; a < 2; ++a) tma_load_2d(sV + a * 16384, &tma, full_bar, p.v_off + h * p.dv + vt * 128 + a * 64, t0);
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer: the whole warp walks, one elected lane issues ----------------
        const uint32_t idesc_kk = idesc_f16(128, 128, true);                    // K-major A, K-major B: Q Kᵀ and Q S
        const uint32_t idesc_y = idesc_f16(128, 128, true, false, true);        // K-major A (P), MN-major B (V)
        const uint32_t idesc_s = idesc_f16(128, DK, true, true, true);          // MN-major A (weighted Vᵀ), MN-major B (K)
        const uint64_t dQ = smem_desc_sw128(sQ), dK = smem_desc_sw128(sK), dS = smem_desc_sw128(sS);
        const uint64_t dV = smem_desc_sw128_mn(sV, 16384, 1024), dKn = smem_desc_sw128_mn(sK, 16384, 1024);
        bool ok = true;
        auto wait = [&](uint64_t* bar, uint32_t parity) {
            const bool got = ok && mbar_wait(bar, parity, abort_flag, p.status, kStatusMmaTimeout);
            ok = __all_sync(0xffffffffu, got);
            if (ok) tc_fence_after_sync();
            return ok;
        };
        for (int c = 0; c < nchunks; ++c) {
            const uint32_t par = (uint32_t)c & 1u;
            if (!wait(full_bar, par)) break;
            if (!STATE_ONLY) {
                if (elect_one()) {
#pragma unroll
                    for (int k = 0; k < DK / 16; ++k) {
                        const uint64_t off = (uint64_t)((k >> 2) * 16384 >> 4) + 2 * (k & 3);
                        umma_f16(tmem_base + kColG, dQ + off, dK + off, idesc_kk, k > 0 ? 1u : 0u);
                    }
                    umma_commit(g_bar);
                }
                __syncwarp();
            }
            if (!wait(s_ready, par)) break;              // completion c: copies of the state before chunk c
            if (!STATE_ONLY) {
                if (elect_one()) {
#pragma unroll
                    for (int part = 0; part < 2; ++part)
#pragma unroll
                        for (int k = 0; k < DK / 16; ++k) {
                            const uint64_t off = (uint64_t)((k >> 2) * 16384 >> 4) + 2 * (k & 3);
                            umma_f16(tmem_base + kColYI, dQ + off, dS + (uint64_t)(part * kAtoms * 16384 >> 4) + off, idesc_kk, part + k > 0 ? 1u : 0u);
                        }
                    umma_commit(yi_bar);
                }
                __syncwarp();
            }
            if (!wait(w_full, par)) break;
            if (elect_one()) {
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    const uint64_t dW = smem_desc_sw128_mn(sW + part * 32768, 16384, 1024);
#pragma unroll
                    for (int k = 0; k < 8; ++k)
                        umma_f16(tmem_base + kColS, dW + (uint64_t)(k * 2048 >> 4), dKn + (uint64_t)(k * 2048 >> 4), idesc_s, part + k > 0 ? 1u : 0u);
                }
                if (STATE_ONLY) umma_commit(y_bar);
            }
            __syncwarp();
            if (STATE_ONLY) continue;
            if (!wait(p_full, par)) break;
            if (elect_one()) {
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    const uint64_t dP = smem_desc_sw128(part == 0 ? sQ : sS);
#pragma unroll
                    for (int k = 0; k < 8; ++k) {
                        const uint64_t off = (uint64_t)((k >> 2) * 16384 >> 4) + 2 * (k & 3);
                        umma_f16(tmem_base + kColY, dP + off, dV + (uint64_t)(k * 2048 >> 4), idesc_y, part + k > 0 ? 1u : 0u);
                    }
                }
                umma_commit(y_bar);
            }
            __syncwarp();
        }
    } else {
        // ---------------- compute threads: token row r of the chunk, value row r of the state, a quarter of the columns ----------------
        const int quad = warp & 3, quarter = (warp - 2) >> 2;
        const int r = quad * 32 + lane;
        const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quad * 32) << 16);
        bool ok = true;
        auto wait = [&](uint64_t* bar, uint32_t parity) {
            const bool got = ok && mbar_wait(bar, parity, abort_flag, p.status, kStatusEpilogueTimeout);
            ok = __all_sync(0xffffffffu, got);
            if (ok) tc_fence_after_sync();
            return ok;
        };
        // 16-byte unit j (of four) of this quarter in row `row` of a 128-column tile
        auto unit = [&](int row, int j) {
            return (quarter >> 1) * 16384 + (row >> 3) * 1024 + (row & 7) * 128 + ((((quarter & 1) * 4 + j) ^ (row & 7)) << 4);
        };
        constexpr int kOwn = DK / 4;                                     // key features of the state row that this thread holds
        const size_t sh_off = (size_t)h * DK * p.dv + vt * 128 + r;      // column r of this tile, rows p.dv apart
        const size_t per_seq = (size_t)p.heads * DK * p.dv;
        float* carry = p.carry + ((size_t)(seq * p.heads + h) * p.segments + seg) * DK * p.dv + vt * 128 + r;
        float* slot = p.state + (size_t)p.slot_ids[seq] * per_seq + sh_off;
        float S[kOwn];
        {
            const float* src = p.segments > 1 ? carry : slot;
            const bool zero = STATE_ONLY || (p.segments == 1 && p.past_len[seq] <= 0);
#pragma unroll
            for (int j = 0; j < kOwn; ++j) S[j] = zero ? 0.f : src[(size_t)(quarter * kOwn + j) * p.dv];
        }
        auto publish_state = [&]() {
            if (!STATE_ONLY) {
#pragma unroll
                for (int q = 0; q < kOwn / 8; ++q) {
                    float x[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) x[i] = S[q * 8 + i];
                    uint4 hi, lo;
                    lightning_split8(x, hi, lo);
                    const int c8 = quarter * (kOwn / 8) + q;
                    uint8_t* dst = sS + (c8 >> 3) * 16384 + (r >> 3) * 1024 + (r & 7) * 128 + (((c8 & 7) ^ (r & 7)) << 4);
                    *reinterpret_cast<uint4*>(dst) = hi;
                    *reinterpret_cast<uint4*>(dst + kAtoms * 16384) = lo;
                }
            }
            tc_fence_before_sync();
            fence_proxy_async_smem();
            mbar_arrive(s_ready);
        };
        publish_state();
        for (int c = 0; c < nchunks; ++c) {
            const uint32_t par = (uint32_t)c & 1u;
            const int len = min(kLtL, ql - c * kLtL);
            const size_t t = (size_t)t_first + (size_t)c * kLtL + r;
            const bool valid = r < len;
            // ---- weighted V (32 features of token r) ----
            if (!wait(full_bar, par)) break;
            {
                const float wgt = valid ? sPw[len - 1 - r] : 0.f;
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const uint32_t off = unit(r, q);
                    const uint4 vu = *reinterpret_cast<const uint4*>(sV + off);
                    const T* ve = reinterpret_cast<const T*>(&vu);
                    float x[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) x[i] = valid ? Cvt<T>::to_f(ve[i]) * wgt : 0.f;
                    uint4 hi, lo;
                    lightning_split8(x, hi, lo);
                    *reinterpret_cast<uint4*>(sW + off) = hi;
                    *reinterpret_cast<uint4*>(sW + 32768 + off) = lo;
                }
                fence_proxy_async_smem();
                mbar_arrive(w_full);
            }
            // gates of this warp's 32 rows, fetched under the products: four lanes share a row, eight rows at a time
            uint4 gate[STATE_ONLY ? 1 : 4];
            const size_t col = (size_t)h * p.dv + vt * 128 + quarter * 32;
            const int row_first = c * kLtL + quad * 32 + (lane >> 2);       // this lane's first row of the segment
            if constexpr (!STATE_ONLY) {
                // ---- P = G ∘ decays: computed under Q S, stored when that has read Q and the state copies ----
                if (!wait(g_bar, par)) break;
                uint4 hi[4], lo[4];
                const int c0 = quarter * 32;
                if (c0 > quad * 32) {                               // wholly above the diagonal
#pragma unroll
                    for (int q = 0; q < 4; ++q) hi[q] = lo[q] = make_uint4(0, 0, 0, 0);
                } else {
#pragma unroll
                    for (int g = 0; g < 2; ++g) {
                        uint32_t gr[16];
                        tmem_ld_x16(lane_addr + kColG + c0 + g * 16, gr);
                        tmem_ld_wait();
                        if (c0 == quad * 32) {                      // the diagonal runs through these columns
#pragma unroll
                            for (int q = 0; q < 2; ++q) {
                                float e[8];
#pragma unroll
                                for (int i = 0; i < 8; ++i) {
                                    const int s = g * 16 + q * 8 + i;
                                    e[i] = s <= lane ? __uint_as_float(gr[q * 8 + i]) * sPw[max(lane - s, 0)] : 0.f;
                                }
                                lightning_split8(e, hi[g * 2 + q], lo[g * 2 + q]);
                            }
                        } else {                                    // λ^{r-s} = λ^{r-c0-31} λ^{c0+31-s}, the second the same for all rows
                            const float far = sPw[r - c0 - 31];
#pragma unroll
                            for (int q = 0; q < 2; ++q) {
                                float e[8];
                                const float4* np = reinterpret_cast<const float4*>(sNear + g * 16 + q * 8);
                                const float4 d0 = np[0], d1 = np[1];
                                const float d[8] = {d0.x, d0.y, d0.z, d0.w, d1.x, d1.y, d1.z, d1.w};
#pragma unroll
                                for (int i = 0; i < 8; ++i) e[i] = __uint_as_float(gr[q * 8 + i]) * (far * d[i]);
                                lightning_split8(e, hi[g * 2 + q], lo[g * 2 + q]);
                            }
                        }
                    }
                }
                tc_fence_before_sync();
                if (!wait(yi_bar, par)) break;
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const uint32_t off = unit(r, q);
                    *reinterpret_cast<uint4*>(sQ + off) = hi[q];
                    *reinterpret_cast<uint4*>(sS + off) = lo[q];
                }
                fence_proxy_async_smem();
                mbar_arrive(p_full);
                const T* gp = reinterpret_cast<const T*>(p.rows) + ((size_t)t_first + row_first) * p.ld + p.g_off + col + (lane & 3) * 8;
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    gate[q] = row_first + q * 8 < ql ? __ldg(reinterpret_cast<const uint4*>(gp + (size_t)q * 8 * p.ld)) : make_uint4(0, 0, 0, 0);
            }
            if (!wait(y_bar, par)) break;
            float o[STATE_ONLY ? 1 : 32];
            if constexpr (!STATE_ONLY) {
                // ---- read-outs: P V + λ^{r+1} Q S ----
                const float carry_in = sPw[r + 1];
#pragma unroll
                for (int g = 0; g < 2; ++g) {
                    uint32_t y[16], yi[16];
                    tmem_ld_x16(lane_addr + kColY + quarter * 32 + g * 16, y);
                    tmem_ld_x16(lane_addr + kColYI + quarter * 32 + g * 16, yi);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[g * 16 + i] = fmaf(carry_in, __uint_as_float(yi[i]), __uint_as_float(y[i]));
                }
            }
            // ---- state: decayed in registers, plus the update ----
            {
                const float keep = sPw[len];
#pragma unroll
                for (int g = 0; g < kOwn / 16; ++g) {
                    uint32_t u[16];
                    tmem_ld_x16(lane_addr + kColS + quarter * kOwn + g * 16, u);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) S[g * 16 + i] = fmaf(keep, S[g * 16 + i], __uint_as_float(u[i]));
                }
            }
            if (c + 1 < nchunks) publish_state();
            if constexpr (!STATE_ONLY) {
                // ---- outputs, under the next chunk's loads and first products.  The products have read the weighted V; in the units that
                // only this warp writes there, lanes that fetched pieces of rows pass them to the rows' lanes and take the results back ----
                const size_t width = (size_t)p.heads * p.dv;
#pragma unroll
                for (int q = 0; q < 4; ++q) *reinterpret_cast<uint4*>(sW + unit(quad * 32 + q * 8 + (lane >> 2), lane & 3)) = gate[q];
                __syncwarp();
                float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    uint4* mine = reinterpret_cast<uint4*>(sW + unit(r, q));
                    const uint4 gu = *mine;
                    const T* ge = reinterpret_cast<const T*>(&gu);
                    const float4* wp = reinterpret_cast<const float4*>(sNw + quarter * 32 + q * 8);
                    const float4 w0 = wp[0], w1 = wp[1];
                    const float w8[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
                    float y[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        part[i & 3] = fmaf(o[q * 8 + i], o[q * 8 + i], part[i & 3]);
                        y[i] = lightning_gate<T>(o[q * 8 + i], w8[i], Cvt<T>::to_f(ge[i]));
                    }
                    uint4 ou;
                    ou.x = Cvt<T>::pack2(y[0], y[1]);
                    ou.y = Cvt<T>::pack2(y[2], y[3]);
                    ou.z = Cvt<T>::pack2(y[4], y[5]);
                    ou.w = Cvt<T>::pack2(y[6], y[7]);
                    *mine = ou;
                }
                if (valid) p.sums[(t * width + col) / 32] = (part[0] + part[1]) + (part[2] + part[3]);
                __syncwarp();
                T* op = reinterpret_cast<T*>(p.out) + ((size_t)t_first + row_first) * width + col + (lane & 3) * 8;
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (row_first + q * 8 < ql)
                        *reinterpret_cast<uint4*>(op + (size_t)q * 8 * width) = *reinterpret_cast<const uint4*>(sW + unit(quad * 32 + q * 8 + (lane >> 2), lane & 3));
                __syncwarp();                             // before this warp's next weighted V
            }
        }
        if (ok && (STATE_ONLY || last_seg)) {
            float* dst = STATE_ONLY ? carry : slot;
#pragma unroll
            for (int j = 0; j < kOwn; ++j) dst[(size_t)(quarter * kOwn + j) * p.dv] = S[j];
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

// Chain the segments of every sequence: in p.carry, local end states become the states in front of the segments.
__global__ void __launch_bounds__(256) lightning_carry_kernel(const __grid_constant__ LightningParams p) {
    pdl_prologue();
    const int sh = blockIdx.x, seq = sh / p.heads, h = sh - seq * p.heads;
    const int ql = p.q_len[seq], seg_rows = p.seg_chunks * kLtL;
    if (ql <= 0) return;
    const int n = (ql + seg_rows - 1) / seg_rows;
    const size_t e = ((size_t)blockIdx.y * 256 + threadIdx.x) * 4, size = (size_t)p.dk * p.dv;
    if (e >= size) return;
    const float chunk = p.powers[(size_t)h * p.n_powers + kLtL];
    float keep = 1.f;
    for (int i = 0; i < p.seg_chunks; ++i) keep *= chunk;
    float4 cur = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.past_len[seq] > 0) cur = *reinterpret_cast<const float4*>(p.state + ((size_t)p.slot_ids[seq] * p.heads + h) * size + e);
    float* seg = p.carry + (size_t)sh * p.segments * size + e;
    constexpr int kAhead = 8;                             // segments whose loads are in flight together
    for (int s0 = 0; s0 < n; s0 += kAhead) {
        float4 local[kAhead];
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            local[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (s0 + i + 1 < n) local[i] = *reinterpret_cast<const float4*>(seg + (size_t)(s0 + i) * size);
        }
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            if (s0 + i >= n) break;
            *reinterpret_cast<float4*>(seg + (size_t)(s0 + i) * size) = cur;
            cur = make_float4(fmaf(cur.x, keep, local[i].x), fmaf(cur.y, keep, local[i].y), fmaf(cur.z, keep, local[i].z), fmaf(cur.w, keep, local[i].w));
        }
    }
}

template <int DK, bool STATE_ONLY>
static int launch_lightning(const CUtensorMap& tma, const LightningParams& p, cudaStream_t stream) {
    constexpr int smem = DK / 64 * 16384 + 32768 + 65536 + (STATE_ONLY ? 0 : 32768 + DK / 64 * 32768) + 528 + 512 + 128 + 128 + 1024;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(lightning_chunk_kernel<DK, STATE_ONLY>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(lightning_chunk)", e);
        configured = true;
    }
    const int segs = STATE_ONLY ? p.segments - 1 : p.segments;
    TELB_LAUNCH("lightning_chunk_kernel", (lightning_chunk_kernel<DK, STATE_ONLY>), dim3((unsigned)(p.num_seqs * p.heads * (p.dv / 128) * segs)), dim3(kLtThreads),
                smem, stream, tma, p);
    TELB_CHECK_LAUNCH("lightning_chunk_kernel");
    return 0;
}

template <int DK>
static int run_chunks(const CUtensorMap& tma, const LightningParams& p, cudaStream_t stream) {
    if (p.segments > 1) {
        if (launch_lightning<DK, true>(tma, p, stream)) return -1;
        TELB_LAUNCH("lightning_carry_kernel", lightning_carry_kernel, dim3(p.num_seqs * p.heads, (DK * p.dv / 4 + 255) / 256), dim3(256), 0, stream, p);
        TELB_CHECK_LAUNCH("lightning_carry_kernel");
    }
    return launch_lightning<DK, false>(tma, p, stream);
}

}  // namespace telb

using namespace telb;

extern "C" int telb_lightning_act(const LightningParams* p, cudaStream_t stream);

// Chunked prefill (see the top of the file): bf16, key heads padded to 64 or 128, value heads to a multiple of 128.  p->act is scratch for the
// activated q | k | v; with p->segments > 1, p->carry too, and no sequence has more than segments * seg_chunks chunks of 128 rows.
extern "C" int telb_lightning_chunk(const LightningParams* p, cudaStream_t stream) {
    if (p->num_seqs <= 0 || p->tokens <= 0) return 0;
    if ((p->dk != 64 && p->dk != 128) || p->dv % 128 || p->n_powers <= kLtL) return fail("telb_lightning_chunk: key heads of 64 or 128, value heads in multiples of 128, 128 powers");
    if (p->ld % 8 || p->g_off % 8 || !p->act) return fail("telb_lightning_chunk: row pitches are multiples of 8, and the activations need their buffer");
    if (p->segments < 1 || (p->segments > 1 && (!p->carry || p->seg_chunks < 1))) return fail("telb_lightning_chunk: segments need their states and a length");
    if (telb_lightning_act(p, stream)) return -1;
    CUtensorMap tma;
    if (make_tmap_2d(&tma, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p->act, p->tokens, p->g_off, (uint64_t)p->g_off * 2, kLtL, 64, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    return p->dk == 64 ? run_chunks<64>(tma, *p, stream) : run_chunks<128>(tma, *p, stream);
}
