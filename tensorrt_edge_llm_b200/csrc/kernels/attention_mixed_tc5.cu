// Attention with scores mixed across heads, on tcgen05, over wide queries (mixed_heads.cu): head h has one query [hkv * pad] that meets the keys
// of all KV heads side by side; its values are those of its own KV head.  Scores lose slope_h * distance, rows see a window, heads leave
// times sigmoid(gate).
//
//   mixed_decode    few rows per sequence.  Every (token, head) pair is a column against the same cached tokens:
//                       Sᵀ[TILE tok, NC] = keys[TILE tok, hkv * pad] · Qᵀ     Oᵀ[128, NC] += valuesᵀ[128, TILE tok] · Pᵀ  per 128 value features
//                   A tile's keys, then its values stream through one ring in pairs of 64-feature chunks; a pair's slot is refilled as
//                   soon as its products are done.  All columns meet all value heads (the products are as narrow as they get); a
//                   column's output is read from the block of its own head.
//   mixed_prefill   prompt portions.  128 rows of one head per CTA; wide queries stay in shared memory, chunks of 128 keys x 64 features stream
//                   through a ring, so that scores of the next tile start while chunks of it still arrive.  Two softmax warpgroups take
//                   64 keys of a tile each, with maxima, sums and outputs of their own, which join at the end; probabilities stay in
//                   TMEM (the A operand of P·V), over the scores they were made from.
//
// HQ = 2: queries come as a high and a low half (2^-17 together), in mixed_decode as further columns, in mixed_prefill as further products.
// Probabilities enter P·V as a high and a low half.  Scores, bias, maxima and sums are fp32.  The producer and the MMA warp walk their loops
// as whole warps and elect a lane only for the instructions themselves.  All waits are bounded.
#include "attention_common.cuh"
#include "host_utils.h"

namespace telb {

using MixT = __nv_bfloat16;
constexpr int kMixPage = 64;
constexpr int kMixSmemLimit = 227 * 1024;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float mix_sigmoid(float g) { return 1.f / (1.f + exp2f(-g * kLog2e)); }

// ---- decode ----------------------------------------------------------------------------------------------
constexpr int kMixMaxSlots = 16;
constexpr int kMixMaxSplits = 64;

struct MixedDecParams {
    void* out;                   // [T, heads * pad]
    float* ws_o;                 // [splits, T * heads, pad] (splits > 1)
    float* ws_lse;               // [splits, T * heads], log2 domain
    const void* gate;            // [T, ld_gate] or null
    const float* slopes;         // [heads]
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* page_table;
    int max_pages, heads, hkv, pad, splits, rows, slots, window, slabs;
    long long ld_gate;
    float scale_log2;
    int* status;
};

constexpr int kMixThreadsDec = 192;

// grid (column blocks, splits, sequences).  NC: (token, head) columns of a block; TILE: cached tokens of a tile, one or two pages.
template <int NC, int TILE, int HQ>
__global__ void __launch_bounds__(kMixThreadsDec, NC == 16 && TILE == 64 ? 2 : 1)
mixed_decode_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_kv, const __grid_constant__ MixedDecParams p) {
    constexpr int NS = HQ * NC;                          // score columns: high halves of the queries, then low ones
    constexpr int kQChunk = NS * 128, kPSpan = 2 * NC * 128, kPBytes = TILE / 64 * kPSpan;
    constexpr int kChunk = TILE * 128, kSlot = 2 * kChunk;
    constexpr int kOCol = 4 * NS, kOBlock = 2 * NC;      // TMEM: four partial scores, then per 128 value features high | low columns
    constexpr int kTmemCols = kOCol + 4 * kOBlock <= 256 ? 256 : 512;
    static_assert(kOCol + 4 * kOBlock <= 512, "scores and four output blocks");

    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int cpp = p.pad / 64, chunks = p.hkv * cpp, pairs = (chunks + 1) / 2;      // chunks of a row's keys (and of its values)
    uint8_t* s_kv = smem;
    uint8_t* s_q = s_kv + p.slots * kSlot;
    uint8_t* s_p = s_q + chunks * kQChunk;
    uint64_t* bars = reinterpret_cast<uint64_t*>(s_p + kPBytes);
    uint64_t* q_full = bars;
    uint64_t* s_full = bars + 1;
    uint64_t* p_full = bars + 2;
    uint64_t* o_done = bars + 3;
    uint64_t* kv_full = bars + 4;
    uint64_t* kv_empty = kv_full + kMixMaxSlots;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(kv_empty + kMixMaxSlots);
    volatile uint32_t* abort_flag = tmem_slot + 1;
    float* s_red = reinterpret_cast<float*>(tmem_slot + 4);          // [2][4 warps][NC] maxima, then sums
    float* s_slope = s_red + 8 * NC;                                 // per column: slope (log2 units), position, head
    int* s_pos = reinterpret_cast<int*>(s_slope + NC);
    int* s_head = s_pos + NC;

    pdl_wait();                                          // dependents start once TMEM is allocated: theirs must not come first
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seq = blockIdx.z, split = blockIdx.y, cb = blockIdx.x;
    const int qlen = p.q_len[seq], past = p.past_len[seq];
    const int ncol = min(NC, qlen * p.heads - cb * NC);
    if (ncol <= 0) return;                               // uniform, before any barrier or TMEM use
    const int row0 = p.q_start[seq] * p.heads + cb * NC; // first (token, head) row of the block
    const int first_pos = past + cb * NC / p.heads, last_pos = past + (cb * NC + ncol - 1) / p.heads;
    const int tile_lo = max(0, first_pos - p.window + 1) / TILE, tile_hi = last_pos / TILE + 1;
    const int per = (tile_hi - tile_lo + p.splits - 1) / p.splits;
    const int j0 = tile_lo + split * per;
    const int ntiles = max(0, min(tile_hi, j0 + per) - j0);

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        mbar_init(s_full, 1);
        mbar_init(p_full, 128);
        mbar_init(o_done, 1);
        for (int s = 0; s < p.slots; ++s) {
            mbar_init(&kv_full[s], 1);
            mbar_init(&kv_empty[s], 1);
        }
        *abort_flag = 0;
        mbar_fence_init();
        prefetch_tensormap(&tma_q);
        prefetch_tensormap(&tma_kv);
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, kTmemCols);
        tmem_relinquish();
    }
    if (threadIdx.x >= 64 && threadIdx.x < 64 + NC) {
        const int c = threadIdx.x - 64, col = cb * NC + min(c, ncol - 1);
        s_head[c] = col % p.heads;
        s_pos[c] = past + col / p.heads;
        s_slope[c] = p.slopes[col % p.heads] * kLog2e;
    }
    for (int i = threadIdx.x; i < kPBytes / 16; i += kMixThreadsDec) reinterpret_cast<uint4*>(s_p)[i] = make_uint4(0, 0, 0, 0);
    fence_proxy_async_smem();
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem_base = *tmem_slot;
    pdl_launch_dependents();

    if (warp == 0) {
        // ---- producer: per tile the keys of all heads, then the values ----
        if (ntiles > 0) {
            const bool leader = elect_one();
            if (leader) {
                mbar_expect_tx(q_full, chunks * kQChunk);
                for (int c = 0; c < chunks; ++c)
#pragma unroll
                    for (int h = 0; h < HQ; ++h) tma_load_2d(s_q + c * kQChunk + h * NC * 128, &tma_q, q_full, (h * chunks + c) * 64, row0);
            }
            const int* pages = p.page_table + (size_t)seq * p.max_pages;
            bool ok = true;
            int slot = 0;
            uint32_t ph = 1;
            constexpr int kPages = TILE / kMixPage, kAhead = 32 / kPages;
            int next = 0;                                // the pages of kAhead tiles are fetched at a time
            for (int j = 0; j < ntiles && ok; ++j) {
                if (j % kAhead == 0) {
                    const int lp = (j0 + j) * kPages + lane;
                    next = lp < p.max_pages ? pages[lp] : -1;
                }
                int page[kPages];                        // tokens past the end are masked
#pragma unroll
                for (int h = 0; h < kPages; ++h) page[h] = max(__shfl_sync(0xffffffffu, next, j % kAhead * kPages + h), 0);
                for (int pr = 0; pr < 2 * pairs; ++pr) {
                    ok = __all_sync(0xffffffffu, mbar_wait(&kv_empty[slot], ph, abort_flag, p.status, kStatusProducerTimeout));
                    if (!ok) break;
                    uint8_t* dst = s_kv + slot * kSlot;
                    const int plane = pr >= pairs ? 1 : 0, c0 = (pr - plane * pairs) * 2;
                    if (leader) {
                        mbar_expect_tx(&kv_full[slot], kSlot);
#pragma unroll
                        for (int c = 0; c < 2; ++c)
#pragma unroll
                            for (int h = 0; h < kPages; ++h) {
                                const int ch = c0 + c, head = ch / cpp;
                                const int slab = ch < chunks ? (page[h] * 2 + plane) * p.hkv + head : p.slabs;      // past the end: zeros
                                tma_load_4d(dst + c * kChunk + h * (kMixPage * 128), &tma_kv, &kv_full[slot], 0, 0, ch - head * cpp, slab);
                            }
                    }
                    if (++slot == p.slots) {
                        slot = 0;
                        ph ^= 1;
                    }
                }
            }
        }
    } else if (warp == 1) {
        // ---- MMA issuer ----
        if (ntiles > 0) {
            const bool leader = elect_one();
            constexpr uint32_t idesc_s = idesc_f16(128, NS, true), idesc_o = idesc_f16(128, 2 * NC, true, true);
            const uint64_t desc_kv = smem_desc_sw128(s_kv), desc_v = smem_desc_sw128_mn(s_kv, kChunk, 1024), desc_q = smem_desc_sw128(s_q),
                           desc_p = smem_desc_sw128(s_p);
            bool ok = __all_sync(0xffffffffu, mbar_wait(q_full, 0, abort_flag, p.status, kStatusMmaTimeout));
            int slot = 0;
            uint32_t ph = 0;
            auto advance = [&]() {
                if (++slot == p.slots) {
                    slot = 0;
                    ph ^= 1;
                }
            };
            for (int j = 0; j < ntiles && ok; ++j) {
                for (int pr = 0; pr < pairs; ++pr) {
                    ok = __all_sync(0xffffffffu, mbar_wait(&kv_full[slot], ph, abort_flag, p.status, kStatusMmaTimeout));
                    if (!ok) break;
                    tc_fence_after_sync();
                    const bool two = pr * 2 + 1 < chunks;
                    const uint64_t dk = desc_kv + (uint64_t)((slot * kSlot) >> 4), dq = desc_q + (uint64_t)((pr * 2 * kQChunk) >> 4);
                    if (leader) {
#pragma unroll
                        for (int k = 0; k < 4; ++k) umma_f16(tmem_base + k * NS, dk + 2 * k, dq + 2 * k, idesc_s, pr ? 1u : 0u);
                        if (two) {
#pragma unroll
                            for (int k = 0; k < 4; ++k)
                                umma_f16(tmem_base + k * NS, dk + (kChunk >> 4) + 2 * k, dq + (kQChunk >> 4) + 2 * k, idesc_s, 1u);
                        }
                        umma_commit(&kv_empty[slot]);
                        if (pr == pairs - 1) umma_commit(s_full);
                    }
                    __syncwarp();
                    advance();
                }
                ok = ok && __all_sync(0xffffffffu, mbar_wait(p_full, j & 1, abort_flag, p.status, kStatusMmaTimeout));
                if (!ok) break;
                tc_fence_after_sync();
                for (int b = 0; b < pairs; ++b) {
                    ok = __all_sync(0xffffffffu, mbar_wait(&kv_full[slot], ph, abort_flag, p.status, kStatusMmaTimeout));
                    if (!ok) break;
                    tc_fence_after_sync();
                    const uint64_t dv = desc_v + (uint64_t)((slot * kSlot) >> 4);
                    const uint32_t d_o = tmem_base + kOCol + b * kOBlock;
                    if (leader) {
#pragma unroll
                        for (int k = 0; k < TILE / 16; ++k)
                            umma_f16(d_o, dv + (uint64_t)((k * 2048) >> 4), desc_p + (uint64_t)(((k >> 2) * kPSpan) >> 4) + 2 * (k & 3), idesc_o, (j | k) ? 1u : 0u);
                        umma_commit(&kv_empty[slot]);
                        if (j == ntiles - 1 && b == pairs - 1) umma_commit(o_done);
                    }
                    __syncwarp();
                    advance();
                }
            }
        }
    } else {
        // ---- softmax / epilogue ----
        const int quad = warp & 3, r = quad * 32 + lane; // cached token within the tile (S), feature within a block (O)
        const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quad * 32) << 16);
        float m_used[NC], l_part[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            m_used[c] = c < ncol ? -INFINITY : INFINITY;
            l_part[c] = 0.f;
        }
        bool ok = true;
        for (int j = 0; j < ntiles && ok; ++j) {
            // the scores of tile j were issued behind P·V of tile j - 1: both are complete now, so P and O may be touched
            if (!mbar_wait(s_full, j & 1, abort_flag, p.status, kStatusEpilogueTimeout)) { ok = false; break; }
            tc_fence_after_sync();
            float s[NC];
#pragma unroll
            for (int c = 0; c < NC; c += 16) {
#pragma unroll
                for (int h = 0; h < HQ; ++h) {
                    uint32_t r0[16], r1[16], r2[16], r3[16];
                    const uint32_t a = lane_addr + h * NC + c;
                    tmem_ld_x16(a, r0);
                    tmem_ld_x16(a + NS, r1);
                    tmem_ld_x16(a + 2 * NS, r2);
                    tmem_ld_x16(a + 3 * NS, r3);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        const float v = __uint_as_float(r0[i]) + __uint_as_float(r1[i]) + (__uint_as_float(r2[i]) + __uint_as_float(r3[i]));
                        s[c + i] = h ? s[c + i] + v : v;
                    }
                }
            }
            const int t0 = (j0 + j) * TILE, tk = t0 + r;
            if (r >= TILE) {                             // lanes behind the tile only help to rescale and to write the output
#pragma unroll
                for (int c = 0; c < NC; ++c) s[c] = -INFINITY;
            } else {
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const int gap = s_pos[c] - tk;
                    s[c] = gap >= 0 && gap < p.window ? fmaf(s[c], p.scale_log2, -s_slope[c] * (float)gap) : -INFINITY;
                }
            }
            // the reference of a column moves only when a score exceeds it by 2^8: most tiles need no maximum
            bool over = false;
#pragma unroll
            for (int c = 0; c < NC; ++c) over = over || s[c] > m_used[c] + 8.0f;
            if (lat_any(over)) {
                float* red = s_red + (j & 1) * 4 * NC;
                float f[NC];
                const float wm = lat_column_max<NC>(s, lane);
                if (lane < NC) red[(warp - 2) * NC + lane] = wm;
                named_barrier_sync(1, 128);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float mt = fmaxf(fmaxf(red[c], red[NC + c]), fmaxf(red[2 * NC + c], red[3 * NC + c]));
                    const bool move = mt > m_used[c] + 8.0f;                      // uniform across the four warps
                    f[c] = !move ? 1.f : m_used[c] == -INFINITY ? 0.f : exp2f(m_used[c] - mt);
                    l_part[c] *= f[c];
                    if (move) m_used[c] = mt;
                }
                if (j > 0) {
                    for (int b = 0; b < pairs; ++b)
#pragma unroll
                        for (int c = 0; c < 2 * NC; c += 16) {
                            uint32_t o[16];
                            tmem_ld_x16(lane_addr + kOCol + b * kOBlock + c, o);
                            tmem_ld_wait();
#pragma unroll
                            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f[(c + i) % NC]);
                            tmem_st_x16(lane_addr + kOCol + b * kOBlock + c, o);
                        }
                    tmem_st_wait();
                }
            }
            if (r < TILE) {
                uint8_t* prow = s_p + (r >> 6) * kPSpan + (r & 7) * 2;
                const int unit = (r & 63) >> 3;
#pragma unroll
                for (int c = 0; c < NC; ++c) {           // columns beyond ncol: reference +inf, probability zero
                    const float e = exp2f(s[c] - (m_used[c] == -INFINITY ? 0.f : m_used[c]));
                    l_part[c] += e;
                    uint8_t* dst = prow + (c >> 3) * 1024 + (c & 7) * 128 + ((unit ^ (c & 7)) << 4);
                    const MixT hi = Cvt<MixT>::from_f(e);
                    *reinterpret_cast<MixT*>(dst) = hi;
                    *reinterpret_cast<MixT*>(dst + NC * 128) = Cvt<MixT>::from_f(e - Cvt<MixT>::to_f(hi));
                }
            }
            fence_proxy_async_smem();
            tc_fence_before_sync();
            mbar_arrive(p_full);
        }
        named_barrier_sync(1, 128);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            float v = l_part[c];
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (lane == (c & 31)) s_red[(warp - 2) * NC + c] = v;
        }
        named_barrier_sync(1, 128);
        if (ok && ntiles > 0) ok = mbar_wait(o_done, 0, abort_flag, p.status, kStatusEpilogueTimeout);
        if (ok) {
            tc_fence_after_sync();
            float inv[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float l = s_red[c] + s_red[NC + c] + s_red[2 * NC + c] + s_red[3 * NC + c];
                const bool have = ntiles > 0 && l > 0.f;
                inv[c] = have ? 1.f / l : 0.f;
                if (p.splits > 1 && r == 0 && c < ncol) p.ws_lse[(size_t)split * p.rows + row0 + c] = have ? m_used[c] + log2f(l) : -INFINITY;
            }
            const int group = p.heads / p.hkv;
            for (int b = 0; b < pairs; ++b) {
                const int ch = 2 * b + (r >> 6), vh = ch / cpp, feat = (ch - vh * cpp) * 64 + (r & 63);      // value head and feature of this lane
#pragma unroll
                for (int c = 0; c < NC; c += 16) {
                    uint32_t o[16], lo[16];
                    tmem_ld_x16(lane_addr + kOCol + b * kOBlock + c, o);       // garbage (never used) without tiles
                    tmem_ld_x16(lane_addr + kOCol + b * kOBlock + NC + c, lo);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        if (c + i >= ncol) continue;
                        const int head = s_head[c + i];
                        if (head < vh * group || head >= (vh + 1) * group) continue;
                        const float v = inv[c + i] > 0.f ? (__uint_as_float(o[i]) + __uint_as_float(lo[i])) * inv[c + i] : 0.f;
                        const size_t row = (size_t)row0 + c + i;
                        if (p.splits == 1) {
                            const size_t tok = (size_t)p.q_start[seq] + s_pos[c + i] - past;
                            const float g = p.gate ? mix_sigmoid(Cvt<MixT>::to_f(reinterpret_cast<const MixT*>(p.gate)[tok * p.ld_gate + head * p.pad + feat])) : 1.f;
                            reinterpret_cast<MixT*>(p.out)[row * p.pad + feat] = Cvt<MixT>::from_f(v * g);
                        } else {
                            p.ws_o[((size_t)split * p.rows + row) * p.pad + feat] = v;
                        }
                    }
                }
            }
            tc_fence_before_sync();
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
        tmem_dealloc(tmem_base, kTmemCols);
    }
}

// out[row] = sigmoid(gate) * sum over splits of 2^(lse - max) O / sum of 2^(lse - max); one warp per (token, head) of the launch's sequences.
__global__ void __launch_bounds__(128) mixed_combine_kernel(const __grid_constant__ MixedDecParams p) {
    pdl_prologue();
    const int lane = threadIdx.x & 31, seq = blockIdx.y, col = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (col >= p.q_len[seq] * p.heads) return;
    const size_t row = (size_t)p.q_start[seq] * p.heads + col;
    float l[2], mx = -INFINITY, den = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int sp = i * 32 + lane;
        l[i] = sp < p.splits ? p.ws_lse[(size_t)sp * p.rows + row] : -INFINITY;
        mx = fmaxf(mx, l[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] = l[i] == -INFINITY ? 0.f : exp2f(l[i] - mx);
        den += l[i];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) den += __shfl_xor_sync(0xffffffffu, den, o);
    const float inv = den > 0.f ? 1.f / den : 0.f;
    const size_t tok = row / p.heads;
    const int head = (int)(row - tok * p.heads), i = lane * 4;           // pad is 64 or 128
    float a[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s = 0; s < p.splits; ++s) {
        const float w = __shfl_sync(0xffffffffu, s < 32 ? l[0] : l[1], s & 31) * inv;
        if (i >= p.pad) continue;
        const float4 v = __ldcg(reinterpret_cast<const float4*>(p.ws_o + ((size_t)s * p.rows + row) * p.pad + i));
        a[0] = fmaf(w, v.x, a[0]);
        a[1] = fmaf(w, v.y, a[1]);
        a[2] = fmaf(w, v.z, a[2]);
        a[3] = fmaf(w, v.w, a[3]);
    }
    if (i >= p.pad) return;
    if (p.gate) {
        const uint2 g2 = *reinterpret_cast<const uint2*>(reinterpret_cast<const MixT*>(p.gate) + tok * p.ld_gate + head * p.pad + i);
        const MixT* g = reinterpret_cast<const MixT*>(&g2);
#pragma unroll
        for (int k = 0; k < 4; ++k) a[k] *= mix_sigmoid(Cvt<MixT>::to_f(g[k]));
    }
    uint2 u;
    u.x = Cvt<MixT>::pack2(a[0], a[1]);
    u.y = Cvt<MixT>::pack2(a[2], a[3]);
    *reinterpret_cast<uint2*>(reinterpret_cast<MixT*>(p.out) + row * p.pad + i) = u;
}

// ---- prefill ---------------------------------------------------------------------------------------------
struct MixedPreParams {
    void* out;                   // [T, heads * pad]
    const void* gate;            // [T, ld_gate] or null
    const float* slopes;         // [heads]
    const int* q_start;          // first row of each sequence
    const int* q_len;
    const int* past_len;
    const int* page_table;
    int max_pages, heads, hkv, chunks, window, kslots, vstages;
    long long ld_gate;
    float scale_log2;
    int* status;
};

constexpr int kMixTile = 128;                // keys per tile: two pages, one per softmax warpgroup
constexpr int kMixKChunk = kMixTile * 128;   // bytes of [128 keys x 64 features]
constexpr int kMixQChunk = 128 * 128;        // bytes of [128 rows x 64 features]
constexpr int kMixKSlots = 8;
constexpr int kMixThreadsPre = 320;          // producer, MMA issuer, two softmax warpgroups

// grid (query tiles of 128 rows, heads, sequences).  VC: 64-feature chunks of a head.
template <int VC, int HQ>
__global__ void __launch_bounds__(kMixThreadsPre, 1)
mixed_prefill_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_kv, const __grid_constant__ MixedPreParams p) {
    constexpr int VP = VC * 64, kVStage = VC * kMixKChunk;
    // TMEM: two score buffers of 128 columns (64 of each warpgroup, which turn into its high | low probabilities), then an output per warpgroup
    constexpr uint32_t kOCol = 256, kTmemCols = 512;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int chunks = p.chunks;
    uint8_t* s_q = smem;                                  // [HQ][chunks]; at the end the warpgroups exchange halves of their outputs here
    uint8_t* s_k = s_q + HQ * chunks * kMixQChunk;
    uint8_t* s_v = s_k + p.kslots * kMixKChunk;
    uint64_t* bars = reinterpret_cast<uint64_t*>(s_v + p.vstages * kVStage);
    uint64_t* q_full = bars;
    uint64_t* s_full = bars + 1;                          // [buffer]
    uint64_t* p_full = s_full + 2;                        // [warpgroup][buffer]
    uint64_t* o_done = p_full + 4;                        // [warpgroup][buffer]: two in turn, so that a wait never meets the phase after next
    uint64_t* k_full = o_done + 4;
    uint64_t* k_empty = k_full + kMixKSlots;
    uint64_t* v_full = k_empty + kMixKSlots;
    uint64_t* v_empty = v_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(v_empty + 2);
    volatile uint32_t* abort_flag = tmem_slot + 1;

    pdl_wait();                                           // dependents start at the end: a long kernel runs slower under waiting ones
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int qt = gridDim.x - 1 - blockIdx.x;            // long rows first
    const int head = blockIdx.y, seq = blockIdx.z;
    const int qlen = p.q_len[seq], past = p.past_len[seq], tok0 = qt * 128;
    if (tok0 >= qlen) return;                             // uniform, before any barrier or TMEM use
    const int qrow0 = p.q_start[seq] + tok0, kvh = head / (p.heads / p.hkv);
    const int row_first = past + tok0, row_last = past + min(qlen, tok0 + 128) - 1;
    const int jlo = max(0, row_first - p.window + 1) / kMixTile, jhi = row_last / kMixTile + 1;      // key tiles [jlo, jhi)

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(&s_full[i], 1);
            mbar_init(&v_full[i], 1);
            mbar_init(&v_empty[i], 1);
        }
        for (int i = 0; i < 4; ++i) {
            mbar_init(&p_full[i], 128);
            mbar_init(&o_done[i], 1);
        }
        for (int s = 0; s < p.kslots; ++s) {
            mbar_init(&k_full[s], 1);
            mbar_init(&k_empty[s], 1);
        }
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, kTmemCols);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        // ---- producer: K(jlo); then K(j + 1), V(j) ----
        const bool leader = elect_one();
        const int* pages = p.page_table + (size_t)seq * p.max_pages;
        const int last_page = row_last / kMixPage;        // pages behind it hold nothing that a row sees: they read page 0, masked
        auto page_of = [&](int j, int half) { return 2 * j + half <= last_page ? max(pages[2 * j + half], 0) : 0; };
        int ks = 0, vs = 0;
        uint32_t kph = 1, vph = 1;
        auto load_keys = [&](int p0, int p1) {
            int part = 0, h = 0;
            for (int c = 0; c < chunks; ++c) {
                if (!__all_sync(0xffffffffu, mbar_wait(&k_empty[ks], kph, abort_flag, p.status, kStatusProducerTimeout))) return false;
                if (leader) {
                    mbar_expect_tx(&k_full[ks], kMixKChunk);
                    tma_load_4d(s_k + ks * kMixKChunk, &tma_kv, &k_full[ks], 0, 0, part, p0 * 2 * p.hkv + h);
                    tma_load_4d(s_k + ks * kMixKChunk + kMixKChunk / 2, &tma_kv, &k_full[ks], 0, 0, part, p1 * 2 * p.hkv + h);
                }
                if (++part == VC) {
                    part = 0;
                    ++h;
                }
                if (++ks == p.kslots) {
                    ks = 0;
                    kph ^= 1;
                }
            }
            return true;
        };
        int p0 = page_of(jlo, 0), p1 = page_of(jlo, 1), n0 = page_of(jlo + 1, 0), n1 = page_of(jlo + 1, 1);
        if (leader) {
            mbar_expect_tx(q_full, HQ * chunks * kMixQChunk);
            for (int c = 0; c < HQ * chunks; ++c) tma_load_3d(s_q + c * kMixQChunk, &tma_q, q_full, c * 64, head, qrow0);
        }
        bool ok = load_keys(p0, p1);
        for (int j = jlo; j < jhi && ok; ++j) {
            const int f0 = page_of(j + 2, 0), f1 = page_of(j + 2, 1);            // fetched a tile before they are used
            if (j + 1 < jhi) ok = load_keys(n0, n1);
            ok = ok && __all_sync(0xffffffffu, mbar_wait(&v_empty[vs], vph, abort_flag, p.status, kStatusProducerTimeout));
            if (!ok) break;
            if (leader) {
                mbar_expect_tx(&v_full[vs], kVStage);
#pragma unroll
                for (int c = 0; c < VC; ++c) {
                    uint8_t* dst = s_v + vs * kVStage + c * kMixKChunk;
                    tma_load_4d(dst, &tma_kv, &v_full[vs], 0, 0, c, (p0 * 2 + 1) * p.hkv + kvh);
                    tma_load_4d(dst + kMixKChunk / 2, &tma_kv, &v_full[vs], 0, 0, c, (p1 * 2 + 1) * p.hkv + kvh);
                }
            }
            if (++vs == p.vstages) {
                vs = 0;
                vph ^= 1;
            }
            p0 = n0, p1 = n1, n0 = f0, n1 = f1;
        }
    } else if (warp == 1) {
        // ---- MMA issuer: S(jlo); then S(j + 1), P·V(j) ----
        const bool leader = elect_one();
        constexpr uint32_t idesc_s = idesc_f16(128, kMixTile, true), idesc_o = idesc_f16(128, VP, true, false, true);
        const uint64_t desc_q = smem_desc_sw128(s_q), desc_k = smem_desc_sw128(s_k), desc_v = smem_desc_sw128_mn(s_v, kMixKChunk, 1024);
        auto wait = [&](uint64_t* bar, uint32_t parity) {
            const bool got = __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, p.status, kStatusMmaTimeout));
            tc_fence_after_sync();
            return got;
        };
        int ks = 0, vs = 0;                               // ring positions of the next key chunk and value tile
        uint32_t kph = 0, vph = 0;
        auto issue_s = [&](int n) {                       // n: tile counted from jlo
            const uint32_t d = tmem_base + (n & 1) * kMixTile;
            for (int c = 0; c < chunks; ++c) {
                if (!wait(&k_full[ks], kph)) return false;
                const uint64_t dk = desc_k + (uint64_t)((ks * kMixKChunk) >> 4), dq = desc_q + (uint64_t)((c * kMixQChunk) >> 4);
                if (leader) {
#pragma unroll
                    for (int h = 0; h < HQ; ++h)
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            umma_f16(d, dq + (uint64_t)((h * chunks * kMixQChunk) >> 4) + 2 * k, dk + 2 * k, idesc_s, (c | h | k) ? 1u : 0u);
                    umma_commit(&k_empty[ks]);
                    if (c == chunks - 1) umma_commit(&s_full[n & 1]);
                }
                __syncwarp();
                if (++ks == p.kslots) {
                    ks = 0;
                    kph ^= 1;
                }
            }
            return true;
        };
        const int ntiles = jhi - jlo;
        bool ok = wait(q_full, 0) && issue_s(0);
        for (int n = 0; n < ntiles && ok; ++n) {
            if (n + 1 < ntiles) ok = issue_s(n + 1);
            ok = ok && wait(&v_full[vs], vph);
            const uint64_t dv = desc_v + (uint64_t)((vs * kVStage) >> 4);
#pragma unroll
            for (int g = 0; g < 2; ++g) {
                ok = ok && wait(&p_full[g * 2 + (n & 1)], (n >> 1) & 1);
                if (!ok) break;
                const uint32_t a = tmem_base + (n & 1) * kMixTile + g * 64, d = tmem_base + kOCol + g * 128;
                if (leader) {
#pragma unroll
                    for (int half = 0; half < 2; ++half)
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            umma_f16_ts(d, a + half * 32 + k * 8, dv + (uint64_t)(((g * 4 + k) * 2048) >> 4), idesc_o, (n | half | k) ? 1u : 0u);
                    umma_commit(&o_done[g * 2 + (n & 1)]);
                    if (g == 1) umma_commit(&v_empty[vs]);
                }
                __syncwarp();
            }
            if (++vs == p.vstages) {
                vs = 0;
                vph ^= 1;
            }
        }
    } else {
        // ---- softmax / epilogue: warpgroup g takes keys g * 64 .. + 63 of every tile, one thread per query row ----
        const int g = (warp - 2) >> 2, quad = warp & 3;
        const int r = quad * 32 + lane, qi = tok0 + r, ntiles = jhi - jlo;
        const uint32_t base = tmem_base + (static_cast<uint32_t>(quad * 32) << 16), s_col = base + g * 64, o_col = base + kOCol + g * 128;
        const int limit = past + qi;                      // last visible key
        const float slope = p.slopes[head] * kLog2e;
        float m_used = -INFINITY, l_sum = 0.f;
        bool ok = true;
        for (int n = 0; n < ntiles && ok; ++n) {
            const int b = n & 1;
            if (!mbar_wait(&s_full[b], (n >> 1) & 1, abort_flag, p.status, kStatusEpilogueTimeout)) { ok = false; break; }
            tc_fence_after_sync();
            float s[64];
            {
                uint32_t r0[32], r1[32];
                tmem_ld_x32(s_col + b * kMixTile, r0);
                tmem_ld_x32(s_col + b * kMixTile + 32, r1);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    s[i] = __uint_as_float(r0[i]);
                    s[32 + i] = __uint_as_float(r1[i]);
                }
            }
            const int c0 = (jlo + n) * kMixTile + g * 64;
            const float bias = slope * (float)(c0 - limit);
#pragma unroll
            for (int i = 0; i < 64; ++i) s[i] = fmaf(s[i], p.scale_log2, fmaf(slope, (float)i, bias));
            if (c0 + 63 > row_first || c0 <= row_last - p.window) {                 // the keys reach the diagonal or the window's start
#pragma unroll
                for (int i = 0; i < 64; ++i) s[i] = c0 + i <= limit && c0 + i > limit - p.window ? s[i] : -INFINITY;
            }
            float mx[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
            for (int i = 4; i < 64; ++i) mx[i & 3] = fmaxf(mx[i & 3], s[i]);
            const float m_new = fmaxf(m_used, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])));
            const bool need = m_new > m_used + 8.0f;
            if (n == 0) {
                m_used = m_new;
            } else if (__any_sync(0xffffffffu, need)) {
                // P·V of tile n - 1 (that of tile n - 2 was issued ahead of these scores and is complete)
                if (!mbar_wait(&o_done[g * 2 + (b ^ 1)], ((n - 1) >> 1) & 1, abort_flag, p.status, kStatusEpilogueTimeout)) { ok = false; break; }
                tc_fence_after_sync();
                const float f = need ? exp2f(m_used - m_new) : 1.f;
#pragma unroll 1
                for (int c = 0; c < VP / 16; ++c) {
                    uint32_t o[16];
                    tmem_ld_x16(o_col + c * 16, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
                    tmem_st_x16(o_col + c * 16, o);
                }
                if (need) {
                    l_sum *= f;
                    m_used = m_new;
                }
            }
            const float mref = m_used == -INFINITY ? 0.f : m_used;
            float acc[2] = {0.f, 0.f};
#pragma unroll
            for (int h = 0; h < 2; ++h) {                             // 32 keys at a time: 16 columns of high halves, 16 of low ones
                uint32_t hw[16], lw[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float e0 = exp2f(s[h * 32 + 2 * i] - mref), e1 = exp2f(s[h * 32 + 2 * i + 1] - mref);
                    acc[0] += e0;
                    acc[1] += e1;
                    hw[i] = Cvt<MixT>::pack2(e0, e1);
                    const MixT* q = reinterpret_cast<const MixT*>(&hw[i]);
                    lw[i] = Cvt<MixT>::pack2(e0 - Cvt<MixT>::to_f(q[0]), e1 - Cvt<MixT>::to_f(q[1]));
                }
                tmem_st_x16(s_col + b * kMixTile + h * 16, hw);
                tmem_st_x16(s_col + b * kMixTile + 32 + h * 16, lw);
            }
            l_sum += acc[0] + acc[1];
            tmem_st_wait();
            tc_fence_before_sync();
            mbar_arrive(&p_full[g * 2 + b]);
        }
        // ---- the two halves of a row join: each warpgroup hands over the features that the other one writes ----
        constexpr int kHalf = VP / 2, kPitch = kHalf + 4;             // fp32 words of a row's half in shared memory, padded
        const size_t tok = (size_t)p.q_start[seq] + qi;
        const MixT* gate = p.gate && qi < qlen ? reinterpret_cast<const MixT*>(p.gate) + tok * p.ld_gate + head * VP + g * kHalf : nullptr;
        if (ok) ok = mbar_wait(&o_done[g * 2 + ((ntiles - 1) & 1)], ((ntiles - 1) >> 1) & 1, abort_flag, p.status, kStatusEpilogueTimeout);
        // Q is read by score products only, and those of the last tile are complete: its room is free
        float* mine = reinterpret_cast<float*>(s_q) + ((size_t)g * 128 + r) * kPitch;
        const float* theirs = reinterpret_cast<const float*>(s_q) + ((size_t)(g ^ 1) * 128 + r) * kPitch;
        float* s_ml = reinterpret_cast<float*>(s_q) + 256 * kPitch;   // [warpgroup][maximum | sum][row]
        if (ok) {
            tc_fence_after_sync();
            s_ml[g * 256 + r] = m_used;
            s_ml[g * 256 + 128 + r] = l_sum;
#pragma unroll 1
            for (int c = 0; c < kHalf / 16; ++c) {
                uint32_t o[16];
                tmem_ld_x16(o_col + (g ^ 1) * kHalf + c * 16, o);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    *reinterpret_cast<uint4*>(mine + c * 16 + i * 4) = make_uint4(o[i * 4], o[i * 4 + 1], o[i * 4 + 2], o[i * 4 + 3]);
            }
        }
        named_barrier_sync(1, 256);
        if (ok && *abort_flag == 0) {
            const float om = s_ml[(g ^ 1) * 256 + r], ol = s_ml[(g ^ 1) * 256 + 128 + r], m = fmaxf(m_used, om);
            float f0 = m_used == -INFINITY ? 0.f : exp2f(m_used - m), f1 = om == -INFINITY ? 0.f : exp2f(om - m);
            const float l = l_sum * f0 + ol * f1, inv = l > 0.f ? 1.f / l : 0.f;
            f0 *= inv;
            f1 *= inv;
            MixT* dst = reinterpret_cast<MixT*>(p.out) + (tok * p.heads + head) * VP + g * kHalf;
#pragma unroll
            for (int c = 0; c < kHalf / 16; ++c) {
                uint32_t o[16];
                tmem_ld_x16(o_col + g * kHalf + c * 16, o);
                alignas(16) MixT gv[16];
                if (gate) {
#pragma unroll
                    for (int i = 0; i < 2; ++i) reinterpret_cast<uint4*>(gv)[i] = reinterpret_cast<const uint4*>(gate + c * 16)[i];
                }
                tmem_ld_wait();
                if (qi < qlen) {
                    float v[16];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float4 t = *reinterpret_cast<const float4*>(theirs + c * 16 + i * 4);
                        v[i * 4] = __uint_as_float(o[i * 4]) * f0 + t.x * f1;
                        v[i * 4 + 1] = __uint_as_float(o[i * 4 + 1]) * f0 + t.y * f1;
                        v[i * 4 + 2] = __uint_as_float(o[i * 4 + 2]) * f0 + t.z * f1;
                        v[i * 4 + 3] = __uint_as_float(o[i * 4 + 3]) * f0 + t.w * f1;
                    }
                    if (gate) {
#pragma unroll
                        for (int i = 0; i < 16; ++i) v[i] *= mix_sigmoid(Cvt<MixT>::to_f(gv[i]));
                    }
                    uint32_t w[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) w[i] = Cvt<MixT>::pack2(v[2 * i], v[2 * i + 1]);
                    reinterpret_cast<uint4*>(dst + c * 16)[0] = make_uint4(w[0], w[1], w[2], w[3]);
                    reinterpret_cast<uint4*>(dst + c * 16)[1] = make_uint4(w[4], w[5], w[6], w[7]);
                }
                __syncwarp();
            }
            tc_fence_before_sync();
        }
    }
    if (*abort_flag) {
        const uint64_t t0 = global_timer_ns();
        while (global_timer_ns() - t0 < 200000ull) __nanosleep(1000);
    }
    tc_fence_before_sync();
    __syncthreads();
    pdl_launch_dependents();
    if (warp == 1) {
        tc_fence_after_sync();
        tmem_dealloc(tmem_base, kTmemCols);
    }
}

template <int NC, int TILE, int HQ>
static int launch_mixed_decode(const CUtensorMap& tq, const CUtensorMap& tkv, MixedDecParams p, int nseq, int max_cols, cudaStream_t stream) {
    // the score MMA of one-page tiles reads one chunk beyond the last slot: Q and P, and a spare
    constexpr int chunk = TILE * 128, slot = 2 * chunk, ctas = NC == 16 && TILE == 64 ? 2 : 1;
    const int chunks = p.hkv * p.pad / 64;
    const int fixed = chunks * HQ * NC * 128 + TILE / 64 * 2 * NC * 128 + (4 + 2 * kMixMaxSlots) * 8 + 16 + (8 + 3) * NC * 4 + 1024 + (TILE == 64 ? chunk : 0);
    p.slots = (kMixSmemLimit / ctas - (ctas - 1) * 1024 - fixed) / slot;
    if (p.slots > kMixMaxSlots) p.slots = kMixMaxSlots;
    if (p.slots < 2) return fail("telb_mixed_attention_decode: rows too wide for shared memory");
    const int smem = fixed + p.slots * slot;
    static int configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(mixed_decode_kernel<NC, TILE, HQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(mixed_decode)", e);
        configured = smem;
    }
    TELB_LAUNCH("mixed_decode_kernel", (mixed_decode_kernel<NC, TILE, HQ>), dim3((max_cols + NC - 1) / NC, p.splits, nseq), dim3(kMixThreadsDec), smem, stream, tq, tkv, p);
    TELB_CHECK_LAUNCH("mixed_decode_kernel");
    if (p.splits > 1) {
        TELB_LAUNCH("mixed_combine_kernel", mixed_combine_kernel, dim3((max_cols + 3) / 4, nseq), dim3(128), 0, stream, p);
        TELB_CHECK_LAUNCH("mixed_combine_kernel");
    }
    return 0;
}

template <int VC, int HQ>
static int launch_mixed_prefill(const CUtensorMap& tq, const CUtensorMap& tkv, MixedPreParams p, int nseq, int max_q, cudaStream_t stream) {
    // the exchange of outputs at the end takes the room of the queries and, where those are narrow, of the keys behind them
    const int fixed = HQ * p.chunks * kMixQChunk + (15 + 2 * kMixKSlots) * 8 + 16 + 1024, v_stage = VC * kMixKChunk;
    p.vstages = kMixSmemLimit - fixed - 2 * v_stage >= 6 * kMixKChunk ? 2 : 1;
    p.kslots = (kMixSmemLimit - fixed - p.vstages * v_stage) / kMixKChunk;
    if (p.kslots > kMixKSlots) p.kslots = kMixKSlots;
    if (p.kslots < 2) return fail("telb_mixed_attention_prefill: queries too wide for shared memory");
    const int smem = fixed + p.kslots * kMixKChunk + p.vstages * v_stage;
    static int configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(mixed_prefill_kernel<VC, HQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(mixed_prefill)", e);
        configured = smem;
    }
    TELB_LAUNCH("mixed_prefill_kernel", (mixed_prefill_kernel<VC, HQ>), dim3((max_q + 127) / 128, p.heads, nseq), dim3(kMixThreadsPre), smem, stream, tq, tkv, p);
    TELB_CHECK_LAUNCH("mixed_prefill_kernel");
    return 0;
}

// Cached heads as [slab = (page, plane, head)][chunk of 64 features][64 tokens][64 features].
static int mixed_kv_map(CUtensorMap* m, const void* kv, int num_pages, int hkv, int pad) {
    const uint64_t dims[4] = {64, kMixPage, (uint64_t)pad / 64, (uint64_t)num_pages * 2 * hkv};
    const uint64_t strides[3] = {(uint64_t)pad * 2, 128, (uint64_t)kMixPage * pad * 2};
    const uint32_t box[4] = {64, kMixPage, 1, 1};
    return make_tmap_nd(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, kv, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
}

}  // namespace telb

using namespace telb;

// bf16 wide queries q [T, heads, halves * hkv * pad], cache [pages, 2, hkv, 64, pad], out [T, heads * pad]; the listed sequences only (q_start: first
// row of each).  pad 64 or 128, hkv * pad at most 512; tile: 64 or 128 cached tokens at a time.  ws holds splits * T * heads * (pad + 1) floats.
extern "C" int telb_mixed_attention_decode(const void* q, const void* kv_layer, void* out, const int* q_start, const int* q_len, const int* past_len,
                                           const int* page_table, int num_seqs, int tokens, int max_q_len, int num_pages, int max_pages, int heads, int hkv, int pad,
                                           int halves, float scale, int window, const float* slopes, const void* gate, long long ld_gate, int splits, int tile,
                                           float* ws, long long ws_floats, int* status, cudaStream_t stream) {
    if (num_seqs <= 0 || tokens <= 0 || max_q_len <= 0) return 0;
    if (tile != 64 && tile != 128) return fail("telb_mixed_attention_decode: tiles of 64 or 128 tokens");
    if ((pad != 64 && pad != 128) || hkv < 1 || hkv * pad > 512 || heads % hkv || (halves != 1 && halves != 2)) return fail("telb_mixed_attention_decode: sizes");
    if (window < 1 || num_seqs > 65535 || (gate && ld_gate % 4)) return fail("telb_mixed_attention_decode: window, sequences or gate pitch");
    MixedDecParams p{};
    p.out = out;
    p.gate = gate;
    p.slopes = slopes;
    p.q_start = q_start;
    p.q_len = q_len;
    p.past_len = past_len;
    p.page_table = page_table;
    p.max_pages = max_pages;
    p.heads = heads;
    p.hkv = hkv;
    p.pad = pad;
    p.rows = tokens * heads;
    p.window = window;
    p.slabs = num_pages * 2 * hkv;
    p.ld_gate = ld_gate;
    p.scale_log2 = scale * kLog2e;
    p.status = status;
    if (splits < 1) splits = 1;
    if (splits > kMixMaxSplits) splits = kMixMaxSplits;
    while (splits > 1 && (long long)splits * p.rows * (pad + 1) > ws_floats) --splits;
    p.splits = splits;
    p.ws_o = ws;
    p.ws_lse = ws + (size_t)splits * p.rows * pad;
    const int max_cols = max_q_len * heads, nc = max_cols <= 16 ? 16 : 32, width = halves * hkv * pad;
    CUtensorMap tq, tkv;
    if (make_tmap_2d(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, q, p.rows, width, (uint64_t)width * 2, nc, 64, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    if (mixed_kv_map(&tkv, kv_layer, num_pages, hkv, pad)) return -1;
#define TELB_MIXED(NC_, TILE_)                                                                          \
    (halves == 2 ? launch_mixed_decode<NC_, TILE_, 2>(tq, tkv, p, num_seqs, max_cols, stream)           \
                 : launch_mixed_decode<NC_, TILE_, 1>(tq, tkv, p, num_seqs, max_cols, stream))
    if (nc == 16) return tile == 64 ? TELB_MIXED(16, 64) : TELB_MIXED(16, 128);
    return tile == 64 ? TELB_MIXED(32, 64) : TELB_MIXED(32, 128);
#undef TELB_MIXED
}

// The same tensors for prompt portions.  hkv * pad at most 512; above 256 only the high halves of the queries are used (halves may be 1).
extern "C" int telb_mixed_attention_prefill(const void* q, const void* kv_layer, void* out, const int* q_start, const int* q_len, const int* past_len,
                                            const int* page_table, int num_seqs, int tokens, int max_q_len, int num_pages, int max_pages, int heads, int hkv, int pad,
                                            int halves, float scale, int window, const float* slopes, const void* gate, long long ld_gate, int* status,
                                            cudaStream_t stream) {
    if (num_seqs <= 0 || tokens <= 0 || max_q_len <= 0) return 0;
    if ((pad != 64 && pad != 128) || hkv < 1 || hkv * pad > 512 || heads % hkv || (halves != 1 && halves != 2)) return fail("telb_mixed_attention_prefill: sizes");
    if (halves == 1 && hkv * pad <= 256) return fail("telb_mixed_attention_prefill: narrow queries come in two halves");
    if (window < 1 || num_seqs > 65535 || heads > 65535 || (gate && ld_gate % 8)) return fail("telb_mixed_attention_prefill: window, sequences, heads or gate pitch");
    MixedPreParams p{out, gate, slopes, q_start, q_len, past_len, page_table, max_pages, heads, hkv, hkv * pad / 64, window, 0, 0, ld_gate, scale * kLog2e, status};
    CUtensorMap tq, tkv;
    {
        const uint64_t width = (uint64_t)halves * hkv * pad;
        const uint64_t dims[3] = {width, (uint64_t)heads, (uint64_t)tokens}, strides[2] = {width * 2, width * 2 * heads};
        const uint32_t box[3] = {64, 1, 128};
        if (make_tmap_nd(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, q, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    }
    if (mixed_kv_map(&tkv, kv_layer, num_pages, hkv, pad)) return -1;
    if (p.chunks <= 4)
        return pad == 64 ? launch_mixed_prefill<1, 2>(tq, tkv, p, num_seqs, max_q_len, stream) : launch_mixed_prefill<2, 2>(tq, tkv, p, num_seqs, max_q_len, stream);
    return pad == 64 ? launch_mixed_prefill<1, 1>(tq, tkv, p, num_seqs, max_q_len, stream) : launch_mixed_prefill<2, 1>(tq, tkv, p, num_seqs, max_q_len, stream);
}
