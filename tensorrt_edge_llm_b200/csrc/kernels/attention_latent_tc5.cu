// Latent attention on tcgen05: cached rows are [latent (rank) | rotated key part], one per token, shared by all heads.
//
//   latent_decode     few rows per sequence.  The key expansion has been folded into the query (one [rank + rot] row per token and head),
//                     so every (token, head) pair is a column against the same cached rows:
//                         Sᵀ[TILE tok, NC] = rows[TILE tok, rank + rot] · Qᵀ    Oᵀ[rank, NC] += latentᵀ[rank, TILE tok] · Pᵀ
//                     A tile of rows is loaded once and serves both products (K-major for the scores, MN-major for the output).  It comes
//                     in pairs of 64-feature chunks through a ring that holds at least one tile: scores start with the first pair, and a
//                     pair's slot is refilled as soon as its 128 output features are done.  The products are narrow, so consecutive ones go
//                     to different accumulators (four for the scores, two output blocks in turn) instead of waiting for one another.
//                     Tiles of two pages use the tensor cores best and fill the ring of the one CTA that an SM holds.  With few rows
//                     in flight tiles of one page spread the work over more CTAs, two per SM; the upper half of their 128-row score
//                     MMA reads whatever lies behind the chunk, and nobody reads its results.
//   latent_prefill    prompt portions, over keys and values expanded from the latents ([rows, heads, k | v], one product per step).  The
//                     rotated key part is not expanded: a K tile is made of chunks of the head's keys and chunks of the shared rows.
//                     256 query rows per CTA in two tiles with a softmax warpgroup each; probabilities stay in TMEM (the A operand
//                     of P·V), over the scores they were made from.
//
// The producer and the MMA warp walk their loops as whole warps and elect a lane only for the instructions themselves: descriptors then
// live in uniform registers (under a divergent branch every issue costs about 100 cycles, more than these narrow products take).
//
// Probabilities enter P·V as a high and a low 16-bit half (2^-17).  Scores, maxima and sums are fp32.  All waits are bounded.
#include <type_traits>

#include "attention_common.cuh"
#include "host_utils.h"

namespace telb {

constexpr int kLatMaxSlots = 16;
constexpr int kLatMaxSplits = 64;

struct LatentDecParams {
    void* out;                 // [rows, rank_pad] 16-bit, rows = T * heads
    float* ws_o;               // [splits, rows, rank_pad] (splits > 1)
    float* ws_lse;             // [splits, rows], log2 domain
    const int* q_start;
    const int* q_len;
    const int* past_len;
    const int* page_table;
    int max_pages, heads, splits, rows, rank_pad, chunks, pairs, vblocks, slots;
    float scale_log2;
    int* status;
};

constexpr int kLatThreads = 192;
constexpr int kLatPage = 64;

// grid (column blocks, splits, sequences).  NC: (token, head) columns of a block; TILE: cached rows of a tile, one or two pages.
template <typename T, int NC, int TILE>
__global__ void __launch_bounds__(kLatThreads, NC == 16 && TILE == 64 ? 2 : 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_kv, const __grid_constant__ LatentDecParams p) {
    constexpr bool kBf16 = std::is_same<T, __nv_bfloat16>::value;
    constexpr int kQChunk = NC * 128, kPSpan = 2 * NC * 128;         // [high | low rows of the columns][64 tokens]
    constexpr int kPBytes = TILE / 64 * kPSpan;
    constexpr int kLatTile = TILE, kLatChunk = TILE * 128, kLatSlot = 2 * kLatChunk;      // chunk: bytes of [TILE rows x 64 features]
    constexpr int kOCol = 4 * NC, kOBlock = 2 * NC;      // TMEM: four partial scores, then per 128 output features high | low columns
    constexpr int kTmemCols = NC == 16 ? 256 : 512;
    static_assert(kOCol + 4 * kOBlock <= kTmemCols, "scores and four output blocks");

    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* s_kv = smem;
    uint8_t* s_q = s_kv + p.slots * kLatSlot;
    uint8_t* s_p = s_q + p.chunks * kQChunk;
    uint64_t* bars = reinterpret_cast<uint64_t*>(s_p + kPBytes);
    uint64_t* q_full = bars;
    uint64_t* s_full = bars + 1;
    uint64_t* p_full = bars + 2;
    uint64_t* o_done = bars + 3;
    uint64_t* kv_full = bars + 4;
    uint64_t* kv_empty = kv_full + kLatMaxSlots;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(kv_empty + kLatMaxSlots);
    volatile uint32_t* abort_flag = tmem_slot + 1;
    float* s_red = reinterpret_cast<float*>(tmem_slot + 4);      // [4 warps][NC] maxima, then sums

    pdl_wait();                                           // dependents start once TMEM is allocated: theirs must not come first
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seq = blockIdx.z, split = blockIdx.y, cb = blockIdx.x;
    const int qlen = p.q_len[seq], past = p.past_len[seq];
    const int ncol = min(NC, qlen * p.heads - cb * NC);
    if (ncol <= 0) return;                               // uniform, before any barrier or TMEM use
    const int row0 = p.q_start[seq] * p.heads + cb * NC; // first (token, head) row of the block
    const int last_q = (cb * NC + ncol - 1) / p.heads;
    const int tiles = (past + last_q + 1 + kLatTile - 1) / kLatTile;
    const int per = (tiles + p.splits - 1) / p.splits;
    const int j0 = split * per;
    const int ntiles = max(0, min(tiles, j0 + per) - j0);

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
    for (int i = threadIdx.x; i < kPBytes / 16; i += kLatThreads) reinterpret_cast<uint4*>(s_p)[i] = make_uint4(0, 0, 0, 0);
    fence_proxy_async_smem();
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem_base = *tmem_slot;
    pdl_launch_dependents();

    if (warp == 0) {
        // ---- producer ----
        if (ntiles > 0) {
            const bool leader = elect_one();
            if (leader) {
                mbar_expect_tx(q_full, p.chunks * kQChunk);
                for (int c = 0; c < p.chunks; ++c) tma_load_2d(s_q + c * kQChunk, &tma_q, q_full, c * 64, row0);
            }
            const int* pages = p.page_table + (size_t)seq * p.max_pages;
            bool ok = true;
            int slot = 0;
            uint32_t ph = 1;
            constexpr int kPages = TILE / kLatPage, kAhead = 32 / kPages;
            int next = 0;                                // the pages of kAhead tiles are fetched at a time
            for (int j = 0; j < ntiles && ok; ++j) {
                if (j % kAhead == 0) {
                    const int lp = (j0 + j) * kPages + lane;
                    next = lp < p.max_pages ? pages[lp] : -1;
                }
                int row[kPages];                         // rows past the end are masked
#pragma unroll
                for (int h = 0; h < kPages; ++h) row[h] = max(__shfl_sync(0xffffffffu, next, j % kAhead * kPages + h), 0) * kLatPage;
                for (int pr = 0; pr < p.pairs; ++pr) {
                    ok = mbar_wait(&kv_empty[slot], ph, abort_flag, p.status, kStatusProducerTimeout);
                    ok = __all_sync(0xffffffffu, ok);
                    if (!ok) break;
                    uint8_t* dst = s_kv + slot * kLatSlot;
                    if (leader) {
                        mbar_expect_tx(&kv_full[slot], kLatSlot);                 // a missing second chunk arrives as zeros
                        if constexpr (kPages == 1) {                              // both chunks in one copy
                            tma_load_3d(dst, &tma_kv, &kv_full[slot], 0, row[0], pr * 2);
                        } else {
#pragma unroll
                            for (int c = 0; c < 2; ++c)
#pragma unroll
                                for (int h = 0; h < kPages; ++h)
                                    tma_load_3d(dst + c * kLatChunk + h * (kLatPage * 128), &tma_kv, &kv_full[slot], 0, row[h], pr * 2 + c);
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
            constexpr uint32_t idesc_s = idesc_f16(128, NC, kBf16), idesc_o = idesc_f16(128, 2 * NC, kBf16, true);
            const uint64_t desc_kv = smem_desc_sw128(s_kv), desc_v = smem_desc_sw128_mn(s_kv, kLatChunk, 1024), desc_q = smem_desc_sw128(s_q),
                           desc_p = smem_desc_sw128(s_p);
            bool ok = __all_sync(0xffffffffu, mbar_wait(q_full, 0, abort_flag, p.status, kStatusMmaTimeout));
            int slot = 0;
            uint32_t ph = 0;
            for (int j = 0; j < ntiles && ok; ++j) {
                const int first = slot;
                for (int pr = 0; pr < p.pairs; ++pr) {
                    ok = __all_sync(0xffffffffu, mbar_wait(&kv_full[slot], ph, abort_flag, p.status, kStatusMmaTimeout));
                    if (!ok) break;
                    tc_fence_after_sync();
                    const bool two = pr * 2 + 1 < p.chunks;
                    const uint64_t dk = desc_kv + (uint64_t)((slot * kLatSlot) >> 4), dq = desc_q + (uint64_t)((pr * 2 * kQChunk) >> 4);
                    if (leader) {
#pragma unroll
                        for (int k = 0; k < 4; ++k) umma_f16(tmem_base + k * NC, dk + 2 * k, dq + 2 * k, idesc_s, pr ? 1u : 0u);
                        if (two) {
#pragma unroll
                            for (int k = 0; k < 4; ++k)
                                umma_f16(tmem_base + k * NC, dk + (kLatChunk >> 4) + 2 * k, dq + (kQChunk >> 4) + 2 * k, idesc_s, 1u);
                        }
                        if (pr >= p.vblocks) umma_commit(&kv_empty[slot]);       // keys only
                        if (pr == p.pairs - 1) umma_commit(s_full);
                    }
                    __syncwarp();
                    if (++slot == p.slots) {
                        slot = 0;
                        ph ^= 1;
                    }
                }
                if (!ok) break;
                ok = __all_sync(0xffffffffu, mbar_wait(p_full, j & 1, abort_flag, p.status, kStatusMmaTimeout));
                if (!ok) break;
                tc_fence_after_sync();
                int s0 = first;
                for (int b = 0; b < p.vblocks; b += 2) {
                    const bool two = b + 1 < p.vblocks;
                    const int s1 = s0 + 1 == p.slots ? 0 : s0 + 1;
                    const uint64_t dv0 = desc_v + (uint64_t)((s0 * kLatSlot) >> 4), dv1 = desc_v + (uint64_t)((s1 * kLatSlot) >> 4);
                    const uint32_t d_o = tmem_base + kOCol + b * kOBlock;
                    if (leader) {
#pragma unroll
                        for (int k = 0; k < kLatTile / 16; ++k) {
                            const uint64_t db = desc_p + (uint64_t)(((k >> 2) * kPSpan) >> 4) + 2 * (k & 3);
                            umma_f16(d_o, dv0 + (uint64_t)((k * 2048) >> 4), db, idesc_o, (j | k) ? 1u : 0u);
                            if (two) umma_f16(d_o + kOBlock, dv1 + (uint64_t)((k * 2048) >> 4), db, idesc_o, (j | k) ? 1u : 0u);
                        }
                        umma_commit(&kv_empty[s0]);
                        if (two) umma_commit(&kv_empty[s1]);
                        if (j == ntiles - 1 && b + 2 >= p.vblocks) umma_commit(o_done);
                    }
                    __syncwarp();
                    s0 = s1 + 1 == p.slots ? 0 : s1 + 1;
                }
            }
        }
    } else {
        // ---- softmax / epilogue ----
        const int quad = warp & 3, r = quad * 32 + lane; // cached row within the tile (S), feature within a block (O)
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
                uint32_t r0[16], r1[16], r2[16], r3[16];
                tmem_ld_x16(lane_addr + c, r0);
                tmem_ld_x16(lane_addr + NC + c, r1);
                tmem_ld_x16(lane_addr + 2 * NC + c, r2);
                tmem_ld_x16(lane_addr + 3 * NC + c, r3);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 16; ++i)
                    s[c + i] = (__uint_as_float(r0[i]) + __uint_as_float(r1[i]) + (__uint_as_float(r2[i]) + __uint_as_float(r3[i]))) * p.scale_log2;
            }
            const int t0 = (j0 + j) * kLatTile, tk = t0 + r;
            if (r >= kLatTile) {                         // lanes behind the tile only help to rescale and to write the output
#pragma unroll
                for (int c = 0; c < NC; ++c) s[c] = -INFINITY;
            } else if (t0 + kLatTile - 1 > past) {       // the tile reaches the first row's own position: mask
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const int qi = qlen == 1 ? 0 : (cb * NC + c) / p.heads;
                    if (tk > past + qi) s[c] = -INFINITY;
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
                    for (int b = 0; b < p.vblocks; ++b)
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
            if (r < kLatTile) {
                uint8_t* prow = s_p + (r >> 6) * kPSpan + (r & 7) * 2;
                const int unit = (r & 63) >> 3;
#pragma unroll
                for (int c = 0; c < NC; ++c) {           // columns beyond ncol: reference +inf, probability zero
                    const float e = exp2f(s[c] - (m_used[c] == -INFINITY ? 0.f : m_used[c]));
                    l_part[c] += e;
                    uint8_t* dst = prow + (c >> 3) * 1024 + (c & 7) * 128 + ((unit ^ (c & 7)) << 4);
                    const T hi = Cvt<T>::from_f(e);
                    *reinterpret_cast<T*>(dst) = hi;
                    *reinterpret_cast<T*>(dst + NC * 128) = Cvt<T>::from_f(e - Cvt<T>::to_f(hi));
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
            for (int b = 0; b < p.vblocks; ++b) {
                const int feat = b * 128 + r;
#pragma unroll
                for (int c = 0; c < NC; c += 16) {
                    uint32_t o[16], lo[16];
                    tmem_ld_x16(lane_addr + kOCol + b * kOBlock + c, o);       // garbage (never used) without tiles
                    tmem_ld_x16(lane_addr + kOCol + b * kOBlock + NC + c, lo);
                    tmem_ld_wait();
                    if (feat >= p.rank_pad) continue;
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        if (c + i >= ncol) continue;
                        const float v = inv[c + i] > 0.f ? (__uint_as_float(o[i]) + __uint_as_float(lo[i])) * inv[c + i] : 0.f;
                        const size_t row = (size_t)row0 + c + i;
                        if (p.splits == 1) reinterpret_cast<T*>(p.out)[row * p.rank_pad + feat] = Cvt<T>::from_f(v);
                        else p.ws_o[((size_t)split * p.rows + row) * p.rank_pad + feat] = v;
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

// out[row] = sum over splits of 2^(lse - max) O / sum of 2^(lse - max)
template <typename T>
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* ws_o, const float* ws_lse, T* out, int rows, int splits, int d) {
    pdl_prologue();
    __shared__ float w[kLatMaxSplits];
    const int row = blockIdx.x;
    if (threadIdx.x < 32) {
        float l[kLatMaxSplits / 32], mx = -INFINITY, den = 0.f;
#pragma unroll
        for (int i = 0; i < kLatMaxSplits / 32; ++i) {
            const int sp = i * 32 + threadIdx.x;
            l[i] = sp < splits ? ws_lse[(size_t)sp * rows + row] : -INFINITY;
            mx = fmaxf(mx, l[i]);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
#pragma unroll
        for (int i = 0; i < kLatMaxSplits / 32; ++i) {
            l[i] = l[i] == -INFINITY ? 0.f : exp2f(l[i] - mx);
            den += l[i];
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) den += __shfl_xor_sync(0xffffffffu, den, o);
#pragma unroll
        for (int i = 0; i < kLatMaxSplits / 32; ++i) w[i * 32 + threadIdx.x] = den > 0.f ? l[i] / den : 0.f;
    }
    __syncthreads();
    for (int i = threadIdx.x * 4; i < d; i += 512) {
        float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
        for (int s = 0; s < splits; ++s) {
            const float4 v = __ldcg(reinterpret_cast<const float4*>(ws_o + ((size_t)s * rows + row) * d + i));
            a[0] = fmaf(w[s], v.x, a[0]);
            a[1] = fmaf(w[s], v.y, a[1]);
            a[2] = fmaf(w[s], v.z, a[2]);
            a[3] = fmaf(w[s], v.w, a[3]);
        }
        uint2 u;
        u.x = Cvt<T>::pack2(a[0], a[1]);
        u.y = Cvt<T>::pack2(a[2], a[3]);
        *reinterpret_cast<uint2*>(out + (size_t)row * d + i) = u;
    }
}

// ---- prefill ---------------------------------------------------------------------------------------------
struct LatentPrefillParams {
    void* out;                 // [T, heads * v_pad]
    const int* q_start;        // first row of each sequence
    const int* q_len;
    const int* past_len;
    const int* kv_start;       // first row of each sequence in the expanded keys / values
    int heads, kn, rc, stages; // 64-feature chunks of the unrotated and the rotated part; K / V ring depth
    float scale_log2;
    int* status;
};

constexpr int kPreThreads = 320;             // producer, MMA issuer, two softmax warpgroups
constexpr int kPreTile = 64;                 // keys per tile
constexpr int kPreMaxStages = 8;
constexpr int kPreChunk = kPreTile * 128;    // bytes of [64 keys x 64 features]
constexpr int kPreQChunk = 128 * 128;        // bytes of [128 rows x 64 features]

// grid (query tiles of 256 rows, heads, sequences).  VC: 64-feature chunks of the values.
template <typename T, int VC>
__global__ void __launch_bounds__(kPreThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_qr, const __grid_constant__ CUtensorMap tma_k,
                      const __grid_constant__ CUtensorMap tma_kr, const __grid_constant__ CUtensorMap tma_v, const __grid_constant__ LatentPrefillParams p) {
    constexpr bool kBf16 = std::is_same<T, __nv_bfloat16>::value;
    constexpr int VP = VC * 64;
    // TMEM per query tile: two score buffers of 64 columns (each turns into high | low probabilities), then the output
    constexpr uint32_t kTileCols = 256, kOCol = 128;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int kc = p.kn + p.rc;
    const int k_bytes = kc * kPreChunk, stage_bytes = k_bytes + VC * kPreChunk;
    uint8_t* s_q = smem;                                  // [2 tiles][kc chunks]
    uint8_t* s_kv = s_q + 2 * kc * kPreQChunk;
    uint64_t* bars = reinterpret_cast<uint64_t*>(s_kv + p.stages * stage_bytes);
    uint64_t* q_full = bars;
    uint64_t* s_full = bars + 1;                          // [tile][buffer]
    uint64_t* p_full = s_full + 4;
    uint64_t* o_done = p_full + 4;                        // [tile][buffer]: two in turn, so that a wait never meets the phase after next
    uint64_t* k_full = o_done + 4;
    uint64_t* k_empty = k_full + kPreMaxStages;
    uint64_t* v_full = k_empty + kPreMaxStages;
    uint64_t* v_empty = v_full + kPreMaxStages;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(v_empty + kPreMaxStages);
    volatile uint32_t* abort_flag = tmem_slot + 1;

    pdl_wait();                                           // dependents start at the end: a long kernel runs slower under waiting ones
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int qt = gridDim.x - 1 - blockIdx.x;            // long rows first
    const int head = blockIdx.y, seq = blockIdx.z;
    const int qlen = p.q_len[seq], past = p.past_len[seq], tok0 = qt * 256;
    if (tok0 >= qlen) return;                             // uniform, before any barrier or TMEM use
    const int qrow0 = p.q_start[seq] + tok0, kvrow0 = p.kv_start[seq];
    // key tiles that query tile t sees (0: the tile has no rows)
    const int nt0 = (past + min(qlen, tok0 + 128) + kPreTile - 1) / kPreTile;
    const int nt1 = qlen > tok0 + 128 ? (past + min(qlen, tok0 + 256) + kPreTile - 1) / kPreTile : 0;
    const int nt = max(nt0, nt1);
    const int qtiles = nt1 > 0 ? 2 : 1;

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int i = 0; i < 4; ++i) {
            mbar_init(&s_full[i], 1);
            mbar_init(&p_full[i], 128);
            mbar_init(&o_done[i], 1);
        }
        for (int s = 0; s < p.stages; ++s) {
            mbar_init(&k_full[s], 1);
            mbar_init(&k_empty[s], 1);
            mbar_init(&v_full[s], 1);
            mbar_init(&v_empty[s], 1);
        }
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, 512);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        // ---- producer ----
        const bool leader = elect_one();
        if (leader) {
            mbar_expect_tx(q_full, qtiles * kc * kPreQChunk);
            for (int t = 0; t < qtiles; ++t)
                for (int c = 0; c < kc; ++c) {
                    uint8_t* dst = s_q + (t * kc + c) * kPreQChunk;
                    if (c < p.kn) tma_load_3d(dst, &tma_q, q_full, c * 64, head, qrow0 + t * 128);
                    else tma_load_3d(dst, &tma_qr, q_full, (c - p.kn) * 64, head, qrow0 + t * 128);
                }
        }
        int st = 0;
        uint32_t ph = 1;
        for (int j = 0; j < nt; ++j) {
            uint8_t* sk = s_kv + st * stage_bytes;
            const int row = kvrow0 + j * kPreTile;
            if (!__all_sync(0xffffffffu, mbar_wait(&k_empty[st], ph, abort_flag, p.status, kStatusProducerTimeout))) break;
            if (leader) {
                mbar_expect_tx(&k_full[st], k_bytes);
                for (int c = 0; c < p.kn; ++c) tma_load_3d(sk + c * kPreChunk, &tma_k, &k_full[st], c * 64, head, row);
                for (int c = 0; c < p.rc; ++c) tma_load_2d(sk + (p.kn + c) * kPreChunk, &tma_kr, &k_full[st], c * 64, row);
            }
            if (!__all_sync(0xffffffffu, mbar_wait(&v_empty[st], ph, abort_flag, p.status, kStatusProducerTimeout))) break;
            if (leader) {
                mbar_expect_tx(&v_full[st], VC * kPreChunk);
#pragma unroll
                for (int c = 0; c < VC; ++c) tma_load_3d(sk + k_bytes + c * kPreChunk, &tma_v, &v_full[st], c * 64, head, row);
            }
            if (++st == p.stages) {
                st = 0;
                ph ^= 1;
            }
        }
    } else if (warp == 1) {
        // ---- MMA issuer: S(0); then S(j + 1), P·V(j) ----
        const bool leader = elect_one();
        constexpr uint32_t idesc_s = idesc_f16(128, kPreTile, kBf16), idesc_o = idesc_f16(128, VP, kBf16, false, true);
        const uint64_t desc_q = smem_desc_sw128(s_q), desc_k = smem_desc_sw128(s_kv), desc_v = smem_desc_sw128_mn(s_kv + k_bytes, kPreChunk, 1024);
        auto wait = [&](uint64_t* bar, uint32_t parity) {
            const bool got = __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, p.status, kStatusMmaTimeout));
            tc_fence_after_sync();
            return got;
        };
        int ks = 0, vs = 0;                               // ring positions of the next key and value tile
        uint32_t kph = 0, vph = 0;
        auto issue_s = [&](int j) {
            if (!wait(&k_full[ks], kph)) return false;
            const uint64_t dk = desc_k + (uint64_t)((ks * stage_bytes) >> 4);
            const uint32_t d = tmem_base + (j & 1) * 64;
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                if (j >= (t == 0 ? nt0 : nt1)) continue;
                const uint64_t dq = desc_q + (uint64_t)((t * kc * kPreQChunk) >> 4);
                if (leader) {
                    for (int c = 0; c < kc; ++c)
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            umma_f16(d + t * kTileCols, dq + (uint64_t)((c * kPreQChunk) >> 4) + 2 * k, dk + (uint64_t)((c * kPreChunk) >> 4) + 2 * k, idesc_s,
                                     (c | k) ? 1u : 0u);
                    umma_commit(&s_full[t * 2 + (j & 1)]);
                }
            }
            if (leader) umma_commit(&k_empty[ks]);
            if (++ks == p.stages) {
                ks = 0;
                kph ^= 1;
            }
            return true;
        };
        bool ok = wait(q_full, 0) && issue_s(0);
        for (int j = 0; j < nt && ok; ++j) {
            if (j + 1 < nt) ok = issue_s(j + 1);
            ok = ok && wait(&v_full[vs], vph);
            const uint64_t dv = desc_v + (uint64_t)((vs * stage_bytes) >> 4);
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                if (!ok || j >= (t == 0 ? nt0 : nt1)) continue;
                ok = wait(&p_full[t * 2 + (j & 1)], (j >> 1) & 1);
                if (!ok) continue;
                const uint32_t a = tmem_base + t * kTileCols + (j & 1) * 64, d = tmem_base + t * kTileCols + kOCol;
                if (leader) {
#pragma unroll
                    for (int half = 0; half < 2; ++half)
#pragma unroll
                        for (int k = 0; k < kPreTile / 16; ++k)
                            umma_f16_ts(d, a + half * 32 + k * 8, dv + (uint64_t)((k * 2048) >> 4), idesc_o, (j | half | k) ? 1u : 0u);
                    umma_commit(&o_done[t * 2 + (j & 1)]);
                }
            }
            if (ok && leader) umma_commit(&v_empty[vs]);
            if (++vs == p.stages) {
                vs = 0;
                vph ^= 1;
            }
        }
    } else {
        // ---- softmax / epilogue: one thread per query row ----
        const int t = (warp - 2) >> 2, quad = warp & 3;
        const int r = quad * 32 + lane, qi = tok0 + t * 128 + r;
        const int mine = t == 0 ? nt0 : nt1;
        const uint32_t base = tmem_base + t * kTileCols + (static_cast<uint32_t>(quad * 32) << 16);
        const int limit = past + qi;                      // last visible key
        float m_used = -INFINITY, l_sum = 0.f;
        bool ok = true;
        for (int j = 0; j < mine && ok; ++j) {
            const int b = j & 1;
            if (!mbar_wait(&s_full[t * 2 + b], (j >> 1) & 1, abort_flag, p.status, kStatusEpilogueTimeout)) { ok = false; break; }
            tc_fence_after_sync();
            float s[kPreTile];
            {
                uint32_t r0[32], r1[32];
                tmem_ld_x32(base + b * 64, r0);
                tmem_ld_x32(base + b * 64 + 32, r1);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    s[i] = __uint_as_float(r0[i]);
                    s[32 + i] = __uint_as_float(r1[i]);
                }
            }
            const int c0 = j * kPreTile;
            if (c0 + kPreTile - 1 > past + tok0 + t * 128) {          // only tiles that reach the first row's diagonal are masked
#pragma unroll
                for (int i = 0; i < kPreTile; ++i) s[i] = c0 + i <= limit ? s[i] : -INFINITY;
            }
            float mx = s[0];
#pragma unroll
            for (int i = 1; i < kPreTile; ++i) mx = fmaxf(mx, s[i]);
            const float m_new = fmaxf(m_used, mx * p.scale_log2);     // the scale is positive
            const bool need = m_new > m_used + 8.0f;
            if (j == 0) {
                m_used = m_new;
            } else if (__any_sync(0xffffffffu, need)) {
                // P·V of tile j - 1 (that of tile j - 2 was issued ahead of these scores and is complete)
                if (!mbar_wait(&o_done[t * 2 + (b ^ 1)], ((j - 1) >> 1) & 1, abort_flag, p.status, kStatusEpilogueTimeout)) { ok = false; break; }
                tc_fence_after_sync();
                const float f = need ? exp2f(m_used - m_new) : 1.f;
#pragma unroll 1
                for (int c = 0; c < VP / 16; ++c) {
                    uint32_t o[16];
                    tmem_ld_x16(base + kOCol + c * 16, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
                    tmem_st_x16(base + kOCol + c * 16, o);
                }
                if (need) {
                    l_sum *= f;
                    m_used = m_new;
                }
            }
            const float mref = m_used == -INFINITY ? 0.f : m_used;
            float acc = 0.f;
#pragma unroll
            for (int h = 0; h < 2; ++h) {                             // 32 keys at a time: 16 columns of high halves, 16 of low ones
                uint32_t hi[16], lo[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float e0 = exp2f(fmaf(s[h * 32 + 2 * i], p.scale_log2, -mref)), e1 = exp2f(fmaf(s[h * 32 + 2 * i + 1], p.scale_log2, -mref));
                    acc += e0 + e1;
                    hi[i] = Cvt<T>::pack2(e0, e1);
                    const T* q = reinterpret_cast<const T*>(&hi[i]);
                    lo[i] = Cvt<T>::pack2(e0 - Cvt<T>::to_f(q[0]), e1 - Cvt<T>::to_f(q[1]));
                }
                tmem_st_x16(base + b * 64 + h * 16, hi);
                tmem_st_x16(base + b * 64 + 32 + h * 16, lo);
            }
            l_sum += acc;
            tmem_st_wait();
            tc_fence_before_sync();
            mbar_arrive(&p_full[t * 2 + b]);
        }
        if (ok && mine > 0) {
            ok = mbar_wait(&o_done[t * 2 + ((mine - 1) & 1)], ((mine - 1) >> 1) & 1, abort_flag, p.status, kStatusEpilogueTimeout);
            if (ok) {
                tc_fence_after_sync();
                const float inv = l_sum > 0.f ? 1.f / l_sum : 0.f;
                T* dst = reinterpret_cast<T*>(p.out) + ((size_t)(p.q_start[seq] + qi) * p.heads + head) * VP;
#pragma unroll 1
                for (int c = 0; c < VP / 16; ++c) {
                    uint32_t o[16];
                    tmem_ld_x16(base + kOCol + c * 16, o);
                    tmem_ld_wait();
                    if (qi < qlen) {
                        uint32_t w[8];
#pragma unroll
                        for (int i = 0; i < 8; ++i) w[i] = Cvt<T>::pack2(__uint_as_float(o[2 * i]) * inv, __uint_as_float(o[2 * i + 1]) * inv);
                        reinterpret_cast<uint4*>(dst + c * 16)[0] = make_uint4(w[0], w[1], w[2], w[3]);
                        reinterpret_cast<uint4*>(dst + c * 16)[1] = make_uint4(w[4], w[5], w[6], w[7]);
                    }
                    __syncwarp();
                }
                tc_fence_before_sync();
            }
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
        tmem_dealloc(tmem_base, 512);
    }
}

constexpr int kSmemLimit = 227 * 1024;

template <typename T, int NC, int TILE>
static int launch_latent_decode(const CUtensorMap& tq, const CUtensorMap& tkv, LatentDecParams p, int nseq, int max_cols, cudaStream_t stream) {
    // the score MMA of one-page tiles reads one chunk beyond the last slot: Q and P, and a spare
    constexpr int chunk = TILE * 128, slot = 2 * chunk, ctas = NC == 16 && TILE == 64 ? 2 : 1;
    const int fixed = p.chunks * NC * 128 + TILE / 64 * 2 * NC * 128 + (4 + 2 * kLatMaxSlots) * 8 + 16 + 8 * NC * 4 + 1024 + (TILE == 64 ? chunk : 0);
    p.slots = (kSmemLimit / ctas - (ctas - 1) * 1024 - fixed) / slot;
    if (p.slots < p.pairs) p.slots = (kSmemLimit - fixed) / slot;
    if (p.slots > kLatMaxSlots) p.slots = kLatMaxSlots;
    if (p.slots > 3 * p.pairs) p.slots = 3 * p.pairs;
    if (p.slots < p.pairs) return fail("telb_latent_attention_decode: rows too wide for shared memory");
    const int smem = fixed + p.slots * slot;
    static int configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<T, NC, TILE>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(latent_decode)", e);
        configured = smem;
    }
    TELB_LAUNCH("latent_decode_kernel", (latent_decode_kernel<T, NC, TILE>), dim3((max_cols + NC - 1) / NC, p.splits, nseq), dim3(kLatThreads), smem, stream, tq, tkv, p);
    TELB_CHECK_LAUNCH("latent_decode_kernel");
    if (p.splits > 1) {
        TELB_LAUNCH("latent_combine_kernel", (latent_combine_kernel<T>), dim3(p.rows), dim3(128), 0, stream, p.ws_o, p.ws_lse, (T*)p.out, p.rows, p.splits, p.rank_pad);
        TELB_CHECK_LAUNCH("latent_combine_kernel");
    }
    return 0;
}

template <typename T, int VC>
static int launch_latent_prefill(const CUtensorMap (&m)[5], LatentPrefillParams p, int nseq, int max_q, cudaStream_t stream) {
    const int kc = p.kn + p.rc, stage = (kc + VC) * kPreChunk;
    const int fixed = 2 * kc * kPreQChunk + (13 + 4 * kPreMaxStages) * 8 + 16 + 1024;
    p.stages = (kSmemLimit - fixed) / stage;
    if (p.stages > kPreMaxStages) p.stages = kPreMaxStages;
    if (p.stages < 1) return fail("telb_latent_attention_prefill: heads too wide for shared memory");
    const int smem = fixed + p.stages * stage;
    static int configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<T, VC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail("cudaFuncSetAttribute(latent_prefill)", e);
        configured = smem;
    }
    TELB_LAUNCH("latent_prefill_kernel", (latent_prefill_kernel<T, VC>), dim3((max_q + 255) / 256, p.heads, nseq), dim3(kPreThreads), smem, stream, m[0], m[1], m[2],
                m[3], m[4], p);
    TELB_CHECK_LAUNCH("latent_prefill_kernel");
    return 0;
}

}  // namespace telb

using namespace telb;

// q [rows = T * heads, rank_pad + rot_pad] with the key expansion folded in, cached rows [pages, 64, rank_pad + rot_pad] → out [rows, rank_pad].
// Sizes are multiples of 64, rank_pad at most 512; tile: 64 or 128 cached rows at a time.  ws holds splits * rows * (rank_pad + 1) floats.
extern "C" int telb_latent_attention_decode(const void* q, const void* kv_layer, void* out, const int* q_start, const int* q_len, const int* past_len,
                                            const int* page_table, int num_seqs, int tokens, int max_q_len, int num_pages, int max_pages, int heads, int rank_pad,
                                            int rot_pad, float scale, int splits, int tile, float* ws, long long ws_floats, int is_bf16, int* status,
                                            cudaStream_t stream) {
    if (num_seqs <= 0 || tokens <= 0) return 0;
    if (tile != 64 && tile != 128) return fail("telb_latent_attention_decode: tiles of 64 or 128 rows");
    if (rank_pad % 64 || rot_pad % 64 || rank_pad < 64 || rank_pad > 512 || rot_pad < 64) return fail("telb_latent_attention_decode: sizes");
    if (num_seqs > 65535) return fail("telb_latent_attention_decode: too many sequences");
    LatentDecParams p{};
    p.out = out;
    p.q_start = q_start;
    p.q_len = q_len;
    p.past_len = past_len;
    p.page_table = page_table;
    p.max_pages = max_pages;
    p.heads = heads;
    p.rows = tokens * heads;
    p.rank_pad = rank_pad;
    p.chunks = (rank_pad + rot_pad) / 64;
    p.pairs = (p.chunks + 1) / 2;
    p.vblocks = (rank_pad + 127) / 128;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.status = status;
    if (splits < 1) splits = 1;
    if (splits > kLatMaxSplits) splits = kLatMaxSplits;
    while (splits > 1 && (long long)splits * p.rows * (rank_pad + 1) > ws_floats) --splits;
    p.splits = splits;
    p.ws_o = ws;
    p.ws_lse = ws + (size_t)splits * p.rows * rank_pad;
    const CUtensorMapDataType dt = is_bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16;
    const int row = rank_pad + rot_pad, max_cols = max_q_len * heads;
    const int nc = max_cols <= 16 ? 16 : 32;
    CUtensorMap tq, tkv;
    if (make_tmap_2d(&tq, dt, 2, q, p.rows, row, (uint64_t)row * 2, nc, 64, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    {   // cached rows as [chunk][row][64 features]: one copy brings a page's rows for a pair of chunks
        const uint64_t dims[3] = {64, (uint64_t)num_pages * kLatPage, (uint64_t)row / 64}, strides[2] = {(uint64_t)row * 2, 128};
        const uint32_t box[3] = {64, kLatPage, tile == 64 ? 2u : 1u};
        if (make_tmap_nd(&tkv, dt, 3, kv_layer, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    }
#define TELB_LATENT(NC_, TILE_)                                                                                          \
    (is_bf16 ? launch_latent_decode<__nv_bfloat16, NC_, TILE_>(tq, tkv, p, num_seqs, max_cols, stream)                   \
             : launch_latent_decode<__half, NC_, TILE_>(tq, tkv, p, num_seqs, max_cols, stream))
    if (nc == 16) return tile == 64 ? TELB_LATENT(16, 64) : TELB_LATENT(16, 128);
    return tile == 64 ? TELB_LATENT(32, 64) : TELB_LATENT(32, 128);
#undef TELB_LATENT
}

// q: packed rows of pitch ldq whose first heads * k_pad columns are the unrotated and next heads * rot_pad the rotated query parts; kv
// [kv_rows, heads * k_pad + heads * v_pad] expanded keys | values; key_rot [kv_rows, rot_pad]; out [T, heads * v_pad].  v_pad 64 or 128.
extern "C" int telb_latent_attention_prefill(const void* q, const void* kv, const void* key_rot, void* out, const int* q_start, const int* q_len,
                                             const int* past_len, const int* kv_start, int num_seqs, int tokens, int max_q_len, int kv_rows, int ldq, int heads,
                                             int k_pad, int rot_pad, int v_pad, float scale, int is_bf16, int* status, cudaStream_t stream) {
    if (num_seqs <= 0 || tokens <= 0 || max_q_len <= 0) return 0;
    if (k_pad % 64 || rot_pad % 64 || ldq % 8 || (v_pad != 64 && v_pad != 128)) return fail("telb_latent_attention_prefill: sizes");
    if (num_seqs > 65535 || heads > 65535) return fail("telb_latent_attention_prefill: too many sequences or heads");
    if (!(scale > 0.f)) return fail("telb_latent_attention_prefill: the scale must be positive");
    LatentPrefillParams p{out, q_start, q_len, past_len, kv_start, heads, k_pad / 64, rot_pad / 64, 0, scale * 1.4426950408889634f, status};
    const CUtensorMapDataType dt = is_bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16;
    const uint8_t* qb = static_cast<const uint8_t*>(q);
    const uint8_t* kvb = static_cast<const uint8_t*>(kv);
    const uint64_t h = heads, pitch_q = (uint64_t)ldq * 2, pitch_kv = h * (uint64_t)(k_pad + v_pad) * 2;
    CUtensorMap m[5];
    auto heads_map = [&](CUtensorMap* out_map, const void* base, int width, uint64_t rows, uint64_t pitch, uint32_t box_rows) {
        const uint64_t dims[3] = {(uint64_t)width, h, rows}, strides[2] = {(uint64_t)width * 2, pitch};
        const uint32_t box[3] = {64, 1, box_rows};
        return make_tmap_nd(out_map, dt, 3, base, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
    };
    if (heads_map(&m[0], qb, k_pad, tokens, pitch_q, 128) || heads_map(&m[1], qb + h * k_pad * 2, rot_pad, tokens, pitch_q, 128) ||
        heads_map(&m[2], kvb, k_pad, kv_rows, pitch_kv, kPreTile) || heads_map(&m[4], kvb + h * k_pad * 2, v_pad, kv_rows, pitch_kv, kPreTile))
        return -1;
    if (make_tmap_2d(&m[3], dt, 2, key_rot, kv_rows, rot_pad, (uint64_t)rot_pad * 2, kPreTile, 64, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
    if (v_pad == 64)
        return is_bf16 ? launch_latent_prefill<__nv_bfloat16, 1>(m, p, num_seqs, max_q_len, stream) : launch_latent_prefill<__half, 1>(m, p, num_seqs, max_q_len, stream);
    return is_bf16 ? launch_latent_prefill<__nv_bfloat16, 2>(m, p, num_seqs, max_q_len, stream) : launch_latent_prefill<__half, 2>(m, p, num_seqs, max_q_len, stream);
}
