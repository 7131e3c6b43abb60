// bfloat16 prompt attention with one or two maps a head on tcgen05 tensor cores (the rules: csrc/attention_maps.cu): key sizes
// that are multiples of 8 up to 128, value sizes likewise, pages of a multiple of 64 tokens. (Queries are loaded through a map of
// [token, head and map, channel], so that channels past a key's size are zeros whatever lies behind the key in its row.)
//
// A CTA carries two groups of 128 query rows that share its value tiles: with one map two groups of queries of one head, with two
// maps the two maps of the same 128 queries (each with its own keys, in the same cache rows). It walks the 64-key tiles that some
// of its queries see: the tiles of kept first keys, then those from the window's first to the diagonal. Per group
//   S = Q K^T    tcgen05.mma 128 x 64 x 16, Q and K in shared memory (TMA, 128-byte swizzle), S in one of two tensor-memory buffers
//   softmax      four warps, a query row a thread: the cap, the mask, a running maximum that may lag by 2^8, 2^x, the row's sum; the
//                weights P go back over the S they came from as bfloat16 pairs
//   O += P V     P from tensor memory, V from shared memory as an MN-major operand
// Warp 0 loads, warp 1 issues the score products and owns the tensor memory, warps 10 and 11 issue the groups' P V products,
// warps 2-5 and 6-9 are the groups' softmax and epilogue. With two maps the epilogue meets: both groups' warps read both outputs
// of their query row (warps of equal rank see the same tensor-memory lanes), a half of the channels each, subtract, exchange
// their shares of the sum of squares through shared memory, scale, gate and store.
//
// The cap c tanh(s / c): where every |s / c| of a warp's tile is at most 1/4 a polynomial of degree 7 on packed pairs (its error is
// below 3e-7 of the value there), else 1 - 2 / (1 + e^(2x)) on the special-function unit. Capped scores lie between -c and c, so
// with c up to 55 the weights need no maximum at all: 2^(c log2 e) stays below 2^80, far inside the range of float32 and bfloat16,
// and neither the search for a row's maximum nor any rescaling is left (CAP 1; larger caps keep the running maximum, CAP 2).
// Keys past a row's length are masked; they are read (a page is loaded whole), which is safe because cache pools start as zeros
// and only ever hold finite values. Every mbarrier wait is bounded (tcgen05.cuh).
#include "tcgen05.cuh"

#define AM_BM 128                                  // query rows a group
#define AM_GROUPS 2
#define AM_BN 64
#define AM_STAGES 3
#define AM_Q_BLOCK (AM_BM * 64 * 2)                // 16 KB: [128 rows x 64 channels], swizzled
#define AM_KV_BLOCK (AM_BN * 64 * 2)               // 8 KB: [64 keys x 64 channels]
#define AM_TMEM_COLS 512                           // per group: S0 [0, 64), S1 [64, 128), O [128, 256)
#define AM_RESCALE 8.0f
#define AM_PV_WARP 10
#define AM_THREADS 384
#define AM_LOG2E 1.4426950408889634f

struct MapsPrompt {
    bf16* out;
    const int32_t* block_table;
    const int32_t* row_slot;
    const int32_t* query_start;
    const int32_t* kv_len;
    const bf16* gate;
    long gate_ld;
    int table_stride, row0, rows, heads, kv_heads, dim, vdim, pages, page_size, window, keep, tile_q;
    float scale, cap, lam, factor, eps;
};

__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float am_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

template <int MAPS, int CAP, int QB, int VB>
__global__ void __launch_bounds__(AM_THREADS, 1) maps_prompt_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                    const __grid_constant__ CUtensorMap map_kv, const MapsPrompt a) {
    extern __shared__ unsigned char smem_raw[];
    constexpr int qb = QB, vb = VB;                                      // 64-channel blocks of a key and of a value
    constexpr uint32_t k_bytes = MAPS * qb * AM_KV_BLOCK, stage_bytes = k_bytes + vb * AM_KV_BLOCK;
    constexpr uint32_t q_bytes = qb * AM_Q_BLOCK;                        // a group's queries
    const uint32_t base = (smem_addr(smem_raw) + 1023u) & ~1023u;
    const uint32_t q_s = base, kv_s = q_s + AM_GROUPS * q_bytes;
    const uint32_t bars = kv_s + AM_STAGES * stage_bytes;
    const uint32_t q_full = bars, kv_full0 = bars + 8, kv_empty0 = kv_full0 + 8 * AM_STAGES;
    // per group g and buffer i, at index (g * 2 + i): scores computed; weights written; weights read (O holds the tile)
    const uint32_t s_full0 = kv_empty0 + 8 * AM_STAGES, p_full0 = s_full0 + 32;
    const uint32_t p_empty0 = p_full0 + 32, o_full0 = p_empty0 + 32, slot = o_full0 + 16;
    __shared__ int s_row, s_q0;
    __shared__ float s_inv[2][AM_BM], s_ss[2][AM_BM];                    // two maps: 1 / l, and shares of the sum of squares
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        int left = (int)blockIdx.y, found = -1, q0 = 0;                  // every head's late query tiles (the longest walks) first
        for (int b = a.rows - 1; b >= a.row0; --b) {
            const int tiles = (a.query_start[b + 1] - a.query_start[b] + a.tile_q - 1) / a.tile_q;
            if (left < tiles) { found = b; q0 = (tiles - 1 - left) * a.tile_q; break; }
            left -= tiles;
        }
        s_row = found; s_q0 = q0;
        mbar_init(q_full, 1);
        for (int s = 0; s < AM_STAGES; ++s) { mbar_init(kv_full0 + 8 * s, 1); mbar_init(kv_empty0 + 8 * s, 1 + AM_GROUPS); }
        for (int i = 0; i < 2 * AM_GROUPS; ++i) {
            mbar_init(s_full0 + 8 * i, 1);
            mbar_init(p_full0 + 8 * i, 4); mbar_init(p_empty0 + 8 * i, 1);
        }
        for (int g = 0; g < AM_GROUPS; ++g) mbar_init(o_full0 + 8 * g, 1);
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(slot), "r"(AM_TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    uint32_t tmem;
    asm volatile("ld.shared.b32 %0, [%1];\n" : "=r"(tmem) : "r"(slot));

    const int b = s_row, h = (int)blockIdx.x, hk = h / (a.heads / a.kv_heads);
    int tile_lo = 0, kt = 0, t0 = 0, p0 = 0, n = 0, nq = 0;
    int g_tiles[AM_GROUPS] = {0, 0}, g_qn[AM_GROUPS] = {0, 0}, g_hi[AM_GROUPS] = {0, 0};
    if (b >= 0) {
        nq = a.query_start[b + 1] - a.query_start[b];
        n = a.kv_len[b];
        t0 = a.query_start[b] + s_q0;
        p0 = n - nq + s_q0;                                              // position of the CTA's first query
        tile_lo = (a.window > 0 ? max(0, p0 - a.window + 1) : 0) / AM_BN;
        kt = min((a.keep + AM_BN - 1) / AM_BN, tile_lo);                 // tiles of kept first keys before the window's
#pragma unroll
        for (int g = 0; g < AM_GROUPS; ++g) {
            const int first = MAPS == 1 ? g * AM_BM : 0;                 // the group's first query among the CTA's
            g_qn[g] = max(0, min(AM_BM, min(nq - s_q0, a.tile_q) - first));
            g_hi[g] = g_qn[g] ? min(n, p0 + first + g_qn[g]) : 0;        // keys below this are visible to some of them
            g_tiles[g] = g_qn[g] ? kt + (g_hi[g] + AM_BN - 1) / AM_BN - tile_lo : 0;
        }
    }
    const int tiles = max(g_tiles[0], g_tiles[1]);
    auto tile_at = [&](int j) -> int { return j < kt ? j : tile_lo + j - kt; };

    if (b >= 0 && warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(q_full, AM_GROUPS * q_bytes);
            for (int g = 0; g < AM_GROUPS; ++g)                          // (a group without queries loads rows it never uses)
                for (int c = 0; c < qb; ++c)
                    tma_load_3d(q_s + g * q_bytes + c * AM_Q_BLOCK, &map_q, q_full, c * 64, MAPS == 1 ? h : h * 2 + g,
                                t0 + (MAPS == 1 ? g * AM_BM : 0));
            const int32_t* table = a.block_table + (size_t)a.row_slot[b] * a.table_stride;
            for (int j = 0; j < tiles; ++j) {
                const int s = j % AM_STAGES;
                if (!mbar_wait(kv_empty0 + 8 * s, ((j / AM_STAGES) & 1) ^ 1, 1)) break;
                const int key0 = tile_at(j) * AM_BN;
                int page = table[key0 / a.page_size];
                page = page < 0 || page >= a.pages ? 0 : page;
                const int row = (page * a.kv_heads + hk) * a.page_size + key0 % a.page_size;      // row of the flattened cache
                const uint32_t dst = kv_s + s * stage_bytes;
                mbar_expect_tx(kv_full0 + 8 * s, stage_bytes);
                for (int m = 0; m < MAPS; ++m)
                    for (int c = 0; c < qb; ++c)
                        tma_load_2d(dst + (m * qb + c) * AM_KV_BLOCK, &map_kv, kv_full0 + 8 * s, m * a.dim + c * 64, row);
                for (int c = 0; c < vb; ++c)
                    tma_load_2d(dst + k_bytes + c * AM_KV_BLOCK, &map_kv, kv_full0 + 8 * s, MAPS * a.dim + c * 64, row);
            }
        }
    } else if (b >= 0 && (warp == 1 || warp >= AM_PV_WARP)) {
        if (lane == 0) {
            // kind::f16, D float32, A and B bfloat16; N / 8 at bit 17, M / 16 at bit 24; bit 16: B is MN-major
            const uint32_t idesc_qk = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(AM_BN >> 3) << 17) | ((uint32_t)(AM_BM >> 4) << 24);
            const uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)((a.vdim + 15) >> 4) << 18) | ((uint32_t)(AM_BM >> 4) << 24);
            if (warp == 1) {
                bool ok = mbar_wait(q_full, 0, 2);
                for (int j = 0; j < tiles && ok; ++j) {
                    const int s = j % AM_STAGES;
                    ok = mbar_wait(kv_full0 + 8 * s, (j / AM_STAGES) & 1, 3);
                    for (int g = 0; g < AM_GROUPS && ok; ++g) {
                        if (j >= g_tiles[g]) continue;
                        const int gb = g * 2 + (j & 1);
                        // S_j overwrites S and P of tile j - 2: wait until P V of that tile has read them
                        if (j >= 2) ok = mbar_wait(p_empty0 + 8 * gb, ((j - 2) >> 1) & 1, 4);
                        if (!ok) break;
                        tc_fence_after();
                        const uint32_t s_t = tmem + g * 256 + (j & 1) * AM_BN;
                        const uint32_t k_src = kv_s + s * stage_bytes + (MAPS == 2 ? g * qb * AM_KV_BLOCK : 0);
#pragma unroll
                        for (int kk = 0; kk < QB * 4; ++kk) {
                            const uint32_t blk = kk >> 2, within = (kk & 3) * 2;
                            tc_mma(s_t, tc_smem_desc(q_s + g * q_bytes + blk * AM_Q_BLOCK) + within,
                                   tc_smem_desc(k_src + blk * AM_KV_BLOCK) + within, idesc_qk, kk != 0);
                        }
                        tc_commit(s_full0 + 8 * gb);
                    }
                    if (ok) tc_commit(kv_empty0 + 8 * s);                // the keys of the stage have been read (all three must arrive)
                }
            } else {
                const int g = warp - AM_PV_WARP, my_tiles = g_tiles[g];
                const uint32_t o_t = tmem + g * 256 + 2 * AM_BN;
                bool ok = true;
                for (int j = 0; j < tiles && ok; ++j) {                  // (a group past its own last tile still paces the stages)
                    const int s = j % AM_STAGES, gb = g * 2 + (j & 1);
                    ok = mbar_wait(kv_full0 + 8 * s, (j / AM_STAGES) & 1, 3);
                    if (ok && j < my_tiles) {                            // O_g += P_g,j V_j
                        ok = mbar_wait(p_full0 + 8 * gb, (j >> 1) & 1, 5);
                        if (!ok) break;
                        tc_fence_after();
                        const uint32_t v_src = kv_s + s * stage_bytes + k_bytes;
                        const uint32_t p_t = tmem + g * 256 + (j & 1) * AM_BN;   // P lies over the first half of its own S
#pragma unroll
                        for (int kk = 0; kk < AM_BN / 16; ++kk)          // 16 keys a step: 8 columns along P, 16 rows down V
                            tc_mma_f16_ts(o_t, p_t + kk * 8, tc_smem_desc_mn(v_src + kk * 16 * 128, AM_KV_BLOCK), idesc_pv, (j | kk) != 0);
                        tc_commit(p_empty0 + 8 * gb);                    // P has been read; O_g holds tile j
                        if (j == my_tiles - 1) tc_commit(o_full0 + 8 * g);   // the group's last tile: its output is complete
                    }
                    if (ok) tc_commit(kv_empty0 + 8 * s);                // the values of the stage have been read
                }
                if (my_tiles == 0 || !ok) tc_commit(o_full0 + 8 * g);    // (nothing was issued for it, or the walk gave up)
            }
        }
    } else if (b >= 0 && warp < AM_PV_WARP) {
        const int g = (warp - 2) >> 2;                                   // this warp's group
        const int q = warp & 3, r = q * 32 + lane;                       // its quarter of the lanes; this thread's query row
        const int pg = p0 + (MAPS == 1 ? g * AM_BM : 0), pos = pg + r;   // the group's first position, and this row's
        const int hi = g_hi[g], qn = g_qn[g], my_tiles = g_tiles[g];
        const uint32_t lane_t = tmem + g * 256 + ((uint32_t)(q * 32) << 16);
        const uint32_t o_t = lane_t + 2 * AM_BN;
        const float scale_log2 = CAP ? 1.f : a.scale * AM_LOG2E;         // capped scores are already in log2 units
        const float to_x = CAP ? a.scale / a.cap : 0.f, from_x = CAP ? a.cap * AM_LOG2E : 0.f;
        const float t2 = to_x * to_x;
        // c log2(e) tanh(s t) = s (scale log2 e) (1 + s^2 (-t^2/3 + s^2 (2 t^4/15 - s^2 17 t^6/315))), t = scale / c
        const uint64_t c7 = pack2(-17.f / 315.f * t2 * t2 * t2, -17.f / 315.f * t2 * t2 * t2), c5 = pack2(2.f / 15.f * t2 * t2, 2.f / 15.f * t2 * t2);
        const uint64_t c3 = pack2(-1.f / 3.f * t2, -1.f / 3.f * t2), one = pack2(1.f, 1.f);
        const uint64_t fx = pack2(a.scale * AM_LOG2E, a.scale * AM_LOG2E);
        float m_used = -INFINITY, l = 0.f;                               // in log2 units; the maximum may lag by AM_RESCALE
        bool ok = true;
        for (int j = 0; j < my_tiles && ok; ++j) {
            const int gb = g * 2 + (j & 1);
            ok = mbar_wait(s_full0 + 8 * gb, (j >> 1) & 1, 6);
            if (!ok) break;
            tc_fence_after();
            uint32_t sr[2][32];
            tc_ld32_nowait(lane_t + (j & 1) * AM_BN, sr[0]);
            tc_ld32_nowait(lane_t + (j & 1) * AM_BN + 32, sr[1]);
            tc_ld_wait();
            if (CAP) {
                float top4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int i = 0; i < 32; ++i) top4[i & 3] = fmaxf(top4[i & 3], fabsf(__uint_as_float(sr[c][i])));
                const float top = fmaxf(fmaxf(top4[0], top4[1]), fmaxf(top4[2], top4[3])) * to_x;
                if (__all_sync(0xffffffffu, top <= 0.25f)) {
#pragma unroll
                    for (int c = 0; c < 2; ++c)
#pragma unroll
                        for (int i = 0; i < 32; i += 2) {
                            const uint64_t x = pack2(__uint_as_float(sr[c][i]), __uint_as_float(sr[c][i + 1])), y = mul2(x, x);
                            const uint64_t w = fma2(y, fma2(y, fma2(y, c7, c5), c3), one);
                            float u, v;
                            unpack2(mul2(mul2(x, fx), w), u, v);
                            sr[c][i] = __float_as_uint(u); sr[c][i + 1] = __float_as_uint(v);
                        }
                } else {
#pragma unroll
                    for (int c = 0; c < 2; ++c)
#pragma unroll
                        for (int i = 0; i < 32; ++i) {
                            const float e = at_ex2(__uint_as_float(sr[c][i]) * to_x * (2.f * AM_LOG2E));     // e^(2x); inf gives 1
                            sr[c][i] = __float_as_uint(from_x * (1.f - __fdividef(2.f, 1.f + e)));
                        }
                }
            }
            const int key0 = tile_at(j) * AM_BN;
            const bool edge = key0 + AM_BN - 1 > pg || key0 + AM_BN > hi
                              || (a.window > 0 && pg + qn - 1 - key0 >= a.window && key0 + AM_BN > a.keep);
            if (edge) {
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        const int key = key0 + c * 32 + i;
                        if (!(key <= pos && key < hi && (a.window <= 0 || pos - key < a.window || key < a.keep))) sr[c][i] = 0xff800000u;
                    }
            }
            if constexpr (CAP != 1) {
                float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY}; // four chains instead of one of 64
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int i = 0; i < 32; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sr[c][i]));
                const float mt = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;
                const bool grow = mt > m_used + AM_RESCALE || (m_used == -INFINITY && mt > -INFINITY);
                if (__any_sync(0xffffffffu, grow)) {                         // rescale what is summed (whole warp: the TMEM ops are collective)
                    const float m_new = grow ? mt : m_used;
                    const float f = m_used == -INFINITY ? 0.f : at_ex2(m_used - m_new);
                    if (j > 0) {
                        ok = mbar_wait(p_empty0 + 8 * (g * 2 + ((j - 1) & 1)), ((j - 1) >> 1) & 1, 7);   // O holds every tile before j
                        tc_fence_after();
                        if (ok) {
                            for (int c = 0; c < (a.vdim + 31) >> 5; ++c) {
                                uint32_t o[32];
                                tc_ld32(o_t + c * 32, o);
#pragma unroll
                                for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
                                tc_st32(o_t + c * 32, o);
                            }
                        }
                    }
                    l *= f;
                    m_used = m_new;
                }
            }
            const float off = CAP == 1 || m_used == -INFINITY ? 0.f : -m_used;
            const uint64_t scale2 = pack2(scale_log2, scale_log2), off2 = pack2(off, off);
            uint64_t sum2[4] = {0ull, 0ull, 0ull, 0ull};                 // four chains of packed sums
            uint32_t pk[32];                                             // 64 weights as bfloat16 pairs
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int i = 0; i < 32; i += 2) {
                    float x, y;
                    if constexpr (CAP == 1) { x = __uint_as_float(sr[c][i]); y = __uint_as_float(sr[c][i + 1]); }
                    else unpack2(fma2(pack2(__uint_as_float(sr[c][i]), __uint_as_float(sr[c][i + 1])), scale2, off2), x, y);
                    x = at_ex2(x);
                    y = at_ex2(y);
                    sum2[(i >> 1) & 3] = add2(sum2[(i >> 1) & 3], pack2(x, y));
                    __nv_bfloat162 pr = __floats2bfloat162_rn(x, y);
                    pk[c * 16 + i / 2] = *(uint32_t*)&pr;
                }
            {
                float x, y;
                unpack2(add2(add2(sum2[0], sum2[1]), add2(sum2[2], sum2[3])), x, y);
                l += x + y;
            }
            if (!ok) break;
            tc_st32(lane_t + (j & 1) * AM_BN, pk);                       // P over the S it came from: 32 columns of bfloat16 pairs
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full0 + 8 * gb);
        }
        constexpr int CHUNKS = VB * 2, MINE = MAPS == 1 ? CHUNKS : VB;   // chunks of 32 channels; this thread's (two maps: g, g + 2)
        const int chunks = (a.vdim + 31) >> 5;
        const size_t token = (size_t)(t0 + (MAPS == 1 ? g * AM_BM : 0) + (r < qn ? r : 0));
        bf16* o_row = a.out + (token * a.heads + h) * a.vdim;
        const bf16* g_row = a.gate ? a.gate + token * a.gate_ld + (size_t)h * a.vdim : nullptr;
        const bool g_vec = (((uintptr_t)a.gate | (uintptr_t)(a.gate_ld * 2)) & 15) == 0;      // (vdim is a multiple of 8)
        uint4 gq[MINE][4];                                               // the row's gates, asked for ahead of the last products
#pragma unroll
        for (int k = 0; k < MINE; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int d = (MAPS == 1 ? k : g + 2 * k) * 32 + i * 8;
                gq[k][i] = make_uint4(0u, 0u, 0u, 0u);
                if (g_row && g_vec && r < qn && d < a.vdim) gq[k][i] = *(const uint4*)(g_row + d);
            }
        if (ok) ok = mbar_wait(o_full0 + 8 * g, 0, 9);
        tc_fence_after();
        const float inv = ok && my_tiles > 0 && l > 0.f ? 1.f / l : 0.f;
        auto store = [&](const float (&v)[32], int c, const uint4 (&gz)[4]) {                  // a chunk of 32 channels of this thread's row, gated
            const int live = min(32, a.vdim - c * 32);                   // a multiple of 8
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
                if (i >= live) break;
                float y[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) y[e] = v[i + e];
                if (g_row) {
                    float z[8];
                    if (g_vec) {
                        const uint4 w = gz[i / 8];
                        const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                        for (int e = 0; e < 4; ++e) { z[2 * e] = __uint_as_float(u[e] << 16); z[2 * e + 1] = __uint_as_float(u[e] & 0xffff0000u); }
                    } else {
#pragma unroll
                        for (int e = 0; e < 8; ++e) z[e] = to_f32(g_row[c * 32 + i + e]);
                    }
#pragma unroll
                    for (int e = 0; e < 8; ++e) y[e] *= am_sigmoid(z[e]);
                }
                uint4 w;
                __nv_bfloat162 a0 = __floats2bfloat162_rn(y[0], y[1]), a1 = __floats2bfloat162_rn(y[2], y[3]);
                __nv_bfloat162 a2 = __floats2bfloat162_rn(y[4], y[5]), a3 = __floats2bfloat162_rn(y[6], y[7]);
                w.x = *(uint32_t*)&a0; w.y = *(uint32_t*)&a1; w.z = *(uint32_t*)&a2; w.w = *(uint32_t*)&a3;
                *(uint4*)(o_row + c * 32 + i) = w;
            }
        };
        if (MAPS == 1) {
            if (ok && qn > 0) {                                          // (the tensor-memory loads are warp-collective: no lane skips them)
#pragma unroll
                for (int c = 0; c < CHUNKS; ++c) {
                    if (c >= chunks) break;
                    uint32_t o[32];
                    tc_ld32(o_t + c * 32, o);
                    float v[32];
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = inv > 0.f ? __uint_as_float(o[i]) * inv : 0.f;
                    if (r < qn) store(v, c, gq[c < MINE ? c : 0]);
                }
            }
        } else {
            s_inv[g][r] = inv;
            tc_fence_before();
            asm volatile("bar.sync 1, 256;\n" ::: "memory");             // both maps' outputs are complete (both groups' softmax warps)
            tc_fence_after();
            const float i1 = s_inv[0][r], i2 = s_inv[1][r] * a.lam;
            const uint32_t row_t = tmem + ((uint32_t)(q * 32) << 16) + 2 * AM_BN;
            float v[VB][32], ss = 0.f;                                   // channels of chunks g, g + 2
#pragma unroll
            for (int k = 0; k < VB; ++k) {
                const int c = g + 2 * k;
#pragma unroll
                for (int i = 0; i < 32; ++i) v[k][i] = 0.f;
                if (c < chunks) {
                    uint32_t o1[32], o2[32];
                    tc_ld32_nowait(row_t + c * 32, o1);
                    tc_ld32_nowait(row_t + 256 + c * 32, o2);
                    tc_ld_wait();
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        if (i < a.vdim - c * 32) {                       // (a row's last chunk may be a part of a chunk)
                            v[k][i] = (i1 > 0.f ? __uint_as_float(o1[i]) * i1 : 0.f) - (s_inv[1][r] > 0.f ? __uint_as_float(o2[i]) * i2 : 0.f);
                            ss = fmaf(v[k][i], v[k][i], ss);
                        }
                    }
                }
            }
            s_ss[g][r] = ss;
            asm volatile("bar.sync 1, 256;\n" ::: "memory");
            const float f = rsqrtf((s_ss[0][r] + s_ss[1][r]) / (float)a.vdim + a.eps) * a.factor;
#pragma unroll
            for (int k = 0; k < VB; ++k) {
                const int c = g + 2 * k;
                if (c < chunks && r < qn) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[k][i] *= f;
                    store(v[k], c, gq[k]);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(AM_TMEM_COLS) : "memory");
    }
}

static int encode_rows(CUtensorMap* map, const void* ptr, uint64_t cols, uint64_t rows, uint32_t box_rows, const char* what) {
    const cuuint64_t dims[2] = {cols, rows};
    const cuuint64_t strides[1] = {cols * 2};
    const cuuint32_t box[2] = {64, box_rows};
    const cuuint32_t elem[2] = {1, 1};
    const CUresult r = cuTensorMapEncodeTiled(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box,
                                              elem, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                              CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) HB_REFUSE("attention_maps_prefill: cuTensorMapEncodeTiled failed with %d for %s", (int)r, what);
    return 0;
}

HB_DEFINE_STATUS_MIRROR(hb_attention_maps_status_mirror)
extern "C" int hb_attention_maps_status(unsigned int* status) {
    HB_CUDA(cudaDeviceSynchronize());
    HB_CUDA(cudaMemcpyFromSymbol(status, g_tc_status, sizeof(unsigned int)));
    const unsigned int zero = 0;
    HB_CUDA(cudaMemcpyToSymbol(g_tc_status, &zero, sizeof(unsigned int)));
    return 0;
}

// Rows row0 .. rows - 1 of the batch; q_tiles is the sum of ceil(queries / tile_q) over them; tokens the step's token count.
// tile_q: 128, or with one map 256.
extern "C" int hb_attention_maps_prefill(void* out, const void* q, const void* kv, const int32_t* block_table, int table_stride,
                                         const int32_t* row_slot, const int32_t* query_start, const int32_t* kv_len, int row0,
                                         int rows, int q_tiles, int tokens, int heads, int kv_heads, int maps, int dim, int vdim,
                                         int pages, int page_size, float scale, float cap, int window, int keep, float lam,
                                         float factor, float eps, const void* gate, long gate_ld, int tile_q, hb_stream stream) {
    if (rows <= row0 || q_tiles == 0) return 0;
    if (maps != 1 && maps != 2) HB_REFUSE("attention_maps_prefill: %d maps (1 or 2)", maps);
    if (dim % 8 || dim < 8 || dim > 128 || vdim % 8 || vdim < 8 || vdim > 128)
        HB_REFUSE("attention_maps_prefill: keys of %d and values of %d: multiples of 8 up to 128", dim, vdim);
    if (tile_q != AM_BM && (maps == 2 || tile_q != AM_GROUPS * AM_BM)) HB_REFUSE("attention_maps_prefill: query tiles of %d", tile_q);
    if (page_size % AM_BN) HB_REFUSE("attention_maps_prefill: page size %d is no multiple of %d", page_size, AM_BN);
    if (kv_heads < 1 || heads % kv_heads) HB_REFUSE("attention_maps_prefill: %d heads, %d kv heads", heads, kv_heads);
    if (q_tiles > 65535) HB_REFUSE("attention_maps_prefill: %d query tiles in one step, above 65535", q_tiles);
    if (!(scale > 0.f) || cap < 0.f || window < 0 || keep < 0) HB_REFUSE("attention_maps_prefill: the score scale must be positive, cap, window and kept keys not negative");
    if ((((uintptr_t)q | (uintptr_t)kv | (uintptr_t)out) % 16) != 0) HB_REFUSE("attention_maps_prefill: pointers must be 16-byte aligned");
    const uint64_t kv_rows = (uint64_t)pages * kv_heads * page_size;
    if (kv_rows > 0x7fffffffull) HB_REFUSE("attention_maps_prefill: the cache has %llu rows, above 2^31", (unsigned long long)kv_rows);
    CUtensorMap map_q, map_kv;
    {
        const cuuint64_t dims[3] = {(cuuint64_t)dim, (cuuint64_t)heads * maps, (cuuint64_t)tokens};
        const cuuint64_t strides[2] = {(cuuint64_t)dim * 2, (cuuint64_t)heads * maps * dim * 2};
        const cuuint32_t box[3] = {64, 1, AM_BM}, elem[3] = {1, 1, 1};
        const CUresult r = cuTensorMapEncodeTiled(&map_q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), dims, strides, box, elem,
                                                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                                  CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
        if (r != CUDA_SUCCESS) HB_REFUSE("attention_maps_prefill: cuTensorMapEncodeTiled failed with %d for q", (int)r);
    }
    int rc = encode_rows(&map_kv, kv, (uint64_t)maps * dim + vdim, kv_rows, AM_BN, "the cache");
    if (rc) return rc;
    const int qb = (dim + 63) / 64, vb = (vdim + 63) / 64;
    const size_t smem = AM_GROUPS * (size_t)qb * AM_Q_BLOCK + AM_STAGES * (size_t)(maps * qb + vb) * AM_KV_BLOCK + 1024 + 256;
    const MapsPrompt p{(bf16*)out, block_table, row_slot, query_start, kv_len, (const bf16*)gate, gate_ld, table_stride, row0, rows,
                       heads, kv_heads, dim, vdim, pages, page_size, window, window > 0 ? keep : 0, tile_q, scale, cap, lam, factor, eps};
    void (*kernel)(const CUtensorMap, const CUtensorMap, const MapsPrompt) = nullptr;
    const int kind = cap <= 0.f ? 0 : cap <= 55.f ? 1 : 2;
#define HB_PICK(M, C) if (maps == M && kind == C) kernel = qb == 1 ? (vb == 1 ? maps_prompt_kernel<M, C, 1, 1> : maps_prompt_kernel<M, C, 1, 2>) \
                                                                   : (vb == 1 ? maps_prompt_kernel<M, C, 2, 1> : maps_prompt_kernel<M, C, 2, 2>)
    HB_PICK(1, 0); HB_PICK(1, 1); HB_PICK(1, 2); HB_PICK(2, 0); HB_PICK(2, 1); HB_PICK(2, 2);
#undef HB_PICK
    HB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kernel<<<dim3(heads, q_tiles), AM_THREADS, smem, (cudaStream_t)stream>>>(map_q, map_kv, p);
    HB_LAUNCH_CHECK("attention_maps_prefill");
    return 0;
}
