// Attention with one or two maps a head over a paged cache that keeps per token and kv head one row [key of map 1 | key of
// map 2 | value] (maps * dim + vdim numbers): cache [pages, kv_heads, page_size, maps dim + vdim].
//
//   s_hm(i, j) = q_hm(i) . k_gm(j) * scale,  with a cap c > 0: c tanh(s / c)
//   a_hm(i)    = sum_j softmax_j(s_hm(i, .)) v_g(j)   over the keys j <= i with i - j < window (0: all) or j < keep
//   o_h        = a_h1, or with two maps (a_h1 - lambda a_h2) / sqrt(mean(.^2) + eps) * factor
//   out_h      = o_h * sigmoid(gate_h)                (gate null: o_h)
//
// g is head h's kv head. The epilogue (difference, its norm, the gate) is 32-bit and part of every kernel here: no map's
// result is ever rounded or written. Scores, weights and sums are 32-bit.
//
// hb_qkv_maps_prepare   a first product's rows [q | k | v | ...] -> norms, rotation, q rows, cache rows
// hb_attention_maps     any sizes on CUDA cores: the float32 engine's kernel, and the bfloat16 engine's for sizes that the
//                       tensor-core kernels refuse
// hb_attention_maps_decode  bfloat16 rows of one token on mma.sync tiles; a row's keys in parts, one CTA each, that meet in a
//                       thread-block cluster
// (Rows of several tokens: csrc/attention_maps_tcgen05.cu.)
#include "attention_mma.cuh"

#define LOG2E 1.4426950408889634f
__device__ __forceinline__ float mp_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// ---------------------------------------------------------------- from the first product to q rows and cache rows
// One warp per token and SL slots: heads * maps queries, kv_heads * maps keys, kv_heads values. norm 1: x / rms(x) * weight, then
// the rotation; norm 2: the rotation, then x / rms(x); 0: no norm. The first rot_dims channels turn in half-split pairs;
// `table` holds, per position, the rot_dims / 2 cosines and then the sines. One rounding, at the end. PAIR: a lane owns runs of
// two neighbouring channels (dim, vdim, the rows and the cache even), else every 32nd channel.
#define MP_WARPS 4
#define MP_PER_LANE 16            // sizes up to 512 (PL: numbers a lane holds, 4 for sizes up to 128)
template <typename T> struct Two;
template <> struct Two<float> {
    static __device__ __forceinline__ float2 load(const float* p) { return *(const float2*)p; }
    static __device__ __forceinline__ void store(float* p, float a, float b) { *(float2*)p = make_float2(a, b); }
};
template <> struct Two<bf16> {
    static __device__ __forceinline__ float2 load(const bf16* p) { return __bfloat1622float2(*(const __nv_bfloat162*)p); }
    static __device__ __forceinline__ void store(bf16* p, float a, float b) { *(__nv_bfloat162*)p = __floats2bfloat162_rn(a, b); }
};

template <typename T, bool PAIR, int PL, int SL>
__global__ void maps_prepare_kernel(T* __restrict__ q_out, T* __restrict__ kv, const T* __restrict__ first, long ld,
                                    const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps, int norm,
                                    const int32_t* __restrict__ positions, const float* __restrict__ table, int rot_dims,
                                    int table_rows, const int32_t* __restrict__ write_index, int pages, int page_size,
                                    int heads, int kv_heads, int maps, int dim, int vdim) {
    extern __shared__ __align__(16) float mp_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nq = heads * maps, nk = kv_heads * maps, slots = nq + nk + kv_heads;
    const long t = blockIdx.x;
    const int slot0 = ((int)blockIdx.y * MP_WARPS + warp) * SL;
    if (slot0 >= slots) return;
    const int rowlen = maps * dim + vdim, last = min(slots, slot0 + SL);
    const long w = write_index ? write_index[t] : -1;
    const bool stored = w >= 0 && w < (long)pages * page_size;
    const long page = stored ? w / page_size : 0, off = stored ? w - page * page_size : 0;
    const T* row = first + t * ld;
    float* ys = mp_smem + (size_t)warp * ((dim + 3) & ~3);
    auto at = [&](int i) -> int { return PAIR ? 2 * lane + 64 * (i >> 1) + (i & 1) : lane + 32 * i; };
    float x[SL][PL];                                                  // every slot's numbers are asked for before any is worked on
#pragma unroll
    for (int s = 0; s < SL; ++s) {
        const T* src = row + (long)(slot0 + s) * dim;                 // (queries, then keys, map by map: one numbering)
        const bool mine = slot0 + s < nq + nk;
#pragma unroll
        for (int i = 0; i < PL; i += PAIR ? 2 : 1) {
            const int d = at(i);
            if (PAIR) {
                const float2 v = mine && d < dim ? Two<T>::load(src + d) : make_float2(0.f, 0.f);
                x[s][i] = v.x; x[s][i + 1] = v.y;
            } else {
                x[s][i] = mine && d < dim ? to_f32(src[d]) : 0.f;
            }
        }
    }
    const int half = rot_dims >> 1;
    float co[PL], si[PL];                                             // the token's angles, for all its slots
    if (rot_dims) {
        int pos = positions[t];
        pos = pos < 0 ? 0 : (pos >= table_rows ? table_rows - 1 : pos);
        const float* cs = table + (size_t)pos * rot_dims;
#pragma unroll
        for (int i = 0; i < PL; ++i) {
            const int d = at(i), c = d < half ? d : d - half;
            co[i] = d < rot_dims ? cs[c] : 1.f;
            si[i] = d < rot_dims ? cs[half + c] : 0.f;
        }
    }
#pragma unroll
    for (int s = 0; s < SL; ++s) {
        const int slot = slot0 + s;
        if (slot >= last) break;
        if (slot >= nq + nk) {                                        // a value head: copied
            if (!stored) continue;
            const int c = slot - nq - nk;
            const T* src = row + (long)(nq + nk) * dim + (long)c * vdim;
            T* dst = kv + ((page * kv_heads + c) * page_size + off) * rowlen + maps * dim;
            if (PAIR) {
                for (int d = 2 * lane; d < vdim; d += 64) { const float2 v = Two<T>::load(src + d); Two<T>::store(dst + d, v.x, v.y); }
            } else {
                for (int d = lane; d < vdim; d += 32) dst[d] = src[d];
            }
            continue;
        }
        const bool is_q = slot < nq;
        T* dst = nullptr;
        if (is_q) dst = q_out + (t * nq + slot) * dim;
        else if (stored) {
            const int c = (slot - nq) / maps, m = (slot - nq) - c * maps;
            dst = kv + ((page * kv_heads + c) * page_size + off) * rowlen + m * dim;
        }
        if (!dst) continue;
        float ss = 0.f;
        if (norm == 1) {
            const float* weight = is_q ? q_weight : k_weight;
#pragma unroll
            for (int i = 0; i < PL; ++i) ss += x[s][i] * x[s][i];
            const float r = rsqrtf(warp_sum(ss) / (float)dim + eps);
#pragma unroll
            for (int i = 0; i < PL; ++i) { const int d = at(i); if (d < dim) x[s][i] *= r * weight[d]; }
        }
        if (rot_dims) {
            __syncwarp();                                             // (the slot before has read its numbers)
#pragma unroll
            for (int i = 0; i < PL; ++i) { const int d = at(i); if (d < rot_dims) ys[d] = x[s][i]; }
            __syncwarp();
#pragma unroll
            for (int i = 0; i < PL; ++i) {
                const int d = at(i);
                if (d < rot_dims) {                                   // u of the pair (u, v), or v
                    const float o = ys[d < half ? d + half : d - half];
                    x[s][i] = d < half ? x[s][i] * co[i] - o * si[i] : x[s][i] * co[i] + o * si[i];
                }
            }
        }
        if (norm == 2) {
            ss = 0.f;
#pragma unroll
            for (int i = 0; i < PL; ++i) ss += x[s][i] * x[s][i];
            const float r = rsqrtf(warp_sum(ss) / (float)dim + eps);
#pragma unroll
            for (int i = 0; i < PL; ++i) x[s][i] *= r;
        }
#pragma unroll
        for (int i = 0; i < PL; i += PAIR ? 2 : 1) {
            const int d = at(i);
            if (d < dim) { if (PAIR) Two<T>::store(dst + d, x[s][i], x[s][i + 1]); else dst[d] = from_f32<T>(x[s][i]); }
        }
    }
}

extern "C" int hb_qkv_maps_prepare(void* q_out, void* kv, const void* first, int dtype, long ld, const float* q_weight,
                                   const float* k_weight, float eps, int norm, const int32_t* positions, const float* table,
                                   int rot_dims, int table_rows, const int32_t* write_index, int pages, int page_size, int tokens,
                                   int heads, int kv_heads, int maps, int dim, int vdim, hb_stream stream) {
    if (tokens == 0) return 0;
    if (dim < 1 || dim > 32 * MP_PER_LANE || vdim < 1) HB_REFUSE("qkv_maps_prepare: key size %d (1 to %d), value size %d", dim, 32 * MP_PER_LANE, vdim);
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > dim) HB_REFUSE("qkv_maps_prepare: %d rotated channels of %d", rot_dims, dim);
    if (rot_dims && (!table || table_rows < 1)) HB_REFUSE("qkv_maps_prepare: a rotation needs its table");
    if (norm < 0 || norm > 2 || (norm == 1 && (!q_weight || !k_weight))) HB_REFUSE("qkv_maps_prepare: norm %d needs both weights", norm);
    if (maps < 1 || kv_heads < 1 || heads % kv_heads) HB_REFUSE("qkv_maps_prepare: %d heads, %d kv heads, %d maps", heads, kv_heads, maps);
    const long slots = (long)heads * maps + (long)kv_heads * maps + kv_heads;
    if (slots > 65535L * MP_WARPS) HB_REFUSE("qkv_maps_prepare: %ld heads a token", slots);
    const int sl = dim <= 128 && tokens >= 64 ? 4 : 1;                // slots a warp takes in turn
    const dim3 grid(tokens, (unsigned)((slots + MP_WARPS * sl - 1) / (MP_WARPS * sl)));
    const size_t smem = (size_t)MP_WARPS * ((dim + 3) & ~3) * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
    const size_t two = dtype == HB_F32 ? 8 : 4;
    const bool pair = dim % 2 == 0 && vdim % 2 == 0 && ld % 2 == 0 && (((uintptr_t)q_out | (uintptr_t)kv | (uintptr_t)first) % two) == 0;
#define HB_ARGS(T) (T*)q_out, (T*)kv, (const T*)first, ld, q_weight, k_weight, eps, norm, positions, table, rot_dims, table_rows, \
    write_index, pages, page_size, heads, kv_heads, maps, dim, vdim
#define HB_RUN(T, P) do { if (sl == 4) maps_prepare_kernel<T, P, 4, 4><<<grid, MP_WARPS * 32, smem, s>>>(HB_ARGS(T)); \
                          else if (dim <= 128) maps_prepare_kernel<T, P, 4, 1><<<grid, MP_WARPS * 32, smem, s>>>(HB_ARGS(T)); \
                          else maps_prepare_kernel<T, P, MP_PER_LANE, 1><<<grid, MP_WARPS * 32, smem, s>>>(HB_ARGS(T)); } while (0)
    if (dtype == HB_F32) { if (pair) HB_RUN(float, true); else HB_RUN(float, false); }
    else if (dtype == HB_BF16) { if (pair) HB_RUN(bf16, true); else HB_RUN(bf16, false); }
    else HB_REFUSE("qkv_maps_prepare: dtype %d", dtype);
#undef HB_RUN
#undef HB_ARGS
    HB_LAUNCH_CHECK("qkv_maps_prepare");
    return 0;
}

// ---------------------------------------------------------------- any sizes, CUDA cores
// One warp per (token, head), its maps one after the other. A lane scores one key of a block of 32, the block's weights then
// sweep the values, a lane owning every 32nd value channel. The visible keys are numbered without the gap between the kept
// first ones and the window.
#define MG_WARPS 4
#define MG_PER_LANE 16            // value sizes up to 512
template <typename T>
__global__ void attention_maps_kernel(T* __restrict__ out, const T* __restrict__ q, const T* __restrict__ kv,
                                      const int32_t* __restrict__ block_table, int table_stride,
                                      const int32_t* __restrict__ row_slot, const int32_t* __restrict__ query_start,
                                      const int32_t* __restrict__ kv_len, int rows, int tokens, int heads, int kv_heads, int maps,
                                      int dim, int vdim, int pages, int page_size, float scale, float cap, int window, int keep,
                                      float lam, float factor, float eps, const T* __restrict__ gate, long gate_ld) {
    extern __shared__ __align__(16) float mp_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long item = (long)blockIdx.x * MG_WARPS + warp;
    if (item >= (long)tokens * heads) return;
    const int t = (int)(item / heads), h = (int)(item % heads);
    float* qs = mp_smem + (size_t)warp * dim;
    int lo = 0, hi = rows;                                   // the row b with query_start[b] <= t < query_start[b + 1]
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (query_start[mid] <= t) lo = mid; else hi = mid;
    }
    const int b = lo, n = kv_len[b];
    const int pos = n - query_start[b + 1] + t;              // the query's position in its sequence
    T* o = out + ((size_t)t * heads + h) * vdim;
    if (n <= 0 || pos < 0) {
        for (int d = lane; d < vdim; d += 32) o[d] = from_f32<T>(0.f);
        return;
    }
    const int rowlen = maps * dim + vdim, hk = h / (heads / kv_heads);
    const int32_t* table = block_table + (size_t)row_slot[b] * table_stride;
    const int first = window > 0 ? max(0, pos - window + 1) : 0;
    const int kept = min(keep, first), count = kept + pos - first + 1;
    float res[MG_PER_LANE];
    for (int m = 0; m < maps; ++m) {
        const T* qr = q + (((size_t)t * heads + h) * maps + m) * dim;
        __syncwarp();
        for (int d = lane; d < dim; d += 32) qs[d] = to_f32(qr[d]);
        __syncwarp();
        float mx = -INFINITY, l = 0.f, acc[MG_PER_LANE];
#pragma unroll
        for (int i = 0; i < MG_PER_LANE; ++i) acc[i] = 0.f;
        for (int i0 = 0; i0 < count; i0 += 32) {
            const int i = i0 + lane, j = i < kept ? i : first + i - kept;
            long base = -1;                                  // element offset of key j's row of this kv head
            if (i < count) {
                const int page = table[j / page_size];
                if (page >= 0 && page < pages) base = (((long)page * kv_heads + hk) * page_size + j % page_size) * rowlen;
            }
            float s = -INFINITY;
            if (base >= 0) {
                const T* kr = kv + base + m * dim;
                float dot = 0.f;
                for (int d = 0; d < dim; ++d) dot = fmaf(qs[d], to_f32(kr[d]), dot);
                s = dot * scale;
                if (cap > 0.f) s = cap * tanhf(s / cap);
            }
            const float m_new = fmaxf(mx, warp_max(s));
            const float corr = m_new == -INFINITY ? 1.f : expf(mx - m_new);
            const float p = base >= 0 ? expf(s - m_new) : 0.f;
            l = l * corr + warp_sum(p);
            mx = m_new;
#pragma unroll
            for (int x = 0; x < MG_PER_LANE; ++x) acc[x] *= corr;
            const int live = min(32, count - i0);
            for (int jj = 0; jj < live; ++jj) {
                const float pj = __shfl_sync(0xffffffffu, p, jj);
                const long bj = __shfl_sync(0xffffffffu, base, jj);
                if (bj < 0) continue;
                const T* vr = kv + bj + maps * dim;
#pragma unroll
                for (int x = 0; x < MG_PER_LANE; ++x) {
                    const int d = lane + 32 * x;
                    if (d < vdim) acc[x] = fmaf(pj, to_f32(vr[d]), acc[x]);
                }
            }
        }
        const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
        for (int x = 0; x < MG_PER_LANE; ++x) res[x] = m == 0 ? acc[x] * inv : res[x] - lam * (acc[x] * inv);
    }
    if (maps > 1) {
        float ss = 0.f;
#pragma unroll
        for (int x = 0; x < MG_PER_LANE; ++x) ss += res[x] * res[x];          // (channels past vdim hold zeros)
        const float r = rsqrtf(warp_sum(ss) / (float)vdim + eps) * factor;
#pragma unroll
        for (int x = 0; x < MG_PER_LANE; ++x) res[x] *= r;
    }
    const T* g = gate ? gate + (size_t)t * gate_ld + (size_t)h * vdim : nullptr;
#pragma unroll
    for (int x = 0; x < MG_PER_LANE; ++x) {
        const int d = lane + 32 * x;
        if (d < vdim) o[d] = from_f32<T>(g ? res[x] * mp_sigmoid(to_f32(g[d])) : res[x]);
    }
}

static int check_maps(const char* what, int heads, int kv_heads, int maps, int dim, int vdim, float scale, float cap, int window, int keep) {
    if (maps != 1 && maps != 2) HB_REFUSE("%s: %d maps (1 or 2)", what, maps);
    if (kv_heads < 1 || heads % kv_heads) HB_REFUSE("%s: %d heads are no multiple of %d kv heads", what, heads, kv_heads);
    if (dim < 1 || vdim < 1 || window < 0 || keep < 0) HB_REFUSE("%s: key size %d, value size %d, window %d, kept %d", what, dim, vdim, window, keep);
    if (!(scale > 0.f) || cap < 0.f) HB_REFUSE("%s: the score scale must be positive, the cap not negative", what);
    return 0;
}

extern "C" int hb_attention_maps(void* out, const void* q, const void* kv, int dtype, const int32_t* block_table, int table_stride,
                                 const int32_t* row_slot, const int32_t* query_start, const int32_t* kv_len, int rows, int tokens,
                                 int heads, int kv_heads, int maps, int dim, int vdim, int pages, int page_size, float scale,
                                 float cap, int window, int keep, float lam, float factor, float eps, const void* gate,
                                 long gate_ld, hb_stream stream) {
    if (tokens == 0 || rows == 0) return 0;
    if (int rc = check_maps("attention_maps", heads, kv_heads, maps, dim, vdim, scale, cap, window, keep)) return rc;
    if (vdim > 32 * MG_PER_LANE) HB_REFUSE("attention_maps: value size %d is above %d", vdim, 32 * MG_PER_LANE);
    if (dim > 2048) HB_REFUSE("attention_maps: key size %d is above 2048", dim);
    const long blocks = ((long)tokens * heads + MG_WARPS - 1) / MG_WARPS;
    const size_t smem = (size_t)MG_WARPS * dim * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
    if (window <= 0) keep = 0;
#define HB_RUN(T) attention_maps_kernel<T><<<(unsigned)blocks, MG_WARPS * 32, smem, s>>>((T*)out, (const T*)q, (const T*)kv, \
    block_table, table_stride, row_slot, query_start, kv_len, rows, tokens, heads, kv_heads, maps, dim, vdim, pages, page_size, \
    scale, cap, window, keep, lam, factor, eps, (const T*)gate, gate_ld)
    if (dtype == HB_F32) HB_RUN(float);
    else if (dtype == HB_BF16) HB_RUN(bf16);
    else HB_REFUSE("attention_maps: dtype %d", dtype);
#undef HB_RUN
    HB_LAUNCH_CHECK("attention_maps");
    return 0;
}

// ---------------------------------------------------------------- rows of one token, bfloat16, tensor cores
// A CTA owns (row, kv head, tile of its query heads, part of the keys) and walks 64-key tiles, 16 keys a warp. The M side of
// mma.sync m16n8k16 holds 16 / maps heads of the kv head's group for each map: the query of map m lies in the columns of that
// map's key and the rest of its row is zero, so one product over the whole key row [key 1 | key 2] scores every map, and the
// 16 rows share one sweep over the values. The parts' CTAs form a cluster; after a barrier each takes a share of the heads,
// merges the parts through distributed shared memory and does the heads' epilogue.
#define MD_PARTS 8                 // parts a row's keys are cut into at most
struct MapsArgs {
    bf16* out;
    const bf16* q;
    const bf16* kv;
    const int32_t* block_table;
    const int32_t* row_slot;
    const int32_t* query_start;
    const int32_t* kv_len;
    const bf16* gate;
    long gate_ld;
    int table_stride, heads, kv_heads, maps, dim, vdim, pages, page_size, page_shift, window, keep, splits;
    float scale, cap, lam, factor, eps;
};

template <int KP, int VP>
__device__ __forceinline__ void load_maps_tile(uint32_t k_s, uint32_t v_s, const MapsArgs& a, const int32_t* table, int hk, int tile,
                                               int lo, int n, int keep, int page_of_tile) {
    constexpr int KC = KP / 8, VC = VP / 8, CPR = KC + VC, STEP = 128 / CPR;
    const int ch = threadIdx.x % CPR, r0 = threadIdx.x / CPR;
    if (r0 >= STEP) return;
    const int kd = a.maps * a.dim, rowlen = kd + a.vdim;
    const bool is_k = ch < KC;
    const int c = is_k ? ch : ch - KC;
    const int have = is_k ? kd >> 3 : a.vdim >> 3, want = is_k ? (kd + 15) >> 4 << 1 : (a.vdim + 15) >> 4 << 1;
    if (c >= want) return;                                    // (columns no product reads)
    const int x = (is_k ? 0 : kd) + c * 8;
    const uint32_t base = is_k ? k_s : v_s;
    const int j0 = tile * TILE_N;
    if (a.page_shift >= 6) {                                  // the tile lies in one page: its rows follow one another
        const bool page_ok = page_of_tile >= 0 && page_of_tile < a.pages && c < have;
        const bool whole = j0 >= lo && j0 + TILE_N <= n;      // no key of the tile is outside the row's range
        const bf16* src = a.kv + (((long)(page_ok ? page_of_tile : 0) * a.kv_heads + hk) * a.page_size + (j0 & (a.page_size - 1))) * rowlen + (page_ok ? x : 0);
#pragma unroll
        for (int r = r0; r < TILE_N; r += STEP) {
            const int j = j0 + r;
            const bool ok = page_ok && (whole || (j < n && (j >= lo || j < keep)));
            cp_async16(base + (is_k ? tile_off<KP>(r, c) : tile_off<VP>(r, c)), src + (ok ? r * rowlen : 0), ok);
        }
        return;
    }
#pragma unroll 4
    for (int r = r0; r < TILE_N; r += STEP) {
        const int j = j0 + r;
        bool ok = j < n && (j >= lo || j < keep) && c < have;
        const bf16* src = a.kv;
        if (ok) {
            const int pi = a.page_shift >= 0 ? j >> a.page_shift : j / a.page_size, po = j - pi * a.page_size, page = table[pi];
            ok = page >= 0 && page < a.pages;
            if (ok) src = a.kv + (((long)page * a.kv_heads + hk) * a.page_size + po) * rowlen + x;
        }
        cp_async16(base + (is_k ? tile_off<KP>(r, c) : tile_off<VP>(r, c)), src, ok);
    }
}

template <int KP, int VP, int STAGES>
__global__ void __launch_bounds__(128, (KP + VP <= 256 ? 3 : 1)) maps_decode_kernel(const MapsArgs a) {
    extern __shared__ __align__(128) unsigned char smem_raw[];
    __shared__ float scratch[33];
    constexpr uint32_t K_BYTES = TILE_N * KP * 2, V_BYTES = TILE_N * VP * 2;
    const uint32_t q_s = smem_u32(smem_raw), k_s = q_s + 16 * KP * 2, v_s = k_s + STAGES * K_BYTES;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int b = blockIdx.x, split = blockIdx.z, splits = a.splits;
    const int group = a.heads / a.kv_heads, hpm = 16 / a.maps, m_tiles = (group + hpm - 1) / hpm;
    const int hk = blockIdx.y / m_tiles, g0 = (blockIdx.y % m_tiles) * hpm, g = min(hpm, group - g0);
    const int n = a.kv_len[b], t = a.query_start[b];
    const int lo = a.window > 0 ? max(0, n - a.window) : 0;          // the one query sits at position n - 1
    const int tile_lo = lo / TILE_N, tile_hi = (n + TILE_N - 1) / TILE_N;
    const int kt = min((a.keep + TILE_N - 1) / TILE_N, tile_lo);     // tiles of kept keys before the window's
    const int total = kt + tile_hi - tile_lo, per = (total + splits - 1) / splits;
    const int first = split * per, last = min(total, first + per);
    const int32_t* table = a.block_table + (size_t)a.row_slot[b] * a.table_stride;
    auto tile_at = [&](int i) -> int { return i < kt ? i : tile_lo + i - kt; };
    auto page_at = [&](int i) -> int { return a.page_shift >= 6 && i < last ? table[tile_at(i) >> (a.page_shift - 6)] : 0; };

    for (int i = threadIdx.x; i < 16 * (KP / 8); i += 128) {
        const int r = i / (KP / 8), ch = i % (KP / 8), m = r / hpm, x = r - m * hpm;
        const bool ok = x < g && ch * 8 >= m * a.dim && ch * 8 < (m + 1) * a.dim;
        const bf16* src = ok ? a.q + (((size_t)t * a.heads + (size_t)hk * group + g0 + x) * a.maps + m) * a.dim + ch * 8 - m * a.dim : a.q;
        cp_async16(q_s + tile_off<KP>(r, ch), src, ok);
    }
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) {
        if (first + s < last)
            load_maps_tile<KP, VP>(k_s + s * K_BYTES, v_s + s * V_BYTES, a, table, hk, tile_at(first + s), lo, n, a.keep, page_at(first + s));
        cp_async_commit();
    }
    int page_ahead = page_at(first + STAGES - 1);

    float o[VP / 8][4];
#pragma unroll
    for (int i = 0; i < VP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;        // rows lane / 4 and lane / 4 + 8, in log2 units
    const int ksteps = (a.maps * a.dim + 15) >> 4, vsteps = (a.vdim + 15) >> 4;
    const FragLanes fk = frag_lanes<KP>(lane), fv = frag_lanes<VP>(lane);
    constexpr bool Q_IN_REGS = KP <= 128;
    uint32_t qf[Q_IN_REGS ? KP / 16 : 1][4];
    bool q_loaded = false;
    for (int i = first; i < last; ++i) {
        const int stage = (i - first) % STAGES, tile = tile_at(i);
        cp_async_wait<STAGES - 2>();
        __syncthreads();
        if (i + STAGES - 1 < last) {
            const int s2 = (i - first + STAGES - 1) % STAGES;
            load_maps_tile<KP, VP>(k_s + s2 * K_BYTES, v_s + s2 * V_BYTES, a, table, hk, tile_at(i + STAGES - 1), lo, n, a.keep, page_ahead);
        }
        cp_async_commit();
        page_ahead = page_at(i + STAGES);
        if (Q_IN_REGS && !q_loaded) {
#pragma unroll
            for (int ks = 0; ks < KP / 16; ++ks)
                if (ks < ksteps) ldmatrix_x4(qf[Q_IN_REGS ? ks : 0], q_s + fk.a_row + ((ks * 32) ^ fk.a_xor));
            q_loaded = true;
        }
        const int key0 = tile * TILE_N + warp * 16;                  // this warp's 16 keys
        if (key0 >= n || (key0 + 16 <= lo && key0 >= a.keep)) continue;   // (uniform per warp; the barrier is above)
        const uint32_t kt_s = k_s + stage * K_BYTES + warp * 16 * (KP * 2) + fk.b_row;
        const uint32_t vt_s = v_s + stage * V_BYTES + warp * 16 * (VP * 2) + fv.t_row;
        float s[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < KP / 16; ++ks) {
            if (ks < ksteps) {
                uint32_t qa[4], kb[4];
                if (!Q_IN_REGS) ldmatrix_x4(qa, q_s + fk.a_row + ((ks * 32) ^ fk.a_xor));
                ldmatrix_x4(kb, kt_s + ((ks * 32) ^ fk.b_xor));
                mma_bf16(s[0], Q_IN_REGS ? qf[Q_IN_REGS ? ks : 0] : qa, kb[0], kb[1]);
                mma_bf16(s[1], Q_IN_REGS ? qf[Q_IN_REGS ? ks : 0] : qa, kb[2], kb[3]);
            }
        }
        if (a.cap > 0.f) {
            const float to_x = a.scale / a.cap, from_x = a.cap * LOG2E;
            float top = 0.f;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) { s[nt][e] *= to_x; top = fmaxf(top, fabsf(s[nt][e])); }
            const bool small = __all_sync(0xffffffffu, top <= 0.25f);
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float x = s[nt][e], y = x * x;              // (the polynomial's error is below 3e-7 of the value here)
                    s[nt][e] = from_x * (small ? x * fmaf(y, fmaf(y, fmaf(y, -17.f / 315.f, 2.f / 15.f), -1.f / 3.f), 1.f) : tanhf(x));
                }
        } else {
            const float f = a.scale * LOG2E;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nt][e] *= f;
        }
        if (!(key0 >= lo && key0 + 16 <= n)) {                       // only tiles at an edge need the mask
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int j = key0 + nt * 8 + (lane & 3) * 2 + (e & 1);
                    if (!(j < n && (j >= lo || j < a.keep))) s[nt][e] = -INFINITY;
                }
        }
        float c0, c1;
        softmax_step<2>(s, m0, m1, l0, l1, 1.f, c0, c1);
        uint32_t p[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
        if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
            for (int x = 0; x < VP / 8; ++x) { o[x][0] *= c0; o[x][1] *= c0; o[x][2] *= c1; o[x][3] *= c1; }
        }
#pragma unroll
        for (int dt = 0; dt < VP / 16; ++dt) {
            if (dt < vsteps) {
                uint32_t vb[4];
                ldmatrix_x4_trans(vb, vt_s + ((dt * 32) ^ fv.t_xor));
                mma_bf16(o[2 * dt], p, vb[0], vb[1]);
                mma_bf16(o[2 * dt + 1], p, vb[2], vb[3]);
            }
        }
    }
    cp_async_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    __syncthreads();                                                 // every warp is done with the tiles: reuse them

    // ---- the four warps' results, then their sum for this part: part_o [16][VP], part_ml [16][2] (maximum in log2 units, sum)
    float* wo = (float*)(smem_raw + 16 * KP * 2);                    // [4][16][VP]
    float* wml = wo + 4 * 16 * VP;                                   // [4][16][2]
    float* part_o = wml + 4 * 16 * 2;
    float* part_ml = part_o + 16 * VP;
    const int r0 = lane >> 2, cq = (lane & 3) * 2;
    const bool up = r0 % hpm < g, down = (r0 + 8) % hpm < g;         // rows that hold a head
#pragma unroll
    for (int i = 0; i < VP / 8; ++i) {
        if (i * 8 < a.vdim) {
            if (up) *(float2*)(wo + (warp * 16 + r0) * VP + i * 8 + cq) = make_float2(o[i][0], o[i][1]);
            if (down) *(float2*)(wo + (warp * 16 + r0 + 8) * VP + i * 8 + cq) = make_float2(o[i][2], o[i][3]);
        }
    }
    if ((lane & 3) == 0) {
        wml[(warp * 16 + r0) * 2] = m0; wml[(warp * 16 + r0) * 2 + 1] = l0;
        wml[(warp * 16 + r0 + 8) * 2] = m1; wml[(warp * 16 + r0 + 8) * 2 + 1] = l1;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < a.maps * g * VP; i += 128) {
        const int d = i % VP, x = i / VP, r = x < g ? x : hpm + x - g;   // (map, head) pairs in a row
        if (d >= a.vdim) continue;
        float mm = -INFINITY;
#pragma unroll
        for (int w = 0; w < 4; ++w) mm = fmaxf(mm, wml[(w * 16 + r) * 2]);
        float acc = 0.f, l = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float mw = wml[(w * 16 + r) * 2];
            const float fw = mw == -INFINITY ? 0.f : ex2(mw - mm);
            acc += fw * wo[(w * 16 + r) * VP + d];
            l += fw * wml[(w * 16 + r) * 2 + 1];
        }
        part_o[r * VP + d] = acc;
        if (d == 0) { part_ml[r * 2] = mm; part_ml[r * 2 + 1] = l; }
    }
    __syncthreads();
    __syncwarp();
    cluster_barrier();                                               // every part of the cluster lies in its shared memory
    // ---- a head at a time, a channel (VP 256: two) a thread: the parts in their order, all their loads in flight at once; then the
    // maps, the norm, the gate
    constexpr int PER = VP > 128 ? 2 : 1;
    const uint32_t po = smem_u32(part_o), pml = smem_u32(part_ml);
    for (int x = split; x < g; x += splits) {
        const int h = hk * group + g0 + x;
        float res[PER];
        for (int m = 0; m < a.maps; ++m) {
            const int r = m * hpm + x;
            float ms[MD_PARTS], ls[MD_PARTS], os[MD_PARTS][PER];
#pragma unroll
            for (int s2 = 0; s2 < MD_PARTS; ++s2) {
                ms[s2] = -INFINITY; ls[s2] = 0.f;
                if (s2 < splits) {
                    ms[s2] = ld_cluster_f32(pml + r * 8, s2);
                    ls[s2] = ld_cluster_f32(pml + r * 8 + 4, s2);
                }
#pragma unroll
                for (int i = 0; i < PER; ++i) {
                    os[s2][i] = 0.f;
                    if (s2 < splits && (int)threadIdx.x + 128 * i < a.vdim) os[s2][i] = ld_cluster_f32(po + (r * VP + threadIdx.x + 128 * i) * 4, s2);
                }
            }
            float mm = -INFINITY, l = 0.f, acc[PER];
#pragma unroll
            for (int i = 0; i < PER; ++i) acc[i] = 0.f;
#pragma unroll
            for (int s2 = 0; s2 < MD_PARTS; ++s2) mm = fmaxf(mm, ms[s2]);
#pragma unroll
            for (int s2 = 0; s2 < MD_PARTS; ++s2) {
                const float f = ms[s2] == -INFINITY ? 0.f : ex2(ms[s2] - mm);
                l += f * ls[s2];
#pragma unroll
                for (int i = 0; i < PER; ++i) acc[i] += f * os[s2][i];
            }
            const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
            for (int i = 0; i < PER; ++i) res[i] = m == 0 ? acc[i] * inv : res[i] - a.lam * (acc[i] * inv);
        }
        if (a.maps > 1) {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < PER; ++i) ss += res[i] * res[i];     // (channels past vdim hold zeros)
            const float f = rsqrtf(block_sum(ss, scratch) / (float)a.vdim + a.eps) * a.factor;
#pragma unroll
            for (int i = 0; i < PER; ++i) res[i] *= f;
        }
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = threadIdx.x + 128 * i;
            if (d < a.vdim) {
                const float y = a.gate ? res[i] * mp_sigmoid(to_f32(a.gate[(size_t)t * a.gate_ld + (size_t)h * a.vdim + d])) : res[i];
                a.out[((size_t)t * a.heads + h) * a.vdim + d] = __float2bfloat16_rn(y);
            }
        }
    }
    __syncwarp();
    cluster_barrier();                                               // nobody leaves while its shared memory may be read
}

template <int KP, int VP, int STAGES>
static int launch_maps_decode(const MapsArgs& a, int rows, cudaStream_t s) {
    auto kernel = maps_decode_kernel<KP, VP, STAGES>;
    const size_t tiles = 16 * KP * 2 + (size_t)STAGES * TILE_N * (KP + VP) * 2;
    const size_t merge = 16 * KP * 2 + (size_t)(4 * 16 * VP + 4 * 16 * 2 + 16 * VP + 16 * 2) * sizeof(float);
    const size_t smem = tiles > merge ? tiles : merge;
    HB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const int group = a.heads / a.kv_heads, hpm = 16 / a.maps;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(rows, a.kv_heads * ((group + hpm - 1) / hpm), a.splits);
    cfg.blockDim = dim3(128);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr = {};
    attr.id = cudaLaunchAttributeClusterDimension;
    attr.val.clusterDim.x = 1; attr.val.clusterDim.y = 1; attr.val.clusterDim.z = a.splits;
    cfg.attrs = &attr;
    cfg.numAttrs = 1;
    HB_CUDA(cudaLaunchKernelEx(&cfg, kernel, a));
    return 0;
}

extern "C" int hb_attention_maps_decode(void* out, const void* q, const void* kv, const int32_t* block_table, int table_stride,
                                        const int32_t* row_slot, const int32_t* query_start, const int32_t* kv_len, int rows,
                                        int heads, int kv_heads, int maps, int dim, int vdim, int pages, int page_size, float scale,
                                        float cap, int window, int keep, float lam, float factor, float eps, const void* gate,
                                        long gate_ld, int splits, hb_stream stream) {
    if (rows == 0) return 0;
    if (int rc = check_maps("attention_maps_decode", heads, kv_heads, maps, dim, vdim, scale, cap, window, keep)) return rc;
    const int kd = maps * dim;
    if (dim % 8 || vdim % 8 || kd > 256 || vdim > 256) HB_REFUSE("attention_maps_decode: %d maps of %d and values of %d: multiples of 8, rows up to 256", maps, dim, vdim);
    if (splits < 1 || splits > 8) HB_REFUSE("attention_maps_decode: %d parts (1 to 8, a cluster's size)", splits);
    if ((((uintptr_t)q | (uintptr_t)kv) & 15) != 0) HB_REFUSE("attention_maps_decode: q and the cache must lie on 16-byte boundaries");
    const MapsArgs a{(bf16*)out, (const bf16*)q, (const bf16*)kv, block_table, row_slot, query_start, kv_len, (const bf16*)gate, gate_ld,
                     table_stride, heads, kv_heads, maps, dim, vdim, pages, page_size, log2_exact(page_size), window,
                     window > 0 ? keep : 0, splits, scale, cap, lam, factor, eps};
    cudaStream_t s = (cudaStream_t)stream;
#define HB_V(K) do { if (vdim <= 64) return launch_maps_decode<K, 64, (K + 64 <= 192 ? 3 : 2)>(a, rows, s); \
                     if (vdim <= 128) return launch_maps_decode<K, 128, (K + 128 <= 192 ? 3 : 2)>(a, rows, s); \
                     return launch_maps_decode<K, 256, 2>(a, rows, s); } while (0)
    if (kd <= 64) HB_V(64);
    if (kd <= 128) HB_V(128);
    HB_V(256);
#undef HB_V
}
