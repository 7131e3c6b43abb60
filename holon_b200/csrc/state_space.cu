// The state-space recurrence for rows of several tokens, in chunks of 64 (the form of Dao and Gu, Transformers are SSMs: Generalized
// Models and Efficient Algorithms Through Structured State Space Duality), everything in 32-bit on CUDA cores:
//     S_t = g_t S_(t-1) + dt_t B_t x_t^T,  y_t = S_t^T C_t + skip x_t,  g_t = exp(-exp(rate_log) dt_t)
// With L_i the sum of the logarithms of g over a chunk's tokens up to i (kept as a pair of float32 whose sum is exact to double
// precision: what the weights need are differences of such sums), a chunk with the state S_in before it gives
//     y_i = sum_(j <= i) (C_i . B_j) exp(L_i - L_j) dt_j x_j + exp(L_i) S_in^T C_i + skip x_i
//     S_out = exp(L_last) S_in + sum_j exp(L_last - L_j) dt_j B_j x_j^T.
// Four kernels: the chunks' products C_i . B_j, per group; the chunks' own contributions to the state, per head; the walk over a
// row's chunks, an element of the state a thread, which leaves every chunk's S_in behind and writes the row's state back; the
// chunks' outputs, per head. Only the third is sequential, one multiply-add a chunk. Blocks find their (row, chunk) in the step's
// rows; launches may have more tiles than the step has chunks. One-token rows: csrc/recurrent.cu.
#include <type_traits>

#include "common.cuh"

#define SS_Q 64                          // tokens a chunk
#define SS_T 64                          // rows and columns of an output tile
#define SS_K 32                          // depth of a staged slice
#define SS_THREADS 128                   // a thread: 8 rows x 4 columns of a tile

struct Chunk { int row, t0, n, first_tile; };              // the batch row, first token, tokens, the row's first tile

// Tile number -> chunk (row -1: there is none). Rows row0 .. rows - 1 in order, each ceil(tokens / 64) tiles.
__device__ __forceinline__ Chunk find_chunk(const int32_t* __restrict__ query_start, int row0, int rows, int tile) {
    int left = tile;
    for (int b = row0; b < rows; ++b) {
        const int n = query_start[b + 1] - query_start[b], tiles = (n + SS_Q - 1) / SS_Q;
        if (left < tiles) return {b, query_start[b] + left * SS_Q, min(SS_Q, n - left * SS_Q), tile - left};
        left -= tiles;
    }
    return {-1, 0, 0, 0};
}

// A slice of an operand in shared memory: element (k, i) in the group of four floats at(k, i / 4). The groups of a row of k are
// permuted by k / 4, so that stores of four k's of one i by eight neighbouring lanes, and of four i's by four, hit different banks.
__device__ __forceinline__ int group_at(int k, int g) { return k * (SS_T / 4) + (g ^ ((k >> 2) & 7)); }

// acc += a^T b over a slice.
__device__ __forceinline__ void tile_step(float (&acc)[8][4], const float* a, const float* b, int depth) {
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const float4* a4 = (const float4*)a;
    const float4* b4 = (const float4*)b;
#pragma unroll 8
    for (int k = 0; k < depth; ++k) {
        const float4 r0 = a4[group_at(k, ty * 2)], r1 = a4[group_at(k, ty * 2 + 1)], c = b4[group_at(k, tx)];
        const float r[8] = {r0.x, r0.y, r0.z, r0.w, r1.x, r1.y, r1.z, r1.w};
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            acc[i][0] = fmaf(r[i], c.x, acc[i][0]); acc[i][1] = fmaf(r[i], c.y, acc[i][1]);
            acc[i][2] = fmaf(r[i], c.z, acc[i][2]); acc[i][3] = fmaf(r[i], c.w, acc[i][3]);
        }
    }
}

// Slices travel through registers (the next one is on its way while the current one is multiplied), 16 bytes a load: four quads a
// thread and operand. `along`: the operand's memory runs along k (element (row i, k) at p[i * stride + k]); eight neighbouring lanes
// load 128 bytes of one row. `across`: it runs along the tile's rows (element (k, i) at p[k * stride + i]).
struct Quads { float4 v[4]; };
__device__ __forceinline__ float4 load_quad(const float* p, int left, bool vec) {        // zeros from `left` on
    if (vec && left >= 4) return *(const float4*)p;
    return make_float4(left > 0 ? p[0] : 0.f, left > 1 ? p[1] : 0.f, left > 2 ? p[2] : 0.f, left > 3 ? p[3] : 0.f);
}
__device__ __forceinline__ void fetch_along(Quads& q, const float* p, size_t stride, int rows, int depth, bool vec) {
    const int i = threadIdx.x >> 3, k = (threadIdx.x & 7) * 4;
#pragma unroll
    for (int r = 0; r < 4; ++r) q.v[r] = load_quad(p + (i + 16 * r) * stride + k, i + 16 * r < rows ? depth - k : 0, vec);
}
__device__ __forceinline__ void store_along(float* a, const Quads& q) {
    const int k = (threadIdx.x & 7) * 4;
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const int i = (threadIdx.x >> 3) + 16 * r, g = i >> 2, e = i & 3;      // (k .. k + 3 share their permutation)
        a[group_at(k, g) * 4 + e] = q.v[r].x; a[group_at(k + 1, g) * 4 + e] = q.v[r].y;
        a[group_at(k + 2, g) * 4 + e] = q.v[r].z; a[group_at(k + 3, g) * 4 + e] = q.v[r].w;
    }
}
__device__ __forceinline__ void fetch_across(Quads& q, const float* p, size_t stride, int rows, int depth, bool vec) {
    const int i = (threadIdx.x & 15) * 4, k = threadIdx.x >> 4;
#pragma unroll
    for (int r = 0; r < 4; ++r) q.v[r] = load_quad(p + (k + 8 * r) * stride + i, k + 8 * r < depth ? rows - i : 0, vec);
}
__device__ __forceinline__ void store_across(float* a, const Quads& q) {
    const int k = threadIdx.x >> 4;
#pragma unroll
    for (int r = 0; r < 4; ++r) ((float4*)a)[group_at(k + 8 * r, threadIdx.x & 15)] = q.v[r];
}
__device__ __forceinline__ void scale_quad(float4& v, float f) { v.x *= f; v.y *= f; v.z *= f; v.w *= f; }

// L_i of a chunk's tokens for one head, by warp 0: hi + lo in two floats; tokens past the chunk repeat the last.
__device__ __forceinline__ void log_decays(float* hi, float* lo, float* steps, const float* __restrict__ dt, const Chunk& c, int heads,
                                           int h, float rate) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        const float d0 = 2 * lane < c.n ? dt[(size_t)(c.t0 + 2 * lane) * heads + h] : 0.f;
        const float d1 = 2 * lane + 1 < c.n ? dt[(size_t)(c.t0 + 2 * lane + 1) * heads + h] : 0.f;
        const double a0 = -(double)rate * d0, a1 = -(double)rate * d1;
        double s = a0 + a1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += up;
        }
        const double l0 = s - a1;
        steps[2 * lane] = d0; steps[2 * lane + 1] = d1;
        hi[2 * lane] = (float)l0; lo[2 * lane] = (float)(l0 - (double)(float)l0);
        hi[2 * lane + 1] = (float)s; lo[2 * lane + 1] = (float)(s - (double)(float)s);
    }
}

// ---- products[tile][group][i][j] = C_i . B_j, [64][64] each. grid (tiles, groups)
__global__ void __launch_bounds__(SS_THREADS, 4) ss_products_kernel(float* __restrict__ products, const float* __restrict__ cb,
                                                                 const int32_t* __restrict__ query_start, int row0, int rows, int groups, int n) {
    __shared__ __align__(16) float a[SS_K * SS_T], b[SS_K * SS_T];
    const Chunk c = find_chunk(query_start, row0, rows, blockIdx.x);
    if (c.row < 0) return;
    const int g = blockIdx.y;
    float acc[8][4] = {};
    Quads qa, qb;
    const float* src = cb + ((size_t)c.t0 * 2 * groups + g) * n;
    const size_t stride = (size_t)2 * groups * n;
    const bool vec = (n & 3) == 0;
    fetch_along(qa, src, stride, c.n, n, vec);
    fetch_along(qb, src + (size_t)groups * n, stride, c.n, n, vec);
    for (int k0 = 0; k0 < n; k0 += SS_K) {
        store_along(a, qa);
        store_along(b, qb);
        __syncthreads();
        if (k0 + SS_K < n) {
            fetch_along(qa, src + k0 + SS_K, stride, c.n, n - k0 - SS_K, vec);
            fetch_along(qb, src + (size_t)groups * n + k0 + SS_K, stride, c.n, n - k0 - SS_K, vec);
        }
        tile_step(acc, a, b, min(SS_K, n - k0));
        __syncthreads();
    }
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float* out = products + ((size_t)blockIdx.x * groups + g) * SS_Q * SS_Q;
#pragma unroll
    for (int i = 0; i < 8; ++i) *(float4*)(out + (ty * 8 + i) * SS_Q + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
}

// ---- own[tile][head][p][n] = sum_j exp(L_last - L_j) dt_j x_j[p] B_j[n]; last[tile][head] = exp(L_last). grid (tiles, heads, tiles of
// p times tiles of n)
__global__ void __launch_bounds__(SS_THREADS, 4) ss_own_kernel(float* __restrict__ own, float* __restrict__ last, const float* __restrict__ cb,
                                                            const float* __restrict__ x, const float* __restrict__ dt,
                                                            const float* __restrict__ rate_log, const int32_t* __restrict__ query_start,
                                                            int row0, int rows, int heads, int groups, int n, int vdim, int n_tiles) {
    __shared__ __align__(16) float a[SS_K * SS_T], b[SS_K * SS_T];
    __shared__ float hi[SS_Q], lo[SS_Q], steps[SS_Q], w[SS_Q];
    const Chunk c = find_chunk(query_start, row0, rows, blockIdx.x);
    if (c.row < 0) return;
    const int h = blockIdx.y, g = h / (heads / groups);
    const int p0 = ((int)blockIdx.z / n_tiles) * SS_T, n0 = ((int)blockIdx.z % n_tiles) * SS_T;
    Quads qa, qb;
    const size_t xs = (size_t)heads * vdim, bs = (size_t)2 * groups * n;
    const float* xp = x + ((size_t)c.t0 * heads + h) * vdim + p0;
    const float* bp = cb + (((size_t)c.t0 * 2 + 1) * groups + g) * n + n0;
    const bool vx = (vdim & 3) == 0, vb = (n & 3) == 0;
    fetch_across(qa, xp, xs, vdim - p0, c.n, vx);                   // (on its way while the decays are added up)
    fetch_across(qb, bp, bs, n - n0, c.n, vb);
    log_decays(hi, lo, steps, dt, c, heads, h, expf(rate_log[h]));
    __syncthreads();
    if (threadIdx.x < SS_Q) {
        const int j = threadIdx.x;
        w[j] = expf((hi[SS_Q - 1] - hi[j]) + (lo[SS_Q - 1] - lo[j])) * steps[j];
        if (j == 0 && blockIdx.z == 0) last[(size_t)blockIdx.x * heads + h] = expf(hi[SS_Q - 1] + lo[SS_Q - 1]);
    }
    __syncthreads();
    float acc[8][4] = {};
    for (int k0 = 0; k0 < c.n; k0 += SS_K) {
#pragma unroll
        for (int r = 0; r < 4; ++r) scale_quad(qa.v[r], w[min(k0 + ((int)threadIdx.x >> 4) + 8 * r, SS_Q - 1)]);
        store_across(a, qa);
        store_across(b, qb);
        __syncthreads();
        if (k0 + SS_K < c.n) {
            fetch_across(qa, xp + (k0 + SS_K) * xs, xs, vdim - p0, c.n - k0 - SS_K, vx);
            fetch_across(qb, bp + (k0 + SS_K) * bs, bs, n - n0, c.n - k0 - SS_K, vb);
        }
        tile_step(acc, a, b, min(SS_K, c.n - k0));
        __syncthreads();
    }
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float* out = own + ((size_t)blockIdx.x * heads + h) * vdim * n;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int p = p0 + ty * 8 + i, col = n0 + tx * 4;
        if (p >= vdim) break;
        if ((n & 3) == 0 && col + 3 < n) *(float4*)(out + (size_t)p * n + col) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        else
#pragma unroll
            for (int k = 0; k < 4; ++k) if (col + k < n) out[(size_t)p * n + col + k] = acc[i][k];
    }
}

// ---- a row's chunks in order: own[tile] <- the state before the chunk, state <- the state behind the last. grid (rows - row0, heads,
// slices of the state), an element (V: four) a thread.
template <bool V>
__global__ void ss_walk_kernel(float* __restrict__ own, const float* __restrict__ last, float* __restrict__ state,
                               const int32_t* __restrict__ query_start, const int32_t* __restrict__ row_slot, int row0, int heads, int size) {
    typedef typename std::conditional<V, float4, float>::type E;
    const int b = row0 + (int)blockIdx.x, h = blockIdx.y, e = blockIdx.z * blockDim.x + threadIdx.x;
    int first = 0;
    for (int r = row0; r < b; ++r) first += (query_start[r + 1] - query_start[r] + SS_Q - 1) / SS_Q;
    const int tiles = (query_start[b + 1] - query_start[b] + SS_Q - 1) / SS_Q;
    if (e >= (V ? size >> 2 : size) || tiles == 0) return;
    E* st = (E*)(state + ((size_t)row_slot[b] * heads + h) * size) + e;
    const size_t stride = (size_t)heads * size / (V ? 4 : 1);
    E* p = (E*)(own + ((size_t)first * heads + h) * size) + e;
    const float* f = last + (size_t)first * heads + h;
    E s = *st;
    auto step = [&](float d, const E& v) {
        if constexpr (V) { s.x = fmaf(d, s.x, v.x); s.y = fmaf(d, s.y, v.y); s.z = fmaf(d, s.z, v.z); s.w = fmaf(d, s.w, v.w); }
        else s = fmaf(d, s, v);
    };
    int i = 0;
    for (; i + 8 <= tiles; i += 8, p += 8 * stride, f += 8 * (size_t)heads) {        // (eight chunks' loads fly together)
        E v[8];
        float d[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) { v[k] = p[k * stride]; d[k] = f[k * (size_t)heads]; }
#pragma unroll
        for (int k = 0; k < 8; ++k) { p[k * stride] = s; step(d[k], v[k]); }
    }
    for (; i < tiles; ++i, p += stride, f += heads) {
        const E v = p[0];
        p[0] = s;
        step(f[0], v);
    }
    *st = s;
}

// ---- y_i[p] of a chunk: the products' part over its own tokens, the state's part over n, the skip. grid (tiles, heads, tiles of p)
__global__ void __launch_bounds__(SS_THREADS, 4) ss_out_kernel(float* __restrict__ y, const float* __restrict__ products,
                                                            const float* __restrict__ before, const float* __restrict__ cb,
                                                            const float* __restrict__ x, const float* __restrict__ dt,
                                                            const float* __restrict__ rate_log, const float* __restrict__ skip,
                                                            const int32_t* __restrict__ query_start, int row0, int rows, int heads,
                                                            int groups, int n, int vdim) {
    __shared__ __align__(16) float a[SS_K * SS_T], b[SS_K * SS_T];
    __shared__ float hi[SS_Q], lo[SS_Q], steps[SS_Q], w[SS_Q];
    const Chunk c = find_chunk(query_start, row0, rows, blockIdx.x);
    if (c.row < 0) return;
    const int h = blockIdx.y, g = h / (heads / groups), p0 = (int)blockIdx.z * SS_T;
    const float* cbp = products + ((size_t)blockIdx.x * groups + g) * SS_Q * SS_Q;
    const float* xp = x + ((size_t)c.t0 * heads + h) * vdim + p0;
    const float* cp = cb + ((size_t)c.t0 * 2 * groups + g) * n;
    const float* sp = before + (((size_t)blockIdx.x * heads + h) * vdim + p0) * n;
    const size_t xs = (size_t)heads * vdim, cs = (size_t)2 * groups * n;
    const bool vx = (vdim & 3) == 0, vn = (n & 3) == 0;
    const int own_slices = (c.n + SS_K - 1) / SS_K, slices = own_slices + (n + SS_K - 1) / SS_K;
    Quads qa, qb;
    auto fetch = [&](int s) {
        if (s < own_slices) {                                       // over the chunk's tokens j
            const int k0 = s * SS_K;
            fetch_along(qa, cbp + k0, SS_Q, SS_Q, SS_K, true);
            fetch_across(qb, xp + k0 * xs, xs, vdim - p0, c.n - k0, vx);
        } else {                                                    // over the state's channels
            const int k0 = (s - own_slices) * SS_K;
            fetch_along(qa, cp + k0, cs, c.n, n - k0, vn);
            fetch_along(qb, sp + k0, n, vdim - p0, n - k0, vn);
        }
    };
    fetch(0);                                                       // (on its way while the decays are added up)
    log_decays(hi, lo, steps, dt, c, heads, h, expf(rate_log[h]));
    __syncthreads();
    if (threadIdx.x < SS_Q) w[threadIdx.x] = expf(hi[threadIdx.x] + lo[threadIdx.x]);
    __syncthreads();
    float acc[8][4] = {};
    for (int s = 0; s < slices; ++s) {
        if (s < own_slices) {                                       // weight of token j in row i: C_i . B_j exp(L_i - L_j) dt_j, j <= i
            const int j = s * SS_K + ((int)threadIdx.x & 7) * 4;
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                const int row = ((int)threadIdx.x >> 3) + 16 * r;
                const float hr = hi[row], lr = lo[row];
                auto weight = [&](int jj, float v) -> float { return jj <= row && jj < c.n ? v * expf((hr - hi[jj]) + (lr - lo[jj])) * steps[jj] : 0.f; };
                qa.v[r].x = weight(j, qa.v[r].x); qa.v[r].y = weight(j + 1, qa.v[r].y);
                qa.v[r].z = weight(j + 2, qa.v[r].z); qa.v[r].w = weight(j + 3, qa.v[r].w);
            }
        } else {
#pragma unroll
            for (int r = 0; r < 4; ++r) scale_quad(qa.v[r], w[((int)threadIdx.x >> 3) + 16 * r]);
        }
        store_along(a, qa);
        if (s < own_slices) store_across(b, qb); else store_along(b, qb);
        __syncthreads();
        if (s + 1 < slices) fetch(s + 1);
        // (the second half of a chunk's tokens weighs nothing in its first half's rows)
        if (s >= own_slices || s == 0 || (int)(threadIdx.x >> 5) * 16 + 15 >= s * SS_K) tile_step(acc, a, b, SS_K);
        __syncthreads();
    }
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const float d = skip[h];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int r = ty * 8 + i;
        if (r >= c.n) break;
        const size_t at = ((size_t)(c.t0 + r) * heads + h) * vdim + p0 + tx * 4;
#pragma unroll
        for (int k = 0; k < 4; ++k) if (p0 + tx * 4 + k < vdim) y[at + k] = fmaf(d, x[at + k], acc[i][k]);
    }
}

extern "C" size_t hb_state_space_prompt_scratch_floats(int tiles, int heads, int groups, int n, int vdim) {
    return (size_t)tiles * ((size_t)heads * vdim * n + (size_t)groups * SS_Q * SS_Q + heads);
}

extern "C" int hb_state_space_prompt(float* y, const float* cb, const float* x, const float* dt, const float* rate_log, const float* skip,
                                     float* state, float* scratch, const int32_t* query_start, const int32_t* row_slot, int row0,
                                     int rows, int tiles, int heads, int groups, int n, int vdim, hb_stream stream) {
    if (rows <= row0 || tiles == 0) return 0;
    if (groups < 1 || heads % groups || n < 1 || vdim < 1) HB_REFUSE("state_space_prompt: %d heads of %d, %d groups of %d", heads, vdim, groups, n);
    if (!scratch || ((uintptr_t)scratch & 15) || ((uintptr_t)state & 15)) HB_REFUSE("state_space_prompt: scratch and state must lie on 16-byte boundaries");
    const int p_tiles = (vdim + SS_T - 1) / SS_T, n_tiles = (n + SS_T - 1) / SS_T;
    if (heads > 65535 || (long)p_tiles * n_tiles > 65535) HB_REFUSE("state_space_prompt: %d heads of %d x %d", heads, vdim, n);
    const int size = vdim * n;
    float* products = scratch;                                     // [tiles][groups][64][64]
    float* own = products + (size_t)tiles * groups * SS_Q * SS_Q;  // [tiles][heads][vdim][n]
    float* last = own + (size_t)tiles * heads * size;              // [tiles][heads]
    cudaStream_t s = (cudaStream_t)stream;
    ss_products_kernel<<<dim3(tiles, groups), SS_THREADS, 0, s>>>(products, cb, query_start, row0, rows, groups, n);
    HB_LAUNCH_CHECK("state_space_products");
    ss_own_kernel<<<dim3(tiles, heads, p_tiles * n_tiles), SS_THREADS, 0, s>>>(own, last, cb, x, dt, rate_log, query_start, row0, rows, heads,
                                                                               groups, n, vdim, n_tiles);
    HB_LAUNCH_CHECK("state_space_own");
    const bool vec = size % 4 == 0;
    const int elements = vec ? size / 4 : size, slices = (elements + 127) / 128;
    if (slices > 65535) HB_REFUSE("state_space_prompt: states of %d numbers", size);
    if (vec) ss_walk_kernel<true><<<dim3(rows - row0, heads, slices), 128, 0, s>>>(own, last, state, query_start, row_slot, row0, heads, size);
    else ss_walk_kernel<false><<<dim3(rows - row0, heads, slices), 128, 0, s>>>(own, last, state, query_start, row_slot, row0, heads, size);
    HB_LAUNCH_CHECK("state_space_walk");
    ss_out_kernel<<<dim3(tiles, heads, p_tiles), SS_THREADS, 0, s>>>(y, products, own, cb, x, dt, rate_log, skip, query_start, row0, rows, heads,
                                                                     groups, n, vdim);
    HB_LAUNCH_CHECK("state_space_out");
    return 0;
}
