// What the mma.sync attention kernels share: asynchronous copies, ldmatrix and mma wrappers, swizzled tiles of 64 keys, the
// online-softmax step, and a cluster's barrier and distributed shared memory.
#pragma once
#include "common.cuh"

#define TILE_N 64

// ---------------------------------------------------------------- small PTX wrappers
__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;                  // src-size 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(n));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *(uint32_t*)&v;
}
__device__ __forceinline__ float ex2(float x) {   // 2^x; -inf gives 0
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}

// Shared-memory tiles hold rows of D_PAD bf16 = D_PAD/8 chunks of 16 bytes; the chunk index is XOR-ed with the low
// three bits of the row so that ldmatrix's 8 rows fall into 8 different bank groups. Byte offset of (row, chunk):
template <int D_PAD> __device__ __forceinline__ uint32_t tile_off(int row, int chunk) {
    return (uint32_t)(row * (D_PAD * 2) + ((chunk ^ (row & 7)) << 4));
}

// Per-lane parts of the ldmatrix addresses, worked out once. A fragment of k-step (or d-step) `step` in a block of 16
// rows that starts at a multiple of 8 lies at  base + rows * (D_PAD * 2) + lane_row + ((step * 32) ^ lane_xor).
struct FragLanes {
    uint32_t a_row, a_xor;         // 16 x 16 A operand (queries): rows lane & 15, k-half lane >> 4
    uint32_t b_row, b_xor;         // two 8-wide B operands from [n][k] memory (keys): rows (lane & 7) + 8 (lane >> 4)
    uint32_t t_row, t_xor;         // two 8-wide B operands from [k][n] memory through .trans (values)
};
template <int D_PAD> __device__ __forceinline__ FragLanes frag_lanes(int lane) {
    const uint32_t x = lane & 7, rb = D_PAD * 2;
    FragLanes f;
    f.a_row = (lane & 15) * rb;                          f.a_xor = ((uint32_t)(lane >> 4) ^ x) << 4;
    f.b_row = ((lane & 7) + ((lane >> 4) << 3)) * rb;    f.b_xor = ((uint32_t)((lane >> 3) & 1) ^ x) << 4;
    f.t_row = ((lane & 7) + (((lane >> 3) & 1) << 3)) * rb;  f.t_xor = ((uint32_t)(lane >> 4) ^ x) << 4;
    return f;
}

// Loads `rows` query rows of one head (row stride heads * head_dim elements) into a tile; the rest become zeros.
template <int D_PAD, int ROWS, int THREADS>
__device__ __forceinline__ void load_q_tile(uint32_t q_s, const bf16* q, long row_stride, int rows, int head_dim) {
    for (int i = threadIdx.x; i < ROWS * (D_PAD / 8); i += THREADS) {
        const int r = i / (D_PAD / 8), ch = i % (D_PAD / 8);
        const bool valid = r < rows && ch < (head_dim >> 3);
        cp_async16(q_s + tile_off<D_PAD>(r, ch), q + (valid ? (long)r * row_stride + ch * 8 : 0), valid);
    }
}

// One online-softmax update of a lane's two rows over NT 8-key blocks of raw scores `s` (masked ones are -inf):
// turns s into weights 2^((s - max) * scale), updates the running maxima and sums, returns the factors by which what
// was summed before must be scaled.
template <int NT>
__device__ __forceinline__ void softmax_step(float (&s)[NT][4], float& m0, float& m1, float& l0, float& l1,
                                             float scale_log2, float& c0, float& c1) {
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
        mx0 = fmaxf(mx0, fmaxf(s[nt][0], s[nt][1]));
        mx1 = fmaxf(mx1, fmaxf(s[nt][2], s[nt][3]));
    }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1)); mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);
    const float nb0 = n0 == -INFINITY ? 0.f : -n0 * scale_log2;    // a row with nothing yet: 2^(-inf) = 0 below
    const float nb1 = n1 == -INFINITY ? 0.f : -n1 * scale_log2;
    c0 = ex2(fmaf(m0, scale_log2, nb0));
    c1 = ex2(fmaf(m1, scale_log2, nb1));
    m0 = n0; m1 = n1;
    float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
        s[nt][0] = ex2(fmaf(s[nt][0], scale_log2, nb0)); s[nt][1] = ex2(fmaf(s[nt][1], scale_log2, nb0));
        s[nt][2] = ex2(fmaf(s[nt][2], scale_log2, nb1)); s[nt][3] = ex2(fmaf(s[nt][3], scale_log2, nb1));
        sum0 += s[nt][0] + s[nt][1]; sum1 += s[nt][2] + s[nt][3];
    }
    l0 = l0 * c0 + sum0; l1 = l1 * c1 + sum1;                       // per-lane partial sums; quads are joined at the end
}

__device__ __forceinline__ float ld_cluster_f32(uint32_t local_addr, uint32_t rank) {
    uint32_t remote;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(remote) : "r"(local_addr), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];\n" : "=f"(v) : "r"(remote) : "memory");
    return v;
}
__device__ __forceinline__ void cluster_barrier() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
}

static inline int log2_exact(int x) {                // log2 of a power of two, else -1
    int s = 0;
    while ((1 << s) < x) ++s;
    return (1 << s) == x ? s : -1;
}
