// A norm on a sublayer's output, added to the stream: dst = src + N(y), N(z) = z * rsqrt(mean(z^2) + eps) * (weight + offset), and
// the same for a pair of outputs that are put together first: with R(y) = y / sqrt(mean(y^2) + pair_eps),
//     z = scale (R(a) * a_weight + R(b) * b_weight),   dst = src + N(z).
// `cast` (or null) gets dst's rows in the storage type, for the next sublayer's products. One block a row, the row in registers
// between the sums over the block; 32-bit arithmetic, z is never rounded. (csrc/elementwise.cu: hb_out_norm_add, the form with a
// bias and the average over depth, sends rows that need neither here.)
#include "common.cuh"

// NV > 0: a thread holds NV groups of four neighbouring numbers (dim a multiple of 4 and at most 4 NV blockDim, pointers on 16-byte
// boundaries). NV == 0: any dim, the row in shared memory.
template <typename T, typename TW, int NV, bool PAIR>
__global__ void out_norm_rows_kernel(float* dst, const float* src, const T* __restrict__ a, const T* __restrict__ b,
                                     const TW* __restrict__ a_weight, const TW* __restrict__ b_weight, float pair_eps, float scale,
                                     const void* __restrict__ weight, int weight_f32, float eps, float offset, T* cast, int dim) {
    extern __shared__ float on_rows[];
    __shared__ float scratch[66];
    const size_t at = (size_t)blockIdx.x * dim;
    auto w1 = [&](int d) -> float { return (weight_f32 ? ((const float*)weight)[d] : to_f32(((const bf16*)weight)[d])) + offset; };
    if constexpr (NV > 0) {
        float z[NV][4], y[PAIR ? NV : 1][4], x[NV][4];
        float sa = 0.f, sb = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * blockDim.x + threadIdx.x) * 4;
            z[n][0] = z[n][1] = z[n][2] = z[n][3] = 0.f;
            if (PAIR) y[PAIR ? n : 0][0] = y[PAIR ? n : 0][1] = y[PAIR ? n : 0][2] = y[PAIR ? n : 0][3] = 0.f;
            if (i < dim) {
                Vec4<T>::load(a + at + i, z[n]);
                if (PAIR) Vec4<T>::load(b + at + i, y[PAIR ? n : 0]);
                Vec4<float>::load(src + at + i, x[n]);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    sa = fmaf(z[n][e], z[n][e], sa);
                    if (PAIR) sb = fmaf(y[PAIR ? n : 0][e], y[PAIR ? n : 0][e], sb);
                }
            }
        }
        if (PAIR) {
            block_sum2(sa, sb, scratch);
            const float fa = rsqrtf(sa / (float)dim + pair_eps) * scale, fb = rsqrtf(sb / (float)dim + pair_eps) * scale;
            sa = 0.f;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int i = (n * blockDim.x + threadIdx.x) * 4;
                if (i < dim) {
                    float wa[4], wb[4];
                    Vec4<TW>::load(a_weight + i, wa);
                    Vec4<TW>::load(b_weight + i, wb);
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        z[n][e] = z[n][e] * fa * wa[e] + y[PAIR ? n : 0][e] * fb * wb[e];
                        sa = fmaf(z[n][e], z[n][e], sa);
                    }
                }
            }
        }
        const float f = rsqrtf(block_sum(sa, scratch) / (float)dim + eps);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * blockDim.x + threadIdx.x) * 4;
            if (i < dim) {
                float w[4];
                if (weight_f32) Vec4<float>::load((const float*)weight + i, w);
                else Vec4<bf16>::load((const bf16*)weight + i, w);
#pragma unroll
                for (int e = 0; e < 4; ++e) x[n][e] = fmaf(z[n][e] * f, w[e] + offset, x[n][e]);
                Vec4<float>::store(dst + at + i, x[n]);
                if (cast) Vec4<T>::store(cast + at + i, x[n]);
            }
        }
    } else {
        float sa = 0.f, sb = 0.f;
        for (int d = threadIdx.x; d < dim; d += blockDim.x) {
            const float z = to_f32(a[at + d]), y = PAIR ? to_f32(b[at + d]) : 0.f;
            sa = fmaf(z, z, sa);
            sb = fmaf(y, y, sb);
            on_rows[d] = z;
        }
        if (PAIR) {
            block_sum2(sa, sb, scratch);
            const float fa = rsqrtf(sa / (float)dim + pair_eps) * scale, fb = rsqrtf(sb / (float)dim + pair_eps) * scale;
            sa = 0.f;
            for (int d = threadIdx.x; d < dim; d += blockDim.x) {
                const float z = on_rows[d] * fa * to_f32(a_weight[d]) + to_f32(b[at + d]) * fb * to_f32(b_weight[d]);
                sa = fmaf(z, z, sa);
                on_rows[d] = z;
            }
        }
        const float f = rsqrtf(block_sum(sa, scratch) / (float)dim + eps);
        for (int d = threadIdx.x; d < dim; d += blockDim.x) {
            const float x = fmaf(on_rows[d] * f, w1(d), src[at + d]);
            dst[at + d] = x;
            if (cast) cast[at + d] = from_f32<T>(x);
        }
    }
}

template <typename T, typename TW, bool PAIR>
static int launch_out_norm(float* dst, const float* src, const void* a, const void* b, const void* a_weight, const void* b_weight,
                           float pair_eps, float scale, const void* weight, int weight_f32, float eps, float offset, void* cast,
                           int rows, int dim, cudaStream_t s) {
    const bool vec = dim % 4 == 0 && (((uintptr_t)dst | (uintptr_t)src | (uintptr_t)a | (uintptr_t)b | (uintptr_t)a_weight |
                                       (uintptr_t)b_weight | (uintptr_t)weight | (uintptr_t)cast) & 15) == 0;
#define HB_RUN(NV, THREADS, SMEM) out_norm_rows_kernel<T, TW, NV, PAIR><<<rows, THREADS, SMEM, s>>>(dst, src, (const T*)a, (const T*)b, \
        (const TW*)a_weight, (const TW*)b_weight, pair_eps, scale, weight, weight_f32, eps, offset, (T*)cast, dim)
    if (vec && dim <= 512) HB_RUN(1, 128, 0);
    else if (vec && dim <= 1024) HB_RUN(1, 256, 0);
    else if (vec && dim <= 2048) HB_RUN(2, 256, 0);
    else if (vec && dim <= 4096) HB_RUN(4, 256, 0);
    else if (vec && dim <= 8192) HB_RUN(4, 512, 0);
    else {
        const size_t smem = (size_t)dim * sizeof(float);
        if (smem > 200 * 1024) HB_REFUSE("out_norm: rows of %d numbers", dim);
        if (smem > 46 * 1024) HB_CUDA(cudaFuncSetAttribute(out_norm_rows_kernel<T, TW, 0, PAIR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        HB_RUN(0, dim >= 1024 ? 256 : 128, smem);
    }
#undef HB_RUN
    HB_LAUNCH_CHECK("out_norm");
    return 0;
}

// dst = src + N(y) with `cast` of y's type.
extern "C" int hb_out_norm_rows(float* dst, const float* src, const void* y, int dtype, const void* weight, int weight_dtype,
                                float eps, float offset, void* cast, int rows, int dim, hb_stream stream) {
    if (rows == 0) return 0;
    if (dim < 1 || !weight) HB_REFUSE("out_norm_rows: rows of %d numbers and a weight", dim);
    const int wf = weight_dtype == HB_F32;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == HB_F32) return launch_out_norm<float, float, false>(dst, src, y, nullptr, nullptr, nullptr, 0.f, 1.f, weight, wf, eps, offset, cast, rows, dim, s);
    if (dtype == HB_BF16) return launch_out_norm<bf16, bf16, false>(dst, src, y, nullptr, nullptr, nullptr, 0.f, 1.f, weight, wf, eps, offset, cast, rows, dim, s);
    HB_REFUSE("out_norm_rows: dtype %d", dtype);
}

extern "C" int hb_out_norm_pair_add(float* dst, const float* src, const void* a, const void* b, int dtype, const void* a_weight,
                                    const void* b_weight, int pair_weight_dtype, float pair_eps, float scale, const void* weight,
                                    int weight_dtype, float eps, float offset, void* cast, int rows, int dim, hb_stream stream) {
    if (rows == 0) return 0;
    if (dim < 1 || !a || !b || !a_weight || !b_weight || !weight) HB_REFUSE("out_norm_pair_add: two rows of %d numbers and their weights", dim);
    const int wf = weight_dtype == HB_F32;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == HB_F32 && pair_weight_dtype == HB_F32) return launch_out_norm<float, float, true>(dst, src, a, b, a_weight, b_weight, pair_eps, scale, weight, wf, eps, offset, cast, rows, dim, s);
    if (dtype == HB_BF16 && pair_weight_dtype == HB_BF16) return launch_out_norm<bf16, bf16, true>(dst, src, a, b, a_weight, b_weight, pair_eps, scale, weight, wf, eps, offset, cast, rows, dim, s);
    if (dtype == HB_BF16 && pair_weight_dtype == HB_F32) return launch_out_norm<bf16, float, true>(dst, src, a, b, a_weight, b_weight, pair_eps, scale, weight, wf, eps, offset, cast, rows, dim, s);
    HB_REFUSE("out_norm_pair_add: dtype %d with weight dtype %d", dtype, pair_weight_dtype);
}
