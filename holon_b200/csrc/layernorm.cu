// Layer norm with a weight and no bias, out = (v - mean v) / sqrt(mean((v - mean v)^2) + eps) * weight, over rows of the
// residual stream to which a pending output is added first, times a factor:
//     v = h[row] + scale * delta[row]                          (one row of a sublayer's output)
//     v = h[row] + scale * sum_k delta[place[row, k]]          (the rows that `top` experts left for the token)
// The sum goes back to h unless rows are gathered by `index`. One block a row; mean and squared deviations are two sums
// over the block, the row waiting in registers (or, for sizes that do not fit them, in shared memory) between them. 32-bit
// arithmetic, one rounding where the output is stored.
#include "common.cuh"

#define LN_PLACES 64                   // places of a token kept in shared memory

// NV > 0: a thread holds NV groups of four neighbouring values (dim a multiple of 4 and at most 4 NV blockDim, pointers on
// 16-byte boundaries). NV == 0: any dim, the row in shared memory.
template <typename TH, typename TD, typename TW, int NV, bool PAIRS>
__global__ void add_layernorm_kernel(TD* __restrict__ out, TH* __restrict__ h, const TD* __restrict__ delta, float scale,
                                     const int32_t* __restrict__ place, int top, const TW* __restrict__ weight, float eps,
                                     const int32_t* __restrict__ index, int dim) {
    extern __shared__ __align__(16) float ln_row[];
    __shared__ float scratch[33];
    __shared__ int places[LN_PLACES];
    const size_t r = blockIdx.x, t = index ? (size_t)index[r] : r;
    TH* hr = h + t * dim;
    const bool write_back = delta != nullptr && index == nullptr;
    if (PAIRS) {
        for (int k = threadIdx.x; k < min(top, LN_PLACES); k += blockDim.x) places[k] = place[t * top + k];
        __syncthreads();
    }
    auto place_of = [&](int k) -> int { return k < LN_PLACES ? places[k] : place[t * top + k]; };
    if constexpr (NV > 0) {
        float v[NV][4], w[NV][4];
        float sum = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * blockDim.x + threadIdx.x) * 4;
            v[n][0] = v[n][1] = v[n][2] = v[n][3] = 0.f;
            if (i < dim) {
                Vec4<TH>::load(hr + i, v[n]);
                Vec4<TW>::load(weight + i, w[n]);
                if (delta) {
                    float d[4];
                    if (PAIRS) {
                        float a[4] = {0.f, 0.f, 0.f, 0.f};
                        for (int k = 0; k < top; ++k) {
                            const int p = place_of(k);
                            if (p < 0) continue;
                            Vec4<TD>::load(delta + (size_t)p * dim + i, d);
#pragma unroll
                            for (int e = 0; e < 4; ++e) a[e] += d[e];
                        }
#pragma unroll
                        for (int e = 0; e < 4; ++e) d[e] = a[e];
                    } else {
                        Vec4<TD>::load(delta + t * dim + i, d);
                    }
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[n][e] = fmaf(scale, d[e], v[n][e]);
                    if (write_back) Vec4<TH>::store(hr + i, v[n]);
                }
                sum += (v[n][0] + v[n][1]) + (v[n][2] + v[n][3]);
            }
        }
        const float mean = block_sum(sum, scratch) / (float)dim;
        float ss = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            if ((int)(n * blockDim.x + threadIdx.x) * 4 < dim) {
#pragma unroll
                for (int e = 0; e < 4; ++e) { v[n][e] -= mean; ss = fmaf(v[n][e], v[n][e], ss); }
            }
        }
        const float f = rsqrtf(block_sum(ss, scratch) / (float)dim + eps);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * blockDim.x + threadIdx.x) * 4;
            if (i < dim) {
#pragma unroll
                for (int e = 0; e < 4; ++e) v[n][e] = v[n][e] * f * w[n][e];
                Vec4<TD>::store(out + r * dim + i, v[n]);
            }
        }
    } else {
        float sum = 0.f;
        for (int i = threadIdx.x; i < dim; i += blockDim.x) {
            float v = to_f32(hr[i]);
            if (delta) {
                float d = 0.f;
                if (PAIRS) {
                    for (int k = 0; k < top; ++k) {
                        const int p = place_of(k);
                        if (p >= 0) d += to_f32(delta[(size_t)p * dim + i]);
                    }
                } else {
                    d = to_f32(delta[t * dim + i]);
                }
                v = fmaf(scale, d, v);
                if (write_back) hr[i] = from_f32<TH>(v);
            }
            ln_row[i] = v;
            sum += v;
        }
        const float mean = block_sum(sum, scratch) / (float)dim;
        float ss = 0.f;
        for (int i = threadIdx.x; i < dim; i += blockDim.x) { const float v = ln_row[i] - mean; ss = fmaf(v, v, ss); }
        const float f = rsqrtf(block_sum(ss, scratch) / (float)dim + eps);
        for (int i = threadIdx.x; i < dim; i += blockDim.x)
            out[r * dim + i] = from_f32<TD>((ln_row[i] - mean) * f * to_f32(weight[i]));
    }
}

template <typename TH, typename TD, typename TW>
static int launch_add_layernorm(void* out, void* h, const void* delta, float scale, const int32_t* place, int top,
                                const void* weight, float eps, const int32_t* index, int rows, int dim, cudaStream_t s) {
    const bool vec = dim % 4 == 0 && (((uintptr_t)out | (uintptr_t)h | (uintptr_t)delta | (uintptr_t)weight) & 15) == 0;
    const int quads = dim / 4;
    int nv = 0, threads = dim >= 1024 ? 512 : 256;
    size_t smem = (size_t)dim * sizeof(float);
    if (vec && quads <= 2048) {
        // few rows (latency counts): a group a thread where a block has that many threads; many rows: blocks of up to 512
        const int wide = rows <= 256 ? 1024 : quads > 512 ? 512 : 256;
        nv = quads <= wide ? 1 : quads <= 2 * wide ? 2 : quads <= 4 * wide ? 4 : 8;
        threads = ((quads + nv - 1) / nv + 31) / 32 * 32;
        smem = 0;
    }
    if (smem > 200 * 1024) HB_REFUSE("add_layernorm: a row of %d values does not fit shared memory (limit 51200)", dim);
#define LN_GO(NV_, P_) do { \
        auto kernel = add_layernorm_kernel<TH, TD, TW, NV_, P_>; \
        if (smem > 46 * 1024) HB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        kernel<<<rows, threads, smem, s>>>((TD*)out, (TH*)h, (const TD*)delta, scale, place, top, (const TW*)weight, eps, index, dim); \
    } while (0)
#define LN_NV(P_) do { if (nv == 0) LN_GO(0, P_); else if (nv == 1) LN_GO(1, P_); else if (nv == 2) LN_GO(2, P_); \
                       else if (nv == 4) LN_GO(4, P_); else LN_GO(8, P_); } while (0)
    if (place) LN_NV(true); else LN_NV(false);
#undef LN_NV
#undef LN_GO
    HB_LAUNCH_CHECK("add_layernorm");
    return 0;
}

extern "C" int hb_add_layernorm(void* out, int out_dtype, void* h, int h_dtype, const void* delta, float scale,
                                const int32_t* place, int top, const void* weight, int weight_dtype, float eps,
                                const int32_t* index, int rows, int dim, hb_stream stream) {
    if (rows == 0 || dim == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (h_dtype != HB_F32 && delta) HB_REFUSE("add_layernorm: the residual stream must be float32 when something is added");
    if (place && (!delta || top < 1)) HB_REFUSE("add_layernorm: places without the rows they name");
#define HB_CASE(H, D, W, TH, TD, TW) if (h_dtype == H && out_dtype == D && weight_dtype == W) \
    return launch_add_layernorm<TH, TD, TW>(out, h, delta, scale, place, top, weight, eps, index, rows, dim, s);
    HB_CASE(HB_F32, HB_F32, HB_F32, float, float, float)
    HB_CASE(HB_F32, HB_BF16, HB_BF16, float, bf16, bf16)
    HB_CASE(HB_F32, HB_BF16, HB_F32, float, bf16, float)
    HB_CASE(HB_BF16, HB_BF16, HB_BF16, bf16, bf16, bf16)
    HB_CASE(HB_BF16, HB_BF16, HB_F32, bf16, bf16, float)
#undef HB_CASE
    HB_REFUSE("add_layernorm: no kernel for dtypes h=%d out=%d weight=%d", h_dtype, out_dtype, weight_dtype);
}
