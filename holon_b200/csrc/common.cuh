// Shared helpers of the kernels: storage types, conversions, warp and block reductions, launch checks.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "api.h"

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float x) { return x; }
__device__ __forceinline__ float to_f32(bf16 x) { return __bfloat162float(x); }
template <typename T> __device__ __forceinline__ T from_f32(float x);
template <> __device__ __forceinline__ float from_f32<float>(float x) { return x; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float x) { return __float2bfloat16_rn(x); }
// The value after one rounding to the storage type, as 32-bit.
template <typename T> __device__ __forceinline__ float rounded(float x) { return to_f32(from_f32<T>(x)); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result. `scratch` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();                       // scratch may still be read from an earlier call
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float w = lane < warps ? scratch[lane] : 0.f;
        w = warp_sum(w);
        if (lane == 0) scratch[32] = w;
    }
    __syncthreads();
    return scratch[32];
}
// Two sums at once (`scratch` holds 66 floats): x and y become the block's sums.
__device__ __forceinline__ void block_sum2(float& x, float& y, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
    x = warp_sum(x);
    y = warp_sum(y);
    __syncthreads();
    if (lane == 0) { scratch[warp] = x; scratch[33 + warp] = y; }
    __syncthreads();
    x = warp_sum(lane < warps ? scratch[lane] : 0.f);             // (every warp adds the warps' sums up in the same order)
    y = warp_sum(lane < warps ? scratch[33 + lane] : 0.f);
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float w = lane < warps ? scratch[lane] : -INFINITY;
        w = warp_max(w);
        if (lane == 0) scratch[32] = w;
    }
    __syncthreads();
    return scratch[32];
}

// Four neighbouring values to and from 32-bit (the address on a 16-byte boundary for float, 8 for bfloat16).
template <typename T> struct Vec4;
template <> struct Vec4<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) { const float4 x = *(const float4*)p; v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *(float4*)p = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Vec4<bf16> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[4]) {
        const uint2 x = *(const uint2*)p;
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&x.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&x.y);
        v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[4]) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 x; x.x = *(uint32_t*)&a; x.y = *(uint32_t*)&b;
        *(uint2*)p = x;
    }
};

// Host side: remembers why a call was refused; hb_last_error() hands the text out.
void hb_set_error(const char* fmt, ...);
#define HB_REFUSE(...) do { hb_set_error(__VA_ARGS__); return HB_ERR_REFUSED; } while (0)
#define HB_LAUNCH_CHECK(name) do { cudaError_t e_ = cudaGetLastError(); if (e_ != cudaSuccess) { \
    hb_set_error("%s: %s", name, cudaGetErrorString(e_)); return HB_ERR_CUDA; } } while (0)
#define HB_CUDA(call) do { cudaError_t e_ = (call); if (e_ != cudaSuccess) { \
    hb_set_error("%s: %s", #call, cudaGetErrorString(e_)); return HB_ERR_CUDA; } } while (0)
