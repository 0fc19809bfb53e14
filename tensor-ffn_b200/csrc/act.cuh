// Activation storage: the row kernels are instantiated for bf16 and for fp32 activations and compute in fp32 either way.
#pragma once
#include "kernels.h"

namespace tffn {

__device__ __forceinline__ float act_load(const float* p) { return __ldcg(p); }
__device__ __forceinline__ float act_load(const bf16* p) {
    return __uint_as_float((uint32_t)__ldcg((const unsigned short*)p) << 16);
}
__device__ __forceinline__ void act_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void act_store(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

// sum over the block (blockDim a multiple of 32, at most 1024); `red` holds 32 floats; every thread gets the result
__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    const int warps = blockDim.x >> 5;
    __syncthreads();  // an earlier use of red is over
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
    for (int w = 0; w < warps; ++w) s += red[w];
    return s;
}

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

}  // namespace tffn
