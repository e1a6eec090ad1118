// Element types and scalar functions shared by the decoder's kernels.  Template parameter E is the element type of
// activations, weights and cached rows: __nv_bfloat16 or float; all arithmetic is fp32.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

namespace tmb {

template<typename E> __device__ __forceinline__ float to_f32(E x);
template<> __device__ __forceinline__ float to_f32<float>(float x) { return x; }
template<> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 x) { return __bfloat162float(x); }
template<typename E> __device__ __forceinline__ E from_f32(float x);
template<> __device__ __forceinline__ float from_f32<float>(float x) { return x; }
template<> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

__device__ __forceinline__ float bf16_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi)
{
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.f / (1.f + expf(-z)); }

// 0.5 z (1 + tanh(u)) with u = sqrt(2/pi) (z + 0.044715 z^3), written as z * sigmoid(2u)
template<bool FAST> __device__ __forceinline__ float gelu_tanh_f32(float z)
{
    const float u2 = 1.5957691216057308f * (z + 0.044715f * z * z * z);
    return FAST ? __fdividef(z, 1.f + __expf(-u2)) : z / (1.f + expf(-u2));
}

// g = min(gate, limit), u = clamp(up, -limit, limit): g * sigmoid(slope * g) * (u + 1)
template<bool FAST> __device__ __forceinline__ float clamped_swish_f32(float gate, float up, float limit, float slope)
{
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit) + 1.f;
    return (FAST ? __fdividef(g, 1.f + __expf(-slope * g)) : g / (1.f + expf(-slope * g))) * u;
}

__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int m = 16; m >= 1; m >>= 1) v += __shfl_xor_sync(0xffffffffu, v, m);
    return v;
}

}  // namespace tmb
