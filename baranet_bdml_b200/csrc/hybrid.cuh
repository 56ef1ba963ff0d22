// Element access and activations shared by the kernels that exist in fp32 and in bf16.
#pragma once

#include "common.cuh"
#include "ptx.cuh"

namespace bn {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
template <typename T> __device__ __forceinline__ float round_to(float v) { return to_f(from_f<T>(v)); }

__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    v[0] = ptx::bf16_lo(u.x); v[1] = ptx::bf16_hi(u.x); v[2] = ptx::bf16_lo(u.y); v[3] = ptx::bf16_hi(u.y);
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(ptx::pack_bf16(v[0], v[1]), ptx::pack_bf16(v[2], v[3]));
}

__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh_exact(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
}
// softplus(z) = log(1 + e^z) without overflow
__device__ __forceinline__ float softplus_exact(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float relu2(float z) { const float t = fmaxf(z, 0.f); return t * t; }
__device__ __forceinline__ float sigmoid_exact(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

// act: BN_ACT_NONE, BN_ACT_SILU, BN_ACT_GELU_TANH, BN_ACT_RELU2
__device__ __forceinline__ float activation_exact(int act, float z) {
    return act == BN_ACT_SILU ? silu_exact(z) : act == BN_ACT_GELU_TANH ? gelu_tanh_exact(z) : act == BN_ACT_RELU2 ? relu2(z) : z;
}
// The epilogues of the bf16 products: the result is rounded to bf16, so the fast exponential suffices.
// gelu_tanh(z) = z * sigmoid(2 u) with u = sqrt(2/pi) (z + 0.044715 z^3), because (1 + tanh u) / 2 = 1 / (1 + e^(-2u)).
__device__ __forceinline__ float activation_fast(int act, float z) {
    if (act == BN_ACT_NONE) return z;
    if (act == BN_ACT_RELU2) return relu2(z);
    const float t = act == BN_ACT_GELU_TANH ? 1.5957691216057308f * fmaf(0.044715f * z * z, z, z) : z;
    return __fdividef(z, 1.f + __expf(-t));
}

// sum over a block of THREADS threads, the same bits in every thread; sh holds THREADS / 32 floats
template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* sh) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();                      // sh may still be read from the sum before
    if (threadIdx.x % 32 == 0) sh[threadIdx.x / 32] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) t += sh[w];
    return t;
}

// cos and sin of position * frequency.  The product and its reduction to one turn are taken in fp64, so that the angle
// is as good far along a sequence as at its start; the functions themselves run in fp32.
__device__ __forceinline__ void rotation(int position, double freq, float* c, float* s) {
    const double turns = (double)position * freq * 0.15915494309189535;
    const float a = (float)((turns - rint(turns)) * 6.283185307179586);
    sincosf(a, s, c);
}

}  // namespace bn
