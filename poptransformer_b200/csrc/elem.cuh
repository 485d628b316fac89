// Element access for kernels that serve fp32 and bf16 activations from one template.
#pragma once
#include <algorithm>

#include "common.cuh"

namespace pt {

static inline bool aligned_to(const void *q, int bytes) { return ((uintptr_t)q & (bytes - 1)) == 0; }

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T> __device__ __forceinline__ T from_f(float x);
template <> __device__ __forceinline__ float from_f<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

template <int VEC> __device__ __forceinline__ void load_vec(const float *p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 r = *reinterpret_cast<const float4 *>(p);
    v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = p[j];
  }
}
template <int VEC> __device__ __forceinline__ void load_vec(const __nv_bfloat16 *p, float (&v)[VEC]) {
  if constexpr (VEC == 8 || VEC == 4) {
    __nv_bfloat162 h[VEC / 2];
    if constexpr (VEC == 8) *reinterpret_cast<uint4 *>(h) = *reinterpret_cast<const uint4 *>(p);
    else *reinterpret_cast<uint2 *>(h) = *reinterpret_cast<const uint2 *>(p);
#pragma unroll
    for (int j = 0; j < VEC / 2; ++j) { v[2 * j] = __low2float(h[j]); v[2 * j + 1] = __high2float(h[j]); }
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = to_f(p[j]);
  }
}
// VEC consecutive values (the address is aligned to VEC elements).
template <int VEC> __device__ __forceinline__ void store_vec(float *p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else if constexpr (VEC == 2) *reinterpret_cast<float2 *>(p) = make_float2(v[0], v[1]);
  else *p = v[0];
}
template <int VEC> __device__ __forceinline__ void store_vec(__nv_bfloat16 *p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    __nv_bfloat162 a[2] = {__floats2bfloat162_rn(v[0], v[1]), __floats2bfloat162_rn(v[2], v[3])};
    *reinterpret_cast<uint2 *>(p) = *reinterpret_cast<const uint2 *>(a);
  } else if constexpr (VEC == 2) {
    *reinterpret_cast<__nv_bfloat162 *>(p) = __floats2bfloat162_rn(v[0], v[1]);
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
// log(1 + exp(x)) without overflow: for x > 0 it is x + log1p(exp(-x)).
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// A bf16 pair as the 32-bit register of a tensor-core fragment, and the pair of what the rounding left over: a value split as
// hi + lo keeps 16 significant bits through two bf16 products (for operands that must not be rounded to 8 bits: softmax weights,
// decay factors, recurrent state).
__device__ __forceinline__ uint32_t pack_bf2(float lo, float hi) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t *>(&h);
}
__device__ __forceinline__ void split_bf2(float a, float b, uint32_t &hi, uint32_t &lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t *>(&h);
  lo = pack_bf2(a - __low2float(h), b - __high2float(h));
}

}  // namespace pt
