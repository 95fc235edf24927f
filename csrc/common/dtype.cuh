// Element-type helpers for kernels that are instantiated for bf16 and for fp32 activations / weights
// (the serving path runs a model either in bf16 with fp32 accumulation or entirely in fp32).
#pragma once
#include "util.cuh"

namespace llmctl {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// VEC (4 or 1) neighbouring numbers; VEC = 4 needs 4 * sizeof(T)-aligned addresses.
template <int VEC>
__device__ __forceinline__ void load_vec(const float* p, float (&v)[VEC]) {
  if (VEC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x, v[VEC > 1 ? 1 : 0] = f.y, v[VEC > 2 ? 2 : 0] = f.z, v[VEC > 3 ? 3 : 0] = f.w;
  } else {
    v[0] = p[0];
  }
}
template <int VEC>
__device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float (&v)[VEC]) {
  if (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(u.x << 16), v[VEC > 1 ? 1 : 0] = __uint_as_float(u.x & 0xffff0000u);
    v[VEC > 2 ? 2 : 0] = __uint_as_float(u.y << 16), v[VEC > 3 ? 3 : 0] = __uint_as_float(u.y & 0xffff0000u);
  } else {
    v[0] = __bfloat162float(p[0]);
  }
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* p, const float (&v)[VEC]) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[VEC > 1 ? 1 : 0], v[VEC > 2 ? 2 : 0], v[VEC > 3 ? 3 : 0]);
  else p[0] = v[0];
}
template <int VEC>
__device__ __forceinline__ void store_vec(__nv_bfloat16* p, const float (&v)[VEC]) {
  if (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[VEC > 1 ? 1 : 0]), pack_bf16x2(v[VEC > 2 ? 2 : 0], v[VEC > 3 ? 3 : 0]));
  else p[0] = __float2bfloat16(v[0]);
}

// Eight neighbouring numbers (16-byte aligned addresses).
__device__ __forceinline__ void load8_f32(const __nv_bfloat16* p, float (&v)[8]) { unpack8(load8(p), v); }
__device__ __forceinline__ void load8_f32(const float* p, float (&v)[8]) {
  *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
  *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(p + 4);
}
__device__ __forceinline__ void store8_f32(__nv_bfloat16* p, const float (&v)[8]) { store8(p, pack8(v)); }
__device__ __forceinline__ void store8_f32(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

}  // namespace llmctl

// Dispatch a templated launch on the `is_fp32` flag of the C ABI.
#define LLMCTL_DISPATCH_DTYPE(is_fp32, T, ...) \
  do {                                         \
    if (is_fp32) {                             \
      using T = float;                         \
      __VA_ARGS__;                             \
    } else {                                   \
      using T = __nv_bfloat16;                 \
      __VA_ARGS__;                             \
    }                                          \
  } while (0)
