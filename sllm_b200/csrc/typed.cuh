// Element access of kernels that are instantiated for bf16 and fp32 storage (arithmetic is fp32 in both).
#pragma once
#include "common.cuh"

namespace sllm {

__device__ __forceinline__ float ld_f(const float* p) { return *p; }
__device__ __forceinline__ float ld_f(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void st_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// N consecutive elements (N = 2 or 4), address aligned to N elements.
template <int N>
__device__ __forceinline__ void ld_vec(const float* p, float (&v)[N]) {
  if constexpr (N == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  } else {
    const float2 x = *reinterpret_cast<const float2*>(p);
    v[0] = x.x; v[1] = x.y;
  }
}
template <int N>
__device__ __forceinline__ void ld_vec(const __nv_bfloat16* p, float (&v)[N]) {
#pragma unroll
  for (int i = 0; i < N; i += 2) {
    const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(p + i);
    v[i] = __bfloat162float(h.x);
    v[i + 1] = __bfloat162float(h.y);
  }
}
template <int N>
__device__ __forceinline__ void st_vec(float* p, const float (&v)[N]) {
  if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
}
template <int N>
__device__ __forceinline__ void st_vec(__nv_bfloat16* p, const float (&v)[N]) {
  if constexpr (N == 4) {
    uint2 o;
    *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = o;
  } else {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
  }
}

// 16 bytes = VEC elements, address aligned to 16 bytes.
template <typename T>
constexpr int kVec16 = 16 / static_cast<int>(sizeof(T));
__device__ __forceinline__ void ld16(const float* p, float (&v)[4]) { ld_vec<4>(p, v); }
__device__ __forceinline__ void ld16(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    v[2 * j] = __bfloat162float(h[j].x);
    v[2 * j + 1] = __bfloat162float(h[j].y);
  }
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

}  // namespace sllm
