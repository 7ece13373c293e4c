// Row access of the layer stacks' kernels, whose operands are bf16 or (all-fp32 mode) float: eight elements at a time, values as fp32.
#pragma once
#include "common.cuh"

template <typename T> __device__ __forceinline__ void load8(const T* p, float* v);
template <> __device__ __forceinline__ void load8<bf16>(const bf16* p, float* v) {
  const uint4 q = *(const uint4*)p;
  const bf162* h = (const bf162*)&q;
#pragma unroll
  for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); v[2 * j] = f.x; v[2 * j + 1] = f.y; }
}
template <> __device__ __forceinline__ void load8<float>(const float* p, float* v) {
  const float4 a = *(const float4*)p, b = *(const float4*)(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float* v);
template <> __device__ __forceinline__ void store8<bf16>(bf16* p, const float* v) {
  uint32_t w[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) { const bf162 h = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]); w[j] = *(const uint32_t*)&h; }
  *(uint4*)p = make_uint4(w[0], w[1], w[2], w[3]);
}
template <> __device__ __forceinline__ void store8<float>(float* p, const float* v) {
  *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
  *(float4*)(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <typename T> __device__ __forceinline__ T to_t(float v);
template <> __device__ __forceinline__ bf16 to_t<bf16>(float v) { return __float2bfloat16(v); }
template <> __device__ __forceinline__ float to_t<float>(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
// Four elements at a time: rows whose threads hold several of them.
template <typename T> __device__ __forceinline__ void load4(const T* p, float* v);
template <> __device__ __forceinline__ void load4<bf16>(const bf16* p, float* v) {
  const uint2 q = *(const uint2*)p;
  const float2 a = __bfloat1622float2(*(const bf162*)&q.x), b = __bfloat1622float2(*(const bf162*)&q.y);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <> __device__ __forceinline__ void load4<float>(const float* p, float* v) {
  const float4 a = *(const float4*)p;
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float* v);
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, const float* v) {
  const bf162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *(uint2*)p = make_uint2(*(const uint32_t*)&a, *(const uint32_t*)&b);
}
template <> __device__ __forceinline__ void store4<float>(float* p, const float* v) { *(float4*)p = make_float4(v[0], v[1], v[2], v[3]); }
