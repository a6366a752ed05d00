// Vector loads and stores of VEC elements of T (bf16 or fp32), widened to fp32 registers, and block reductions.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <cstdint>

namespace omni {

template <typename T, int V>
struct alignas(sizeof(T) * V < 16 ? sizeof(T) * V : 16) VecOf {
  T v[V];
};

__device__ __forceinline__ float to_f32(float x) { return x; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T>
__device__ __forceinline__ T from_f32(float x);
template <>
__device__ __forceinline__ float from_f32<float>(float x) { return x; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float x) { return __float2bfloat16(x); }

template <int V, typename T>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[V]) {
  const VecOf<T, V> a = *reinterpret_cast<const VecOf<T, V>*>(p);
#pragma unroll
  for (int i = 0; i < V; ++i) f[i] = to_f32(a.v[i]);
}
template <int V, typename T>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[V]) {
  VecOf<T, V> a;
#pragma unroll
  for (int i = 0; i < V; ++i) a.v[i] = from_f32<T>(f[i]);
  *reinterpret_cast<VecOf<T, V>*>(p) = a;
}

__device__ __forceinline__ float warp_sum32(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum of two values over the block (at most 1024 threads); every thread gets both.
__device__ __forceinline__ float2 block_sum2(float a, float b) {
  __shared__ float2 part[32];
  a = warp_sum32(a);
  b = warp_sum32(b);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  float2 s = make_float2(0.f, 0.f);
  const int nw = (blockDim.x + 31) >> 5;
  for (int i = 0; i < nw; ++i) { s.x += part[i].x; s.y += part[i].y; }
  __syncthreads();
  return s;
}

// silu and the tanh form of gelu: exact exponentials and divisions for fp32 activations, the fast ones where the result is
// rounded to bf16 anyway
template <typename T>
__device__ __forceinline__ float exp_for(float x) { return expf(x); }
template <>
__device__ __forceinline__ float exp_for<__nv_bfloat16>(float x) { return __expf(x); }
template <typename T>
__device__ __forceinline__ float div_for(float a, float b) { return a / b; }
template <>
__device__ __forceinline__ float div_for<__nv_bfloat16>(float a, float b) { return __fdividef(a, b); }
template <typename T>
__device__ __forceinline__ float silu_for(float x) { return div_for<T>(x, 1.0f + exp_for<T>(-x)); }
template <typename T>
__device__ __forceinline__ float gelu_tanh_for(float x) {
  return div_for<T>(x, 1.0f + exp_for<T>(-1.5957691216057308f * (x + 0.044715f * x * x * x)));
}

}  // namespace omni
