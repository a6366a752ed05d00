// What may happen to an attention score between q k^T and the softmax, and which keys a query sees.
#pragma once
#include <cuda_runtime.h>

namespace omni {

// score = cap tanh(raw scale / cap) - slope distance - r1 ln(1 + r2 distance) (each part optional), in units of log 2
struct ScoreMod {
  float scale_log2;        // scale * log2(e)
  float cap_in;            // 2 log2(e) scale / cap
  float cap_log2;          // cap * log2(e); 0 = no cap
  const float* slopes;     // [heads] or null
  const float *r1, *r2;    // [heads] or null
};

inline ScoreMod make_score_mod(float scale, float cap, const float* slopes, const float* r1 = nullptr, const float* r2 = nullptr) {
  constexpr float kLog2e = 1.4426950408889634f;
  return {scale * kLog2e, cap > 0.f ? 2.f * kLog2e * scale / cap : 0.f, cap > 0.f ? cap * kLog2e : 0.f, slopes, r1, r2};
}

__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lg2_fast(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// r1 ln(1 + r2 distance) in units of log 2; absolute error of some 1e-7, which r1 multiplies
__device__ __forceinline__ float log_bias(float r1, float r2, float distance) { return r1 * lg2_fast(fmaf(r2, distance, 1.f)); }
__device__ __forceinline__ float rcp_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// tanh(z) = 1 - 2 / (1 + e^2z): absolute error of some 1e-7, which the cap multiplies.  `add` comes on top.
__device__ __forceinline__ float capped(const ScoreMod& m, float raw, float add) {
  return fmaf(-2.f * m.cap_log2, rcp_fast(1.f + ex2_fast(raw * m.cap_in)), m.cap_log2 + add);
}
__device__ __forceinline__ float cap_score(const ScoreMod& m, float raw) {
  return m.cap_log2 > 0.f ? capped(m, raw, 0.f) : raw * m.scale_log2;
}

// two fp32 values in one register pair
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack_f32x2(float a, float b) {
  f32x2 v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(a), "f"(b));
  return v;
}
__device__ __forceinline__ void unpack_f32x2(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 fma_f32x2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 v;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(v) : "l"(a), "l"(b), "l"(c));
  return v;
}
__device__ __forceinline__ f32x2 add_f32x2(f32x2 a, f32x2 b) {
  f32x2 v;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(v) : "l"(a), "l"(b));
  return v;
}

// First key that a query at `pos` sees through its window (of `window` keys) and in its chunk (of `chunk` positions); 0 = none.
// Kept first keys come on top.
__host__ __device__ __forceinline__ int first_key(int pos, int window, int chunk) {
  int lo = window > 0 ? pos - window + 1 : 0;
  if (chunk > 0 && pos >= 0) {
    const int c = pos / chunk * chunk;
    lo = c > lo ? c : lo;
  }
  return lo > 0 ? lo : 0;
}

}  // namespace omni
