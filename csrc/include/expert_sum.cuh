// Columns c .. c + V of a token's expert mixture: the chosen experts' rows (already weighted; rows < 0 are none) and the shared
// expert's row (may be null) added up in fp32.
#pragma once
#include "omni_vec.cuh"

namespace omni {

template <typename T, int V>
__device__ __forceinline__ void expert_sum(const T* y, int y_ld, const int* rows, int top_k, const T* shared, int t, int c,
                                           float (&out)[V]) {
#pragma unroll
  for (int i = 0; i < V; ++i) out[i] = 0.f;
  for (int k = 0; k < top_k; ++k) {
    if (rows[k] < 0) continue;
    float v[V];
    load_vec<V>(y + (size_t)rows[k] * y_ld + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) out[i] += v[i];
  }
  if (shared != nullptr) {
    float v[V];
    load_vec<V>(shared + (size_t)t * y_ld + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) out[i] += v[i];
  }
}

}  // namespace omni
