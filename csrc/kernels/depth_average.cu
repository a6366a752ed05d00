// Row kernels of models with norms on both sides of the sublayers, one fp32 residual, learned positions, and a learned average
// over depth after every layer:
//   omni_embed_positions   x = embedding row + position row, and the normed input of the first sublayer
//   omni_both_norms_step   x' = x + mult rmsnorm(sublayer output) w_out; at the end of a layer x' is also what the layer gave, X_n,
//                          and the residual becomes sum_j average[j] X_j over the embedding output X_0 and all layers' results so
//                          far; then the normed input of the next sublayer
// The sublayer's output is a tensor, or the parts of an expert mixture.  Activations are bf16 or fp32 (`f32`); the residual, the
// results [layers + 1, T, ld], all weights and sums are fp32.  Columns past the width are written as zeros where they may be an
// operand of the next GEMM.
#include "../include/expert_sum.cuh"
#include "../include/omni_vec.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

struct EmbedParams {
  const int64_t* ids;
  const void* table;         // [rows, table_ld]
  int rows, table_ld;
  const int64_t* positions;
  const void* pos_table;     // [pos_rows, pos_ld] or null
  int pos_rows, pos_ld;
  float* x;                  // [T, ld]
  int H, ld;
  const float* w;
  float eps;
  void* h;                   // [T, h_ld]
  int h_ld;
};

// KEEP vectors per thread stay in registers between the two passes; what is beyond them is read again.
template <typename T, int V, int KEEP>
__global__ void embed_positions_kernel(const EmbedParams p) {
  const int t = blockIdx.x;
  const int64_t id = p.ids[t], pos = p.pos_table != nullptr ? p.positions[t] : 0;
  const bool known = id >= 0 && id < p.rows, placed = p.pos_table != nullptr && pos >= 0 && pos < p.pos_rows;
  float* xr = p.x + (size_t)t * p.ld;
  float keep[KEEP][V], ss = 0.f;
  const int step = blockDim.x * V;
  auto gather = [&](int c, float (&a)[V]) {
#pragma unroll
    for (int i = 0; i < V; ++i) a[i] = 0.f;
    if (known) load_vec<V>((const T*)p.table + (size_t)id * p.table_ld + c, a);
    if (placed) {
      float b[V];
      load_vec<V>((const T*)p.pos_table + (size_t)pos * p.pos_ld + c, b);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] += b[i];
    }
    store_vec<V>(xr + c, a);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += a[i] * a[i];
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < p.H) gather(c, keep[k]);
  }
  for (int c = threadIdx.x * V + KEEP * step; c < p.H; c += step) {
    float a[V];
    gather(c, a);
  }
  const float r = 1.0f / sqrtf(block_sum2(ss, 0.f).x / (float)p.H + p.eps);
  T* hr = (T*)p.h + (size_t)t * p.h_ld;
  auto finish = [&](int c, float (&a)[V]) {
    float g[V];
    load_vec<V>(p.w + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) a[i] = a[i] * r * g[i];
    store_vec<V>(hr + c, a);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < p.H) finish(c, keep[k]);
  }
  for (int c = threadIdx.x * V + KEEP * step; c < p.H; c += step) {
    float a[V];
    load_vec<V>(xr + c, a);
    finish(c, a);
  }
  for (int c = p.H + threadIdx.x; c < p.h_ld; c += blockDim.x) hr[c] = from_f32<T>(0.f);
}

struct StepParams {
  const float* x_in;     // [T, ld]
  float* x_out;          // [T, ld], may be x_in
  const void* y;         // sublayer output rows of pitch y_ld; expert mixtures: the sorted expert rows
  int y_ld;
  const int* row_of;     // expert mixtures: [T, top_k] row of y, or -1; null: y has one row per token
  int top_k;
  const void* shared;    // expert mixtures: [T, y_ld] or null
  const float* w_out;    // [H]
  float mult;
  float* results;        // [n (+ 1), T, ld]; null: no average
  const float* average;  // [n + 1]
  int n, store;          // store: there is room for results[n]
  const float* w;        // [H]
  float eps;
  void* h;               // [T, h_ld]
  int H, ld, h_ld;
};

template <typename T, int V, int KEEP, bool AVG>
__global__ void both_norms_step_kernel(const StepParams p, int T_rows) {
  const int t = blockIdx.x;
  __shared__ int rows[32];
  if (p.row_of != nullptr) {
    if (threadIdx.x < p.top_k) rows[threadIdx.x] = p.row_of[(size_t)t * p.top_k + threadIdx.x];
    __syncthreads();
  }
  const size_t row = (size_t)t * p.ld, layer = (size_t)T_rows * p.ld;
  const int step = blockDim.x * V;
  auto sublayer = [&](int c, float (&y)[V]) {
    if (p.row_of != nullptr) expert_sum<T, V>((const T*)p.y, p.y_ld, rows, p.top_k, (const T*)p.shared, t, c, y);
    else load_vec<V>((const T*)p.y + (size_t)t * p.y_ld + c, y);
  };
  // what does not wait for the norm: x, or (with an average) x apart from the part of the earlier results
  float yk[KEEP][V], xk[KEEP][V], past[AVG ? KEEP : 1][V], ss = 0.f;
  auto earlier = [&](int c, float (&a)[V]) {
#pragma unroll
    for (int i = 0; i < V; ++i) a[i] = 0.f;
    for (int j = 0; j < p.n; ++j) {
      float b[V];
      load_vec<V>(p.results + j * layer + row + c, b);
      const float f = p.average[j];
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] = fmaf(f, b[i], a[i]);
    }
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < p.H) {
      sublayer(c, yk[k]);
      load_vec<V>(p.x_in + row + c, xk[k]);
      if constexpr (AVG) earlier(c, past[k]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += yk[k][i] * yk[k][i];
    }
  }
  for (int c = threadIdx.x * V + KEEP * step; c < p.H; c += step) {
    float y[V];
    sublayer(c, y);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += y[i] * y[i];
  }
  const float r = p.mult / sqrtf(block_sum2(ss, 0.f).x / (float)p.H + p.eps);
  const float last = AVG ? p.average[p.n] : 1.f;
  ss = 0.f;
  auto update = [&](int c, float (&y)[V], float (&x)[V], float (&a)[V]) {      // leaves the new residual in x
    float g[V];
    load_vec<V>(p.w_out + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] = fmaf(y[i] * r, g[i], x[i]);
    if constexpr (AVG) {
      if (p.store) store_vec<V>(p.results + p.n * layer + row + c, x);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] = fmaf(last, x[i], a[i]);
    }
    store_vec<V>(p.x_out + row + c, x);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += x[i] * x[i];
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < p.H) update(c, yk[k], xk[k], past[AVG ? k : 0]);
  }
  for (int c = threadIdx.x * V + KEEP * step; c < p.H; c += step) {
    float y[V], x[V], a[V];
    sublayer(c, y);
    load_vec<V>(p.x_in + row + c, x);
    if constexpr (AVG) earlier(c, a);
    update(c, y, x, a);
  }
  const float rn = 1.0f / sqrtf(block_sum2(ss, 0.f).x / (float)p.H + p.eps);
  T* hr = (T*)p.h + (size_t)t * p.h_ld;
  auto finish = [&](int c, float (&x)[V]) {
    float g[V];
    load_vec<V>(p.w + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] = x[i] * rn * g[i];
    store_vec<V>(hr + c, x);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < p.H) finish(c, xk[k]);
  }
  for (int c = threadIdx.x * V + KEEP * step; c < p.H; c += step) {
    float x[V];
    load_vec<V>(p.x_out + row + c, x);
    finish(c, x);
  }
  for (int c = p.H + threadIdx.x; c < p.h_ld; c += blockDim.x) hr[c] = from_f32<T>(0.f);
}

static inline int da_threads(int n, int v) {
  const int th = ((n + v - 1) / v + 31) / 32 * 32;
  return th > 256 ? 256 : (th < 32 ? 32 : th);
}

}  // namespace omni

using namespace omni;

#define FOR_TYPE(CALL)          \
  if (f32) { typedef float T; CALL } else { typedef bf16 T; CALL }

extern "C" int omni_embed_positions(const int64_t* ids, const void* table, int rows, int table_ld, const int64_t* positions,
                                    const void* pos_table, int pos_rows, int pos_ld, void* x, int T_rows, int H, int ld,
                                    const float* w, float eps, void* h, int h_ld, int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H || h_ld < H || table_ld < H || (pos_table != nullptr && (pos_ld < H || positions == nullptr))) return -1;
  const EmbedParams p = {ids, table, rows, table_ld, positions, pos_table, pos_rows, pos_ld, (float*)x, H, ld, w, eps, h, h_ld};
  if (H % 8 == 0 && ld % 8 == 0 && h_ld % 8 == 0 && table_ld % 8 == 0 && (pos_table == nullptr || pos_ld % 8 == 0)) {
    FOR_TYPE((embed_positions_kernel<T, 8, 2><<<T_rows, da_threads(H, 8), 0, st>>>(p));)
  } else {
    FOR_TYPE((embed_positions_kernel<T, 1, 2><<<T_rows, da_threads(H, 1), 0, st>>>(p));)
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_both_norms_step(const void* x_in, void* x_out, int T_rows, int H, int ld, const void* y, int y_ld,
                                    const int* row_of, int top_k, const void* shared, const float* w_out, float mult, void* results,
                                    const float* average, int n, int store, const float* w, float eps, void* h, int h_ld, int f32,
                                    cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H || h_ld < H || y_ld < H || y == nullptr) return -1;
  if (row_of != nullptr && (top_k < 1 || top_k > 32)) return -2;
  if (results != nullptr && (average == nullptr || n < 1)) return -3;
  const StepParams p = {(const float*)x_in, (float*)x_out, y, y_ld, row_of, top_k, shared, w_out, mult, (float*)results, average, n, store,
                        w, eps, h, H, ld, h_ld};
#define STEP(V, KEEP)                                                                                                            \
  if (results != nullptr) { FOR_TYPE((both_norms_step_kernel<T, V, KEEP, true><<<T_rows, da_threads(H, V), 0, st>>>(p, T_rows));) } \
  else { FOR_TYPE((both_norms_step_kernel<T, V, KEEP, false><<<T_rows, da_threads(H, V), 0, st>>>(p, T_rows));) }
  const bool v8 = H % 8 == 0 && ld % 8 == 0 && h_ld % 8 == 0 && y_ld % 8 == 0;
  if (v8 && H <= 2048) { STEP(8, 1) }
  else if (v8) { STEP(8, 2) }
  else { STEP(1, 2) }
#undef STEP
  return (int)cudaGetLastError();
}
#undef FOR_TYPE
