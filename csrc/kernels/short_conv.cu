// Short causal convolution per channel ahead of a mixer (Mamba-2: bias and silu; attention: neither): y_t = sum_k w[k] u_(t - taps + 1 + k).
// Earlier inputs of a request come from its slot of the state [slots, taps - 1, channels] (activation type), which the same
// call moves on.  A request whose first token of the call is at position 0 starts from zeros whatever its slot holds; a row with
// a negative slot is padding.  bias (may be null) and w [taps, channels] are fp32; act 1: silu.
#include "../include/omni_vec.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

template <int V>
__device__ __forceinline__ void load_bias(const float* bias, int c, float (&v)[V]) {
  if (bias != nullptr) {
    load_vec<V>(bias + c, v);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = 0.f;
  }
}

// Input of `pos - back` of the request whose rows start at `row0` (position `pos0`): from this call's rows, from the
// state, or zero before the start of the sequence.
template <typename T, int V>
__device__ __forceinline__ void conv_input(const T* u, int ld, const T* state, int taps, int C, int c, int row, long long pos,
                                           int row0, int back, float (&v)[V]) {
  if (pos - back < 0) {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = 0.f;
  } else if (row - back >= row0) {
    load_vec<V>(u + (size_t)(row - back) * ld + c, v);
  } else {
    // state[k] holds the input k - (taps - 1) places before row0
    load_vec<V>(state + (size_t)(taps - 1 - (row0 - (row - back))) * C + c, v);
  }
}

// ragged rows; blockDim (32, 8): 32 channel vectors x 8 rows
template <typename T, int V>
__global__ void short_conv_kernel(const T* __restrict__ u, int ld, int C, int taps, const float* __restrict__ w,
                                 const float* __restrict__ bias, const T* __restrict__ state,
                                 const int64_t* __restrict__ positions, const int* __restrict__ q_to_seq,
                                 const int* __restrict__ cu_q, const int* __restrict__ state_slots, T* __restrict__ out,
                                 int out_ld, int rows, bool silu) {
  const int row = blockIdx.x * blockDim.y + threadIdx.y;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (row >= rows || c >= C) return;
  const int r = q_to_seq[row];
  const long long pos = positions[row];
  const int row0 = cu_q[r];
  const T* st = state + (size_t)max(state_slots[r], 0) * (taps - 1) * C;
  float acc[V];
  load_bias<V>(bias, c, acc);
  for (int k = 0; k < taps; ++k) {
    float v[V], g[V];
    conv_input<T, V>(u, ld, st, taps, C, c, row, pos, row0, taps - 1 - k, v);
    load_vec<V>(w + (size_t)k * C + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = fmaf(g[i], v[i], acc[i]);
  }
#pragma unroll
  for (int i = 0; i < V; ++i) acc[i] = silu ? silu_for<T>(acc[i]) : acc[i];
  store_vec<V>(out + (size_t)row * out_ld + c, acc);
}

// The same for up to four taps: a thread walks CONV_ROWS rows with the taps' inputs in registers, so that every input is
// read once.  blockDim (32, 4).
constexpr int CONV_ROWS = 16;
template <typename T, int V, int TAPS>
__global__ void short_conv_walk_kernel(const T* __restrict__ u, int ld, int C, const float* __restrict__ w,
                                      const float* __restrict__ bias, const T* __restrict__ state,
                                      const int64_t* __restrict__ positions, const int* __restrict__ q_to_seq,
                                      const int* __restrict__ cu_q, const int* __restrict__ state_slots, T* __restrict__ out,
                                      int out_ld, int rows, bool silu) {
  const int t0 = (blockIdx.x * blockDim.y + threadIdx.y) * CONV_ROWS;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (t0 >= rows || c >= C) return;
  float g[TAPS][V], b[V], x[TAPS][V];      // x[k]: the input TAPS - 1 - k rows back
#pragma unroll
  for (int k = 0; k < TAPS; ++k) load_vec<V>(w + (size_t)k * C + c, g[k]);
  load_bias<V>(bias, c, b);
  int next_start = t0;                     // first row of the next request (or of this walk): the window is fetched anew
#pragma unroll 4
  for (int e = 0; e < CONV_ROWS; ++e) {
    const int t = t0 + e;
    if (t >= rows) break;
    if (t == next_start) {
      const int r = q_to_seq[t], row0 = cu_q[r];
      next_start = cu_q[r + 1];
      const T* st = state + (size_t)max(state_slots[r], 0) * (TAPS - 1) * C;
      const long long pos = positions[t];
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k) conv_input<T, V>(u, ld, st, TAPS, C, c, t, pos, row0, TAPS - 1 - k, x[k]);
    }
    load_vec<V>(u + (size_t)t * ld + c, x[TAPS - 1]);
    float acc[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      acc[i] = b[i];
#pragma unroll
      for (int k = 0; k < TAPS; ++k) acc[i] = fmaf(g[k][i], x[k][i], acc[i]);
      if (silu) acc[i] = silu_for<T>(acc[i]);
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k) x[k][i] = x[k + 1][i];
    }
    store_vec<V>(out + (size_t)t * out_ld + c, acc);
  }
}

// after the convolution of ragged rows: the last taps - 1 inputs of every request go to its slot
template <typename T, int V>
__global__ void conv_state_kernel(const T* __restrict__ u, int ld, int C, int taps, T* __restrict__ state,
                                  const int64_t* __restrict__ positions, const int* __restrict__ cu_q,
                                  const int* __restrict__ state_slots) {
  const int r = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  const int slot = state_slots[r];
  const int row0 = cu_q[r], n = cu_q[r + 1] - row0;
  if (c >= C || slot < 0 || n <= 0) return;
  T* st = state + (size_t)slot * (taps - 1) * C;
  const int last = row0 + n - 1;
  const long long pos = positions[last];
  for (int k = 0; k < taps - 1; ++k) {           // ascending: reads lie ahead of what has been written
    float v[V];
    conv_input<T, V>(u, ld, st, taps, C, c, last, pos, row0, taps - 2 - k, v);
    store_vec<V>(st + (size_t)k * C + c, v);
  }
}

// one token per request: convolution and state shift together
template <typename T, int V>
__global__ void conv_step_kernel(const T* __restrict__ u, int ld, int C, int taps, const float* __restrict__ w,
                                 const float* __restrict__ bias, T* __restrict__ state, const int64_t* __restrict__ positions,
                                 const int* __restrict__ state_slots, T* __restrict__ out, int out_ld, bool silu) {
  const int r = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  const int slot = state_slots[r];
  float acc[V];
  if (slot < 0) {
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = 0.f;
    store_vec<V>(out + (size_t)r * out_ld + c, acc);
    return;
  }
  const long long pos = positions[r];
  T* st = state + (size_t)slot * (taps - 1) * C;
  load_bias<V>(bias, c, acc);
  for (int k = 0; k < taps; ++k) {
    float v[V], g[V];
    const int back = taps - 1 - k;
    conv_input<T, V>(u, ld, st, taps, C, c, r, pos, r, back, v);
    load_vec<V>(w + (size_t)k * C + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = fmaf(g[i], v[i], acc[i]);
    if (k > 0) store_vec<V>(st + (size_t)(k - 1) * C + c, v);       // entry k - 1 has been read
  }
#pragma unroll
  for (int i = 0; i < V; ++i) acc[i] = silu ? silu_for<T>(acc[i]) : acc[i];
  store_vec<V>(out + (size_t)r * out_ld + c, acc);
}

}  // namespace omni

using namespace omni;

// u: first channel of the convolution's input in row 0 (a column slice of the projection).  cu_q null: one row per request.
template <typename T, int V>
static int short_conv_t(const void* u, int ld, int C, int taps, const float* w, const float* bias, void* state,
                       const int64_t* positions, const int* q_to_seq, const int* cu_q, const int* state_slots, int B, int rows,
                       void* out, int out_ld, bool silu, cudaStream_t st) {
  const int vecs = (C + V - 1) / V;
  if (cu_q == nullptr) {
    conv_step_kernel<T, V><<<dim3((vecs + 127) / 128, B), 128, 0, st>>>((const T*)u, ld, C, taps, w, bias, (T*)state, positions,
                                                                       state_slots, (T*)out, out_ld, silu);
    return (int)cudaGetLastError();
  }
#define CONV_WALK(TAPS)                                                                                                   \
  short_conv_walk_kernel<T, V, TAPS><<<dim3((rows + 4 * CONV_ROWS - 1) / (4 * CONV_ROWS), (vecs + 31) / 32), dim3(32, 4), 0, st>>>( \
      (const T*)u, ld, C, w, bias, (const T*)state, positions, q_to_seq, cu_q, state_slots, (T*)out, out_ld, rows, silu)
  if (taps == 2) CONV_WALK(2);
  else if (taps == 3) CONV_WALK(3);
  else if (taps == 4) CONV_WALK(4);
  else
    short_conv_kernel<T, V><<<dim3((rows + 7) / 8, (vecs + 31) / 32), dim3(32, 8), 0, st>>>(
        (const T*)u, ld, C, taps, w, bias, (const T*)state, positions, q_to_seq, cu_q, state_slots, (T*)out, out_ld, rows, silu);
#undef CONV_WALK
  if (taps > 1)
    conv_state_kernel<T, V><<<dim3(B, (vecs + 127) / 128), 128, 0, st>>>((const T*)u, ld, C, taps, (T*)state, positions, cu_q,
                                                                        state_slots);
  return (int)cudaGetLastError();
}

extern "C" int omni_short_conv(const void* u, int ld, int C, int taps, const void* w, const void* bias, void* state,
                              const int64_t* positions, const int* q_to_seq, const int* cu_q, const int* state_slots, int B,
                              int rows, void* out, int out_ld, int act, int f32, cudaStream_t st) {
  if (B <= 0 || rows <= 0) return 0;
  if (C < 1 || taps < 1 || out_ld < C || act < 0 || act > 1 || B > 65535 || (cu_q == nullptr && rows != B)) return -1;
  const bool v8 = C % 8 == 0 && ld % 8 == 0 && out_ld % 8 == 0 &&
                  (((uintptr_t)u | (uintptr_t)out | (uintptr_t)state) % 16 == 0);
  const float *wf = (const float*)w, *bf = (const float*)bias;
  if (f32) {
    if (v8) return short_conv_t<float, 8>(u, ld, C, taps, wf, bf, state, positions, q_to_seq, cu_q, state_slots, B, rows, out, out_ld, act != 0, st);
    return short_conv_t<float, 1>(u, ld, C, taps, wf, bf, state, positions, q_to_seq, cu_q, state_slots, B, rows, out, out_ld, act != 0, st);
  }
  if (v8) return short_conv_t<bf16, 8>(u, ld, C, taps, wf, bf, state, positions, q_to_seq, cu_q, state_slots, B, rows, out, out_ld, act != 0, st);
  return short_conv_t<bf16, 1>(u, ld, C, taps, wf, bf, state, positions, q_to_seq, cu_q, state_slots, B, rows, out, out_ld, act != 0, st);
}
