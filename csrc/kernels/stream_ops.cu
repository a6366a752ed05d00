// Row kernels of models with several residual streams (hyper-connections) and a layer norm ahead of every sublayer, and the
// token shift of WKV mixers:
//   omni_embed_streams   embedding gather times a constant -> all streams, and the first sublayer's normed input
//   omni_stream_step     sublayer output -> every stream anew, x_t <- sum_s mix[s, t] x_s + out[t] y, and the next sublayer's
//                        normed input, layer_norm(sum_s in[s] x_s) w, in one pass.  The output is a tensor, or the parts of
//                        an expert mixture (sorted expert rows, identity weights, shared expert) that are summed here
//   omni_token_shift     h + (h_prev - h) mu for several mu at once; h_prev of a request's first row comes from its state slot,
//                        which is moved on
//   omni_tanh_split      tanh of fp32 values as bf16 hi | lo, so that a product keeps 16 bits of mantissa on that side
// Streams are fp32, [T, streams, ld]; activations are bf16 or fp32 (`f32`), their padding columns are written as zeros.
#include "../include/expert_sum.cuh"
#include "../include/omni_vec.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

// u (fp32, H values in shared memory, `sum` this thread's part of their sum) -> layer_norm(u) w as activations
template <typename T, int V>
__device__ __forceinline__ void layer_norm_row(const float* u, float sum, const float* __restrict__ w, T* __restrict__ h, int H,
                                               int ld, float eps) {
  const float mean = block_sum2(sum, 0.f).x / (float)H;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V)
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float d = u[c + i] - mean;
      ss += d * d;
    }
  const float r = 1.0f / sqrtf(block_sum2(ss, 0.f).x / (float)H + eps);
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float g[V], o[V];
    load_vec<V>(w + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] = (u[c + i] - mean) * r * g[i];
    store_vec<V>(h + c, o);
  }
  for (int c = H + threadIdx.x; c < ld; c += blockDim.x) h[c] = from_f32<T>(0.f);
}

template <typename T, int V>
__global__ void embed_streams_kernel(const int64_t* __restrict__ ids, const T* __restrict__ table, int rows, int H, int ld,
                                     float scale, int streams, const float* __restrict__ in, const float* __restrict__ w,
                                     float eps, float* __restrict__ x, T* __restrict__ h) {
  extern __shared__ float so_u[];
  const int t = blockIdx.x;
  const int64_t id = ids[t];
  const bool ok = id >= 0 && id < rows;
  float tot = 0.f;
  for (int s = 0; s < streams; ++s) tot += in[s];
  float sum = 0.f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float v[V];
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = 0.f;
    if (ok) load_vec<V>(table + (size_t)id * ld + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] *= scale;
    for (int s = 0; s < streams; ++s) store_vec<V>(x + ((size_t)t * streams + s) * ld + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float u = v[i] * tot;
      so_u[c + i] = u;
      sum += u;
    }
  }
  layer_norm_row<T, V>(so_u, sum, w, h + (size_t)t * ld, H, ld, eps);
}

struct StepParams {
  float* x;              // [T, streams, ld]
  const void* y;         // sublayer output rows of pitch y_ld; expert mixtures: the sorted expert rows
  int y_ld;
  const int* row_of;     // expert mixtures: [T, top_k] row of y, or -1; null: y has one row per token
  const int* ids;        // [T, top_k] chosen experts
  const float* wts;      // [T, top_k]
  int top_k, experts;    // choices >= experts are identity experts: the sublayer's input times their weight
  const void* h_in;      // [T, h_ld] the sublayer's input
  const void* shared;    // [T, y_ld] or null
  const float *mix, *out, *in, *w;
  void* h;               // [T, h_ld]
  int H, ld, h_ld, streams;
  float eps;
  int last;              // the streams are not needed any more
};

template <typename T, int V, int S>
__global__ void stream_step_kernel(const StepParams p) {
  extern __shared__ float so_u[];
  const int t = blockIdx.x, n = S > 4 ? p.streams : S;
  __shared__ float mix[S * S], out[S], in[S];
  __shared__ int rows[32];
  __shared__ float same;
  for (int i = threadIdx.x; i < n * n; i += blockDim.x) mix[i] = p.mix[i];
  if (threadIdx.x < n) { out[threadIdx.x] = p.out[threadIdx.x]; in[threadIdx.x] = p.in[threadIdx.x]; }
  if (p.row_of != nullptr) {
    if (threadIdx.x < p.top_k) rows[threadIdx.x] = p.row_of[(size_t)t * p.top_k + threadIdx.x];
    if (threadIdx.x == 0) {
      float s = 0.f;
      for (int k = 0; k < p.top_k; ++k)
        if (p.ids[(size_t)t * p.top_k + k] >= p.experts) s += p.wts[(size_t)t * p.top_k + k];
      same = s;
    }
  }
  __syncthreads();
  float sum = 0.f;
  for (int c = threadIdx.x * V; c < p.H; c += blockDim.x * V) {
    float y[V];
    if (p.row_of == nullptr) {
      load_vec<V>((const T*)p.y + (size_t)t * p.y_ld + c, y);
    } else {
      expert_sum<T, V>((const T*)p.y, p.y_ld, rows, p.top_k, (const T*)p.shared, t, c, y);
      if (same != 0.f) {
        float v[V];
        load_vec<V>((const T*)p.h_in + (size_t)t * p.h_ld + c, v);
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = fmaf(same, v[i], y[i]);
      }
    }
    float a[S][V], u[V];
    float* xr = p.x + (size_t)t * n * p.ld + c;
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (s < n) load_vec<V>(xr + (size_t)s * p.ld, a[s]);
#pragma unroll
    for (int i = 0; i < V; ++i) u[i] = 0.f;
#pragma unroll
    for (int q = 0; q < S; ++q) {
      if (q >= n) break;
      float b[V];
#pragma unroll
      for (int i = 0; i < V; ++i) b[i] = out[q] * y[i];
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s < n)
#pragma unroll
          for (int i = 0; i < V; ++i) b[i] = fmaf(mix[s * n + q], a[s][i], b[i]);
      if (!p.last) store_vec<V>(xr + (size_t)q * p.ld, b);
#pragma unroll
      for (int i = 0; i < V; ++i) u[i] = fmaf(in[q], b[i], u[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
      so_u[c + i] = u[i];
      sum += u[i];
    }
  }
  layer_norm_row<T, V>(so_u, sum, p.w, (T*)p.h + (size_t)t * p.h_ld, p.H, p.h_ld, p.eps);
}

// out [T, parts, part_ld]; rows of request r are cu_q[r] .. cu_q[r + 1] (null: one each).  state [slots, H].
template <typename T, int V>
__global__ void token_shift_kernel(const T* __restrict__ h, int ld, const float* __restrict__ mu, int parts, int H,
                                   T* __restrict__ state, const int64_t* __restrict__ positions,
                                   const int* __restrict__ q_to_seq, const int* __restrict__ cu_q,
                                   const int* __restrict__ state_slots, T* __restrict__ out, int part_ld) {
  const int t = blockIdx.x;
  const int r = cu_q ? q_to_seq[t] : t;
  const int row0 = cu_q ? cu_q[r] : t, row1 = cu_q ? cu_q[r + 1] : t + 1;
  const int slot = state_slots[r];
  T* st = slot >= 0 ? state + (size_t)slot * H : nullptr;
  const bool stored = t == row0, start = positions[t] == 0;
  T* o = out + (size_t)t * parts * part_ld;
  for (int c = threadIdx.x * V; c < part_ld; c += blockDim.x * V) {
    float x[V], d[V];
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] = d[i] = 0.f;
    if (c < H) {
      load_vec<V>(h + (size_t)t * ld + c, x);
      if (!stored) load_vec<V>(h + (size_t)(t - 1) * ld + c, d);
      else if (!start && st != nullptr) load_vec<V>(st + c, d);
#pragma unroll
      for (int i = 0; i < V; ++i) d[i] -= x[i];
      if (stored && st != nullptr) {       // this CTA alone reads the slot, so it may also move it on
        float n[V];
        load_vec<V>(h + (size_t)(row1 - 1) * ld + c, n);
        store_vec<V>(st + c, n);
      }
    }
    for (int k = 0; k < parts; ++k) {
      float m[V], v[V];
#pragma unroll
      for (int i = 0; i < V; ++i) m[i] = 0.f;
      if (c < H) load_vec<V>(mu + (size_t)k * H + c, m);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = fmaf(d[i], m[i], x[i]);
      store_vec<V>(o + (size_t)k * part_ld + c, v);
    }
  }
}

template <typename T>
__global__ void tanh_split_kernel(const float* __restrict__ a, int a_ld, int R, T* __restrict__ out, int half, int rows) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * half) return;
  const int t = i / half, c = i % half;
  const float v = c < R ? tanhf(a[(size_t)t * a_ld + c]) : 0.f;
  const T hi = from_f32<T>(v);
  if (sizeof(T) == 4) {
    out[(size_t)t * half + c] = hi;
  } else {
    out[(size_t)t * 2 * half + c] = hi;
    out[(size_t)t * 2 * half + half + c] = from_f32<T>(v - to_f32(hi));
  }
}

static inline int so_threads(int n, int v) {
  int th = ((n + v - 1) / v + 31) / 32 * 32;
  return th > 256 ? 256 : (th < 32 ? 32 : th);
}

template <typename T, int V>
static int launch_step(const StepParams& p, int rows, cudaStream_t st) {
  const int th = so_threads(p.H, V), sm = p.H * (int)sizeof(float);
  switch (p.streams) {
    case 1: stream_step_kernel<T, V, 1><<<rows, th, sm, st>>>(p); break;
    case 2: stream_step_kernel<T, V, 2><<<rows, th, sm, st>>>(p); break;
    case 3: stream_step_kernel<T, V, 3><<<rows, th, sm, st>>>(p); break;
    case 4: stream_step_kernel<T, V, 4><<<rows, th, sm, st>>>(p); break;
    default: stream_step_kernel<T, 1, 16><<<rows, so_threads(p.H, 1), sm, st>>>(p); break;
  }
  return (int)cudaGetLastError();
}

}  // namespace omni

using namespace omni;

#define FOR_TYPE(CALL)          \
  if (f32) { typedef float T; CALL } else { typedef bf16 T; CALL }

constexpr int SO_MAX_H = 12288 - 64;      // one row in fp32 fits the default shared memory

extern "C" int omni_embed_streams(const int64_t* ids, const void* table, int rows, int T_rows, int H, int ld, float scale,
                                  int streams, const void* in, const void* w, float eps, void* x, void* h, int f32,
                                  cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H || H > SO_MAX_H || streams < 1 || streams > 16) return -1;
  const int sm = H * (int)sizeof(float);
  if (H % 4 == 0 && ld % 4 == 0) {
    FOR_TYPE((embed_streams_kernel<T, 4><<<T_rows, so_threads(H, 4), sm, st>>>(
                  ids, (const T*)table, rows, H, ld, scale, streams, (const float*)in, (const float*)w, eps, (float*)x, (T*)h));)
  } else {
    FOR_TYPE((embed_streams_kernel<T, 1><<<T_rows, so_threads(H, 1), sm, st>>>(
                  ids, (const T*)table, rows, H, ld, scale, streams, (const float*)in, (const float*)w, eps, (float*)x, (T*)h));)
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_stream_step(void* x, int T_rows, int H, int ld, int streams, const void* y, int y_ld, const int* row_of,
                                const int* ids, const float* wts, int top_k, int experts, const void* h_in,
                                const void* shared, const void* mix, const void* out, const void* in, const void* w, float eps,
                                void* h, int h_ld, int last, int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H || y_ld < H || h_ld < H || H > SO_MAX_H || streams < 1 || streams > 16) return -1;
  if (row_of != nullptr && (top_k < 1 || top_k > 32 || h_in == h)) return -2;
  StepParams p = {(float*)x, y, y_ld, row_of, ids, wts, top_k, experts, h_in, shared, (const float*)mix, (const float*)out,
                  (const float*)in, (const float*)w, h, H, ld, h_ld, streams, eps, last};
  if (H % 4 == 0 && ld % 4 == 0 && y_ld % 4 == 0 && h_ld % 4 == 0) {
    if (f32) return launch_step<float, 4>(p, T_rows, st);
    return launch_step<bf16, 4>(p, T_rows, st);
  }
  if (f32) return launch_step<float, 1>(p, T_rows, st);
  return launch_step<bf16, 1>(p, T_rows, st);
}

extern "C" int omni_token_shift(const void* h, int ld, const void* mu, int parts, int H, void* state, const int64_t* positions,
                                const int* q_to_seq, const int* cu_q, const int* state_slots, int T_rows, void* out, int part_ld,
                                int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H || part_ld < H || parts < 1) return -1;
  if (H % 8 == 0 && ld % 8 == 0 && part_ld % 8 == 0) {
    FOR_TYPE((token_shift_kernel<T, 8><<<T_rows, so_threads(part_ld, 8), 0, st>>>(
                  (const T*)h, ld, (const float*)mu, parts, H, (T*)state, positions, q_to_seq, cu_q, state_slots, (T*)out, part_ld));)
  } else {
    FOR_TYPE((token_shift_kernel<T, 1><<<T_rows, so_threads(part_ld, 1), 0, st>>>(
                  (const T*)h, ld, (const float*)mu, parts, H, (T*)state, positions, q_to_seq, cu_q, state_slots, (T*)out, part_ld));)
  }
  return (int)cudaGetLastError();
}

// a [T, a_ld] fp32, R columns -> bf16 [T, 2 half] (hi | lo) or fp32 [T, half], zeros past R.
extern "C" int omni_tanh_split(const void* a, int a_ld, int R, void* out, int half, int T_rows, int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (R < 1 || half < R || a_ld < R || (long long)T_rows * half > 0x7fffffffLL) return -1;
  const int n = T_rows * half;
  FOR_TYPE((tanh_split_kernel<T><<<(n + 255) / 256, 256, 0, st>>>((const float*)a, a_ld, R, (T*)out, half, T_rows));)
  return (int)cudaGetLastError();
}
#undef FOR_TYPE
