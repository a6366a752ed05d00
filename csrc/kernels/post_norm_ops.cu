// Row kernels of models with one fp32 residual stream and norms on the sublayers' outputs or ahead of the sublayers:
//   omni_embed_residual      embedding gather -> fp32 residual and its activation copy (the first sublayer's input)
//   omni_post_norm_add       residual += rmsnorm(sublayer output) * w, and the activation copy for the next sublayer
//   omni_rmsnorm_residual    final norm: fp32 residual -> activations
//   omni_residual_norm       norms ahead: embedding gather, or residual += sublayer output (a tensor, or the parts of an expert
//                            mixture) + bias, and the normed input of the next sublayer in the same pass
//   omni_qk_norm_rope_cache  optional RMSNorm over the whole q and the whole k projection, rotate-half RoPE on the first
//                            dimensions of every head, K/V scatter into the paged cache
//   omni_gated_mul           gelu(gate) * up, silu(gate) * up or the clamped form, for widths the GEMM epilogue does not take
//   omni_gemm_f32            plain fp32 matrix products: dense, by row segments, or by column groups (fp32 runs of a model)
// Activations are bf16 or fp32 (`f32` argument).  Rows have a pitch (`ld`, elements) that may exceed their width: the
// padding columns of an output are written as zeros so that it can be a TMA operand of the next GEMM.  Norm weights are
// fp32.  Every value between two roundings to the activation type is fp32.
#include "../include/expert_sum.cuh"
#include "../include/omni_vec.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

template <typename T, int V>
__global__ void embed_residual_kernel(const int64_t* __restrict__ ids, const T* __restrict__ table, int rows, int ld,
                                      float* __restrict__ x, T* __restrict__ xa) {
  const int t = blockIdx.x;
  const int64_t id = ids[t];
  const bool ok = id >= 0 && id < rows;
  for (int c = threadIdx.x * V; c < ld; c += blockDim.x * V) {
    float v[V];
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = 0.f;
    if (ok) load_vec<V>(table + (size_t)id * ld + c, v);
    store_vec<V>(x + (size_t)t * ld + c, v);
    if (xa != nullptr) store_vec<V>(xa + (size_t)t * ld + c, v);
  }
}

// KEEP vectors per thread stay in registers between the two passes; what is beyond them is read again.
template <typename T, int V, int KEEP>
__global__ void post_norm_add_kernel(const T* __restrict__ y, int y_ld, const float* __restrict__ w, float* __restrict__ x,
                                     T* __restrict__ xa, int H, int ld, float eps) {
  const int t = blockIdx.x;
  const T* yr = y + (size_t)t * y_ld;
  float keep[KEEP][V];
  float ss = 0.f;
  const int step = blockDim.x * V;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < H) {
      load_vec<V>(yr + c, keep[k]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += keep[k][i] * keep[k][i];
    }
  }
  for (int c = threadIdx.x * V + KEEP * step; c < H; c += step) {
    float v[V];
    load_vec<V>(yr + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += v[i] * v[i];
  }
  const float r = 1.0f / sqrtf(block_sum2(ss, 0.f).x / (float)H + eps);
  auto finish = [&](int c, const float (&v)[V]) {
    float g[V], a[V];
    load_vec<V>(w + c, g);
    load_vec<V>(x + (size_t)t * ld + c, a);
#pragma unroll
    for (int i = 0; i < V; ++i) a[i] += v[i] * r * g[i];
    store_vec<V>(x + (size_t)t * ld + c, a);
    if (xa != nullptr) store_vec<V>(xa + (size_t)t * ld + c, a);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < H) finish(c, keep[k]);
  }
  for (int c = threadIdx.x * V + KEEP * step; c < H; c += step) {
    float v[V];
    load_vec<V>(yr + c, v);
    finish(c, v);
  }
  if (xa != nullptr)
    for (int c = H + threadIdx.x; c < ld; c += blockDim.x) xa[(size_t)t * ld + c] = from_f32<T>(0.f);
}

template <typename T, int V>
__global__ void rmsnorm_residual_kernel(const float* __restrict__ x, const float* __restrict__ w, T* __restrict__ out, int H,
                                        int ld, float eps) {
  const int t = blockIdx.x;
  const float* xr = x + (size_t)t * ld;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float v[V];
    load_vec<V>(xr + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += v[i] * v[i];
  }
  const float r = 1.0f / sqrtf(block_sum2(ss, 0.f).x / (float)H + eps);
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float v[V], g[V];
    load_vec<V>(xr + c, v);
    load_vec<V>(w + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = v[i] * r * g[i];
    store_vec<V>(out + (size_t)t * ld + c, v);
  }
  for (int c = H + threadIdx.x; c < ld; c += blockDim.x) out[(size_t)t * ld + c] = from_f32<T>(0.f);
}

struct ResidualParams {
  float* x;              // [T, ld]
  const int64_t* ids;    // embedding gather: x = table[ids[t]]; null: x += y
  const void* table;     // [rows, table_ld]
  int rows, table_ld;
  const void* y;         // sublayer output rows of pitch y_ld; expert mixtures: the sorted expert rows; null: x as it is
  int y_ld;
  const int* row_of;     // expert mixtures: [T, top_k] row of y, or -1; null: y has one row per token
  int top_k;
  const void* shared;    // expert mixtures: [T, y_ld] or null
  const float* bias;     // [H] or null, added with y
  const float* w;        // norm weight
  float eps, out_scale;  // factor on the normed row
  void* h;               // [T, h_ld]
  int H, ld, h_ld;
  int ones;              // column H of h is one (the column that carries the next projection's bias)
};

// KEEP vectors per thread stay in registers between the two passes; what is beyond them is read again.
template <typename T, int V, int KEEP>
__global__ void residual_norm_kernel(const ResidualParams p) {
  const int t = blockIdx.x;
  __shared__ int rows[32];
  if (p.row_of != nullptr) {
    if (threadIdx.x < p.top_k) rows[threadIdx.x] = p.row_of[(size_t)t * p.top_k + threadIdx.x];
    __syncthreads();
  }
  float* xr = p.x + (size_t)t * p.ld;
  const int64_t id = p.ids != nullptr ? p.ids[t] : 0;
  const bool known = id >= 0 && id < p.rows;
  float keep[KEEP][V], ss = 0.f;
  const int step = blockDim.x * V;
  auto update = [&](int c, float (&a)[V]) {
    if (p.ids != nullptr) {
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] = 0.f;
      if (known) load_vec<V>((const T*)p.table + (size_t)id * p.table_ld + c, a);
    } else {
      load_vec<V>(xr + c, a);
      if (p.y != nullptr) {
        float y[V];
        if (p.row_of != nullptr) expert_sum<T, V>((const T*)p.y, p.y_ld, rows, p.top_k, (const T*)p.shared, t, c, y);
        else load_vec<V>((const T*)p.y + (size_t)t * p.y_ld + c, y);
#pragma unroll
        for (int i = 0; i < V; ++i) a[i] += y[i];
        if (p.bias != nullptr) {
          load_vec<V>(p.bias + c, y);
#pragma unroll
          for (int i = 0; i < V; ++i) a[i] += y[i];
        }
      }
    }
    store_vec<V>(xr + c, a);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += a[i] * a[i];
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < p.H) update(c, keep[k]);
  }
  for (int c = threadIdx.x * V + KEEP * step; c < p.H; c += step) {
    float a[V];
    update(c, a);
  }
  const float r = p.out_scale / sqrtf(block_sum2(ss, 0.f).x / (float)p.H + p.eps);
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
  for (int c = p.H + threadIdx.x; c < p.h_ld; c += blockDim.x) hr[c] = from_f32<T>(p.ones && c == p.H ? 1.f : 0.f);
}

// One CTA per token, one warp per head.  q rows are normed (qw null: not) and rotated in place, k rows go to the cache the same way,
// v rows are copied.  Hkv = 0: the layer reads another layer's cache and has q rows only.
template <typename T, int V>
__global__ void qk_norm_rope_cache_kernel(T* __restrict__ qkv, int ld, int Hq, int Hkv, int D, int DV,
                                          const float* __restrict__ qw, const float* __restrict__ kw, float eps,
                                          const float* __restrict__ cos_sin, int rot, const int64_t* __restrict__ positions,
                                          const int64_t* __restrict__ slots, T* __restrict__ k_cache,
                                          T* __restrict__ v_cache) {
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  T* row = qkv + (size_t)t * ld;
  const int nq = Hq * D, nk = Hkv * D;
  const bool normed = qw != nullptr;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * V; normed && c < nq + nk; c += blockDim.x * V) {
    float v[V];
    load_vec<V>(row + c, v);
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) s += v[i] * v[i];
    if (c < nq) sq += s; else sk += s;
  }
  float rq = 1.0f, rk = 1.0f;
  if (normed) {
    const float2 tot = block_sum2(sq, sk);
    rq = 1.0f / sqrtf(tot.x / (float)nq + eps);
    rk = nk > 0 ? 1.0f / sqrtf(tot.y / (float)nk + eps) : 0.f;
  }
  const int64_t slot = slots[t];
  const int half = rot >> 1;
  const float* cs = cos_sin + (size_t)positions[t] * rot;
  for (int hd = warp; hd < Hq + Hkv; hd += nwarps) {
    const bool is_q = hd < Hq;
    const T* src = row + (size_t)hd * D;
    T* dst = is_q ? row + (size_t)hd * D : k_cache + ((size_t)slot * Hkv + (hd - Hq)) * D;
    if (!is_q && slot < 0) continue;
    const float* w = !normed ? nullptr : (is_q ? qw + (size_t)hd * D : kw + (size_t)(hd - Hq) * D);
    const float r = is_q ? rq : rk;
    for (int c = lane * V; c < D; c += 32 * V) {
      if (c >= half && c < rot) continue;      // written together with its partner
      float a[V], wa[V];
      load_vec<V>(src + c, a);
      if (normed) {
        load_vec<V>(w + c, wa);
#pragma unroll
        for (int i = 0; i < V; ++i) a[i] = a[i] * r * wa[i];
      }
      if (c < half) {
        float b[V], wb[V], co[V], si[V];
        load_vec<V>(src + c + half, b);
        if (normed) {
          load_vec<V>(w + c + half, wb);
#pragma unroll
          for (int i = 0; i < V; ++i) b[i] = b[i] * r * wb[i];
        }
        load_vec<V>(cs + c, co);
        load_vec<V>(cs + half + c, si);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          const float u = a[i];
          a[i] = u * co[i] - b[i] * si[i];
          b[i] = b[i] * co[i] + u * si[i];
        }
        store_vec<V>(dst + c + half, b);
      }
      store_vec<V>(dst + c, a);
    }
  }
  if (slot >= 0) {
    const T* vr = row + nq + nk;
    T* vd = v_cache + (size_t)slot * Hkv * DV;
    for (int c = threadIdx.x * V; c < Hkv * DV; c += blockDim.x * V)
      *reinterpret_cast<VecOf<T, V>*>(vd + c) = *reinterpret_cast<const VecOf<T, V>*>(vr + c);
  }
}

// KIND 0: gelu(g) u, 2: silu(g) u, 1: min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u, +-limit) + 1)
template <typename T, int V, int KIND>
__global__ void gated_mul_kernel(const T* __restrict__ x, int x_ld, int up_off, T* __restrict__ out, int out_ld, int T_rows,
                                 int I, float limit) {
  const int row = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= out_ld) return;
  float o[V];
#pragma unroll
  for (int i = 0; i < V; ++i) o[i] = 0.f;
  if (c < I) {
    float g[V], u[V];
    load_vec<V>(x + (size_t)row * x_ld + c, g);
    load_vec<V>(x + (size_t)row * x_ld + up_off + c, u);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      if (KIND == 0) {
        o[i] = gelu_tanh_for<T>(g[i]) * u[i];
      } else if (KIND == 2) {
        o[i] = silu_for<T>(g[i]) * u[i];
      } else {
        const float gc = fminf(g[i], limit);
        o[i] = div_for<T>(gc, 1.0f + exp_for<T>(-1.702f * gc)) * (fminf(fmaxf(u[i], -limit), limit) + 1.0f);
      }
    }
  }
  store_vec<V>(out + (size_t)row * out_ld + c, o);
}

struct GemmF32Params {
  const float *x, *w;
  float* out;
  int T, N, K, x_ld, out_ld;
  const int *seg_start, *seg_len;      // [G] row segment of every group, or null: all rows
  const float* row_scale;              // [T] or null
  int x_group_col, out_group_col;      // first column of a group's x and out rows is group * this
};

// out[t, n] = sum_k x[t, k] w[g, n, k].  64 x 64 tile per CTA, 16 k per step, 4 x 4 outputs per thread; blockIdx.z = group.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32Params p) {
  const int g = blockIdx.z;
  const int first = p.seg_len ? p.seg_start[g] : 0, rows = p.seg_len ? p.seg_len[g] : p.T;
  const int t0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  if (t0 >= rows) return;
  const float* x = p.x + (size_t)first * p.x_ld + (size_t)g * p.x_group_col;
  const float* w = p.w + (size_t)g * p.N * p.K;
  float* out = p.out + (size_t)first * p.out_ld + (size_t)g * p.out_group_col;
  __shared__ float xs[16][68], ws[16][68];
  const int tr = (threadIdx.x >> 4) * 4, tc = (threadIdx.x & 15) * 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      xs[lk + i][lr] = (t0 + lr < rows && k < p.K) ? x[(size_t)(t0 + lr) * p.x_ld + k] : 0.f;
      ws[lk + i][lr] = (n0 + lr < p.N && k < p.K) ? w[(size_t)(n0 + lr) * p.K + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = xs[k][tr + i]; b[i] = ws[k][tc + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (t0 + tr + i >= rows) break;
    const float s = p.row_scale ? p.row_scale[first + t0 + tr + i] : 1.0f;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n0 + tc + j < p.N) out[(size_t)(t0 + tr + i) * p.out_ld + n0 + tc + j] = acc[i][j] * s;
  }
}

static inline int row_threads(int n, int v) {
  int th = ((n + v - 1) / v + 31) / 32 * 32;
  return th > 256 ? 256 : (th < 32 ? 32 : th);
}

}  // namespace omni

using namespace omni;

#define FOR_TYPE(CALL)          \
  if (f32) { typedef float T; CALL } else { typedef bf16 T; CALL }

extern "C" int omni_embed_residual(const int64_t* ids, const void* table, int rows, int T_rows, int ld, void* x, void* xa,
                                   int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (ld % 4 != 0) return -1;
  FOR_TYPE((embed_residual_kernel<T, 4><<<T_rows, row_threads(ld, 4), 0, st>>>(ids, (const T*)table, rows, ld, (float*)x,
                                                                               (T*)xa));)
  return (int)cudaGetLastError();
}

extern "C" int omni_post_norm_add(const void* y, int y_ld, const void* w, void* x, void* xa, int T_rows, int H, int ld,
                                  float eps, int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H || y_ld < H) return -1;
  if (H % 8 == 0 && y_ld % 8 == 0 && ld % 8 == 0) {
    FOR_TYPE((post_norm_add_kernel<T, 8, 2><<<T_rows, row_threads(H, 8), 0, st>>>((const T*)y, y_ld, (const float*)w,
                                                                                   (float*)x, (T*)xa, H, ld, eps));)
  } else {
    FOR_TYPE((post_norm_add_kernel<T, 1, 1><<<T_rows, row_threads(H, 1), 0, st>>>((const T*)y, y_ld, (const float*)w,
                                                                                   (float*)x, (T*)xa, H, ld, eps));)
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_rmsnorm_residual(const void* x, const void* w, void* out, int T_rows, int H, int ld, float eps, int f32,
                                     cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H) return -1;
  if (H % 8 == 0 && ld % 8 == 0) {
    FOR_TYPE((rmsnorm_residual_kernel<T, 8><<<T_rows, row_threads(H, 8), 0, st>>>((const float*)x, (const float*)w, (T*)out, H,
                                                                                  ld, eps));)
  } else {
    FOR_TYPE((rmsnorm_residual_kernel<T, 1><<<T_rows, row_threads(H, 1), 0, st>>>((const float*)x, (const float*)w, (T*)out, H,
                                                                                  ld, eps));)
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_residual_norm(void* x, int T_rows, int H, int ld, const int64_t* ids, const void* table, int rows, int table_ld,
                                  const void* y, int y_ld, const int* row_of, int top_k, const void* shared, const float* bias,
                                  const float* w, float eps, float out_scale, void* h, int h_ld, int ones, int f32,
                                  cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || ld < H || h_ld < H + (ones ? 1 : 0) || (ids != nullptr && table_ld < H) || (y != nullptr && y_ld < H)) return -1;
  if (row_of != nullptr && (top_k < 1 || top_k > 32 || y == nullptr)) return -2;
  const ResidualParams p = {(float*)x, ids, table, rows, table_ld, y, y_ld, row_of, top_k, shared, bias, w, eps, out_scale, h, H, ld, h_ld, ones};
  if (H % 8 == 0 && ld % 8 == 0 && h_ld % 8 == 0 && (ids == nullptr || table_ld % 8 == 0) && (y == nullptr || y_ld % 8 == 0)) {
    FOR_TYPE((residual_norm_kernel<T, 8, 2><<<T_rows, row_threads(H, 8), 0, st>>>(p));)
  } else {
    FOR_TYPE((residual_norm_kernel<T, 1, 1><<<T_rows, row_threads(H, 1), 0, st>>>(p));)
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_qk_norm_rope_cache(void* qkv, int ld, int Hq, int Hkv, int D, int DV, const void* qw, const void* kw,
                                       float eps, const void* cos_sin, int rot, const int64_t* positions,
                                       const int64_t* slots, void* k_cache, void* v_cache, int T_rows, int f32,
                                       cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (Hq < 1 || D < 1 || rot < 0 || rot > D || rot % 2 != 0 || (rot > 0 && cos_sin == nullptr)) return -1;
  if (Hkv > 0 && (k_cache == nullptr || v_cache == nullptr || (qw != nullptr && kw == nullptr))) return -2;
  if (D % 4 == 0 && DV % 4 == 0 && (rot / 2) % 4 == 0 && ld % 4 == 0) {
    FOR_TYPE((qk_norm_rope_cache_kernel<T, 4><<<T_rows, 256, 0, st>>>(
                  (T*)qkv, ld, Hq, Hkv, D, DV, (const float*)qw, (const float*)kw, eps, (const float*)cos_sin, rot, positions,
                  slots, (T*)k_cache, (T*)v_cache));)
  } else {
    FOR_TYPE((qk_norm_rope_cache_kernel<T, 1><<<T_rows, 256, 0, st>>>(
                  (T*)qkv, ld, Hq, Hkv, D, DV, (const float*)qw, (const float*)kw, eps, (const float*)cos_sin, rot, positions,
                  slots, (T*)k_cache, (T*)v_cache));)
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_gated_mul(const void* x, int x_ld, int up_off, void* out, int out_ld, int T_rows, int I, int kind, float limit,
                              int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (I < 1 || out_ld < I || T_rows > 65535 * 16 || kind < 0 || kind > 2) return -1;
  const int vec = (I % 8 == 0 && x_ld % 8 == 0 && up_off % 8 == 0 && out_ld % 8 == 0) ? 8 : 1;
#define GATED(V, KIND)                                                                                                        \
  FOR_TYPE((gated_mul_kernel<T, V, KIND><<<grid, 128, 0, st>>>((const T*)x + (size_t)r0 * x_ld, x_ld, up_off,                 \
                                                               (T*)out + (size_t)r0 * out_ld, out_ld, n, I, limit));)
  for (int r0 = 0; r0 < T_rows; r0 += 65535) {      // grid.y limit
    const int n = T_rows - r0 < 65535 ? T_rows - r0 : 65535;
    const dim3 grid((out_ld / vec + 127) / 128 + (out_ld % vec ? 1 : 0), n);
    if (vec == 8 && kind == 0) { GATED(8, 0) }
    else if (vec == 8 && kind == 2) { GATED(8, 2) }
    else if (vec == 8) { GATED(8, 1) }
    else if (kind == 0) { GATED(1, 0) }
    else if (kind == 2) { GATED(1, 2) }
    else { GATED(1, 1) }
  }
#undef GATED
  return (int)cudaGetLastError();
}

// w [G, N, K] contiguous.  Groups by row segments (seg_start / seg_len), by columns (x_group_col / out_group_col), or one.
extern "C" int omni_gemm_f32(const void* x, const void* w, void* out, int T_rows, int N, int K, int x_ld, int out_ld, int G,
                             const int* seg_start, const int* seg_len, const float* row_scale, int x_group_col,
                             int out_group_col, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (N < 1 || K < 1 || G < 1 || G > 65535 || x_ld < K || out_ld < N) return -1;
  if ((seg_len == nullptr) != (seg_start == nullptr)) return -3;
  const dim3 grid((N + 63) / 64, (T_rows + 63) / 64, G);
  if (grid.y > 65535) return -2;
  const GemmF32Params p = {(const float*)x, (const float*)w, (float*)out, T_rows, N, K, x_ld, out_ld, seg_start, seg_len,
                           row_scale, x_group_col, out_group_col};
  gemm_f32_kernel<<<grid, 256, 0, st>>>(p);
  return (int)cudaGetLastError();
}
#undef FOR_TYPE
