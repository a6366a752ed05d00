// Between the input projections of an attention layer and the attention itself:
//   omni_qkv_prepare     optional RMSNorm of every q and k head, rotation of the first dimensions of every head (halves or
//                        neighbours), values mixed with those of an earlier layer or divided by their head's root mean square, K/V
//                        scatter into the paged cache
//   omni_latent_prepare  latent attention: RMSNorm of the query latent (if there is one) and of the key/value latent, rotation of
//                        the shared key part; latent | key part go to the cache and, if asked for, to contiguous rows
//   omni_rotate_heads    rotation of a part of every head, in place or into another layout
//   omni_gather_pages    rows of the paged cache to contiguous rows, a range of positions per request
// Activations are bf16 or fp32 (`f32`), norm weights and angles fp32; every value between two roundings is fp32.  cos_sin
// [positions, rot] holds cos | sin.  A row with a negative slot is padding and leaves nothing in the cache.
#include "../include/omni_vec.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

struct QkvParams {
  int ld, Hq, Hkv, D, DV;      // rows: q heads | k heads | v heads
  const float *qw, *kw;        // [D] each, or null: no norm
  float eps;
  const float* cos_sin;
  int rot, pairs;              // rotated dimensions; neighbours (1) or halves (0)
  const int64_t *positions, *slots;
  const float* mix;            // one value: v <- (1 - mix) v + mix v_first; null: v as it is
  const void* v_first;         // [T, vf_ld]
  int vf_ld;
  int v_norm;                  // v <- v / rms(v) by head (without mix)
};

// One CTA per token, one warp per head.  q in place, k and v into the cache.
template <typename T, int V>
__global__ void qkv_prepare_kernel(T* __restrict__ qkv, const QkvParams p, T* __restrict__ k_cache, T* __restrict__ v_cache) {
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  T* row = qkv + (size_t)t * p.ld;
  const int64_t slot = p.slots[t];
  const int D = p.D, half = p.rot >> 1;
  const float* cs = p.cos_sin + (size_t)p.positions[t] * p.rot;
  const bool normed = p.qw != nullptr;
  // q heads stay as they are without norm and rotation
  for (int hd = warp + (normed || p.rot > 0 ? 0 : p.Hq); hd < p.Hq + p.Hkv; hd += nwarps) {
    const bool is_q = hd < p.Hq;
    if (!is_q && slot < 0) continue;
    const T* src = row + (size_t)hd * D;
    T* dst = is_q ? row + (size_t)hd * D : k_cache + ((size_t)slot * p.Hkv + (hd - p.Hq)) * D;
    const float* w = is_q ? p.qw : p.kw;
    float r = 1.0f;
    if (normed) {
      float ss = 0.f;
      for (int c = lane * V; c < D; c += 32 * V) {
        float v[V];
        load_vec<V>(src + c, v);
#pragma unroll
        for (int i = 0; i < V; ++i) ss += v[i] * v[i];
      }
      r = 1.0f / sqrtf(warp_sum32(ss) / (float)D + p.eps);
    }
    for (int c = lane * V; c < D; c += 32 * V) {
      if (c < p.rot && (p.pairs ? V == 1 && (c & 1) : c >= half)) continue;      // written together with its partner
      float a[V];
      load_vec<V>(src + c, a);
      if (normed) {
        float g[V];
        load_vec<V>(w + c, g);
#pragma unroll
        for (int i = 0; i < V; ++i) a[i] = a[i] * r * g[i];
      }
      if (c < p.rot && p.pairs) {
        if (V == 1) {
          float b = to_f32(src[c + 1]);
          if (normed) b = b * r * w[c + 1];
          const float co = cs[c >> 1], si = cs[half + (c >> 1)], u = a[0];
          a[0] = u * co - b * si;
          dst[c + 1] = from_f32<T>(b * co + u * si);
        } else {
#pragma unroll
          for (int i = 0; i + 1 < V; i += 2) {
            const float co = cs[(c + i) >> 1], si = cs[half + ((c + i) >> 1)], u = a[i];
            a[i] = u * co - a[i + 1] * si;
            a[i + 1] = a[i + 1] * co + u * si;
          }
        }
      } else if (c < half) {
        float b[V], co[V], si[V];
        load_vec<V>(src + c + half, b);
        if (normed) {
          float g[V];
          load_vec<V>(w + c + half, g);
#pragma unroll
          for (int i = 0; i < V; ++i) b[i] = b[i] * r * g[i];
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
  if (slot >= 0 && p.v_norm) {
    for (int hd = warp; hd < p.Hkv; hd += nwarps) {
      const T* vr = row + (size_t)(p.Hq + p.Hkv) * D + (size_t)hd * p.DV;
      T* vd = v_cache + ((size_t)slot * p.Hkv + hd) * p.DV;
      float ss = 0.f;
      for (int c = lane * V; c < p.DV; c += 32 * V) {
        float v[V];
        load_vec<V>(vr + c, v);
#pragma unroll
        for (int i = 0; i < V; ++i) ss += v[i] * v[i];
      }
      const float r = 1.0f / sqrtf(warp_sum32(ss) / (float)p.DV + p.eps);
      for (int c = lane * V; c < p.DV; c += 32 * V) {
        float v[V];
        load_vec<V>(vr + c, v);
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] *= r;
        store_vec<V>(vd + c, v);
      }
    }
  } else if (slot >= 0) {
    const T* vr = row + (size_t)(p.Hq + p.Hkv) * D;
    const int n = p.Hkv * p.DV;
    T* vd = v_cache + (size_t)slot * n;
    const float lam = p.mix != nullptr ? *p.mix : 0.f;
    for (int c = threadIdx.x * V; c < n; c += blockDim.x * V) {
      float v[V];
      load_vec<V>(vr + c, v);
      if (p.mix != nullptr) {
        float f[V];
        load_vec<V>((const T*)p.v_first + (size_t)t * p.vf_ld + c, f);
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = (1.0f - lam) * v[i] + lam * f[i];
      }
      store_vec<V>(vd + c, v);
    }
  }
}

struct LatentParams {
  int a_ld, q_rank, kv0, kv_rank, rot;   // columns of a row: [0, q_rank) query latent (0: none), from kv0 on kv_rank latent | rot key part
  const float *qw, *cw;
  float eps;
  const float* cos_sin;
  const int64_t *positions, *slots;
  int q_cols;                            // of the normed query latent's rows
  int c_cols, r_cols;                    // latent and key part in a cache row
};

// A CTA per token, or (ONE_WARP) a warp per token.
template <typename T, int V, bool ONE_WARP>
__global__ void latent_prepare_kernel(const T* __restrict__ a, const LatentParams p, T* __restrict__ cq, T* __restrict__ cache,
                                      T* __restrict__ rows, int T_rows) {
  const int t = ONE_WARP ? blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.x;
  if (ONE_WARP && t >= T_rows) return;
  const int tid = ONE_WARP ? threadIdx.x & 31 : threadIdx.x, nt = ONE_WARP ? 32 : blockDim.x;
  const T* ar = a + (size_t)t * p.a_ld;
  const T* cr = ar + p.kv0;
  float sq = 0.f, sc = 0.f;
  for (int c = tid * V; c < p.q_rank; c += nt * V) {
    float v[V];
    load_vec<V>(ar + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) sq += v[i] * v[i];
  }
  for (int c = tid * V; c < p.kv_rank; c += nt * V) {
    float v[V];
    load_vec<V>(cr + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) sc += v[i] * v[i];
  }
  const float2 tot = ONE_WARP ? make_float2(warp_sum32(sq), warp_sum32(sc)) : block_sum2(sq, sc);
  const float rq = 1.0f / sqrtf(tot.x / (float)max(p.q_rank, 1) + p.eps), rc = 1.0f / sqrtf(tot.y / (float)p.kv_rank + p.eps);
  T* qd = cq + (size_t)t * p.q_cols;
  for (int c = tid * V; c < p.q_cols; c += nt * V) {
    float v[V], g[V];
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = 0.f;
    if (c < p.q_rank) {
      load_vec<V>(ar + c, v);
      load_vec<V>(p.qw + c, g);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = v[i] * rq * g[i];
    }
    store_vec<V>(qd + c, v);
  }
  const int64_t slot = p.slots[t];
  const int D = p.c_cols + p.r_cols;
  T* d0 = slot >= 0 ? cache + (size_t)slot * D : nullptr;
  T* d1 = rows != nullptr ? rows + (size_t)t * D : nullptr;
  for (int c = tid * V; c < p.c_cols; c += nt * V) {
    float v[V], g[V];
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = 0.f;
    if (c < p.kv_rank) {
      load_vec<V>(cr + c, v);
      load_vec<V>(p.cw + c, g);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = v[i] * rc * g[i];
    }
    if (d0 != nullptr) store_vec<V>(d0 + c, v);
    if (d1 != nullptr) store_vec<V>(d1 + c, v);
  }
  const int half = p.rot >> 1;
  const float* cs = p.cos_sin + (size_t)p.positions[t] * p.rot;
  for (int c = tid; c < p.r_cols; c += nt) {
    float v = 0.f;
    if (c < p.rot) {
      const int i = c < half ? c : c - half;
      const float u = to_f32(cr[p.kv_rank + i]), w = to_f32(cr[p.kv_rank + half + i]), co = cs[i], si = cs[half + i];
      v = c < half ? u * co - w * si : w * co + u * si;
    }
    if (d0 != nullptr) d0[p.c_cols + c] = from_f32<T>(v);
    if (d1 != nullptr) d1[p.c_cols + c] = from_f32<T>(v);
  }
}

// src row t, head h: columns t src_ld + h src_head + [0, rot); dst alike with [0, cols), zeros past rot.  May be the same memory.
template <typename T, int V>
__global__ void rotate_heads_kernel(const T* src, long long src_ld, int src_head, int rows, int H, int rot, const float* __restrict__ cos_sin,
                                    const int64_t* __restrict__ positions, T* dst, long long dst_ld, int dst_head, int cols) {
  const int half = rot >> 1, per = half / V;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)rows * H * per) return;
  const int k = (int)(i % per) * V, h = (int)(i / per % H), t = (int)(i / per / H);
  const T* s = src + (size_t)t * src_ld + (size_t)h * src_head;
  T* d = dst + (size_t)t * dst_ld + (size_t)h * dst_head;
  const float* cs = cos_sin + (size_t)positions[t] * rot;
  float a[V], b[V], co[V], si[V];
  load_vec<V>(s + k, a);
  load_vec<V>(s + half + k, b);
  load_vec<V>(cs + k, co);
  load_vec<V>(cs + half + k, si);
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const float u = a[j];
    a[j] = u * co[j] - b[j] * si[j];
    b[j] = b[j] * co[j] + u * si[j];
  }
  store_vec<V>(d + k, a);
  store_vec<V>(d + half + k, b);
  if (k == 0)
    for (int c = rot; c < cols; ++c) d[c] = from_f32<T>(0.f);
}

// dst rows first[b] .. end[b] <- the cached rows of request req[b] from position pos0[b] on.  16-byte pieces, one warp per row.
__global__ void gather_pages_kernel(const uint4* __restrict__ cache, int pieces, const int* __restrict__ block_table, int bt_ld,
                                    int block_size, const int* __restrict__ req, const int* __restrict__ pos0,
                                    const int* __restrict__ first, const int* __restrict__ end, uint4* __restrict__ dst) {
  const int b = blockIdx.y, r = first[b] + blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (r >= end[b]) return;
  const int pos = pos0[b] + r - first[b];
  const size_t slot = (size_t)block_table[(size_t)req[b] * bt_ld + pos / block_size] * block_size + pos % block_size;
  for (int c = threadIdx.x & 31; c < pieces; c += 32) dst[(size_t)r * pieces + c] = cache[slot * pieces + c];
}

}  // namespace omni

using namespace omni;

#define FOR_TYPE(CALL)          \
  if (f32) { typedef float T; CALL } else { typedef bf16 T; CALL }

static bool aligned16(const void* p) { return (uintptr_t)p % 16 == 0; }

extern "C" int omni_qkv_prepare(void* qkv, int ld, int Hq, int Hkv, int D, int DV, const float* qw, const float* kw, float eps,
                                const float* cos_sin, int rot, int pairs, const int64_t* positions, const int64_t* slots,
                                const float* mix, const void* v_first, int vf_ld, int v_norm, void* k_cache, void* v_cache, int T_rows,
                                int f32, cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (Hq < 1 || Hkv < 1 || D < 1 || DV < 1 || rot < 0 || rot > D || rot % 2 != 0 || (rot > 0 && cos_sin == nullptr)) return -1;
  if (k_cache == nullptr || v_cache == nullptr || (qw == nullptr) != (kw == nullptr) || (mix != nullptr && (v_first == nullptr || v_norm))) return -2;
  const QkvParams p = {ld, Hq, Hkv, D, DV, qw, kw, eps, cos_sin, rot, pairs, positions, slots, mix, v_first, vf_ld, v_norm};
  const bool v4 = D % 4 == 0 && DV % 4 == 0 && (rot / 2) % 4 == 0 && ld % 4 == 0 && (mix == nullptr || (vf_ld % 4 == 0 && (uintptr_t)v_first % (f32 ? 16 : 8) == 0)) &&
                  aligned16(qkv);
  if (v4) {
    FOR_TYPE((qkv_prepare_kernel<T, 4><<<T_rows, 256, 0, st>>>((T*)qkv, p, (T*)k_cache, (T*)v_cache));)
  } else {
    FOR_TYPE((qkv_prepare_kernel<T, 1><<<T_rows, 256, 0, st>>>((T*)qkv, p, (T*)k_cache, (T*)v_cache));)
  }
  return (int)cudaGetLastError();
}

// cache [slots, c_cols + r_cols]; rows [T, c_cols + r_cols] or null; cq [T, q_cols].
extern "C" int omni_latent_prepare(const void* a, int a_ld, int q_rank, int kv0, int kv_rank, int rot, const float* qw, const float* cw,
                                   float eps, const float* cos_sin, const int64_t* positions, const int64_t* slots, void* cq,
                                   int q_cols, void* cache, void* rows, int c_cols, int r_cols, int T_rows, int f32,
                                   cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (q_rank < 0 || (q_rank > 0 && (cq == nullptr || qw == nullptr))) return -2;
  if (kv_rank < 1 || rot < 2 || rot % 2 != 0 || q_cols < q_rank || c_cols < kv_rank || r_cols < rot || kv0 < q_rank ||
      a_ld < kv0 + kv_rank + rot || cos_sin == nullptr)
    return -1;
  if (q_rank == 0) q_cols = 0;
  const LatentParams p = {a_ld, q_rank, kv0, kv_rank, rot, qw, cw, eps, cos_sin, positions, slots, q_cols, c_cols, r_cols};
#define LATENT(V)                                                                                                                     \
  if (q_rank == 0) { FOR_TYPE((latent_prepare_kernel<T, V, true><<<(T_rows + 3) / 4, 128, 0, st>>>((const T*)a, p, (T*)cq, (T*)cache, (T*)rows, T_rows));) } \
  else { FOR_TYPE((latent_prepare_kernel<T, V, false><<<T_rows, 128, 0, st>>>((const T*)a, p, (T*)cq, (T*)cache, (T*)rows, T_rows));) }
  const int sizes = q_rank | kv0 | kv_rank | a_ld | q_cols | c_cols | r_cols;
  if (q_rank == 0 && sizes % 8 == 0) { LATENT(8) }
  else if (sizes % 4 == 0) { LATENT(4) }
  else { LATENT(1) }
#undef LATENT
  return (int)cudaGetLastError();
}

extern "C" int omni_rotate_heads(const void* src, long long src_ld, int src_head, int T_rows, int H, int rot, const float* cos_sin,
                                 const int64_t* positions, void* dst, long long dst_ld, int dst_head, int cols, int f32,
                                 cudaStream_t st) {
  if (T_rows <= 0) return 0;
  if (H < 1 || rot < 2 || rot % 2 != 0 || cols < rot) return -1;
  const int half = rot / 2;
  const bool v4 = half % 4 == 0 && src_ld % 4 == 0 && src_head % 4 == 0 && dst_ld % 4 == 0 && dst_head % 4 == 0 && aligned16(cos_sin) &&
                  (uintptr_t)src % (f32 ? 16 : 8) == 0 && (uintptr_t)dst % (f32 ? 16 : 8) == 0;
  const long long n = (long long)T_rows * H * (half / (v4 ? 4 : 1));
  const unsigned grid = (unsigned)((n + 255) / 256);
  if (v4) {
    FOR_TYPE((rotate_heads_kernel<T, 4><<<grid, 256, 0, st>>>((const T*)src, src_ld, src_head, T_rows, H, rot, cos_sin, positions,
                                                               (T*)dst, dst_ld, dst_head, cols));)
  } else {
    FOR_TYPE((rotate_heads_kernel<T, 1><<<grid, 256, 0, st>>>((const T*)src, src_ld, src_head, T_rows, H, rot, cos_sin, positions,
                                                               (T*)dst, dst_ld, dst_head, cols));)
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_gather_pages(const void* cache, int row_bytes, const int* block_table, int bt_ld, int block_size, const int* req,
                                 const int* pos0, const int* first, const int* end, int B, int max_rows, void* dst, cudaStream_t st) {
  if (B <= 0 || max_rows <= 0) return 0;
  if (row_bytes < 16 || row_bytes % 16 != 0 || B > 65535 || !aligned16(cache) || !aligned16(dst)) return -1;
  gather_pages_kernel<<<dim3((max_rows + 7) / 8, B), 256, 0, st>>>((const uint4*)cache, row_bytes / 16, block_table, bt_ld, block_size,
                                                                  req, pos0, first, end, (uint4*)dst);
  return (int)cudaGetLastError();
}
#undef FOR_TYPE
