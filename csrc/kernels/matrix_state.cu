// Mixers whose state is a matrix per head, between their projections: the matrix memory of xLSTM (mLSTM), WKV and gated linear
// attention (GLA).
//
//   mLSTM   S <- keep S + add k v^T,  n <- keep n + add k,  o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
//           with m the running maximum of the log gates, keep = exp(f + m' - m), add = exp(i - m)
//   WKV     o = (S + diag(u) k v^T)^T r,  S <- diag(w) S + k v^T,  w = exp(-exp(z + w0)) per head and key channel
//   GLA     S <- diag(a) S + k v^T,  o = S^T q,  a = sigmoid(z + w0)^(1 / tau) per head and key channel
//
// State slots (fp32): S [slots, H, P or P + 1, N] with N the key size and P the value size; the last row of the mLSTM's is n,
// which is what a value of one would accumulate.  m [slots, H].  A request whose first token of the call is at position 0
// starts from zeros; a row with a negative slot is padding.
//
//   omni_mlstm_gates   i, f and m of every token (one scan per request and head over pairs (sum of f, maximum)): keep and add
//                      for the token-by-token form, and per chunk of 128 tokens what the tensor-core form needs
//   omni_state_rows    token by token, the state in registers: a warp owns a few rows of P, N lies across its lanes.  One token
//                      per request (decode) makes it a stream over the state; fp32 runs and short portions take it too
//   omni_head_norm     o of every head divided by its root mean square, times a weight, a gate and a constant
// The chunked forms for portions of prompts: ssd_sm100.cu (mLSTM), wkv_chunk.cu (WKV, GLA).
#include "../include/omni_vec.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;
constexpr float kL2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------------ gates
struct MlstmGateParams {
  const float* z;            // [T, z_ld]: input gate of head h at column h, forget gate at f_col + h, before the biases
  int z_ld, f_col;
  const float *ib, *fb;      // [H]
  float cap;
  float* m_state;            // [slots, H]
  const int* cu_q;
  const int64_t* positions;
  const int* state_slots;
  int H;
  float2* ka;                // [T, H] keep, add
  float* m;                  // [T, H]
  float* den;                // [T, H], zeroed: where the chunked form adds up n . q
  // chunks of 128 tokens (null: not wanted); chunk c of request r is row cu_q[r] / 128 + r + c; all in log2 units
  float *row, *cp, *g;       // [chunks, H, 128]: b - m, b - i, and 2^(-cp - gmax of its block of 32), b the sum of f in the chunk
  float* gmax;               // [chunks, H, 4]
  float* m_in;               // [chunks, H]: m before the chunk
};

__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

__global__ void mlstm_gates_step_kernel(const MlstmGateParams p, int rows) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * p.H) return;
  const int t = i / p.H, h = i % p.H, slot = p.state_slots[t];
  float keep = 0.f, add = 0.f, m = 0.f;
  if (slot >= 0) {
    const float gi = p.cap * tanhf((p.z[(size_t)t * p.z_ld + h] + p.ib[h]) / p.cap);
    const float gf = log_sigmoid(p.cap * tanhf((p.z[(size_t)t * p.z_ld + p.f_col + h] + p.fb[h]) / p.cap));
    float* ms = p.m_state + (size_t)slot * p.H + h;
    const float old = gf + (p.positions[t] == 0 ? 0.f : *ms);
    m = fmaxf(old, gi);
    keep = expf(old - m);
    add = expf(gi - m);
    *ms = m;
  }
  p.ka[i] = make_float2(keep, add);
  p.m[i] = m;
}

constexpr int GT_THREADS = 512;      // four chunks at a time
__global__ void __launch_bounds__(GT_THREADS) mlstm_gates_kernel(const MlstmGateParams p) {
  const int h = blockIdx.x, r = blockIdx.y;
  const int row0 = p.cu_q[r], n_rows = p.cu_q[r + 1] - row0, slot = p.state_slots[r];
  if (n_rows <= 0) return;
  const int i = threadIdx.x, warp = i >> 5, lane = i & 31, ch = i >> 7;
  __shared__ float2 wtot[16];
  __shared__ float2 ctot[4];
  __shared__ float ms[GT_THREADS];
  float carry = (slot >= 0 && p.positions[row0] != 0) ? p.m_state[(size_t)slot * p.H + h] : 0.f;
  for (int base = 0; base < n_rows; base += GT_THREADS) {
    const int t = base + i;
    const bool ok = t < n_rows;
    float f = 0.f, gi = -INFINITY;
    if (ok) {
      const float* z = p.z + (size_t)(row0 + t) * p.z_ld;
      gi = p.cap * tanhf((z[h] + p.ib[h]) / p.cap);
      f = log_sigmoid(p.cap * tanhf((z[p.f_col + h] + p.fb[h]) / p.cap));
    }
    // (F, M): sum of f, and the largest i plus the f after it
    float F = f, M = gi;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float F1 = __shfl_up_sync(0xffffffffu, F, o), M1 = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) { M = fmaxf(M1 + F, M); F += F1; }
    }
    if (lane == 31) wtot[warp] = make_float2(F, M);
    __syncthreads();
    {
      float Fp = 0.f, Mp = -INFINITY;
      for (int w = ch * 4; w < warp; ++w) { Mp = fmaxf(Mp + wtot[w].x, wtot[w].y); Fp += wtot[w].x; }
      M = fmaxf(Mp + F, M);
      F += Fp;
    }
    if ((i & 127) == 127) ctot[ch] = make_float2(F, M);
    __syncthreads();
    float m_in = carry;
    for (int c = 0; c < ch; ++c) m_in = fmaxf(m_in + ctot[c].x, ctot[c].y);
    const float m = fmaxf(m_in + F, M);
    ms[i] = m;
    __syncthreads();
    const float before = (i & 127) ? ms[i - 1] : m_in;
    if (ok) {
      const size_t at = (size_t)(row0 + t) * p.H + h;
      p.ka[at] = make_float2(expf(f + before - m), expf(gi - m));
      p.m[at] = m;
      p.den[at] = 0.f;
    }
    if (p.row != nullptr && base + ch * 128 < n_rows) {      // uniform per warp
      const size_t chunk = ((size_t)(row0 / 128 + r + base / 128 + ch) * p.H + h);
      const float c = -((F - gi) * kL2e);                    // -inf for rows past the end
      float mx = c;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      mx = fmaxf(mx, -1e30f);
      p.row[chunk * 128 + (i & 127)] = (F - m) * kL2e;
      p.cp[chunk * 128 + (i & 127)] = -c;
      p.g[chunk * 128 + (i & 127)] = exp2f(c - mx);
      if (lane == 0) p.gmax[chunk * 4 + (warp & 3)] = mx;
      if ((i & 127) == 0) p.m_in[chunk] = m_in * kL2e;
    }
    carry = ms[GT_THREADS - 1];
    __syncthreads();
  }
  if (i == 0 && slot >= 0) p.m_state[(size_t)slot * p.H + h] = carry;
}

// ------------------------------------------------------------------------------------------------ token by token
struct StateParams {
  const void *a, *b, *v;     // query, key [T, ld] with head h at column h N, value with head h at column h P
  int a_ld, b_ld, v_ld;
  float a_scale;             // mLSTM, GLA: multiplies the query
  const float2* ka;          // mLSTM [T, H]
  float* den;                // mLSTM [T, H]: n . q
  const float* z;            // WKV, GLA [T, z_ld]
  int z_ld;
  const float *w0, *u;       // WKV, GLA (w0 alone) [H N]
  float inv_tau;             // GLA
  float* state;
  const int* cu_q;           // [B + 1], null = one row per request
  const int64_t* positions;
  const int* state_slots;
  void* y;                   // [T, y_ld], head h at column h P
  int y_ld;
  int H, P, N;
  int max_rows;              // requests with more rows are left to another kernel (0: none are)
  int vec;                   // rows allow NV-wide loads
};

enum { ST_MLSTM = 0, ST_WKV = 1, ST_GLA = 2 };

// NV values of N per lane (VECN: neighbours, otherwise 32 apart), R rows of the state per warp.
template <typename T, int KIND, int NV, int R, bool VECN>
__global__ void __launch_bounds__(128) state_rows_kernel(const StateParams p) {
  constexpr bool MLSTM = KIND == ST_MLSTM;         // the others have a decay per channel
  const int h = blockIdx.x, r = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p0 = (blockIdx.y * 4 + warp) * R, PR = MLSTM ? p.P + 1 : p.P;
  if (p0 >= PR) return;
  const int row0 = p.cu_q ? p.cu_q[r] : r, row1 = p.cu_q ? p.cu_q[r + 1] : r + 1;
  if (row1 <= row0 || (p.max_rows > 0 && row1 - row0 > p.max_rows)) return;
  const int slot = p.state_slots[r];
  T* y = (T*)p.y;
  if (slot < 0) {
    for (int t = row0; t < row1; ++t)
      for (int i = lane; i < R; i += 32) {
        if (p0 + i < p.P) y[(size_t)t * p.y_ld + h * p.P + p0 + i] = from_f32<T>(0.f);
        if (MLSTM && p0 + i == p.P) p.den[(size_t)t * p.H + h] = 0.f;
      }
    return;
  }
  constexpr int W = NV < 4 ? NV : 4;              // vector width of the state
  float* st = p.state + (((size_t)slot * p.H + h) * PR + p0) * p.N;
  auto n_of = [&](int i) { return VECN ? lane * NV + i : i * 32 + lane; };
  float S[R][NV];
  const bool fresh = p.positions[row0] == 0;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    if constexpr (VECN) {
#pragma unroll
      for (int j = 0; j < NV; j += W) {
        float v[W];
#pragma unroll
        for (int e = 0; e < W; ++e) v[e] = 0.f;
        if (!fresh && p0 + i < PR && lane * NV < p.N) load_vec<W>(st + (size_t)i * p.N + lane * NV + j, v);
#pragma unroll
        for (int e = 0; e < W; ++e) S[i][j + e] = v[e];
      }
    } else {
#pragma unroll
      for (int j = 0; j < NV; ++j) S[i][j] = (!fresh && p0 + i < PR && n_of(j) < p.N) ? st[(size_t)i * p.N + n_of(j)] : 0.f;
    }
  }
  float w0[MLSTM ? 1 : NV], u[KIND == ST_WKV ? NV : 1];
  if constexpr (!MLSTM) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const bool in = n_of(j) < p.N;
      w0[j] = in ? p.w0[h * p.N + n_of(j)] : 0.f;
      if constexpr (KIND == ST_WKV) u[j] = in ? p.u[h * p.N + n_of(j)] : 0.f;
    }
  }
  struct Tok {
    float a[NV], b[NV], z[MLSTM ? 1 : NV], x;
    float2 ka;
  };
  auto fetch = [&](int t, Tok& k) {
    const T* ar = (const T*)p.a + (size_t)t * p.a_ld + h * p.N;
    const T* br = (const T*)p.b + (size_t)t * p.b_ld + h * p.N;
    const float* zr = MLSTM ? nullptr : p.z + (size_t)t * p.z_ld + h * p.N;
    bool done = false;
    if constexpr (VECN && NV <= 4) {
      if (p.vec) {
        done = true;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          k.a[j] = k.b[j] = 0.f;
          if constexpr (!MLSTM) k.z[j] = 0.f;
        }
        if (lane * NV < p.N) {
          load_vec<NV>(ar + lane * NV, k.a);
          load_vec<NV>(br + lane * NV, k.b);
          if constexpr (!MLSTM) load_vec<NV>(zr + lane * NV, k.z);
        }
      }
    }
    if (!done) {
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const bool in = n_of(j) < p.N;
        k.a[j] = in ? to_f32(ar[n_of(j)]) : 0.f;
        k.b[j] = in ? to_f32(br[n_of(j)]) : 0.f;
        if constexpr (!MLSTM) k.z[j] = in ? zr[n_of(j)] : 0.f;
      }
    }
    const int pr = p0 + lane;                      // lane i holds the value of row i
    k.x = (lane < R && pr < p.P) ? to_f32(((const T*)p.v)[(size_t)t * p.v_ld + h * p.P + pr]) : 0.f;
    if constexpr (MLSTM) {
      if (lane < R && pr == p.P) k.x = 1.f;
      k.ka = p.ka[(size_t)t * p.H + h];
    }
  };
  Tok cur, nxt;
  fetch(row0, cur);
  for (int t = row0; t < row1; ++t) {
    if (t + 1 < row1) fetch(t + 1, nxt);
    float v[R];
    if constexpr (KIND == ST_GLA) {
      float dec[NV];
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        dec[j] = expf(log_sigmoid(cur.z[j] + w0[j]) * p.inv_tau);
        cur.a[j] *= p.a_scale;
      }
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const float x = __shfl_sync(0xffffffffu, cur.x, i);
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          S[i][j] = fmaf(dec[j], S[i][j], x * cur.b[j]);
          s = fmaf(S[i][j], cur.a[j], s);
        }
        v[i] = s;
      }
    } else if constexpr (KIND == ST_WKV) {
      float dec[NV], uk = 0.f;
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        dec[j] = expf(-expf(cur.z[j] + w0[j]));
        uk = fmaf(u[j] * cur.b[j], cur.a[j], uk);
      }
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const float x = __shfl_sync(0xffffffffu, cur.x, i);
        float s = x * uk;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          s = fmaf(S[i][j], cur.a[j], s);
          S[i][j] = fmaf(dec[j], S[i][j], x * cur.b[j]);
        }
        v[i] = s;
      }
    } else {
#pragma unroll
      for (int j = 0; j < NV; ++j) cur.a[j] *= p.a_scale;
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const float x = cur.ka.y * __shfl_sync(0xffffffffu, cur.x, i);
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          S[i][j] = fmaf(cur.ka.x, S[i][j], x * cur.b[j]);
          s = fmaf(S[i][j], cur.a[j], s);
        }
        v[i] = s;
      }
    }
    // sum over the lanes; halving the number of values with each of the first steps leaves row i in the lanes whose
    // leading bits are i
    int o = 16;
#pragma unroll
    for (int n = R; n > 1; n >>= 1, o >>= 1) {
      const bool up = (lane & o) != 0;
#pragma unroll
      for (int i = 0; i < n / 2; ++i) {
        const float send = up ? v[i] : v[i + n / 2];
        const float mine = up ? v[i + n / 2] : v[i];
        v[i] = mine + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    float s = v[0];
    for (; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    const int i = lane / (32 / R);
    if (lane % (32 / R) == 0) {
      if (p0 + i < p.P) y[(size_t)t * p.y_ld + h * p.P + p0 + i] = from_f32<T>(s);
      if (MLSTM && p0 + i == p.P) p.den[(size_t)t * p.H + h] = s;
    }
    cur = nxt;
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    if (p0 + i >= PR) break;
    if constexpr (VECN) {
      if (lane * NV < p.N) {
#pragma unroll
        for (int j = 0; j < NV; j += W) {
          float v[W];
#pragma unroll
          for (int e = 0; e < W; ++e) v[e] = S[i][j + e];
          store_vec<W>(st + (size_t)i * p.N + lane * NV + j, v);
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < NV; ++j)
        if (n_of(j) < p.N) st[(size_t)i * p.N + n_of(j)] = S[i][j];
    }
  }
}

template <typename T, int KIND>
static int launch_state_rows(StateParams p, int B, cudaStream_t stream) {
  const int PR = KIND == ST_MLSTM ? p.P + 1 : p.P;
#define ST_CASE(NV, R, VECN)                                                                                              \
  {                                                                                                                       \
    const uintptr_t al = NV * sizeof(T) - 1;                                                                              \
    p.vec = VECN && p.N % NV == 0 && ((p.a_ld | p.b_ld) % NV) == 0 && (((uintptr_t)p.a | (uintptr_t)p.b) & al) == 0 &&     \
            (KIND == ST_MLSTM || (p.z_ld % NV == 0 && ((uintptr_t)p.z & (NV * 4 - 1)) == 0));                                          \
    const dim3 grid(p.H, (PR + 4 * R - 1) / (4 * R), B);                                                                  \
    state_rows_kernel<T, KIND, NV, R, VECN><<<grid, 128, 0, stream>>>(p);                                                  \
    return (int)cudaGetLastError();                                                                                       \
  }
  if (p.N <= 32) ST_CASE(1, 8, true)
  if (p.N <= 64 && p.N % 2 == 0) ST_CASE(2, 8, true)
  if (p.N <= 64) ST_CASE(2, 8, false)
  if (p.N <= 128 && p.N % 4 == 0) ST_CASE(4, 8, true)
  if (p.N <= 128) ST_CASE(4, 8, false)
  if (p.N <= 256 && p.N % 8 == 0) ST_CASE(8, 4, true)
  if (p.N <= 256) ST_CASE(8, 4, false)
  if (p.N <= 1024) ST_CASE(32, 2, false)
#undef ST_CASE
  return -3;
}

// ------------------------------------------------------------------------------------------------ norm and gate
// LANES lanes per (token, head).  ACT 0: sigmoid gate, 1: silu gate.
template <typename T, int V, int LANES, int ACT>
__global__ void __launch_bounds__(256) head_norm_kernel(const T* __restrict__ y, int y_ld, const float* __restrict__ den,
                                                        const float* __restrict__ m, const T* __restrict__ gate, int gate_ld,
                                                        const float* __restrict__ w, float scale, T* __restrict__ out, int out_ld,
                                                        int rows, int H, int P, float eps) {
  const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / LANES;
  const int lane = threadIdx.x & (LANES - 1);
  const bool ok = item < (long long)rows * H;            // every lane takes part in the sums
  const int t = ok ? (int)(item / H) : 0, h = ok ? (int)(item % H) : 0;
  const T* yr = y + (size_t)t * y_ld + h * P;
  const T* gr = gate + (size_t)t * gate_ld + h * P;
  T* o = out + (size_t)t * out_ld + h * P;
  const float div = (ok && den) ? 1.0f / (fmaxf(fabsf(den[item]), expf(-m[item])) + 1e-6f) : 1.0f;
  float first[V], ss = 0.f;                              // the first vector stays in registers
#pragma unroll
  for (int i = 0; i < V; ++i) first[i] = 0.f;
  if (ok && lane * V < P) load_vec<V>(yr + lane * V, first);
#pragma unroll
  for (int i = 0; i < V; ++i) { first[i] *= div; ss += first[i] * first[i]; }
  for (int c = (LANES + lane) * V; ok && c < P; c += LANES * V) {
    float v[V];
    load_vec<V>(yr + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) { v[i] *= div; ss += v[i] * v[i]; }
  }
#pragma unroll
  for (int s = LANES / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!ok) return;
  const float r = 1.0f / sqrtf(ss / (float)P + eps) * scale;
  auto finish = [&](int c, const float (&v)[V]) {
    float g[V], g2[V], a[V];
    load_vec<V>(gr + c, g);
    load_vec<V>(w + h * P + c, g2);
#pragma unroll
    for (int i = 0; i < V; ++i)
      a[i] = v[i] * r * g2[i] * (ACT == 0 ? div_for<T>(1.0f, 1.0f + exp_for<T>(-g[i])) : silu_for<T>(g[i]));
    store_vec<V>(o + c, a);
  };
  if (lane * V < P) finish(lane * V, first);
  for (int c = (LANES + lane) * V; c < P; c += LANES * V) {
    float v[V];
    load_vec<V>(yr + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] *= div;
    finish(c, v);
  }
}

}  // namespace omni

using namespace omni;

extern "C" int omni_mlstm_gates(const float* z, int z_ld, int f_col, const void* ib, const void* fb, float cap, void* m_state,
                                const int* cu_q, const int64_t* positions, const int* state_slots, int B, int rows, int H, void* ka,
                                float* m, float* den, float* chunks, int n_chunks, cudaStream_t st) {
  if (B <= 0 || rows <= 0) return 0;
  if (H < 1 || B > 65535 || !(cap > 0.f)) return -1;
  MlstmGateParams p = {z, z_ld, f_col, (const float*)ib, (const float*)fb, cap, (float*)m_state, cu_q, positions, state_slots, H,
                       (float2*)ka, m, den, nullptr, nullptr, nullptr, nullptr, nullptr};
  if (cu_q == nullptr) {
    mlstm_gates_step_kernel<<<(rows * H + 255) / 256, 256, 0, st>>>(p, rows);
    return (int)cudaGetLastError();
  }
  if (chunks != nullptr) {
    const size_t a = (size_t)n_chunks * H * 128;
    p.row = chunks; p.cp = chunks + a; p.g = chunks + 2 * a; p.gmax = chunks + 3 * a; p.m_in = p.gmax + (size_t)n_chunks * H * 4;
  }
  mlstm_gates_kernel<<<dim3(H, B), GT_THREADS, 0, st>>>(p);
  return (int)cudaGetLastError();
}

// kind 0: mLSTM (ka, den), 1: WKV (z, w0, u), 2: GLA (z, w0, inv_tau).
extern "C" int omni_state_rows(int kind, const void* a, int a_ld, float a_scale, const void* b, int b_ld, const void* v, int v_ld,
                               const void* ka, float* den, const float* z, int z_ld, const void* w0, const void* u, float inv_tau,
                               void* state, const int* cu_q, const int64_t* positions, const int* state_slots, int B, void* y, int y_ld,
                               int H, int P, int N, int f32, int max_rows, cudaStream_t st) {
  if (B <= 0) return 0;
  if (H < 1 || P < 1 || N < 1 || B > 65535 || P > 65535 * 8 || kind < 0 || kind > 2) return -1;
  StateParams p = {a, b, v, a_ld, b_ld, v_ld, a_scale, (const float2*)ka, den, z, z_ld, (const float*)w0, (const float*)u,
                   inv_tau, (float*)state, cu_q, positions, state_slots, y, y_ld, H, P, N, max_rows, 0};
  if (kind == ST_MLSTM) return f32 ? launch_state_rows<float, ST_MLSTM>(p, B, st) : launch_state_rows<bf16, ST_MLSTM>(p, B, st);
  if (kind == ST_WKV) return f32 ? launch_state_rows<float, ST_WKV>(p, B, st) : launch_state_rows<bf16, ST_WKV>(p, B, st);
  return f32 ? launch_state_rows<float, ST_GLA>(p, B, st) : launch_state_rows<bf16, ST_GLA>(p, B, st);
}

// y, gate, out: head h at column h P of rows of their pitches.  den / m [T, H] null: y is what is normed.  act 0 sigmoid, 1 silu.
extern "C" int omni_head_norm(const void* y, int y_ld, const float* den, const float* m, const void* gate, int gate_ld,
                              const void* w, float scale, void* out, int out_ld, int rows, int H, int P, float eps, int act, int f32,
                              cudaStream_t st) {
  if (rows <= 0) return 0;
  if (H < 1 || P < 1 || act < 0 || act > 1) return -1;
  const size_t esz = f32 ? 4 : 2;
  const bool v8 = P % 8 == 0 && y_ld % 8 == 0 && gate_ld % 8 == 0 && out_ld % 8 == 0 &&
                  (((uintptr_t)y | (uintptr_t)gate | (uintptr_t)out) & (esz == 4 ? 15 : 8 * esz - 1)) == 0;
#define HEAD_NORM(T, V, LANES, ACT)                                                                                            \
  head_norm_kernel<T, V, LANES, ACT><<<(unsigned)(((long long)rows * H * LANES + 255) / 256), 256, 0, st>>>(                   \
      (const T*)y, y_ld, den, m, (const T*)gate, gate_ld, (const float*)w, scale, (T*)out, out_ld, rows, H, P, eps)
#define HEAD_NORM_V(T, ACT)                            \
  do {                                                 \
    if (!v8) HEAD_NORM(T, 1, 32, ACT);                 \
    else if (P <= 64) HEAD_NORM(T, 8, 8, ACT);         \
    else if (P <= 128) HEAD_NORM(T, 8, 16, ACT);       \
    else HEAD_NORM(T, 8, 32, ACT);                     \
  } while (0)
  if (f32) { if (act == 0) HEAD_NORM_V(float, 0); else HEAD_NORM_V(float, 1); }
  else { if (act == 0) HEAD_NORM_V(bf16, 0); else HEAD_NORM_V(bf16, 1); }
#undef HEAD_NORM_V
#undef HEAD_NORM
  return (int)cudaGetLastError();
}
