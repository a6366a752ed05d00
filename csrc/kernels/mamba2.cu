// Mamba-2 (state-space duality) layer between its two projections.
//
// The input projection's rows are [z: inner | x: inner | B: G N | C: G N | dt: heads], inner = heads * P.
// x, B, C go through the short convolution of short_conv.cu first.
//   omni_ssm_scan         the recurrence  S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x  with
//                         dt = softplus(dt + dt_bias), S fp32 in the request's slot
//   omni_gated_group_norm y * silu(z), RMSNorm in equal parts, weight
//
// State slots: [slots, heads, P, N] fp32.  A request whose first
// token of the call is at position 0 starts from zeros whatever its slot holds; a row with a negative slot is padding.
//
// The scan has two forms here.
//   ssm_rows_kernel   token by token, the state in registers: a warp owns a few rows of P, N lies across its lanes.  One
//                     token per request (decode) makes it a stream over the state; it also is the fp32 path and takes the
//                     shapes the other form does not.
//   ssd_chunk_kernel  portions of prompts, bf16, states of more than 128 (up to that size ssd_sm100.cu runs the same scheme
//                     on tcgen05): chunks of 64 tokens,
//                       Y = (C B^T o L) (dt x) + exp(cum) C S,   S <- exp(cum_end) S + B^T (exp(cum_end - cum) dt x)
//                     with L_ij = exp(cum_i - cum_j) for j <= i and cum the running sum of -exp(A_log) dt in the chunk.
//                     One CTA walks the chunks of one (request, head, 32 columns of P); S stays in fp32 accumulators.
//                     Every fp32 operand (the decayed scores, S, the decayed inputs) enters its MMA as a pair of bf16
//                     values hi + lo, so products keep 16 bits of mantissa on that side; C, B and x are bf16 as stored.
#include "../include/omni_vec.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// ------------------------------------------------------------------------------------------------ recurrence by rows
struct SsmParams {
  const void* xbc;        // [T, xbc_ld] = x | B | C after the convolution
  int xbc_ld;
  const void* dt;         // dt of head h of row t: dt[t * dt_ld + h], before bias and softplus
  int dt_ld;
  const float* A_log;
  const float* dt_bias;
  const float* D;
  float* state;           // [slots, H, P, N]
  const int* cu_q;        // [B + 1], null = one row per request
  const int64_t* positions;
  const int* state_slots;
  void* y;                // [T, y_ld]
  int y_ld;
  int H, P, N, G;
  int max_rows;           // requests with more rows are left to another kernel (0: none are)
};

// NV values of N per lane.  VECN: a lane's values are neighbours (N a multiple of NV, 16-byte accesses); otherwise they are
// 32 apart.  R rows of P per warp.
template <typename T, int NV, int R, bool VECN>
__global__ void __launch_bounds__(128) ssm_rows_kernel(const SsmParams p) {
  const int h = blockIdx.x, r = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p0 = (blockIdx.y * 4 + warp) * R;
  if (p0 >= p.P) return;
  const int row0 = p.cu_q ? p.cu_q[r] : r, row1 = p.cu_q ? p.cu_q[r + 1] : r + 1;
  if (row1 <= row0 || (p.max_rows > 0 && row1 - row0 > p.max_rows)) return;
  const int slot = p.state_slots[r];
  const int inner = p.H * p.P, g = h / (p.H / p.G);
  const T* xbc = (const T*)p.xbc;
  T* y = (T*)p.y;
  if (slot < 0) {
    for (int t = row0; t < row1; ++t)
      for (int i = lane; i < R; i += 32)
        if (p0 + i < p.P) y[(size_t)t * p.y_ld + h * p.P + p0 + i] = from_f32<T>(0.f);
    return;
  }
  constexpr int W = NV < 4 ? NV : 4;              // vector width
  float* st = p.state + (((size_t)slot * p.H + h) * p.P + p0) * p.N;
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
        if (!fresh && p0 + i < p.P && lane * NV < p.N) load_vec<W>(st + (size_t)i * p.N + lane * NV + j, v);
#pragma unroll
        for (int e = 0; e < W; ++e) S[i][j + e] = v[e];
      }
    } else {
#pragma unroll
      for (int j = 0; j < NV; ++j)
        S[i][j] = (!fresh && p0 + i < p.P && n_of(j) < p.N) ? st[(size_t)i * p.N + n_of(j)] : 0.f;
    }
  }
  const float a = -expf(p.A_log[h]), bias = p.dt_bias[h], Dh = p.D[h];
  for (int t = row0; t < row1; ++t) {
    const T* row = xbc + (size_t)t * p.xbc_ld;
    const float dt = softplus_f(to_f32(((const T*)p.dt)[(size_t)t * p.dt_ld + h]) + bias);
    const float decay = expf(a * dt);
    float Bv[NV], Cv[NV];
    const T* Br = row + inner + g * p.N;
    const T* Cr = Br + p.G * p.N;
    if constexpr (VECN && NV <= 4) {
#pragma unroll
      for (int j = 0; j < NV; ++j) Bv[j] = Cv[j] = 0.f;
      if (lane * NV < p.N) {
        if (((p.N | inner | p.xbc_ld) & (NV - 1)) == 0) {
          load_vec<NV>(Br + lane * NV, Bv);
          load_vec<NV>(Cr + lane * NV, Cv);
        } else {
#pragma unroll
          for (int j = 0; j < NV; ++j) { Bv[j] = to_f32(Br[lane * NV + j]); Cv[j] = to_f32(Cr[lane * NV + j]); }
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const bool in = n_of(j) < p.N;
        Bv[j] = in ? to_f32(Br[n_of(j)]) : 0.f;
        Cv[j] = in ? to_f32(Cr[n_of(j)]) : 0.f;
      }
    }
    // lane i holds x of row i
    const float xl = (lane < R && p0 + lane < p.P) ? to_f32(row[h * p.P + p0 + lane]) : 0.f;
    float out[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const float w = dt * __shfl_sync(0xffffffffu, xl, i);
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        S[i][j] = fmaf(decay, S[i][j], w * Bv[j]);
        s = fmaf(S[i][j], Cv[j], s);
      }
      out[i] = s;
    }
    // sum over the lanes; halving the number of values with each of the first steps leaves row i in the lanes whose
    // leading bits are i
    float v[R];
#pragma unroll
    for (int i = 0; i < R; ++i) v[i] = out[i];
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
    const float xi = __shfl_sync(0xffffffffu, xl, i);
    if (lane % (32 / R) == 0 && p0 + i < p.P)
      y[(size_t)t * p.y_ld + h * p.P + p0 + i] = from_f32<T>(fmaf(Dh, xi, s));
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    if (p0 + i >= p.P) break;
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

template <typename T>
static int launch_ssm_rows(const SsmParams& p, int B, cudaStream_t stream) {
#define SSM_CASE(NV, R, VECN)                                                     \
  {                                                                               \
    const dim3 grid(p.H, (p.P + 4 * R - 1) / (4 * R), B);                         \
    ssm_rows_kernel<T, NV, R, VECN><<<grid, 128, 0, stream>>>(p);                 \
    return (int)cudaGetLastError();                                               \
  }
  if (p.N <= 32) SSM_CASE(1, 8, true)
  if (p.N <= 64 && p.N % 2 == 0) SSM_CASE(2, 8, true)
  if (p.N <= 64) SSM_CASE(2, 8, false)
  if (p.N <= 128 && p.N % 4 == 0) SSM_CASE(4, 8, true)
  if (p.N <= 128) SSM_CASE(4, 8, false)
  if (p.N <= 256 && p.N % 8 == 0) SSM_CASE(8, 4, true)
  if (p.N <= 256) SSM_CASE(8, 4, false)
  if (p.N <= 1024) SSM_CASE(32, 2, false)
#undef SSM_CASE
  return -3;
}

// ------------------------------------------------------------------------------------------------ chunked scan
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (a, b) -> packed bf16 pair and the packed remainder
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

constexpr int SD_Q = 64, SD_PT = 32;
// byte offset of 16-byte chunk `ch` of a row, rotated so that ldmatrix reads are free of bank conflicts
template <int ROWB>
__device__ __forceinline__ uint32_t sd_off(int row, int ch) {
  return (uint32_t)(row * ROWB) + (uint32_t)((ROWB >= 128 ? (ch ^ (row & 7)) : (ch ^ ((row >> 1) & 3))) << 4);
}

template <int NP>
struct SdSmem {
  static constexpr int BC = SD_Q * NP * 2, X = SD_Q * SD_PT * 2, S = NP * SD_PT * 2;
  static constexpr int STAGE = 2 * BC + X;              // B, C, x of one chunk
  static constexpr int W_OFF = 2 * STAGE, S_OFF = W_OFF + 2 * X;
  static constexpr int F_OFF = S_OFF + 2 * S;           // cum[64], dt[64], warp total
  static constexpr int TOTAL = F_OFF + (3 * SD_Q + 4) * 4;
};

template <int NP>
__global__ void __launch_bounds__(128) ssd_chunk_kernel(const SsmParams p) {
  extern __shared__ __align__(128) uint8_t sd_smem[];
  using L = SdSmem<NP>;
  const int pt = blockIdx.x, h = blockIdx.y, r = blockIdx.z;
  const int row0 = p.cu_q[r], n_rows = p.cu_q[r + 1] - row0;
  const int slot = p.state_slots[r];
  if (n_rows <= 0 || slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int p0 = pt * SD_PT, pw = min(SD_PT, p.P - p0);
  const int inner = p.H * p.P, g = h / (p.H / p.G);
  const bf16* xbc = (const bf16*)p.xbc + (size_t)row0 * p.xbc_ld;
  const bf16* dtp = (const bf16*)p.dt + (size_t)row0 * p.dt_ld + h;
  const int n_chunks = (n_rows + SD_Q - 1) / SD_Q;
  const uint32_t base = smem_addr(sd_smem);
  float* cum = reinterpret_cast<float*>(sd_smem + L::F_OFF);   // log2 units
  float* dts = cum + SD_Q;
  float* ecum = dts + SD_Q;                                    // exp of the running sum
  float* wtot = ecum + SD_Q;

  auto load_chunk = [&](int c) {
    const uint32_t sb = base + (c & 1) * L::STAGE, sc = sb + L::BC, sx = sc + L::BC;
    const int t0 = c * SD_Q;
    constexpr int CH = NP / 8;
    for (int i = tid; i < SD_Q * CH; i += 128) {
      const int row = i / CH, ch = i % CH;
      const bool ok = t0 + row < n_rows && ch * 8 < p.N;
      const bf16* src = xbc + (size_t)(ok ? t0 + row : 0) * p.xbc_ld + inner + g * p.N + (ok ? ch * 8 : 0);
      cp_async16(sb + sd_off<NP * 2>(row, ch), src, ok);
      cp_async16(sc + sd_off<NP * 2>(row, ch), src + p.G * p.N, ok);
    }
    for (int i = tid; i < SD_Q * (SD_PT / 8); i += 128) {
      const int row = i / (SD_PT / 8), ch = i % (SD_PT / 8);
      const bool ok = t0 + row < n_rows && ch * 8 < pw;
      const bf16* src = xbc + (size_t)(ok ? t0 + row : 0) * p.xbc_ld + h * p.P + p0 + (ok ? ch * 8 : 0);
      cp_async16(sx + sd_off<SD_PT * 2>(row, ch), src, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_dt = [&](int c) -> float {       // threads 0..63: dt of the chunk's token, rows past the end count as -inf
    const int t = c * SD_Q + tid;
    return (tid < SD_Q && t < n_rows) ? __bfloat162float(dtp[(size_t)t * p.dt_ld]) : -INFINITY;
  };

  // state accumulators: rows n = warp * NP/4 + mt * 16 + (lane / 4) (+ 8), columns p = nt * 8 + (lane % 4) * 2 (+ 1)
  constexpr int MT = NP / 64;
  float S[MT][4][4];
  const int lg = lane >> 2, lc = (lane & 3) * 2;
  float* st = p.state + (((size_t)slot * p.H + h) * p.P + p0) * p.N;
  const bool fresh = p.positions[row0] == 0;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = warp * (NP / 4) + mt * 16 + lg + (e >> 1) * 8, pc = nt * 8 + lc + (e & 1);
        S[mt][nt][e] = (!fresh && n < p.N && pc < pw) ? st[(size_t)pc * p.N + n] : 0.f;
      }

  const float a2 = -expf(p.A_log[h]) * kLog2e, bias = p.dt_bias[h], Dh = p.D[h];
  load_chunk(0);
  float dt_raw = load_dt(0);
  for (int c = 0; c < n_chunks; ++c) {
    const bool more = c + 1 < n_chunks;
    if (more) load_chunk(c + 1);
    // ---- dt and the running decay (warps 0 and 1), S as bf16 pairs in shared memory (all warps)
    const float dt = (tid < SD_Q && dt_raw != -INFINITY) ? softplus_f(dt_raw + bias) : 0.f;
    if (more) dt_raw = load_dt(c + 1);
    float run = a2 * dt;
    if (warp < 2) {
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      if (warp == 0 && lane == 31) wtot[0] = run;
    }
    const uint32_t sh = base + L::S_OFF, sl = sh + L::S;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split2(S[mt][nt][half * 2], S[mt][nt][half * 2 + 1], hi, lo);
          const int n = warp * (NP / 4) + mt * 16 + lg + half * 8;
          const uint32_t off = sd_off<SD_PT * 2>(n, nt) + lc * 2;
          asm volatile("st.shared.b32 [%0], %1;" ::"r"(sh + off), "r"(hi) : "memory");
          asm volatile("st.shared.b32 [%0], %1;" ::"r"(sl + off), "r"(lo) : "memory");
        }
    if (more) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (warp < 2) {
      if (warp == 1) run += wtot[0];
      cum[tid] = run;
      dts[tid] = dt;
      ecum[tid] = exp2f(run);
    }
    __syncthreads();
    const uint32_t sb = base + (c & 1) * L::STAGE, sc = sb + L::BC, sx = sc + L::BC;
    const float cend = cum[SD_Q - 1];
    // ---- decayed inputs exp(cum_end - cum) dt x as bf16 pairs
    const uint32_t swh = base + L::W_OFF, swl = swh + L::X;
    for (int i = tid; i < SD_Q * (SD_PT / 8); i += 128) {
      const int row = i / (SD_PT / 8);
      const uint32_t off = sd_off<SD_PT * 2>(row, i % (SD_PT / 8));
      const float wt = exp2f(cend - cum[row]) * dts[row];
      uint32_t v[4], hi[4], lo[4];
      asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(sx + off));
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v[e]));
        split2(f.x * wt, f.y * wt, hi[e], lo[e]);
      }
      asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(swh + off), "r"(hi[0]), "r"(hi[1]), "r"(hi[2]), "r"(hi[3]) : "memory");
      asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(swl + off), "r"(lo[0]), "r"(lo[1]), "r"(lo[2]), "r"(lo[3]) : "memory");
    }
    // ---- this warp's 16 rows: scores C B^T (key tiles up to the diagonal) and C S
    float sc_acc[8][4], y[4][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) sc_acc[j][0] = sc_acc[j][1] = sc_acc[j][2] = sc_acc[j][3] = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
    const int arow = warp * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll 2
    for (int ks = 0; ks < NP / 16; ++ks) {
      uint32_t ca[4];
      ldsm_x4(sc + sd_off<NP * 2>(arow, ks * 2 + (lane >> 4)), ca);
#pragma unroll
      for (int jp = 0; jp < 4; ++jp) {                 // pairs of 8-key tiles = 16 keys
        if (jp <= warp) {
          uint32_t kb[4];
          const int krow = jp * 16 + (lane >> 4) * 8 + (lane & 7);
          ldsm_x4(sb + sd_off<NP * 2>(krow, ks * 2 + ((lane >> 3) & 1)), kb);
          mma16816(sc_acc[2 * jp], ca, kb[0], kb[1]);
          mma16816(sc_acc[2 * jp + 1], ca, kb[2], kb[3]);
        }
      }
      const int srow = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
      for (int jp = 0; jp < 2; ++jp) {
        const uint32_t off = sd_off<SD_PT * 2>(srow, jp * 2 + (lane >> 4));
        uint32_t sv[4];
        ldsm_x4_trans(sh + off, sv);
        mma16816(y[2 * jp], ca, sv[0], sv[1]);
        mma16816(y[2 * jp + 1], ca, sv[2], sv[3]);
        ldsm_x4_trans(sl + off, sv);
        mma16816(y[2 * jp], ca, sv[0], sv[1]);
        mma16816(y[2 * jp + 1], ca, sv[2], sv[3]);
      }
    }
    const int i0 = warp * 16 + lg, i1 = i0 + 8;        // this thread's rows of the chunk
    const float c0 = cum[i0], c1 = cum[i1], e0 = ecum[i0], e1 = ecum[i1];
#pragma unroll
    for (int j = 0; j < 4; ++j) { y[j][0] *= e0; y[j][1] *= e0; y[j][2] *= e1; y[j][3] *= e1; }
    // ---- Y += (scores o decay o dt) x
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      if (ks <= warp) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int j0 = ks * 16 + q * 8 + lc;
          const float2 cj = *reinterpret_cast<const float2*>(cum + j0), dj = *reinterpret_cast<const float2*>(dts + j0);
          const float (&s)[4] = sc_acc[2 * ks + q];
          const float m0 = j0 <= i0 ? s[0] * exp2f(c0 - cj.x) * dj.x : 0.f;
          const float m1 = j0 + 1 <= i0 ? s[1] * exp2f(c0 - cj.y) * dj.y : 0.f;
          const float m2 = j0 <= i1 ? s[2] * exp2f(c1 - cj.x) * dj.x : 0.f;
          const float m3 = j0 + 1 <= i1 ? s[3] * exp2f(c1 - cj.y) * dj.y : 0.f;
          split2(m0, m1, ah[2 * q], al[2 * q]);
          split2(m2, m3, ah[2 * q + 1], al[2 * q + 1]);
        }
        const int xrow = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
        for (int jp = 0; jp < 2; ++jp) {
          uint32_t xv[4];
          ldsm_x4_trans(sx + sd_off<SD_PT * 2>(xrow, jp * 2 + (lane >> 4)), xv);
          mma16816(y[2 * jp], ah, xv[0], xv[1]);
          mma16816(y[2 * jp + 1], ah, xv[2], xv[3]);
          mma16816(y[2 * jp], al, xv[0], xv[1]);
          mma16816(y[2 * jp + 1], al, xv[2], xv[3]);
        }
      }
    }
    // ---- + D x, out
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = half ? i1 : i0;
      if (c * SD_Q + i < n_rows) {
        bf16* yr = (bf16*)p.y + (size_t)(row0 + c * SD_Q + i) * p.y_ld + h * p.P + p0;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          if (nt * 8 + lc < pw) {
            uint32_t xr;
            asm volatile("ld.shared.b32 %0, [%1];" : "=r"(xr) : "r"(sx + sd_off<SD_PT * 2>(i, nt) + lc * 2));
            const float2 xf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&xr));
            *reinterpret_cast<__nv_bfloat162*>(yr + nt * 8 + lc) =
                __floats2bfloat162_rn(fmaf(Dh, xf.x, y[nt][half * 2]), fmaf(Dh, xf.y, y[nt][half * 2 + 1]));
          }
        }
      }
    }
    __syncthreads();                                   // the decayed inputs are complete
    // ---- S <- exp(cum_end) S + B^T W
    const float eend = ecum[SD_Q - 1];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mt][nt][e] *= eend;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t wh[2][4], wl[2][4];
      const int wrow = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
      for (int jp = 0; jp < 2; ++jp) {
        const uint32_t off = sd_off<SD_PT * 2>(wrow, jp * 2 + (lane >> 4));
        ldsm_x4_trans(swh + off, wh[jp]);
        ldsm_x4_trans(swl + off, wl[jp]);
      }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        // A = B^T: rows n, columns t; stored [t][n], so the four 8x8 blocks are (t, n), (t, n + 8), (t + 8, n), (t + 8, n + 8)
        uint32_t ba[4];
        const int trow = ks * 16 + (lane >> 4) * 8 + (lane & 7);
        const int nch = (warp * (NP / 4) + mt * 16) / 8 + ((lane >> 3) & 1);
        ldsm_x4_trans(sb + sd_off<NP * 2>(trow, nch), ba);
#pragma unroll
        for (int jp = 0; jp < 2; ++jp) {
          mma16816(S[mt][2 * jp], ba, wh[jp][0], wh[jp][1]);
          mma16816(S[mt][2 * jp + 1], ba, wh[jp][2], wh[jp][3]);
          mma16816(S[mt][2 * jp], ba, wl[jp][0], wl[jp][1]);
          mma16816(S[mt][2 * jp + 1], ba, wl[jp][2], wl[jp][3]);
        }
      }
    }
    __syncthreads();                                   // before the next chunk's buffers are written
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = warp * (NP / 4) + mt * 16 + lg + (e >> 1) * 8, pc = nt * 8 + lc + (e & 1);
        if (n < p.N && pc < pw) st[(size_t)pc * p.N + n] = S[mt][nt][e];
      }
}

template <int NP>
static int launch_ssd(const SsmParams& p, int B, cudaStream_t stream) {
  static bool configured[64] = {false};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return (int)e;
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    e = cudaFuncSetAttribute(ssd_chunk_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, SdSmem<NP>::TOTAL);
    if (e != cudaSuccess) return (int)e;
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  ssd_chunk_kernel<NP><<<dim3((p.P + SD_PT - 1) / SD_PT, p.H, B), 128, SdSmem<NP>::TOTAL, stream>>>(p);
  return (int)cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------ gate and norm
template <typename T, int V>
__global__ void gated_group_norm_kernel(const T* __restrict__ y, int y_ld, const T* __restrict__ z, int z_ld,
                                        const float* __restrict__ w, T* __restrict__ out, int out_ld, int inner, int part,
                                        float eps) {
  const int t = blockIdx.x, c0 = blockIdx.y * part;
  const T* yr = y + (size_t)t * y_ld + c0;
  const T* zr = z + (size_t)t * z_ld + c0;
  auto gate = [&](int c, float (&v)[V]) {
    float g[V];
    load_vec<V>(yr + c, v);
    load_vec<V>(zr + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] *= silu_for<T>(g[i]);
  };
  constexpr int KEEP = 2;                     // gated vectors that stay in registers between the two passes
  float keep[KEEP][V];
  float ss = 0.f;
  const int step = blockDim.x * V;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < part) {
      gate(c, keep[k]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += keep[k][i] * keep[k][i];
    }
  }
  for (int c = threadIdx.x * V + KEEP * step; c < part; c += step) {
    float v[V];
    gate(c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += v[i] * v[i];
  }
  const float r = 1.0f / sqrtf(block_sum2(ss, 0.f).x / (float)part + eps);
  auto finish = [&](int c, const float (&v)[V]) {
    float g[V], o[V];
    load_vec<V>(w + c0 + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] = v[i] * r * g[i];
    store_vec<V>(out + (size_t)t * out_ld + c0 + c, o);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = threadIdx.x * V + k * step;
    if (c < part) finish(c, keep[k]);
  }
  for (int c = threadIdx.x * V + KEEP * step; c < part; c += step) {
    float v[V];
    gate(c, v);
    finish(c, v);
  }
  if (blockIdx.y == 0)
    for (int c = inner + threadIdx.x; c < out_ld; c += blockDim.x) out[(size_t)t * out_ld + c] = from_f32<T>(0.f);
}

}  // namespace omni

using namespace omni;

// cu_q null: one row per request.  max_rows > 0: token by token, requests of up to max_rows rows only; < 0: token by token
// for all of them.
extern "C" int omni_ssm_scan(const void* xbc, int xbc_ld, const void* dt, int dt_ld, const void* A_log, const void* dt_bias,
                             const void* D, void* state, const int* cu_q, const int64_t* positions, const int* state_slots,
                             int B, void* y, int y_ld, int H, int P, int N, int G, int f32, int max_rows, cudaStream_t st) {
  if (B <= 0) return 0;
  if (H < 1 || P < 1 || N < 1 || G < 1 || H % G != 0 || B > 65535 || H > 65535) return -1;
  SsmParams p;
  p.xbc = xbc; p.xbc_ld = xbc_ld; p.dt = dt; p.dt_ld = dt_ld; p.A_log = (const float*)A_log;
  p.dt_bias = (const float*)dt_bias; p.D = (const float*)D; p.state = (float*)state; p.cu_q = cu_q; p.positions = positions;
  p.state_slots = state_slots; p.y = y; p.y_ld = y_ld; p.H = H; p.P = P; p.N = N; p.G = G; p.max_rows = max_rows > 0 ? max_rows : 0;
  const bool chunked = cu_q != nullptr && !f32 && max_rows == 0 && P % 8 == 0 && N % 8 == 0 && N > 128 && N <= 256 &&
                       xbc_ld % 8 == 0 && y_ld % 2 == 0 && (uintptr_t)xbc % 16 == 0 && (uintptr_t)y % 4 == 0;
  if (chunked) return launch_ssd<256>(p, B, st);
  return f32 ? launch_ssm_rows<float>(p, B, st) : launch_ssm_rows<bf16>(p, B, st);
}

extern "C" int omni_gated_group_norm(const void* y, int y_ld, const void* z, int z_ld, const void* w, void* out, int out_ld,
                                     int rows, int inner, int parts, float eps, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (inner < 1 || parts < 1 || inner % parts != 0 || parts > 65535 || out_ld < inner) return -1;
  const int part = inner / parts;
  const bool v8 = part % 8 == 0 && y_ld % 8 == 0 && z_ld % 8 == 0 && out_ld % 8 == 0 &&
                  (((uintptr_t)y | (uintptr_t)z | (uintptr_t)out) % 16 == 0);
  const int v = v8 ? 8 : 1;
  int th = ((part + v - 1) / v + 31) / 32 * 32;
  th = th > 256 ? 256 : th;
  const dim3 grid(rows, parts);
  const float* wf = (const float*)w;
  if (f32) {
    if (v8) gated_group_norm_kernel<float, 8><<<grid, th, 0, st>>>((const float*)y, y_ld, (const float*)z, z_ld, wf, (float*)out, out_ld, inner, part, eps);
    else gated_group_norm_kernel<float, 1><<<grid, th, 0, st>>>((const float*)y, y_ld, (const float*)z, z_ld, wf, (float*)out, out_ld, inner, part, eps);
  } else {
    if (v8) gated_group_norm_kernel<bf16, 8><<<grid, th, 0, st>>>((const bf16*)y, y_ld, (const bf16*)z, z_ld, wf, (bf16*)out, out_ld, inner, part, eps);
    else gated_group_norm_kernel<bf16, 1><<<grid, th, 0, st>>>((const bf16*)y, y_ld, (const bf16*)z, z_ld, wf, (bf16*)out, out_ld, inner, part, eps);
  }
  return (int)cudaGetLastError();
}
