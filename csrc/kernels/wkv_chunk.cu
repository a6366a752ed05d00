// Recurrences with a decay per head and key channel over portions of prompts, bf16 activations (matrix_state.cu holds the
// token-by-token forms):
//   WKV  o_t = (S + diag(u) k_t v_t^T)^T r_t, S <- diag(w_t) S + k_t v_t^T with w = exp(-exp(z + w0)); head sizes up to 128 that are
//        multiples of 8
//   GLA  S <- diag(w_t) S + k_t v_t^T, o_t = S^T r_t with w = sigmoid(z + w0)^(1 / tau); key sizes up to 256 and value sizes that are
//        multiples of 8
//
// Chunks of 16 tokens.  With c_t the running sum of log2 w inside the chunk (c_-1 = 0),
//   O = (r 2^(c_t-1)) S + A v,   A_ij = sum over channels r_i k_j 2^(c_i-1 - c_j) for j < i, r_i u k_i on the diagonal
//   S <- 2^(c_15) S + (k 2^(c_15 - c_t))^T v
// for WKV; in GLA a token's own decay and pair come ahead of its output: c_t and c_i stand where c_t-1 and c_i-1 do, and r_i k_i is
// on the diagonal.
// A decay per channel leaves no common factor to take out of a block of scores, and k 2^(-c_j) alone may overflow: every
// exponent that is taken here is a difference whose sign makes it at most zero.  A is made of 4 x 4 tiles: below the diagonal
// tiles both sides refer to the tile's first row (8 exponentials for 16 products), on it every pair has its own.
//
// One CTA walks the chunks of one (request, head) and 32, 64 or 128 of its value columns; two kinds of warps, stages of shared memory
// between them:
//   prep   (one to three groups of 4 warps that take turns) elementwise part with a thread per channel and 8 tokens, the next
//          chunk's inputs already in registers, then the tiles of A with lanes over channels
//   state  (one warp per 16 value columns) S^T in fp32 accumulators; O^T = S^T R^T + V^T A^T and S^T += V^T K on mma.sync, S^T being
//          its own A operand.  A chunk of 16 tokens is too short for tcgen05: the chain from S to S would go through tensor memory
//          and two commits per chunk, where it is a handful of dependent MMAs here.
// Every fp32 operand of an MMA is a pair of bf16 values hi + lo (products keep 16 bits of mantissa); v is bf16 as stored.  All
// waits are bounded.
#include "../include/omni_ptx.cuh"
#include "../include/omni_vec.cuh"
#include "../include/tma_host.h"

namespace omni {

struct WkvParams {
  const __nv_bfloat16 *r, *k, *v;      // [T, ld], head h at column h D
  int r_ld, k_ld, v_ld;
  const float* z;                      // [T, z_ld]
  int z_ld;
  const float *w0, *u;                 // [H D]; u: WKV
  float r_scale, inv_tau;              // GLA: multiplies r; 1 / tau
  float* state;                        // [slots, H, P (value), D (key)]
  const int* cu_q;
  const int64_t* positions;
  const int* state_slots;
  __nv_bfloat16* y;
  int y_ld;
  int H, D, P, min_rows;
  OmniStatus* status;
};

constexpr int WK_L = 16;                           // tokens per chunk
constexpr int WK_PREP = 4;                         // warps of a prep group
constexpr int WK_TP = 20;                          // floats per channel of the arrays [channel][token]
constexpr int WK_APITCH = 48;                      // bytes per row of A
template <int DP, int VP>                            // key channels, value columns of a CTA
struct WkLayout {
  static constexpr int GROUPS = DP > 128 ? 1 : (DP > 64 && VP != 64 ? 2 : 3);   // prep groups, as many as fit
  static constexpr int STAGES = 2 * GROUPS;
  static constexpr int PITCH = DP * 2 + 16;        // bytes per token row; ldmatrix rows fall into different banks
  static constexpr int TILE = WK_L * PITCH;
  static constexpr int VPITCH = VP * 2 + 16;
  static constexpr int A_OFF = 4 * TILE + WK_L * VPITCH;      // after R hi, R lo, K hi, K lo, V
  static constexpr int DS_OFF = A_OFF + 2 * WK_L * WK_APITCH;
  static constexpr int STAGE = DS_OFF + DP * 4;
  static constexpr int T_OFF = STAGES * STAGE;  // per group r, k, c: [DP][WK_TP] floats each
  static constexpr int T_ARR = DP * WK_TP * 4;
  static constexpr int U_OFF = T_OFF + GROUPS * 3 * T_ARR;
  static constexpr int BAR_OFF = U_OFF + DP * 4;
  static constexpr int SMEM = BAR_OFF + ((2 * STAGES + GROUPS) * 8 + 4 + 15) / 16 * 16;      // barriers, abort flag
  static_assert(SMEM <= 232448, "exceeds the 227 KB shared-memory limit of one CTA");
  static constexpr int STATE_WARPS = VP / 16;
  static constexpr int THREADS = 32 * (GROUPS * WK_PREP + STATE_WARPS);
};

__device__ __forceinline__ void wk_ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr) : "memory");
}
__device__ __forceinline__ void wk_ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr) : "memory");
}
__device__ __forceinline__ void wk_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void wk_split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float wk_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Sum of v[16] over the GROUP lanes of a group (GROUP 8 or 16, groups aligned): lane e of the group ends up with element(s)
// e * 16 / GROUP ... in v[0 .. 16 / GROUP).
template <int GROUP>
__device__ __forceinline__ void wk_group_sum(float (&v)[16], int lane) {
  int n = 16;
#pragma unroll
  for (int o = GROUP / 2; o > 0; o >>= 1) {
    n >>= 1;
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i < n) {
        const float send = up ? v[i] : v[i + n];
        const float mine = up ? v[i + n] : v[i];
        v[i] = mine + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
  }
}

// log2 of the decay, from z + w0
template <bool GLA>
__device__ __forceinline__ float wk_log2_decay(float z, float inv_tau) {
  if (GLA) {      // log2 of the sigmoid; its absolute error of some 1e-7 is what a whole sequence multiplies at most
    const float z2 = z * 1.4426950408889634f;
    float l;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(1.f + wk_ex2(-fabsf(z2))));
    return (fminf(z2, 0.f) - l) * inv_tau;
  }
  return -1.4426950408889634f * expf(z);
}

template <int DP, int VP, bool GLA>
__global__ void __launch_bounds__(WkLayout<DP, VP>::THREADS) wkv_chunk_kernel(const WkvParams p) {
  using L = WkLayout<DP, VP>;
  const int h = blockIdx.x, q = blockIdx.y, v_col0 = blockIdx.z * VP, P = p.P;
  const int row0 = p.cu_q[q], n_rows = p.cu_q[q + 1] - row0, slot = p.state_slots[q];
  if (n_rows <= 0 || n_rows < p.min_rows || slot < 0) return;
  const int n = (n_rows + WK_L - 1) / WK_L, D = p.D;
  extern __shared__ __align__(16) uint8_t wk_smem[];
  uint64_t* bars = reinterpret_cast<uint64_t*>(wk_smem + L::BAR_OFF);
  uint64_t *full = bars, *empty = bars + L::STAGES, *tiles = bars + 2 * L::STAGES;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 2 * L::STAGES + L::GROUPS);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < L::STAGES; ++s) { mbar_init(&full[s], WK_PREP); mbar_init(&empty[s], L::STATE_WARPS); }
    for (int g = 0; g < L::GROUPS; ++g) mbar_init(&tiles[g], WK_PREP);
    *abort_flag = 0;
    mbar_fence_init();
  }
  // what is never written later: A above the diagonal, channels past the head size
  for (int i = threadIdx.x; i < L::BAR_OFF / 4; i += L::THREADS) reinterpret_cast<uint32_t*>(wk_smem)[i] = 0u;
  __syncthreads();
  for (int c = threadIdx.x; c < D; c += L::THREADS) reinterpret_cast<float*>(wk_smem + L::U_OFF)[c] = GLA ? 1.f : p.u[h * D + c];
  __syncthreads();

  if (warp < L::GROUPS * WK_PREP) {
    // ------------------------------------------------------------------ prep
    constexpr int PASS = (DP + 63) / 64;
    const int grp = warp / WK_PREP, gw = warp % WK_PREP, tid = threadIdx.x % (32 * WK_PREP);
    const int half = lane >> 4;                          // tokens 8 half .. 8 half + 7
    const float* us = reinterpret_cast<const float*>(wk_smem + L::U_OFF);
    __nv_bfloat16 rn[PASS][8], kn[PASS][8];              // the coming chunk
    float zn[PASS][8], w0[PASS];
    const __nv_bfloat16 zero = __float2bfloat16(0.f);
#pragma unroll
    for (int a = 0; a < PASS; ++a) {
      const int c = a * 64 + gw * 16 + (lane & 15);
      w0[a] = c < D ? p.w0[h * D + c] : 0.f;
    }
    auto fetch = [&](int ch) {
#pragma unroll
      for (int a = 0; a < PASS; ++a) {
        const int c = a * 64 + gw * 16 + (lane & 15), t0 = ch * WK_L + half * 8;
        const size_t row = (size_t)(row0 + t0);
        const __nv_bfloat16 *rp = p.r + row * p.r_ld + h * D + c, *kp = p.k + row * p.k_ld + h * D + c;
        const float* zp = p.z + row * p.z_ld + h * D + c;
        const int left = c < D ? n_rows - t0 : 0;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const bool ok = e < left;
          rn[a][e] = ok ? *rp : zero;
          kn[a][e] = ok ? *kp : zero;
          zn[a][e] = ok ? *zp : (GLA ? INFINITY : -INFINITY);      // no decay
          rp += p.r_ld; kp += p.k_ld; zp += p.z_ld;
        }
      }
    };
    if (grp < n) fetch(grp);
    for (int ch = grp; ch < n; ch += L::GROUPS) {
      const int s = ch % L::STAGES, ph = (ch / L::STAGES) & 1;
      uint8_t* st = wk_smem + s * L::STAGE;
      float* rT = reinterpret_cast<float*>(wk_smem + L::T_OFF + grp * 3 * L::T_ARR);
      float* kT = rT + DP * WK_TP;
      float* cT = kT + DP * WK_TP;                       // cT[channel][t] = c_t-1, t = 0 .. 16; GLA: c_t
      float w2[PASS][8];
#pragma unroll
      for (int a = 0; a < PASS; ++a)
#pragma unroll
        for (int e = 0; e < 8; ++e) w2[a][e] = fmaxf(wk_log2_decay<GLA>(zn[a][e] + w0[a], p.inv_tau), -256.f);   // 2^-256 is 0
      if (!mbar_wait(&empty[s], ph ^ 1, abort_flag, p.status, 71, ch)) break;
      // ---- v rows
      const int v8 = min(VP, P - v_col0) / 8;
      for (int i = tid; i < WK_L * v8; i += 32 * WK_PREP) {
        const int t = i / v8, c8 = i % v8;
        const bool ok = ch * WK_L + t < n_rows;
        const __nv_bfloat16* src = p.v + (size_t)(row0 + (ok ? ch * WK_L + t : 0)) * p.v_ld + h * P + v_col0 + c8 * 8;
        const int bytes = ok ? 16 : 0;                   // the rest is zero-filled
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;"
                     ::"r"(smem_u32(st + 4 * L::TILE + t * L::VPITCH + c8 * 16)), "l"(src), "r"(bytes) : "memory");
      }
      // ---- elementwise; the arrays are free once the whole group has handed over its chunk before
      if (ch >= L::GROUPS && !mbar_wait(&full[(ch - L::GROUPS) % L::STAGES], ((ch - L::GROUPS) / L::STAGES) & 1, abort_flag, p.status, 74, ch)) break;
#pragma unroll
      for (int a = 0; a < PASS; ++a) {
        const int c = a * 64 + gw * 16 + (lane & 15);
        float cum[8], run = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) { run += w2[a][e]; cum[e] = run; }
        const float other = __shfl_xor_sync(0xffffffffu, run, 16);
        const float base = half ? other : 0.f, tot = run + other;
        if (c < DP) {
          float rf[8], kf[8], pv[8];
          uint8_t* o = st + half * 8 * L::PITCH + c * 2;
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            rf[e] = __bfloat162float(rn[a][e]) * (GLA ? p.r_scale : 1.f);
            kf[e] = __bfloat162float(kn[a][e]);
            pv[e] = GLA ? base + cum[e] : base + (e ? cum[e - 1] : 0.f);
            const float R = rf[e] * wk_ex2(pv[e]), K = kf[e] * wk_ex2(fminf(tot - (base + cum[e]), 0.f));
            const __nv_bfloat16 rh = __float2bfloat16(R), kh = __float2bfloat16(K);
            *reinterpret_cast<__nv_bfloat16*>(o + e * L::PITCH) = rh;
            *reinterpret_cast<__nv_bfloat16*>(o + L::TILE + e * L::PITCH) = __float2bfloat16(R - __bfloat162float(rh));
            *reinterpret_cast<__nv_bfloat16*>(o + 2 * L::TILE + e * L::PITCH) = kh;
            *reinterpret_cast<__nv_bfloat16*>(o + 3 * L::TILE + e * L::PITCH) = __float2bfloat16(K - __bfloat162float(kh));
          }
          const int at = c * WK_TP + half * 8;
          *reinterpret_cast<float4*>(rT + at) = make_float4(rf[0], rf[1], rf[2], rf[3]);
          *reinterpret_cast<float4*>(rT + at + 4) = make_float4(rf[4], rf[5], rf[6], rf[7]);
          *reinterpret_cast<float4*>(kT + at) = make_float4(kf[0], kf[1], kf[2], kf[3]);
          *reinterpret_cast<float4*>(kT + at + 4) = make_float4(kf[4], kf[5], kf[6], kf[7]);
          *reinterpret_cast<float4*>(cT + at) = make_float4(pv[0], pv[1], pv[2], pv[3]);
          *reinterpret_cast<float4*>(cT + at + 4) = make_float4(pv[4], pv[5], pv[6], pv[7]);
          if (half) {
            if (!GLA) cT[c * WK_TP + 16] = base + cum[7];
            reinterpret_cast<float*>(st + L::DS_OFF)[c] = wk_ex2(tot);
          }
        }
      }
      if (ch + L::GROUPS < n) fetch(ch + L::GROUPS);
      __syncwarp();
      if (lane == 0) mbar_arrive(&tiles[grp]);
      if (!mbar_wait(&tiles[grp], (ch / L::GROUPS) & 1, abort_flag, p.status, 72, ch)) break;
      // ---- A
      float acc[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) acc[i] = 0.f;
      uint8_t* At = st + L::A_OFF;
      auto put = [&](int i, int j, float x) {
        const __nv_bfloat16 hi = __float2bfloat16(x);
        *reinterpret_cast<__nv_bfloat16*>(At + i * WK_APITCH + j * 2) = hi;
        *reinterpret_cast<__nv_bfloat16*>(At + WK_L * WK_APITCH + i * WK_APITCH + j * 2) = __float2bfloat16(x - __bfloat162float(hi));
      };
      if (gw == 0) {                                     // the four diagonal tiles, eight lanes each
        const int b = (lane >> 3) * 4;
#pragma unroll 4
        for (int cc = 0; cc < DP; cc += 8) {
          const int c = cc + (lane & 7);
          const float4 r4 = *reinterpret_cast<const float4*>(rT + c * WK_TP + b), k4 = *reinterpret_cast<const float4*>(kT + c * WK_TP + b);
          const float4 p4 = *reinterpret_cast<const float4*>(cT + c * WK_TP + b);
          const float rv[4] = {r4.x, r4.y, r4.z, r4.w}, kv[4] = {k4.x, k4.y, k4.z, k4.w}, cv[4] = {p4.x, p4.y, p4.z, p4.w};
          const float uc = us[c];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            acc[i * 4 + i] = fmaf(rv[i] * uc, kv[i], acc[i * 4 + i]);
#pragma unroll
            for (int j = 0; j < i; ++j) {                // c_i-1 - c_j; GLA: c_i - c_j
              if (GLA) acc[i * 4 + j] = fmaf(rv[i] * kv[j], wk_ex2(fminf(cv[i] - cv[j], 0.f)), acc[i * 4 + j]);
              else acc[i * 4 + j] = fmaf(rv[i] * kv[j], j + 1 == i ? 1.f : wk_ex2(fminf(cv[i] - cv[j + 1], 0.f)), acc[i * 4 + j]);
            }
          }
        }
        wk_group_sum<8>(acc, lane);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int x = (lane & 7) * 2 + e, i = x >> 2, j = x & 3;
          if (j <= i) put(b + i, b + j, acc[e]);
        }
      } else {                                           // two tiles below it per warp, sixteen lanes each
        const int tile = (gw - 1) * 2 + (lane >> 4);   // (1,0) (2,0) (2,1) (3,0) (3,1) (3,2)
        const int I = tile == 0 ? 1 : (tile < 3 ? 2 : 3), J = tile == 0 ? 0 : (tile < 3 ? tile - 1 : tile - 3);
#pragma unroll 4
        for (int cc = 0; cc < DP; cc += 16) {
          const int c = cc + (lane & 15);
          const float4 r4 = *reinterpret_cast<const float4*>(rT + c * WK_TP + I * 4), k4 = *reinterpret_cast<const float4*>(kT + c * WK_TP + J * 4);
          const float4 pi = *reinterpret_cast<const float4*>(cT + c * WK_TP + I * 4), pj = *reinterpret_cast<const float4*>(cT + c * WK_TP + J * 4);
          const float ref = pi.x, pj4 = GLA ? 0.f : cT[c * WK_TP + J * 4 + 4];
          const float cj[4] = {GLA ? pj.x : pj.y, GLA ? pj.y : pj.z, GLA ? pj.z : pj.w, GLA ? pj.w : pj4};      // c of the tile's keys
          const float rv[4] = {r4.x, r4.y * wk_ex2(fminf(pi.y - ref, 0.f)), r4.z * wk_ex2(fminf(pi.z - ref, 0.f)), r4.w * wk_ex2(fminf(pi.w - ref, 0.f))};
          const float kv[4] = {k4.x * wk_ex2(fminf(ref - cj[0], 0.f)), k4.y * wk_ex2(fminf(ref - cj[1], 0.f)),
                               k4.z * wk_ex2(fminf(ref - cj[2], 0.f)), k4.w * wk_ex2(fminf(ref - cj[3], 0.f))};
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i * 4 + j] = fmaf(rv[i], kv[j], acc[i * 4 + j]);
        }
        wk_group_sum<16>(acc, lane);
        const int x = lane & 15;
        put(I * 4 + (x >> 2), J * 4 + (x & 3), acc[0]);
      }
      asm volatile("cp.async.wait_all;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(&full[s]);
    }
  } else {
    // ------------------------------------------------------------------ state
    const int vc0 = (warp - L::GROUPS * WK_PREP) * 16, p0 = v_col0 + vc0, g = lane >> 2, t2 = (lane & 3) * 2;
    float S[DP / 8][4];                                  // rows p0 + g (+ 8) of S^T, channels nt * 8 + t2 (+ 1)
    float* gs = p.state + ((size_t)slot * p.H + h) * P * D;
    const bool fresh = p.positions[row0] == 0;
#pragma unroll
    for (int nt = 0; nt < DP / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int pr = p0 + g + e * 4, c = nt * 8 + t2;
        float2 v = make_float2(0.f, 0.f);
        if (!fresh && pr < P && c < D) v = *reinterpret_cast<const float2*>(gs + (size_t)pr * D + c);
        S[nt][e] = v.x;
        S[nt][e + 1] = v.y;
      }
    const int lrow = (lane >> 4) * 8 + (lane & 7), lcol = ((lane >> 3) & 1) * 16;      // matrices ordered (rows, columns): 00 01 10 11
    const uint32_t sb = smem_u32(wk_smem);
    bool ok = true;
    for (int ch = 0; ch < n; ++ch) {
      const int s = ch % L::STAGES;
      if (!mbar_wait(&full[s], (ch / L::STAGES) & 1, abort_flag, p.status, 73, ch)) { ok = false; break; }
      __syncwarp();
      const uint32_t st = sb + s * L::STAGE;
      float o[2][4], o2[2][4], o3[2][4];               // sums of their own: short chains of dependent MMAs
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = o2[i][e] = o3[i][e] = 0.f;
      // ---- O^T = S^T R^T
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        wk_split2(S[2 * ks][0], S[2 * ks][1], ah[0], al[0]);
        wk_split2(S[2 * ks][2], S[2 * ks][3], ah[1], al[1]);
        wk_split2(S[2 * ks + 1][0], S[2 * ks + 1][1], ah[2], al[2]);
        wk_split2(S[2 * ks + 1][2], S[2 * ks + 1][3], ah[3], al[3]);
        const uint32_t at = st + lrow * L::PITCH + ks * 32 + lcol;
        wk_ldsm4(at, bh);
        wk_ldsm4(at + L::TILE, bl);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          wk_mma(o[i], ah, bh[2 * i], bh[2 * i + 1]);
          wk_mma(o2[i], ah, bl[2 * i], bl[2 * i + 1]);
          wk_mma(o3[i], al, bh[2 * i], bh[2 * i + 1]);
        }
      }
      // ---- + V^T A^T
      uint32_t va[4];
      wk_ldsm4t(st + 4 * L::TILE + lrow * L::VPITCH + vc0 * 2 + lcol, va);      // (tokens, values) 00 01 10 11 transposed: a0 a1 a2 a3
      {
        uint32_t bh[4], bl[4];
        const uint32_t at = st + L::A_OFF + lrow * WK_APITCH + lcol;
        wk_ldsm4(at, bh);
        wk_ldsm4(at + WK_L * WK_APITCH, bl);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          wk_mma(o2[i], va, bh[2 * i], bh[2 * i + 1]);
          wk_mma(o3[i], va, bl[2 * i], bl[2 * i + 1]);
        }
      }
      // ---- S^T <- 2^c_15 S^T + V^T K
      const float* ds = reinterpret_cast<const float*>(wk_smem + s * L::STAGE + L::DS_OFF);
#pragma unroll
      for (int n2 = 0; n2 < DP / 16; ++n2) {
        uint32_t bh[4], bl[4];
        // (tokens 0-7, channels 0-7), (tokens 8-15, channels 0-7), then the next 8 channels; transposed
        const uint32_t at = st + 2 * L::TILE + (((lane >> 3) & 1) * 8 + (lane & 7)) * L::PITCH + n2 * 32 + (lane >> 4) * 16;
        wk_ldsm4t(at, bh);
        wk_ldsm4t(at + L::TILE, bl);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          float (&sv)[4] = S[n2 * 2 + i];
          const float2 d = *reinterpret_cast<const float2*>(ds + (n2 * 2 + i) * 8 + t2);
          sv[0] *= d.x; sv[1] *= d.y; sv[2] *= d.x; sv[3] *= d.y;
          wk_mma(sv, va, bh[2 * i], bh[2 * i + 1]);
          wk_mma(sv, va, bl[2 * i], bl[2 * i + 1]);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[s]);
      // ---- output rows: o[i][e] belongs to value p0 + g (+ 8 for e >= 2) of token i * 8 + t2 (+ 1 for odd e)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = ch * WK_L + i * 8 + t2 + (e & 1), pr = p0 + g + (e >> 1) * 8;
          if (t < n_rows && pr < P) p.y[(size_t)(row0 + t) * p.y_ld + h * P + pr] = __float2bfloat16(o[i][e] + (o2[i][e] + o3[i][e]));
        }
    }
    if (ok) {
#pragma unroll
      for (int nt = 0; nt < DP / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int pr = p0 + g + e * 4, c = nt * 8 + t2;
          if (pr < P && c < D) *reinterpret_cast<float2*>(gs + (size_t)pr * D + c) = make_float2(S[nt][e], S[nt][e + 1]);
        }
    }
  }
  asm volatile("cp.async.wait_all;" ::: "memory");      // nothing in flight when a wait has given up either
  __syncthreads();
  if (threadIdx.x == 0 && *abort_flag) report_abort(abort_flag, p.status);
}

template <int DP, int VP, bool GLA>
static int launch_wkv(const WkvParams& p, int B, cudaStream_t stream) {
  using L = WkLayout<DP, VP>;
  static bool configured[64] = {false};
  if (int e = ensure_dyn_smem((const void*)wkv_chunk_kernel<DP, VP, GLA>, L::SMEM, configured)) return e;
  wkv_chunk_kernel<DP, VP, GLA><<<dim3(p.H, B, (p.P + VP - 1) / VP), L::THREADS, L::SMEM, stream>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace omni

using namespace omni;

// Requests with fewer than min_rows rows, and padding, are not touched.
extern "C" int omni_wkv_chunks(const void* r, int r_ld, const void* k, int k_ld, const void* v, int v_ld, const float* z, int z_ld,
                               const void* w0, const void* u, void* state, const int* cu_q, const int64_t* positions,
                               const int* state_slots, int B, int max_q, void* y, int y_ld, int H, int D, int min_rows, void* status,
                               cudaStream_t stream) {
  if (B <= 0 || max_q < min_rows) return 0;
  if (H < 1 || B > 65535 || min_rows < 1 || D < 8 || D % 8 != 0 || D > 128) return -1;
  if (v_ld % 8 != 0 || (uintptr_t)v % 16 != 0 || (uintptr_t)state % 16 != 0) return -2;
  WkvParams p = {(const __nv_bfloat16*)r, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, r_ld, k_ld, v_ld, z, z_ld, (const float*)w0,
                 (const float*)u, 1.f, 0.f, (float*)state, cu_q, positions, state_slots, (__nv_bfloat16*)y, y_ld, H, D, D, min_rows,
                 (OmniStatus*)status};
  if (D <= 32) return launch_wkv<32, 32, false>(p, B, stream);
  if (D <= 64) return launch_wkv<64, 64, false>(p, B, stream);
  return launch_wkv<128, 128, false>(p, B, stream);
}

// q, k with head h at column h N, v and y at column h P, z and bias [H N], state [slots, H, P, N].
extern "C" int omni_gla_chunks(const void* q, int q_ld, const void* k, int k_ld, const void* v, int v_ld, const float* z, int z_ld,
                               const float* bias, float q_scale, float inv_tau, void* state, const int* cu_q, const int64_t* positions,
                               const int* state_slots, int B, int max_q, void* y, int y_ld, int H, int P, int N, int min_rows,
                               void* status, cudaStream_t stream) {
  if (B <= 0 || max_q < min_rows) return 0;
  if (H < 1 || B > 65535 || min_rows < 1 || N < 8 || N % 8 != 0 || N > 256 || P < 8 || P % 8 != 0 || P > 65535 || !(inv_tau > 0.f)) return -1;
  if (v_ld % 8 != 0 || (uintptr_t)v % 16 != 0 || (uintptr_t)state % 16 != 0) return -2;
  WkvParams p = {(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, q_ld, k_ld, v_ld, z, z_ld, bias, nullptr,
                 q_scale, inv_tau, (float*)state, cu_q, positions, state_slots, (__nv_bfloat16*)y, y_ld, H, N, P, min_rows,
                 (OmniStatus*)status};
  // every CTA prepares its chunks anew: 64 columns each only where that leaves no SM with two CTAs
  const bool narrow = (long long)H * B * ((P + 63) / 64) <= 148;
#define GLA_CASE(DP)                                                       \
  if (N <= DP) {                                                           \
    if (P <= 32) return launch_wkv<DP, 32, true>(p, B, stream);            \
    if (P <= 64 || narrow) return launch_wkv<DP, 64, true>(p, B, stream);  \
    return launch_wkv<DP, 128, true>(p, B, stream);                        \
  }
  GLA_CASE(32) GLA_CASE(64) GLA_CASE(128) GLA_CASE(256)
#undef GLA_CASE
  return -3;
}
