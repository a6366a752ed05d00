// Mamba-2 recurrence over portions of prompts on tcgen05: chunks of 128 tokens, state size up to 128, bf16 activations.
// (mamba2.cu holds the other forms: single tokens, fp32, larger states.)
//
// Per chunk of one (request, head, 64 columns of P), with cum the running sum of -exp(A_log) dt inside the chunk:
//   SC = C B^T                                  [128 i x 128 j]  A = C (smem, K-major)      B = B (smem, K-major)
//   M  = SC o exp(cum_i - cum_j) dt_j + D I     j <= i, in TMEM over SC as bf16 hi | lo
//   YD = M x                                    [128 i x 64 p]   A = M (TMEM)               B = x (smem, MN-major)
//   YO = C S                                    [128 i x 64 p]   A = C                      B = S hi, lo (smem, MN-major)
//   ST = B^T W, W = exp(cum_end - cum) dt x     [128 n x 64 p]   A = B (smem, MN-major)     B = W hi, lo (smem, MN-major)
//   y  = YD + exp(cum_i) YO,   S <- exp(cum_end) S + ST
// S lives in fp32 registers (thread = row n).  Every fp32 operand of an MMA is a pair of bf16 values hi + lo (two MMAs), so
// products keep 16 bits of mantissa on that side; C, B and x are bf16 as stored.
//
// One CTA walks the chunks of its request.  Warps: 0 TMA producer (two stages of C, B, x), 1 MMA issue, 2..5 scores -> M and
// the output rows (thread = token), 6..9 decays, W and the state (thread = token, then thread = state row).  Left of the
// diagonal block a warp's 32 rows need no exponentials per element: exp(cum_i - cum_j) dt_j = exp(cum_i - cum_b) *
// (exp(cum_b - cum_j) dt_j) with b the last token of j's block of 32, both factors at most 1 and the second shared by
// all rows.  Every wait is bounded.
#include "../include/omni_ptx.cuh"
#include "../include/omni_vec.cuh"
#include "../include/tma_host.h"

namespace omni {

struct SsdParams {
  const __nv_bfloat16* dt;   // dt of head h of row t: dt[t * dt_ld + h], before bias and softplus
  int dt_ld;
  const float* A_log;
  const float* dt_bias;
  const float* D;
  float* state;              // [slots, H, P, N]
  const int* cu_q;
  const int64_t* positions;
  const int* state_slots;
  __nv_bfloat16* y;          // [T, y_ld]
  int y_ld;
  int H, P, N, G;
  int min_rows;              // requests with fewer rows are left to another kernel
  OmniStatus* status;
};

constexpr int SQ = 128;                        // tokens per chunk
constexpr int SQ_TILE = SQ * 128;              // 128 rows of one 128-byte swizzle span: 16 KB
constexpr int SQ_STAGE = 5 * SQ_TILE;          // C (2 tiles), B (2 tiles), x
constexpr int SQ_W = 2 * SQ_STAGE;             // W hi, W lo
constexpr int SQ_S = SQ_W + 2 * SQ_TILE;       // S hi, S lo
constexpr int SQ_F = SQ_S + 2 * SQ_TILE;       // cum, g, dt: 128 floats each
constexpr int SQ_BAR = SQ_F + 3 * SQ * 4;
constexpr int SQ_SMEM = SQ_BAR + 192;
static_assert(SQ_SMEM <= 232448, "shared memory of one CTA");
constexpr int SQ_THREADS = 320;
// TMEM columns: SC / M two buffers of 128, YO two of 64, YD, ST
constexpr int TC_SC = 0, TC_YO = 256, TC_YD = 384, TC_ST = 448, TC_COLS = 512;

__device__ __forceinline__ void sq_umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void sq_split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float sq_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// eight values -> 16-byte chunk `ch` of row `row` of a hi and a lo tile
__device__ __forceinline__ void sq_store8(uint8_t* hi_tile, uint8_t* lo_tile, int row, int ch, const float (&v)[8]) {
  uint32_t hi[4], lo[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) sq_split2(v[2 * e], v[2 * e + 1], hi[e], lo[e]);
  const int off = row * 128 + ((ch ^ (row & 7)) << 4);
  *reinterpret_cast<uint4*>(hi_tile + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
  *reinterpret_cast<uint4*>(lo_tile + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
}

__global__ void __launch_bounds__(SQ_THREADS, 1)
ssd_sm100_kernel(const __grid_constant__ CUtensorMap tmap_bc, const __grid_constant__ CUtensorMap tmap_x, const SsdParams p) {
  const int pt = blockIdx.x, h = blockIdx.y, r = blockIdx.z;
  const int row0 = p.cu_q[r], n_rows = p.cu_q[r + 1] - row0;
  const int slot = p.state_slots[r];
  if (n_rows <= 0 || n_rows < p.min_rows || slot < 0) return;      // uniform, before any barrier / TMEM use
  const int p0 = pt * 64, pw = min(64, p.P - p0);
  const int g = h / (p.H / p.G);
  const int n = (n_rows + SQ - 1) / SQ;
  const int nch = (p.N + 63) / 64, ksn = (p.N + 15) / 16;          // 64-wide tiles and 16-wide steps of the state size

  extern __shared__ __align__(1024) uint8_t sq_smem[];
  uint64_t* bars = (uint64_t*)(sq_smem + SQ_BAR);
  uint64_t *full = bars, *empty = bars + 2, *sc_full = bars + 4;   // two each
  uint64_t *m_full = bars + 6, *cum_full = bars + 7, *w_full = bars + 8, *st_full = bars + 9, *s_full = bars + 10,
           *yo_done = bars + 11, *y_full = bars + 12, *y_empty = bars + 13;
  uint32_t* tmem_slot = (uint32_t*)(bars + 14);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
  float* cum = reinterpret_cast<float*>(sq_smem + SQ_F);           // log2 units
  float* gs = cum + SQ;
  float* dts = gs + SQ;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < 2; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); mbar_init(&sc_full[s], 1); }
    mbar_init(m_full, 4); mbar_init(cum_full, 4); mbar_init(w_full, 4); mbar_init(st_full, 1);
    mbar_init(s_full, 4); mbar_init(yo_done, 1); mbar_init(y_full, 1); mbar_init(y_empty, 4);
    *abort_flag = (smem_u32(sq_smem) & 1023) ? (0x40000000 | (51 << 16)) : 0;      // swizzled tiles need the alignment
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, TC_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const bool aligned = (smem_u32(sq_smem) & 1023) == 0;

  if (!aligned) {
    // nothing runs; reported below
  } else if (warp == 0) {
    if (lane == 0) {
      for (int c = 0; c < n; ++c) {
        const int s = c & 1, row = row0 + c * SQ;
        if (!mbar_wait(&empty[s], ((c >> 1) & 1) ^ 1, abort_flag, p.status, 51, c)) break;
        uint8_t* st = sq_smem + s * SQ_STAGE;
        mbar_expect_tx(&full[s], (2 * nch + 1) * SQ_TILE);
        for (int k = 0; k < nch; ++k) {
          tma_load_3d(st + k * SQ_TILE, &tmap_bc, &full[s], k * 64, p.G + g, row);
          tma_load_3d(st + (2 + k) * SQ_TILE, &tmap_bc, &full[s], k * 64, g, row);
        }
        tma_load_3d(st + 4 * SQ_TILE, &tmap_x, &full[s], p0, h, row);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t id_sc = umma_idesc(128, 128, 1, 1, 0, 0);
      constexpr uint32_t id_y = umma_idesc(128, 64, 1, 1, 0, 1);
      constexpr uint32_t id_st = umma_idesc(128, 64, 1, 1, 1, 1);
      const uint32_t sbase = smem_u32(sq_smem);
      auto mn = [&](uint32_t addr, int k) { return umma_desc_mnmajor_sw128(addr + k * 2048, SQ_TILE, 1024); };
      auto issue_sc = [&](int c) -> bool {
        if (!mbar_wait(&full[c & 1], (c >> 1) & 1, abort_flag, p.status, 52, c)) return false;
        tc_fence_after();
        const uint32_t cb = sbase + (c & 1) * SQ_STAGE;
        for (int k = 0; k < ksn; ++k)
          umma_bf16(tmem + TC_SC + (c & 1) * 128, umma_desc_kmajor_sw128(cb + (k >> 2) * SQ_TILE) + 2 * (k & 3),
                    umma_desc_kmajor_sw128(cb + (2 + (k >> 2)) * SQ_TILE) + 2 * (k & 3), id_sc, k > 0);
        umma_commit(&sc_full[c & 1]);
        return true;
      };
      bool ok = issue_sc(0);
      for (int c = 0; c < n && ok; ++c) {
        const uint32_t ph = c & 1, cb = sbase + (c & 1) * SQ_STAGE;
        // ---- YO = C S
        if (!mbar_wait(s_full, ph, abort_flag, p.status, 53, c)) { ok = false; break; }
        tc_fence_after();
        for (int k = 0; k < ksn; ++k) {
          const uint64_t ad = umma_desc_kmajor_sw128(cb + (k >> 2) * SQ_TILE) + 2 * (k & 3);
          umma_bf16(tmem + TC_YO + (c & 1) * 64, ad, mn(sbase + SQ_S, k), id_y, k > 0);
          umma_bf16(tmem + TC_YO + (c & 1) * 64, ad, mn(sbase + SQ_S + SQ_TILE, k), id_y, 1u);
        }
        umma_commit(yo_done);
        // ---- ST = B^T W
        if (!mbar_wait(w_full, ph, abort_flag, p.status, 54, c)) { ok = false; break; }
        tc_fence_after();
        for (int k = 0; k < 8; ++k) {
          const uint64_t ad = mn(cb + 2 * SQ_TILE, k);
          umma_bf16(tmem + TC_ST, ad, mn(sbase + SQ_W, k), id_st, k > 0);
          umma_bf16(tmem + TC_ST, ad, mn(sbase + SQ_W + SQ_TILE, k), id_st, 1u);
        }
        umma_commit(st_full);
        // ---- the next chunk's scores, while this one's are worked on
        if (c + 1 < n && !issue_sc(c + 1)) { ok = false; break; }
        // ---- YD = M x
        if (!mbar_wait(m_full, ph, abort_flag, p.status, 55, c)) { ok = false; break; }
        if (c > 0 && !mbar_wait(y_empty, (c - 1) & 1, abort_flag, p.status, 56, c)) { ok = false; break; }
        tc_fence_after();
        for (int k = 0; k < 8; ++k) {
          const uint32_t m = tmem + TC_SC + (c & 1) * 128 + (k >> 1) * 32 + (k & 1) * 8;
          const uint64_t xd = mn(cb + 4 * SQ_TILE, k);
          sq_umma_ts(tmem + TC_YD, m, xd, id_y, k > 0);
          sq_umma_ts(tmem + TC_YD, m + 16, xd, id_y, 1u);
        }
        umma_commit(y_full);
        umma_commit(&empty[c & 1]);
      }
    }
  } else if (warp < 6) {
    // ------------------------------------------------------------------ scores -> M, output rows
    const int qd = warp & 3, i = qd * 32 + lane;
    const uint32_t la = tmem + ((uint32_t)(qd * 32) << 16);
    const float Dh = p.D[h];
    float e_prev = 0.f;
    auto output = [&](int c, float e) -> bool {          // rows of chunk c: YD + e YO
      if (!mbar_wait(y_full, c & 1, abort_flag, p.status, 57, c)) return false;
      tc_fence_after();
      const int t = c * SQ + i;
      __nv_bfloat16* yr = p.y + (size_t)(row0 + t) * p.y_ld + h * p.P + p0;
#pragma unroll 1
      for (int q = 0; q < 64; q += 32) {
        if (q >= pw) break;
        uint32_t yd[32], yo[32];
        tmem_ld_x32(la + TC_YD + q, yd);
        tmem_ld_x32(la + TC_YO + (c & 1) * 64 + q, yo);
        tmem_ld_wait();
        if (t < n_rows) {
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (q + j < pw) {
              float v[8];
#pragma unroll
              for (int k = 0; k < 8; ++k) v[k] = fmaf(e, __uint_as_float(yo[j + k]), __uint_as_float(yd[j + k]));
              store_vec<8>(yr + q + j, v);
            }
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(y_empty);
      return true;
    };
    bool ok = true;
    for (int c = 0; c < n; ++c) {
      if (!mbar_wait(cum_full, c & 1, abort_flag, p.status, 58, c) ||
          !mbar_wait(&sc_full[c & 1], (c >> 1) & 1, abort_flag, p.status, 59, c)) { ok = false; break; }
      tc_fence_after();
      const float ci = cum[i];
#pragma unroll 1
      for (int b = 0; b < 4; ++b) {
        const uint32_t col = la + TC_SC + (c & 1) * 128 + b * 32;
        uint32_t hi[16], lo[16];
        if (b > qd) {                                    // right of the diagonal
#pragma unroll
          for (int j = 0; j < 16; ++j) hi[j] = lo[j] = 0u;
        } else {
          uint32_t s[32];
          tmem_ld_x32(col, s);
          tmem_ld_wait();
          if (b < qd) {
            const float f = exp2f(ci - cum[b * 32 + 31]);
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
              const float4 gj = *reinterpret_cast<const float4*>(gs + b * 32 + j);
              sq_split2(__uint_as_float(s[j]) * (f * gj.x), __uint_as_float(s[j + 1]) * (f * gj.y), hi[j / 2], lo[j / 2]);
              sq_split2(__uint_as_float(s[j + 2]) * (f * gj.z), __uint_as_float(s[j + 3]) * (f * gj.w), hi[j / 2 + 1],
                        lo[j / 2 + 1]);
            }
          } else {
#pragma unroll
            for (int j = 0; j < 32; j += 2) {
              const float2 cj = *reinterpret_cast<const float2*>(cum + b * 32 + j);
              const float2 dj = *reinterpret_cast<const float2*>(dts + b * 32 + j);
              float m0 = j <= lane ? __uint_as_float(s[j]) * (exp2f(fminf(ci - cj.x, 0.f)) * dj.x) : 0.f;
              float m1 = j + 1 <= lane ? __uint_as_float(s[j + 1]) * (exp2f(fminf(ci - cj.y, 0.f)) * dj.y) : 0.f;
              if (j == lane) m0 += Dh;
              if (j + 1 == lane) m1 += Dh;
              sq_split2(m0, m1, hi[j / 2], lo[j / 2]);
            }
          }
        }
        tmem_st_x16(col, hi);
        tmem_st_x16(col + 16, lo);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(m_full);
      if (c > 0 && !output(c - 1, e_prev)) { ok = false; break; }
      e_prev = exp2f(ci);
    }
    if (ok) output(n - 1, e_prev);
  } else {
    // ------------------------------------------------------------------ decays, W, state
    const int qd = warp & 3, i = qd * 32 + lane;         // token of the chunk, and row n of the state
    const uint32_t la = tmem + ((uint32_t)(qd * 32) << 16);
    const float a2 = -expf(p.A_log[h]) * 1.4426950408889634f, bias = p.dt_bias[h];
    float* st = p.state + (((size_t)slot * p.H + h) * p.P + p0) * p.N + i;
    const bool fresh = p.positions[row0] == 0, in_n = i < p.N;
    float S[64];
#pragma unroll
    for (int k = 0; k < 64; ++k) S[k] = (!fresh && in_n && k < pw) ? st[(size_t)k * p.N] : 0.f;
    auto write_state = [&]() {
#pragma unroll
      for (int ch = 0; ch < 8; ++ch) {
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = S[ch * 8 + e];
        sq_store8(sq_smem + SQ_S, sq_smem + SQ_S + SQ_TILE, i, ch, v);
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(s_full);
    };
    write_state();
    const __nv_bfloat16* dtp = p.dt + (size_t)row0 * p.dt_ld + h;
    auto load_dt = [&](int c, float (&d)[4]) {           // every warp sees the whole chunk: it needs all four block sums
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        const int t = c * SQ + b * 32 + lane;
        d[b] = t < n_rows ? __bfloat162float(dtp[(size_t)t * p.dt_ld]) : 0.f;
      }
    };
    float raw[4];
    load_dt(0, raw);
    for (int c = 0; c < n; ++c) {
      float off = 0.f, cend = 0.f, ci = 0.f, dt = 0.f;
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        const float d = c * SQ + b * 32 + lane < n_rows ? sq_softplus(raw[b] + bias) : 0.f;
        float run = a2 * d;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float up = __shfl_up_sync(0xffffffffu, run, o);
          if (lane >= o) run += up;
        }
        if (b == qd) { dt = d; ci = run; off = cend; }
        cend += __shfl_sync(0xffffffffu, run, 31);
      }
      ci += off;
      if (c + 1 < n) load_dt(c + 1, raw);
      const float c31 = __shfl_sync(0xffffffffu, ci, 31);
      if (c > 0 && !mbar_wait(m_full, (c - 1) & 1, abort_flag, p.status, 60, c)) break;    // the arrays have been read
      cum[i] = ci;
      gs[i] = exp2f(fminf(c31 - ci, 0.f)) * dt;
      dts[i] = dt;
      __syncwarp();
      if (lane == 0) mbar_arrive(cum_full);
      // ---- W = exp(cum_end - cum) dt x, this token's row
      if (!mbar_wait(&full[c & 1], (c >> 1) & 1, abort_flag, p.status, 61, c)) break;
      const float w = exp2f(fminf(cend - ci, 0.f)) * dt;
      const uint8_t* xr = sq_smem + (c & 1) * SQ_STAGE + 4 * SQ_TILE + i * 128;
      const bool live = c * SQ + i < n_rows;             // rows past the end hold another request's values
#pragma unroll
      for (int ch = 0; ch < 8; ++ch) {
        float v[8];
        load_vec<8>(reinterpret_cast<const __nv_bfloat16*>(xr + ((ch ^ (i & 7)) << 4)), v);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = live ? v[e] * w : 0.f;
        sq_store8(sq_smem + SQ_W, sq_smem + SQ_W + SQ_TILE, i, ch, v);
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(w_full);
      // ---- S <- exp(cum_end) S + ST
      if (!mbar_wait(st_full, c & 1, abort_flag, p.status, 62, c)) break;
      tc_fence_after();
      const float eend = exp2f(cend);
#pragma unroll
      for (int q = 0; q < 64; q += 16) {
        uint32_t v[16];
        tmem_ld_x16(la + TC_ST + q, v);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; ++j) S[q + j] = fmaf(eend, S[q + j], __uint_as_float(v[j]));
      }
      tc_fence_before();
      if (c + 1 < n) {
        if (!mbar_wait(yo_done, c & 1, abort_flag, p.status, 63, c)) break;      // C S has read the old state
        write_state();
      }
    }
    if (!*abort_flag) {
#pragma unroll
      for (int k = 0; k < 64; ++k)
        if (in_n && k < pw) st[(size_t)k * p.N] = S[k];
    }
  }

  if (*abort_flag) {
    if (threadIdx.x == 0) report_abort(abort_flag, p.status);
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, TC_COLS);
  }
}

}  // namespace omni

using namespace omni;

// Arguments as omni_ssm_scan (mamba2.cu); `rows` rows of xbc in all.  Requests with fewer than min_rows rows are not touched.
extern "C" int omni_ssd_chunks(const void* xbc, int xbc_ld, long long rows, const void* dt, int dt_ld, const void* A_log,
                               const void* dt_bias, const void* D, void* state, const int* cu_q, const int64_t* positions,
                               const int* state_slots, int B, void* y, int y_ld, int H, int P, int N, int G, int min_rows,
                               void* status, cudaStream_t stream) {
  if (B <= 0 || rows <= 0) return 0;
  if (H < 1 || G < 1 || H % G != 0 || B > 65535 || H > 65535) return -1;
  if (P < 8 || P % 8 != 0 || N < 8 || N % 8 != 0 || N > 128 || xbc_ld % 8 != 0 || y_ld % 8 != 0) return -2;
  if (((uintptr_t)xbc | (uintptr_t)y) % 16 != 0) return -3;
  CUtensorMap tbc, tx;
  const uint64_t pitch = (uint64_t)xbc_ld * 2;
  if (make_tmap_3d(&tbc, (const __nv_bfloat16*)xbc + H * P, 2, N, 2 * G, (uint64_t)rows, (uint64_t)N * 2, pitch, 64, 1, SQ, true))
    return -10;
  if (make_tmap_3d(&tx, xbc, 2, P, H, (uint64_t)rows, (uint64_t)P * 2, pitch, 64, 1, SQ, true)) return -11;
  SsdParams p;
  p.dt = (const __nv_bfloat16*)dt; p.dt_ld = dt_ld; p.A_log = (const float*)A_log; p.dt_bias = (const float*)dt_bias;
  p.D = (const float*)D; p.state = (float*)state; p.cu_q = cu_q; p.positions = positions; p.state_slots = state_slots;
  p.y = (__nv_bfloat16*)y; p.y_ld = y_ld; p.H = H; p.P = P; p.N = N; p.G = G; p.min_rows = min_rows;
  p.status = (OmniStatus*)status;
  static bool configured[64] = {false};
  if (int e = ensure_dyn_smem((const void*)ssd_sm100_kernel, SQ_SMEM, configured)) return e;
  ssd_sm100_kernel<<<dim3((P + 63) / 64, H, B), SQ_THREADS, SQ_SMEM, stream>>>(tbc, tx, p);
  return (int)cudaGetLastError();
}
