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
// A first small kernel turns dt into what both sides need per (chunk, head): cum, cp = cum - log2(dt) (so that
// exp(cum_i - cum_j) dt_j = 2^(cum_i - cp_j)) and g_j = 2^(cum_b - cp_j) with b the last token of j's block of 32.  Left of the
// diagonal block a warp's 32 rows then need no exponential per element: 2^(cum_i - cp_j) = 2^(cum_i - cum_b) g_j, both
// factors at most 1 (times dt) and the second shared by all rows.  All of it is in log2 units.
//
// The matrix memory of xLSTM (MEM) is the same scheme with C = q, B = k, x = v, and its own pre-pass (matrix_state.cu: gates):
// with b the running sum of the log forget gates, i the log input gate and m the running maximum,
//   M = SC o exp(b_i - m_i + i_j - b_j) N^-1/2,   y = YD + exp(b_i + m_in - m_i) N^-1/2 YO,   S <- exp(b_end + m_in - m_end) S + ST
// so `cum` holds b - m, cp = b - i, the factor of YO and S has m_in (m before the chunk) added, and blocks left of the diagonal
// take the largest i - b of the block as the reference between their two factors.  The CTA of the first 64 columns also moves
// the normaliser n (the last state row) and adds up n . q: row sums of M beside the dot products of q with n, in fp32.
//
// One CTA walks the chunks of its request.  Warps: 0 TMA producer (two stages of C, B, x, cp, g), 1 MMA issue, 2..9 scores ->
// M and the output rows (thread = token and half of the columns), 10..17 W and the state (thread = token, then state row, and
// half of the columns).  Every wait is bounded.
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
  float *cum, *cp, *g;       // [chunks, H, 128]; chunk c of request r is row cu_q[r] / 128 + r + c
  const float *gmax, *m_in;  // MEM: [chunks, H, 4], [chunks, H]
  float* den;                // MEM: [T, H], zeroed: n . q
  float log2_scale;          // MEM: of the factor on q
  OmniStatus* status;
};

constexpr int SQ = 128;                        // tokens per chunk
constexpr int SQ_TILE = SQ * 128;              // 128 rows of one 128-byte swizzle span: 16 KB
constexpr int SQ_STAGE = 5 * SQ_TILE;          // C (2 tiles), B (2 tiles), x
constexpr int SQ_W = 2 * SQ_STAGE;             // W hi, W lo
constexpr int SQ_S = SQ_W + 2 * SQ_TILE;       // S hi, S lo
constexpr int SQ_F = SQ_S + 2 * SQ_TILE;       // two stages of cp and g
constexpr int SQ_FB = SQ * 4;                  // bytes of one such array
constexpr int SQ_BAR = SQ_F + 4 * SQ_FB;
constexpr int SQ_N = SQ_BAR + 192;             // MEM: n
constexpr int SQ_SMEM = SQ_N + SQ_FB;
static_assert(SQ_SMEM <= 232448, "shared memory of one CTA");
constexpr int SQ_THREADS = 576;
// TMEM columns: SC / M two buffers of 128, YO two of 64, YD, ST.  M takes the columns of the scores it came from: 16 tokens
// are 8 columns hi and 8 columns lo.
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
__device__ __forceinline__ float sq_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void sq_tmem_st_x8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};"
               ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}
// 16 columns at each of two addresses.  The wait belongs to the same statement: between a load and its wait the compiler
// must not touch the destination registers, and it would not know.
__device__ __forceinline__ void sq_tmem_ld_2x16(uint32_t addr_a, uint32_t addr_b, uint32_t (&a)[16], uint32_t (&b)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%32];\n\t"
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%33];\n\t"
      "tcgen05.wait::ld.sync.aligned;"
      : "=&r"(a[0]), "=&r"(a[1]), "=&r"(a[2]), "=&r"(a[3]), "=&r"(a[4]), "=&r"(a[5]), "=&r"(a[6]), "=&r"(a[7]), "=&r"(a[8]), "=&r"(a[9]), "=&r"(a[10]), "=&r"(a[11]), "=&r"(a[12]), "=&r"(a[13]), "=&r"(a[14]), "=&r"(a[15]),
        "=&r"(b[0]), "=&r"(b[1]), "=&r"(b[2]), "=&r"(b[3]), "=&r"(b[4]), "=&r"(b[5]), "=&r"(b[6]), "=&r"(b[7]), "=&r"(b[8]), "=&r"(b[9]), "=&r"(b[10]), "=&r"(b[11]), "=&r"(b[12]), "=&r"(b[13]), "=&r"(b[14]), "=&r"(b[15])
      : "r"(addr_a), "r"(addr_b)
      : "memory");
}
__device__ __forceinline__ void sq_bulk_load(void* smem_dst, const void* gsrc, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(smem_dst)), "l"(gsrc), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
// byte offset of 16-byte chunk `ch` of row `row` of a swizzled tile
__device__ __forceinline__ int sq_off(int row, int ch) { return row * 128 + ((ch ^ (row & 7)) << 4); }

// One CTA per (chunk, request, 8 heads); thread = token of the chunk.
__global__ void __launch_bounds__(SQ) ssd_decay_kernel(const SsdParams p) {
  const int c = blockIdx.x, r = blockIdx.y, h0 = blockIdx.z * 8;
  const int row0 = p.cu_q[r], n_rows = p.cu_q[r + 1] - row0;
  if (c * SQ >= n_rows || n_rows < p.min_rows) return;
  const int i = threadIdx.x, warp = i >> 5, lane = i & 31, t = c * SQ + i;
  __shared__ float tot[4][8];
  float dt[8], run[8];
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    const int h = h0 + k;
    dt[k] = (h < p.H && t < n_rows) ? sq_softplus(__bfloat162float(p.dt[(size_t)(row0 + t) * p.dt_ld + h]) + p.dt_bias[h]) : 0.f;
    run[k] = h < p.H ? -expf(p.A_log[h]) * 1.4426950408889634f * dt[k] : 0.f;
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1)
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const float up = __shfl_up_sync(0xffffffffu, run[k], o);
      if (lane >= o) run[k] += up;
    }
  if (lane == 31)
#pragma unroll
    for (int k = 0; k < 8; ++k) tot[warp][k] = run[k];
  __syncthreads();
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    const float c31 = __shfl_sync(0xffffffffu, run[k], 31);
    if (h0 + k >= p.H) break;
    float off = 0.f;
    for (int w = 0; w < warp; ++w) off += tot[w][k];
    const float cum = run[k] + off;
    const size_t at = ((size_t)(row0 / SQ + r + c) * p.H + h0 + k) * SQ + i;
    p.cum[at] = cum;
    p.cp[at] = cum - log2f(dt[k]);               // dt 0 (rows past the end): +inf, i.e. no contribution
    p.g[at] = exp2f(fminf(c31 - run[k], 0.f)) * dt[k];
  }
}

template <bool MEM>
__global__ void __launch_bounds__(SQ_THREADS, 1)
ssd_sm100_kernel(const __grid_constant__ CUtensorMap tmap_c, const __grid_constant__ CUtensorMap tmap_b,
                 const __grid_constant__ CUtensorMap tmap_x, const SsdParams p) {
  const int pt = blockIdx.x, h = blockIdx.y, r = blockIdx.z;
  const int row0 = p.cu_q[r], n_rows = p.cu_q[r + 1] - row0;
  const int slot = p.state_slots[r];
  if (n_rows <= 0 || n_rows < p.min_rows || slot < 0) return;      // uniform, before any barrier / TMEM use
  const int p0 = pt * 64, pw = min(64, p.P - p0);
  const int g = MEM ? h : h / (p.H / p.G);
  const bool own_n = MEM && pt == 0;
  const int n = (n_rows + SQ - 1) / SQ;
  const int nch = (p.N + 63) / 64, ksn = (p.N + 15) / 16;          // 64-wide tiles and 16-wide steps of the state size
  const size_t arr0 = ((size_t)(row0 / SQ + r) * p.H + h) * SQ, arr_step = (size_t)p.H * SQ;

  extern __shared__ __align__(1024) uint8_t sq_smem[];
  uint64_t* bars = (uint64_t*)(sq_smem + SQ_BAR);
  uint64_t *full = bars, *empty = bars + 2, *sc_full = bars + 4;   // two each
  uint64_t *m_full = bars + 6, *w_full = bars + 7, *st_full = bars + 8, *s_full = bars + 9, *yo_done = bars + 10,
           *y_full = bars + 11, *y_empty = bars + 12, *n_full = bars + 13;
  uint32_t* tmem_slot = (uint32_t*)(bars + 14);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool aligned = (smem_u32(sq_smem) & 1023) == 0;            // the swizzled tiles need it
  if (threadIdx.x == 0) {
    for (int s = 0; s < 2; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); mbar_init(&sc_full[s], 1); }
    mbar_init(m_full, 8); mbar_init(w_full, 8); mbar_init(st_full, 1); mbar_init(s_full, 8);
    mbar_init(yo_done, 1); mbar_init(y_full, 1); mbar_init(y_empty, 8);
    if (MEM) mbar_init(n_full, 8);
    *abort_flag = aligned ? 0 : (0x40000000 | (51 << 16));
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

  if (!aligned) {
    // nothing runs; reported below
  } else if (warp == 0) {
    if (lane == 0) {
      for (int c = 0; c < n; ++c) {
        const int s = c & 1, row = row0 + c * SQ;
        if (!mbar_wait(&empty[s], ((c >> 1) & 1) ^ 1, abort_flag, p.status, 51, c)) break;
        uint8_t* st = sq_smem + s * SQ_STAGE;
        mbar_expect_tx(&full[s], (2 * nch + 1) * SQ_TILE + 2 * SQ_FB);
        for (int k = 0; k < nch; ++k) {
          tma_load_3d(st + k * SQ_TILE, &tmap_c, &full[s], k * 64, MEM ? h : p.G + g, row);
          tma_load_3d(st + (2 + k) * SQ_TILE, &tmap_b, &full[s], k * 64, g, row);
        }
        tma_load_3d(st + 4 * SQ_TILE, &tmap_x, &full[s], p0, h, row);
        sq_bulk_load(sq_smem + SQ_F + s * 2 * SQ_FB, p.cp + arr0 + c * arr_step, SQ_FB, &full[s]);
        sq_bulk_load(sq_smem + SQ_F + s * 2 * SQ_FB + SQ_FB, p.g + arr0 + c * arr_step, SQ_FB, &full[s]);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t id_sc = umma_idesc(128, 128, 1, 1, 0, 0);
      constexpr uint32_t id_y = umma_idesc(128, 64, 1, 1, 0, 1);
      constexpr uint32_t id_st = umma_idesc(128, 64, 1, 1, 1, 1);
      const uint32_t sbase = smem_u32(sq_smem);
      // 16-wide step k of a tile pair: along the 128-byte rows (K-major), or 16 rows further down (MN-major)
      auto kd = [](uint32_t tile, int k) { return umma_desc_kmajor_sw128(tile + (k >> 2) * SQ_TILE + (k & 3) * 32); };
      auto mn = [](uint32_t tile, int k) { return umma_desc_mnmajor_sw128(tile + k * 2048, SQ_TILE, 1024); };
      auto issue_sc = [&](int c) -> bool {
        if (!mbar_wait(&full[c & 1], (c >> 1) & 1, abort_flag, p.status, 52, c)) return false;
        tc_fence_after();
        const uint32_t cb = sbase + (c & 1) * SQ_STAGE, d = tmem + TC_SC + (c & 1) * 128;
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (k < ksn) umma_bf16(d, kd(cb, k), kd(cb + 2 * SQ_TILE, k), id_sc, k > 0);
        umma_commit(&sc_full[c & 1]);
        return true;
      };
      bool ok = issue_sc(0);
      for (int c = 0; c < n && ok; ++c) {
        const uint32_t ph = c & 1, cb = sbase + (c & 1) * SQ_STAGE;
        // ---- YO = C S
        if (!mbar_wait(s_full, ph, abort_flag, p.status, 53, c)) { ok = false; break; }
        tc_fence_after();
        {
          const uint32_t d = tmem + TC_YO + (c & 1) * 64;
#pragma unroll
          for (int k = 0; k < 8; ++k)
            if (k < ksn) {
              umma_bf16(d, kd(cb, k), mn(sbase + SQ_S, k), id_y, k > 0);
              umma_bf16(d, kd(cb, k), mn(sbase + SQ_S + SQ_TILE, k), id_y, 1u);
            }
        }
        umma_commit(yo_done);
        // ---- ST = B^T W
        if (!mbar_wait(w_full, ph, abort_flag, p.status, 54, c)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          umma_bf16(tmem + TC_ST, mn(cb + 2 * SQ_TILE, k), mn(sbase + SQ_W, k), id_st, k > 0);
          umma_bf16(tmem + TC_ST, mn(cb + 2 * SQ_TILE, k), mn(sbase + SQ_W + SQ_TILE, k), id_st, 1u);
        }
        umma_commit(st_full);
        // ---- the next chunk's scores, while this one's are worked on
        if (c + 1 < n && !issue_sc(c + 1)) { ok = false; break; }
        // ---- YD = M x
        if (!mbar_wait(m_full, ph, abort_flag, p.status, 55, c)) { ok = false; break; }
        if (c > 0 && !mbar_wait(y_empty, (c - 1) & 1, abort_flag, p.status, 56, c)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const uint32_t m = tmem + TC_SC + (c & 1) * 128 + k * 16;
          sq_umma_ts(tmem + TC_YD, m, mn(cb + 4 * SQ_TILE, k), id_y, k > 0);
          sq_umma_ts(tmem + TC_YD, m + 8, mn(cb + 4 * SQ_TILE, k), id_y, 1u);
        }
        umma_commit(y_full);
        umma_commit(&empty[c & 1]);
      }
    }
  } else if (warp < 10) {
    // ------------------------------------------------------------------ scores -> M, output rows
    const int qd = warp & 3, i = qd * 32 + lane, half = (warp - 2) >> 2;
    const uint32_t la = tmem + ((uint32_t)(qd * 32) << 16);
    const float Dh = MEM ? 0.f : p.D[h];
    const float* cumg = p.cum + arr0;
    const float* gm = MEM ? p.gmax + ((size_t)(row0 / SQ + r) * p.H + h) * 4 : nullptr;
    const float* min_g = MEM ? p.m_in + (size_t)(row0 / SQ + r) * p.H + h : nullptr;
    // this row's sum and the references of the first three blocks: the sums at their ends, or minus their largest i - b
    float ci = cumg[i], cb[3], mi = MEM ? min_g[0] : 0.f;
#pragma unroll
    for (int b = 0; b < 3; ++b) cb[b] = MEM ? -gm[b] : cumg[b * 32 + 31];
    float e_prev = 0.f;
    auto output = [&](int c, float e) -> bool {          // rows of chunk c: YD + e YO, 32 columns
      if (!mbar_wait(y_full, c & 1, abort_flag, p.status, 57, c)) return false;
      tc_fence_after();
      const int t = c * SQ + i;
      __nv_bfloat16* yr = p.y + (size_t)(row0 + t) * p.y_ld + h * p.P + p0;
#pragma unroll
      for (int q0 = 0; q0 < 32; q0 += 16) {
        const int q = half * 32 + q0;
        if (q < pw) {
          uint32_t yd[16], yo[16];
          __syncwarp();
          sq_tmem_ld_2x16(la + TC_YD + q, la + TC_YO + (c & 1) * 64 + q, yd, yo);
          if (t < n_rows) {
#pragma unroll
            for (int j = 0; j < 16; j += 8) {
              if (q + j < pw) {
                float v[8];
#pragma unroll
                for (int k = 0; k < 8; ++k) v[k] = fmaf(e, __uint_as_float(yo[j + k]), __uint_as_float(yd[j + k]));
                store_vec<8>(yr + q + j, v);
              }
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
      const float my = MEM ? ci + p.log2_scale : ci, c0 = cb[0], c1 = cb[1], c2 = cb[2];
      const float my_in = MEM ? my + mi : my;
      if (c + 1 < n) {                                   // the next chunk's, on their way while this one is worked on
        const float* nx = cumg + (c + 1) * arr_step;
        ci = nx[i];
#pragma unroll
        for (int b = 0; b < 3; ++b) cb[b] = MEM ? -gm[(size_t)(c + 1) * p.H * 4 + b] : nx[b * 32 + 31];
        if (MEM) mi = min_g[(size_t)(c + 1) * p.H];
      }
      if (!mbar_wait(&full[c & 1], (c >> 1) & 1, abort_flag, p.status, 58, c) ||
          !mbar_wait(&sc_full[c & 1], (c >> 1) & 1, abort_flag, p.status, 59, c)) { ok = false; break; }
      tc_fence_after();
      const float* cps = reinterpret_cast<const float*>(sq_smem + SQ_F + (c & 1) * 2 * SQ_FB) + half * 16;
      const float* gs = cps + SQ;
      const uint32_t col0 = la + TC_SC + (c & 1) * 128 + half * 16;
      uint32_t s[4][16];
      float rs = 0.f;                                    // MEM: sum of this thread's part of the row of M
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        if (b == 0) sq_tmem_ld_2x16(col0, col0 + 32, s[0], s[1]);          // blocks right of the diagonal are not used
        if (b == 2 && qd >= 2) sq_tmem_ld_2x16(col0 + 64, col0 + 96, s[2], s[3]);
        uint32_t hi[8], lo[8];
        if (b > qd) {                                    // right of the diagonal
#pragma unroll
          for (int j = 0; j < 8; ++j) hi[j] = lo[j] = 0u;
        } else if (b < qd) {
          const float f = sq_ex2(my - (b == 0 ? c0 : (b == 1 ? c1 : c2)));
#pragma unroll
          for (int j = 0; j < 16; j += 4) {
            const float4 gj = *reinterpret_cast<const float4*>(gs + b * 32 + j);
            const float m0 = __uint_as_float(s[b][j]) * (f * gj.x), m1 = __uint_as_float(s[b][j + 1]) * (f * gj.y);
            const float m2 = __uint_as_float(s[b][j + 2]) * (f * gj.z), m3 = __uint_as_float(s[b][j + 3]) * (f * gj.w);
            if (MEM) rs += (m0 + m1) + (m2 + m3);
            sq_split2(m0, m1, hi[j / 2], lo[j / 2]);
            sq_split2(m2, m3, hi[j / 2 + 1], lo[j / 2 + 1]);
          }
        } else {
          const int d = lane - half * 16;                // column of the diagonal among these 16
#pragma unroll
          for (int j = 0; j < 16; j += 4) {
            const float4 cj = *reinterpret_cast<const float4*>(cps + b * 32 + j);
            float m[4] = {cj.x, cj.y, cj.z, cj.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              m[e] = j + e <= d ? __uint_as_float(s[b][j + e]) * sq_ex2(my - m[e]) : 0.f;
              if (!MEM && j + e == d) m[e] += Dh;
            }
            if (MEM) rs += (m[0] + m[1]) + (m[2] + m[3]);
            sq_split2(m[0], m[1], hi[j / 2], lo[j / 2]);
            sq_split2(m[2], m[3], hi[j / 2 + 1], lo[j / 2 + 1]);
          }
        }
        __syncwarp();
        sq_tmem_st_x8(col0 + b * 32, hi);
        sq_tmem_st_x8(col0 + b * 32 + 8, lo);
      }
      tmem_st_wait();
      tc_fence_before();
      if (own_n) {                                       // n . q of this row: before m_full, which lets go of the chunk's tiles
        if (!mbar_wait(n_full, c & 1, abort_flag, p.status, 64, c)) { ok = false; break; }
        const float* sn = reinterpret_cast<const float*>(sq_smem + SQ_N);
        float dot = 0.f;
        for (int k8 = half; k8 * 8 < p.N; k8 += 2) {
          const uint4 q8 = *reinterpret_cast<const uint4*>(sq_smem + (c & 1) * SQ_STAGE + (k8 >> 3) * SQ_TILE + sq_off(i, k8 & 7));
          const float4 na = *reinterpret_cast<const float4*>(sn + k8 * 8), nb = *reinterpret_cast<const float4*>(sn + k8 * 8 + 4);
          const uint32_t v[4] = {q8.x, q8.y, q8.z, q8.w};
          float2 f[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) f[e] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v[e]));
          dot += (f[0].x * na.x + f[0].y * na.y) + (f[1].x * na.z + f[1].y * na.w) + (f[2].x * nb.x + f[2].y * nb.y) +
                 (f[3].x * nb.z + f[3].y * nb.w);
        }
        const int t = c * SQ + i;
        if (t < n_rows) atomicAdd(p.den + (size_t)(row0 + t) * p.H + h, fmaf(sq_ex2(my_in), dot, rs));      // two addends: order-free
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(m_full);
      if (c > 0 && !output(c - 1, e_prev)) { ok = false; break; }
      e_prev = sq_ex2(my_in);
    }
    if (ok) output(n - 1, e_prev);
  } else {
    // ------------------------------------------------------------------ W, state
    const int qd = warp & 3, i = qd * 32 + lane, half = (warp - 10) >> 2;      // token of the chunk, and row n of the state
    const uint32_t la = tmem + ((uint32_t)(qd * 32) << 16);
    const int q0 = half * 32, kn = i < p.N ? pw - q0 : 0;                      // columns of this half that exist
    const int PR = MEM ? p.P + 1 : p.P;
    float* st = p.state + (((size_t)slot * p.H + h) * PR + p0 + q0) * p.N + i;
    const bool fresh = p.positions[row0] == 0;
    // MEM: a lane owns channel nc of n for half of the tokens (those with bit 2 of their number set or not)
    const int nc = (warp - 10) * 16 + (lane & 15), nth = lane >> 4;
    float* st_n = p.state + (((size_t)slot * p.H + h) * PR + p.P) * p.N + nc;
    float n_now = 0.f, n_part = 0.f;
    auto write_n = [&]() {
      if (nth == 0) reinterpret_cast<float*>(sq_smem + SQ_N)[nc] = n_now;
      __syncwarp();
      if (lane == 0) mbar_arrive(n_full);
    };
    if (own_n) {
      if (!fresh && nc < p.N) n_now = *st_n;
      write_n();
    }
    float S[32];
    {
#pragma unroll
      for (int k = 0; k < 32; ++k) S[k] = (!fresh && k < kn) ? st[(size_t)k * p.N] : 0.f;
    }
    auto write_state = [&]() {
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) sq_split2(S[ch * 8 + 2 * e], S[ch * 8 + 2 * e + 1], hi[e], lo[e]);
        uint8_t* d = sq_smem + SQ_S + sq_off(i, half * 4 + ch);
        *reinterpret_cast<uint4*>(d) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(d + SQ_TILE) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(s_full);
    };
    write_state();
    const float* cend_g = p.cum + arr0 + SQ - 1;
    float cend = cend_g[0], cend_next = 0.f;
    const float* min_g = MEM ? p.m_in + (size_t)(row0 / SQ + r) * p.H + h : nullptr;
    const float* gm = MEM ? p.gmax + ((size_t)(row0 / SQ + r) * p.H + h) * 4 : nullptr;
    uint32_t wh[16], wl[16];                             // this token's W of the coming chunk
    auto prepare = [&](int c, float ce) -> bool {
      if (!mbar_wait(&full[c & 1], (c >> 1) & 1, abort_flag, p.status, 61, c)) return false;
      const uint8_t* xt = sq_smem + (c & 1) * SQ_STAGE + 4 * SQ_TILE;
      uint4 x[4];
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) x[ch] = *reinterpret_cast<const uint4*>(xt + sq_off(i, half * 4 + ch));
      const float cp = *(reinterpret_cast<const float*>(sq_smem + SQ_F + (c & 1) * 2 * SQ_FB) + i);
      const float w = sq_ex2(ce - cp);                   // 0 for rows past the end
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
        const uint32_t v[4] = {x[ch].x, x[ch].y, x[ch].z, x[ch].w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v[e]));
          sq_split2(f.x * w, f.y * w, wh[ch * 4 + e], wl[ch * 4 + e]);
        }
      }
      if (own_n) {                                       // sum of w_j k_j; before w_full, which lets go of the chunk's tiles
        n_part = 0.f;
        if (nc < p.N) {
          const uint8_t* kt = sq_smem + (c & 1) * SQ_STAGE + (2 + (nc >> 6)) * SQ_TILE + (nc & 7) * 2;
          const float* gs = reinterpret_cast<const float*>(sq_smem + SQ_F + (c & 1) * 2 * SQ_FB) + SQ;
#pragma unroll
          for (int b = 0; b < 4; ++b) {
            float acc = 0.f;
#pragma unroll
            for (int j4 = 0; j4 < 32; j4 += 8) {
              const int j = b * 32 + j4 + nth * 4;
              const float4 gj = *reinterpret_cast<const float4*>(gs + j);
              const float gv[4] = {gj.x, gj.y, gj.z, gj.w};
#pragma unroll
              for (int e = 0; e < 4; ++e)
                acc = fmaf(gv[e], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(kt + sq_off(j + e, (nc >> 3) & 7))), acc);
            }
            n_part = fmaf(sq_ex2(ce + gm[(size_t)c * p.H * 4 + b]), acc, n_part);
          }
        }
        n_part += __shfl_xor_sync(0xffffffffu, n_part, 16);
      }
      return true;
    };
    bool ok = prepare(0, cend);
    for (int c = 0; c < n && ok; ++c) {
      // W of the chunk before has been read: its ST was waited for
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
        uint8_t* d = sq_smem + SQ_W + sq_off(i, half * 4 + ch);
        *reinterpret_cast<uint4*>(d) = make_uint4(wh[4 * ch], wh[4 * ch + 1], wh[4 * ch + 2], wh[4 * ch + 3]);
        *reinterpret_cast<uint4*>(d + SQ_TILE) = make_uint4(wl[4 * ch], wl[4 * ch + 1], wl[4 * ch + 2], wl[4 * ch + 3]);
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(w_full);
      const float eend = sq_ex2(MEM ? cend + min_g[(size_t)c * p.H] : cend);
      if (own_n) n_now = fmaf(eend, n_now, n_part);      // n after this chunk; the next prepare overwrites n_part
      if (c + 1 < n) {
        cend_next = cend_g[(c + 1) * arr_step];
        if (!prepare(c + 1, cend_next)) break;
      }
      // ---- S <- exp(cum_end) S + ST
      if (!mbar_wait(st_full, c & 1, abort_flag, p.status, 62, c)) break;
      tc_fence_after();
      {
        uint32_t v[2][16];
        __syncwarp();
        sq_tmem_ld_2x16(la + TC_ST + q0, la + TC_ST + q0 + 16, v[0], v[1]);
#pragma unroll
        for (int j = 0; j < 32; ++j) S[j] = fmaf(eend, S[j], __uint_as_float(v[j >> 4][j & 15]));
      }
      tc_fence_before();
      if (c + 1 < n) {
        if (!mbar_wait(yo_done, c & 1, abort_flag, p.status, 63, c)) break;      // C S has read the old state
        write_state();
        if (own_n) {
          if (!mbar_wait(y_full, c & 1, abort_flag, p.status, 65, c)) break;     // every row has read the old n
          write_n();
        }
      }
      cend = cend_next;
    }
    if (!*abort_flag) {
#pragma unroll
      for (int k = 0; k < 32; ++k)
        if (k < kn) st[(size_t)k * p.N] = S[k];
      if (own_n && nth == 0 && nc < p.N) *st_n = n_now;
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

// Arguments as omni_ssm_scan (mamba2.cu); `rows` rows of xbc in all, at most max_q of one request.  Requests with fewer than
// min_rows rows are not touched.  scratch: 3 * (rows / 128 + B) * H * 128 floats.
extern "C" int omni_ssd_chunks(const void* xbc, int xbc_ld, long long rows, const void* dt, int dt_ld, const void* A_log,
                               const void* dt_bias, const void* D, void* state, const int* cu_q, const int64_t* positions,
                               const int* state_slots, int B, int max_q, void* y, int y_ld, int H, int P, int N, int G,
                               int min_rows, float* scratch, void* status, cudaStream_t stream) {
  if (B <= 0 || rows <= 0 || max_q < min_rows) return 0;
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
  const size_t arr = (size_t)(rows / SQ + B) * H * SQ;
  p.cum = scratch; p.cp = scratch + arr; p.g = scratch + 2 * arr;
  ssd_decay_kernel<<<dim3((max_q + SQ - 1) / SQ, B, (H + 7) / 8), SQ, 0, stream>>>(p);
  static bool configured[64] = {false};
  if (int e = ensure_dyn_smem((const void*)ssd_sm100_kernel<false>, SQ_SMEM, configured)) return e;
  ssd_sm100_kernel<false><<<dim3((P + 63) / 64, H, B), SQ_THREADS, SQ_SMEM, stream>>>(tbc, tbc, tx, p);
  return (int)cudaGetLastError();
}

// Matrix memory over portions of prompts.  q, k, v [rows, ld] with head h at column h N / h N / h P; chunks: what omni_mlstm_gates
// left (n_chunks = rows / 128 + B of them); state [slots, H, P + 1, N]; den [rows, H] zeroed; y = S^T q N^-1/2.
extern "C" int omni_mlstm_chunks(const void* q, int q_ld, const void* k, int k_ld, const void* v, int v_ld, long long rows,
                                 const float* chunks, int n_chunks, float* den, float scale, void* state, const int* cu_q,
                                 const int64_t* positions, const int* state_slots, int B, int max_q, void* y, int y_ld, int H, int P,
                                 int N, int min_rows, void* status, cudaStream_t stream) {
  if (B <= 0 || rows <= 0 || max_q < min_rows) return 0;
  if (H < 1 || B > 65535 || H > 65535 || !(scale > 0.f) || chunks == nullptr || n_chunks < rows / SQ + B) return -1;
  if (P < 8 || P % 8 != 0 || N < 8 || N % 8 != 0 || N > 128 || (q_ld | k_ld | v_ld | y_ld) % 8 != 0) return -2;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)y | (uintptr_t)chunks) % 16 != 0) return -3;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d(&tq, q, 2, N, H, (uint64_t)rows, (uint64_t)N * 2, (uint64_t)q_ld * 2, 64, 1, SQ, true)) return -10;
  if (make_tmap_3d(&tk, k, 2, N, H, (uint64_t)rows, (uint64_t)N * 2, (uint64_t)k_ld * 2, 64, 1, SQ, true)) return -11;
  if (make_tmap_3d(&tv, v, 2, P, H, (uint64_t)rows, (uint64_t)P * 2, (uint64_t)v_ld * 2, 64, 1, SQ, true)) return -12;
  SsdParams p;
  memset(&p, 0, sizeof(p));
  const size_t arr = (size_t)n_chunks * H * SQ;
  p.cum = const_cast<float*>(chunks); p.cp = p.cum + arr; p.g = p.cum + 2 * arr; p.gmax = p.cum + 3 * arr;
  p.m_in = p.gmax + (size_t)n_chunks * H * 4; p.den = den; p.log2_scale = log2f(scale);
  p.state = (float*)state; p.cu_q = cu_q; p.positions = positions; p.state_slots = state_slots;
  p.y = (__nv_bfloat16*)y; p.y_ld = y_ld; p.H = H; p.P = P; p.N = N; p.G = H; p.min_rows = min_rows;
  p.status = (OmniStatus*)status;
  static bool configured[64] = {false};
  if (int e = ensure_dyn_smem((const void*)ssd_sm100_kernel<true>, SQ_SMEM, configured)) return e;
  ssd_sm100_kernel<true><<<dim3((P + 63) / 64, H, B), SQ_THREADS, SQ_SMEM, stream>>>(tq, tk, tv, p);
  return (int)cudaGetLastError();
}
