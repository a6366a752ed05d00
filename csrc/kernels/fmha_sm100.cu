// Variable-length causal attention for prefill (tcgen05 + TMEM) and GQA paged decode.
//
// omni_fmha_varlen: one CTA per (q head, request, 128-query tile).
//   S = Q K^T     A = Q tile (smem, K-major, 64-dim chunks)   B = K tile of 64 keys (smem, K-major)
//   P = softmax   kept in TMEM as packed bf16                  (thread = query row: no cross-thread reductions)
//   O += P V      A = P (TMEM)                                 B = V tile (smem, MN-major), 128 output dims
// The key dimension may come from two tensors: `k` (per kv head) and `k2` (shared by all heads).  That is how
// MLA prefill runs without materialising [k_nope | k_pe]: k/v are column slices of the kv_b_proj output,
// k2 is the roped k_pe slice of the latent rows.  GQA (Qwen) uses k only, with q heads mapped to kv heads.
// omni_fmha_paged: the same kernel reading K and V tiles from the paged cache through the block table (any head sizes
// up to 192 / 128 that are multiples of 8: the tensor maps are [rows, heads, head size], so a partial 64-wide chunk is
// zero-filled), with an optional sliding window - key tiles outside every query's window are never loaded - and with the
// softmax weights carried as a pair of bf16 values (p = hi + lo, two MMAs), i.e. to 16 bits of mantissa; optionally a sink per
// head in the softmax denominator and a factor on the result, kept first keys beside the window (their tiles come first), chunks
// instead of it, a gate per output element, and capped or biased scores (an instantiation of its own).
// omni_fmha_latent: contiguous key rows as in the first form, but with any head sizes, the window, the pair of bf16 weights and a
// gate per row and head, and with the sinks of the second: latent attention over keys and values that were projected from their latents.
// Causal mask is aligned to the end of the key range (query i of a request with Lq queries and Lk keys sees
// keys <= Lk - Lq + i), which also covers chunked prefill and prefix-cache hits.
//
// The paged decode of the GQA models (one query token per request) is a separate kernel: gqa_decode.cu.
//
// Reference call sites: npu_fused_infer_attention_score / npu_fusion_attention
// (omni/models/common/layers/attention/deepseek_mla.py:386-400, omni/models/common/layers/attention/backend/attention.py:590-666).
#include "../include/omni_ptx.cuh"
#include "../include/score_mod.cuh"
#include "../include/tma_host.h"

namespace omni {

enum { FM_DENSE = 0, FM_PAGED = 1, FM_PAGED_MOD = 2, FM_LATENT = 3 };

struct FmhaParams {
  const int* cu_q;   // [B] first row of each request
  const int* end_q;  // [B] and the row after its last: cu_q + 1 where requests follow one another
  const int* cu_k;
  const int* end_k;
  int Hq, Hkv;
  int q_head_stride, k_head_stride, v_head_stride;  // in elements (column offset per head)
  int v_col0, k2_col0;
  int nk1, nk2;      // number of 64-wide key chunks taken from k and from k2
  float scale_log2;
  int causal;
  __nv_bfloat16* out;  // [Tq, Hq * dv], row pitch out_ld
  int dv, out_ld;
  // paged variant: keys of request b live in blocks of the cache, kv_len[b] of them (cu_k is not used)
  const int* kv_len;
  const int* block_table;
  int bt_ld, block_size;
  int window;          // a query sees the last `window` keys up to its own; 0 = all
  int chunk, keep;     // see first_key; the first `keep` keys are visible in any case
  ScoreMod score;      // FM_PAGED_MOD
  // [Tq, gate_ld] or null: the result of head h is multiplied by sigmoid(gate[t, h]) (latent), or of column d of it by
  // sigmoid(gate[t, h dv + d]) (paged)
  const __nv_bfloat16* gate;
  int gate_ld;
  const float* sink;   // [Hq] or null: exp(sink) is one more term of the softmax denominator
  float out_scale;     // multiplies the result before it is rounded
  OmniStatus* status;
};

constexpr int FM_BQ = 128, FM_BK = 64, FM_DV = 128;
constexpr int FM_QCHUNK = FM_BQ * 128;          // 16 KB
constexpr int FM_KCHUNK = FM_BK * 128;          // 8 KB
constexpr int FM_MAXC = 3;                      // up to 192 qk dims
constexpr int FM_V_STAGE = 2 * FM_KCHUNK;       // 16 KB
constexpr int FM_THREADS = 192;
// Shared memory and TMEM layout.  MAXC: 64-wide chunks of the qk size that fit.  The paged kernel with two chunks and two
// stages takes 98 KB and 256 TMEM columns, so that two CTAs share an SM and one's softmax overlaps the other's MMAs; its P
// (32 columns hi, 32 columns lo) replaces the 64 columns of the S tile that it was computed from, which the next QK^T but
// one writes again only after the PV that reads P (the MMAs of a CTA complete in order).
template <int MODE, int MAXC, int STAGES>
struct FmLayout {
  static constexpr bool EXACT = MODE != FM_DENSE;
  static constexpr int K_STAGE = MAXC * FM_KCHUNK;
  static constexpr int SMEM = MAXC * FM_QCHUNK + STAGES * (K_STAGE + FM_V_STAGE) + 1024 + 1024;
  static constexpr int T_O = 0, T_S = 128, T_P = EXACT ? T_S : 256, T_P_STRIDE = EXACT ? FM_BK : FM_BK / 2;
  static constexpr int T_COLS = EXACT ? 256 : 512;
};

__device__ __forceinline__ void fm_umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc,
                                           uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

template <int MODE, int MAXC, int STAGES>
__global__ void __launch_bounds__(FM_THREADS, (MODE != FM_DENSE && MAXC == 2) ? 2 : 1)
fmha_varlen_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_q2,
                   const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_k2,
                   const __grid_constant__ CUtensorMap tmap_v, const FmhaParams p) {
  constexpr bool PAGED = MODE == FM_PAGED || MODE == FM_PAGED_MOD;      // keys through the block table
  constexpr bool EXACT = MODE != FM_DENSE;                              // any head sizes, masks, softmax weights as hi + lo
  // the last query tiles of the requests see the most keys: they come first, so that the short ones fill the gaps at the end
  const int b = blockIdx.y, h = blockIdx.x;
  const int q_begin = p.cu_q[b], q_end = p.end_q[b];
  const int k_begin = PAGED ? 0 : p.cu_k[b];
  const int Lq = q_end - q_begin, Lk = PAGED ? p.kv_len[b] : p.end_k[b] - k_begin;
  const int q0 = (gridDim.z - 1 - blockIdx.z) * FM_BQ;
  if (q0 >= Lq) return;  // uniform for the whole CTA, before any barrier / TMEM use
  const int ctx = Lk - Lq;
  const int hk = h / (p.Hq / p.Hkv);
  const int nc = p.nk1 + p.nk2;
  // keys this tile can see
  int k_hi = p.causal ? min(Lk, ctx + q0 + FM_BQ) : Lk;
  // first key tile that the tile's first query sees, but for those of kept keys, which come ahead of it
  const int t_first = EXACT ? first_key(ctx + q0, p.window, p.chunk) / FM_BK : 0;
  const int n_keep = PAGED ? min((p.keep + FM_BK - 1) / FM_BK, t_first) : 0;
  const int n = n_keep + (k_hi + FM_BK - 1) / FM_BK - t_first;
  auto first_of_tile = [&](int i) { return (PAGED && i < n_keep ? i : t_first - n_keep + i) * FM_BK; };
  const int nv = EXACT ? (p.dv + 63) / 64 : 2;         // 64-wide chunks of the value size

  using L = FmLayout<MODE, MAXC, STAGES>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* sq = smem;
  uint8_t* sk = smem + MAXC * FM_QCHUNK;
  uint8_t* sv = sk + STAGES * L::K_STAGE;
  uint64_t* bars = (uint64_t*)(sv + STAGES * FM_V_STAGE);
  uint64_t* q_full = bars;                       // 1
  uint64_t* k_full = bars + 1;                   // STAGES
  uint64_t* k_empty = k_full + STAGES;
  uint64_t* v_full = k_empty + STAGES;
  uint64_t* v_empty = v_full + STAGES;
  uint64_t* s_full = v_empty + STAGES;        // 2
  uint64_t* p_full = s_full + 2;                 // 2
  uint64_t* o_done = p_full + 2;                 // 1
  uint64_t* o_final = o_done + 1;                // 1
  uint32_t* tmem_slot = (uint32_t*)(o_final + 1);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&p_full[s], 4); }
    mbar_init(o_done, 1);
    mbar_init(o_final, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, L::T_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, nc * FM_QCHUNK);
      for (int c = 0; c < nc; ++c) {
        if (EXACT && c < p.nk1) tma_load_3d(sq + c * FM_QCHUNK, &tmap_q, q_full, c * 64, h, q_begin + q0);
        else if (EXACT) tma_load_3d(sq + c * FM_QCHUNK, &tmap_q2, q_full, (c - p.nk1) * 64, h, q_begin + q0);
        else tma_load_2d(sq + c * FM_QCHUNK, &tmap_q, q_full, h * p.q_head_stride + c * 64, q_begin + q0);
      }
      for (int i = 0; i < n; ++i) {
        const int st = i % STAGES;
        const uint32_t ph = (i / STAGES) & 1;
        const int key0 = first_of_tile(i);
        int row = k_begin + key0;
        if (PAGED) {
          row = p.block_table[(size_t)b * p.bt_ld + key0 / p.block_size] * p.block_size + key0 % p.block_size;
        }
        if (!mbar_wait(&k_empty[st], ph ^ 1, abort_flag, p.status, 11, i)) break;
        mbar_expect_tx(&k_full[st], nc * FM_KCHUNK);
        for (int c = 0; c < p.nk1; ++c) {
          if (EXACT) tma_load_3d(sk + st * L::K_STAGE + c * FM_KCHUNK, &tmap_k, &k_full[st], c * 64, hk, row);
          else tma_load_2d(sk + st * L::K_STAGE + c * FM_KCHUNK, &tmap_k, &k_full[st], hk * p.k_head_stride + c * 64, row);
        }
        for (int c = 0; c < p.nk2; ++c)
          tma_load_2d(sk + st * L::K_STAGE + (p.nk1 + c) * FM_KCHUNK, &tmap_k2, &k_full[st], p.k2_col0 + c * 64, row);
        if (!mbar_wait(&v_empty[st], ph ^ 1, abort_flag, p.status, 12, i)) break;
        mbar_expect_tx(&v_full[st], nv * FM_KCHUNK);
        for (int c = 0; c < nv; ++c) {
          if (EXACT) tma_load_3d(sv + st * FM_V_STAGE + c * FM_KCHUNK, &tmap_v, &v_full[st], c * 64, hk, row);
          else tma_load_2d(sv + st * FM_V_STAGE + c * FM_KCHUNK, &tmap_v, &v_full[st],
                           hk * p.v_head_stride + p.v_col0 + c * 64, row);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_qk = umma_idesc(128, FM_BK, 1, 1, 0, 0);
      const uint32_t idesc_pv = umma_idesc(128, nv * 64, 1, 1, 0, 1);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status, 13, 0);
      auto issue_qk = [&](int j) -> bool {
        const int st = j % STAGES;
        if (!mbar_wait(&k_full[st], (j / STAGES) & 1, abort_flag, p.status, 14, j)) return false;
        tc_fence_after();
        const uint32_t d = tmem_base + L::T_S + (j & 1) * FM_BK;
        uint32_t accum = 0;
        for (int c = 0; c < nc; ++c) {
          const uint64_t ad = umma_desc_kmajor_sw128(smem_u32(sq) + c * FM_QCHUNK);
          const uint64_t bd = umma_desc_kmajor_sw128(smem_u32(sk) + st * L::K_STAGE + c * FM_KCHUNK);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            umma_bf16(d, ad + 2 * k, bd + 2 * k, idesc_qk, accum);
            accum = 1;
          }
        }
        umma_commit(&k_empty[st]);
        umma_commit(&s_full[j & 1]);
        return true;
      };
      if (ok) ok = issue_qk(0);
      if (ok && n > 1) ok = issue_qk(1);
      for (int i = 0; i < n && ok; ++i) {
        const int st = i % STAGES;
        if (!mbar_wait(&p_full[i & 1], (i >> 1) & 1, abort_flag, p.status, 15, i)) { ok = false; break; }
        if (!mbar_wait(&v_full[st], (i / STAGES) & 1, abort_flag, p.status, 16, i)) { ok = false; break; }
        tc_fence_after();
        const uint32_t vbase = smem_u32(sv) + st * FM_V_STAGE;
#pragma unroll
        for (int k = 0; k < FM_BK / 16; ++k) {
          const uint64_t bd = umma_desc_mnmajor_sw128(vbase + k * 2048, FM_KCHUNK, 1024);
          fm_umma_ts(tmem_base + L::T_O, tmem_base + L::T_P + (i & 1) * L::T_P_STRIDE + k * 8, bd, idesc_pv,
                     (i > 0 || k > 0) ? 1u : 0u);
          if (EXACT) fm_umma_ts(tmem_base + L::T_O, tmem_base + L::T_P + FM_BK / 2 + (i & 1) * L::T_P_STRIDE + k * 8, bd, idesc_pv, 1u);
        }
        umma_commit(&v_empty[st]);
        umma_commit(o_done);
        if (i == n - 1) umma_commit(o_final);
        if (i + 2 < n) ok = issue_qk(i + 2);
      }
    }
  } else {
    const int qd = warp & 3;
    const int row = qd * 32 + lane;          // query row inside the tile
    const uint32_t lane_addr = tmem_base + ((uint32_t)(qd * 32) << 16);
    const int q_pos = ctx + q0 + row;        // last key index this row may see (causal)
    const int first = EXACT ? first_key(q_pos, p.window, p.chunk) : 0;
    float slope = 0.f;
    if (MODE == FM_PAGED_MOD && p.score.slopes != nullptr) slope = p.score.slopes[h] * 1.4426950408889634f;
    float r1 = 0.f, r2 = 0.f;
    if (MODE == FM_PAGED_MOD && p.score.r1 != nullptr) { r1 = p.score.r1[h]; r2 = p.score.r2[h]; }
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n; ++i) {
      if (!mbar_wait(&s_full[i & 1], (i >> 1) & 1, abort_flag, p.status, 17, i)) { ok = false; break; }
      tc_fence_after();
      const int kbase = first_of_tile(i);
      int lim = Lk - kbase;                        // keys beyond the request end are masked
      if (p.causal) lim = min(lim, q_pos - kbase + 1);
      const int low = first - kbase;               // and those before the window, but for the kept ones
      const int kept = p.keep - kbase;
      float dist_bias = 0.f;                       // of column 0
      if (MODE == FM_PAGED_MOD) dist_bias = slope * (float)(q_pos - kbase);
      // raw scores (their scale is positive and enters with the subtraction of the maximum), or final ones in log2 units
      float s[FM_BK];
      {
        uint32_t lo32[32], hi32[32];
        tmem_ld_x32(lane_addr + L::T_S + (i & 1) * FM_BK, lo32);
        tmem_ld_x32(lane_addr + L::T_S + (i & 1) * FM_BK + 32, hi32);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) { s[j] = __uint_as_float(lo32[j]); s[32 + j] = __uint_as_float(hi32[j]); }
      }
      if (MODE == FM_PAGED_MOD) {
        if (p.score.cap_log2 > 0.f) {
#pragma unroll
          for (int j = 0; j < FM_BK; ++j) s[j] = capped(p.score, s[j], fmaf(slope, (float)j, -dist_bias));
        } else {
#pragma unroll
          for (int j = 0; j < FM_BK; ++j) s[j] = fmaf(s[j], p.scale_log2, fmaf(slope, (float)j, -dist_bias));
        }
        if (p.score.r1 != nullptr) {
          const float dist = (float)(q_pos - kbase);      // to column 0; keys ahead of the query are masked below
#pragma unroll
          for (int j = 0; j < FM_BK; ++j) s[j] -= log_bias(r1, r2, fmaxf(dist - (float)j, 0.f));
        }
      }
      if (!__all_sync(0xffffffffu, lim >= FM_BK && (!EXACT || low <= 0 || (PAGED && kept >= FM_BK)))) {
#pragma unroll
        for (int j = 0; j < FM_BK; ++j)
          if (!(j < lim && (!EXACT || j >= low || (PAGED && j < kept)))) s[j] = -INFINITY;
      }
      float mx4[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int j = 4; j < FM_BK; j += 4) {
        mx4[0] = fmaxf(mx4[0], s[j]); mx4[1] = fmaxf(mx4[1], s[j + 1]);
        mx4[2] = fmaxf(mx4[2], s[j + 2]); mx4[3] = fmaxf(mx4[3], s[j + 3]);
      }
      const float unit = MODE == FM_PAGED_MOD ? 1.f : p.scale_log2;
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * unit;
      // A row that has seen no key yet (its window starts in a later tile, or it lies past the end of the request)
      // has nothing accumulated: it takes the maximum over as it is.
      const float m_new = fmaxf(m, mx);
      const bool grow = m != -INFINITY && (m_new - m) > 8.0f;
      if (m == -INFINITY) m = m_new;
      if (i > 0 && __any_sync(0xffffffffu, grow)) {
        if (!mbar_wait(o_done, (i - 1) & 1, abort_flag, p.status, 18, i)) { ok = false; break; }
        tc_fence_after();
        const float f = grow ? ex2_fast(m - m_new) : 1.0f;
        if (grow) { l *= f; m = m_new; }
#pragma unroll 1
        for (int c = 0; c < nv * 64; c += 32) {
          uint32_t ov[32];
          tmem_ld_x32(lane_addr + L::T_O + c, ov);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) ov[j] = __float_as_uint(__uint_as_float(ov[j]) * f);
          tmem_st_x32(lane_addr + L::T_O + c, ov);
        }
        tmem_st_wait();
      }
      uint32_t pk[32], pl[32];
      const float m_ref = m == -INFINITY ? 0.f : m;
      const f32x2 unit2 = pack_f32x2(unit, unit), neg_m2 = pack_f32x2(-m_ref, -m_ref), minus2 = pack_f32x2(-1.f, -1.f);
      f32x2 rs2[2] = {0ull, 0ull};
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        float p0, p1;
        unpack_f32x2(fma_f32x2(pack_f32x2(s[2 * j], s[2 * j + 1]), unit2, neg_m2), p0, p1);
        p0 = ex2_fast(p0);
        p1 = ex2_fast(p1);
        const f32x2 pp = pack_f32x2(p0, p1);
        rs2[j & 1] = add_f32x2(rs2[j & 1], pp);
        __nv_bfloat162 h2 = __floats2bfloat162_rn(p0, p1);
        const uint32_t hb = *reinterpret_cast<uint32_t*>(&h2);
        pk[j] = hb;
        if (EXACT) {      // what the rounding to bf16 left over
          unpack_f32x2(fma_f32x2(pack_f32x2(__uint_as_float(hb << 16), __uint_as_float(hb & 0xffff0000u)), minus2, pp), p0, p1);
          h2 = __floats2bfloat162_rn(p0, p1);
          pl[j] = *reinterpret_cast<uint32_t*>(&h2);
        }
      }
      {
        float a, b;
        unpack_f32x2(add_f32x2(rs2[0], rs2[1]), a, b);
        l += a + b;
      }
      tmem_st_x32(lane_addr + L::T_P + (i & 1) * L::T_P_STRIDE, pk);
      if (EXACT) tmem_st_x32(lane_addr + L::T_P + FM_BK / 2 + (i & 1) * L::T_P_STRIDE, pl);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[i & 1]);
    }
    if (ok) ok = mbar_wait(o_final, 0, abort_flag, p.status, 19, n);
    if (ok) {
      tc_fence_after();
      const bool row_ok = (q0 + row) < Lq;
      float den = l;
      if (EXACT && p.sink != nullptr && m != -INFINITY) den += exp2f(p.sink[h] * 1.4426950408889634f - m);
      float inv_l = l > 0.f ? (EXACT ? p.out_scale : 1.0f) / den : 0.f;
      if (MODE == FM_LATENT && p.gate != nullptr && row_ok)
        inv_l /= 1.f + __expf(-__bfloat162float(p.gate[(size_t)(q_begin + q0 + row) * p.gate_ld + h]));
      __nv_bfloat16* orow = p.out + (size_t)(q_begin + q0 + row) * p.out_ld + h * p.dv;
#pragma unroll 1
      for (int c = 0; c < p.dv; c += 32) {
        uint32_t ov[32];
        tmem_ld_x32(lane_addr + L::T_O + c, ov);
        tmem_ld_wait();
        if (row_ok) {
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (EXACT && c + j >= p.dv) break;
            float g8[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) g8[e] = inv_l;
            if (PAGED && p.gate != nullptr) {
              const uint4 gv = *reinterpret_cast<const uint4*>(p.gate + (size_t)(q_begin + q0 + row) * p.gate_ld + h * p.dv + c + j);
              const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(g2[e]);
                g8[2 * e] = __fdividef(inv_l, 1.f + __expf(-f.x));
                g8[2 * e + 1] = __fdividef(inv_l, 1.f + __expf(-f.y));
              }
            }
            __nv_bfloat16 o8[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) o8[e] = __float2bfloat16(__uint_as_float(ov[j + e]) * g8[e]);
            *reinterpret_cast<uint4*>(orow + c + j) = *reinterpret_cast<uint4*>(o8);
          }
        }
      }
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
    tmem_dealloc(tmem_base, L::T_COLS);
  }
}

}  // namespace omni

using namespace omni;

template <int MODE, int MAXC, int STAGES>
static int launch_fmha(dim3 grid, const CUtensorMap& tq, const CUtensorMap& tq2, const CUtensorMap& tk, const CUtensorMap& tk2,
                       const CUtensorMap& tv, const FmhaParams& p, cudaStream_t stream) {
  constexpr int smem = FmLayout<MODE, MAXC, STAGES>::SMEM;
  static bool configured[64] = {false};
  if (int e = ensure_dyn_smem((const void*)fmha_varlen_kernel<MODE, MAXC, STAGES>, smem, configured)) return e;
  fmha_varlen_kernel<MODE, MAXC, STAGES><<<grid, FM_THREADS, smem, stream>>>(tq, tq2, tk, tk2, tv, p);
  return (int)cudaGetLastError();
}

// q/k/k2/v are 2-D row-major bf16 matrices given by (pointer, rows, row pitch in elements, columns).
extern "C" int omni_fmha_varlen(const void* q, long long q_rows, int q_ld, int q_cols, const void* k, long long k_rows,
                                int k_ld, int k_cols, const void* k2, int k2_ld, int k2_cols, const void* v, int v_ld,
                                int v_cols, const int* cu_q, const int* cu_k, int B, int max_q, int Hq, int Hkv,
                                int q_head_stride, int k_head_stride, int v_head_stride, int v_col0, int k2_col0,
                                int d_k1, int d_k2, int d_v, float scale, int causal, void* out, void* status,
                                cudaStream_t stream) {
  if (B <= 0 || max_q <= 0) return 0;
  if (d_v != 128 || d_k1 % 64 != 0 || d_k2 % 64 != 0 || (d_k1 + d_k2) > 64 * FM_MAXC) return -1;
  if (Hq % Hkv != 0) return -2;
  CUtensorMap tq, tk, tk2, tv;
  if (make_tmap_2d(&tq, q, 2, (uint64_t)q_rows, q_cols, q_ld, FM_BQ, 64, true)) return -10;
  if (make_tmap_2d(&tk, k, 2, (uint64_t)k_rows, k_cols, k_ld, FM_BK, 64, true)) return -11;
  if (d_k2 > 0) {
    if (make_tmap_2d(&tk2, k2, 2, (uint64_t)k_rows, k2_cols, k2_ld, FM_BK, 64, true)) return -12;
  } else {
    tk2 = tk;
  }
  if (make_tmap_2d(&tv, v, 2, (uint64_t)k_rows, v_cols, v_ld, FM_BK, 64, true)) return -13;
  FmhaParams p;
  memset(&p, 0, sizeof(p));
  p.cu_q = cu_q; p.end_q = cu_q + 1; p.cu_k = cu_k; p.end_k = cu_k + 1; p.Hq = Hq; p.Hkv = Hkv; p.q_head_stride = q_head_stride;
  p.k_head_stride = k_head_stride; p.v_head_stride = v_head_stride; p.v_col0 = v_col0; p.k2_col0 = k2_col0;
  p.nk1 = d_k1 / 64; p.nk2 = d_k2 / 64; p.scale_log2 = scale * 1.4426950408889634f; p.causal = causal;
  p.out = (__nv_bfloat16*)out; p.status = (OmniStatus*)status;
  p.dv = FM_DV; p.out_ld = Hq * FM_DV;
  p.out_scale = 1.0f;
  return launch_fmha<FM_DENSE, FM_MAXC, 3>(dim3(Hq, B, (max_q + FM_BQ - 1) / FM_BQ), tq, tq, tk, tk2, tv, p, stream);
}

// Ragged queries against the paged cache.  q: rows of pitch q_ld holding Hq heads of d_k; k_cache / v_cache
// [slots, Hkv, d_k / d_v]; kv_len[b] keys of request b, of which its cu_q segment is the end; out rows of pitch out_ld.
extern "C" int omni_fmha_paged(const void* q, long long q_rows, int q_ld, const void* k_cache, const void* v_cache,
                               long long slots, const int* cu_q, const int* kv_len, const int* block_table, int bt_ld, int B,
                               int max_q, int Hq, int Hkv, int d_k, int d_v, int block_size, int window, int chunk, int keep,
                               float scale, float softcap, const float* slopes, const float* r1, const float* r2, const float* sink,
                               const void* gate, int gate_ld, float out_scale, void* out, int out_ld, void* status, cudaStream_t stream) {
  if (B <= 0 || max_q <= 0) return 0;
  if (d_k < 8 || d_v < 8 || d_k % 8 != 0 || d_v % 8 != 0 || d_k > 64 * FM_MAXC || d_v > FM_DV) return -1;
  if (Hkv < 1 || Hq % Hkv != 0 || B > 65535 || max_q > 65535 * FM_BQ || window < 0 || chunk < 0 || keep < 0) return -2;
  if (block_size < FM_BK || block_size % FM_BK != 0 || q_ld % 8 != 0 || out_ld % 8 != 0) return -3;
  if ((r1 == nullptr) != (r2 == nullptr) || (gate != nullptr && (gate_ld % 8 != 0 || (uintptr_t)gate % 16 != 0 || gate_ld < Hq * d_v))) return -5;
  if (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)out) % 16 != 0) return -4;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d(&tq, q, 2, d_k, Hq, (uint64_t)q_rows, (uint64_t)d_k * 2, (uint64_t)q_ld * 2, 64, 1, FM_BQ, true)) return -10;
  if (make_tmap_3d(&tk, k_cache, 2, d_k, Hkv, (uint64_t)slots, (uint64_t)d_k * 2, (uint64_t)Hkv * d_k * 2, 64, 1, FM_BK, true))
    return -11;
  if (make_tmap_3d(&tv, v_cache, 2, d_v, Hkv, (uint64_t)slots, (uint64_t)d_v * 2, (uint64_t)Hkv * d_v * 2, 64, 1, FM_BK, true))
    return -13;
  FmhaParams p;
  memset(&p, 0, sizeof(p));
  p.cu_q = cu_q; p.end_q = cu_q + 1; p.Hq = Hq; p.Hkv = Hkv; p.nk1 = (d_k + 63) / 64; p.nk2 = 0;
  p.scale_log2 = scale * 1.4426950408889634f; p.causal = 1; p.out = (__nv_bfloat16*)out; p.status = (OmniStatus*)status;
  p.dv = d_v; p.out_ld = out_ld; p.kv_len = kv_len; p.block_table = block_table; p.bt_ld = bt_ld;
  p.block_size = block_size; p.window = window; p.chunk = chunk; p.keep = keep; p.sink = sink; p.out_scale = out_scale;
  p.score = make_score_mod(scale, softcap, slopes, r1, r2); p.gate = (const __nv_bfloat16*)gate; p.gate_ld = gate_ld;
  const dim3 grid(Hq, B, (max_q + FM_BQ - 1) / FM_BQ);
  if (softcap > 0.f || slopes != nullptr || r1 != nullptr) {
    if (p.nk1 <= 2) return launch_fmha<FM_PAGED_MOD, 2, 2>(grid, tq, tq, tk, tk, tv, p, stream);
    return launch_fmha<FM_PAGED_MOD, FM_MAXC, 3>(grid, tq, tq, tk, tk, tv, p, stream);
  }
  if (p.nk1 <= 2) return launch_fmha<FM_PAGED, 2, 2>(grid, tq, tq, tk, tk, tv, p, stream);
  return launch_fmha<FM_PAGED, FM_MAXC, 3>(grid, tq, tq, tk, tk, tv, p, stream);
}

// Latent attention of ragged queries over projected keys.  q rows of pitch q_ld: per head d1 unrotated | d2 rotated; kv rows of
// pitch kv_ld: per head d1 keys | d_v values; k2 rows of pitch k2_ld: the d2 rotated key columns that all heads share.  Request
// b has query rows q_start[b] .. q_end[b] and key rows k_start[b] .. k_end[b], whose last ones belong to its queries.
extern "C" int omni_fmha_latent(const void* q, long long q_rows, int q_ld, const void* kv, long long k_rows, int kv_ld,
                                const void* k2, int k2_ld, const int* q_start, const int* q_end, const int* k_start,
                                const int* k_end, int B, int max_q, int H, int d1, int d2, int d_v, int window, float scale,
                                const void* gate, int gate_ld, const float* sink, void* out, int out_ld, void* status, cudaStream_t stream) {
  if (B <= 0 || max_q <= 0) return 0;
  const int nk1 = (d1 + 63) / 64, nk2 = (d2 + 63) / 64;
  if (d1 < 8 || d2 < 8 || d_v < 8 || d1 % 8 != 0 || d2 % 8 != 0 || d_v % 8 != 0 || nk1 + nk2 > FM_MAXC || d_v > FM_DV) return -1;
  if (H < 1 || B > 65535 || max_q > 65535 * FM_BQ || window < 0 || q_rows < 1 || k_rows < 1) return -2;
  if (q_ld % 8 != 0 || kv_ld % 8 != 0 || k2_ld % 8 != 0 || out_ld % 8 != 0 || q_ld < H * (d1 + d2) || kv_ld < H * (d1 + d_v)) return -3;
  if (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)k2 | (uintptr_t)out) % 16 != 0) return -4;
  CUtensorMap tq, tq2, tk, tk2, tv;
  const __nv_bfloat16 *qb = (const __nv_bfloat16*)q, *kb = (const __nv_bfloat16*)kv;
  const uint64_t q_head = (uint64_t)(d1 + d2) * 2, k_head = (uint64_t)(d1 + d_v) * 2;
  if (make_tmap_3d(&tq, qb, 2, d1, H, (uint64_t)q_rows, q_head, (uint64_t)q_ld * 2, 64, 1, FM_BQ, true)) return -10;
  if (make_tmap_3d(&tq2, qb + d1, 2, d2, H, (uint64_t)q_rows, q_head, (uint64_t)q_ld * 2, 64, 1, FM_BQ, true)) return -11;
  if (make_tmap_3d(&tk, kb, 2, d1, H, (uint64_t)k_rows, k_head, (uint64_t)kv_ld * 2, 64, 1, FM_BK, true)) return -12;
  if (make_tmap_2d(&tk2, k2, 2, (uint64_t)k_rows, d2, k2_ld, FM_BK, 64, true)) return -13;
  if (make_tmap_3d(&tv, kb + d1, 2, d_v, H, (uint64_t)k_rows, k_head, (uint64_t)kv_ld * 2, 64, 1, FM_BK, true)) return -14;
  FmhaParams p;
  memset(&p, 0, sizeof(p));
  p.cu_q = q_start; p.end_q = q_end; p.cu_k = k_start; p.end_k = k_end; p.Hq = H; p.Hkv = H; p.nk1 = nk1; p.nk2 = nk2;
  p.scale_log2 = scale * 1.4426950408889634f; p.causal = 1; p.out = (__nv_bfloat16*)out; p.status = (OmniStatus*)status;
  p.dv = d_v; p.out_ld = out_ld; p.window = window; p.out_scale = 1.0f; p.gate = (const __nv_bfloat16*)gate; p.gate_ld = gate_ld; p.sink = sink;
  const dim3 grid(H, B, (max_q + FM_BQ - 1) / FM_BQ);
  if (nk1 + nk2 <= 2) return launch_fmha<FM_LATENT, 2, 2>(grid, tq, tq2, tk, tk2, tv, p, stream);
  return launch_fmha<FM_LATENT, FM_MAXC, 3>(grid, tq, tq2, tk, tk2, tv, p, stream);
}
