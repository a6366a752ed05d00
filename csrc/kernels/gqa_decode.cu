// Grouped-query attention decode over a paged K/V cache: one query token per request, D = 128, up to 16 query heads
// per KV head.
//
//   q        [B, Hq, 128] bf16
//   k_cache  [blocks, block_size, Hkv, 128] bf16 (v_cache alike)
//   out      [B, Hq, 128] bf16 = softmax(q k^T * scale) v over the first seq_lens[b] cache rows of request b
//
// The op is a stream over the cache (every K and V row is read once), so the kernel is built around keeping many
// independent 16 KB pieces of that stream in flight per SM.  grid (Hkv, splits, B), four warps per CTA; each warp owns a
// private 16 KB staging area and walks tiles of 32 keys on its own: it copies the tile's K and V rows with 16-byte
// cp.async (coalesced 256-byte rows, rows of keys past the end zero-filled), waits for them, and runs the tile's math
// on the tensor cores.  With three CTAs per SM twelve such streams run side by side, which covers the memory latency
// without any block-level synchronisation in the loop.
//
// Math per tile: the query heads that share the KV head are the rows of the MMA (mma.sync m16n8k16, rows past the
// group size are zero), S = Q K^T from ldmatrix fragments of the staged K rows, online softmax in registers (one row
// per lane quad), and O += P V with P taken straight from the S accumulators and V fragments from ldmatrix.trans.
// Staged rows are XOR-swizzled by 16-byte chunk so that both ldmatrix forms are free of bank conflicts.  The four
// warps' partial results are merged through shared memory at the end; a split-KV launch writes fp32 partials and
// log-sum-exps that a small second kernel combines.  This is a bandwidth-bound op on a few query rows, so the
// warp-level MMA is enough: the tensor pipe is idle most of the time either way.
//
// omni_gqa_paged_decode_window runs the general form of the same kernel: key and value sizes of their own (multiples of
// 8 up to 256; staged rows are DP = 64, 128 or 256 wide and the columns past the real size stay zero), any number of query
// heads per KV head (16 per CTA), a sliding window (tiles before it are not read), and softmax weights carried as a pair
// of bf16 values (two MMAs per value tile), i.e. to 16 bits of mantissa.  Beside the window it knows kept first keys and
// chunks, a soft cap of the scores, a linear and a logarithmic distance bias per head (an instantiation of its own), cache rows of
// any pitch (latent attention: the values are the first columns of the key rows), rows that share a request (q_to_seq), and a gate
// per row and head or per output element.
//
// Reference counterpart: the paged decode attention of the GQA backend
// (omni/models/common/layers/attention/backend/attention.py:507-702).
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <cstdint>

#include "../include/score_mod.cuh"

namespace omni {

constexpr int GQ_D = 128;                              // head size of the special form
constexpr int GQ_TILE = 32;                            // keys per warp tile
constexpr int GQ_WARPS = 4;
template <int DP>
struct GqSmem {
  static constexpr int ROW_BYTES = DP * 2;
  static constexpr int STAGE_BYTES = 2 * GQ_TILE * ROW_BYTES;   // K and V of one tile: 16 KB for DP = 128
  static constexpr int Q_BYTES = 16 * ROW_BYTES;                // 16 query rows (zero padded)
  static constexpr int TOTAL = GQ_WARPS * STAGE_BYTES + Q_BYTES;
  static_assert(GQ_WARPS * STAGE_BYTES >= GQ_WARPS * 16 * DP * 4 + 2 * GQ_WARPS * 16 * 4,
                "the staging area is reused for the merge of the four warps");
};

struct GqShape {           // used by the general form only
  int q_ld, out_ld, dk, dv, window;
  const float* sink;       // [Hq] or null: exp(sink) is one more term of the softmax denominator
  float out_scale;         // multiplies the result before it is rounded
  int chunk, keep;         // see first_key; the first `keep` keys are visible in any case
  long long k_row, v_row;  // elements from one token's row to the next in the caches
  const int* q_to_seq;     // [B] block-table row of each q row, or null (identity)
  ScoreMod score;          // GEN 2
  const __nv_bfloat16* gate;   // [B, gate_ld] or null: the result of head h is multiplied by sigmoid(gate[b, h gate_cols (+ d)])
  int gate_ld, gate_cols;      // per head: 1, or dv
};
__device__ __forceinline__ float gq_gate(const __nv_bfloat16* gate, int ld, int cols, int b, int h, int d) {
  return gate == nullptr ? 1.f : 1.f / (1.f + __expf(-__bfloat162float(gate[(size_t)b * ld + h * cols + (cols > 1 ? d : 0)])));
}

__device__ __forceinline__ uint32_t gq_smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
template <int DP>
__device__ __forceinline__ uint32_t gq_swz(int row, int chunk) { return (uint32_t)(row * DP * 2 + ((chunk ^ (row & 7)) << 4)); }

__device__ __forceinline__ void gq_cp_async16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;     // 0 source bytes: the 16 destination bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void gq_cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

__device__ __forceinline__ void gq_ldmatrix_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void gq_ldmatrix_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void gq_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t gq_pack(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ uint32_t gq_rest(uint32_t packed, float lo, float hi) {
  const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&packed));
  return gq_pack(lo - f.x, hi - f.y);
}

// GEN 0: the special form, 1: general, 2: general with capped or biased scores
template <int DP, int GEN>
__global__ void __launch_bounds__(GQ_WARPS * 32, DP > 128 ? 1 : 3)
gqa_decode_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
                  const __nv_bfloat16* __restrict__ v_cache, const int* __restrict__ block_table, int bt_ld,
                  const int* __restrict__ seq_lens, int block_size, int Hq, int Hkv, float scale_log2, int splits,
                  float* __restrict__ o_part, float* __restrict__ lse_part, __nv_bfloat16* __restrict__ out,
                  const GqShape sh) {
  extern __shared__ __align__(1024) uint8_t gq_smem[];
  using SM = GqSmem<DP>;
  const int split = blockIdx.y, b = blockIdx.z;
  const int Gall = Hq / Hkv;
  const int nsub = GEN ? (Gall + 15) >> 4 : 1;                // CTAs per KV head
  const int hk = GEN ? blockIdx.x / nsub : blockIdx.x;
  const int g0 = GEN ? (blockIdx.x - hk * nsub) * 16 : 0;     // first query head of this CTA within the group
  const int G = GEN ? min(16, Gall - g0) : Gall;
  const int dk = GEN ? sh.dk : DP, dv = GEN ? sh.dv : DP;
  const int q_ld = GEN ? sh.q_ld : Hq * DP, out_ld = GEN ? sh.out_ld : Hq * DP;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int L = seq_lens[b];
  const int low = GEN ? first_key(L - 1, sh.window, sh.chunk) : 0;        // first visible key, but for those kept
  const int tile0 = low / GQ_TILE;
  const int nkeep = GEN ? min((sh.keep + GQ_TILE - 1) / GQ_TILE, tile0) : 0;   // tiles of kept keys ahead of it
  const int tiles = nkeep + (L + GQ_TILE - 1) / GQ_TILE - tile0;
  const int seq = (GEN && sh.q_to_seq != nullptr) ? sh.q_to_seq[b] : b;
  const int tps = (tiles + splits - 1) / splits;
  const int u_begin = split * tps, u_end = min(tiles, u_begin + tps);

  uint8_t* stage = gq_smem + warp * SM::STAGE_BYTES;          // [K tile][V tile]
  uint8_t* sq = gq_smem + GQ_WARPS * SM::STAGE_BYTES;         // 16 x DP bf16, swizzled like the tiles
  const uint32_t stage_k = gq_smem_u32(stage), stage_v = stage_k + GQ_TILE * SM::ROW_BYTES, sq_addr = gq_smem_u32(sq);

  // query rows of this group (rows >= G are zero)
  constexpr int CH = DP / 8;                                  // 16-byte chunks of a staged row
  for (int i = threadIdx.x; i < 16 * CH; i += blockDim.x) {
    const int row = i / CH, chunk = i % CH;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (row < G && chunk * 8 < dk)
      v = *reinterpret_cast<const uint4*>(q + (size_t)b * q_ld + (hk * Gall + g0 + row) * dk + chunk * 8);
    *reinterpret_cast<uint4*>(sq + gq_swz<DP>(row, chunk)) = v;
  }
  if (GEN && (dk < DP || dv < DP)) {                          // the columns past the head size are never staged
    for (int i = threadIdx.x; i < GQ_WARPS * SM::STAGE_BYTES / 16; i += blockDim.x)
      reinterpret_cast<uint4*>(gq_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
  }
  __syncthreads();
  // A fragments of Q for the 16-wide steps over the head dimension
  constexpr int KS = DP / 16, JT = DP / 8;                    // 16-wide steps over the head size, 8-wide output tiles
  uint32_t qa[KS][4];
  {
    const int row = ((lane >> 3) & 1) * 8 + (lane & 7), chalf = lane >> 4;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) gq_ldmatrix_x4(sq_addr + gq_swz<DP>(row, ks * 2 + chalf), qa[ks]);
  }

  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[JT][4];
#pragma unroll
  for (int j = 0; j < JT; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }

  float slope[2] = {0.f, 0.f}, r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};      // of the two rows of this lane; slopes in log2 units
  if (GEN == 2 && sh.score.slopes != nullptr) {
#pragma unroll
    for (int r = 0; r < 2; ++r)
      if ((lane >> 2) + 8 * r < G) slope[r] = sh.score.slopes[hk * Gall + g0 + (lane >> 2) + 8 * r] * 1.4426950408889634f;
  }
  if (GEN == 2 && sh.score.r1 != nullptr) {
#pragma unroll
    for (int r = 0; r < 2; ++r)
      if ((lane >> 2) + 8 * r < G) {
        r1[r] = sh.score.r1[hk * Gall + g0 + (lane >> 2) + 8 * r];
        r2[r] = sh.score.r2[hk * Gall + g0 + (lane >> 2) + 8 * r];
      }
  }

  for (int u = u_begin + warp; u < u_end; u += GQ_WARPS) {
    const int t = u < nkeep ? u : tile0 + u - nkeep;
    // ---- stage the tile: lane `r` knows where key row r of the tile lives
    const int my_key = t * GQ_TILE + lane;
    const bool my_valid = my_key < L;
    long long my_slot = 0;
    if (my_valid) my_slot = (long long)block_table[(size_t)seq * bt_ld + my_key / block_size] * block_size + my_key % block_size;
#pragma unroll 4
    for (int it = 0; it < GQ_TILE * CH / 32; ++it) {
      const int row = (it * 32 + lane) / CH, chunk = (it * 32 + lane) % CH;
      const long long slot = __shfl_sync(0xffffffffu, my_slot, row);
      const bool valid = __shfl_sync(0xffffffffu, (int)my_valid, row) != 0;
      const size_t k_at = GEN ? (size_t)slot * sh.k_row + (size_t)hk * dk : ((size_t)slot * Hkv + hk) * dk;
      const size_t v_at = GEN ? (size_t)slot * sh.v_row + (size_t)hk * dv : ((size_t)slot * Hkv + hk) * dv;
      if (!GEN || chunk * 8 < dk) gq_cp_async16(stage_k + gq_swz<DP>(row, chunk), k_cache + k_at + chunk * 8, valid);
      if (!GEN || chunk * 8 < dv) gq_cp_async16(stage_v + gq_swz<DP>(row, chunk), v_cache + v_at + chunk * 8, valid);
    }
    gq_cp_async_wait_all();
    __syncwarp();

    // ---- S = Q K^T : four 8-key column tiles
    float s[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) { s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f; }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int krow = j * 8 + (lane & 7);
#pragma unroll
      for (int kp = 0; kp < KS / 2; ++kp) {     // two 16-wide steps per ldmatrix.x4
        uint32_t kb[4];
        gq_ldmatrix_x4(stage_k + gq_swz<DP>(krow, kp * 4 + (lane >> 3)), kb);
        gq_mma(s[j], qa[2 * kp], kb[0], kb[1]);
        gq_mma(s[j], qa[2 * kp + 1], kb[2], kb[3]);
      }
    }
    // ---- online softmax: rows g = lane / 4 and g + 8; this lane holds 8 of the 32 scores of each
    const int key0 = t * GQ_TILE + (lane & 3) * 2;
    float mt[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = key0 + j * 8 + (e & 1);
        const bool see = key < L && (!GEN || key >= low || key < sh.keep);
        float w = GEN == 2 ? cap_score(sh.score, s[j][e]) - slope[e >> 1] * (float)(L - 1 - key) : s[j][e] * scale_log2;
        if (GEN == 2 && sh.score.r1 != nullptr) w -= log_bias(r1[e >> 1], r2[e >> 1], (float)max(L - 1 - key, 0));
        const float v = see ? w : -INFINITY;
        s[j][e] = v;
        mt[e >> 1] = fmaxf(mt[e >> 1], v);
      }
    }
    float f[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 1));
      mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 2));
      const float m_new = fmaxf(m[r], mt[r]);
      f[r] = m_new == -INFINITY ? 1.f : exp2f(m[r] - m_new);
      m[r] = m_new;
    }
    float rs[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float p = m[e >> 1] == -INFINITY ? 0.f : exp2f(s[j][e] - m[e >> 1]);
        s[j][e] = p;
        rs[e >> 1] += p;
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      rs[r] += __shfl_xor_sync(0xffffffffu, rs[r], 1);
      rs[r] += __shfl_xor_sync(0xffffffffu, rs[r], 2);
      l[r] = l[r] * f[r] + rs[r];
    }
#pragma unroll
    for (int j = 0; j < JT; ++j) { o[j][0] *= f[0]; o[j][1] *= f[0]; o[j][2] *= f[1]; o[j][3] *= f[1]; }
    // ---- O += P V : two 16-key steps, 8-wide output tiles
#pragma unroll
    for (int ks = 0; ks < 2; ++ks) {
      uint32_t pa[4];
      pa[0] = gq_pack(s[2 * ks][0], s[2 * ks][1]);
      pa[1] = gq_pack(s[2 * ks][2], s[2 * ks][3]);
      pa[2] = gq_pack(s[2 * ks + 1][0], s[2 * ks + 1][1]);
      pa[3] = gq_pack(s[2 * ks + 1][2], s[2 * ks + 1][3]);
      uint32_t pl[4];                           // general form: what the rounding of the weights left over
      if (GEN) {
        pl[0] = gq_rest(pa[0], s[2 * ks][0], s[2 * ks][1]);
        pl[1] = gq_rest(pa[1], s[2 * ks][2], s[2 * ks][3]);
        pl[2] = gq_rest(pa[2], s[2 * ks + 1][0], s[2 * ks + 1][1]);
        pl[3] = gq_rest(pa[3], s[2 * ks + 1][2], s[2 * ks + 1][3]);
      }
      const int vrow = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
      for (int jp = 0; jp < JT / 2; ++jp) {     // two output tiles per ldmatrix.x4.trans
        uint32_t vb[4];
        gq_ldmatrix_x4_trans(stage_v + gq_swz<DP>(vrow, jp * 2 + (lane >> 4)), vb);
        gq_mma(o[2 * jp], pa, vb[0], vb[1]);
        gq_mma(o[2 * jp + 1], pa, vb[2], vb[3]);
        if (GEN) {
          gq_mma(o[2 * jp], pl, vb[0], vb[1]);
          gq_mma(o[2 * jp + 1], pl, vb[2], vb[3]);
        }
      }
    }
    __syncwarp();      // every lane is done with the staged tile before the next copies land
  }

  // ---- merge the four warps (staging memory is free now)
  __syncthreads();
  float* s_o = reinterpret_cast<float*>(gq_smem);                     // [4][16][DP]
  float* s_m = s_o + GQ_WARPS * 16 * DP;                              // [4][16]
  float* s_l = s_m + GQ_WARPS * 16;
  {
    const int g = lane >> 2, c = (lane & 3) * 2;
#pragma unroll
    for (int j = 0; j < JT; ++j) {
      float* r0 = s_o + ((size_t)warp * 16 + g) * DP + j * 8 + c;
      float* r1 = s_o + ((size_t)warp * 16 + g + 8) * DP + j * 8 + c;
      r0[0] = o[j][0]; r0[1] = o[j][1]; r1[0] = o[j][2]; r1[1] = o[j][3];
    }
    if ((lane & 3) == 0) {
      s_m[warp * 16 + g] = m[0]; s_m[warp * 16 + g + 8] = m[1];
      s_l[warp * 16 + g] = l[0]; s_l[warp * 16 + g + 8] = l[1];
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < G * DP; idx += blockDim.x) {
    const int g = idx / DP, d = idx - g * DP;
    if (GEN && d >= dv) continue;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < GQ_WARPS; ++w) mm = fmaxf(mm, s_m[w * 16 + g]);
    float ll = 0.f, acc = 0.f;
    if (mm > -INFINITY) {
#pragma unroll
      for (int w = 0; w < GQ_WARPS; ++w) {
        const float mw = s_m[w * 16 + g];
        const float fw = mw == -INFINITY ? 0.f : exp2f(mw - mm);
        ll += s_l[w * 16 + g] * fw;
        acc += s_o[((size_t)w * 16 + g) * DP + d] * fw;
      }
    }
    const int hq = hk * Gall + g0 + g;
    if (splits == 1) {
      float den = ll;
      if (GEN && sh.sink != nullptr && ll > 0.f) den += exp2f(sh.sink[hq] * 1.4426950408889634f - mm);
      const float f = GEN ? sh.out_scale * gq_gate(sh.gate, sh.gate_ld, sh.gate_cols, b, hq, d) : 1.f;
      out[(size_t)b * out_ld + hq * dv + d] = __float2bfloat16(ll > 0.f ? acc / den * f : 0.f);
    } else {
      o_part[(((size_t)b * splits + split) * Hq + hq) * dv + d] = ll > 0.f ? acc / ll : 0.f;
      if (d == 0) lse_part[((size_t)b * splits + split) * Hq + hq] = ll > 0.f ? mm + log2f(ll) : -INFINITY;
    }
  }
}

__global__ void gqa_combine_kernel(const float* __restrict__ o_part, const float* __restrict__ lse_part, int splits,
                                   int Hq, int dv, int out_ld, const float* __restrict__ sink, float out_scale,
                                   const __nv_bfloat16* __restrict__ gate, int gate_ld, int gate_cols, __nv_bfloat16* out) {
  const int bh = blockIdx.x;
  const int b = bh / Hq, h = bh - b * Hq;
  const int d = threadIdx.x;
  if (d >= dv) return;
  float mx = -INFINITY;
  for (int s = 0; s < splits; ++s) mx = fmaxf(mx, lse_part[((size_t)b * splits + s) * Hq + h]);
  float den = 0.f, acc = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float v = lse_part[((size_t)b * splits + s) * Hq + h];
    if (v == -INFINITY) continue;
    const float w = exp2f(v - mx);
    den += w;
    acc += w * o_part[(((size_t)b * splits + s) * Hq + h) * dv + d];
  }
  if (sink != nullptr && den > 0.f) den += exp2f(sink[h] * 1.4426950408889634f - mx);
  out[(size_t)b * out_ld + h * dv + d] = __float2bfloat16(den > 0.f ? acc / den * out_scale * gq_gate(gate, gate_ld, gate_cols, b, h, d) : 0.f);
}

}  // namespace omni

using namespace omni;

template <int DP, int GEN>
static int launch_gqa(dim3 grid, const void* q, const void* k_cache, const void* v_cache, const int* block_table, int bt_ld,
                      const int* seq_lens, int B, int block_size, int Hq, int Hkv, float scale, int splits, float* o_part,
                      float* lse_part, void* out, const GqShape& sh, int dv, int out_ld, cudaStream_t stream) {
  static bool configured[64] = {false};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return (int)e;
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    e = cudaFuncSetAttribute(gqa_decode_kernel<DP, GEN>, cudaFuncAttributeMaxDynamicSharedMemorySize, GqSmem<DP>::TOTAL);
    if (e != cudaSuccess) return (int)e;
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  gqa_decode_kernel<DP, GEN><<<grid, GQ_WARPS * 32, GqSmem<DP>::TOTAL, stream>>>(
      (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, block_table, bt_ld, seq_lens,
      block_size, Hq, Hkv, scale * 1.4426950408889634f, splits, o_part, lse_part, (__nv_bfloat16*)out, sh);
  e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  if (splits > 1) {
    gqa_combine_kernel<<<B * Hq, (dv + 31) / 32 * 32, 0, stream>>>(o_part, lse_part, splits, Hq, dv, out_ld, sh.sink,
                                                                   sh.out_scale, sh.gate, sh.gate_ld, sh.gate_cols, (__nv_bfloat16*)out);
    e = cudaGetLastError();
  }
  return (int)e;
}

extern "C" int omni_gqa_paged_decode(const void* q, const void* k_cache, const void* v_cache, const int* block_table,
                                     int bt_ld, const int* seq_lens, int B, int Hq, int Hkv, int D, int block_size,
                                     float scale, int splits, float* o_part, float* lse_part, void* out,
                                     cudaStream_t stream) {
  if (B <= 0) return 0;
  if (D != GQ_D || Hq % Hkv != 0 || Hq / Hkv > 16 || splits < 1) return -1;
  if (splits > 1 && (o_part == nullptr || lse_part == nullptr)) return -2;
  GqShape sh = {};
  sh.out_scale = 1.f;
  return launch_gqa<GQ_D, 0>(dim3(Hkv, splits, B), q, k_cache, v_cache, block_table, bt_ld, seq_lens, B, block_size, Hq,
                                 Hkv, scale, splits, o_part, lse_part, out, sh, GQ_D, Hq * GQ_D, stream);
}

// General form: q rows of pitch q_ld, key size dk, value size dv, out rows of pitch out_ld, window / chunk 0 = all keys.
extern "C" int omni_gqa_paged_decode_window(const void* q, int q_ld, const void* k_cache, const void* v_cache, long long k_row,
                                            long long v_row, const int* q_to_seq, const int* block_table, int bt_ld,
                                            const int* seq_lens, int B, int Hq, int Hkv, int dk, int dv, int block_size,
                                            int window, int chunk, int keep, float scale, float softcap, const float* slopes,
                                            const float* r1, const float* r2, const float* sink, const void* gate, int gate_ld,
                                            int gate_cols, float out_scale, int splits, float* o_part, float* lse_part, void* out, int out_ld, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (Hkv < 1 || Hq % Hkv != 0 || splits < 1 || splits > 65535 || B > 65535 || window < 0) return -1;
  if (splits > 1 && (o_part == nullptr || lse_part == nullptr)) return -2;
  if (dk < 8 || dv < 8 || dk % 8 != 0 || dv % 8 != 0 || dk > 256 || dv > 256) return -3;
  if (q_ld % 8 != 0 || ((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16 != 0) return -4;
  if (chunk < 0 || keep < 0 || k_row < (long long)Hkv * dk || v_row < (long long)Hkv * dv || k_row % 8 != 0 || v_row % 8 != 0) return -6;
  if ((r1 == nullptr) != (r2 == nullptr) || (gate != nullptr && ((gate_cols != 1 && gate_cols != dv) || gate_ld < Hq * gate_cols))) return -7;
  const GqShape sh = {q_ld, out_ld, dk, dv, window, sink, out_scale, chunk, keep, k_row, v_row, q_to_seq,
                      make_score_mod(scale, softcap, slopes, r1, r2), (const __nv_bfloat16*)gate, gate_ld, gate_cols};
  const bool mod = softcap > 0.f || slopes != nullptr || r1 != nullptr;
  const dim3 grid(Hkv * ((Hq / Hkv + 15) / 16), splits, B);
  const int d = dk > dv ? dk : dv;
#define GQA_CASE(DP)                                                                                                     \
  if (d <= DP && mod)                                                                                                    \
    return launch_gqa<DP, 2>(grid, q, k_cache, v_cache, block_table, bt_ld, seq_lens, B, block_size, Hq, Hkv, scale,     \
                             splits, o_part, lse_part, out, sh, dv, out_ld, stream);                                     \
  if (d <= DP)                                                                                                           \
    return launch_gqa<DP, 1>(grid, q, k_cache, v_cache, block_table, bt_ld, seq_lens, B, block_size, Hq, Hkv, scale,  \
                                splits, o_part, lse_part, out, sh, dv, out_ld, stream);
  GQA_CASE(64) GQA_CASE(128) GQA_CASE(256)
#undef GQA_CASE
  return -5;
}
