// Windowed causal attention over the paged cache for any head sizes, block size and activation type (bf16 or fp32): one
// warp per (query row, head).  This is the fp32 path of the models and takes the head shapes that the tensor-core kernels
// (fmha_sm100.cu for prompt portions, gqa_decode.cu for single tokens) do not.
//
//   lane = key     32 scores at a time, each lane reads its key row
//   lane = column  P V, value rows read coalesced
// Scores, softmax and the accumulation over the values are fp32.  `sink` (per head, may be null): exp(sink) stands in the
// softmax denominator; `out_scale` multiplies the result before it is rounded, and so does sigmoid(gate[row, head]) if there is a
// gate (or of gate[row, head, column]).  Optionally: the first `keep` keys beside the window, chunks, a soft cap of the scores, a linear
// and a logarithmic distance bias per head.
// Rows of the caches have a pitch of their own, so that values may be a part of the key rows (latent attention).
#include "../include/omni_vec.cuh"
#include "../include/score_mod.cuh"

namespace omni {

constexpr int AA_WARPS = 4;
constexpr int AA_MAXV = 64;      // value columns per lane, at most: d_v <= 2048

struct AttnAnyOpts {
  long long k_row, v_row;        // elements from one token's row to the next in the caches
  int window, chunk, keep;
  float softcap;
  const float* slopes;           // [Hq] or null
  const float *r1, *r2;          // [Hq] or null
  const void* gate;              // [rows, gate_ld] of the activation type, or null
  int gate_ld, gate_cols;        // per head: 1, or dv
};

// MAXV: value columns per lane
template <typename T, int MAXV>
__global__ void __launch_bounds__(AA_WARPS * 32) attn_any_kernel(
    const T* __restrict__ q, int q_ld, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
    const int64_t* __restrict__ positions, const int* __restrict__ q_to_seq, const int64_t* __restrict__ slots,
    const int* __restrict__ block_table, int bt_ld, int rows, int Hq, int Hkv, int dk, int dv, int block_size,
    float scale, const float* __restrict__ sink, float out_scale, T* __restrict__ out, int out_ld, const AttnAnyOpts o) {
  extern __shared__ float aa_q[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * AA_WARPS + warp;
  if (item >= (long long)rows * Hq) return;      // no block-level synchronisation below
  const int t = (int)(item / Hq), h = (int)(item % Hq), hk = h / (Hq / Hkv);
  float* sq = aa_q + warp * dk;
  T* orow = out + (size_t)t * out_ld + h * dv;
  if (slots[t] < 0) {                            // padding row
    for (int d = lane; d < dv; d += 32) orow[d] = from_f32<T>(0.f);
    return;
  }
  for (int d = lane; d < dk; d += 32) sq[d] = to_f32(q[(size_t)t * q_ld + h * dk + d]);
  __syncwarp();
  const int pos = (int)positions[t];
  const int lo = first_key(pos, o.window, o.chunk);
  const float slope = o.slopes != nullptr ? o.slopes[h] : 0.f;
  const float r1 = o.r1 != nullptr ? o.r1[h] : 0.f, r2 = o.r1 != nullptr ? o.r2[h] : 0.f;
  const int* bt = block_table + (size_t)q_to_seq[t] * bt_ld;
  float m = -INFINITY, l = 0.f, acc[MAXV];
#pragma unroll
  for (int i = 0; i < MAXV; ++i) acc[i] = 0.f;
  const int kept = min(o.keep, lo);                 // keys ahead of the window that stay visible
  for (int k0 = kept > 0 ? 0 : lo; k0 <= pos; k0 = k0 < lo && k0 + 32 >= kept ? lo : k0 + 32) {
    const int key = k0 + lane, end = k0 < lo ? kept : pos + 1;
    float s = -INFINITY;
    size_t slot = 0;
    if (key < end) {
      slot = (size_t)bt[key / block_size] * block_size + key % block_size;
      const T* kr = k_cache + slot * o.k_row + (size_t)hk * dk;
      float dot = 0.f;
      for (int d = 0; d < dk; ++d) dot = fmaf(sq[d], to_f32(kr[d]), dot);
      s = dot * scale;
      if (o.softcap > 0.f) s = o.softcap * tanhf(s / o.softcap);
      s -= slope * (float)(pos - key);
      if (o.r1 != nullptr) s -= r1 * log1pf(r2 * (float)(pos - key));
    }
    float mx = s;
#pragma unroll
    for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
    const float m_new = fmaxf(m, mx);            // finite: at least one key of the group is visible
    const float f = expf(m - m_new);
    const float p = expf(s - m_new);
    l = l * f + warp_sum32(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < MAXV; ++i) acc[i] *= f;
    const int n = min(32, end - k0);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const T* vr = v_cache + (size_t)__shfl_sync(0xffffffffu, (unsigned long long)slot, j) * o.v_row + (size_t)hk * dv;
#pragma unroll
      for (int i = 0; i < MAXV; ++i)
        if (i * 32 + lane < dv) acc[i] = fmaf(pj, to_f32(vr[i * 32 + lane]), acc[i]);
    }
  }
  if (sink != nullptr) l += expf(sink[h] - m);      // one more term of the denominator, without a value
  const T* gate = o.gate != nullptr ? (const T*)o.gate + (size_t)t * o.gate_ld + h * o.gate_cols : nullptr;
  if (gate != nullptr && o.gate_cols == 1) out_scale /= 1.f + expf(-to_f32(gate[0]));
#pragma unroll
  for (int i = 0; i < MAXV; ++i)
    if (i * 32 + lane < dv) {
      float v = acc[i] / l * out_scale;
      if (gate != nullptr && o.gate_cols > 1) v /= 1.f + expf(-to_f32(gate[i * 32 + lane]));
      orow[i * 32 + lane] = from_f32<T>(v);
    }
}

template <typename T>
static int launch_attn_any(const void* q, int q_ld, const void* k, const void* v, const int64_t* positions,
                           const int* q_to_seq, const int64_t* slots, const int* bt, int bt_ld, int rows, int Hq, int Hkv,
                           int dk, int dv, int block_size, float scale, const float* sink, float out_scale, void* out,
                           int out_ld, const AttnAnyOpts& o, cudaStream_t st) {
  const long long items = (long long)rows * Hq;
  const auto kernel = dv <= 32 * 16 ? attn_any_kernel<T, 16> : attn_any_kernel<T, AA_MAXV>;
  kernel<<<(unsigned)((items + AA_WARPS - 1) / AA_WARPS), AA_WARPS * 32, AA_WARPS * dk * sizeof(float), st>>>(
      (const T*)q, q_ld, (const T*)k, (const T*)v, positions, q_to_seq, slots, bt, bt_ld, rows, Hq, Hkv, dk, dv, block_size,
      scale, sink, out_scale, (T*)out, out_ld, o);
  return (int)cudaGetLastError();
}

}  // namespace omni

using namespace omni;

extern "C" int omni_attn_any(const void* q, int q_ld, const void* k_cache, const void* v_cache, long long k_row, long long v_row,
                             const int64_t* positions, const int* q_to_seq, const int64_t* slots, const int* block_table, int bt_ld,
                             int rows, int Hq, int Hkv, int dk, int dv, int block_size, int window, int chunk, int keep, float scale,
                             float softcap, const float* slopes, const float* r1, const float* r2, const float* sink, const void* gate,
                             int gate_ld, int gate_cols, float out_scale, void* out, int out_ld, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (Hkv < 1 || Hq % Hkv != 0 || dk < 1 || dk > 2048 || dv < 1 || dv > 32 * AA_MAXV || block_size < 1 || window < 0) return -1;
  if (chunk < 0 || keep < 0 || k_row < (long long)Hkv * dk || v_row < (long long)Hkv * dv) return -2;
  if ((r1 == nullptr) != (r2 == nullptr) || (gate != nullptr && ((gate_cols != 1 && gate_cols != dv) || gate_ld < Hq * gate_cols))) return -3;
  const AttnAnyOpts o = {k_row, v_row, window, chunk, keep, softcap, slopes, r1, r2, gate, gate_ld, gate_cols};
  if (f32)
    return launch_attn_any<float>(q, q_ld, k_cache, v_cache, positions, q_to_seq, slots, block_table, bt_ld, rows, Hq, Hkv, dk,
                                  dv, block_size, scale, sink, out_scale, out, out_ld, o, st);
  return launch_attn_any<__nv_bfloat16>(q, q_ld, k_cache, v_cache, positions, q_to_seq, slots, block_table, bt_ld, rows, Hq,
                                        Hkv, dk, dv, block_size, scale, sink, out_scale, out, out_ld, o, st);
}
