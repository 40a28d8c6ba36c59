// Float32 grouped-query attention over the paged cache, for prefill and decode
// alike: one warp per (token, query head); the token attends to the keys of
// its own sequence at positions [max(0, pos-window+1), pos] (window 0 = all);
// with chunk > 0 only to those of them that lie in its own chunk of positions,
// [floor(pos/chunk) chunk, pos]; with softcap > 0 a score s becomes softcap tanh(s/softcap); with sink = 1 the
// softmax's denominator has one more term, exp(0): a key of score 0 that has no value.
// Formulas: crates/janus-engine/src/compute/shaders/attention.wgsl:96-115
// (kv head = h*nkv/nh, score = dot * scale), softmax.wgsl:29-50 (exp(s-max)/sum),
// attention.wgsl:170-185 (sum of p*v).  The softmax runs online over chunks of
// 32 keys that start at multiples of 32 of the absolute key index, so a
// token's result does not depend on how its sequence was cut into steps.
//
// The values are the first `vd` numbers of rows of ld_v numbers (latent attention: a row is key and value at once).
// slopes (one per query head): slope (position - key position) is taken off the score; sinks (one per query head): the
// denominator has one more term, exp(sink); gate (rows of ld_gate numbers, one a query head): its sigmoid multiplies the
// head's output.
//
// Cache layout of one layer: [page][kv_head][PAGE][hd]; block_table[slot][i] is
// the page of keys [i*PAGE, (i+1)*PAGE) of the sequence in `slot`.
#include <math_constants.h>
#include <stdio.h>

#include "common.cuh"

namespace {

constexpr int WARPS = 4;
constexpr int SMALL_HD = 256, MAX_HD = 1280;

// VEC: head sizes that are multiples of 4 (16-byte loads of the keys).  HDM bounds the head size; U value rows are
// loaded at a time.
template <bool VEC, int HDM, int U>
__global__ void __launch_bounds__(WARPS * 32) attention_f32_kernel(
    const float* __restrict__ q, const float* __restrict__ k_cache, const float* __restrict__ v_cache,
    float* __restrict__ out, const int* __restrict__ block_table, const int* __restrict__ token_slot,
    const int* __restrict__ positions, int T, int nh, int nkv, int hd, int vd, int page_size, int max_pages,
    int window, float scale, int chunk, float softcap, float sink, int ld_v, const float* __restrict__ slopes,
    const float* __restrict__ sinks, const float* __restrict__ gate, int ld_gate) {
  __shared__ __align__(16) float q_s[WARPS][HDM];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * WARPS + warp;
  if (item >= (long long)T * nh) return;  // whole warp leaves together
  const int t = (int)(item / nh), h = (int)(item % nh);
  const int kvh = (h * nkv) / nh;
  const int pos = positions[t];
  const int* pages = block_table + (size_t)token_slot[t] * max_pages;
  int kstart = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
  if (chunk > 0) kstart = max(kstart, (pos / chunk) * chunk);   // only the keys of the query's own chunk of positions

  const float* qv = q + ((size_t)t * nh + h) * hd;
  for (int d = lane; d < hd; d += 32) q_s[warp][d] = qv[d];
  __syncwarp();

  const float slope = slopes != nullptr ? slopes[h] : 0.0f;
  float m = -CUDART_INF_F, l = 0.0f;
  float acc[HDM / 32];
#pragma unroll
  for (int j = 0; j < HDM / 32; ++j) acc[j] = 0.0f;

  for (int c0 = (kstart / 32) * 32; c0 <= pos; c0 += 32) {
    const int key = c0 + lane;
    const bool valid = key >= kstart && key <= pos;
    float s = -CUDART_INF_F;
    if (valid) {
      const int page = pages[key / page_size], row = key % page_size;
      const float* kr = k_cache + (((size_t)page * nkv + kvh) * page_size + row) * hd;
      float dot = 0.0f;
      if (VEC) {
        // 16-byte loads, eight in flight, consumed in the order d = 0, 1, 2, ... (the sum is the same as below)
        const float4* kr4 = reinterpret_cast<const float4*>(kr);
        const float4* q4 = reinterpret_cast<const float4*>(q_s[warp]);
#pragma unroll 8
        for (int d4 = 0; d4 < hd / 4; ++d4) {
          const float4 kk = kr4[d4], qq = q4[d4];
          dot = fmaf(qq.x, kk.x, dot);
          dot = fmaf(qq.y, kk.y, dot);
          dot = fmaf(qq.z, kk.z, dot);
          dot = fmaf(qq.w, kk.w, dot);
        }
      } else {
        for (int d = 0; d < hd; ++d) dot = fmaf(q_s[warp][d], kr[d], dot);
      }
      s = dot * scale;
      if (softcap > 0.0f) s = softcap * tanhf(s / softcap);
      s = fmaf(slope, (float)(key - pos), s);
    }
    const float m_new = fmaxf(m, jb::warp_max(s));
    const float p = valid ? expf(s - m_new) : 0.0f;
    const float corr = expf(m - m_new);  // exp(-inf) = 0 on the first chunk
    l = l * corr + jb::warp_sum(p);
#pragma unroll
    for (int j = 0; j < HDM / 32; ++j) acc[j] *= corr;
    const int n_keys = min(32, pos - c0 + 1);
    // several value rows are loaded before their products are added, in key order (the same sums as one by one,
    // with the rows' latencies side by side)
    const int first = max(c0, kstart) - c0;
    for (int kk0 = first; kk0 < n_keys; kk0 += U) {
      float vreg[U][HDM / 32];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int key2 = c0 + min(kk0 + u, n_keys - 1);
        const int page = pages[key2 / page_size], row = key2 % page_size;
        const float* vr = v_cache + (((size_t)page * nkv + kvh) * page_size + row) * ld_v;
#pragma unroll
        for (int j = 0; j < HDM / 32; ++j) {
          const int d = lane + 32 * j;
          vreg[u][j] = d < vd ? vr[d] : 0.0f;
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (kk0 + u < n_keys) {   // uniform across the warp
          const float pk = __shfl_sync(0xffffffffu, p, kk0 + u);
#pragma unroll
          for (int j = 0; j < HDM / 32; ++j)
            if (lane + 32 * j < vd) acc[j] = fmaf(pk, vreg[u][j], acc[j]);
        }
      }
    }
    m = m_new;
  }
  if (sink > 0.0f) l += sink * expf(m == -CUDART_INF_F ? 0.0f : -m);
  if (sinks != nullptr) l += expf(sinks[h] - (m == -CUDART_INF_F ? 0.0f : m));
  const float open = gate != nullptr ? 1.0f / (1.0f + expf(-gate[(size_t)t * ld_gate + h])) : 1.0f;
  float* o = out + ((size_t)t * nh + h) * vd;
#pragma unroll
  for (int j = 0; j < HDM / 32; ++j) {
    const int d = lane + 32 * j;
    if (d < vd) o[d] = acc[j] / l * open;
  }
}

}  // namespace

JB_EXPORT int jb_attention_f32(const float* q, const float* k_cache, const float* v_cache, float* out,
                               const int* block_table, const int* token_slot, const int* positions, int T,
                               int nh, int nkv, int hd, int vd, int page_size, int max_pages, int window, float scale,
                               int chunk, float softcap, float sink, int ld_v, const float* slopes, const float* sinks,
                               const float* gate, int ld_gate, cudaStream_t stream) {
  if (T <= 0) return 0;
  JB_REFUSE(hd > MAX_HD || hd <= 0 || vd <= 0 || vd > ld_v || vd > (hd <= SMALL_HD ? SMALL_HD : MAX_HD),
            "attention_f32: head_dim %d is outside (0, %d], or its values (%d) are wider than their rows or the kernel", hd,
            MAX_HD, vd);
  JB_REFUSE(nkv <= 0 || nh % nkv != 0, "attention_f32: %d heads are not a multiple of %d kv heads", nh, nkv);
  const long long items = (long long)T * nh;
  const unsigned blocks = (unsigned)((items + WARPS - 1) / WARPS);
  const bool vec = hd % 4 == 0 && (((uintptr_t)k_cache) & 15) == 0;
#define JB_GO(VEC, HDM, U)                                                                                         \
  attention_f32_kernel<VEC, HDM, U><<<blocks, WARPS * 32, 0, stream>>>(q, k_cache, v_cache, out, block_table,      \
                                                                       token_slot, positions, T, nh, nkv, hd, vd,  \
                                                                       page_size, max_pages, window, scale, chunk, \
                                                                       softcap, sink, ld_v, slopes, sinks, gate,   \
                                                                       ld_gate)
  if (hd <= SMALL_HD) {
    if (vec) JB_GO(true, SMALL_HD, 8);
    else JB_GO(false, SMALL_HD, 8);
  } else {
    if (vec) JB_GO(true, MAX_HD, 2);
    else JB_GO(false, MAX_HD, 2);
  }
#undef JB_GO
  JB_CHECK_LAUNCH();
  return 0;
}
