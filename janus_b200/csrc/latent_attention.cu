// bfloat16 attention over cached latent rows: every query head of a token reads the same rows, a row's first N numbers
// are its value, all D of them its key (multi-query attention whose values are a part of its keys, with head sizes far
// above what the other attention kernels keep in registers).  Compiled for one row (-DJB_LATENT_D: numbers a row is
// stored with, a multiple of 8; -DJB_LATENT_N: value numbers).
//
// A block owns a tile of 16 MB rows = (token, head) pairs of one sequence (tokens outside, heads inside, as the queries
// lie in memory) and a share of the keys (the key range cut into splits), in tiles of KT keys that come through a ring of
// stages by bulk copies, one a row (the copy engine puts the rows at a padded pitch, free of bank conflicts).  A row of
// the tile in shared memory serves the scores (Q K^T, all D numbers) and the weighted sum (P V, the first N): it is read
// from memory once.  Per tile, with sixteen warps:
//   scores     a warp takes 8 keys and a half or a quarter of the D numbers; partial sums in shared memory
//   softmax    a warp takes MB rows, online in float32 (exp2 of log2e-scaled scores); P in bfloat16 to shared memory
//   sums       a warp takes every sixteenth group of 16 value columns of all rows, float32 in registers
// Every wait for a copy is bounded in time and reports through `*status` (code 31); the rest of such a launch runs on
// without waiting, and its result is not used.
// Works for single tokens (their heads are the rows) and for several tokens a sequence alike; position i sees j <= i.
// With one split the result is written as bfloat16 rows [T H, N], else as float32 partial sums (unnormalised), maxima and
// sums for the kernel that follows.
#include <math_constants.h>
#include <stdio.h>

#include "common.cuh"

#ifndef JB_LATENT_QREGS
#define JB_LATENT_QREGS 40   // registers a thread may spend on its part of the queries; more of them stay in shared memory
#endif
#ifndef JB_LATENT_D
#define JB_LATENT_D 576
#endif
#ifndef JB_LATENT_N
#define JB_LATENT_N 512
#endif

namespace {

typedef __nv_bfloat16 bf16;

constexpr int D = JB_LATENT_D, N = JB_LATENT_N;
static_assert(D % 8 == 0 && D >= 8 && N >= 1 && N <= D, "a row is whole 16-byte vectors and holds its value");
constexpr int DP = (D + 15) / 16 * 16;     // as the MMAs see a row
constexpr int LD = DP + 8;                 // padded shared row: an odd number of 16-byte chunks, conflict-free ldmatrix
constexpr int CHUNKS = D / 8;
constexpr int PAGE = 64;
constexpr int WARPS = 16, THREADS = WARPS * 32;
constexpr int KT = D > 320 ? 32 : 64;      // keys per tile
constexpr int GROUPS = KT / 8;             // groups of 8 keys
constexpr int KS = WARPS / GROUPS;         // warps that share a group of keys, each with a part of the D numbers
constexpr int STEPS = DP / 16;             // 16-number steps of a score
constexpr int WSTEPS = (STEPS + KS - 1) / KS;
constexpr int UNITS = (N + 15) / 16;       // groups of 16 value columns
constexpr int WUNITS = (UNITS + WARPS - 1) / WARPS;
constexpr int TILE = KT * LD;              // elements of a stage
constexpr int S_LD = KT + 4, P_LD = KT + 8;
constexpr float LOG2E = 1.4426950408889634f;
constexpr int SMEM_LIMIT = 227 * 1024;

constexpr int fixed_smem(int mb) {         // everything but the stages; 64 spare bytes: the last pair of steps reads past its row
  return mb * 16 * LD * 2 + KS * mb * 16 * S_LD * 4 + mb * 16 * P_LD * 2 + 2 * mb * 16 * 4 + 64 + 4 * 8;
}
constexpr int stages_for(int mb) {
  const int fit = (SMEM_LIMIT - fixed_smem(mb)) / (TILE * 2);
  return fit > 4 ? 4 : fit;
}
constexpr int smem_for(int mb) { return fixed_smem(mb) + stages_for(mb) * TILE * 2; }
constexpr bool takes(int mb) { return stages_for(mb) >= 2; }

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
constexpr unsigned long long WAIT_LIMIT_NS = 2000000000ull;
__device__ __forceinline__ unsigned long long global_ns() {
  unsigned long long t;
  asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
  return t;
}
__device__ __forceinline__ uint32_t mbar_try(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(bar), "r"(parity)
      : "memory");
  return ok;
}
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, int* status) {
  if (mbar_try(bar, parity)) return true;
  const unsigned long long t0 = global_ns();
  for (;;) {
#pragma unroll 1
    for (int i = 0; i < 256; ++i)
      if (mbar_try(bar, parity)) return true;
    if (global_ns() - t0 > WAIT_LIMIT_NS) {
      atomicCAS(status, 0, 31);
      return false;
    }
  }
}
__device__ __forceinline__ void bulk_copy(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src),
               "r"(bytes), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// q: [T][H][D]; cache: pages [page][64][D]; part_o: [T][H][splits][N], part_ml: [T][H][splits][2] (maximum, sum).
template <int MB>
__global__ void __launch_bounds__(THREADS) latent_attention_kernel(
    const bf16* __restrict__ q, const bf16* __restrict__ cache, bf16* __restrict__ out, float* __restrict__ part_o,
    float* __restrict__ part_ml, const int* __restrict__ block_table, const int* __restrict__ q_start,
    const int* __restrict__ kv_len, int H, int max_pages, float scale_log2, int n_splits, int* __restrict__ status) {
  constexpr int ROWS = MB * 16, STAGES = stages_for(MB), RPW = ROWS / WARPS;
  constexpr bool Q_IN_REGS = WSTEPS * 4 * MB <= JB_LATENT_QREGS;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);                    // [ROWS][LD]
  bf16* kv_s = q_s + ROWS * LD;                                     // [STAGES][KT][LD]
  float* s_s = reinterpret_cast<float*>(kv_s + STAGES * TILE + 32); // [KS][ROWS][S_LD] (behind the spare bytes)
  bf16* p_s = reinterpret_cast<bf16*>(s_s + KS * ROWS * S_LD);      // [ROWS][P_LD]
  float* corr_s = reinterpret_cast<float*>(p_s + ROWS * P_LD);      // [ROWS]
  float* l_s = corr_s + ROWS;                                       // [ROWS]
  uint64_t* bars = reinterpret_cast<uint64_t*>(l_s + ROWS);         // [STAGES]
  jb::pdl_launch_dependents();
  const int seq = blockIdx.z, split = blockIdx.y;
  const int qs = q_start[seq], q_len = q_start[seq + 1] - qs;
  const int len = kv_len[seq], pos0 = len - q_len;
  const int row0 = blockIdx.x * ROWS;                               // first row of the tile within the sequence's rows
  const int n_rows = min(ROWS, q_len * H - row0);
  if (n_rows <= 0) return;                                          // (nothing of an earlier kernel was touched)
  const int pos_last = pos0 + (row0 + n_rows - 1) / H;
  const int tiles = pos_last / KT + 1;
  const int j0 = (int)(((long long)split * tiles) / n_splits), j1 = (int)(((long long)(split + 1) * tiles) / n_splits);
  const int* pages = block_table + (size_t)seq * max_pages;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  // tile j into its stage: one bulk copy a row, issued by the lanes of one warp
  auto issue = [&](int j) {
    const bf16* src = cache + ((size_t)pages[j * KT / PAGE] * PAGE + j * KT % PAGE) * D;
    const uint32_t dst = smem_u32(kv_s + ((j - j0) % STAGES) * TILE), bar = smem_u32(bars + (j - j0) % STAGES);
    if (lane == 0) asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(KT * D * 2) : "memory");
    __syncwarp();
#pragma unroll
    for (int r = lane; r < KT; r += 32) bulk_copy(dst + r * LD * 2, src + (size_t)r * D, D * 2, bar);
  };
  auto issue_first = [&]() {
#pragma unroll 1
    for (int s = 0; s < STAGES - 1; ++s)
      if (j0 + s < j1) issue(j0 + s);
  };
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s)
      asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(smem_u32(bars + s)) : "memory");
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncwarp();
  // rows below pos0 were cached by earlier steps: tiles that lie wholly below are asked for before the wait on the
  // kernel that appends this step's rows (the barriers' only other users meet them behind a barrier of the block)
  const bool early = min(j1, j0 + STAGES - 1) * KT <= pos0;
  if (early && warp == 0) issue_first();
  jb::pdl_wait();
  if (!early && warp == 0) issue_first();
  bool waits = true;
  if constexpr (DP != D) {   // columns that no load writes
    constexpr int PAD = DP > D ? DP - D : 1;
    for (int i = threadIdx.x; i < (ROWS + STAGES * KT) * PAD; i += THREADS)
      q_s[(i / PAD) * LD + D + i % PAD] = __float2bfloat16_rn(0.0f);
  }
  for (int ch = threadIdx.x; ch < ROWS * CHUNKS; ch += THREADS) {
    const int r = ch / CHUNKS, c = ch % CHUNKS;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < n_rows) v = *reinterpret_cast<const uint4*>(q + ((size_t)qs * H + row0 + r) * D + c * 8);
    *reinterpret_cast<uint4*>(q_s + r * LD + c * 8) = v;
  }
  __syncthreads();

  const int kg = warp % GROUPS, part = warp / GROUPS;
  const int step0 = part * WSTEPS, step1 = min(STEPS, step0 + WSTEPS);
  uint32_t qa[Q_IN_REGS ? MB * WSTEPS : 1][4];
  if constexpr (Q_IN_REGS) {
#pragma unroll
    for (int b = 0; b < MB; ++b)
#pragma unroll
      for (int s = 0; s < WSTEPS; ++s)
        if (step0 + s < STEPS)
          ldmatrix_x4(qa[b * WSTEPS + s], q_s + (b * 16 + (lane & 15)) * LD + (step0 + s) * 16 + (lane >> 4) * 8);
  }
  float m[RPW], l[RPW];
  int row_pos[RPW];
#pragma unroll
  for (int i = 0; i < RPW; ++i) {
    m[i] = -CUDART_INF_F;
    l[i] = 0.0f;
    const int r = warp * RPW + i;
    row_pos[i] = r < n_rows ? pos0 + (row0 + r) / H : -1;
  }
  float o[MB][WUNITS][2][4];
#pragma unroll
  for (int b = 0; b < MB; ++b)
#pragma unroll
    for (int u = 0; u < WUNITS; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[b][u][0][e] = o[b][u][1][e] = 0.0f;

  for (int j = j0; j < j1; ++j) {
    __syncthreads();         // everybody is done with tile j - 1: its stage is free
    if (warp == 0 && j + STAGES - 1 < j1) issue(j + STAGES - 1);
    if (waits) waits = mbar_wait(smem_u32(bars + (j - j0) % STAGES), ((j - j0) / STAGES) & 1, status);
    const bf16* tile = kv_s + ((j - j0) % STAGES) * TILE;
    // ---- scores ----
    {
      float s[MB][2][4];     // two chains a block of rows
#pragma unroll
      for (int b = 0; b < MB; ++b)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[b][0][e] = s[b][1][e] = 0.0f;
      const bf16* k_rows = tile + (kg * 8 + (lane & 7)) * LD + (lane >> 3) * 8;
#pragma unroll
      for (int st = 0; st < WSTEPS; st += 2) {
        if (step0 + st >= step1) break;
        uint32_t kb[4];      // two steps of 16 numbers of 8 keys
        ldmatrix_x4(kb, k_rows + (step0 + st) * 16);
#pragma unroll
        for (int b = 0; b < MB; ++b) {
          if constexpr (Q_IN_REGS) {
            mma_bf16(s[b][0], qa[b * WSTEPS + st], kb[0], kb[1]);
            if (st + 1 < WSTEPS && step0 + st + 1 < step1) mma_bf16(s[b][1], qa[b * WSTEPS + (st + 1 < WSTEPS ? st + 1 : st)], kb[2], kb[3]);
          } else {
            uint32_t a[4];
            const bf16* q_rows = q_s + (b * 16 + (lane & 15)) * LD + (step0 + st) * 16 + (lane >> 4) * 8;
            ldmatrix_x4(a, q_rows);
            mma_bf16(s[b][0], a, kb[0], kb[1]);
            if (step0 + st + 1 < step1) {
              ldmatrix_x4(a, q_rows + 16);
              mma_bf16(s[b][1], a, kb[2], kb[3]);
            }
          }
        }
      }
      float* dst = s_s + part * ROWS * S_LD + kg * 8 + 2 * (lane & 3);
#pragma unroll
      for (int b = 0; b < MB; ++b) {
        const int r = b * 16 + (lane >> 2);
        *reinterpret_cast<float2*>(dst + r * S_LD) = make_float2(s[b][0][0] + s[b][1][0], s[b][0][1] + s[b][1][1]);
        *reinterpret_cast<float2*>(dst + (r + 8) * S_LD) = make_float2(s[b][0][2] + s[b][1][2], s[b][0][3] + s[b][1][3]);
      }
    }
    __syncthreads();
    // ---- softmax ----
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int r = warp * RPW + i;
      float v[KT / 32];
      float mx = -CUDART_INF_F;
#pragma unroll
      for (int c = 0; c < KT / 32; ++c) {
        const int key = c * 32 + lane;
        float x = s_s[r * S_LD + key];
#pragma unroll
        for (int k = 1; k < KS; ++k) x += s_s[(k * ROWS + r) * S_LD + key];
        v[c] = j * KT + key <= row_pos[i] ? x * scale_log2 : -CUDART_INF_F;
        mx = fmaxf(mx, v[c]);
      }
      const float m_new = fmaxf(m[i], jb::warp_max(mx));
      const float m_use = m_new == -CUDART_INF_F ? 0.0f : m_new;
      const float corr = exp2f(m[i] - m_use);       // 0 when nothing was seen before
      m[i] = m_new;
      l[i] *= corr;
#pragma unroll
      for (int c = 0; c < KT / 32; ++c) {
        const float p = exp2f(v[c] - m_use);
        l[i] += p;
        p_s[r * P_LD + c * 32 + lane] = __float2bfloat16_rn(p);
      }
      if (lane == 0) corr_s[r] = corr;
    }
    __syncthreads();
    // ---- weighted sums ----
#pragma unroll
    for (int b = 0; b < MB; ++b) {
      const float c0 = corr_s[b * 16 + (lane >> 2)], c1 = corr_s[b * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int u = 0; u < WUNITS; ++u)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          o[b][u][h][0] *= c0;
          o[b][u][h][1] *= c0;
          o[b][u][h][2] *= c1;
          o[b][u][h][3] *= c1;
        }
    }
#pragma unroll
    for (int ks = 0; ks < KT / 16; ++ks) {
      uint32_t a[MB][4];
#pragma unroll
      for (int b = 0; b < MB; ++b) ldmatrix_x4(a[b], p_s + (b * 16 + (lane & 15)) * P_LD + ks * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int u = 0; u < WUNITS; ++u) {
        const int unit = warp + u * WARPS;
        if (unit < UNITS) {
          uint32_t v[4];
          ldmatrix_x4_trans(v, tile + (ks * 16 + (lane & 15)) * LD + unit * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int b = 0; b < MB; ++b) {
            mma_bf16(o[b][u][0], a[b], v[0], v[1]);
            mma_bf16(o[b][u][1], a[b], v[2], v[3]);
          }
        }
      }
    }
  }
  // ---- results ----
#pragma unroll
  for (int i = 0; i < RPW; ++i) {
    const float sum = jb::warp_sum(l[i]);
    const int r = warp * RPW + i;
    if (lane == 0) {
      l_s[r] = sum;
      if (n_splits > 1 && r < n_rows) {
        float* ml = part_ml + (((size_t)qs * H + row0 + r) * n_splits + split) * 2;
        ml[0] = m[i];
        ml[1] = sum;
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int b = 0; b < MB; ++b)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = b * 16 + (lane >> 2) + 8 * half;
      if (r >= n_rows) continue;
      const size_t row = (size_t)qs * H + row0 + r;
      const float inv = n_splits == 1 ? 1.0f / l_s[r] : 1.0f;
#pragma unroll
      for (int u = 0; u < WUNITS; ++u)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int c = (warp + u * WARPS) * 16 + h * 8 + 2 * (lane & 3);
          const float x = o[b][u][h][2 * half] * inv, y = o[b][u][h][2 * half + 1] * inv;
          if (n_splits > 1) {
            float* dst = part_o + (row * n_splits + split) * N + c;
            if (N % 2 == 0) {
              if (c < N) *reinterpret_cast<float2*>(dst) = make_float2(x, y);
            } else {
              if (c < N) dst[0] = x;
              if (c + 1 < N) dst[1] = y;
            }
          } else {
            bf16* dst = out + row * N + c;
            if (c < N) dst[0] = __float2bfloat16_rn(x);
            if (c + 1 < N) dst[1] = __float2bfloat16_rn(y);
          }
        }
    }
}

template <int MB>
int go(const bf16* q, const bf16* cache, bf16* out, float* part_o, float* part_ml, const int* block_table, const int* q_start,
       const int* kv_len, int n_seqs, int max_q_len, int H, int max_pages, float scale, int n_splits, int* status,
       cudaStream_t stream) {
  if constexpr (takes(MB)) {
    static bool configured = false;
    if (!configured) {
      cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<MB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_for(MB));
      if (e != cudaSuccess) return (int)e;
      configured = true;
    }
    const long long tiles = ((long long)max_q_len * H + MB * 16 - 1) / (MB * 16);
    JB_REFUSE(tiles > 0x7fffffffLL, "latent_attention: %d tokens of %d heads are too many", max_q_len, H);
    jb::Launch cfg(dim3((unsigned)tiles, n_splits, n_seqs), dim3(THREADS), smem_for(MB), stream);
    return (int)cudaLaunchKernelEx(&cfg.c, latent_attention_kernel<MB>, q, cache, out, part_o, part_ml, block_table, q_start,
                                   kv_len, H, max_pages, scale * LOG2E, n_splits, status);
  } else {
    JB_REFUSE(true, "latent_attention: %d rows of %d numbers do not fit shared memory", MB * 16, D);
    return 0;
  }
}

}  // namespace

// Row blocks of 16 that a launch of this build may give one CTA (2, 1, or 0: the rows do not fit at all).
JB_EXPORT int jb_latent_attention_blocks() { return takes(2) ? 2 : takes(1) ? 1 : 0; }

// q: [T, H D] bf16; cache: pages [page][1][64][D]; out: [T, H N] bf16 (n_splits == 1) or part_o, part_ml (n_splits > 1);
// blocks: row blocks of 16 a CTA takes (1 or 2).
JB_EXPORT int jb_latent_attention(const void* q, const void* cache, void* out, float* part_o, float* part_ml,
                                  const int* block_table, const int* q_start, const int* kv_len, int n_seqs, int max_q_len,
                                  int H, int d, int n, int page_size, int max_pages, float scale, int n_splits, int blocks,
                                  int* status, cudaStream_t stream) {
  if (n_seqs <= 0 || max_q_len <= 0) return 0;
  JB_REFUSE(d != D || n != N, "latent_attention: built for rows of %d with values of %d, called with %d and %d", D, N, d, n);
  JB_REFUSE(page_size != PAGE, "latent_attention: page size %d (need %d)", page_size, PAGE);
  JB_REFUSE(H < 1 || n_splits < 1 || n_splits > 65535 || n_seqs > 65535 || (n_splits > 1 ? !part_o || !part_ml : !out),
            "latent_attention: %d heads, %d splits, or no room for the result", H, n_splits);
  JB_REFUSE(((uintptr_t)q | (uintptr_t)cache) & 15, "latent_attention: operands must be 16-byte aligned");
  if (blocks == 2)
    return go<2>((const bf16*)q, (const bf16*)cache, (bf16*)out, part_o, part_ml, block_table, q_start, kv_len, n_seqs,
                 max_q_len, H, max_pages, scale, n_splits, status, stream);
  return go<1>((const bf16*)q, (const bf16*)cache, (bf16*)out, part_o, part_ml, block_table, q_start, kv_len, n_seqs,
               max_q_len, H, max_pages, scale, n_splits, status, stream);
}
