// Latent attention with a rotated part: what happens around the attention kernels.  Per token a place caches one row
// [c | p]: the latent c (n numbers, normed) and a key part p (r numbers, rotated) that all heads share; a head's key is
// [Wuk_h c | p], its value Wuv_h c.  All arithmetic is float32 on the projections' float32 accumulators
//
//   proj [T, ld]:  q at q_col (H heads of d unrotated then r rotated numbers), the row's projection at c_col (n + r)
//
//   latent_prep      queries as heads: q_out[t, h] = [q | turned q], for attention over keys and values per head;
//                    the token's row is normed, turned and appended to the pages (and to `rows` [T, stored], if given)
//   latent_queries   queries in the latents' space: q_out[t, h] = [Wuk_h^T q | turned q], so that the score with the
//                    cached row itself is the head's score; the token's row as above
//   latent_down      where the queries have a latent of their own (m numbers at column 0): it is normed and written for the
//                    product that makes the queries from it; the token's row as above
//   latent_values    out[t, h] = Wuv_h o, o = sum_j p_j c_j the attention's output in the latents' space, from rows
//                    [T, H, n] or straight from the partial sums that the splits of the keys left; times the sigmoid
//                    of an output gate, if there is one (a number for every value, or one per head)
//   gather_rows      the cached rows of a step's sequences, sequence after sequence, in one matrix
//
// The rotation turns the pair (i, i + r/2) by the position's angle; cos and sin come from a table [positions][r/2][2].
// Pages of one place: [page][1][page_size][stored], stored >= n + r, extra columns never written (they stay zero).
#include <cooperative_groups.h>
#include <math_constants.h>
#include <stdio.h>

#include "common.cuh"

namespace {

namespace cg = cooperative_groups;
typedef __nv_bfloat16 bf16;

struct Row {                 // the token's own row: where it comes from and where it goes (c_cache null: none)
  int c_col, n, r, stored;
  const float* w;            // norm weight of the latent
  float eps;
  const int* dest;
  void* c_cache;
  void* rows;                // a second copy, row t of [T, stored] (null: none)
  int vec;                   // n, r / 2 and stored are whole groups of four, everything lies at aligned addresses
};

template <typename TO>
__device__ __forceinline__ void store4(TO* p, const float4& v) {
  if constexpr (sizeof(TO) == 4) {
    *reinterpret_cast<float4*>(p) = v;
  } else {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&lo);
    u.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
  }
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float squares4(const float4& v, float ss) {
  return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, fmaf(v.x, v.x, ss))));
}
__device__ __forceinline__ float4 scaled4(const float4& v, float f, const float4& w) {
  return make_float4((v.x * f) * w.x, (v.y * f) * w.y, (v.z * f) * w.z, (v.w * f) * w.w);
}
// The pairs (u, v) of four neighbouring numbers and of those half a row further, turned by cs (cos and sin of the four).
__device__ __forceinline__ void turn4(const float4& u, const float4& v, const float* cs, float4& a, float4& b) {
  const float4 p = load4(cs), q = load4(cs + 4);
  a = make_float4(u.x * p.x - v.x * p.y, u.y * p.z - v.y * p.w, u.z * q.x - v.z * q.y, u.w * q.z - v.w * q.w);
  b = make_float4(v.x * p.x + u.x * p.y, v.y * p.z + u.y * p.w, v.z * q.x + u.z * q.y, v.w * q.z + u.w * q.w);
}

// One block norms, turns and writes the row of token t, four numbers a thread.
template <typename TO>
__device__ void write_row_vec(const float* x, const Row& row, const float* cs, int t, float* scratch) {
  float ss = 0.0f;
  for (int i = threadIdx.x * 4; i < row.n; i += blockDim.x * 4) ss = squares4(load4(x + i), ss);
  ss = jb::block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)row.n + row.eps);
  TO* out = (TO*)row.c_cache + (size_t)row.dest[t] * row.stored;
  TO* copy = row.rows != nullptr ? (TO*)row.rows + (size_t)t * row.stored : nullptr;
  const int half = row.r >> 1;
  auto put = [&](int i, const float4& v) {
    store4(out + i, v);
    if (copy != nullptr) store4(copy + i, v);
  };
  for (int i = threadIdx.x * 4; i < row.stored; i += blockDim.x * 4) {
    if (i < row.n) {
      put(i, scaled4(load4(x + i), inv, load4(row.w + i)));
    } else if (i < row.n + row.r) {
      const int j = i - row.n;
      if (cs == nullptr) {
        put(i, load4(x + i));
      } else if (j < half) {
        float4 a, b;
        turn4(load4(x + i), load4(x + i + half), cs + 2 * j, a, b);
        put(i, a);
        put(i + half, b);
      }
    } else if (copy != nullptr) {
      store4(copy + i, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
    }
  }
}

// One block norms, turns and writes the row of token t.
template <typename TO>
__device__ void write_row(const float* pr, const Row& row, const float* cs, int t, float* scratch) {
  const float* x = pr + row.c_col;
  if (row.vec) {
    write_row_vec<TO>(x, row, cs, t, scratch);
    return;
  }
  float ss = 0.0f;
  for (int i = threadIdx.x; i < row.n; i += blockDim.x) ss = fmaf(x[i], x[i], ss);
  ss = jb::block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)row.n + row.eps);
  TO* out = (TO*)row.c_cache + (size_t)row.dest[t] * row.stored;
  TO* copy = row.rows != nullptr ? (TO*)row.rows + (size_t)t * row.stored : nullptr;
  const int half = row.r >> 1;
  for (int i = threadIdx.x; i < row.stored; i += blockDim.x) {
    float v;
    if (i < row.n) {
      v = (x[i] * inv) * row.w[i];
    } else if (i < row.n + row.r) {
      const int j = i - row.n;
      v = x[i];
      if (cs != nullptr) {
        const int k = j < half ? j : j - half;
        const float other = x[row.n + (j < half ? j + half : k)];
        const float co = cs[2 * k], si = cs[2 * k + 1];
        v = j < half ? v * co - other * si : v * co + other * si;
      }
    } else {
      if (copy != nullptr) copy[i] = jb::from_f32<TO>(0.0f);
      continue;
    }
    out[i] = jb::from_f32<TO>(v);
    if (copy != nullptr) copy[i] = jb::from_f32<TO>(v);
  }
}

// Queries as heads (`dp` numbers each, the extra ones zero), one block per token (blockIdx.y == 0), and the token's row,
// another one (blockIdx.y == 1).
// VEC: d, r / 2, dp, the columns and the rows are whole groups of four at aligned addresses.
template <typename TO, bool VEC>
__global__ void __launch_bounds__(256) latent_prep_kernel(const float* __restrict__ proj, int ld, int q_col, int H, int d,
                                                          int r, int dp, const float* __restrict__ table,
                                                          const int* __restrict__ positions, TO* __restrict__ q_out,
                                                          Row row) {
  __shared__ float scratch[33];
  jb::pdl_launch_dependents();
  jb::pdl_wait();
  const int t = blockIdx.x;
  const float* pr = proj + (size_t)t * ld;
  const int half = r >> 1;
  const float* cs = table != nullptr && r > 0 ? table + (size_t)positions[t] * half * 2 : nullptr;
  if (blockIdx.y == 1) {
    write_row<TO>(pr, row, cs, t, scratch);
    return;
  }
  TO* q = q_out + (size_t)t * H * dp;
  if constexpr (VEC) {
    const int per = dp >> 2;                           // groups of four per stored head
    for (int i = threadIdx.x; i < H * per; i += blockDim.x) {
      const int h = i / per, j = (i - h * per) << 2;
      const float* x = pr + q_col + (size_t)h * (d + r);
      TO* o = q + (size_t)h * dp;
      if (j < d || (j < d + r && cs == nullptr)) {
        store4(o + j, *reinterpret_cast<const float4*>(x + j));
      } else if (j < d + half) {
        float4 a, b;
        turn4(load4(x + j), load4(x + j + half), cs + 2 * (j - d), a, b);
        store4(o + j, a);
        store4(o + j + half, b);
      } else if (j >= d + r) {
        store4(o + j, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
      }
    }
  } else {
    for (int i = threadIdx.x; i < H * dp; i += blockDim.x) {
      const int h = i / dp, j = i - h * dp;
      const float* x = pr + q_col + (size_t)h * (d + r);
      float v = j < d + r ? x[j] : 0.0f;
      if (j >= d && j < d + r && cs != nullptr) {
        const int k = j - d < half ? j - d : j - d - half;
        const float co = cs[2 * k], si = cs[2 * k + 1];
        v = j - d < half ? v * co - x[j + half] * si : v * co + x[j - half] * si;
      }
      q[i] = jb::from_f32<TO>(v);
    }
  }
}

// a_out[t] = x / rms(x) * w with x = proj[t, 0 : m], a block per token (blockIdx.y == 0); the token's row, another one
// (blockIdx.y == 1).  All blocks together set the n_clear float4 at `clear` to zero.  VEC: m and ld are whole groups of
// four at aligned addresses.
template <typename TO, bool VEC>
__global__ void __launch_bounds__(256) latent_down_kernel(const float* __restrict__ proj, int ld, int m,
                                                          const float* __restrict__ w, float eps, TO* __restrict__ a_out,
                                                          const float* __restrict__ table, const int* __restrict__ positions,
                                                          float4* __restrict__ clear, long long n_clear, Row row) {
  __shared__ float scratch[33];
  jb::pdl_launch_dependents();
  jb::pdl_wait();
  const int t = blockIdx.x;
  const float* x = proj + (size_t)t * ld;
  const long long blocks = (long long)gridDim.x * gridDim.y, block = (long long)blockIdx.y * gridDim.x + t;
  for (long long i = block * blockDim.x + threadIdx.x; i < n_clear; i += blocks * blockDim.x)
    clear[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if (blockIdx.y == 1) {
    const float* cs = table != nullptr && row.r > 0 ? table + (size_t)positions[t] * (row.r >> 1) * 2 : nullptr;
    write_row<TO>(x, row, cs, t, scratch);
    return;
  }
  float ss = 0.0f;
  if constexpr (VEC) {
    for (int i = threadIdx.x * 4; i < m; i += blockDim.x * 4) ss = squares4(load4(x + i), ss);
    ss = jb::block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)m + eps);
    for (int i = threadIdx.x * 4; i < m; i += blockDim.x * 4)
      store4(a_out + (size_t)t * m + i, scaled4(load4(x + i), inv, load4(w + i)));
    return;
  }
  for (int i = threadIdx.x; i < m; i += blockDim.x) ss = fmaf(x[i], x[i], ss);
  ss = jb::block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)m + eps);
  for (int i = threadIdx.x; i < m; i += blockDim.x) a_out[(size_t)t * m + i] = jb::from_f32<TO>((x[i] * inv) * w[i]);
}

// V numbers of a weight row (16 bytes, or one number): the bits are loaded early and unpacked late.
template <int V> struct Raw {
  uint4 bits;
  template <typename T> __device__ __forceinline__ void load(const T* p) { bits = *reinterpret_cast<const uint4*>(p); }
  template <typename T> __device__ __forceinline__ void unpack(float (&v)[V]) const {
    const uint32_t w[4] = {bits.x, bits.y, bits.z, bits.w};
    if constexpr (sizeof(T) == 2) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
      }
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) v[i] = __uint_as_float(w[i]);
    }
  }
};
template <> struct Raw<1> {
  float x;
  template <typename T> __device__ __forceinline__ void load(const T* p) { x = jb::to_f32(*p); }
  template <typename T> __device__ __forceinline__ void unpack(float (&v)[1]) const { v[0] = x; }
};

constexpr int QT = 8;             // tokens of a block of latent_queries
constexpr int Q_THREADS = 128;

// q_out[t, h, :n] = sum_j q[t, h, j] uk[h d + j, :], q_out[t, h, n : n + r] = the turned part, the rest zero; and, by
// the blocks behind the heads' (blockIdx.x >= H * chunks: a block per token), the tokens' rows.
// A block owns (head, a chunk of COLS latent columns, QT tokens): COLS / V threads a row of uk, the others take other
// rows j; the partial sums meet in shared memory.  The first rows of uk are asked for before the wait on the kernel
// that makes the projections.
template <typename T, int V>
__global__ void __launch_bounds__(Q_THREADS) latent_queries_kernel(
    const float* __restrict__ proj, int ld, int q_col, int H, int d, int r, int n, int dp, const T* __restrict__ uk,
    const float* __restrict__ table, const int* __restrict__ positions, T* __restrict__ q_out, int n_tokens, Row row) {
  constexpr int CT = 8;                         // threads along the columns
  constexpr int COLS = CT * V;
  constexpr int SL = Q_THREADS / CT;            // slices of the rows j
  extern __shared__ __align__(16) float sm[];   // q [QT][d], then the slices' sums [SL][QT][COLS]
  __shared__ float scratch[33];
  jb::pdl_launch_dependents();
  const int chunks = (n + COLS - 1) / COLS;
  const int t0 = blockIdx.y * QT, nt = min(QT, n_tokens - t0);
  const int half = r >> 1;
  if (blockIdx.x >= H * chunks) {
    jb::pdl_wait();
    const int t = t0 + blockIdx.x - H * chunks;
    if (t >= n_tokens) return;
    const float* cs = table != nullptr && r > 0 ? table + (size_t)positions[t] * half * 2 : nullptr;
    write_row<T>(proj + (size_t)t * ld, row, cs, t, scratch);
    return;
  }
  const int h = blockIdx.x / chunks, chunk = blockIdx.x - h * chunks;
  const int ct = threadIdx.x % CT, sl = threadIdx.x / CT;
  const int col = chunk * COLS + ct * V;
  const bool active = col < n;                  // with V > 1 n is a multiple of V: no column group is cut
  const T* w = uk + (size_t)h * d * n + (active ? col : 0);
  constexpr int AHEAD = 8;                      // rows of uk a thread has in flight
  Raw<V> raw[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i) raw[i].load(w + (size_t)min(sl + i * SL, d - 1) * n);
  jb::pdl_wait();
  float* q_s = sm;
  float* part = sm + (QT * d + 3) / 4 * 4;
  for (int i = threadIdx.x; i < nt * d; i += Q_THREADS)
    q_s[i] = proj[(size_t)(t0 + i / d) * ld + q_col + (size_t)h * (d + r) + i % d];
  if (chunk == 0) {                             // the turned part and the zero columns, once per head
    const int extra = dp - n;
    for (int i = threadIdx.x; i < nt * extra; i += Q_THREADS) {
      const int t = t0 + i / extra, j = i % extra;
      const float* x = proj + (size_t)t * ld + q_col + (size_t)h * (d + r) + d;
      float v = j < r ? x[j] : 0.0f;
      if (j < r && table != nullptr) {
        const int k = j < half ? j : j - half;
        const float* cs = table + ((size_t)positions[t] * half + k) * 2;
        v = j < half ? v * cs[0] - x[j + half] * cs[1] : v * cs[0] + x[k] * cs[1];
      }
      q_out[((size_t)t * H + h) * dp + n + j] = jb::from_f32<T>(v);
    }
  }
  __syncthreads();
  float acc[QT][V];
#pragma unroll
  for (int k = 0; k < QT; ++k)
#pragma unroll
    for (int v = 0; v < V; ++v) acc[k][v] = 0.0f;
  for (int j0 = sl; j0 < d; j0 += AHEAD * SL) {
    if (j0 != sl) {
#pragma unroll
      for (int i = 0; i < AHEAD; ++i) raw[i].load(w + (size_t)min(j0 + i * SL, d - 1) * n);
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int j = j0 + i * SL;
      if (j < d && active) {
        float wv[V];
        raw[i].template unpack<T>(wv);
#pragma unroll
        for (int k = 0; k < QT; ++k) {
          const float x = k < nt ? q_s[k * d + j] : 0.0f;
#pragma unroll
          for (int v = 0; v < V; ++v) acc[k][v] = fmaf(wv[v], x, acc[k][v]);
        }
      }
    }
  }
#pragma unroll
  for (int k = 0; k < QT; ++k)
#pragma unroll
    for (int v = 0; v < V; ++v) part[(sl * QT + k) * COLS + ct * V + v] = acc[k][v];
  __syncthreads();
  for (int i = threadIdx.x; i < nt * COLS; i += Q_THREADS) {
    const int k = i / COLS, c = i % COLS;
    if (chunk * COLS + c >= n) continue;
    float v = 0.0f;
#pragma unroll
    for (int s = 0; s < SL; ++s) v += part[(s * QT + k) * COLS + c];
    q_out[((size_t)(t0 + k) * H + h) * dp + chunk * COLS + c] = jb::from_f32<T>(v);
  }
}

constexpr int VT = 4;              // tokens of a block of latent_values
constexpr int V_WARPS = 8, V_ROWS = 4;

// out[t, h, c] = (uv[h e + c, :] . o[t, h]) * sigmoid(gate[t, h e + c]) for c < e, zero for e <= c < ep (gate_per_head:
// the gate's column is h).  o comes from
// `o_rows` [T, H, n] (splits == 0), or from the key splits' partial sums: part_o [T, H, splits, n] and part_ml
// [T, H, splits, 2] (maximum in units of log2, sum), o = sum_s f_s part_o[s] / sum_s f_s l_s with f_s = 2^(m_s - max).
// A block owns (a chunk of V_WARPS * V_ROWS value rows, head, VT tokens); a warp takes V_ROWS rows, whose first columns
// it asks for before the wait on the attention kernel.  The blocks of a head's chunks form a cluster: each of them joins
// a part of o's columns and leaves it in the shared memory of all.
template <typename T, int V>
__global__ void __launch_bounds__(V_WARPS * 32) latent_values_kernel(
    const T* __restrict__ o_rows, const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits,
    const T* __restrict__ uv, const float* __restrict__ gate, int ld_gate, int gate_per_head, T* __restrict__ out,
    int n_tokens, int H, int n, int e, int ep) {
  extern __shared__ __align__(16) float o_s[];   // [VT][n padded to 8], then the splits' factors [VT][splits]
  jb::pdl_launch_dependents();
  cg::cluster_group cluster = cg::this_cluster();
  const int members = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
  if (members > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");   // (waited for before the first write to another block)
  const int h = blockIdx.y, t0 = blockIdx.z * VT, nt = min(VT, n_tokens - t0);
  const int np = (n + 7) / 8 * 8, nv = np / V;
  auto place = [&](int c) { return (c % V) * nv + c / V; };      // column c of a row of o_s: lanes read neighbours
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = (blockIdx.x * V_WARPS + warp) * V_ROWS;
  const T* w[V_ROWS];
  Raw<V> raw[V_ROWS][2];                         // the columns lane V and (lane + 32) V of the warp's rows
#pragma unroll
  for (int q = 0; q < V_ROWS; ++q) {
    w[q] = uv + ((size_t)h * e + min(c0 + q, e - 1)) * n;
#pragma unroll
    for (int x = 0; x < 2; ++x)
      if ((lane + 32 * x) * V < n) raw[q][x].load(w[q] + (lane + 32 * x) * V);
  }
  jb::pdl_wait();
  // the sum this lane will write: row my_c of token my_k; its gate is asked for early (no gate: z -> infinity, sigmoid 1)
  const int my_c = c0 + (lane >> 1) / VT, my_k = (lane >> 1) % VT;
  float z = CUDART_INF_F;
  if (gate != nullptr && my_k < nt && my_c < e) z = gate[(size_t)(t0 + my_k) * ld_gate + (gate_per_head ? (size_t)h : (size_t)h * e + my_c)];
  if (splits > 0) {
    float* f_s = o_s + VT * np;
    if (warp < nt) {                             // a warp per token: lanes over the splits
      const float* ml = part_ml + ((size_t)(t0 + warp) * H + h) * splits * 2;
      float m = -CUDART_INF_F, l = 0.0f;
      for (int s = lane; s < splits; s += 32) m = fmaxf(m, ml[2 * s]);
      m = jb::warp_max(m);
      for (int s = lane; s < splits; s += 32) {
        const float f = exp2f(ml[2 * s] - m);    // a split without keys weighs 0
        f_s[warp * splits + s] = f;
        l = fmaf(ml[2 * s + 1], f, l);
      }
      const float inv = 1.0f / jb::warp_sum(l);
      for (int s = lane; s < splits; s += 32) f_s[warp * splits + s] *= inv;
    }
    __syncthreads();
    if (members > 1) asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    auto put = [&](int at, float v) {
      if (members == 1) {
        o_s[at] = v;
      } else {
        for (int m = 0; m < members; ++m) *cluster.map_shared_rank(o_s + at, m) = v;
      }
    };
    if (n % 4 == 0) {
      const int n4 = n >> 2;
      for (int i = threadIdx.x + rank * blockDim.x; i < nt * n4; i += blockDim.x * members) {
        const int k = i / n4, c = i - k * n4;
        const float4* p = reinterpret_cast<const float4*>(part_o + ((size_t)(t0 + k) * H + h) * splits * n) + c;
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
        for (int s = 0; s < splits; ++s) {
          const float f = f_s[k * splits + s];
          const float4 x = p[(size_t)s * n4];
          v.x = fmaf(f, x.x, v.x), v.y = fmaf(f, x.y, v.y), v.z = fmaf(f, x.z, v.z), v.w = fmaf(f, x.w, v.w);
        }
        const int o = k * np;
        put(o + place(4 * c), v.x), put(o + place(4 * c + 1), v.y), put(o + place(4 * c + 2), v.z), put(o + place(4 * c + 3), v.w);
      }
    } else {
      for (int i = threadIdx.x + rank * blockDim.x; i < nt * n; i += blockDim.x * members) {
        const int k = i / n, c = i - k * n;
        const float* p = part_o + ((size_t)(t0 + k) * H + h) * splits * n + c;
        float v = 0.0f;
#pragma unroll 8
        for (int s = 0; s < splits; ++s) v = fmaf(f_s[k * splits + s], p[(size_t)s * n], v);
        put(k * np + place(c), v);
      }
    }
    if (members > 1) cluster.sync();
  } else {
    for (int i = threadIdx.x; i < nt * n; i += blockDim.x)
      o_s[(i / n) * np + place(i % n)] = jb::to_f32(o_rows[((size_t)(t0 + i / n) * H + h) * n + i % n]);
    if (members > 1) asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
  }
  __syncthreads();
  if (c0 >= ep) return;
  float acc[V_ROWS * VT];
#pragma unroll
  for (int i = 0; i < V_ROWS * VT; ++i) acc[i] = 0.0f;
  auto add = [&](const Raw<V>* r, int stride, int i) {      // columns i .. i + V - 1 of the warp's rows
#pragma unroll
    for (int q = 0; q < V_ROWS; ++q) {
      float a[V];
      r[q * stride].template unpack<T>(a);
#pragma unroll
      for (int k = 0; k < VT; ++k) {
        if (k < nt) {
#pragma unroll
          for (int v = 0; v < V; ++v) acc[q * VT + k] = fmaf(a[v], o_s[k * np + v * nv + i / V], acc[q * VT + k]);
        }
      }
    }
  };
#pragma unroll
  for (int x = 0; x < 2; ++x)
    if ((lane + 32 * x) * V < n) add(&raw[0][x], 2, (lane + 32 * x) * V);
  for (int i = (lane + 64) * V; i < n; i += 32 * V) {
    Raw<V> more[V_ROWS];
#pragma unroll
    for (int q = 0; q < V_ROWS; ++q) more[q].load(w[q] + i);
    add(more, 1, i);
  }
  // the warp's 16 sums: every exchange halves what a lane still holds, so lanes 2 i and 2 i + 1 end with sum i
  static_assert(V_ROWS * VT == 16, "sixteen sums a warp");
#pragma unroll
  for (int half = 8; half >= 1; half >>= 1) {
    const bool upper = lane & (2 * half);
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float send = upper ? acc[i] : acc[i + half];
      const float keep = upper ? acc[i + half] : acc[i];
      acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, 2 * half);
    }
  }
  const float sum = acc[0] + __shfl_xor_sync(0xffffffffu, acc[0], 1);
  if (lane % 2 == 0 && my_k < nt && my_c < ep)
    out[((size_t)(t0 + my_k) * H + h) * ep + my_c] = jb::from_f32<T>(my_c < e ? sum * (1.0f / (1.0f + expf(-z))) : 0.0f);
}

// rows[start[s] + i] = the cached row of position i of sequence s; a block per (GATHER rows of a page, sequence), rows
// of `vecs` 16-byte vectors.
constexpr int GATHER = 8;
__global__ void __launch_bounds__(256) gather_rows_kernel(const uint4* __restrict__ cache, const int* __restrict__ block_table,
                                                          int max_pages, int page_size, const int* __restrict__ kv_len,
                                                          const int* __restrict__ start, uint4* __restrict__ rows, int vecs) {
  jb::pdl_launch_dependents();
  jb::pdl_wait();
  const int s = blockIdx.y, first = blockIdx.x * GATHER;
  const int count = min(GATHER, kv_len[s] - first);
  if (count <= 0) return;
  const uint4* src = cache + ((size_t)block_table[(size_t)s * max_pages + first / page_size] * page_size + first % page_size) * vecs;
  uint4* dst = rows + (size_t)(start[s] + first) * vecs;
  for (int i = threadIdx.x; i < count * vecs; i += blockDim.x) dst[i] = src[i];
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

Row make_row(const float* proj, int ld, const float* table, int c_col, int n, int r, int stored, const float* w, float eps,
             const int* dest, void* c_cache, void* rows) {
  const bool vec = ld % 4 == 0 && c_col % 4 == 0 && n % 4 == 0 && r % 8 == 0 && stored % 4 == 0 && aligned16(proj) &&
                   aligned16(table) && aligned16(w) && aligned16(c_cache) && aligned16(rows);
  return Row{c_col, n, r, stored, w, eps, dest, c_cache, rows, vec ? 1 : 0};
}

int check_row(int ld, int r, const Row& row) {
  JB_REFUSE(r < 0 || (r & 1), "latent: %d rotated numbers", r);
  JB_REFUSE(row.c_cache != nullptr && (ld < row.c_col + row.n + row.r || row.stored < row.n + row.r || row.n < 1 ||
                                       row.r != r || row.w == nullptr || row.dest == nullptr),
            "latent: rows of %d floats do not hold a row of %d + %d numbers, or %d columns do not store it", ld, row.n,
            row.r, row.stored);
  return 0;
}
int check_queries(int ld, int q_col, int H, int d, int r, const Row& row) {
  JB_REFUSE(H < 1 || d < 0 || d + r < 1, "latent: %d heads of %d + %d numbers", H, d, r);
  JB_REFUSE(ld < q_col + H * (d + r), "latent: rows of %d floats do not hold the queries", ld);
  return check_row(ld, r, row);
}

}  // namespace

// proj: float32 [T, ld]; q_out [T, H dp], the pages and `rows` in out_dtype; table: float32 [positions][r/2][2] or null
// (no rotation); c_cache null: queries only; rows null: no second copy.
JB_EXPORT int jb_latent_heads(const float* proj, int ld, int q_col, int H, int d, int r, int dp, const float* table,
                              const int* positions, void* q_out, int out_dtype, int c_col, int n, int stored,
                              const float* w, float eps, const int* dest, void* c_cache, void* rows, int T,
                              cudaStream_t stream) {
  if (T <= 0) return 0;
  const Row row = make_row(proj, ld, table, c_col, n, r, stored, w, eps, dest, c_cache, rows);
  if (const int bad = check_queries(ld, q_col, H, d, r, row)) return bad;
  JB_REFUSE(dp < d + r, "latent_heads: heads of %d numbers cannot be stored in %d columns", d + r, dp);
  const bool vec = ld % 4 == 0 && q_col % 4 == 0 && d % 4 == 0 && r % 8 == 0 && dp % 4 == 0 && aligned16(proj) &&
                   aligned16(q_out) && (table == nullptr || aligned16(table));
  jb::Launch cfg(dim3(T, c_cache != nullptr ? 2 : 1), dim3(256), 0, stream);
  cudaError_t e;
#define JB_GO(TO, VEC) \
  e = cudaLaunchKernelEx(&cfg.c, latent_prep_kernel<TO, VEC>, proj, ld, q_col, H, d, r, dp, table, positions, (TO*)q_out, row)
  if (out_dtype == JB_F32) {
    if (vec) JB_GO(float, true);
    else JB_GO(float, false);
  } else if (out_dtype == JB_BF16) {
    if (vec) JB_GO(bf16, true);
    else JB_GO(bf16, false);
  } else {
    return JB_ERR_BAD_DTYPE;
  }
#undef JB_GO
  return (int)e;
}

// proj: float32 [T, ld] with the queries' latent in columns [0, m); w [m] float32; a_out [T, m], the pages and `rows` in
// out_dtype; the row's arguments as in jb_latent_heads.  clear: n_clear floats (whole 16-byte vectors) set to zero, or null.
JB_EXPORT int jb_latent_down(const float* proj, int ld, int m, const float* w, float eps, void* a_out, int out_dtype, int r,
                             const float* table, const int* positions, int c_col, int n, int stored, const float* row_w,
                             const int* dest, void* c_cache, void* rows, float* clear, long long n_clear, int T,
                             cudaStream_t stream) {
  if (T <= 0) return 0;
  const Row row = make_row(proj, ld, table, c_col, n, r, stored, row_w, eps, dest, c_cache, rows);
  JB_REFUSE(m < 1 || ld < m, "latent_down: rows of %d floats do not hold %d numbers", ld, m);
  if (const int bad = check_row(ld, r, row)) return bad;
  JB_REFUSE(clear != nullptr && (n_clear % 4 != 0 || !aligned16(clear)), "latent_down: %lld floats to clear", n_clear);
  const long long vecs = clear != nullptr ? n_clear / 4 : 0;
  jb::Launch cfg(dim3(T, c_cache != nullptr ? 2 : 1), dim3(256), 0, stream);
  const bool vec = ld % 4 == 0 && m % 4 == 0 && aligned16(proj) && aligned16(w) && aligned16(a_out);
#define JB_GO(TO, VEC)                                                                                                    \
  return (int)cudaLaunchKernelEx(&cfg.c, latent_down_kernel<TO, VEC>, proj, ld, m, w, eps, (TO*)a_out, table, positions, \
                                 (float4*)clear, vecs, row)
  if (out_dtype == JB_F32) {
    if (vec) JB_GO(float, true);
    JB_GO(float, false);
  }
  if (out_dtype == JB_BF16) {
    if (vec) JB_GO(bf16, true);
    JB_GO(bf16, false);
  }
#undef JB_GO
  return JB_ERR_BAD_DTYPE;
}

// As jb_latent_heads, the queries multiplied into the latents' space: q_out [T, H dp], dp >= n + r; uk: [H d, n]
// row-major in dtype.
JB_EXPORT int jb_latent_queries(const float* proj, int ld, int q_col, int H, int d, int r, int n, int dp, const void* uk,
                                const float* table, const int* positions, void* q_out, int dtype, int c_col, int stored,
                                const float* w, float eps, const int* dest, void* c_cache, int T, cudaStream_t stream) {
  if (T <= 0) return 0;
  const Row row = make_row(proj, ld, table, c_col, n, r, stored, w, eps, dest, c_cache, nullptr);
  if (const int bad = check_queries(ld, q_col, H, d, r, row)) return bad;
  JB_REFUSE(dp < n + r || n < 1 || d < 1, "latent_queries: %d + %d numbers cannot be stored in %d columns", n, r, dp);
  const int vw = dtype == JB_BF16 ? 8 : 4;
  const bool vec = n % vw == 0 && aligned16(uk);
  const int cols = 8 * (vec ? vw : 1);
  const int chunks = (n + cols - 1) / cols;
  const size_t smem = ((size_t)(QT * d + 3) / 4 * 4 + (size_t)(Q_THREADS / 8) * QT * cols) * sizeof(float);
  JB_REFUSE(smem > 200 * 1024, "latent_queries: heads of %d numbers (%zu bytes) do not fit shared memory", d, smem);
  jb::Launch cfg(dim3(H * chunks + (c_cache != nullptr ? (T < QT ? T : QT) : 0), (T + QT - 1) / QT), dim3(Q_THREADS), smem, stream);
  cudaError_t e = cudaSuccess;
#define JB_GO(T_, V_)                                                                                               \
  do {                                                                                                              \
    auto k = latent_queries_kernel<T_, V_>;                                                                         \
    if (smem > 48 * 1024) e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
    if (e == cudaSuccess)                                                                                           \
      e = cudaLaunchKernelEx(&cfg.c, k, proj, ld, q_col, H, d, r, n, dp, (const T_*)uk, table, positions, (T_*)q_out, T, row); \
  } while (0)
  if (dtype == JB_F32) {
    if (vec) JB_GO(float, 4);
    else JB_GO(float, 1);
  } else if (dtype == JB_BF16) {
    if (vec) JB_GO(bf16, 8);
    else JB_GO(bf16, 1);
  } else {
    return JB_ERR_BAD_DTYPE;
  }
#undef JB_GO
  return (int)e;
}

// uv: [H e, n] row-major; o_rows [T, H n] and out [T, H ep] in dtype; gate: float32 rows of ld_gate numbers, column
// h e + c for number c of head h, or h with gate_per_head (null: no gate).  splits > 0: from part_o and part_ml instead of o_rows.
JB_EXPORT int jb_latent_values(const void* o_rows, const float* part_o, const float* part_ml, int splits, const void* uv,
                               const float* gate, int ld_gate, int gate_per_head, void* out, int dtype, int T, int H, int n,
                               int e, int ep, cudaStream_t stream) {
  if (T <= 0) return 0;
  JB_REFUSE(e < 1 || ep < e || n < 1 || H < 1 || splits < 0, "latent_values: %d values in %d columns from %d numbers", e, ep, n);
  JB_REFUSE(splits > 0 ? (part_o == nullptr || part_ml == nullptr) : o_rows == nullptr, "latent_values: no input");
  const int vw = dtype == JB_BF16 ? 8 : 4;
  const bool vec = n % vw == 0 && aligned16(uv);
  const size_t smem = ((size_t)VT * ((n + 7) / 8 * 8) + (size_t)VT * splits) * sizeof(float);
  JB_REFUSE(smem > 200 * 1024, "latent_values: latents of %d numbers do not fit shared memory", n);
  const int rows = V_WARPS * V_ROWS;
  const int chunks = (ep + rows - 1) / rows;
  jb::Launch cfg(dim3(chunks, H, (T + VT - 1) / VT), dim3(V_WARPS * 32), smem, stream);
  cudaLaunchAttribute attrs[2];
  attrs[0].id = cudaLaunchAttributeClusterDimension;
  attrs[0].val.clusterDim.x = chunks % 8 == 0 ? 8 : chunks % 4 == 0 ? 4 : chunks % 2 == 0 ? 2 : 1;
  attrs[0].val.clusterDim.y = attrs[0].val.clusterDim.z = 1;
  if (cfg.c.numAttrs) attrs[1] = cfg.attr[0];
  cfg.c.attrs = attrs;
  cfg.c.numAttrs += 1;
  cudaError_t err = cudaSuccess;
#define JB_GO(T_, V_)                                                                                               \
  do {                                                                                                              \
    auto k = latent_values_kernel<T_, V_>;                                                                          \
    if (smem > 48 * 1024) err = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
    if (err == cudaSuccess)                                                                                         \
      err = cudaLaunchKernelEx(&cfg.c, k, (const T_*)o_rows, part_o, part_ml, splits, (const T_*)uv, gate, ld_gate, \
                               gate_per_head, (T_*)out, T, H, n, e, ep);                                            \
  } while (0)
  if (dtype == JB_F32) {
    if (vec) JB_GO(float, 4);
    else JB_GO(float, 1);
  } else if (dtype == JB_BF16) {
    if (vec) JB_GO(bf16, 8);
    else JB_GO(bf16, 1);
  } else {
    return JB_ERR_BAD_DTYPE;
  }
#undef JB_GO
  return (int)err;
}

// cache: pages [page][1][page_size][stored] of 16-byte rows (row_bytes a multiple of 16); block_table [n_seqs][max_pages];
// start[s]: the matrix row of position 0 of sequence s; pages: the most pages a sequence has.
JB_EXPORT int jb_gather_rows(const void* cache, const int* block_table, int max_pages, int page_size, const int* kv_len,
                             const int* start, void* rows, int row_bytes, int n_seqs, int pages, cudaStream_t stream) {
  if (n_seqs <= 0 || pages <= 0) return 0;
  JB_REFUSE(page_size % GATHER != 0, "gather_rows: pages of %d rows", page_size);
  JB_REFUSE(row_bytes % 16 != 0 || !aligned16(cache) || !aligned16(rows), "gather_rows: rows of %d bytes", row_bytes);
  jb::Launch cfg(dim3(pages * (page_size / GATHER), n_seqs), dim3(256), 0, stream);
  return (int)cudaLaunchKernelEx(&cfg.c, gather_rows_kernel, (const uint4*)cache, block_table, max_pages, page_size, kv_len,
                                 start, (uint4*)rows, row_bytes / 16);
}
