// Dynamic tanh in the place of a norm, N(x) = tanh(alpha x) * w + b feature by feature (no mean, no variance), and
// the sum of a sublayer's output into the residual stream around it, in one launch.  All arithmetic is float32.
// For one number of the stream r [T, W]:
//
//   r <- r + mult * Na(y)        (y: a sublayer's float32 output, set to zero afterwards; skipped without y)
//   r <- Na(r)                   (replace = 1, no y: the stream itself passes the norm)
//   x  = Nb(r)                   (in the engine dtype; without Nb the cast alone; skipped without x)
//
// With row_index the rows of x are picked (x[i] from r[row_index[i]]) and the stream is only read.  `clear`, `clear2`:
// float32 buffers of whole 16-byte vectors that the launch sets to zero on the way.  A thread takes four neighbours
// (rows of whole, aligned 16-byte vectors) or one number.
#include <stdio.h>

#include "common.cuh"

namespace {

typedef __nv_bfloat16 bf16;

struct Squash {
  const float* w;
  const float* b;
  float alpha;
};

__device__ __forceinline__ void clear_slice(float4* buf, size_t n4) {
  if (buf == nullptr) return;
  const float4 z = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n4; i += (size_t)gridDim.x * blockDim.x) buf[i] = z;
}

template <int V>
__device__ __forceinline__ void load(const float* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
  } else {
    v[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void store(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int V>
__device__ __forceinline__ void store(bf16* p, const float (&v)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&lo);
    u.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

template <int V>
__device__ __forceinline__ void squash(float (&v)[V], const Squash& n, int c) {
  float w[V], b[V];
  load<V>(n.w + c, w);
  load<V>(n.b + c, b);
#pragma unroll
  for (int j = 0; j < V; ++j) v[j] = fmaf(tanhf(n.alpha * v[j]), w[j], b[j]);
}

template <typename TO, int V>
__global__ void __launch_bounds__(256) tanh_norm_kernel(float* __restrict__ stream, float* __restrict__ y, Squash na,
                                                        float mult, int replace, Squash nb, TO* __restrict__ x_out,
                                                        const int* __restrict__ row_index, unsigned n, int W,
                                                        float4* __restrict__ clear, size_t clear_n4,
                                                        float4* __restrict__ clear2, size_t clear2_n4) {
  jb::pdl_launch_dependents();
  jb::pdl_wait();
  clear_slice(clear, clear_n4);
  clear_slice(clear2, clear2_n4);
  const unsigned per_row = (unsigned)W / V;
  for (unsigned i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
    const unsigned row = i / per_row;
    const int c = (int)(i - row * per_row) * V;
    const size_t at = (size_t)i * V;
    const size_t src = row_index != nullptr ? (size_t)row_index[row] * W + c : at;
    float r[V];
    load<V>(stream + src, r);
    if (y != nullptr) {
      float d[V], zero[V];
      load<V>(y + src, d);
#pragma unroll
      for (int j = 0; j < V; ++j) zero[j] = 0.0f;
      store<V>(y + src, zero);
      squash<V>(d, na, c);
#pragma unroll
      for (int j = 0; j < V; ++j) r[j] = fmaf(mult, d[j], r[j]);
      store<V>(stream + src, r);
    } else if (replace) {
      squash<V>(r, na, c);
      store<V>(stream + src, r);
    }
    if (x_out != nullptr) {
      if (nb.w != nullptr) squash<V>(r, nb, c);
      store<V>(x_out + at, r);
    }
  }
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace

// stream: float32 [., W]; y: float32, as the stream, or null; (wa, ba, alpha_a) the norm on y (or, with replace, on
// the stream), (wb, bb, alpha_b) the norm of x_out's rows (null: a cast); x_out: [rows, W] in out_dtype, or null;
// row_index: int32 [rows] or null.
JB_EXPORT int jb_tanh_norm(float* stream, float* y, const float* wa, const float* ba, float alpha_a, float mult,
                           int replace, const float* wb, const float* bb, float alpha_b, void* x_out, int out_dtype,
                           const int* row_index, int rows, int W, float* clear, long long clear_n, float* clear2,
                           long long clear2_n, cudaStream_t s) {
  if (rows <= 0) return 0;
  JB_REFUSE(W <= 0, "tanh_norm: rows of %d numbers", W);
  JB_REFUSE((y != nullptr || replace) && (wa == nullptr || ba == nullptr), "tanh_norm: the first norm has no weights");
  JB_REFUSE((wb == nullptr) != (bb == nullptr), "tanh_norm: the second norm needs a weight and a bias");
  JB_REFUSE(row_index != nullptr && (y != nullptr || replace), "tanh_norm: picked rows are only read");
  JB_REFUSE(((clear_n | clear2_n) & 3) || !aligned16(clear) || !aligned16(clear2),
            "tanh_norm: buffers to clear must be whole, aligned 16-byte vectors");
  const bool vec = W % 4 == 0 && aligned16(stream) && aligned16(y) && aligned16(wa) && aligned16(ba) && aligned16(wb) &&
                   aligned16(bb) && aligned16(x_out);
  const size_t n = (size_t)rows * W / (vec ? 4 : 1);
  JB_REFUSE(n >= 0x7fffffffull, "tanh_norm: %d rows of %d numbers are too many", rows, W);
  const int threads = n <= 148 * 256 ? 64 : 256;      // few numbers: spread over the SMs
  const size_t want = (n + threads - 1) / threads;
  jb::Launch cfg(dim3((unsigned)(want < 148 * 16 ? want : 148 * 16)), dim3(threads), 0, s);
  const Squash na{wa, ba, alpha_a}, nb{wb, bb, alpha_b};
  cudaError_t e;
#define JB_GO(TO, V)                                                                                             \
  e = cudaLaunchKernelEx(&cfg.c, tanh_norm_kernel<TO, V>, stream, y, na, mult, replace, nb, (TO*)x_out, row_index, (unsigned)n, \
                         W, (float4*)clear, (size_t)(clear_n / 4), (float4*)clear2, (size_t)(clear2_n / 4))
  if (out_dtype == JB_F32) {
    if (vec) JB_GO(float, 4);
    else JB_GO(float, 1);
  } else if (out_dtype == JB_BF16) {
    if (vec) JB_GO(bf16, 4);
    else JB_GO(bf16, 1);
  } else {
    return JB_ERR_BAD_DTYPE;
  }
#undef JB_GO
  return (int)e;
}
