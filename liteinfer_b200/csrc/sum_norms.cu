// A residual stream in 32-bit that takes a sum of several sublayers' outputs at once, and the norms that read it next.
//
//   li_sum_norms   d = sum of terms;  v = x[row] + d;  x[row] = v (optional);  out_i = v / sqrt(mean(v^2) + eps) * w_i
//                  for one or two weights (the norms in front of sublayers that run side by side: one pass over the
//                  row, one sum of squares); or only the sum is made; or, without a stream, out_1 = d.
//
// The terms: up to two dense ones [tokens, width] in the engine's type, each times a constant and optionally times a
// float of its row; and optionally rows of experts: `top` rows of `routed` per token, row place[token * top + s] (or the
// pair itself), already multiplied by their weights.  Everything is summed in 32-bit, dense terms in order, then the
// experts' rows in slot order, then the stream.  One block a row, the row in registers by 16-byte accesses where the
// width allows, else in shared memory.  The order of every sum depends on the row's width only.
#include "common.cuh"

namespace li {

struct SumTerms {
  const void* dense[2];
  float factor[2];
  const float* row_factor[2];
  const void* routed;
  const int* place;
  int top;
};

template <typename T> __device__ __forceinline__ void four(const T* p, float (&o)[4]);
template <> __device__ __forceinline__ void four<float>(const float* p, float (&o)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
}
template <> __device__ __forceinline__ void four<bf16>(const bf16* p, float (&o)[4]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  o[0] = __uint_as_float(v.x << 16); o[1] = __uint_as_float(v.x & 0xffff0000u);
  o[2] = __uint_as_float(v.y << 16); o[3] = __uint_as_float(v.y & 0xffff0000u);
}
__device__ __forceinline__ void put_four(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void put_four(bf16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}

// NV: groups of four columns a thread keeps.  x may be null (the sum itself goes to out_1).
template <typename T, int NV>
__global__ void __launch_bounds__(1024)
sum_norms_kernel(float* __restrict__ x, const SumTerms terms, const float* __restrict__ w1, const float* __restrict__ w2,
                 T* __restrict__ out1, T* __restrict__ out2, const int* __restrict__ rows, int width, float eps,
                 int write_stream) {
  __shared__ float scratch[33];
  float w[2][NV][4];
  int col[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    col[i] = (i * blockDim.x + threadIdx.x) * 4;
    if (col[i] < width) {
      if (w1 != nullptr) four<float>(w1 + col[i], w[0][i]);
      if (w2 != nullptr) four<float>(w2 + col[i], w[1][i]);
    }
  }
  grid_dependency_wait();
  const int r = blockIdx.x, row = rows != nullptr ? rows[r] : r;
  float v[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const T* dense = static_cast<const T*>(terms.dense[k]);
    if (dense == nullptr) continue;
    const float factor = terms.factor[k] * (terms.row_factor[k] != nullptr ? terms.row_factor[k][row] : 1.0f);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < width) {
        float y[4];
        four<T>(dense + (size_t)row * width + col[i], y);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[i][e] = fmaf(factor, y[e], v[i][e]);
      }
  }
  if (terms.routed != nullptr) {
    const T* routed = static_cast<const T*>(terms.routed);
    const size_t first = (size_t)row * terms.top;
#pragma unroll 4
    for (int s = 0; s < terms.top; ++s) {
      const size_t at = terms.place != nullptr ? (size_t)terms.place[first + s] : first + s;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (col[i] < width) {
          float y[4];
          four<T>(routed + at * width + col[i], y);
#pragma unroll
          for (int e = 0; e < 4; ++e) v[i][e] += y[e];
        }
    }
  }
  if (x == nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < width) put_four(out1 + (size_t)r * width + col[i], v[i]);
    return;
  }
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col[i] < width) {
      float base[4];
      four<float>(x + (size_t)row * width + col[i], base);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[i][e] += base[e];
        q = fmaf(v[i][e], v[i][e], q);
      }
      if (write_stream) put_four(x + (size_t)row * width + col[i], v[i]);
    }
  if (out1 == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum(q, scratch) / (float)width + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col[i] < width) {
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = v[i][e] * inv * w[0][i][e];
      put_four(out1 + (size_t)r * width + col[i], y);
      if (out2 != nullptr) {
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = v[i][e] * inv * w[1][i][e];
        put_four(out2 + (size_t)r * width + col[i], y);
      }
    }
}

// The same, any width, a column at a time.
template <typename T>
__global__ void __launch_bounds__(256)
sum_norms_plain_kernel(float* __restrict__ x, const SumTerms terms, const float* __restrict__ w1,
                       const float* __restrict__ w2, T* __restrict__ out1, T* __restrict__ out2,
                       const int* __restrict__ rows, int width, float eps, int write_stream) {
  extern __shared__ float kept[];      // [width]
  __shared__ float scratch[33];
  grid_dependency_wait();
  const int r = blockIdx.x, row = rows != nullptr ? rows[r] : r;
  float q = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float v = 0.f;
    for (int k = 0; k < 2; ++k) {
      const T* dense = static_cast<const T*>(terms.dense[k]);
      if (dense == nullptr) continue;
      const float factor = terms.factor[k] * (terms.row_factor[k] != nullptr ? terms.row_factor[k][row] : 1.0f);
      v = fmaf(factor, to_float(dense[(size_t)row * width + c]), v);
    }
    if (terms.routed != nullptr)
      for (int s = 0; s < terms.top; ++s) {
        const size_t pair = (size_t)row * terms.top + s;
        v += to_float(static_cast<const T*>(terms.routed)[(terms.place != nullptr ? (size_t)terms.place[pair] : pair) * width + c]);
      }
    if (x == nullptr) {
      out1[(size_t)r * width + c] = from_float<T>(v);
      continue;
    }
    v += x[(size_t)row * width + c];
    if (write_stream) x[(size_t)row * width + c] = v;
    kept[c] = v;
    q = fmaf(v, v, q);
  }
  if (x == nullptr || out1 == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum(q, scratch) / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    out1[(size_t)r * width + c] = from_float<T>(kept[c] * inv * w1[c]);
    if (out2 != nullptr) out2[(size_t)r * width + c] = from_float<T>(kept[c] * inv * w2[c]);
  }
}

}  // namespace li

using namespace li;

// x [tokens, width] float32 or null; out_1, out_2 [n, width] in `dtype` (out_2 may be null; out_1 null: only the sum is
// made); weights [width] float32; rows (optional) [n]: the rows to be made.  dense_i null: no such term.
LI_EXPORT int li_sum_norms(int dtype, float* x, const void* dense_0, float factor_0, const float* row_factor_0,
                           const void* dense_1, float factor_1, const float* row_factor_1, const void* routed,
                           const int* place, int top, const float* w1, const float* w2, void* out_1, void* out_2,
                           const int* rows, int n, int width, float eps, int write_stream, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width < 1 || (size_t)width * sizeof(float) > 48 * 1024 * 4) return LI_ERR_UNSUPPORTED;
  if ((x == nullptr && out_1 == nullptr) || (x != nullptr && out_1 != nullptr && w1 == nullptr) ||
      (out_2 != nullptr && (w2 == nullptr || out_1 == nullptr)))
    return LI_ERR_UNSUPPORTED;
  const SumTerms terms{{dense_0, dense_1}, {factor_0, factor_1}, {row_factor_0, row_factor_1}, routed, place, top};
  const bool vec = width % 4 == 0 && width <= 16384 && aligned16(x) && aligned16(dense_0) && aligned16(dense_1) &&
                   aligned16(routed) && aligned16(w1) && aligned16(w2) && aligned16(out_1) && aligned16(out_2);
  if (vec) {
    const int quads = width / 4;
    const int block = quads >= 1024 ? 1024 : (quads + 31) / 32 * 32;
    const int per_thread = (quads + block - 1) / block;
#define LI_SUM(T, NV)                                                                                                 \
  return (int)launch_pdl(n, sum_norms_kernel<T, NV>, dim3(n), dim3(block), 0, stream, x, terms, w1, w2, (T*)out_1,    \
                         (T*)out_2, rows, width, eps, write_stream)
#define LI_SUM_NV(T)                                                                                                  \
  {                                                                                                                   \
    if (per_thread == 1) LI_SUM(T, 1);                                                                                \
    if (per_thread == 2) LI_SUM(T, 2);                                                                                \
    LI_SUM(T, 4);                                                                                                     \
  }
    if (dtype == kFloat32) LI_SUM_NV(float)
    LI_SUM_NV(bf16)
#undef LI_SUM_NV
#undef LI_SUM
  }
  const size_t smem = (size_t)width * sizeof(float);
#define LI_SUM_PLAIN(T)                                                                                               \
  {                                                                                                                   \
    if (smem > 48 * 1024) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(sum_norms_plain_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,     \
                                           (int)smem);                                                                \
      if (e != cudaSuccess) return (int)e;                                                                            \
    }                                                                                                                 \
    return (int)launch_pdl(n, sum_norms_plain_kernel<T>, dim3(n), dim3(256), smem, stream, x, terms, w1, w2, (T*)out_1, \
                           (T*)out_2, rows, width, eps, write_stream);                                                \
  }
  if (dtype == kFloat32) LI_SUM_PLAIN(float)
  LI_SUM_PLAIN(bf16)
#undef LI_SUM_PLAIN
}
