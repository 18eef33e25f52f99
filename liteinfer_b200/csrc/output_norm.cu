// What a sublayer gives back, put together, normalised and added into a residual stream in 32-bit, in one pass.
//
//   li_output_norm   y = sum of terms;  v = x[row] + y / sqrt(mean(y^2) + eps_y) * w_y;  x[row] = v (optional);
//                    out = v, rounded, or v / sqrt(mean(v^2) + eps) * w;  or out is left out.
//
// The terms of y: up to two dense ones [tokens, width] in the engine's type, each optionally divided by its own root mean
// square over the row and multiplied by a weight (mixers side by side that are each normalised on their way out), times a
// constant, and optionally times a float of its row; and optionally rows of experts: row place[token * top + s] of `routed`
// for s < top (a negative place: the slot has no row; place null: the pair itself), already multiplied by their weights.
// Everything is 32-bit; dense terms in order, then the experts' rows in slot order.  One block a row, the row in registers
// by 16-byte accesses where the width allows, else in shared memory.  The order of every sum depends on the width only.
#include "common.cuh"

namespace li {

struct OutputTerms {
  const void* dense[2];
  float factor[2];
  const float* row_factor[2];
  const float* norm_weight[2];      // not null: the term is normalised first
  float norm_eps[2];
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

// NV: groups of four columns a thread keeps.  (x and a dense term may be the same rows: a thread reads its columns of all
// terms before it stores any of x.)
template <typename T, int NV>
__global__ void __launch_bounds__(1024)
output_norm_kernel(float* x, const OutputTerms terms, const float* __restrict__ w_y, float eps_y, const float* __restrict__ w,
                   float eps, T* __restrict__ out, const int* __restrict__ rows, int width, int write_stream) {
  __shared__ float scratch[66];
  constexpr bool kEarly = NV == 1;            // the weights wait in registers only where there are enough of them
  float wy[NV][4], wo[NV][4], wt[2][NV][4];
  int col[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    col[i] = (i * blockDim.x + threadIdx.x) * 4;
    if (kEarly && col[i] < width) {           // the weights are inputs of the model: on their way before the wait
      four<float>(w_y + col[i], wy[i]);
      if (w != nullptr) four<float>(w + col[i], wo[i]);
#pragma unroll
      for (int k = 0; k < 2; ++k)
        if (terms.norm_weight[k] != nullptr) four<float>(terms.norm_weight[k] + col[i], wt[k][i]);
    }
  }
  grid_dependency_wait();
  const int r = blockIdx.x, row = rows != nullptr ? rows[r] : r;
  const float n = (float)width;
  float y[NV][4], base[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
    if (kEarly && col[i] < width) four<float>(x + (size_t)row * width + col[i], base[i]);
  }
  float t[2][NV][4];
  float2 ss = make_float2(0.f, 0.f);
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const T* dense = static_cast<const T*>(terms.dense[k]);
    if (dense == nullptr) continue;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < width) {
        four<T>(dense + (size_t)row * width + col[i], t[k][i]);
#pragma unroll
        for (int e = 0; e < 4; ++e) (k == 0 ? ss.x : ss.y) = fmaf(t[k][i][e], t[k][i][e], k == 0 ? ss.x : ss.y);
      }
  }
  if (terms.norm_weight[0] != nullptr || terms.norm_weight[1] != nullptr) ss = block_sum2(ss, scratch);
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    if (terms.dense[k] == nullptr) continue;
    float factor = terms.factor[k] * (terms.row_factor[k] != nullptr ? terms.row_factor[k][row] : 1.0f);
    const bool normed = terms.norm_weight[k] != nullptr;
    if (normed) factor *= 1.0f / sqrtf((k == 0 ? ss.x : ss.y) / n + terms.norm_eps[k]);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < width) {
        if (!kEarly && normed) four<float>(terms.norm_weight[k] + col[i], wt[k][i]);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[i][e] = fmaf(factor, normed ? t[k][i][e] * wt[k][i][e] : t[k][i][e], y[i][e]);
      }
  }
  if (terms.routed != nullptr) {
    const T* routed = static_cast<const T*>(terms.routed);
    const size_t first = (size_t)row * terms.top;
#pragma unroll 4
    for (int s = 0; s < terms.top; ++s) {
      const long at = terms.place != nullptr ? (long)terms.place[first + s] : (long)(first + s);
      if (at < 0) continue;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (col[i] < width) {
          float v[4];
          four<T>(routed + (size_t)at * width + col[i], v);
#pragma unroll
          for (int e = 0; e < 4; ++e) y[i][e] += v[e];
        }
    }
  }
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col[i] < width)
#pragma unroll
      for (int e = 0; e < 4; ++e) q = fmaf(y[i][e], y[i][e], q);
  const float inv_y = 1.0f / sqrtf(block_sum(q, scratch) / n + eps_y);
  q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col[i] < width) {
      if (!kEarly) {
        four<float>(x + (size_t)row * width + col[i], base[i]);
        four<float>(w_y + col[i], wy[i]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        y[i][e] = base[i][e] + y[i][e] * inv_y * wy[i][e];
        q = fmaf(y[i][e], y[i][e], q);
      }
      if (write_stream) put_four(x + (size_t)row * width + col[i], y[i]);
    }
  if (out == nullptr) return;
  float inv = 1.0f;
  if (w != nullptr) inv = 1.0f / sqrtf(block_sum(q, scratch) / n + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col[i] < width) {
      if (w != nullptr) {
        if (!kEarly) four<float>(w + col[i], wo[i]);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[i][e] = y[i][e] * inv * wo[i][e];
      }
      put_four(out + (size_t)r * width + col[i], y[i]);
    }
}

// The same, any width, a column at a time.
template <typename T>
__global__ void __launch_bounds__(256)
output_norm_plain_kernel(float* x, const OutputTerms terms, const float* __restrict__ w_y, float eps_y,
                         const float* __restrict__ w, float eps, T* __restrict__ out, const int* __restrict__ rows, int width,
                         int write_stream) {
  extern __shared__ float kept[];      // [width]
  __shared__ float scratch[66];
  grid_dependency_wait();
  const int r = blockIdx.x, row = rows != nullptr ? rows[r] : r;
  const float n = (float)width;
  float2 ss = make_float2(0.f, 0.f);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    if (terms.norm_weight[0] != nullptr) {
      const float v = to_float(static_cast<const T*>(terms.dense[0])[(size_t)row * width + c]);
      ss.x = fmaf(v, v, ss.x);
    }
    if (terms.norm_weight[1] != nullptr) {
      const float v = to_float(static_cast<const T*>(terms.dense[1])[(size_t)row * width + c]);
      ss.y = fmaf(v, v, ss.y);
    }
  }
  ss = block_sum2(ss, scratch);
  float factor[2];
  for (int k = 0; k < 2; ++k) {
    factor[k] = terms.factor[k] * (terms.row_factor[k] != nullptr ? terms.row_factor[k][row] : 1.0f);
    if (terms.norm_weight[k] != nullptr) factor[k] *= 1.0f / sqrtf((k == 0 ? ss.x : ss.y) / n + terms.norm_eps[k]);
  }
  float q = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float y = 0.f;
    for (int k = 0; k < 2; ++k) {
      if (terms.dense[k] == nullptr) continue;
      const float v = to_float(static_cast<const T*>(terms.dense[k])[(size_t)row * width + c]);
      y = fmaf(factor[k], terms.norm_weight[k] != nullptr ? v * terms.norm_weight[k][c] : v, y);
    }
    if (terms.routed != nullptr)
      for (int s = 0; s < terms.top; ++s) {
        const size_t pair = (size_t)row * terms.top + s;
        const long at = terms.place != nullptr ? (long)terms.place[pair] : (long)pair;
        if (at >= 0) y += to_float(static_cast<const T*>(terms.routed)[(size_t)at * width + c]);
      }
    kept[c] = y;
    q = fmaf(y, y, q);
  }
  const float inv_y = 1.0f / sqrtf(block_sum(q, scratch) / n + eps_y);
  q = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = x[(size_t)row * width + c] + kept[c] * inv_y * w_y[c];
    if (write_stream) x[(size_t)row * width + c] = v;
    kept[c] = v;
    q = fmaf(v, v, q);
  }
  if (out == nullptr) return;
  const float inv = w != nullptr ? 1.0f / sqrtf(block_sum(q, scratch) / n + eps) : 1.0f;
  for (int c = threadIdx.x; c < width; c += blockDim.x)
    out[(size_t)r * width + c] = from_float<T>(w != nullptr ? kept[c] * inv * w[c] : kept[c]);
}

}  // namespace li

using namespace li;

// x [tokens, width] float32; out [n, width] in `dtype` or null; w_y, w [width] float32 (w null: out is the sum itself);
// rows (optional) [n]: the rows to be made.  dense_i null: no such term; norm_i null: the term as it is.
LI_EXPORT int li_output_norm(int dtype, float* x, const void* dense_0, float factor_0, const float* row_factor_0,
                             const float* norm_0, float norm_eps_0, const void* dense_1, float factor_1,
                             const float* row_factor_1, const float* norm_1, float norm_eps_1, const void* routed,
                             const int* place, int top, const float* w_y, float eps_y, const float* w, float eps, void* out,
                             const int* rows, int n, int width, int write_stream, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width < 1 || (size_t)width * sizeof(float) > 48 * 1024 * 4 || x == nullptr || w_y == nullptr) return LI_ERR_UNSUPPORTED;
  if ((norm_0 != nullptr && dense_0 == nullptr) || (norm_1 != nullptr && dense_1 == nullptr) || (out == nullptr && !write_stream))
    return LI_ERR_UNSUPPORTED;
  const OutputTerms terms{{dense_0, dense_1}, {factor_0, factor_1}, {row_factor_0, row_factor_1}, {norm_0, norm_1},
                          {norm_eps_0, norm_eps_1}, routed, place, top};
  const bool vec = width % 4 == 0 && width <= 16384 && aligned16(x) && aligned16(dense_0) && aligned16(dense_1) &&
                   aligned16(norm_0) && aligned16(norm_1) && aligned16(routed) && aligned16(w_y) && aligned16(w) && aligned16(out);
  if (vec) {
    const int quads = width / 4;
    const int block = quads >= 1024 ? 1024 : (quads + 31) / 32 * 32;
    const int per_thread = (quads + block - 1) / block;
#define LI_OUT(T, NV)                                                                                                 \
  return (int)launch_pdl(n, output_norm_kernel<T, NV>, dim3(n), dim3(block), 0, stream, x, terms, w_y, eps_y, w, eps, \
                         (T*)out, rows, width, write_stream)
#define LI_OUT_NV(T)                                                                                                  \
  {                                                                                                                   \
    if (per_thread == 1) LI_OUT(T, 1);                                                                                \
    if (per_thread == 2) LI_OUT(T, 2);                                                                                \
    LI_OUT(T, 4);                                                                                                     \
  }
    if (dtype == kFloat32) LI_OUT_NV(float)
    LI_OUT_NV(bf16)
#undef LI_OUT_NV
#undef LI_OUT
  }
  const size_t smem = (size_t)width * sizeof(float);
#define LI_OUT_PLAIN(T)                                                                                               \
  {                                                                                                                   \
    if (smem > 48 * 1024) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(output_norm_plain_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,   \
                                           (int)smem);                                                                \
      if (e != cudaSuccess) return (int)e;                                                                            \
    }                                                                                                                 \
    return (int)launch_pdl(n, output_norm_plain_kernel<T>, dim3(n), dim3(256), smem, stream, x, terms, w_y, eps_y, w, eps, \
                           (T*)out, rows, width, write_stream);                                                       \
  }
  if (dtype == kFloat32) LI_OUT_PLAIN(float)
  LI_OUT_PLAIN(bf16)
#undef LI_OUT_PLAIN
}
