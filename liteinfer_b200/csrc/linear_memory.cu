// Two memories that are linear in what they hold: per request and head a matrix S [dim, vdim] in 32-bit, from zero.
//
//   state space (Mamba-2): with B, C [dim] of the head's group, x [vdim], dt = softplus(z + dt_bias), one number a head:
//     S <- exp(-exp(A_log) dt) S + B (dt x)^T;  y = S^T C          (y + D x, the gate and the norm come behind:
//                                                                   li_gated_group_norm)
//   time mixing (RWKV-6):  with r, k [dim], v [vdim = dim], decay w = exp(-exp(W2 tanh(l) + w0)) [dim], bonus u [dim]:
//     o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T
//
//   li_ssd_steps / li_wkv_steps   steps in which some sequence brings several tokens.  Two kernels: the first turns every
//                                 token's inputs into records of floats (dim and vdim rounded up, the places past them
//                                 zero), so that the second only copies; the second runs the recurrence and writes
//                                 S^T C, or S^T r (with the bonus (r . u k) v added by li_gated_rmsnorm behind it).
//   li_ssd_token                  steps of single tokens: gates and recurrence in one kernel.
//   li_wkv_token                  steps of single tokens: decay, recurrence, the norm per head and the gate in one.
//   li_token_shift                out[i][t] = x[t] + (x[t - 1] - x[t]) mu[i] for several mu at once; before a step's first
//                                 token of a sequence stands what the request keeps (zeros at its start).
//
// The state is kept column by column, state[slot][head][vdim][dim]: a column is a chain of its own over the tokens.  In
// the steps form a block takes 16 columns of one head of one sequence, a warp two of them, each lane dim / 32 of their
// entries in registers for the whole step, so an entry read from shared memory serves two columns.  Records come in
// chunks of up to 16 tokens by cp.async, three chunks deep, one block barrier a chunk, and a lane has the next token's
// entries on their way to its registers while it works on this one's.  The read-outs of eight tokens are added up over the
// lanes together: sixteen shuffles for sixteen sums, each the same tree whatever the token's place in a step.  In the
// token form a block takes one head of one sequence and walks its columns, sixteen lanes a column and several columns in
// flight: the state's bytes are all the work there.  Sequences that bring no token touch nothing.
#include "common.cuh"

namespace li {

constexpr int kColumns = 16;        // of a block of the steps form: eight warps x two columns
constexpr int kStepThreads = 256;
constexpr int kStages = 3;
constexpr int kRowGroups = 16;      // of a block of the token form: eight warps x two groups of lanes

// Two floats in one 64-bit register, and the two-wide arithmetic on them (each lane of the pair rounds on its own).
typedef unsigned long long pair_t;
__device__ __forceinline__ pair_t make_pair2(float a, float b) {
  pair_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ pair_t mul2(pair_t a, pair_t b) {
  pair_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ pair_t fma2(pair_t a, pair_t b, pair_t c) {
  pair_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ float sum2(pair_t a) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
  return x + y;
}
__device__ __forceinline__ void copy16(float* smem, const float* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem));
}

__device__ __forceinline__ float softplus_of(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// ------------------------------------------------------------------------------------------ several tokens
// A record of a token lies in two parts: `shared_part` floats that all heads of a group read (or one head, with as many
// groups as heads) and behind a pointer of its own the head's part.
//   kScalar (state space): group part C [dimp] | B [dimp]; head part dt x [vdimp] | decay, 0, 0, 0.
//   else (time mixing):    group part r [dimp] | k [dimp] | w [dimp]; head part v [vdimp].
// kScalar also says when a token reads: behind its own update (state space) or before it.

template <int N, bool kScalar>
struct Entries {
  pair_t q[N], k[N], w[kScalar ? 1 : N];
  float2 v;
};

// The entry that the first half of pair `i` of a lane is.
template <int N> __device__ __forceinline__ int entry_of(int i, int lane) {
  return N == 1 ? 2 * lane : 4 * (lane + 32 * (i >> 1)) + 2 * (i & 1);
}

template <int N>
__device__ __forceinline__ void fetch_pairs(pair_t (&p)[N], const float* __restrict__ row, int lane) {
  if (N == 1) {
    p[0] = *reinterpret_cast<const pair_t*>(row + 2 * lane);
  } else {
#pragma unroll
    for (int j = 0; j < N / 2; ++j) {
      const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(row + 4 * (lane + 32 * j));
      p[2 * j] = v.x;
      p[2 * j + 1] = v.y;
    }
  }
}

template <int N, bool kScalar>
__device__ __forceinline__ void fetch_entries(Entries<N, kScalar>& t, const float* __restrict__ row, int lane, int warp) {
  constexpr int dimp = 64 * N, group_part = (kScalar ? 2 : 3) * dimp;
  fetch_pairs<N>(t.q, row, lane);
  fetch_pairs<N>(t.k, row + dimp, lane);
  if constexpr (kScalar) {
    const float a = row[group_part + kColumns];
    t.w[0] = make_pair2(a, a);
  } else {
    fetch_pairs<N>(t.w, row + 2 * dimp, lane);
  }
  t.v = *reinterpret_cast<const float2*>(row + group_part + 2 * warp);
}

template <int N, bool kScalar>
__device__ __forceinline__ void memory_step(pair_t (&S)[2][N], const Entries<N, kScalar>& t, float& read0, float& read1) {
  const pair_t v0 = make_pair2(t.v.x, t.v.x), v1 = make_pair2(t.v.y, t.v.y);
  pair_t a0, a1;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    if (!kScalar) {
      a0 = i == 0 ? mul2(S[0][i], t.q[i]) : fma2(S[0][i], t.q[i], a0);
      a1 = i == 0 ? mul2(S[1][i], t.q[i]) : fma2(S[1][i], t.q[i], a1);
    }
    const pair_t w = t.w[kScalar ? 0 : i];
    S[0][i] = fma2(w, S[0][i], mul2(t.k[i], v0));
    S[1][i] = fma2(w, S[1][i], mul2(t.k[i], v1));
    if (kScalar) {
      a0 = i == 0 ? mul2(S[0][i], t.q[i]) : fma2(S[0][i], t.q[i], a0);
      a1 = i == 0 ? mul2(S[1][i], t.q[i]) : fma2(S[1][i], t.q[i], a1);
    }
  }
  read0 = sum2(a0);
  read1 = sum2(a1);
}

// N: pairs of entries of a column that a lane keeps; dimp = 64 N.
template <int N, int CHUNK, bool kScalar>
__global__ void __launch_bounds__(kStepThreads)
memory_steps_kernel(const float* __restrict__ group_records, const float* __restrict__ head_records,
                    float* __restrict__ state, const int* __restrict__ query_start_loc, const int* __restrict__ state_slots,
                    float* __restrict__ out, int heads, int groups, int dim, int vdim, int vdimp) {
  extern __shared__ __align__(16) float staged[];       // kStages x CHUNK x (group part, v [kColumns], decay [4])
  constexpr int dimp = 64 * N, group_part = (kScalar ? 2 : 3) * dimp;
  constexpr int kPerToken = group_part + kColumns + (kScalar ? 4 : 0);
  constexpr int kCopies = kPerToken / 4;                // 16-byte copies of a token
  const int seq = blockIdx.z, head = blockIdx.y, first_column = blockIdx.x * kColumns;
  const int begin = query_start_loc[seq], end = query_start_loc[seq + 1];
  if (end <= begin) return;
  const int slot = state_slots[seq];
  if (slot < 0) return;
  const int chunks = (end - begin + CHUNK - 1) / CHUNK;
  const int head_part = vdimp + (kScalar ? 4 : 0);
  const float* group_source = group_records + ((size_t)begin * groups + head / (heads / groups)) * group_part;
  const float* head_source = head_records + ((size_t)begin * heads + head) * head_part;
  const size_t group_stride = (size_t)groups * group_part, head_stride = (size_t)heads * head_part;

  auto stage = [&](int c) {
    float* dst = staged + (c % kStages) * CHUNK * kPerToken;
    const int n = min(CHUNK, end - begin - c * CHUNK) * kCopies;
    for (int i = threadIdx.x; i < n; i += kStepThreads) {
      const int tok = i / kCopies, e = (i - tok * kCopies) * 4;
      const size_t t = c * CHUNK + tok;
      const float* src;
      if (e < group_part) src = group_source + t * group_stride + e;
      else if (e < group_part + kColumns) src = head_source + t * head_stride + first_column + (e - group_part);
      else src = head_source + t * head_stride + vdimp;
      copy16(dst + tok * kPerToken + e, src);
    }
  };

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col0 = first_column + 2 * warp;             // and the next one
  grid_dependency_wait();
#pragma unroll
  for (int c = 0; c < kStages - 1; ++c) {
    if (c < chunks) stage(c);
    asm volatile("cp.async.commit_group;\n" ::);
  }
  float* mine = state + (((size_t)slot * heads + head) * vdim + col0) * dim;
  const bool vec = dim % 2 == 0;                        // (the caller's state is 16-byte aligned)
  pair_t S[2][N];
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int at = entry_of<N>(i, lane);
      const float* p = mine + (size_t)c * dim + at;
      float2 v = make_float2(0.f, 0.f);
      if (col0 + c < vdim) {
        if (vec) { if (at < dim) v = *reinterpret_cast<const float2*>(p); }
        else {
          if (at < dim) v.x = p[0];
          if (at + 1 < dim) v.y = p[1];
        }
      }
      S[c][i] = make_pair2(v.x, v.y);
    }
  // Lane s writes (in the warp's first half) the read-out of column col0 + (s >> 3) of token s & 7 of every eight.
  const int out_col = col0 + ((lane >> 3) & 1);
  float* target = out + (size_t)begin * heads * vdim + (size_t)head * vdim + out_col;

  for (int c = 0; c < chunks; ++c) {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(kStages - 2));
    __syncthreads();                                    // chunk c is here; everybody is done with chunk c - 1
    if (c + kStages - 1 < chunks) stage(c + kStages - 1);
    asm volatile("cp.async.commit_group;\n" ::);
    const int n = min(CHUNK, end - begin - c * CHUNK);
    const float* tokens = staged + (c % kStages) * CHUNK * kPerToken;
#pragma unroll 1
    for (int g0 = 0; g0 < n; g0 += 8) {
      float p[16];
      const float* row = tokens + g0 * kPerToken;
      Entries<N, kScalar> part[2];
      fetch_entries<N, kScalar>(part[0], row, lane, warp);
      if (n - g0 >= 8) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          if (i < 7) fetch_entries<N, kScalar>(part[(i + 1) & 1], row + (i + 1) * kPerToken, lane, warp);
          memory_step<N, kScalar>(S, part[i & 1], p[i], p[i + 8]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          p[i] = p[i + 8] = 0.f;
          if (g0 + i < n) {
            if (i > 0) fetch_entries<N, kScalar>(part[0], row + i * kPerToken, lane, warp);
            memory_step<N, kScalar>(S, part[0], p[i], p[i + 8]);
          }
        }
      }
      // Sixteen sums over the warp: lane s ends with sum s & 15 of its half, then the halves meet.
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) {
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (i < o) {
            const float send = up ? p[i] : p[i + o], keep = up ? p[i + o] : p[i];
            p[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
          }
      }
      p[0] += __shfl_xor_sync(0xffffffffu, p[0], 16);
      const int tok = g0 + (lane & 7);
      if (lane < 16 && tok < n && out_col < vdim) target[(size_t)(c * CHUNK + tok) * heads * vdim] = p[0];
    }
  }
  grid_launch_dependents();
#pragma unroll
  for (int c = 0; c < 2; ++c) {
    if (col0 + c >= vdim) continue;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int at = entry_of<N>(i, lane);
      float* p = mine + (size_t)c * dim + at;
      float2 v;
      asm("mov.b64 {%0, %1}, %2;" : "=f"(v.x), "=f"(v.y) : "l"(S[c][i]));
      if (vec) { if (at < dim) *reinterpret_cast<float2*>(p) = v; }
      else {
        if (at < dim) p[0] = v.x;
        if (at + 1 < dim) p[1] = v.y;
      }
    }
  }
}

// ------------------------------------------------------------------------------------------ records
// State space.  conved [tokens, heads * vdim + 2 * groups * dim] = x | B | C; dt: column slice of the projection.
template <typename T>
__global__ void __launch_bounds__(256)
ssd_record_kernel(const T* __restrict__ conved, size_t conved_stride, const T* __restrict__ dt, size_t dt_stride,
                  const float* __restrict__ dt_bias, const float* __restrict__ a_log, float* __restrict__ group_records,
                  float* __restrict__ head_records, int heads, int groups, int dim, int dimp, int vdim, int vdimp) {
  grid_dependency_wait();
  const int t = blockIdx.x;
  const T* row = conved + (size_t)t * conved_stride;
  const T* dt_row = dt + (size_t)t * dt_stride;
  const int inner = heads * vdim, width = groups * dim;
  float4* group_out = reinterpret_cast<float4*>(group_records) + (size_t)t * groups * (dimp / 2);
  float4* head_out = reinterpret_cast<float4*>(head_records) + (size_t)t * heads * (vdimp / 4 + 1);
  const int group_items = groups * (dimp / 2), head_items = heads * (vdimp / 4 + 1);
  for (int i = threadIdx.x; i < group_items + head_items; i += blockDim.x) {
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (i < group_items) {
      const int g = i / (dimp / 2), c = (i - g * (dimp / 2)) * 4;
      const bool first = c < dimp;                       // C, then B
      const int e0 = first ? c : c - dimp;
      const T* src = row + inner + (first ? width : 0) + g * dim;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (e0 + e < dim) v[e] = widen(src[e0 + e]);
      group_out[i] = make_float4(v[0], v[1], v[2], v[3]);
    } else {
      const int j = i - group_items, h = j / (vdimp / 4 + 1), e0 = (j - h * (vdimp / 4 + 1)) * 4;
      const float step = softplus_of(widen(dt_row[h]) + dt_bias[h]);
      if (e0 == vdimp) v[0] = expf(-expf(a_log[h]) * step);
      else
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (e0 + e < vdim) v[e] = step * widen(row[h * vdim + e0 + e]);
      head_out[j] = make_float4(v[0], v[1], v[2], v[3]);
    }
  }
}

// Time mixing.  r, k, v [tokens, heads * dim] (rows row_stride apart), low [tokens, rank] the decay's inner product
// (before its tanh), w2t [rank, heads * dim] (transposed), w0, u [heads * dim].  A block: 16 tokens x a few heads.
constexpr int kRecordTokens = 16, kRecordThreads = 128;
template <typename T> __device__ __forceinline__ float2 two(const T* p);
template <> __device__ __forceinline__ float2 two<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 two<bf16>(const bf16* p) {
  const unsigned v = *reinterpret_cast<const unsigned*>(p);
  return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
}

// kPairs: two neighbouring channels a thread and access (dim even, rows aligned for it), else one.
template <typename T, bool kPairs>
__global__ void __launch_bounds__(kRecordThreads)
wkv_record_kernel(const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v, size_t row_stride,
                  const T* __restrict__ low, size_t low_stride, int rank, const T* __restrict__ w2t,
                  const float* __restrict__ w0, const float* __restrict__ u, float* __restrict__ group_records,
                  float* __restrict__ head_records, float* __restrict__ bonus, int tokens, int heads, int heads_per_block,
                  int dim, int dimp, int vdimp) {
  constexpr int C = kPairs ? 2 : 1;
  extern __shared__ __align__(16) float tanhs[];         // [rank][kRecordTokens]
  grid_dependency_wait();
  const int t0 = blockIdx.x * kRecordTokens, n = min(kRecordTokens, tokens - t0);
  const int h0 = blockIdx.y * heads_per_block, h1 = min(heads, h0 + heads_per_block);
  const int width = heads * dim, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < rank * kRecordTokens; i += kRecordThreads) {
    const int t = i / rank, c = i - t * rank;
    tanhs[c * kRecordTokens + t] = t < n ? tanhf(to_float(low[(size_t)(t0 + t) * low_stride + c])) : 0.f;
  }
  __syncthreads();
  for (int c = h0 * dim + threadIdx.x * C; c < h1 * dim; c += kRecordThreads * C) {
    float acc[C][kRecordTokens];
#pragma unroll
    for (int e = 0; e < C; ++e)
#pragma unroll
      for (int t = 0; t < kRecordTokens; ++t) acc[e][t] = 0.f;
#pragma unroll 8
    for (int i = 0; i < rank; ++i) {
      float w[2];
      if constexpr (kPairs) {
        const float2 p = two<T>(w2t + (size_t)i * width + c);
        w[0] = p.x; w[1] = p.y;
      } else {
        w[0] = widen(w2t[(size_t)i * width + c]);
      }
      const float4* th = reinterpret_cast<const float4*>(tanhs + i * kRecordTokens);
#pragma unroll
      for (int t = 0; t < kRecordTokens / 4; ++t) {
        const float4 x = th[t];
#pragma unroll
        for (int e = 0; e < C; ++e) {
          acc[e][4 * t] = fmaf(w[e], x.x, acc[e][4 * t]);
          acc[e][4 * t + 1] = fmaf(w[e], x.y, acc[e][4 * t + 1]);
          acc[e][4 * t + 2] = fmaf(w[e], x.z, acc[e][4 * t + 2]);
          acc[e][4 * t + 3] = fmaf(w[e], x.w, acc[e][4 * t + 3]);
        }
      }
    }
    const int h = c / dim, d = c - h * dim;              // (a pair lies within one head: dim is even)
    float* out = group_records + ((size_t)t0 * heads + h) * 3 * dimp + 2 * dimp + d;
    float base[2] = {w0[c], kPairs ? w0[c + C - 1] : 0.f};
#pragma unroll
    for (int t = 0; t < kRecordTokens; ++t)
      if (t < n) {
        float* o = out + (size_t)t * heads * 3 * dimp;
        if constexpr (kPairs)
          *reinterpret_cast<float2*>(o) = make_float2(expf(-expf(acc[0][t] + base[0])), expf(-expf(acc[C - 1][t] + base[1])));
        else
          o[0] = expf(-expf(acc[0][t] + base[0]));
      }
  }
  // r, k and v as floats, zeros in the places past dim, and the bonus r . (u k): a warp a (token, head).
#pragma unroll 4
  for (int item = warp; item < n * (h1 - h0); item += kRecordThreads / 32) {
    const int t = item / (h1 - h0), h = h0 + item - t * (h1 - h0);
    const size_t row = (size_t)(t0 + t) * row_stride + (size_t)h * dim, rec = (size_t)(t0 + t) * heads + h;
    float* group_out = group_records + rec * 3 * dimp;
    float* head_out = head_records + rec * vdimp;
    float sum = 0.f;
    for (int d = lane * C; d < dimp; d += 32 * C) {
      float rv[2] = {0.f, 0.f}, kv[2] = {0.f, 0.f}, vv[2] = {0.f, 0.f};
      if (d < dim) {
        if constexpr (kPairs) {
          const float2 a = two<T>(r + row + d), b = two<T>(k + row + d), c = two<T>(v + row + d);
          rv[0] = a.x; rv[1] = a.y; kv[0] = b.x; kv[1] = b.y; vv[0] = c.x; vv[1] = c.y;
        } else {
          rv[0] = widen(r[row + d]);
          kv[0] = widen(k[row + d]);
          vv[0] = widen(v[row + d]);
        }
#pragma unroll
        for (int e = 0; e < C; ++e) sum = fmaf(rv[e] * u[h * dim + d + e], kv[e], sum);
      }
      if constexpr (kPairs) {
        *reinterpret_cast<float2*>(group_out + d) = make_float2(rv[0], rv[1]);
        *reinterpret_cast<float2*>(group_out + dimp + d) = make_float2(kv[0], kv[1]);
        if (d >= dim) *reinterpret_cast<float2*>(group_out + 2 * dimp + d) = make_float2(0.f, 0.f);
        if (d < vdimp) *reinterpret_cast<float2*>(head_out + d) = make_float2(vv[0], vv[1]);
      } else {
        group_out[d] = rv[0];
        group_out[dimp + d] = kv[0];
        if (d >= dim) group_out[2 * dimp + d] = 0.f;
        if (d < vdimp) head_out[d] = vv[0];
      }
    }
    sum = warp_sum(sum);
    if (lane == 0) bonus[rec] = sum;
  }
}

// ------------------------------------------------------------------------------------------ single tokens
// The walk over the columns of one head's state that both token kernels do: S_j <- w S_j + k v_j entry by entry, the
// read-out before (kBefore) or behind that.  Every lane of a warp runs every round.
template <int NPL, bool kBefore, typename Read>
__device__ __forceinline__ void walk_columns(float* base, int dim, int vdim, const float* qs, const float* ks, const float* ws,
                                             float decay, const float* vs, float4 (&s)[NPL <= 8 ? 4 : (NPL == 16 ? 2 : 1)][NPL / 4],
                                             int sub, int group, Read read) {
  constexpr int kAhead = NPL <= 8 ? 4 : (NPL == 16 ? 2 : 1);     // columns of a group in flight
  const bool vec = dim % 4 == 0;
  for (int c0 = group; c0 - group < vdim; c0 += kRowGroups * kAhead) {
    if (c0 != group) {
#pragma unroll
      for (int a = 0; a < kAhead; ++a)
#pragma unroll
        for (int j = 0; j < NPL / 4; ++j) {
          const int at = 4 * (sub + 16 * j), column = c0 + kRowGroups * a;
          const float* p = base + (size_t)column * dim + at;
          float4& x = s[a][j];
          x = make_float4(0.f, 0.f, 0.f, 0.f);
          if (column >= vdim) continue;
          if (vec) { if (at < dim) x = *reinterpret_cast<const float4*>(p); }
          else {
            if (at < dim) x.x = p[0];
            if (at + 1 < dim) x.y = p[1];
            if (at + 2 < dim) x.z = p[2];
            if (at + 3 < dim) x.w = p[3];
          }
        }
    }
    float p[kAhead];
#pragma unroll
    for (int a = 0; a < kAhead; ++a) {
      const int column = c0 + kRowGroups * a;
      const float v = column < vdim ? vs[column] : 0.f;
      p[a] = 0.f;
#pragma unroll
      for (int j = 0; j < NPL / 4; ++j) {
        const int at = 4 * (sub + 16 * j);
        const float4 q = *reinterpret_cast<const float4*>(qs + at), k = *reinterpret_cast<const float4*>(ks + at);
        const float4 w = ws != nullptr ? *reinterpret_cast<const float4*>(ws + at) : make_float4(decay, decay, decay, decay);
        float4& x = s[a][j];
        if (kBefore) p[a] = fmaf(x.w, q.w, fmaf(x.z, q.z, fmaf(x.y, q.y, fmaf(x.x, q.x, p[a]))));
        x.x = fmaf(w.x, x.x, k.x * v);
        x.y = fmaf(w.y, x.y, k.y * v);
        x.z = fmaf(w.z, x.z, k.z * v);
        x.w = fmaf(w.w, x.w, k.w * v);
        if (!kBefore) p[a] = fmaf(x.w, q.w, fmaf(x.z, q.z, fmaf(x.y, q.y, fmaf(x.x, q.x, p[a]))));
        if (column < vdim) {
          float* dst = base + (size_t)column * dim + at;
          if (vec) { if (at < dim) *reinterpret_cast<float4*>(dst) = x; }
          else {
            if (at < dim) dst[0] = x.x;
            if (at + 1 < dim) dst[1] = x.y;
            if (at + 2 < dim) dst[2] = x.z;
            if (at + 3 < dim) dst[3] = x.w;
          }
        }
      }
    }
#pragma unroll
    for (int a = 0; a < kAhead; ++a) {
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) p[a] += __shfl_xor_sync(0xffffffffu, p[a], o);
      const int column = c0 + kRowGroups * a;
      if (sub == 0 && column < vdim) read(column, p[a]);
    }
  }
}

// The first columns of a walk, asked for while the token's inputs are made.
template <int NPL>
__device__ __forceinline__ void first_columns(const float* base, int dim, int vdim,
                                              float4 (&s)[NPL <= 8 ? 4 : (NPL == 16 ? 2 : 1)][NPL / 4], int sub, int group) {
  constexpr int kAhead = NPL <= 8 ? 4 : (NPL == 16 ? 2 : 1);
  const bool vec = dim % 4 == 0;
#pragma unroll
  for (int a = 0; a < kAhead; ++a)
#pragma unroll
    for (int j = 0; j < NPL / 4; ++j) {
      const int at = 4 * (sub + 16 * j), column = group + kRowGroups * a;
      const float* p = base + (size_t)column * dim + at;
      float4& x = s[a][j];
      x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (column >= vdim) continue;
      if (vec) { if (at < dim) x = *reinterpret_cast<const float4*>(p); }
      else {
        if (at < dim) x.x = p[0];
        if (at + 1 < dim) x.y = p[1];
        if (at + 2 < dim) x.z = p[2];
        if (at + 3 < dim) x.w = p[3];
      }
    }
}

// Every sequence brings one token (token row = query_start_loc[seq]) or none.  out [tokens, heads * vdim] float32 = S^T C.
template <typename T, int NPL>
__global__ void __launch_bounds__(256)
ssd_token_kernel(const T* __restrict__ conved, size_t conved_stride, const T* __restrict__ dt, size_t dt_stride,
                 const float* __restrict__ dt_bias, const float* __restrict__ a_log, float* __restrict__ state,
                 const int* __restrict__ query_start_loc, const int* __restrict__ state_slots, float* __restrict__ out,
                 int heads, int groups, int dim, int vdim) {
  extern __shared__ __align__(16) float shared[];       // C [dimp], B [dimp], dt x [vdim]
  constexpr int dimp = 16 * NPL;
  constexpr int kAhead = NPL <= 8 ? 4 : (NPL == 16 ? 2 : 1);
  const int head = blockIdx.x, seq = blockIdx.y;
  const int begin = query_start_loc[seq], end = query_start_loc[seq + 1];
  if (end <= begin) return;
  const int slot = state_slots[seq];
  if (slot < 0) return;
  float* qs = shared;
  float* ks = qs + dimp;
  float* vs = ks + dimp;
  const int lane = threadIdx.x & 31, sub = lane & 15, group = (threadIdx.x >> 5) * 2 + (lane >> 4);
  float* base = state + ((size_t)slot * heads + head) * (size_t)vdim * dim;
  grid_dependency_wait();
  float4 s[kAhead][NPL / 4];
  first_columns<NPL>(base, dim, vdim, s, sub, group);
  const T* row = conved + (size_t)begin * conved_stride;
  const T* b = row + heads * vdim + (head / (heads / groups)) * dim;
  const T* c = b + groups * dim;
  const float step = softplus_of(to_float(dt[(size_t)begin * dt_stride + head]) + dt_bias[head]);
  for (int i = threadIdx.x; i < dimp; i += 256) {
    qs[i] = i < dim ? to_float(c[i]) : 0.f;
    ks[i] = i < dim ? to_float(b[i]) : 0.f;
  }
  for (int i = threadIdx.x; i < vdim; i += 256) vs[i] = step * to_float(row[head * vdim + i]);
  __syncthreads();
  float* o = out + (size_t)begin * heads * vdim + (size_t)head * vdim;
  walk_columns<NPL, false>(base, dim, vdim, qs, ks, nullptr, expf(-expf(a_log[head]) * step), vs, s, sub, group,
                           [&](int column, float value) { o[column] = value; });
  grid_launch_dependents();
}

// Decay, recurrence, bonus, the norm of the head's read-out over its numbers, weight and gate:
// out[t, h] = o / sqrt(mean(o^2) + eps) * norm_weight * silu(g).
template <typename T, int NPL>
__global__ void __launch_bounds__(256)
wkv_token_kernel(const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v, const T* __restrict__ g,
                 size_t row_stride, const T* __restrict__ low, size_t low_stride, int rank, const T* __restrict__ w2,
                 const float* __restrict__ w0, const float* __restrict__ u, float* __restrict__ state,
                 const int* __restrict__ query_start_loc, const int* __restrict__ state_slots,
                 const float* __restrict__ norm_weight, float eps, T* __restrict__ out, size_t out_stride, int heads, int dim) {
  extern __shared__ __align__(16) float shared[];       // r, k, w [dimp each], v, o [dim each], tanh [rank]
  __shared__ float scratch[33];
  constexpr int dimp = 16 * NPL;
  constexpr int kAhead = NPL <= 8 ? 4 : (NPL == 16 ? 2 : 1);
  const int head = blockIdx.x, seq = blockIdx.y;
  const int begin = query_start_loc[seq], end = query_start_loc[seq + 1];
  if (end <= begin) return;
  const int slot = state_slots[seq];
  if (slot < 0) return;
  float* rs = shared;
  float* ks = rs + dimp;
  float* ws = ks + dimp;
  float* vs = ws + dimp;
  float* os = vs + dim;
  float* th = os + dim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane & 15, group = warp * 2 + (lane >> 4);
  float* base = state + ((size_t)slot * heads + head) * (size_t)dim * dim;
  // The decay's second product, a group of lanes a channel (channels group, group + 16, ...), four of the rank a lane: up to
  // a rank of 64 its weights are on their way to registers before the wait.
  constexpr bool kEarly = NPL <= 8;
  const bool early = kEarly && rank <= 64 && rank % 4 == 0 && reinterpret_cast<uintptr_t>(w2) % (4 * sizeof(T)) == 0;
  float wr[kEarly ? NPL : 1][4];
  if (early) {
#pragma unroll
    for (int i = 0; i < (kEarly ? NPL : 1); ++i) {
      const int d = i * kRowGroups + group;
      wr[i][0] = wr[i][1] = wr[i][2] = wr[i][3] = 0.f;
      if (d < dim && 4 * sub < rank) {
        const T* p = w2 + ((size_t)head * dim + d) * rank + 4 * sub;
        const float2 a = two<T>(p), b = two<T>(p + 2);
        wr[i][0] = a.x; wr[i][1] = a.y; wr[i][2] = b.x; wr[i][3] = b.y;
      }
    }
  }
  grid_dependency_wait();
  float4 s[kAhead][NPL / 4];
  first_columns<NPL>(base, dim, dim, s, sub, group);
  const size_t at = (size_t)begin * row_stride + (size_t)head * dim;
  for (int i = threadIdx.x; i < rank; i += 256) th[i] = tanhf(to_float(low[(size_t)begin * low_stride + i]));
  float mine = 0.f;
  for (int i = threadIdx.x; i < dimp; i += 256) {
    const bool live = i < dim;
    const float rv = live ? to_float(r[at + i]) : 0.f, kv = live ? to_float(k[at + i]) : 0.f;
    rs[i] = rv;
    ks[i] = kv;
    if (live) {
      vs[i] = to_float(v[at + i]);
      mine = fmaf(rv * u[head * dim + i], kv, mine);
    } else {
      ws[i] = 0.f;
    }
  }
  const float bonus = block_sum(mine, scratch);         // (its barriers also show the tanhs to everybody)
  auto finish = [&](int d, float z) {
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
    if (sub == 0 && d < dim) ws[d] = expf(-expf(z + w0[head * dim + d]));
  };
  if (early) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (4 * sub < rank) x = make_float4(th[4 * sub], th[4 * sub + 1], th[4 * sub + 2], th[4 * sub + 3]);
#pragma unroll
    for (int i = 0; i < (kEarly ? NPL : 1); ++i)
      finish(i * kRowGroups + group, fmaf(wr[i][3], x.w, fmaf(wr[i][2], x.z, fmaf(wr[i][1], x.y, wr[i][0] * x.x))));
  }
  for (int d0 = early ? dim : 0; d0 < dim; d0 += kRowGroups) {
    const int d = d0 + group;
    float z = 0.f;
    if (d < dim)
      for (int i = sub; i < rank; i += 16) z = fmaf(to_float(w2[((size_t)head * dim + d) * rank + i]), th[i], z);
    finish(d, z);
  }
  __syncthreads();
  walk_columns<NPL, true>(base, dim, dim, rs, ks, ws, 0.f, vs, s, sub, group,
                          [&](int column, float value) { os[column] = fmaf(bonus, vs[column], value); });
  grid_launch_dependents();
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < dim; i += 256) ss = fmaf(os[i], os[i], ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)dim + eps);
  T* o = out + (size_t)begin * out_stride + (size_t)head * dim;
  for (int i = threadIdx.x; i < dim; i += 256) {
    const float gate = to_float(g[at + i]);
    o[i] = from_float<T>(os[i] * inv * norm_weight[head * dim + i] * (gate / (1.0f + expf(-gate))));
  }
}

// ------------------------------------------------------------------------------------------ token shift
// x [tokens, width]; mu [count, width]; out [count][tokens, width]; before [slots, width]: each request's last token so
// far.  move: every sequence brings one token, and the thread that has read `before` for its columns writes it on.
template <typename T, int E>
__global__ void token_shift_kernel(const T* __restrict__ x, const float* __restrict__ mu, int count, T* before,
                                   const int* __restrict__ seq_of_token, const int* __restrict__ query_start_loc,
                                   const int* __restrict__ state_slots, T* __restrict__ out, int tokens, int width, int move) {
  const int t = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * E;
  if (c >= width) return;
  grid_dependency_wait();
  const int seq = seq_of_token[t];
  float now[E], diff[E];
#pragma unroll
  for (int e = 0; e < E; ++e) now[e] = diff[e] = 0.f;
  if (seq >= 0) {
    const T* mine = x + (size_t)t * width + c;
    T* kept = before + (size_t)state_slots[seq] * width + c;
    const T* last = t > query_start_loc[seq] ? mine - width : kept;
    if (E > 1) {
      const Vec16<T> a = load16(mine), b = load16(last);
      float f[Vec16<T>::N];
      unpack16(a, f);
#pragma unroll
      for (int e = 0; e < E; ++e) now[e] = f[e];
      unpack16(b, f);
#pragma unroll
      for (int e = 0; e < E; ++e) diff[e] = f[e] - now[e];
      if (move) store16(kept, a);
    } else {
      now[0] = to_float(mine[0]);
      diff[0] = to_float(last[0]) - now[0];
      if (move) kept[0] = mine[0];
    }
  }
  for (int i = 0; i < count; ++i) {
    const float* m = mu + (size_t)i * width + c;
    T* o = out + ((size_t)i * tokens + t) * width + c;
    if (E > 1) {
      Vec16<T> v;
#pragma unroll
      for (int e = 0; e < E; e += 4) {
        const float4 w = *reinterpret_cast<const float4*>(m + e);
        v.set(e, fmaf(diff[e], w.x, now[e]));
        v.set(e + 1, fmaf(diff[e + 1], w.y, now[e + 1]));
        v.set(e + 2, fmaf(diff[e + 2], w.z, now[e + 2]));
        v.set(e + 3, fmaf(diff[e + 3], w.w, now[e + 3]));
      }
      store16(o, v);
    } else {
      o[0] = from_float<T>(fmaf(diff[0], m[0], now[0]));
    }
  }
}

template <int N, int CHUNK, bool kScalar>
int launch_memory(int tokens, int num_seqs, cudaStream_t stream, const float* group_records, const float* head_records,
                  float* state, const int* qsl, const int* slots, float* out, int heads, int groups, int dim, int vdim,
                  int vdimp) {
  constexpr size_t per_token = (kScalar ? 2 : 3) * 64 * N + kColumns + (kScalar ? 4 : 0);
  constexpr size_t smem = (size_t)kStages * CHUNK * per_token * sizeof(float);
  static bool configured = false;
  if (!configured && smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(memory_steps_kernel<N, CHUNK, kScalar>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(tokens, memory_steps_kernel<N, CHUNK, kScalar>, dim3(vdimp / kColumns, heads, num_seqs),
                         dim3(kStepThreads), smem, stream, group_records, head_records, state, qsl, slots, out, heads, groups,
                         dim, vdim, vdimp);
}

}  // namespace li

using namespace li;

static int rounded_dim(int dim) { return dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 512; }
static int rounded_columns(int vdim) { return (vdim + kColumns - 1) / kColumns * kColumns; }
static bool refused(int num_seqs, int heads, int groups, int dim, int vdim, const void* state) {
  return heads < 1 || heads > 65535 || groups < 1 || heads % groups || num_seqs > 65535 || dim < 1 || dim > 512 || vdim < 1 ||
         vdim > 4096 || !aligned16(state);
}

// Floats of a token's records: of one group and of one head (scalar: the state space; else time mixing).
LI_EXPORT int li_memory_record_floats(int scalar, int dim, int vdim, int* head_floats) {
  *head_floats = rounded_columns(vdim) + (scalar ? 4 : 0);
  return (scalar ? 2 : 3) * rounded_dim(dim);
}

// conved [tokens, conved_stride]: x (heads x vdim), B, C (groups x dim each) side by side; dt [tokens, dt_stride] (heads).
// records: scratch, 16-byte aligned.  state [slots, heads, vdim, dim] float32 is read and written; out [tokens, heads *
// vdim] float32.
LI_EXPORT int li_ssd_steps(int dtype, const void* conved, size_t conved_stride, const void* dt, size_t dt_stride,
                           const float* dt_bias, const float* a_log, float* group_records, float* head_records, float* state,
                           const int* query_start_loc, const int* state_slots, int tokens, int num_seqs, float* out,
                           int heads, int groups, int dim, int vdim, cudaStream_t stream) {
  if (tokens <= 0 || num_seqs <= 0) return 0;
  if (refused(num_seqs, heads, groups, dim, vdim, state) || !aligned16(group_records) || !aligned16(head_records))
    return LI_ERR_UNSUPPORTED;
  const int dimp = rounded_dim(dim), vdimp = rounded_columns(vdim);
  cudaError_t e;
  if (dtype == kFloat32)
    e = launch_pdl(tokens, ssd_record_kernel<float>, dim3(tokens), dim3(256), 0, stream, (const float*)conved, conved_stride,
                   (const float*)dt, dt_stride, dt_bias, a_log, group_records, head_records, heads, groups, dim, dimp, vdim, vdimp);
  else
    e = launch_pdl(tokens, ssd_record_kernel<bf16>, dim3(tokens), dim3(256), 0, stream, (const bf16*)conved, conved_stride,
                   (const bf16*)dt, dt_stride, dt_bias, a_log, group_records, head_records, heads, groups, dim, dimp, vdim, vdimp);
  if (e != cudaSuccess) return (int)e;
#define LI_STEPS(N, CHUNK)                                                                                            \
  return launch_memory<N, CHUNK, true>(tokens, num_seqs, stream, group_records, head_records, state, query_start_loc, \
                                       state_slots, out, heads, groups, dim, vdim, vdimp)
  if (dimp == 64) LI_STEPS(1, 16);
  if (dimp == 128) LI_STEPS(2, 16);
  if (dimp == 256) LI_STEPS(4, 8);
  LI_STEPS(8, 8);
#undef LI_STEPS
}

LI_EXPORT int li_ssd_token(int dtype, const void* conved, size_t conved_stride, const void* dt, size_t dt_stride,
                           const float* dt_bias, const float* a_log, float* state, const int* query_start_loc,
                           const int* state_slots, int num_seqs, float* out, int heads, int groups, int dim, int vdim,
                           cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (refused(num_seqs, heads, groups, dim, vdim, state)) return LI_ERR_UNSUPPORTED;
  const int dimp = rounded_dim(dim);
  const size_t smem = (size_t)(2 * dimp + vdim) * sizeof(float);
#define LI_TOKEN(T, NPL)                                                                                              \
  return (int)launch_pdl(num_seqs, ssd_token_kernel<T, NPL>, dim3(heads, num_seqs), dim3(256), smem, stream,          \
                         (const T*)conved, conved_stride, (const T*)dt, dt_stride, dt_bias, a_log, state,             \
                         query_start_loc, state_slots, out, heads, groups, dim, vdim)
#define LI_TOKEN_T(T)                                                                                                 \
  {                                                                                                                   \
    if (dimp == 64) LI_TOKEN(T, 4);                                                                                   \
    if (dimp == 128) LI_TOKEN(T, 8);                                                                                  \
    if (dimp == 256) LI_TOKEN(T, 16);                                                                                 \
    LI_TOKEN(T, 32);                                                                                                  \
  }
  if (dtype == kFloat32) LI_TOKEN_T(float)
  LI_TOKEN_T(bf16)
#undef LI_TOKEN_T
#undef LI_TOKEN
}

// r, k, v [tokens, heads * dim] (rows row_stride apart); low [tokens, low_stride] (rank numbers: the decay's inner product
// before its tanh); w2t [rank, heads * dim] in the engine's type; w0, u [heads * dim] float32.  bonus [tokens, heads] float32
// receives r . (u k).  out [tokens, heads * dim] float32 = S^T r (S before the token's own update).
LI_EXPORT int li_wkv_steps(int dtype, const void* r, const void* k, const void* v, size_t row_stride, const void* low,
                           size_t low_stride, int rank, const void* w2t, const float* w0, const float* u,
                           float* group_records, float* head_records, float* bonus, float* state,
                           const int* query_start_loc, const int* state_slots, int tokens, int num_seqs, float* out,
                           int heads, int dim, cudaStream_t stream) {
  if (tokens <= 0 || num_seqs <= 0) return 0;
  if (refused(num_seqs, heads, heads, dim, dim, state) || rank < 1 || rank > 512 || !aligned16(group_records) ||
      !aligned16(head_records))
    return LI_ERR_UNSUPPORTED;
  const int dimp = rounded_dim(dim), vdimp = rounded_columns(dim);
  const int per_block = dim >= 256 ? 1 : 256 / dim;
  const dim3 grid((tokens + kRecordTokens - 1) / kRecordTokens, (heads + per_block - 1) / per_block);
  const size_t smem = (size_t)rank * kRecordTokens * sizeof(float), pair = dtype == kFloat32 ? 8 : 4;
  const bool pairs = dim % 2 == 0 && row_stride % 2 == 0 && (uintptr_t)r % pair == 0 && (uintptr_t)k % pair == 0 &&
                     (uintptr_t)v % pair == 0 && (uintptr_t)w2t % pair == 0;
  cudaError_t e;
#define LI_RECORD(T, P)                                                                                               \
  e = launch_pdl(tokens, wkv_record_kernel<T, P>, grid, dim3(kRecordThreads), smem, stream, (const T*)r, (const T*)k, \
                 (const T*)v, row_stride, (const T*)low, low_stride, rank, (const T*)w2t, w0, u, group_records,       \
                 head_records, bonus, tokens, heads, per_block, dim, dimp, vdimp)
  if (dtype == kFloat32) { if (pairs) LI_RECORD(float, true); else LI_RECORD(float, false); }
  else if (pairs) LI_RECORD(bf16, true);
  else LI_RECORD(bf16, false);
#undef LI_RECORD
  if (e != cudaSuccess) return (int)e;
#define LI_STEPS(N, CHUNK)                                                                                            \
  return launch_memory<N, CHUNK, false>(tokens, num_seqs, stream, group_records, head_records, state, query_start_loc, \
                                        state_slots, out, heads, heads, dim, dim, vdimp)
  if (dimp == 64) LI_STEPS(1, 16);
  if (dimp == 128) LI_STEPS(2, 16);
  if (dimp == 256) LI_STEPS(4, 8);
  LI_STEPS(8, 8);
#undef LI_STEPS
}

// The same for steps in which every sequence brings one token (or none), up to the normed and gated read-out: out [tokens,
// out_stride] in the engine's type.  w2 [heads * dim, rank] (as stored); norm_weight [heads * dim] float32.
LI_EXPORT int li_wkv_token(int dtype, const void* r, const void* k, const void* v, const void* g, size_t row_stride,
                           const void* low, size_t low_stride, int rank, const void* w2, const float* w0, const float* u,
                           float* state, const int* query_start_loc, const int* state_slots, int num_seqs,
                           const float* norm_weight, float eps, void* out, size_t out_stride, int heads, int dim,
                           cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (refused(num_seqs, heads, heads, dim, dim, state) || rank < 1 || rank > 512) return LI_ERR_UNSUPPORTED;
  const int dimp = rounded_dim(dim);
  const size_t smem = (size_t)(3 * dimp + 2 * dim + rank) * sizeof(float);
#define LI_TOKEN(T, NPL)                                                                                              \
  return (int)launch_pdl(num_seqs, wkv_token_kernel<T, NPL>, dim3(heads, num_seqs), dim3(256), smem, stream,          \
                         (const T*)r, (const T*)k, (const T*)v, (const T*)g, row_stride, (const T*)low, low_stride,   \
                         rank, (const T*)w2, w0, u, state, query_start_loc, state_slots, norm_weight, eps, (T*)out,   \
                         out_stride, heads, dim)
#define LI_TOKEN_T(T)                                                                                                 \
  {                                                                                                                   \
    if (dimp == 64) LI_TOKEN(T, 4);                                                                                   \
    if (dimp == 128) LI_TOKEN(T, 8);                                                                                  \
    if (dimp == 256) LI_TOKEN(T, 16);                                                                                 \
    LI_TOKEN(T, 32);                                                                                                  \
  }
  if (dtype == kFloat32) LI_TOKEN_T(float)
  LI_TOKEN_T(bf16)
#undef LI_TOKEN_T
#undef LI_TOKEN
}

// x [tokens, width] contiguous; mu [count, width] float32; before [slots, width] in the engine's type; out [count, tokens,
// width].  move: every sequence brings one token, and `before` becomes it in the same launch.
LI_EXPORT int li_token_shift(int dtype, const void* x, const float* mu, int count, void* before, const int* seq_of_token,
                             const int* query_start_loc, const int* state_slots, void* out, int tokens, int width, int move,
                             cudaStream_t stream) {
  if (tokens <= 0 || count <= 0) return 0;
  if (width < 1) return LI_ERR_UNSUPPORTED;
  const int n = dtype == kFloat32 ? 4 : 8;
  const bool vec = width % n == 0 && aligned16(x) && aligned16(mu) && aligned16(before) && aligned16(out);
  const int per_row = vec ? width / n : width;
  const int block = per_row >= 256 ? 256 : (per_row + 31) / 32 * 32;
  const dim3 grid(tokens, (per_row + block - 1) / block);
  if (grid.y > 65535) return LI_ERR_UNSUPPORTED;
#define LI_SHIFT(T, E)                                                                                                \
  return (int)launch_pdl(tokens, token_shift_kernel<T, E>, grid, dim3(block), 0, stream, (const T*)x, mu, count,      \
                         (T*)before, seq_of_token, query_start_loc, state_slots, (T*)out, tokens, width, move)
  if (dtype == kFloat32) { if (vec) LI_SHIFT(float, 4); LI_SHIFT(float, 1); }
  if (vec) LI_SHIFT(bf16, 8);
  LI_SHIFT(bf16, 1);
#undef LI_SHIFT
}
