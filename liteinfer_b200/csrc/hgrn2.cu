// The memory of an HGRN2 layer: linear attention whose forget gate also decides what is written.  Per request and head a
// state S [dim, vdim] in 32-bit; per token, with raw projections z_q, z_f of the head (dim numbers each) and v (vdim):
//
//   q = silu(z_q);  f = l + (1 - l) sigmoid(z_f + b)            # b and the lower bound l: one number a channel
//   S <- diag(f) S + (1 - f) v^T;  o = S^T q
//
//   li_hgrn2_steps   steps in which some sequence brings several tokens.  Two kernels: the first turns q, f and v of
//                    every token and head into a record of floats (dim and vdim rounded up, the places past dim zero),
//                    so that the second only copies; the second runs the recurrence and writes o as float32.
//   li_hgrn2_token   steps of single tokens, in one kernel: gates, recurrence, and behind them the root-mean-square norm
//                    of each head's o over vdim with its weight, rounded to the engine's type.  (After the other entry
//                    li_gated_rmsnorm does that norm.)
//
// The state is kept column by column, state[slot][head][vdim][dim]: a column is a chain of its own over the tokens,
// S_j <- f S_j + (1 - f) v_j entry by entry (a gate of exactly 1 leaves the entry as it is).  In the first form a block
// takes 16 columns of one head of one sequence; a warp takes two of them, each lane with dim / 32 of their entries in
// registers for the whole step, so an entry of q and f read from shared memory serves two columns.  The records come in
// chunks of up to 16 tokens by cp.async, three chunks deep, one block barrier a chunk, and a lane has the next token's
// entries on their way to its registers while it works on this one's.  A token's update of S needs nothing of its
// read-out, so the lanes keep their parts of eight tokens' read-outs of both columns and add them up together: sixteen
// shuffles for sixteen sums, and every sum is the same tree whatever the token's place in a step.  In the second form a
// block takes one head of one sequence and walks its columns, sixteen lanes a column and several columns in flight, since
// there the state's bytes are all the work.
// Sequences that bring no token touch nothing.
#include "common.cuh"

namespace li {

constexpr int kColumns = 16;        // of a block of the first form: eight warps x two columns
constexpr int kStepThreads = 256;
constexpr int kStages = 3;
constexpr int kRowGroups = 16;      // of a block of the second form: eight warps x two groups of lanes

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

__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float forget_of(float z, float bias, float lower) {
  return lower + (1.0f - lower) * sigmoid_of(z + bias);
}

__device__ __forceinline__ void copy16(float* smem, const float* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem));
}

// A lane's entries of one token: N pairs each of q and f, and the token's values of the lane's two columns.
template <int N>
struct TokenPart {
  pair_t q[N], f[N];
  float2 v;
};

// row: the token's q [32 * 2N], f [32 * 2N], values.  Pairs of a lane lie side by side in fours of floats where N allows.
template <int N>
__device__ __forceinline__ void fetch_part(TokenPart<N>& t, const float* __restrict__ row, int lane, int warp) {
  constexpr int dimp = 64 * N;
  if (N == 1) {
    t.q[0] = *reinterpret_cast<const pair_t*>(row + 2 * lane);
    t.f[0] = *reinterpret_cast<const pair_t*>(row + dimp + 2 * lane);
  } else {
#pragma unroll
    for (int j = 0; j < N / 2; ++j) {
      const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(row + 4 * (lane + 32 * j));
      const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(row + dimp + 4 * (lane + 32 * j));
      t.q[2 * j] = q.x; t.q[2 * j + 1] = q.y;
      t.f[2 * j] = f.x; t.f[2 * j + 1] = f.y;
    }
  }
  t.v = *reinterpret_cast<const float2*>(row + 2 * dimp + 2 * warp);
}

// The entry that the first half of pair `i` of a lane is.
template <int N> __device__ __forceinline__ int entry_of(int i, int lane) {
  return N == 1 ? 2 * lane : 4 * (lane + 32 * (i >> 1)) + 2 * (i & 1);
}

// One token on a lane's part of two columns: S <- f S + (1 - f) v, and the lane's parts of the columns' read-outs.
template <int N>
__device__ __forceinline__ void hgrn2_step(pair_t (&S)[2][N], const TokenPart<N>& t, float& read0, float& read1) {
  const pair_t v0 = make_pair2(t.v.x, t.v.x), v1 = make_pair2(t.v.y, t.v.y);
  const pair_t one = make_pair2(1.f, 1.f), minus = make_pair2(-1.f, -1.f);
  pair_t a0, a1;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const pair_t g = fma2(t.f[i], minus, one);
    S[0][i] = fma2(t.f[i], S[0][i], mul2(g, v0));
    S[1][i] = fma2(t.f[i], S[1][i], mul2(g, v1));
    a0 = i == 0 ? mul2(S[0][i], t.q[i]) : fma2(S[0][i], t.q[i], a0);
    a1 = i == 0 ? mul2(S[1][i], t.q[i]) : fma2(S[1][i], t.q[i], a1);
  }
  read0 = sum2(a0);
  read1 = sum2(a1);
}

// ------------------------------------------------------------------------------------------ records
// record[token][head]: q [dimp] | f [dimp] | v [vdimp].  A block per token; a thread four neighbouring numbers.
template <typename T>
__global__ void __launch_bounds__(256)
hgrn2_record_kernel(const T* __restrict__ proj, size_t row_stride, int q_off, int f_off, int v_off,
                    const float* __restrict__ f_bias, const float* __restrict__ lower, float* __restrict__ records,
                    int heads, int dim, int dimp, int vdim, int vdimp, int vec) {
  grid_dependency_wait();
  const int t = blockIdx.x;
  const T* row = proj + (size_t)t * row_stride;
  const int per_head = (2 * dimp + vdimp) >> 2;
  float4* out = reinterpret_cast<float4*>(records) + (size_t)t * heads * per_head;
  for (int i = threadIdx.x; i < heads * per_head; i += blockDim.x) {
    const int h = i / per_head, c = (i - h * per_head) << 2;
    const int kind = c < dimp ? 0 : c < 2 * dimp ? 1 : 2;
    const int e0 = c - kind * dimp, n = kind == 2 ? vdim : dim;
    const int at = (kind == 0 ? q_off : kind == 1 ? f_off : v_off) + h * n + e0;
    float x[4];
    if (vec && e0 + 4 <= n) {
      if (sizeof(T) == 4) {
        const float4 v = *reinterpret_cast<const float4*>(row + at);
        x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
      } else {
        const uint2 v = *reinterpret_cast<const uint2*>(row + at);
        x[0] = __uint_as_float(v.x << 16); x[1] = __uint_as_float(v.x & 0xffff0000u);
        x[2] = __uint_as_float(v.y << 16); x[3] = __uint_as_float(v.y & 0xffff0000u);
      }
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] = e0 + e < n ? to_float(row[at + e]) : 0.f;
    }
    if (kind < 2) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (e0 + e >= n) x[e] = 0.f;
        else if (kind == 0) x[e] = x[e] * sigmoid_of(x[e]);
        else x[e] = forget_of(x[e], f_bias[h * dim + e0 + e], lower[h * dim + e0 + e]);
      }
    }
    out[i] = make_float4(x[0], x[1], x[2], x[3]);
  }
}

// ----------------------------------------------------------------------------------------- several tokens
// N: pairs of entries of a column that a lane keeps; dimp = 64 N.
template <int N, int CHUNK>
__global__ void __launch_bounds__(kStepThreads)
hgrn2_steps_kernel(const float* __restrict__ records, float* __restrict__ state, const int* __restrict__ query_start_loc,
                   const int* __restrict__ state_slots, float* __restrict__ out, int heads, int dim, int vdim, int vdimp) {
  extern __shared__ __align__(16) float shared[];       // kStages x CHUNK x (q [dimp], f [dimp], v [kColumns])
  constexpr int dimp = 64 * N;
  constexpr int kPerToken = 2 * dimp + kColumns;
  constexpr int kCopies = kPerToken / 4;                // 16-byte copies of a token
  const int seq = blockIdx.z, head = blockIdx.y, first_column = blockIdx.x * kColumns;
  const int begin = query_start_loc[seq], end = query_start_loc[seq + 1];
  if (end <= begin) return;
  const int slot = state_slots[seq];
  if (slot < 0) return;
  const int chunks = (end - begin + CHUNK - 1) / CHUNK;
  const size_t record = 2 * dimp + vdimp;
  const float* source = records + ((size_t)begin * heads + head) * record;

  auto stage = [&](int c) {
    float* dst = shared + (c % kStages) * CHUNK * kPerToken;
    const int n = min(CHUNK, end - begin - c * CHUNK) * kCopies;
    for (int i = threadIdx.x; i < n; i += kStepThreads) {
      const int tok = i / kCopies, e = (i - tok * kCopies) * 4;
      const float* src = source + (size_t)(c * CHUNK + tok) * heads * record;
      copy16(dst + tok * kPerToken + e, src + (e < 2 * dimp ? e : e + first_column));
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
    const float* tokens = shared + (c % kStages) * CHUNK * kPerToken;
#pragma unroll 1
    for (int g0 = 0; g0 < n; g0 += 8) {
      float p[16];
      const float* row = tokens + g0 * kPerToken;
      TokenPart<N> part[2];
      fetch_part<N>(part[0], row, lane, warp);
      if (n - g0 >= 8) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          if (i < 7) fetch_part<N>(part[(i + 1) & 1], row + (i + 1) * kPerToken, lane, warp);
          hgrn2_step<N>(S, part[i & 1], p[i], p[i + 8]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          p[i] = p[i + 8] = 0.f;
          if (g0 + i < n) {
            if (i > 0) fetch_part<N>(part[0], row + i * kPerToken, lane, warp);
            hgrn2_step<N>(S, part[0], p[i], p[i + 8]);
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

// ------------------------------------------------------------------------------------------ single tokens
// Every sequence brings one token (token row = query_start_loc[seq]) or none.
template <typename T, int NPL>
__global__ void __launch_bounds__(256)
hgrn2_token_kernel(const T* __restrict__ proj, size_t row_stride, int q_off, int f_off, int v_off,
                   const float* __restrict__ f_bias, const float* __restrict__ lower, float* __restrict__ state,
                   const int* __restrict__ query_start_loc, const int* __restrict__ state_slots,
                   const float* __restrict__ norm_weight, float eps, T* __restrict__ out, size_t out_stride, int heads,
                   int dim, int vdim) {
  extern __shared__ __align__(16) float shared[];       // q [dimp], f [dimp], v [vdim], o [vdim]
  __shared__ float scratch[33];
  constexpr int dimp = 16 * NPL;
  constexpr int kAhead = NPL <= 8 ? 4 : (NPL == 16 ? 2 : 1);     // columns of a group in flight
  const int head = blockIdx.x, seq = blockIdx.y;
  const int begin = query_start_loc[seq], end = query_start_loc[seq + 1];
  if (end <= begin) return;
  const int slot = state_slots[seq];
  if (slot < 0) return;
  float* qs = shared;
  float* fs = qs + dimp;
  float* vs = fs + dimp;
  float* os = vs + vdim;
  grid_dependency_wait();
  const T* row = proj + (size_t)begin * row_stride;
  const int lane = threadIdx.x & 31, sub = lane & 15, group = (threadIdx.x >> 5) * 2 + (lane >> 4);
  float* base = state + ((size_t)slot * heads + head) * (size_t)vdim * dim;
  const bool vec = dim % 4 == 0;
  auto fetch = [&](int column, float4 (&s)[NPL / 4]) {
#pragma unroll
    for (int j = 0; j < NPL / 4; ++j) {
      const int at = 4 * (sub + 16 * j);
      const float* p = base + (size_t)column * dim + at;
      s[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (column >= vdim) continue;
      if (vec) { if (at < dim) s[j] = *reinterpret_cast<const float4*>(p); }
      else {
        if (at < dim) s[j].x = p[0];
        if (at + 1 < dim) s[j].y = p[1];
        if (at + 2 < dim) s[j].z = p[2];
        if (at + 3 < dim) s[j].w = p[3];
      }
    }
  };
  float4 s[kAhead][NPL / 4];
#pragma unroll
  for (int a = 0; a < kAhead; ++a) fetch(group + kRowGroups * a, s[a]);      // on their way while the gates are made
  for (int i = threadIdx.x; i < dimp; i += 256) {
    float q = 0.f, f = 0.f;
    if (i < dim) {
      q = to_float(row[q_off + head * dim + i]);
      q = q * sigmoid_of(q);
      f = forget_of(to_float(row[f_off + head * dim + i]), f_bias[head * dim + i], lower[head * dim + i]);
    }
    qs[i] = q;
    fs[i] = f;
  }
  for (int i = threadIdx.x; i < vdim; i += 256) vs[i] = to_float(row[v_off + head * vdim + i]);
  __syncthreads();
  for (int c0 = group; c0 - group < vdim; c0 += kRowGroups * kAhead) {       // every lane of a warp runs every round
    if (c0 != group) {
#pragma unroll
      for (int a = 0; a < kAhead; ++a) fetch(c0 + kRowGroups * a, s[a]);
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
        const float4 q = *reinterpret_cast<const float4*>(qs + at), f = *reinterpret_cast<const float4*>(fs + at);
        float4& x = s[a][j];
        x.x = fmaf(f.x, x.x, (1.0f - f.x) * v);
        x.y = fmaf(f.y, x.y, (1.0f - f.y) * v);
        x.z = fmaf(f.z, x.z, (1.0f - f.z) * v);
        x.w = fmaf(f.w, x.w, (1.0f - f.w) * v);
        p[a] = fmaf(x.w, q.w, fmaf(x.z, q.z, fmaf(x.y, q.y, fmaf(x.x, q.x, p[a]))));
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
      if (sub == 0 && column < vdim) os[column] = p[a];
    }
  }
  grid_launch_dependents();
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < vdim; i += 256) ss = fmaf(os[i], os[i], ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)vdim + eps);
  T* o = out + (size_t)begin * out_stride + (size_t)head * vdim;
  for (int i = threadIdx.x; i < vdim; i += 256) o[i] = from_float<T>(os[i] * inv * norm_weight[i]);
}

template <int N, int CHUNK>
int launch_steps(int tokens, int num_seqs, cudaStream_t stream, const float* records, float* state, const int* qsl,
                 const int* slots, float* out, int heads, int dim, int vdim, int vdimp) {
  constexpr size_t smem = (size_t)kStages * CHUNK * (128 * N + kColumns) * sizeof(float);
  static bool configured = false;
  if (!configured && smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(hgrn2_steps_kernel<N, CHUNK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(tokens, hgrn2_steps_kernel<N, CHUNK>, dim3(vdimp / kColumns, heads, num_seqs), dim3(kStepThreads),
                         smem, stream, records, state, qsl, slots, out, heads, dim, vdim, vdimp);
}

}  // namespace li

using namespace li;

static int rounded_dim(int dim) { return dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 512; }
static bool refused(int num_seqs, int heads, int dim, int vdim, const void* state) {
  return heads < 1 || heads > 65535 || num_seqs > 65535 || dim < 1 || dim > 512 || vdim < 1 || vdim > 4096 || !aligned16(state);
}

// Floats of a record of one token and head.
LI_EXPORT int li_hgrn2_record_floats(int dim, int vdim) {
  return 2 * rounded_dim(dim) + (vdim + kColumns - 1) / kColumns * kColumns;
}

// proj [tokens, row_stride]: q at column q_off and f at f_off (heads x dim), v at v_off (heads x vdim).  f_bias, lower
// [heads * dim] float32.  records: scratch of tokens * heads * li_hgrn2_record_floats floats, 16-byte aligned.  state
// [slots, heads, vdim, dim] float32 is read and written; out [tokens, heads * vdim] float32.
LI_EXPORT int li_hgrn2_steps(int dtype, const void* proj, size_t row_stride, int q_off, int f_off, int v_off,
                             const float* f_bias, const float* lower, float* records, float* state,
                             const int* query_start_loc, const int* state_slots, int tokens, int num_seqs, float* out,
                             int heads, int dim, int vdim, cudaStream_t stream) {
  if (tokens <= 0 || num_seqs <= 0) return 0;
  if (refused(num_seqs, heads, dim, vdim, state) || !aligned16(records)) return LI_ERR_UNSUPPORTED;
  const int dimp = rounded_dim(dim), vdimp = (vdim + kColumns - 1) / kColumns * kColumns;
  const int vec = dim % 4 == 0 && vdim % 4 == 0 && row_stride % 4 == 0 && q_off % 4 == 0 && f_off % 4 == 0 &&
                  v_off % 4 == 0 && reinterpret_cast<uintptr_t>(proj) % (dtype == kFloat32 ? 16 : 8) == 0;
  cudaError_t e;
  if (dtype == kFloat32)
    e = launch_pdl(tokens, hgrn2_record_kernel<float>, dim3(tokens), dim3(256), 0, stream, (const float*)proj, row_stride,
                   q_off, f_off, v_off, f_bias, lower, records, heads, dim, dimp, vdim, vdimp, vec);
  else
    e = launch_pdl(tokens, hgrn2_record_kernel<bf16>, dim3(tokens), dim3(256), 0, stream, (const bf16*)proj, row_stride,
                   q_off, f_off, v_off, f_bias, lower, records, heads, dim, dimp, vdim, vdimp, vec);
  if (e != cudaSuccess) return (int)e;
#define LI_STEPS(N, CHUNK)                                                                                            \
  return launch_steps<N, CHUNK>(tokens, num_seqs, stream, records, state, query_start_loc, state_slots, out, heads, dim, \
                                  vdim, vdimp)
  if (dimp == 64) LI_STEPS(1, 16);
  if (dimp == 128) LI_STEPS(2, 16);
  if (dimp == 256) LI_STEPS(4, 8);
  LI_STEPS(8, 8);
#undef LI_STEPS
}

// Steps in which every sequence brings one token (or none): everything up to the normed read-out, out [tokens, out_stride]
// in the engine's type with head h at column h * vdim.  norm_weight [vdim] float32.
LI_EXPORT int li_hgrn2_token(int dtype, const void* proj, size_t row_stride, int q_off, int f_off, int v_off,
                             const float* f_bias, const float* lower, float* state, const int* query_start_loc,
                             const int* state_slots, int num_seqs, const float* norm_weight, float eps, void* out,
                             size_t out_stride, int heads, int dim, int vdim, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (refused(num_seqs, heads, dim, vdim, state)) return LI_ERR_UNSUPPORTED;
  const int dimp = rounded_dim(dim);
  const size_t smem = (size_t)(2 * dimp + 2 * vdim) * sizeof(float);
#define LI_TOKEN(T, NPL)                                                                                              \
  return (int)launch_pdl(num_seqs, hgrn2_token_kernel<T, NPL>, dim3(heads, num_seqs), dim3(256), smem, stream,        \
                         (const T*)proj, row_stride, q_off, f_off, v_off, f_bias, lower, state, query_start_loc,      \
                         state_slots, norm_weight, eps, (T*)out, out_stride, heads, dim, vdim)
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
