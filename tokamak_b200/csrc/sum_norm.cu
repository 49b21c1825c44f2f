// The residual sum of several branches at once, and the RMS norm of the result:
//
//   x = resid + branch_0 + branch_1 + extra + vector        float32
//   out = w * x / sqrt(mean(x^2) + eps)                     rounded once on store
//
// A block whose sublayers read the same input side by side leaves all their outputs to the next norm; what else
// joins the stream between two blocks (rows kept from earlier, one vector for every token) rides along.  A
// branch is one of
//   1  rows in the activation type
//   2  the float32 partial sums of a split product
//   3  the experts' output rows (bfloat16) of a mixture: sum_k weights[t, k] * y[pair_row[t * top + k]]
//   4  the same with float32 rows
//      (row t * top + k without a list; a choice of weight 0 is skipped: it may have no row)
// each formed in float32 in a fixed order before it joins, so a row does not depend on what else is in the step.
// With a list of rows only those are summed and normed and the stream is left as it is (the model's last norm).
// One block per row.
#include "common.cuh"
#include "stacked_input.cuh"

namespace tk {

constexpr int kSumTerms = 3;

struct SumTerm {
  const void* data;         // null: no branch
  int kind;
  int count;                // 2: number of partial sums; 3, 4: choices of a token
  long long stride;         // 2: elements from one partial sum to the next
  const float* weights;     // 3, 4: [n_tokens, count]
  const int* pair_row;      // 3, 4: [n_tokens * count] or null
};

struct SumNormParams {
  float* resid;             // [n_tokens, width]
  SumTerm term[kSumTerms];
  const float* extra;       // [n_tokens, width] or null
  const float* vector;      // [width] or null
  const float* weight;      // [width]
  void* out;                // [n_rows, width] activation type
  const int* rows;          // [n_rows] or null: every row, and the sum is written back
  int n_rows, n_tokens, width;
  float eps;
};

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 axpy4(float w, float4 v, float4 a) {
  return make_float4(a.x + w * v.x, a.y + w * v.y, a.z + w * v.z, a.w + w * v.w);
}

// Columns c .. c + 3 of row t of a branch (term1: one column).
template <typename T>
__device__ __forceinline__ float4 term4(const SumTerm& s, int t, int c, int width) {
  const size_t at = (size_t)t * width + c;
  float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if (s.kind == 1) return ld4<T>((const T*)s.data + at);
  if (s.kind == 2) {
    for (int i = 0; i < s.count; ++i) acc = add4(acc, ld4<float>((const float*)s.data + (size_t)i * s.stride + at));
    return acc;
  }
  for (int k = 0; k < s.count; ++k) {
    const size_t pair = (size_t)t * s.count + k;
    const float w = s.weights[pair];
    if (w == 0.0f) continue;
    const size_t row = s.pair_row != nullptr ? (size_t)s.pair_row[pair] : pair;
    if (s.kind == 3) acc = axpy4(w, ld4<__nv_bfloat16>((const __nv_bfloat16*)s.data + row * width + c), acc);
    else acc = axpy4(w, ld4<float>((const float*)s.data + row * width + c), acc);
  }
  return acc;
}

template <typename T>
__device__ __forceinline__ float term1(const SumTerm& s, int t, int c, int width) {
  const size_t at = (size_t)t * width + c;
  float acc = 0.0f;
  if (s.kind == 1) return to_f32<T>(((const T*)s.data)[at]);
  if (s.kind == 2) {
    for (int i = 0; i < s.count; ++i) acc += ((const float*)s.data)[(size_t)i * s.stride + at];
    return acc;
  }
  for (int k = 0; k < s.count; ++k) {
    const size_t pair = (size_t)t * s.count + k;
    const float w = s.weights[pair];
    if (w == 0.0f) continue;
    const size_t row = s.pair_row != nullptr ? (size_t)s.pair_row[pair] : pair;
    acc += w * (s.kind == 3 ? __bfloat162float(((const __nv_bfloat16*)s.data)[row * width + c])
                            : ((const float*)s.data)[row * width + c]);
  }
  return acc;
}

// Rows of any width: the row is kept in shared memory between the sum of squares and the scaling.
template <typename T>
__global__ void sum_rmsnorm_kernel(SumNormParams p) {
  extern __shared__ float row[];
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int t = p.rows != nullptr ? p.rows[blockIdx.x] : blockIdx.x;
  if (t < 0 || t >= p.n_tokens) return;
  float* x = p.resid + (size_t)t * p.width;
  float ss = 0.0f;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    float v = x[c];
#pragma unroll
    for (int i = 0; i < kSumTerms; ++i) {
      if (p.term[i].data != nullptr) v += term1<T>(p.term[i], t, c, p.width);
    }
    if (p.extra != nullptr) v += p.extra[(size_t)t * p.width + c];
    if (p.vector != nullptr) v += p.vector[c];
    if (p.rows == nullptr) x[c] = v;
    row[c] = v;
    ss += v * v;
  }
  const float rstd = rsqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
  T* out = (T*)p.out + (size_t)blockIdx.x * p.width;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) out[c] = from_f32<T>(row[c] * rstd * p.weight[c]);
}

constexpr int kSumPieces = 4;

// Widths that are a multiple of 4: 16-byte accesses, the row in registers (K pieces of four columns a thread), the
// norm's weight and the vector asked for before the wait for the kernel in front.
template <typename T, int K>
__global__ void __launch_bounds__(512) sum_rmsnorm_vec_kernel(SumNormParams p) {
  __shared__ float scratch[32];
  pdl_trigger();
  const int chunks = p.width >> 2;
  float4 w[K], v[K];
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    w[k] = v[k] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (i < chunks) {
      w[k] = reinterpret_cast<const float4*>(p.weight)[i];
      if (p.vector != nullptr) v[k] = reinterpret_cast<const float4*>(p.vector)[i];
    }
  }
  pdl_wait();
  const int t = p.rows != nullptr ? p.rows[blockIdx.x] : blockIdx.x;
  if (t < 0 || t >= p.n_tokens) return;
  float* x = p.resid + (size_t)t * p.width;
  float ss = 0.0f;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i >= chunks) continue;
    float4 a = *reinterpret_cast<const float4*>(x + 4 * i);
#pragma unroll
    for (int j = 0; j < kSumTerms; ++j) {
      if (p.term[j].data != nullptr) a = add4(a, term4<T>(p.term[j], t, 4 * i, p.width));
    }
    if (p.extra != nullptr) a = add4(a, ld4<float>(p.extra + (size_t)t * p.width + 4 * i));
    a = add4(a, v[k]);
    if (p.rows == nullptr) *reinterpret_cast<float4*>(x + 4 * i) = a;
    v[k] = a;
    ss += (a.x * a.x + a.y * a.y) + (a.z * a.z + a.w * a.w);
  }
  const float rstd = rsqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
  T* out = (T*)p.out + (size_t)blockIdx.x * p.width;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < chunks) {
      st4<T>(out + 4 * i, make_float4(v[k].x * rstd * w[k].x, v[k].y * rstd * w[k].y, v[k].z * rstd * w[k].z,
                                      v[k].w * rstd * w[k].w));
    }
  }
}

static bool sum_term_ok(const SumTerm& s) {
  if (s.data == nullptr) return true;
  if (s.kind < 1 || s.kind > 4 || s.count < 1) return false;
  return s.kind < 3 || s.weights != nullptr;
}

}  // namespace tk

TK_API int tk_sum_rmsnorm(float* resid, const void* a, int a_kind, int a_count, long long a_stride, const float* a_weights,
                          const int* a_pair_row, const void* b, int b_kind, int b_count, long long b_stride,
                          const float* b_weights, const int* b_pair_row, const void* c, int c_kind, int c_count,
                          long long c_stride, const float* c_weights, const int* c_pair_row, const float* extra, const float* vector,
                          const float* weight, void* out, const int* rows, int n_rows, int n_tokens, int width, float eps,
                          int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  tk::SumNormParams p;
  p.resid = resid;
  p.term[0] = tk::SumTerm{a, a_kind, a_count, a_stride, a_weights, a_pair_row};
  p.term[1] = tk::SumTerm{b, b_kind, b_count, b_stride, b_weights, b_pair_row};
  p.term[2] = tk::SumTerm{c, c_kind, c_count, c_stride, c_weights, c_pair_row};
  p.extra = extra; p.vector = vector; p.weight = weight; p.out = out; p.rows = rows;
  p.n_rows = n_rows; p.n_tokens = n_tokens; p.width = width; p.eps = eps;
  if (resid == nullptr || weight == nullptr || out == nullptr || width < 1 || !tk::sum_term_ok(p.term[0]) ||
      !tk::sum_term_ok(p.term[1]) || !tk::sum_term_ok(p.term[2]) || (size_t)width * sizeof(float) > 200 * 1024) {
    return (int)cudaErrorInvalidValue;
  }
  cudaError_t e = cudaSuccess;
  const int chunks = width / 4;
  if (width % 4 == 0 && a_stride % 4 == 0 && b_stride % 4 == 0 && c_stride % 4 == 0 && chunks <= 512 * tk::kSumPieces) {
    // few rows get a thread per piece of four columns, many rows two pieces a thread
    int threads = ((n_rows <= 296 ? chunks : (chunks + 1) / 2) + 31) / 32 * 32;
    if (threads > 512) threads = 512;
    if (threads < 64) threads = 64;
    const int pieces = (chunks + threads - 1) / threads;
#define TK_SUM_VEC(K) \
    TK_DISPATCH_DTYPE(dtype, T, (e = tk::launch(tk::sum_rmsnorm_vec_kernel<T, K>, dim3((unsigned)n_rows), dim3(threads), 0, stream, p)))
    if (pieces <= 1) { TK_SUM_VEC(1); } else if (pieces <= 2) { TK_SUM_VEC(2); } else { TK_SUM_VEC(4); }
#undef TK_SUM_VEC
    return (int)e;
  }
  const size_t smem = (size_t)width * sizeof(float);
  int threads = n_rows <= 64 ? 512 : 256;
  while (threads > 64 && threads / 2 >= width) threads /= 2;
#define TK_SUM(T)                                                                                                     \
  do {                                                                                                                \
    if (smem > 48 * 1024) {                                                                                           \
      e = cudaFuncSetAttribute(tk::sum_rmsnorm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
      if (e != cudaSuccess) return (int)e;                                                                            \
    }                                                                                                                 \
    e = tk::launch(tk::sum_rmsnorm_kernel<T>, dim3((unsigned)n_rows), dim3(threads), smem, stream, p);                \
  } while (0)
  if (dtype == tk::kF32) { TK_SUM(float); } else if (dtype == tk::kBF16) { TK_SUM(__nv_bfloat16); }
  else return (int)cudaErrorInvalidValue;
#undef TK_SUM
  return (int)e;
}
