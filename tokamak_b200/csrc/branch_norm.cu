// A branch that is normalised before it joins the residual stream:
//
//   y = branch * rsqrt(mean(branch^2) + eps_b) * post_w (* layer_scale)
//   x = resid + y                      (written back to resid unless `rows` selects rows)
//   out = x * rsqrt(mean(x^2) + eps_n) * next_w          (when a norm follows)
//   out = x                                              (next_w null: the next sublayer reads the stream itself)
//
// in one pass: the norm after a sublayer, the per-channel layer scale, the 32-bit residual sum
// and the norm in front of the next sublayer.  Statistics, sums and the residual stream are
// float32; `out` is rounded once to the activation type.  The branch comes in the activation
// type or as float32 partial sums [parts, tokens, hidden] of a split-K product.
//
// Either norm may work in groups: the row is split into equal consecutive parts and each is divided by
// its own root mean square (branch_norm_add_groups_kernel; one group is the plain norm).  That kernel also
// takes a row without a branch: the norm in front alone.
#include "common.cuh"
#include "group_norm.cuh"

namespace tk {

template <typename T>
__global__ void branch_norm_add_kernel(float* __restrict__ resid, const T* __restrict__ branch,
                                       const float* __restrict__ parts, int n_parts, size_t part_stride,
                                       const float* __restrict__ post_w, const float* __restrict__ layer_scale,
                                       const float* __restrict__ next_w, T* __restrict__ out,
                                       const int* __restrict__ rows, int hidden, float eps_b, float eps_n) {
  extern __shared__ float row[];          // the branch, then the new residual row
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  float* x = resid + (size_t)r * hidden;
  float ss = 0.0f;
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
    float b;
    if (branch != nullptr) {
      b = to_f32<T>(branch[(size_t)r * hidden + h]);
    } else {
      b = 0.0f;
      for (int s = 0; s < n_parts; ++s) b += parts[(size_t)s * part_stride + (size_t)r * hidden + h];
    }
    row[h] = b;
    ss += b * b;
  }
  ss = block_sum(ss, scratch);
  const float rstd_b = rsqrtf(ss / (float)hidden + eps_b);
  float ss2 = 0.0f;
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
    float y = row[h] * rstd_b;
    if (post_w != nullptr) y *= post_w[h];
    if (layer_scale != nullptr) y *= layer_scale[h];
    const float v = x[h] + y;
    if (rows == nullptr) x[h] = v;
    row[h] = v;
    ss2 += v * v;
  }
  if (out == nullptr) return;
  T* o = out + (size_t)i * hidden;
  if (next_w == nullptr) {
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) o[h] = from_f32<T>(row[h]);
    return;
  }
  ss2 = block_sum(ss2, scratch);
  const float rstd = rsqrtf(ss2 / (float)hidden + eps_n);
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) o[h] = from_f32<T>(row[h] * rstd * next_w[h]);
}

// The general form with groups: the row lies in shared memory, a warp takes a group at a time.
template <typename T>
__global__ void branch_norm_add_groups_kernel(float* __restrict__ resid, const T* __restrict__ branch,
                                              const float* __restrict__ parts, int n_parts, size_t part_stride,
                                              const float* __restrict__ post_w, const float* __restrict__ layer_scale,
                                              const float* __restrict__ next_w, T* __restrict__ out,
                                              const int* __restrict__ rows, int hidden, float eps_b, float eps_n,
                                              int groups_b, int groups_n) {
  extern __shared__ float row[];          // the branch, then the new residual row; behind it the groups' statistics
  float* rstd = row + hidden;
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  float* x = resid + (size_t)r * hidden;
  const bool has_branch = branch != nullptr || parts != nullptr;
  if (has_branch) {
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
      float b;
      if (branch != nullptr) {
        b = to_f32<T>(branch[(size_t)r * hidden + h]);
      } else {
        b = 0.0f;
        for (int s = 0; s < n_parts; ++s) b += parts[(size_t)s * part_stride + (size_t)r * hidden + h];
      }
      row[h] = b;
    }
    group_rstd(row, hidden, groups_b, eps_b, rstd);
  }
  const int size_b = hidden / groups_b;
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
    float v = x[h];
    if (has_branch) {
      float y = row[h] * rstd[h / size_b];
      if (post_w != nullptr) y *= post_w[h];
      if (layer_scale != nullptr) y *= layer_scale[h];
      v += y;
      if (rows == nullptr) x[h] = v;
    }
    row[h] = v;
  }
  if (out == nullptr) return;
  T* o = out + (size_t)i * hidden;
  if (next_w == nullptr) {
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) o[h] = from_f32<T>(row[h]);
    return;
  }
  group_rstd(row, hidden, groups_n, eps_n, rstd);
  const int size_n = hidden / groups_n;
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) o[h] = from_f32<T>(row[h] * rstd[h / size_n] * next_w[h]);
}

// Four neighbouring elements at once (the address is a multiple of four elements).
template <typename T> __device__ __forceinline__ float4 ld4(const T* p);
template <> __device__ __forceinline__ float4 ld4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 ld4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
template <typename T> __device__ __forceinline__ void st4(T* p, float4 v);
template <> __device__ __forceinline__ void st4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void st4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  uint2 o;
  *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = o;
}

// The same for rows whose length is a multiple of 4: a thread keeps kChunks pieces of four elements
// in registers through all three steps, so a row is read once and nothing goes through shared memory;
// the weights, which no kernel writes, are on their way before the kernel in front has finished.
// With a few rows (decoding) the kernel is three memory latencies long instead of a loop of them.
template <typename T, int kChunks>
__global__ void __launch_bounds__(512) branch_norm_add_vec_kernel(float* __restrict__ resid, const T* __restrict__ branch,
                                           const float* __restrict__ parts, int n_parts, size_t part_stride,
                                           const float* __restrict__ post_w, const float* __restrict__ layer_scale,
                                           const float* __restrict__ next_w, T* __restrict__ out,
                                           const int* __restrict__ rows, int hidden, float eps_b, float eps_n) {
  __shared__ float scratch[32];
  pdl_trigger();
  const float4 ones = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
  float4 w[kChunks], nw[kChunks];
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    w[c] = ones; nw[c] = ones;
    if (h < hidden) {
      if (post_w != nullptr) w[c] = ld4<float>(post_w + h);
      if (layer_scale != nullptr) {
        const float4 l = ld4<float>(layer_scale + h);
        w[c].x *= l.x; w[c].y *= l.y; w[c].z *= l.z; w[c].w *= l.w;
      }
      if (out != nullptr && next_w != nullptr) nw[c] = ld4<float>(next_w + h);
    }
  }
  pdl_wait();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  float* x = resid + (size_t)r * hidden;
  float4 b[kChunks], xv[kChunks];
  float ss = 0.0f;
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    b[c] = make_float4(0.0f, 0.0f, 0.0f, 0.0f); xv[c] = b[c];
    if (h < hidden) {
      xv[c] = ld4<float>(x + h);
      if (branch != nullptr) {
        b[c] = ld4<T>(branch + (size_t)r * hidden + h);
      } else {
        const float* src = parts + (size_t)r * hidden + h;
        for (int s = 0; s < n_parts; ++s) {
          const float4 v = ld4<float>(src + (size_t)s * part_stride);
          b[c].x += v.x; b[c].y += v.y; b[c].z += v.z; b[c].w += v.w;
        }
      }
      ss += b[c].x * b[c].x + b[c].y * b[c].y + b[c].z * b[c].z + b[c].w * b[c].w;
    }
  }
  ss = block_sum(ss, scratch);
  const float rstd_b = rsqrtf(ss / (float)hidden + eps_b);
  float ss2 = 0.0f;
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    // (branch * rstd) * (post_w * layer_scale): the two weights were multiplied on the way in
    float4 y = make_float4(b[c].x * rstd_b, b[c].y * rstd_b, b[c].z * rstd_b, b[c].w * rstd_b);
    if (post_w != nullptr || layer_scale != nullptr) { y.x *= w[c].x; y.y *= w[c].y; y.z *= w[c].z; y.w *= w[c].w; }
    xv[c].x += y.x; xv[c].y += y.y; xv[c].z += y.z; xv[c].w += y.w;
    if (h < hidden) {
      if (rows == nullptr) st4<float>(x + h, xv[c]);
      ss2 += xv[c].x * xv[c].x + xv[c].y * xv[c].y + xv[c].z * xv[c].z + xv[c].w * xv[c].w;
    }
  }
  if (out == nullptr) return;
  // without a norm in front of the next sublayer the row goes out as it is (every thread takes the same branch)
  const float rstd = next_w != nullptr ? rsqrtf(block_sum(ss2, scratch) / (float)hidden + eps_n) : 1.0f;
  T* o = out + (size_t)i * hidden;
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    if (h < hidden) {
      st4<T>(o + h, make_float4(xv[c].x * rstd * nw[c].x, xv[c].y * rstd * nw[c].y, xv[c].z * rstd * nw[c].z,
                                xv[c].w * rstd * nw[c].w));
    }
  }
}

// Two branches that join together, each after a norm of its own:
//   x = resid + a * rsqrt(mean(a^2) + eps_b) * w_a + b * rsqrt(mean(b^2) + eps_b) * w_b,   out = x * rsqrt(mean(x^2) + eps_n) * next_w
struct BranchPairParams {
  float* resid;
  const void* branch[2];        // activation type, or null: float32 partial sums
  const float* parts[2];
  int n_parts[2];
  size_t part_stride[2];
  const float* post_w[2];
  const float* next_w;
  void* out;
  const int* rows;
  int hidden;
  float eps_b, eps_n;
};

__device__ __forceinline__ float2 block_sum2(float2 v, float2* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
  v.x = warp_sum(v.x); v.y = warp_sum(v.y);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  const float2 r = lane < nwarps ? scratch[lane] : make_float2(0.0f, 0.0f);
  return make_float2(warp_sum(r.x), warp_sum(r.y));
}

// Any width: both branches lie in shared memory, the first's place takes the new row.
template <typename T>
__global__ void branch_pair_norm_add_kernel(BranchPairParams p) {
  extern __shared__ float row[];          // [2][hidden]
  __shared__ float2 scratch[32];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x, r = p.rows ? p.rows[i] : i, hidden = p.hidden;
  float* x = p.resid + (size_t)r * hidden;
  float2 ss = make_float2(0.0f, 0.0f);
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
    float v[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      if (p.branch[j] != nullptr) {
        v[j] = to_f32<T>(((const T*)p.branch[j])[(size_t)r * hidden + h]);
      } else {
        v[j] = 0.0f;
        for (int s = 0; s < p.n_parts[j]; ++s) v[j] += p.parts[j][(size_t)s * p.part_stride[j] + (size_t)r * hidden + h];
      }
      row[j * hidden + h] = v[j];
    }
    ss.x += v[0] * v[0]; ss.y += v[1] * v[1];
  }
  ss = block_sum2(ss, scratch);
  const float ra = rsqrtf(ss.x / (float)hidden + p.eps_b), rb = rsqrtf(ss.y / (float)hidden + p.eps_b);
  float2 sx = make_float2(0.0f, 0.0f);
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
    const float v = x[h] + (row[h] * ra * p.post_w[0][h] + row[hidden + h] * rb * p.post_w[1][h]);
    if (p.rows == nullptr) x[h] = v;
    row[h] = v;
    sx.x += v * v;
  }
  const float rstd = rsqrtf(block_sum2(sx, scratch).x / (float)hidden + p.eps_n);
  T* o = (T*)p.out + (size_t)i * hidden;
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) o[h] = from_f32<T>(row[h] * rstd * p.next_w[h]);
}

// Rows of a multiple of 4: everything stays in registers, the weights are asked for before the wait.
template <typename T, int kChunks>
__global__ void __launch_bounds__(512) branch_pair_norm_add_vec_kernel(BranchPairParams p) {
  __shared__ float2 scratch[32];
  pdl_trigger();
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  const int hidden = p.hidden;
  float4 wa[kChunks], wb[kChunks], nw[kChunks];
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    wa[c] = wb[c] = nw[c] = zero;
    if (h < hidden) { wa[c] = ld4<float>(p.post_w[0] + h); wb[c] = ld4<float>(p.post_w[1] + h); nw[c] = ld4<float>(p.next_w + h); }
  }
  pdl_wait();
  const int i = blockIdx.x, r = p.rows ? p.rows[i] : i;
  float* x = p.resid + (size_t)r * hidden;
  float4 v[2][kChunks], xv[kChunks];
  float2 ss = make_float2(0.0f, 0.0f);
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    v[0][c] = v[1][c] = xv[c] = zero;
    if (h >= hidden) continue;
    xv[c] = ld4<float>(x + h);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      if (p.branch[j] != nullptr) {
        v[j][c] = ld4<T>((const T*)p.branch[j] + (size_t)r * hidden + h);
      } else {
        const float* src = p.parts[j] + (size_t)r * hidden + h;
        for (int s = 0; s < p.n_parts[j]; ++s) {
          const float4 u = ld4<float>(src + (size_t)s * p.part_stride[j]);
          v[j][c].x += u.x; v[j][c].y += u.y; v[j][c].z += u.z; v[j][c].w += u.w;
        }
      }
    }
    ss.x += v[0][c].x * v[0][c].x + v[0][c].y * v[0][c].y + v[0][c].z * v[0][c].z + v[0][c].w * v[0][c].w;
    ss.y += v[1][c].x * v[1][c].x + v[1][c].y * v[1][c].y + v[1][c].z * v[1][c].z + v[1][c].w * v[1][c].w;
  }
  ss = block_sum2(ss, scratch);
  const float ra = rsqrtf(ss.x / (float)hidden + p.eps_b), rb = rsqrtf(ss.y / (float)hidden + p.eps_b);
  float2 sx = make_float2(0.0f, 0.0f);
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    if (h >= hidden) continue;
    xv[c].x += v[0][c].x * ra * wa[c].x + v[1][c].x * rb * wb[c].x;
    xv[c].y += v[0][c].y * ra * wa[c].y + v[1][c].y * rb * wb[c].y;
    xv[c].z += v[0][c].z * ra * wa[c].z + v[1][c].z * rb * wb[c].z;
    xv[c].w += v[0][c].w * ra * wa[c].w + v[1][c].w * rb * wb[c].w;
    if (p.rows == nullptr) st4<float>(x + h, xv[c]);
    sx.x += xv[c].x * xv[c].x + xv[c].y * xv[c].y + xv[c].z * xv[c].z + xv[c].w * xv[c].w;
  }
  const float rstd = rsqrtf(block_sum2(sx, scratch).x / (float)hidden + p.eps_n);
  T* o = (T*)p.out + (size_t)i * hidden;
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int h = (threadIdx.x + c * blockDim.x) * 4;
    if (h < hidden) st4<T>(o + h, make_float4(xv[c].x * rstd * nw[c].x, xv[c].y * rstd * nw[c].y, xv[c].z * rstd * nw[c].z,
                                              xv[c].w * rstd * nw[c].w));
  }
}

}  // namespace tk

TK_API int tk_branch_norm_add(float* resid, const void* branch, const float* parts, int n_parts,
                              long long part_stride, const float* post_w, const float* layer_scale,
                              const float* next_w, void* out, const int* rows, int n_rows, int hidden,
                              float eps_b, float eps_n, int groups_b, int groups_n, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  const bool grouped = groups_b > 1 || groups_n > 1 || (branch == nullptr && parts == nullptr);
  if (hidden < 1 || hidden > 12288 || (branch != nullptr && parts != nullptr) || groups_b < 1 || groups_n < 1 ||
      hidden % groups_b || hidden % groups_n) {
    return (int)cudaErrorInvalidValue;
  }
  cudaError_t e = cudaSuccess;
  if (grouped) {
    // few rows fill few SMs: more threads a row then (a group's sum is a warp's in either shape, the same bits)
    const int threads = hidden >= 4096 && n_rows <= 64 ? 1024 : hidden >= 2048 && n_rows <= 64 ? 512 : hidden >= 1024 ? 256 : 128;
    const int most = groups_b > groups_n ? groups_b : groups_n;
    const size_t smem = (size_t)(hidden + most) * sizeof(float);
    if (smem > 96 * 1024) return (int)cudaErrorInvalidValue;
#define TK_BRANCH_NORM_GROUPS(T)                                                                                       \
    do {                                                                                                               \
      if (smem > 48 * 1024) {                                                                                          \
        e = cudaFuncSetAttribute(tk::branch_norm_add_groups_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                 (int)smem);                                                                           \
        if (e != cudaSuccess) return (int)e;                                                                           \
      }                                                                                                                \
      e = tk::launch(tk::branch_norm_add_groups_kernel<T>, dim3((unsigned)n_rows), dim3(threads), smem, stream, resid, \
                     (const T*)branch, parts, n_parts, (size_t)part_stride, post_w, layer_scale, next_w, (T*)out,      \
                     rows, hidden, eps_b, eps_n, groups_b, groups_n);                                                  \
    } while (0)
    if (dtype == tk::kF32) { TK_BRANCH_NORM_GROUPS(float); }
    else if (dtype == tk::kBF16) { TK_BRANCH_NORM_GROUPS(__nv_bfloat16); }
    else return (int)cudaErrorInvalidValue;
#undef TK_BRANCH_NORM_GROUPS
    return (int)e;
  }
  if (hidden % 4 == 0) {
    const int quads = hidden / 4;
    const int threads = quads >= 512 ? 512 : (quads + 31) / 32 * 32;
    const int chunks = (quads + threads - 1) / threads;        // at most 6: hidden <= 12288
#define TK_BRANCH_NORM_VEC(K)                                                                                         \
    TK_DISPATCH_DTYPE(dtype, T,                                                                                      \
                      e = tk::launch(tk::branch_norm_add_vec_kernel<T, K>, dim3((unsigned)n_rows), dim3(threads), 0, \
                                     stream, resid, (const T*)branch, parts, n_parts, (size_t)part_stride, post_w,   \
                                     layer_scale, next_w, (T*)out, rows, hidden, eps_b, eps_n))
    if (chunks <= 1) { TK_BRANCH_NORM_VEC(1); }
    else if (chunks <= 2) { TK_BRANCH_NORM_VEC(2); }
    else if (chunks <= 4) { TK_BRANCH_NORM_VEC(4); }
    else { TK_BRANCH_NORM_VEC(8); }
#undef TK_BRANCH_NORM_VEC
    return (int)e;
  }
  const int threads = hidden >= 1024 ? 256 : 128;
  TK_DISPATCH_DTYPE(dtype, T,
                    e = tk::launch(tk::branch_norm_add_kernel<T>, dim3((unsigned)n_rows), dim3(threads),
                                   (size_t)hidden * sizeof(float), stream, resid, (const T*)branch, parts, n_parts,
                                   (size_t)part_stride, post_w, layer_scale, next_w, (T*)out, rows, hidden, eps_b,
                                   eps_n));
  return (int)e;
}

TK_API int tk_branch_pair_norm_add(float* resid, const void* a, const float* a_parts, int a_n, long long a_stride,
                                   const float* a_w, const void* b, const float* b_parts, int b_n, long long b_stride,
                                   const float* b_w, const float* next_w, void* out, const int* rows, int n_rows,
                                   int hidden, float eps_b, float eps_n, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (hidden < 1 || hidden > 12288 || (a == nullptr) == (a_parts == nullptr) || (b == nullptr) == (b_parts == nullptr) ||
      a_w == nullptr || b_w == nullptr || next_w == nullptr || out == nullptr) {
    return (int)cudaErrorInvalidValue;
  }
  tk::BranchPairParams p;
  p.resid = resid; p.branch[0] = a; p.branch[1] = b; p.parts[0] = a_parts; p.parts[1] = b_parts;
  p.n_parts[0] = a_n; p.n_parts[1] = b_n; p.part_stride[0] = (size_t)a_stride; p.part_stride[1] = (size_t)b_stride;
  p.post_w[0] = a_w; p.post_w[1] = b_w; p.next_w = next_w; p.out = out; p.rows = rows; p.hidden = hidden;
  p.eps_b = eps_b; p.eps_n = eps_n;
  cudaError_t e = cudaSuccess;
  if (hidden % 4 == 0 && hidden <= 8192) {
    const int quads = hidden / 4;
    const int threads = quads >= 512 ? 512 : (quads + 31) / 32 * 32;
    const int chunks = (quads + threads - 1) / threads;
#define TK_BRANCH_PAIR_VEC(K)                                                                                            \
    TK_DISPATCH_DTYPE(dtype, T, (e = tk::launch(tk::branch_pair_norm_add_vec_kernel<T, K>, dim3((unsigned)n_rows),       \
                                                dim3(threads), 0, stream, p)))
    if (chunks <= 1) { TK_BRANCH_PAIR_VEC(1); }
    else if (chunks <= 2) { TK_BRANCH_PAIR_VEC(2); }
    else { TK_BRANCH_PAIR_VEC(4); }
#undef TK_BRANCH_PAIR_VEC
    return (int)e;
  }
  const size_t smem = (size_t)2 * hidden * sizeof(float);
  const int threads = hidden >= 1024 ? 256 : 128;
#define TK_BRANCH_PAIR(T)                                                                                              \
  do {                                                                                                                 \
    if (smem > 48 * 1024) {                                                                                            \
      e = cudaFuncSetAttribute(tk::branch_pair_norm_add_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,        \
                               (int)smem);                                                                             \
      if (e != cudaSuccess) return (int)e;                                                                             \
    }                                                                                                                  \
    e = tk::launch(tk::branch_pair_norm_add_kernel<T>, dim3((unsigned)n_rows), dim3(threads), smem, stream, p);        \
  } while (0)
  if (dtype == tk::kF32) { TK_BRANCH_PAIR(float); }
  else if (dtype == tk::kBF16) { TK_BRANCH_PAIR(__nv_bfloat16); }
  else return (int)cudaErrorInvalidValue;
#undef TK_BRANCH_PAIR
  return (int)e;
}
