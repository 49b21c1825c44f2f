// Embedding lookup, residual add + RMSNorm, and the SwiGLU gate.
//
// The residual stream is float32 in every engine dtype, so the residual sum is
// always a 32-bit sum; the normalised output is rounded once to the activation
// type.  RMSNorm statistics are 32-bit as in the reference
// (src/tokamak/model/layers.py:28-33).
#include "common.cuh"
#include "stacked_input.cuh"
#include "timeline.cuh"

namespace tk {

// resid[t, :] = float(table[ids[t], :]) * scale                 (src/tokamak/model/transformer.py:140)
template <typename T>
__global__ void embed_gather_kernel(const T* __restrict__ table, const int* __restrict__ ids,
                                    float* __restrict__ resid, int hidden, int vocab, float scale, int accumulate,
                                    int* err) {
  pdl_trigger();
  if (threadIdx.x == 0) tl_mark(4, 0);
  pdl_wait();
  if (threadIdx.x == 0) tl_mark(4, 1);
  const int t = blockIdx.x;
  const int id = ids[t];
  float* out = resid + (size_t)t * hidden;
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) set_error(err, kErrTokenId, t, id, vocab);
    if (!accumulate) {
      for (int h = threadIdx.x; h < hidden; h += blockDim.x) out[h] = 0.0f;
    }
    return;
  }
  const T* row = table + (size_t)id * hidden;
  if (accumulate) {     // a second table's rows join the rows that are there (a learned position table)
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) out[h] += to_f32<T>(row[h]) * scale;
    return;
  }
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) out[h] = to_f32<T>(row[h]) * scale;
}

// resid[t, :] = float(table[ids[t], :]) * scale + float(pairs[row, :]), where row is a hash of the request's
// previous token and this one, (prev * mul_prev + cur * mul_cur) mod buckets, and `buckets` (the table's last row)
// for a request's first token.  The previous token is the one before in the step or, for the first token of a
// request's portion, the one that last[slot] holds from the step before; the block of that first token also moves
// last[slot] on to the portion's last token, after it has read it, so no other block touches the entry.
// keep: a second copy of the rows, or null.
struct EmbedBigramParams {
  const void* table; const void* pairs;
  const int* ids; const int* positions; const int* tok_req; const int* req_q_start; const int* req_q_len;
  const int* req_slot;
  int* last;                // [max_slots]
  float* resid; float* keep;
  int n_tokens, n_reqs, max_slots, hidden, vocab, buckets;
  long long mul_prev, mul_cur;
  float scale;
  int* err;
};

template <typename T>
__global__ void embed_bigram_kernel(EmbedBigramParams p) {
  __shared__ int s_id, s_row;
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  if (threadIdx.x == 0) {
    int id = p.ids[t], row = -1;
    const int pos = p.positions[t], r = p.tok_req[t];
    if (id < 0 || id >= p.vocab) {
      set_error(p.err, kErrTokenId, t, id, p.vocab);
      id = -1;
    }
    if (pos < 0) {
      set_error(p.err, kErrPosition, t, pos, 0);
    } else if (r < 0 || r >= p.n_reqs) {
      set_error(p.err, kErrRequest, t, r, p.n_reqs);
    } else {
      const int first = p.req_q_start[r], end = first + p.req_q_len[r], slot = p.req_slot[r];
      if (slot < 0 || slot >= p.max_slots || first < 0 || t < first || t >= end || end > p.n_tokens) {
        set_error(p.err, kErrRequest, t, r, slot);
      } else {
        int prev = 0;
        if (pos > 0) prev = t > first ? p.ids[t - 1] : p.last[slot];
        if (t == first) p.last[slot] = p.ids[end - 1];
        if (pos == 0) {
          row = p.buckets;
        } else if (prev < 0 || prev >= p.vocab) {
          set_error(p.err, kErrTokenId, t, prev, p.vocab);
        } else if (id >= 0) {
          const long long hash = ((long long)prev * p.mul_prev + (long long)id * p.mul_cur) % p.buckets;
          row = (int)(hash < 0 ? hash + p.buckets : hash);
        }
      }
    }
    s_id = id; s_row = row;
  }
  __syncthreads();
  const int id = s_id, row = s_row;
  const bool ok = id >= 0 && row >= 0;
  const T* a = (const T*)p.table + (size_t)(ok ? id : 0) * p.hidden;
  const T* b = (const T*)p.pairs + (size_t)(ok ? row : 0) * p.hidden;
  float* out = p.resid + (size_t)t * p.hidden;
  float* copy = p.keep != nullptr ? p.keep + (size_t)t * p.hidden : nullptr;
  if ((p.hidden & 3) == 0) {
    for (int h = threadIdx.x * 4; h < p.hidden; h += blockDim.x * 4) {
      float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (ok) {
        const float4 x = ld4<T>(a + h), y = ld4<T>(b + h);
        v = make_float4(x.x * p.scale + y.x, x.y * p.scale + y.y, x.z * p.scale + y.z, x.w * p.scale + y.w);
      }
      *reinterpret_cast<float4*>(out + h) = v;
      if (copy != nullptr) *reinterpret_cast<float4*>(copy + h) = v;
    }
    return;
  }
  for (int h = threadIdx.x; h < p.hidden; h += blockDim.x) {
    const float v = ok ? to_f32<T>(a[h]) * p.scale + to_f32<T>(b[h]) : 0.0f;
    out[h] = v;
    if (copy != nullptr) copy[h] = v;
  }
}

// x = resid[r] (+ delta[r]);  resid[r] = x (when written back);
// out[i] = weight * x * rsqrt(mean(x^2) + eps)
// rows == nullptr: r = i = blockIdx.x and the sum is written back to resid.
// rows != nullptr: r = rows[i]; resid is left untouched (used for the final norm
// over the positions whose logits are wanted).
template <typename TOut, typename TDelta>
__global__ void add_rmsnorm_kernel(float* __restrict__ resid, const TDelta* __restrict__ delta,
                                   const float* __restrict__ parts, int n_parts, size_t part_stride,
                                   const float* __restrict__ weight, TOut* __restrict__ out,
                                   const int* __restrict__ rows, int hidden, float eps) {
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  float* x = resid + (size_t)r * hidden;
  const TDelta* d = delta ? delta + (size_t)r * hidden : nullptr;
  const float* ps = parts ? parts + (size_t)r * hidden : nullptr;
  const bool has_delta = (d != nullptr) || (ps != nullptr);
  const bool write_back = (rows == nullptr) && has_delta;
  auto branch = [&](int h) -> float {
    if (d) return to_f32<TDelta>(d[h]);
    float acc = 0.0f;
    for (int s = 0; s < n_parts; ++s) acc += ps[(size_t)s * part_stride + h];
    return acc;
  };
  float ss = 0.0f;
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
    float v = x[h];
    if (has_delta) v += branch(h);
    if (write_back) x[h] = v;
    ss += v * v;
  }
  ss = block_sum(ss, scratch);
  const float rstd = rsqrtf(ss / (float)hidden + eps);
  TOut* o = out + (size_t)i * hidden;
  for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
    float v;
    if (write_back || !has_delta) {
      v = x[h];
    } else {
      v = x[h] + branch(h);
    }
    o[h] = from_f32<TOut>(v * rstd * weight[h]);
  }
}

// Same operation for widths that are a multiple of 8: every thread keeps its values in
// registers between the sum of squares and the scaling, so the row is read once, with
// 16- and 32-byte accesses.
template <typename T> struct Vec8;
template <> struct Vec8<float> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    const float4 b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
};
template <> struct Vec8<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[8]) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
  }
};

template <typename T, int ITERS>
__global__ void add_rmsnorm_vec_kernel(float* __restrict__ resid, const T* __restrict__ delta,
                                       const float* __restrict__ parts, int n_parts, size_t part_stride,
                                       const float* __restrict__ weight, T* __restrict__ out,
                                       const int* __restrict__ rows, int hidden, float eps) {
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  float* x = resid + (size_t)r * hidden;
  const T* d = delta ? delta + (size_t)r * hidden : nullptr;
  const float* ps = parts ? parts + (size_t)r * hidden : nullptr;
  const bool write_back = (rows == nullptr) && (d != nullptr || ps != nullptr);
  float v[ITERS][8];
  float ss = 0.0f;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int h = (it * blockDim.x + threadIdx.x) * 8;
    if (h < hidden) {
      Vec8<float>::load(x + h, v[it]);
      if (d) {
        float dv[8];
        Vec8<T>::load(d + h, dv);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[it][e] += dv[e];
      } else if (ps) {
        for (int s = 0; s < n_parts; ++s) {
          float dv[8];
          Vec8<float>::load(ps + (size_t)s * part_stride + h, dv);
#pragma unroll
          for (int e = 0; e < 8; ++e) v[it][e] += dv[e];
        }
      }
      if (write_back) Vec8<float>::store(x + h, v[it]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += v[it][e] * v[it][e];
    }
  }
  ss = block_sum(ss, scratch);
  const float rstd = rsqrtf(ss / (float)hidden + eps);
  T* o = out + (size_t)i * hidden;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int h = (it * blockDim.x + threadIdx.x) * 8;
    if (h < hidden) {
      float w[8], y[8];
      Vec8<float>::load(weight + h, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = v[it][e] * rstd * w[e];
      Vec8<T>::store(o + h, y);
    }
  }
}

// out[t, j] = act(gate[t, j]) * up[t, j]           (act = silu: src/tokamak/model/layers.py:103)
// A row of gu holds gate and up alternating in blocks: `block` gate values, then the `block` up
// values of the same outputs (block = inter: all gate values, then all up values).
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gu, const float* __restrict__ parts, int n_parts,
                              size_t part_stride, T* __restrict__ out, int inter, int block, size_t total, int act) {
  pdl_trigger();
  pdl_wait();
  size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; idx < total; idx += stride) {
    const size_t t = idx / inter;
    const int j = (int)(idx - t * inter);
    const size_t at = t * 2 * inter + (size_t)(j / block) * 2 * block + (j % block);
    float g, u;
    if (parts == nullptr) {
      g = to_f32<T>(gu[at]);
      u = to_f32<T>(gu[at + block]);
    } else {
      g = 0.0f; u = 0.0f;
      for (int s = 0; s < n_parts; ++s) {
        g += parts[s * part_stride + at];
        u += parts[s * part_stride + at + block];
      }
    }
    out[idx] = from_f32<T>(glu_act(g, act) * u);
  }
}

// The same for an intermediate size and a block that are multiples of 8: 16-byte loads and stores.
template <typename T>
__global__ void swiglu_vec_kernel(const T* __restrict__ gu, const float* __restrict__ parts, int n_parts,
                                  size_t part_stride, T* __restrict__ out, int inter, int block, size_t total8, int act) {
  pdl_trigger();
  pdl_wait();
  size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  const int per_row = inter / 8;
  for (; idx < total8; idx += stride) {
    const size_t t = idx / per_row;
    const int j = (int)(idx - t * per_row) * 8;
    const size_t at = t * 2 * inter + (size_t)(j / block) * 2 * block + (j % block);
    float g[8], u[8], y[8];
    if (parts == nullptr) {
      Vec8<T>::load(gu + at, g);
      Vec8<T>::load(gu + at + block, u);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) { g[e] = 0.0f; u[e] = 0.0f; }
      for (int s = 0; s < n_parts; ++s) {
        float a[8], b[8];
        Vec8<float>::load(parts + s * part_stride + at, a);
        Vec8<float>::load(parts + s * part_stride + at + block, b);
#pragma unroll
        for (int e = 0; e < 8; ++e) { g[e] += a[e]; u[e] += b[e]; }
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) y[e] = glu_act(g[e], act) * u[e];
    Vec8<T>::store(out + t * inter + j, y);
  }
}

// Ungated feed-forward activations, out[t, j] = act(x[t, j]): 0 = silu, 1 = the tanh form of gelu, 2 = relu(x)^2.
// x may be the float32 partial sums of a split-K product.
template <typename T>
__global__ void unary_act_kernel(const T* __restrict__ x, const float* __restrict__ parts, int n_parts,
                                 size_t part_stride, T* __restrict__ out, size_t total, int act) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    float z;
    if (parts == nullptr) z = to_f32<T>(x[i]);
    else { z = 0.0f; for (int s = 0; s < n_parts; ++s) z += parts[(size_t)s * part_stride + i]; }
    out[i] = from_f32<T>(unary_act(z, act));
  }
}

}  // namespace tk

TK_TIMELINE_SETTER(elementwise)

TK_API int tk_embed_gather(const void* table, int dtype, const int* ids, float* resid, int n_tokens,
                           int hidden, int vocab, float scale, int accumulate, int* err, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  const int threads = hidden >= 1024 ? 256 : 128;
  cudaError_t e = cudaSuccess;
  TK_DISPATCH_DTYPE(dtype, T,
                    e = tk::launch(tk::embed_gather_kernel<T>, dim3(n_tokens), dim3(threads), 0, stream,
                                       (const T*)table, ids, resid, hidden, vocab, scale, accumulate, err));
  return (int)e;
}

TK_API int tk_embed_bigram(const void* table, const void* pairs, int dtype, const int* ids, const int* positions,
                           const int* tok_req, const int* req_q_start, const int* req_q_len, const int* req_slot, int* last,
                           float* resid, float* keep, int n_tokens, int n_reqs, int max_slots, int hidden, int vocab,
                           int buckets, long long mul_prev, long long mul_cur, float scale, int* err, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (buckets < 1 || hidden < 1 || last == nullptr) return (int)cudaErrorInvalidValue;
  tk::EmbedBigramParams p;
  p.table = table; p.pairs = pairs; p.ids = ids; p.positions = positions; p.tok_req = tok_req;
  p.req_q_start = req_q_start; p.req_q_len = req_q_len; p.req_slot = req_slot; p.last = last;
  p.resid = resid; p.keep = keep; p.n_tokens = n_tokens; p.n_reqs = n_reqs; p.max_slots = max_slots; p.hidden = hidden;
  p.vocab = vocab; p.buckets = buckets; p.mul_prev = mul_prev; p.mul_cur = mul_cur; p.scale = scale; p.err = err;
  const int threads = hidden >= 2048 ? 256 : (hidden >= 512 ? 128 : 64);
  cudaError_t e = cudaSuccess;
  TK_DISPATCH_DTYPE(dtype, T, e = tk::launch(tk::embed_bigram_kernel<T>, dim3(n_tokens), dim3(threads), 0, stream, p));
  return (int)e;
}

// delta: branch output in the activation type, or null.  parts: float32 partial sums of the
// branch output [n_parts, rows of resid, hidden] (part_stride elements apart), or null.
TK_API int tk_add_rmsnorm(float* resid, const void* delta, const float* parts, int n_parts,
                          long long part_stride, const float* weight, void* out, const int* rows,
                          int n_rows, int hidden, float eps, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (parts != nullptr && (delta != nullptr || n_parts < 1)) return (int)cudaErrorInvalidValue;
  cudaError_t e = cudaSuccess;
  if (hidden % 8 == 0 && hidden <= 4 * 512 * 8) {
    // one pass with the row in registers: threads * 8 * ITERS >= hidden
    int threads = ((hidden / 8 + 31) / 32) * 32;
    int iters = 1;
    if (threads > 512) { iters = (hidden / 8 + 511) / 512; threads = 512; }
    if (threads > 256 && iters == 1 && n_rows >= 64) { threads = (threads / 2 + 31) / 32 * 32; iters = 2; }
    if (iters == 3) iters = 4;
#define TK_LAUNCH_VEC(IT)                                                                       \
    TK_DISPATCH_DTYPE(dtype, T,                                                                 \
                      (e = tk::launch(tk::add_rmsnorm_vec_kernel<T, IT>, dim3(n_rows), dim3(threads), 0, \
                                      stream, resid, (const T*)delta, parts, n_parts,             \
                                      (size_t)part_stride, weight, (T*)out, rows, hidden, eps)))
    if (iters == 1) { TK_LAUNCH_VEC(1); } else if (iters == 2) { TK_LAUNCH_VEC(2); } else { TK_LAUNCH_VEC(4); }
#undef TK_LAUNCH_VEC
    return (int)e;
  }
  const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
  TK_DISPATCH_DTYPE(dtype, T,
                    (e = tk::launch(tk::add_rmsnorm_kernel<T, T>, dim3(n_rows), dim3(threads), 0, stream,
                                    resid, (const T*)delta, parts, n_parts, (size_t)part_stride, weight,
                                    (T*)out, rows, hidden, eps)));
  return (int)e;
}

TK_API int tk_swiglu(const void* gate_up, const float* parts, int n_parts, long long part_stride,
                     void* out, int n_tokens, int inter, int block, int dtype, int act, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (block <= 0 || inter % block != 0) return (int)cudaErrorInvalidValue;
  const size_t total = (size_t)n_tokens * inter;
  const int threads = 256;
  cudaError_t e = cudaSuccess;
  if (inter % 8 == 0 && block % 8 == 0) {
    const size_t total8 = total / 8;
    size_t vblocks = (total8 + threads - 1) / threads;
    if (vblocks > 148 * 32) vblocks = 148 * 32;
    TK_DISPATCH_DTYPE(dtype, T,
                      e = tk::launch(tk::swiglu_vec_kernel<T>, dim3((unsigned)vblocks), dim3(threads), 0, stream,
                                     (const T*)gate_up, parts, n_parts, (size_t)part_stride, (T*)out, inter,
                                     block, total8, act));
    return (int)e;
  }
  size_t blocks = (total + threads - 1) / threads;
  if (blocks > 148 * 16) blocks = 148 * 16;
  TK_DISPATCH_DTYPE(dtype, T,
                    e = tk::launch(tk::swiglu_kernel<T>, dim3((unsigned)blocks), dim3(threads), 0, stream,
                                   (const T*)gate_up, parts, n_parts, (size_t)part_stride, (T*)out, inter,
                                   block, total, act));
  return (int)e;
}

TK_API int tk_unary_act(const void* x, const float* parts, int n_parts, long long part_stride, void* out,
                        long long total, int dtype, int act, cudaStream_t stream) {
  if (total <= 0) return 0;
  if ((x == nullptr) == (parts == nullptr) || act < 0 || act > 3) return (int)cudaErrorInvalidValue;
  size_t blocks = ((size_t)total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  cudaError_t e = cudaSuccess;
  TK_DISPATCH_DTYPE(dtype, T, e = tk::launch(tk::unary_act_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, stream,
                                             (const T*)x, parts, n_parts, (size_t)part_stride, (T*)out, (size_t)total,
                                             act));
  return (int)e;
}
