// What follows the two attention maps of a differential attention head: per token and head
//
//   o = a_1 - lambda * a_2;    y = o / sqrt(mean(o^2) + eps) * factor
//
// a: [tokens, 2 heads, v_row], the maps' outputs side by side (the first `dv` elements of a row count); y: rows of
// heads * dv elements.  Differences, mean and scaling are float32, rounded once on store.  A warp takes a head.
#include "common.cuh"
#include "stacked_input.cuh"

namespace tk {

constexpr int kMapWarps = 4;
constexpr int kMapMaxDim = 512;

// kVec: four neighbouring elements at a time (dv and v_row multiples of 4).
template <typename T, bool kVec>
__global__ void map_difference_kernel(const T* __restrict__ a, T* __restrict__ y, long long y_stride, int n_tokens,
                                      int heads, int dv, int v_row, float lambda, float eps, float factor) {
  constexpr int kStep = kVec ? 4 : 1;
  constexpr int kRounds = kMapMaxDim / (32 * kStep);
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * kMapWarps + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * heads) return;
  const int t = (int)(item / heads), h = (int)(item - (long long)t * heads);
  const T* a1 = a + (size_t)item * 2 * v_row;
  const T* a2 = a1 + v_row;
  float o[kRounds][kStep];
  float ss = 0.0f;
#pragma unroll
  for (int k = 0; k < kRounds; ++k) {
    const int e = (lane + 32 * k) * kStep;
    if (e >= dv) continue;
    if constexpr (kVec) {
      const float4 u = ld4<T>(a1 + e), w = ld4<T>(a2 + e);
      o[k][0] = u.x - lambda * w.x; o[k][1] = u.y - lambda * w.y;
      o[k][2] = u.z - lambda * w.z; o[k][3] = u.w - lambda * w.w;
    } else {
      o[k][0] = to_f32<T>(a1[e]) - lambda * to_f32<T>(a2[e]);
    }
#pragma unroll
    for (int i = 0; i < kStep; ++i) ss += o[k][i] * o[k][i];
  }
  const float f = rsqrtf(warp_sum(ss) / (float)dv + eps) * factor;
  T* dst = y + (size_t)t * y_stride + (size_t)h * dv;
#pragma unroll
  for (int k = 0; k < kRounds; ++k) {
    const int e = (lane + 32 * k) * kStep;
    if (e >= dv) continue;
    if constexpr (kVec) st4<T>(dst + e, make_float4(o[k][0] * f, o[k][1] * f, o[k][2] * f, o[k][3] * f));
    else dst[e] = from_f32<T>(o[k][0] * f);
  }
}

}  // namespace tk

TK_API int tk_map_difference(const void* a, void* y, long long y_stride, int n_tokens, int heads, int dv, int v_row,
                             float lambda, float eps, float factor, int dtype, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (a == nullptr || y == nullptr || heads < 1 || dv < 1 || dv > tk::kMapMaxDim || v_row < dv) return (int)cudaErrorInvalidValue;
  const long long items = (long long)n_tokens * heads;
  const dim3 grid((unsigned)((items + tk::kMapWarps - 1) / tk::kMapWarps)), block(tk::kMapWarps * 32);
  cudaError_t e = cudaSuccess;
  if (dv % 4 == 0 && v_row % 4 == 0 && y_stride % 4 == 0 && (((uintptr_t)a | (uintptr_t)y) & 15) == 0) {
    TK_DISPATCH_DTYPE(dtype, T, (e = tk::launch(tk::map_difference_kernel<T, true>, grid, block, 0, stream, (const T*)a, (T*)y,
                                                y_stride, n_tokens, heads, dv, v_row, lambda, eps, factor)));
  } else {
    TK_DISPATCH_DTYPE(dtype, T, (e = tk::launch(tk::map_difference_kernel<T, false>, grid, block, 0, stream, (const T*)a, (T*)y,
                                                y_stride, n_tokens, heads, dv, v_row, lambda, eps, factor)));
  }
  return (int)e;
}
