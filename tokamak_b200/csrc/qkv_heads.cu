// Preparation of queries, keys and values head by head, with the options that several attention
// mixers share:
//
//   biases             z <- z + b                                   (q, k, v; each may be absent)
//   head norm          x <- x / sqrt(mean_head(x^2) + eps) * w      (q and k; w of one head's size, shared by all
//                                                                    heads, or absent: unit norm); before the
//                                                                    rotation, or after it (norm_after)
//   query temperature  q <- q * (1 + coef * ln(floor((p + 1) / every) + 1))   at position p
//   rotation           over the first `rotary_dim` elements of every q and k head, either of neighbouring
//                      pairs (2i, 2i + 1) or of halves (i, i + rotary_dim / 2); the pair (u, w) at angle a
//                      becomes (u cos a - w sin a, w cos a + u sin a)
//   values from keys   v = the key projection (with its bias) as it was before norm and rotation; the
//                      projection then has no value columns
//
//   maps               a head's query and key are `maps` pieces of k_dim elements, each normed and rotated like a
//                      head of its own.  The key row holds the pieces one after the other; every query piece
//                      goes to a row of its own, at its key piece's place and with zeros elsewhere, so that its
//                      product with the key row is the product of the two pieces
//   stored rows        key (and query) rows of k_row >= maps * k_dim and value rows of v_row >= v_dim elements,
//                      the rest zero (attention kernels that are built for a few row sizes)
//
// and the write of keys and values into their pages.  Everything is float32 and rounded once on store.
// One warp per (token, head); a row of the input is a stacked projection (activation type or float32
// partial sums) in which the queries, keys and values start at q_off, k_off and v_off.
#include "common.cuh"
#include "stacked_input.cuh"

namespace tk {

constexpr int kHeadsWarps = 4;
constexpr int kHeadsMaxDim = 512;

struct QkvHeadsParams {
  StackedInput in;
  int q_off, k_off, v_off;                  // v_off < 0: values from keys
  const float* q_bias; const float* k_bias; const float* v_bias;
  const float* q_norm; const float* k_norm; // [k_dim] or null
  int head_norm;                            // 0: no norm
  int norm_after;                           // the norm follows the rotation
  float eps;
  const float2* rope_table;                 // [n_tokens, rotary_dim / 2] (cos, sin) or null
  int rotary_dim, halves;
  float temp_coef; int temp_every;          // temp_every <= 0: no temperature
  void* q_out;                              // [n_tokens, n_q_heads, k_row]
  void* k_cache;                            // [num_pages, n_kv_heads, page_size, k_row]
  void* v_cache;                            // [num_pages, n_kv_heads, page_size, v_row]
  const int* positions; const int* tok_req; const int* req_slot; const int* block_table;
  const int* req_q_len; const int* req_kv_len;
  int* err;
  int n_tokens, n_reqs, n_q_heads, n_kv_heads, k_dim, v_dim, page_size, max_pages, num_pages;
  int maps, k_row, v_row;                   // n_q_heads counts the pieces of the queries, n_kv_heads the key rows
};

template <typename T>
__global__ void qkv_heads_kernel(QkvHeadsParams p) {
  __shared__ float s_head[kHeadsWarps][kHeadsMaxDim];
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int own_v = p.v_off >= 0 ? p.n_kv_heads : 0;
  const int k_heads = p.n_kv_heads * p.maps;
  const int heads_total = p.n_q_heads + k_heads + own_v;
  const int t = blockIdx.x;
  const int h = blockIdx.y * kHeadsWarps + warp;
  if (h >= heads_total) return;
  int kind, head;     // 0 = q, 1 = k, 2 = v
  if (h < p.n_q_heads) { kind = 0; head = h; }
  else if (h < p.n_q_heads + k_heads) { kind = 1; head = h - p.n_q_heads; }
  else { kind = 2; head = h - p.n_q_heads - k_heads; }
  const int d = kind == 2 ? p.v_dim : p.k_dim;
  const int col = (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + head * d;
  const float* bias = kind == 0 ? p.q_bias : kind == 1 ? p.k_bias : p.v_bias;
  const size_t src = (size_t)t * p.in.row_stride + col;
  const int pos = p.positions[t];
  if (pos < 0) { if (lane == 0) set_error(p.err, kErrPosition, t, pos, 0); return; }

  T* dst = nullptr;
  T* dst_v = nullptr;          // values from keys: the same head of the value pages
  int zero_rows = 0;
  // this warp's part of the stored row: [off, off + d), the row's rest behind the last piece, and all of a query's row
  const int row_len = kind == 2 ? p.v_row : p.k_row;
  const int piece = kind == 2 ? 0 : head % p.maps, off = piece * d;
  const int tail = kind == 2 || piece == p.maps - 1 ? row_len - off : d;
  if (kind == 0) {
    dst = (T*)p.q_out + ((size_t)t * p.n_q_heads + head) * row_len;
  } else {
    const int r = p.tok_req[t];
    if (r < 0 || r >= p.n_reqs) { if (lane == 0) set_error(p.err, kErrRequest, t, r, p.n_reqs); return; }
    const int pidx = pos / p.page_size;
    const int slot = pos - pidx * p.page_size;
    const int page = (pidx < p.max_pages) ? p.block_table[(size_t)p.req_slot[r] * p.max_pages + pidx] : -1;
    if (page < 0 || page >= p.num_pages) { if (lane == 0) set_error(p.err, kErrPage, t, pidx, page); return; }
    const size_t row = ((size_t)page * p.n_kv_heads + (kind == 1 ? head / p.maps : head)) * p.page_size + slot;
    dst = (T*)(kind == 1 ? p.k_cache : p.v_cache) + row * row_len;
    if (kind == 1 && p.v_off < 0) dst_v = (T*)p.v_cache + row * p.v_row;
    // the request's last token of this step clears the rest of a page that was begun in this step, so
    // that a live page never holds stale values behind the last position
    if (p.req_kv_len != nullptr) {
      const int kv_len = p.req_kv_len[r], q_len = p.req_q_len[r];
      if (pos == kv_len - 1 && pos - slot >= kv_len - q_len) zero_rows = p.page_size - 1 - slot;
    }
  }
  for (int z = 1; z <= zero_rows; ++z) {
    for (int e = lane; e < tail; e += 32) {
      dst[(size_t)z * row_len + off + e] = from_f32<T>(0.0f);
      if (dst_v != nullptr) dst_v[(size_t)z * row_len + e] = from_f32<T>(0.0f);
    }
  }
  if (kind == 0) {
    for (int e = lane; e < off; e += 32) dst[e] = from_f32<T>(0.0f);
    for (int e = off + d + lane; e < row_len; e += 32) dst[e] = from_f32<T>(0.0f);
  } else {
    for (int e = d + lane; e < tail; e += 32) {
      dst[off + e] = from_f32<T>(0.0f);
      if (dst_v != nullptr) dst_v[e] = from_f32<T>(0.0f);
    }
  }
  dst += off;

  float* x = s_head[warp];
  float ss = 0.0f;
  for (int e = lane; e < d; e += 32) {
    const float v = stacked_ld<T>(p.in, src + e) + (bias != nullptr ? bias[head * d + e] : 0.0f);
    x[e] = v;
    ss += v * v;
    if (kind == 2) dst[e] = from_f32<T>(v);
    if (dst_v != nullptr) dst_v[e] = from_f32<T>(v);
  }
  if (kind == 2) return;
  float factor = 1.0f, last = 1.0f;        // in front of the rotation, behind it
  if (p.head_norm && !p.norm_after) factor = rsqrtf(warp_sum(ss) / (float)d + p.eps);
  if (kind == 0 && p.temp_every > 0) {
    (p.norm_after ? last : factor) *= 1.0f + p.temp_coef * logf(floorf((float)(pos + 1) / (float)p.temp_every) + 1.0f);
  }
  const float* w_norm = p.head_norm ? (kind == 0 ? p.q_norm : p.k_norm) : nullptr;
  const float* w = p.norm_after ? nullptr : w_norm;
  __syncwarp();
  const int r = p.rope_table != nullptr ? p.rotary_dim : 0, half = r >> 1;
  const float2* tab = p.rope_table + (size_t)t * half;
  float kept[kHeadsMaxDim / 32];
  float ss_after = 0.0f;
#pragma unroll
  for (int k = 0; k < kHeadsMaxDim / 32; ++k) {
    const int e = lane + 32 * k;
    kept[k] = 0.0f;
    if (e >= d) continue;
    float v = x[e] * factor * (w != nullptr ? w[e] : 1.0f);
    if (e < r) {
      int partner, idx; bool first;
      if (p.halves) { first = e < half; partner = first ? e + half : e - half; idx = first ? e : e - half; }
      else { first = !(e & 1); partner = e ^ 1; idx = e >> 1; }
      const float o = x[partner] * factor * (w != nullptr ? w[partner] : 1.0f);
      const float2 cs = tab[idx];
      v = first ? v * cs.x - o * cs.y : v * cs.x + o * cs.y;
    }
    if (!p.norm_after) { dst[e] = from_f32<T>(v); continue; }
    kept[k] = v;
    ss_after += v * v;
  }
  if (!p.norm_after) return;
  if (p.head_norm) last *= rsqrtf(warp_sum(ss_after) / (float)d + p.eps);
#pragma unroll
  for (int k = 0; k < kHeadsMaxDim / 32; ++k) {
    const int e = lane + 32 * k;
    if (e < d) dst[e] = from_f32<T>(kept[k] * last * (w_norm != nullptr ? w_norm[e] : 1.0f));
  }
}

// The same with 16-byte accesses, for head sizes, column offsets and row lengths that are multiples of 4: a lane
// keeps up to four pieces of four elements of its head in registers; rotation partners are read from the
// warp's copy of the head in shared memory.  Sums and products are formed as in the kernel above.
template <typename T>
__global__ void qkv_heads_vec_kernel(QkvHeadsParams p) {
  __shared__ __align__(16) float s_head[kHeadsWarps][kHeadsMaxDim];
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int own_v = p.v_off >= 0 ? p.n_kv_heads : 0;
  const int k_heads = p.n_kv_heads * p.maps;
  const int heads_total = p.n_q_heads + k_heads + own_v;
  const int t = blockIdx.x;
  const int h = blockIdx.y * kHeadsWarps + warp;
  if (h >= heads_total) return;
  int kind, head;     // 0 = q, 1 = k, 2 = v
  if (h < p.n_q_heads) { kind = 0; head = h; }
  else if (h < p.n_q_heads + k_heads) { kind = 1; head = h - p.n_q_heads; }
  else { kind = 2; head = h - p.n_q_heads - k_heads; }
  const int d = kind == 2 ? p.v_dim : p.k_dim;
  const int col = (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + head * d;
  const float* bias = kind == 0 ? p.q_bias : kind == 1 ? p.k_bias : p.v_bias;
  const size_t src = (size_t)t * p.in.row_stride + col;
  const int pos = p.positions[t];
  if (pos < 0) { if (lane == 0) set_error(p.err, kErrPosition, t, pos, 0); return; }

  T* dst = nullptr;
  T* dst_v = nullptr;
  int zero_rows = 0;
  // this warp's part of the stored row: [off, off + d), the row's rest behind the last piece, and all of a query's row
  const int row_len = kind == 2 ? p.v_row : p.k_row;
  const int piece = kind == 2 ? 0 : head % p.maps, off = piece * d;
  const int tail = kind == 2 || piece == p.maps - 1 ? row_len - off : d;
  if (kind == 0) {
    dst = (T*)p.q_out + ((size_t)t * p.n_q_heads + head) * row_len;
  } else {
    const int r = p.tok_req[t];
    if (r < 0 || r >= p.n_reqs) { if (lane == 0) set_error(p.err, kErrRequest, t, r, p.n_reqs); return; }
    const int pidx = pos / p.page_size;
    const int slot = pos - pidx * p.page_size;
    const int page = (pidx < p.max_pages) ? p.block_table[(size_t)p.req_slot[r] * p.max_pages + pidx] : -1;
    if (page < 0 || page >= p.num_pages) { if (lane == 0) set_error(p.err, kErrPage, t, pidx, page); return; }
    const size_t row = ((size_t)page * p.n_kv_heads + (kind == 1 ? head / p.maps : head)) * p.page_size + slot;
    dst = (T*)(kind == 1 ? p.k_cache : p.v_cache) + row * row_len;
    if (kind == 1 && p.v_off < 0) dst_v = (T*)p.v_cache + row * p.v_row;
    if (p.req_kv_len != nullptr) {
      const int kv_len = p.req_kv_len[r], q_len = p.req_q_len[r];
      if (pos == kv_len - 1 && pos - slot >= kv_len - q_len) zero_rows = p.page_size - 1 - slot;
    }
  }
  const int chunks = d >> 2;
  const float4 zero4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  for (int z = 1; z <= zero_rows; ++z) {
    for (int i = lane; i < tail >> 2; i += 32) {
      st4<T>(dst + (size_t)z * row_len + off + 4 * i, zero4);
      if (dst_v != nullptr) st4<T>(dst_v + (size_t)z * row_len + 4 * i, zero4);
    }
  }
  if (kind == 0) {
    for (int e = 4 * lane; e < row_len; e += 128) {
      if (e < off || e >= off + d) st4<T>(dst + e, zero4);
    }
  } else {
    for (int e = d + 4 * lane; e < tail; e += 128) {
      st4<T>(dst + off + e, zero4);
      if (dst_v != nullptr) st4<T>(dst_v + e, zero4);
    }
  }
  dst += off;

  float* x = s_head[warp];
  float4 own[4];
  float ss = 0.0f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int i = lane + 32 * k;
    own[k] = zero4;
    if (i >= chunks) continue;
    float4 v = stacked_ld4<T>(p.in, src + 4 * i);
    if (bias != nullptr) {
      const float4 b = *reinterpret_cast<const float4*>(bias + head * d + 4 * i);
      v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
    }
    own[k] = v;
    *reinterpret_cast<float4*>(x + 4 * i) = v;
    ss += v.x * v.x; ss += v.y * v.y; ss += v.z * v.z; ss += v.w * v.w;
    if (kind == 2) st4<T>(dst + 4 * i, v);
    if (dst_v != nullptr) st4<T>(dst_v + 4 * i, v);
  }
  if (kind == 2) return;
  float factor = 1.0f, last = 1.0f;        // in front of the rotation, behind it
  if (p.head_norm && !p.norm_after) factor = rsqrtf(warp_sum(ss) / (float)d + p.eps);
  if (kind == 0 && p.temp_every > 0) {
    (p.norm_after ? last : factor) *= 1.0f + p.temp_coef * logf(floorf((float)(pos + 1) / (float)p.temp_every) + 1.0f);
  }
  const float* w_norm = p.head_norm ? (kind == 0 ? p.q_norm : p.k_norm) : nullptr;
  const float* w = p.norm_after ? nullptr : w_norm;
  __syncwarp();
  const int r = p.rope_table != nullptr ? p.rotary_dim : 0, half = r >> 1;
  const float2* tab = p.rope_table + (size_t)t * half;
  float ss_after = 0.0f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int i = lane + 32 * k;
    if (i >= chunks) continue;
    const float4 w4 = w != nullptr ? *reinterpret_cast<const float4*>(w + 4 * i) : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
    float v[4] = {own[k].x * factor * w4.x, own[k].y * factor * w4.y, own[k].z * factor * w4.z, own[k].w * factor * w4.w};
    if (4 * i < r) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int e = 4 * i + j;
        if (e < r) {
          int partner, idx; bool first;
          if (p.halves) { first = e < half; partner = first ? e + half : e - half; idx = first ? e : e - half; }
          else { first = !(e & 1); partner = e ^ 1; idx = e >> 1; }
          const float o = x[partner] * factor * (w != nullptr ? w[partner] : 1.0f);
          const float2 cs = tab[idx];
          v[j] = first ? v[j] * cs.x - o * cs.y : v[j] * cs.x + o * cs.y;
        }
      }
    }
    own[k] = make_float4(v[0], v[1], v[2], v[3]);
    if (!p.norm_after) st4<T>(dst + 4 * i, own[k]);
    ss_after += v[0] * v[0]; ss_after += v[1] * v[1]; ss_after += v[2] * v[2]; ss_after += v[3] * v[3];
  }
  if (!p.norm_after) return;
  if (p.head_norm) last *= rsqrtf(warp_sum(ss_after) / (float)d + p.eps);
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int i = lane + 32 * k;
    if (i >= chunks) continue;
    float4 v = make_float4(own[k].x * last, own[k].y * last, own[k].z * last, own[k].w * last);
    if (w_norm != nullptr) {
      const float4 w4 = *reinterpret_cast<const float4*>(w_norm + 4 * i);
      v.x *= w4.x; v.y *= w4.y; v.z *= w4.z; v.w *= w4.w;
    }
    st4<T>(dst + 4 * i, v);
  }
}

// The same for pieces of up to 128 elements (sizes, offsets and row lengths multiples of 4, the rotated part in whole
// fours per half, values of their own): kLanes lanes take a piece, four elements each, so that a warp works on 32 /
// kLanes pieces (a value head longer than that is cut: nothing passes between its elements), and rotation partners and sums of squares pass between lanes instead of through shared memory.
template <typename T, int kLanes>
__global__ void __launch_bounds__(kHeadsWarps * 32) qkv_heads_lanes_kernel(QkvHeadsParams p) {
  constexpr int kPieces = 32 / kLanes;
  pdl_trigger();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int first = (blockIdx.y * kHeadsWarps + warp) * kPieces;
  const int v_cuts = (p.v_dim + 4 * kLanes - 1) / (4 * kLanes);
  const int k_heads = p.n_kv_heads * p.maps, heads_total = p.n_q_heads + k_heads + p.n_kv_heads * v_cuts;
  if (first >= heads_total) return;                    // the whole warp
  const int t = blockIdx.x;
  const int h = min(first + lane / kLanes, heads_total - 1);
  const bool real = first + lane / kLanes < heads_total;
  const int kind = h < p.n_q_heads ? 0 : h < p.n_q_heads + k_heads ? 1 : 2;       // 0 = q, 1 = k, 2 = v
  const int v_item = h - p.n_q_heads - k_heads;
  const int head = kind == 0 ? h : kind == 1 ? h - p.n_q_heads : v_item / v_cuts;
  const int d = kind == 2 ? p.v_dim : p.k_dim;
  const int c = lane % kLanes, e = 4 * (c + (kind == 2 ? (v_item % v_cuts) * kLanes : 0));
  const bool live = real && e < d;
  const int r = p.rope_table != nullptr && kind != 2 ? p.rotary_dim : 0, half = r >> 1;
  pdl_wait();
  float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if (live) {
    x = stacked_ld4<T>(p.in, (size_t)t * p.in.row_stride + (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + head * d + e);
  }
  // the angles of these four elements: four pairs (halves) or two (neighbours)
  float4 cs0 = make_float4(1.0f, 0.0f, 1.0f, 0.0f), cs1 = cs0;
  const bool turned = e < r;
  if (turned) {
    const float2* tab = p.rope_table + (size_t)t * half;
    if (p.halves) {
      const int i = e < half ? e : e - half;
      cs0 = *reinterpret_cast<const float4*>(tab + i); cs1 = *reinterpret_cast<const float4*>(tab + i + 2);
    } else {
      const float2 a = tab[e >> 1], b = tab[(e >> 1) + 1];
      cs0 = make_float4(a.x, a.y, b.x, b.y);
    }
  }
  const int pos = p.positions[t];
  bool ok = real;
  if (pos < 0) { if (lane == 0) set_error(p.err, kErrPosition, t, pos, 0); return; }      // the whole warp
  const int row_len = kind == 2 ? p.v_row : p.k_row;
  const int piece = kind == 2 ? 0 : head % p.maps, off = piece * d;
  const int tail = kind == 2 || piece == p.maps - 1 ? row_len - off : d;
  T* dst = (T*)p.q_out + ((size_t)t * p.n_q_heads + (kind == 0 ? head : 0)) * row_len;
  int zero_rows = 0;
  if (kind != 0) {
    const int req = p.tok_req[t];
    const int pidx = pos / p.page_size, slot = pos - pidx * p.page_size;
    int page = -1;
    if (req < 0 || req >= p.n_reqs) {
      if (lane % kLanes == 0) set_error(p.err, kErrRequest, t, req, p.n_reqs);
    } else {
      page = pidx < p.max_pages ? p.block_table[(size_t)p.req_slot[req] * p.max_pages + pidx] : -1;
      if (page < 0 || page >= p.num_pages) { if (lane % kLanes == 0) set_error(p.err, kErrPage, t, pidx, page); page = -1; }
    }
    ok = ok && page >= 0;
    const size_t row = ((size_t)max(page, 0) * p.n_kv_heads + (kind == 1 ? head / p.maps : head)) * p.page_size + slot;
    dst = (T*)(kind == 1 ? p.k_cache : p.v_cache) + row * row_len;
    // the request's last token of this step clears the rest of a page that was begun in this step
    if (ok && p.req_kv_len != nullptr) {
      const int kv_len = p.req_kv_len[req], q_len = p.req_q_len[req];
      if (pos == kv_len - 1 && pos - slot >= kv_len - q_len) zero_rows = p.page_size - 1 - slot;
    }
  }
  if (live) {
    const float* bias = kind == 0 ? p.q_bias : kind == 1 ? p.k_bias : p.v_bias;
    if (bias != nullptr) {
      const float4 b = *reinterpret_cast<const float4*>(bias + head * d + e);
      x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
    }
  }
  auto piece_sum = [&](float v) {
#pragma unroll
    for (int o = kLanes / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
  };
  auto scale4 = [](float4 v, float f) { return make_float4(v.x * f, v.y * f, v.z * f, v.w * f); };
  const float* w = p.head_norm && kind != 2 ? (kind == 0 ? p.q_norm : p.k_norm) : nullptr;
  auto norm = [&]() {
    const float f = rsqrtf(piece_sum((x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w)) / (float)d + p.eps);
    if (kind == 2) return;
    x = scale4(x, f);
    if (w != nullptr && live) {
      const float4 g = *reinterpret_cast<const float4*>(w + e);
      x.x *= g.x; x.y *= g.y; x.z *= g.z; x.w *= g.w;
    }
  };
  if (p.head_norm && !p.norm_after) norm();
  if (p.rope_table != nullptr) {
    if (p.halves) {
      const int q4 = half >> 2;
      const int from = (lane - c) + (e < half ? c + q4 : c - q4);
      const int src = turned ? from : lane;
      float4 o;
      o.x = __shfl_sync(0xffffffffu, x.x, src); o.y = __shfl_sync(0xffffffffu, x.y, src);
      o.z = __shfl_sync(0xffffffffu, x.z, src); o.w = __shfl_sync(0xffffffffu, x.w, src);
      if (turned) {
        const float s = e < half ? -1.0f : 1.0f;
        x = make_float4(x.x * cs0.x + s * (o.x * cs0.y), x.y * cs0.z + s * (o.y * cs0.w), x.z * cs1.x + s * (o.z * cs1.y),
                        x.w * cs1.z + s * (o.w * cs1.w));
      }
    } else if (turned) {
      x = make_float4(x.x * cs0.x - x.y * cs0.y, x.y * cs0.x + x.x * cs0.y, x.z * cs0.z - x.w * cs0.w, x.w * cs0.z + x.z * cs0.w);
    }
  }
  if (p.head_norm && p.norm_after) norm();
  if (kind == 0 && p.temp_every > 0) x = scale4(x, 1.0f + p.temp_coef * logf(floorf((float)(pos + 1) / (float)p.temp_every) + 1.0f));
  if (!ok) return;
  const float4 zero4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if (live) st4<T>(dst + off + e, x);
  if (kind == 0) {
    for (int i = e; i < row_len; i += 4 * kLanes) {
      if (i < off || i >= off + d) st4<T>(dst + i, zero4);
    }
    return;
  }
  const int step = 4 * kLanes * (kind == 2 ? v_cuts : 1);
  for (int i = d + e; i < tail; i += step) st4<T>(dst + off + i, zero4);
  for (int z = 1; z <= zero_rows; ++z) {
    for (int i = e; i < tail; i += step) st4<T>(dst + (size_t)z * row_len + off + i, zero4);
  }
}

}  // namespace tk

TK_API int tk_qkv_heads(const void* x, const float* parts, int n_parts, long long part_stride, int row_stride,
                        int q_off, int k_off, int v_off, const float* q_bias, const float* k_bias,
                        const float* v_bias, const float* q_norm, const float* k_norm, int head_norm, float eps,
                        const float* rope_table, int rotary_dim, int halves, float temp_coef, int temp_every,
                        void* q_out, void* k_cache, void* v_cache, const int* positions, const int* tok_req,
                        const int* req_slot, const int* block_table, const int* req_q_len, const int* req_kv_len,
                        int* err, int n_tokens, int n_reqs, int n_q_heads, int n_kv_heads, int k_dim, int v_dim,
                        int page_size, int max_pages, int num_pages, int norm_after, int maps, int k_row, int v_row,
                        int dtype, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (maps < 1 || n_q_heads % maps || k_row < maps * k_dim || v_row < v_dim ||
      (v_off < 0 && (maps != 1 || k_row != v_row))) {
    return (int)cudaErrorInvalidValue;
  }
  if ((x == nullptr) == (parts == nullptr) || n_q_heads < 1 || n_kv_heads < 1 || k_dim < 1 || v_dim < 1 ||
      k_dim > tk::kHeadsMaxDim || v_dim > tk::kHeadsMaxDim || rotary_dim < 0 || rotary_dim > k_dim ||
      (rotary_dim & 1) || (v_off < 0 && v_dim != k_dim)) {
    return (int)cudaErrorInvalidValue;
  }
  tk::QkvHeadsParams p;
  p.in.x = x; p.in.parts = parts; p.in.n_parts = n_parts; p.in.row_stride = row_stride; p.in.part_stride = part_stride;
  p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.q_bias = q_bias; p.k_bias = k_bias; p.v_bias = v_bias;
  p.q_norm = q_norm; p.k_norm = k_norm; p.head_norm = head_norm; p.eps = eps;
  p.rope_table = (const float2*)rope_table; p.rotary_dim = rotary_dim; p.halves = halves;
  p.temp_coef = temp_coef; p.temp_every = temp_every;
  p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache;
  p.positions = positions; p.tok_req = tok_req; p.req_slot = req_slot; p.block_table = block_table;
  p.req_q_len = req_q_len; p.req_kv_len = req_kv_len; p.err = err;
  p.n_tokens = n_tokens; p.n_reqs = n_reqs; p.n_q_heads = n_q_heads; p.n_kv_heads = n_kv_heads; p.k_dim = k_dim;
  p.v_dim = v_dim; p.page_size = page_size; p.max_pages = max_pages; p.num_pages = num_pages;
  p.norm_after = norm_after; p.maps = maps; p.k_row = k_row; p.v_row = v_row;
  const int heads_total = n_q_heads + n_kv_heads * maps + (v_off >= 0 ? n_kv_heads : 0);
  const dim3 grid((unsigned)n_tokens, (unsigned)((heads_total + tk::kHeadsWarps - 1) / tk::kHeadsWarps));
  cudaError_t e = cudaSuccess;
  const bool vec = k_dim % 4 == 0 && v_dim % 4 == 0 && k_row % 4 == 0 && v_row % 4 == 0 && row_stride % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 &&
                   (v_off < 0 || v_off % 4 == 0);
  if (vec && k_dim <= 128 && v_off >= 0 && (rope_table == nullptr || rotary_dim % (halves ? 8 : 4) == 0) &&
      ((uintptr_t)rope_table & 15) == 0) {
    const int lanes = k_dim <= 32 ? 8 : k_dim <= 64 ? 16 : 32, per_block = tk::kHeadsWarps * (32 / lanes);
    const int items = n_q_heads + n_kv_heads * maps + n_kv_heads * ((v_dim + 4 * lanes - 1) / (4 * lanes));
    const dim3 g((unsigned)n_tokens, (unsigned)((items + per_block - 1) / per_block));
#define TK_QKV_LANES(L) \
    TK_DISPATCH_DTYPE(dtype, T, (e = tk::launch(tk::qkv_heads_lanes_kernel<T, L>, g, dim3(tk::kHeadsWarps * 32), 0, stream, p)))
    if (lanes == 8) { TK_QKV_LANES(8); } else if (lanes == 16) { TK_QKV_LANES(16); } else { TK_QKV_LANES(32); }
#undef TK_QKV_LANES
    return (int)e;
  }
  if (vec) {
    TK_DISPATCH_DTYPE(dtype, T, e = tk::launch(tk::qkv_heads_vec_kernel<T>, grid, dim3(tk::kHeadsWarps * 32), 0, stream, p));
    return (int)e;
  }
  TK_DISPATCH_DTYPE(dtype, T, e = tk::launch(tk::qkv_heads_kernel<T>, grid, dim3(tk::kHeadsWarps * 32), 0, stream, p));
  return (int)e;
}
