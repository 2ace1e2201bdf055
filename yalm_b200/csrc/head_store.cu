// What follows a q/k(/v) product whose heads are each on their own (parts/exact_attention.py), a warp per
// head of one token: sums the product's split-K slices; norms a head of q or k over its own root mean
// square times a weight shared by the heads; turns its first `dims` features in pairs (i, i + dims/2) by the
// step's cosines and sines; multiplies q by a temperature that grows with the position,
// 1 + coef ln(floor((pos + 1) / every) + 1); and writes q, this step's keys and values and the cache rows in
// the storage type.  Keys and values have sizes of their own.  Without v columns the values are the keys as
// projected, before the norm.  Norms, angles and temperatures are 32-bit.
#include "api.h"
#include "common.cuh"

namespace yalm {

struct HeadStore {
  const float* qkv;            // slices [n_partials][tokens][row], row = H dk + G dk (+ G dv)
  int n_partials;
  long long partial_stride;
  const float *q_norm, *k_norm;        // [dk] (zero beyond the true size) or null
  float eps, true_dk;
  const float2* table;         // [tokens][dims / 2] (cos, sin) or null
  int dims;
  float temp_coef, temp_every; // temp_every <= 0: no temperature
  const int *token_seq, *q_start, *seq_slot, *slot_pos;
  void *q_out, *kv_step, *k_cache, *v_cache;
  int H, G, dk, dv, has_v, capacity, write_cache;
  const int* page_table;
  int pps, n_pages;
};

template <int W>
__device__ __forceinline__ void head_load(const float* __restrict__ p, int n, long long stride, float* v) {
  if constexpr (W == 4) {
    v[0] = v[1] = v[2] = v[3] = 0.f;
    for (int s0 = 0; s0 < n; s0 += 4) {
      float4 t[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        t[j] = s0 + j < n ? *reinterpret_cast<const float4*>(p + (size_t)(s0 + j) * stride) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < 4; ++j) { v[0] += t[j].x; v[1] += t[j].y; v[2] += t[j].z; v[3] += t[j].w; }
    }
  } else {
    v[0] = sum_slices(p, n, stride);
  }
}
template <typename T, int W>
__device__ __forceinline__ void head_put(T* __restrict__ p, const float* v) {
  if constexpr (W == 4 && sizeof(T) == 2) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack2<T>(v[0], v[1]), pack2<T>(v[2], v[3]));
  } else if constexpr (W == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    p[0] = from_float<T>(v[0]);
  }
}

// An item is W features and, where they turn, their W partners; E items per lane.  grid (tokens, units / 8)
template <typename T, int W, int E>
__global__ void __launch_bounds__(256) head_store_kernel(HeadStore a) {
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5);                // q heads, k heads, v heads
  if (unit >= a.H + a.G * (a.has_v ? 2 : 1)) return;
  const int b = a.token_seq[t], slot = a.seq_slot[b], qs = a.q_start[b], ql = a.q_start[b + 1] - qs;
  const int past = a.slot_pos[slot], pos = past + (t - qs);
  const bool keep = a.write_cache && pos >= past + ql - a.capacity;
  const bool is_q = unit < a.H, is_v = unit >= a.H + a.G;
  const int head = is_q ? unit : is_v ? unit - a.H - a.G : unit - a.H;
  const int size = is_v ? a.dv : a.dk;
  const int nq = a.H * a.dk, nk = a.G * a.dk, row = nq + nk + (a.has_v ? a.G * a.dv : 0);
  const int at = is_q ? head * a.dk : is_v ? nq + nk + head * a.dv : nq + head * a.dk;
  const float* norm = is_v ? nullptr : is_q ? a.q_norm : a.k_norm;
  const int half = is_v ? 0 : a.dims >> 1, pairs = half / W, items = pairs + (size - 2 * half) / W;
  const int step_row = a.G * (a.dk + a.dv), cache_row = pos % a.capacity;
  pdl_wait();
  const float* src = a.qkv + (size_t)t * row + at;
  float v[E][2][W], ss = 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int it = e * 32 + lane;
#pragma unroll
    for (int j = 0; j < W; ++j) v[e][0][j] = v[e][1][j] = 0.f;
    if (it < items) {
      head_load<W>(src + (it < pairs ? it * W : 2 * half + (it - pairs) * W), a.n_partials, a.partial_stride, v[e][0]);
      if (it < pairs) head_load<W>(src + half + it * W, a.n_partials, a.partial_stride, v[e][1]);
    }
#pragma unroll
    for (int j = 0; j < W; ++j) ss += v[e][0][j] * v[e][0][j] + v[e][1][j] * v[e][1][j];
  }
  // where this head's row goes; a key head without v columns also leaves its raw row as the value
  T* out = is_q ? reinterpret_cast<T*>(a.q_out) + ((size_t)t * a.H + head) * a.dk
                : reinterpret_cast<T*>(a.kv_step) + (size_t)t * step_row + (is_v ? nk + head * a.dv : head * a.dk);
  T* cached = nullptr;
  if (!is_q && keep)
    cached = reinterpret_cast<T*>(is_v ? a.v_cache : a.k_cache) +
             kv_row_offset(a.page_table, a.pps, a.n_pages, slot, head, a.G, a.capacity, cache_row, size);
  if (!is_q && !a.has_v) {
    T* vo = reinterpret_cast<T*>(a.kv_step) + (size_t)t * step_row + nk + head * a.dv;
    T* vc = keep ? reinterpret_cast<T*>(a.v_cache) +
                       kv_row_offset(a.page_table, a.pps, a.n_pages, slot, head, a.G, a.capacity, cache_row, a.dv) : nullptr;
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int it = e * 32 + lane;
      if (it >= items) continue;
      const int i0 = it < pairs ? it * W : 2 * half + (it - pairs) * W;
      head_put<T, W>(vo + i0, v[e][0]);
      if (vc != nullptr) head_put<T, W>(vc + i0, v[e][0]);
      if (it < pairs) {
        head_put<T, W>(vo + half + i0, v[e][1]);
        if (vc != nullptr) head_put<T, W>(vc + half + i0, v[e][1]);
      }
    }
  }
  const float r = norm != nullptr ? 1.0f / sqrtf(warp_sum(ss) / a.true_dk + a.eps) : 1.f;
  const float temp = is_q && a.temp_every > 0.f
                         ? 1.0f + a.temp_coef * logf(floorf((float)(pos + 1) / a.temp_every) + 1.0f) : 1.f;
  const float2* cs = a.table != nullptr ? a.table + (size_t)t * (a.dims >> 1) : nullptr;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int it = e * 32 + lane;
    if (it >= items) continue;
    const int i0 = it < pairs ? it * W : 2 * half + (it - pairs) * W;
#pragma unroll
    for (int j = 0; j < W; ++j) {
      if (norm != nullptr) {
        v[e][0][j] *= r * norm[i0 + j];
        if (it < pairs) v[e][1][j] *= r * norm[half + i0 + j];
      }
      if (it < pairs) {
        const float2 c = cs[i0 + j];
        const float lo = rotate_lo(v[e][0][j], v[e][1][j], c.x, c.y);
        v[e][1][j] = rotate_hi(v[e][0][j], v[e][1][j], c.x, c.y) * temp;
        v[e][0][j] = lo * temp;
      } else {
        v[e][0][j] *= temp;
      }
    }
    head_put<T, W>(out + i0, v[e][0]);
    if (cached != nullptr) head_put<T, W>(cached + i0, v[e][0]);
    if (it < pairs) {
      head_put<T, W>(out + half + i0, v[e][1]);
      if (cached != nullptr) head_put<T, W>(cached + half + i0, v[e][1]);
    }
  }
}

}  // namespace yalm

using namespace yalm;

// qkv: float32 slices [n_partials][tokens][H dk + G dk + (has_v ? G dv : 0)]; q_norm, k_norm float32 [dk] or null
// (true_dk: the features that the mean counts); table float32 [tokens][dims / 2][2] or null (dims 0); q_out
// [tokens][H][dk], kv_step [tokens][G dk + G dv], caches with rows of dk and of dv.  dk and dv up to 256; without
// v columns dv == dk.
extern "C" int yalm_head_store(const float* qkv, int n_partials, long long partial_stride, const float* q_norm,
                               const float* k_norm, float eps, int true_dk, const float* table, int dims,
                               float temp_coef, float temp_every, const int* token_seq, const int* q_start,
                               const int* seq_slot, const int* slot_pos, void* q_out, void* kv_step, void* k_cache,
                               void* v_cache, int dtype, int n_tokens, int H, int G, int dk, int dv, int has_v,
                               int capacity, int write_cache, const int* page_table, int pages_per_slot, int n_pages,
                               cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || dk <= 0 || dv <= 0 || dk > 256 || dv > 256 || true_dk <= 0 || true_dk > dk || capacity <= 0 ||
      (!has_v && dv != dk) || dims < 0 || (dims & 1) || dims > dk || (dims > 0 && table == nullptr) ||
      (q_norm == nullptr) != (k_norm == nullptr))
    return -2;
  const HeadStore a = {qkv, n_partials, partial_stride, q_norm, k_norm, eps, (float)true_dk,
                       reinterpret_cast<const float2*>(table), dims, temp_coef, temp_every, token_seq, q_start, seq_slot,
                       slot_pos, q_out, kv_step, k_cache, v_cache, H, G, dk, dv, has_v, capacity, write_cache,
                       page_table, pages_per_slot, n_pages};
  const int units = H + G * (has_v ? 2 : 1);
  const dim3 grid(n_tokens, (units + 7) / 8), block(256);
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && dims % 8 == 0 && (partial_stride & 3) == 0 &&
                   ((((uintptr_t)qkv) | ((uintptr_t)q_out) | ((uintptr_t)kv_step) | ((uintptr_t)k_cache) | ((uintptr_t)v_cache)) & 15) == 0;
#define YALM_HS(T)                                                                       \
  do {                                                                                   \
    if (vec && dk <= 128 && dv <= 128) launch_pdl(head_store_kernel<T, 4, 1>, grid, block, 0, stream, a); \
    else if (vec) launch_pdl(head_store_kernel<T, 4, 2>, grid, block, 0, stream, a);     \
    else launch_pdl(head_store_kernel<T, 1, 8>, grid, block, 0, stream, a);              \
  } while (0)
  if (dtype == DT_F32) YALM_HS(float);
  else if (dtype == DT_BF16) YALM_HS(__nv_bfloat16);
  else if (dtype == DT_F16) YALM_HS(__half);
  else return -3;
#undef YALM_HS
  YALM_LAUNCH_CHECK();
  return 0;
}
