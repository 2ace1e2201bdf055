// Attention over a cached latent: a token leaves one row [c | kr] in the cache, c = norm(Wdkv h)[:rank]
// times a weight, kr the rot_dim rotated features shared by all heads.  Per head the key is
// [Wuk c | kr] and the value Wuv c, so with q = [qa | qr]
//     q . k = (Wuk^T qa) . c + qr . kr,        sum_j p_j v_j = Wuv (sum_j p_j c_j):
// in the absorbed form queries are moved into the latent space once per token and head, the
// attention runs over the cached rows themselves, and the mixed latent is expanded by Wuv
// afterwards.  In the expanded form (whole prompts) Wuk c and Wuv c are one product over the step's
// rows and the queries are only rotated.  The kernels around the attention (latent_attention.cu):
//  * latent_store: sums the down projection's split-K slices, norms c, rotates kr (angle in 32 bits;
//    pairs of neighbours or of halves, cos and sin times a factor), writes the row to this step's
//    buffer (as key and as value), to the cache (the positions that a ring keeps) and, where asked,
//    c alone as a matrix for the expanded form's product;
//  * latent_rotate_q: q = [qa | rot(qr)] in the storage type, for the expanded form;
//  * latent_absorb_q: q' = [Wuk_h^T qa | rot(qr) | 0] per token and head;
//  * latent_expand: out_h = (Wuv_h o_h) * sigmoid(gate), o_h the first `rank` features of the
//    attention's output for head h, or the merge of the partial results of a split attention.
// Sources are columns of one stacked product: a row pitch and a first column each.
#include "api.h"
#include "common.cuh"

namespace yalm {

// float32 slices [n][tokens][row], the columns of interest from p on
struct Cols {
  const float* p;
  int n;
  long long stride;      // between slices
  int row;
};
__device__ __forceinline__ float col(const Cols& a, int t, int c) {
  return sum_slices(a.p + (size_t)t * a.row + c, a.n, a.stride);
}

template <int V> struct Int { static constexpr int value = V; };

struct Rotation {
  const float* freq;     // [rd / 2]
  int rd, halves;        // pairs (i, i + rd/2), else (2i, 2i + 1)
  float mult;            // on cos and sin
};
// feature e of the rotated part at position pos; load(e) gives the part before the rotation
template <typename Load>
__device__ __forceinline__ float rotated(const Rotation& r, int e, int pos, Load load) {
  const int half = r.rd >> 1;
  const bool low = r.halves ? e < half : !(e & 1);
  const int pair = r.halves ? (low ? e : e - half) : e >> 1;
  const int other = r.halves ? (low ? e + half : e - half) : e ^ 1;
  const float ang = (float)pos * r.freq[pair];
  const float c = cosf(ang) * r.mult, s = sinf(ang) * r.mult;
  const float me = load(e), ot = load(other);
  return low ? rotate_lo(me, ot, c, s) : rotate_hi(ot, me, c, s);
}

struct Seqs {
  const int *token_seq, *q_start, *seq_slot, *slot_pos;
};
__device__ __forceinline__ int position_of(const Seqs& s, int t) {
  const int b = s.token_seq[t];
  return s.slot_pos[s.seq_slot[b]] + (t - s.q_start[b]);
}

// sigmoid gate of an output feature: mode 1 one logit per head, 2 one per feature
struct Gate {
  Cols z;
  int mode;
};
__device__ __forceinline__ float gated(const Gate& g, int t, int h, int feature, int vdim, float v) {
  if (g.mode == 0) return v;
  const float z = col(g.z, t, g.mode == 1 ? h : h * vdim + feature);
  return v / (1.0f + expf(-z));
}

template <typename T>
__device__ __forceinline__ void put4(T* __restrict__ p, const float* v) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    uint2 u;
    u.x = pack2<T>(v[0], v[1]);
    u.y = pack2<T>(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = u;
  }
}
// four neighbouring columns
__device__ __forceinline__ float4 col4(const Cols& a, int t, int c) {
  const float* p = a.p + (size_t)t * a.row + c;
  float4 v = *reinterpret_cast<const float4*>(p);
  for (int k = 1; k < a.n; ++k) {
    const float4 e = *reinterpret_cast<const float4*>(p + (size_t)k * a.stride);
    v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
  }
  return v;
}

// VEC: everything in multiples of four and 16-byte aligned, a thread takes four neighbouring features
template <typename T, bool VEC>
__global__ void latent_store_kernel(Cols src, const float* __restrict__ c_norm, float eps, Rotation rot, Seqs sq,
                                    T* __restrict__ kv_step, T* __restrict__ cache, T* __restrict__ c_rows,
                                    int rank, int hd, int capacity, int write_cache,
                                    const int* __restrict__ page_table, int pps, int n_pages) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float row_s[];
  __shared__ float scratch[33];
  constexpr int W = VEC ? 4 : 1;
  const int t = blockIdx.x;
  pdl_wait();
  const int row = rank + rot.rd;
  float ss = 0.f;
  for (int i = threadIdx.x * W; i < row; i += blockDim.x * W) {
    if constexpr (VEC) {
      const float4 v = col4(src, t, i);
      *reinterpret_cast<float4*>(row_s + i) = v;
      if (i < rank) ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    } else {
      const float v = col(src, t, i);
      row_s[i] = v;
      if (i < rank) ss += v * v;
    }
  }
  const int b = sq.token_seq[t];
  const int slot = sq.seq_slot[b];
  const int past = sq.slot_pos[slot];
  const int pos = past + (t - sq.q_start[b]);
  // of a step longer than the ring only the last positions stay
  const bool keep = write_cache && pos >= past + (sq.q_start[b + 1] - sq.q_start[b]) - capacity;
  const size_t off = keep ? kv_row_offset(page_table, pps, n_pages, slot, 0, 1, capacity, pos % capacity, hd) : 0;
  const float rs = 1.0f / sqrtf(block_sum(ss, scratch) / (float)rank + eps);
  for (int i = threadIdx.x * W; i < hd; i += blockDim.x * W) {
    float v[W];
#pragma unroll
    for (int j = 0; j < W; ++j) {
      const int f = i + j;
      v[j] = f < rank ? row_s[f] * rs * c_norm[f]
           : f < row ? rotated(rot, f - rank, pos, [&](int e) { return row_s[rank + e]; }) : 0.f;
    }
    if constexpr (VEC) {
      put4<T>(kv_step + (size_t)t * 2 * hd + i, v);
      put4<T>(kv_step + (size_t)t * 2 * hd + hd + i, v);
      if (keep) put4<T>(cache + off + i, v);
      if (c_rows != nullptr && i < rank) put4<T>(c_rows + (size_t)t * rank + i, v);
    } else {
      const T val = from_float<T>(v[0]);
      kv_step[(size_t)t * 2 * hd + i] = val;
      kv_step[(size_t)t * 2 * hd + hd + i] = val;
      if (keep) cache[off + i] = val;
      if (c_rows != nullptr && i < rank) c_rows[(size_t)t * rank + i] = val;
    }
  }
}

// grid (tokens, parts of the heads): a block takes `per` heads of one token, the token's cosines and
// sines once through shared memory
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
latent_rotate_q_kernel(Cols q, Rotation rot, Seqs sq, T* __restrict__ q_out, int H, int dim, int per) {
  pdl_launch_dependents();
  extern __shared__ float cs[];                         // cos [rd/2], sin [rd/2]
  const int t = blockIdx.x;
  const int pos = position_of(sq, t);
  const int half = rot.rd >> 1;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float ang = (float)pos * rot.freq[i];
    cs[i] = cosf(ang) * rot.mult;
    cs[half + i] = sinf(ang) * rot.mult;
  }
  __syncthreads();
  pdl_wait();
  const int qd = dim + rot.rd;
  const int h0 = blockIdx.y * per, h1 = min(H, h0 + per);
  auto turn = [&](int h, int e) {
    const bool low = rot.halves ? e < half : !(e & 1);
    const int pair = rot.halves ? (low ? e : e - half) : e >> 1;
    const int other = rot.halves ? (low ? e + half : e - half) : e ^ 1;
    const float me = col(q, t, h * qd + dim + e), ot = col(q, t, h * qd + dim + other);
    return low ? rotate_lo(me, ot, cs[pair], cs[half + pair]) : rotate_hi(ot, me, cs[pair], cs[half + pair]);
  };
  if constexpr (VEC) {                                  // everything in multiples of four
    T* dst = q_out + (size_t)t * H * qd;
    for (int i = h0 * qd + threadIdx.x * 4; i < h1 * qd; i += blockDim.x * 4) {
      const int h = i / qd, e = i - h * qd - dim;       // e >= 0: feature of the rotated part
      const float4 a = col4(q, t, i);
      float v[4] = {a.x, a.y, a.z, a.w};
      if (e >= 0 && rot.halves) {
        const bool low = e < half;
        const float4 c = col4(q, t, low ? i + half : i - half);
        const float o[4] = {c.x, c.y, c.z, c.w};
        const int p0 = low ? e : e - half;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float cc = cs[p0 + j], sn = cs[half + p0 + j];
          v[j] = low ? rotate_lo(v[j], o[j], cc, sn) : rotate_hi(o[j], v[j], cc, sn);
        }
      } else if (e >= 0) {
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          const int p0 = (e + j) >> 1;
          const float lo = v[j], hi = v[j + 1];
          v[j] = rotate_lo(lo, hi, cs[p0], cs[half + p0]);
          v[j + 1] = rotate_hi(lo, hi, cs[p0], cs[half + p0]);
        }
      }
      put4<T>(dst + i, v);
    }
  } else {
    for (int i = h0 * qd + threadIdx.x; i < h1 * qd; i += blockDim.x) {
      const int h = i / qd, e = i - h * qd;
      q_out[(size_t)t * H * qd + i] = from_float<T>(e < dim ? col(q, t, i) : turn(h, e - dim));
    }
  }
}

// ---- per-head products of few tokens (a decode step): a block takes TOK tokens x 8 CT columns of one
// head.  A thread owns eight neighbouring columns and every (256 / CT)-th row of the head's matrix B [K][N]
// (one 16-byte load feeds 8 TOK multiply-adds); the partial sums of a warp's row groups are added through
// shuffles, those of the warps through shared memory.  x [K][TOK] float32 in shared memory.
constexpr int LT_TOK = 4;              // the most tokens of a block; a step of few tokens takes them one by one
constexpr int LT_ONE = 16;             // up to this many tokens
constexpr int LT_CT_Q = 32, LT_CT_V = 16;      // column threads of the two products (256 and 128 columns)

template <typename T>
__device__ __forceinline__ void load8(const T* __restrict__ p, float* f) {
  if constexpr (sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  } else {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = to_float(e[j]);
  }
}

template <typename T, bool VEC, int TOK, int CT, typename Epi>
__device__ __forceinline__ void few_tokens_product(const T* __restrict__ B, const float* xs, float* red, int K, int N,
                                                   int n0, Epi epi) {
  constexpr int KG = 256 / CT, COLS = 8 * CT;
  const int c8 = threadIdx.x % CT, kg = threadIdx.x / CT;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int n = n0 + c8 * 8;
  float acc[TOK][8];
#pragma unroll
  for (int tt = 0; tt < TOK; ++tt)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[tt][j] = 0.f;
  if (n < N) {
#pragma unroll 8
    for (int k = kg; k < K; k += KG) {
      float w[8], x[TOK];
      if constexpr (VEC) {
        load8(B + (size_t)k * N + n, w);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) w[j] = n + j < N ? to_float(B[(size_t)k * N + n + j]) : 0.f;
      }
      if constexpr (TOK % 4 == 0) {
#pragma unroll
        for (int tt = 0; tt < TOK; tt += 4) {
          const float4 a = *reinterpret_cast<const float4*>(xs + (size_t)k * TOK + tt);
          x[tt] = a.x; x[tt + 1] = a.y; x[tt + 2] = a.z; x[tt + 3] = a.w;
        }
      } else {
#pragma unroll
        for (int tt = 0; tt < TOK; ++tt) x[tt] = xs[(size_t)k * TOK + tt];
      }
#pragma unroll
      for (int tt = 0; tt < TOK; ++tt)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[tt][j] = fmaf(w[j], x[tt], acc[tt][j]);
    }
  }
#pragma unroll
  for (int o = CT; o < 32; o <<= 1)
#pragma unroll
    for (int tt = 0; tt < TOK; ++tt)
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[tt][j] += __shfl_xor_sync(0xffffffffu, acc[tt][j], o);
  if (lane < CT)
#pragma unroll
    for (int tt = 0; tt < TOK; ++tt) {
      float* r = red + ((size_t)warp * TOK + tt) * COLS + c8 * 8;
      *reinterpret_cast<float4*>(r) = make_float4(acc[tt][0], acc[tt][1], acc[tt][2], acc[tt][3]);
      *reinterpret_cast<float4*>(r + 4) = make_float4(acc[tt][4], acc[tt][5], acc[tt][6], acc[tt][7]);
    }
  __syncthreads();
  for (int i = threadIdx.x; i < TOK * COLS; i += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) v += red[(size_t)w * TOK * COLS + i];
    const int tt = i / COLS, nn = n0 + i % COLS;
    if (nn < N) epi(tt, nn, v);
  }
}

// grid (token tiles, heads, column tiles over rank); q slices [tokens][H (dim + rd)]; w_uk [H][dim][rank];
// q_out [tokens][H][hd].  The blocks of the first column tile also write the rotated part and the padding.
template <typename T, bool VEC, int TOK>
__global__ void __launch_bounds__(256)
latent_absorb_q_kernel(Cols q, const T* __restrict__ w_uk, Rotation rot, Seqs sq, T* __restrict__ q_out,
                       int n_tokens, int H, int dim, int rank, int hd) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float lt_smem[];
  float* red = lt_smem;                                  // [8][TOK][8 LT_CT_Q]
  float* xs = red + 64 * TOK * LT_CT_Q;                  // [dim + rd][TOK]
  __shared__ int pos_s[TOK];
  const int t0 = blockIdx.x * TOK, h = blockIdx.y;
  const int qd = dim + rot.rd;
  if (threadIdx.x < TOK) pos_s[threadIdx.x] = position_of(sq, min(t0 + (int)threadIdx.x, n_tokens - 1));
  pdl_wait();
  for (int idx = threadIdx.x; idx < TOK * qd; idx += blockDim.x) {
    const int tt = idx / qd, e = idx - tt * qd;
    xs[(size_t)e * TOK + tt] = t0 + tt < n_tokens ? col(q, t0 + tt, h * qd + e) : 0.f;
  }
  __syncthreads();
  few_tokens_product<T, VEC, TOK, LT_CT_Q>(
      w_uk + (size_t)h * dim * rank, xs, red, dim, rank, blockIdx.z * 8 * LT_CT_Q, [&](int tt, int n, float v) {
        if (t0 + tt < n_tokens) q_out[((size_t)(t0 + tt) * H + h) * hd + n] = from_float<T>(v);
      });
  if (blockIdx.z != 0) return;
  const int tail = hd - rank;
  for (int idx = threadIdx.x; idx < TOK * tail; idx += blockDim.x) {
    const int tt = idx / tail, e = idx - tt * tail;
    const int t = t0 + tt;
    if (t >= n_tokens) continue;
    float v = 0.f;
    if (e < rot.rd) v = rotated(rot, e, pos_s[tt], [&](int f) { return xs[(size_t)(dim + f) * TOK + tt]; });
    q_out[((size_t)t * H + h) * hd + rank + e] = from_float<T>(v);
  }
}

// Partial results of an attention whose keys were split over blocks: part_o float32
// [tokens][H][nsplit][rank] (unnormalised), part_ml [tokens][H][nsplit][2] = (maximum in units of
// log2, sum); a part without keys has maximum -inf.
struct Parts {
  const float *o, *ml;
  int nsplit;
};
constexpr int LT_MAX_SPLIT = 64;

// grid (token tiles, heads, column tiles over vdim).  o [tokens][H][hd] or `parts`; w_uv [H][rank][vdim]
// (transposed when bound); out [tokens][H vdim]
template <typename T, bool VEC, int TOK>
__global__ void __launch_bounds__(256)
latent_expand_kernel(const T* __restrict__ o, Parts parts, const T* __restrict__ w_uv, Gate gate,
                     T* __restrict__ out, int n_tokens, int H, int rank, int vdim, int hd) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float lt_smem[];
  float* red = lt_smem;                                  // [8][TOK][8 LT_CT_V]
  float* xs = red + 64 * TOK * LT_CT_V;                  // [rank][TOK]
  __shared__ float w_s[TOK][LT_MAX_SPLIT];
  const int t0 = blockIdx.x * TOK, h = blockIdx.y;
  pdl_wait();
  if (parts.nsplit > 1) {
    // a warp per token: the parts' weights exp2(m_s - M) / L
    const int lane = threadIdx.x & 31, tt = threadIdx.x >> 5;
    if (tt < TOK && t0 + tt < n_tokens) {
      const float* ml = parts.ml + ((size_t)(t0 + tt) * H + h) * parts.nsplit * 2;
      float m[LT_MAX_SPLIT / 32], l[LT_MAX_SPLIT / 32], M = -INFINITY, L = 0.f;
#pragma unroll
      for (int k = 0; k < LT_MAX_SPLIT / 32; ++k) {
        const int s = lane + 32 * k;
        m[k] = s < parts.nsplit ? ml[2 * s] : -INFINITY;
        l[k] = s < parts.nsplit ? ml[2 * s + 1] : 0.f;
        M = fmaxf(M, m[k]);
      }
      M = warp_max(M);
#pragma unroll
      for (int k = 0; k < LT_MAX_SPLIT / 32; ++k) {
        m[k] = m[k] > -INFINITY ? exp2f(m[k] - M) : 0.f;
        L += l[k] * m[k];
      }
      L = warp_sum(L);
#pragma unroll
      for (int k = 0; k < LT_MAX_SPLIT / 32; ++k)
        if (lane + 32 * k < parts.nsplit) w_s[tt][lane + 32 * k] = m[k] / L;
    }
    __syncthreads();
    // four features per thread where the rows allow it, all loads of eight parts in flight
    auto merge = [&](auto vec4) {
      constexpr int W = decltype(vec4)::value;
      const int per = rank / W;
      for (int idx = threadIdx.x; idx < TOK * per; idx += blockDim.x) {
        const int u = idx / per, c = (idx - u * per) * W;
        float v[W];
#pragma unroll
        for (int j = 0; j < W; ++j) v[j] = 0.f;
        if (t0 + u < n_tokens) {
          const float* po = parts.o + ((size_t)(t0 + u) * H + h) * parts.nsplit * rank + c;
          for (int s0 = 0; s0 < parts.nsplit; s0 += 8) {
            float p[8][W];
#pragma unroll
            for (int j = 0; j < 8; ++j) {                // a part of weight zero may never have been written
              const bool on = s0 + j < parts.nsplit && w_s[u][min(s0 + j, LT_MAX_SPLIT - 1)] > 0.f;
              if constexpr (W == 4) {
                const float4 a = on ? *reinterpret_cast<const float4*>(po + (size_t)(s0 + j) * rank) : make_float4(0.f, 0.f, 0.f, 0.f);
                p[j][0] = a.x; p[j][1] = a.y; p[j][2] = a.z; p[j][3] = a.w;
              } else {
                p[j][0] = on ? po[(size_t)(s0 + j) * rank] : 0.f;
              }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j)
              if (s0 + j < parts.nsplit)
#pragma unroll
                for (int i = 0; i < W; ++i) v[i] = fmaf(w_s[u][s0 + j], p[j][i], v[i]);
          }
        }
#pragma unroll
        for (int i = 0; i < W; ++i) xs[(size_t)(c + i) * TOK + u] = v[i];
      }
    };
    if (rank % 4 == 0) merge(Int<4>());
    else merge(Int<1>());
  } else {
    for (int idx = threadIdx.x; idx < TOK * rank; idx += blockDim.x) {
      const int tt = idx / rank, c = idx - tt * rank;
      xs[(size_t)c * TOK + tt] = t0 + tt < n_tokens ? to_float(o[((size_t)(t0 + tt) * H + h) * hd + c]) : 0.f;
    }
  }
  __syncthreads();
  few_tokens_product<T, VEC, TOK, LT_CT_V>(
      w_uv + (size_t)h * rank * vdim, xs, red, rank, vdim, blockIdx.z * 8 * LT_CT_V, [&](int tt, int n, float v) {
        const int t = t0 + tt;
        if (t < n_tokens) out[((size_t)t * H + h) * vdim + n] = from_float<T>(gated(gate, t, h, n, vdim, v));
      });
}

// ---- the two per-head products for many tokens: a block of 256 threads takes 64 tokens x 64
// columns of one head, a thread 4 x 4 of them; A and the head's matrix come through shared memory in
// slabs of 16 of K, so that a loaded element feeds 64 multiply-adds.
constexpr int HP_BM = 64, HP_BN = 64, HP_BK = 16;

template <typename T, typename LoadA, typename Epi>
__device__ __forceinline__ void head_product_tile(const T* __restrict__ B, int K, int N, int t0, int n0,
                                                  int n_tokens, LoadA load_a, Epi epi) {
  __shared__ __align__(16) float As[HP_BK][HP_BM + 4];     // [k][token]
  __shared__ __align__(16) float Bs[HP_BK][HP_BN + 4];     // [k][column]
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += HP_BK) {
#pragma unroll
    for (int r = 0; r < HP_BM * HP_BK / 256; ++r) {
      const int i = threadIdx.x + r * 256;
      const int tt = i / HP_BK, kk = i % HP_BK;
      As[kk][tt] = (t0 + tt < n_tokens && k0 + kk < K) ? load_a(t0 + tt, k0 + kk) : 0.f;
    }
#pragma unroll
    for (int r = 0; r < HP_BK * HP_BN / 256; ++r) {
      const int i = threadIdx.x + r * 256;
      const int kk = i / HP_BN, nn = i % HP_BN;
      Bs[kk][nn] = (k0 + kk < K && n0 + nn < N) ? to_float(B[(size_t)(k0 + kk) * N + n0 + nn]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < HP_BK; ++kk) {
      const float4 a = *reinterpret_cast<const float4*>(&As[kk][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Bs[kk][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(bv[j], av[i], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (t < n_tokens && n < N) epi(t, n, acc[i][j]);
    }
}

// grid (token tiles of 64, heads, column tiles of 64 over rank); the blocks of the first column
// tile also write the rotated part and the zero padding
template <typename T>
__global__ void __launch_bounds__(256)
latent_absorb_q_tiled_kernel(Cols q, const T* __restrict__ w_uk, Rotation rot, Seqs sq, T* __restrict__ q_out,
                             int n_tokens, int H, int dim, int rank, int hd) {
  pdl_launch_dependents();
  const int t0 = blockIdx.x * HP_BM, h = blockIdx.y, n0 = blockIdx.z * HP_BN;
  const int qd = dim + rot.rd;
  pdl_wait();
  head_product_tile<T>(
      w_uk + (size_t)h * dim * rank, dim, rank, t0, n0, n_tokens,
      [&](int t, int k) { return col(q, t, h * qd + k); },
      [&](int t, int n, float v) { q_out[((size_t)t * H + h) * hd + n] = from_float<T>(v); });
  if (blockIdx.z != 0) return;
  const int tail = hd - rank;
  for (int idx = threadIdx.x; idx < HP_BM * tail; idx += blockDim.x) {
    const int tt = idx / tail, e = idx - tt * tail;
    const int t = t0 + tt;
    if (t >= n_tokens) continue;
    float v = 0.f;
    if (e < rot.rd) v = rotated(rot, e, position_of(sq, t), [&](int f) { return col(q, t, h * qd + dim + f); });
    q_out[((size_t)t * H + h) * hd + rank + e] = from_float<T>(v);
  }
}

// grid (token tiles of 64, heads, column tiles of 64 over vdim)
template <typename T>
__global__ void __launch_bounds__(256)
latent_expand_tiled_kernel(const T* __restrict__ o, const T* __restrict__ w_uv, Gate gate, T* __restrict__ out,
                           int n_tokens, int H, int rank, int vdim, int hd) {
  pdl_launch_dependents();
  const int t0 = blockIdx.x * HP_BM, h = blockIdx.y, n0 = blockIdx.z * HP_BN;
  pdl_wait();
  head_product_tile<T>(
      w_uv + (size_t)h * rank * vdim, rank, vdim, t0, n0, n_tokens,
      [&](int t, int k) { return to_float(o[((size_t)t * H + h) * hd + k]); },
      [&](int t, int n, float v) {
        out[((size_t)t * H + h) * vdim + n] = from_float<T>(gated(gate, t, h, n, vdim, v));
      });
}

// Beyond this many tokens the tiled kernels run, in the 16-bit types; in 32 bits every result is the same
// chain of additions whatever else is in the step.
constexpr int HP_MANY = 128;

}  // namespace yalm

using namespace yalm;

#define YALM_BY_TYPE(dtype, CALL)                 \
  do {                                            \
    if ((dtype) == DT_F32) { CALL(float); }       \
    else if ((dtype) == DT_BF16) { CALL(__nv_bfloat16); } \
    else if ((dtype) == DT_F16) { CALL(__half); } \
    else return -3;                               \
  } while (0)
// CALL(T, VEC) with a run-time choice of VEC
#define YALM_BY_TYPE_VEC(dtype, vec, CALL)                                        \
  do {                                                                            \
    if ((dtype) == DT_F32) { if (vec) { CALL(float, true); } else { CALL(float, false); } }                   \
    else if ((dtype) == DT_BF16) { if (vec) { CALL(__nv_bfloat16, true); } else { CALL(__nv_bfloat16, false); } } \
    else if ((dtype) == DT_F16) { if (vec) { CALL(__half, true); } else { CALL(__half, false); } }            \
    else return -3;                                                               \
  } while (0)
#define YALM_LT_SMEM(KERNEL, smem)                                                                          \
  do {                                                                                                      \
    static size_t attr = 40 * 1024;            /* static shared memory comes on top */                      \
    if ((smem) > attr) {                                                                                    \
      cudaError_t e = cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem)); \
      if (e != cudaSuccess) return (int)e;                                                                  \
      attr = (smem);                                                                                        \
    }                                                                                                       \
  } while (0)

// src: float32 slices [n_partials][tokens][src_row], the down projection's rank + rd columns from col0 on;
// c_norm [rank]; freq [rd / 2]; kv_step [tokens][2][hd] and the cache ([slots][1][capacity][hd], or
// pages) in `dtype`, c_rows (optional) [tokens][rank]; hd >= rank + rd (the rest is zero)
extern "C" int yalm_latent_store(const float* src, int n_partials, long long partial_stride, int src_row, int col0,
                                 const float* c_norm, float eps, const float* freq, int halves, float mult,
                                 const int* token_seq, const int* q_start, const int* seq_slot,
                                 const int* slot_pos, void* kv_step, void* cache, void* c_rows, int dtype,
                                 int n_tokens, int rank, int rd, int hd, int capacity, int write_cache,
                                 const int* page_table, int pages_per_slot, int n_pages, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (rank <= 0 || rd < 0 || rd % 2 || hd < rank + rd || rank + rd > 12 * 1024 || capacity <= 0) return -2;
  const Cols s = {src + col0, n_partials, partial_stride, src_row};
  const Rotation rot = {freq, rd, halves, mult};
  const Seqs sq = {token_seq, q_start, seq_slot, slot_pos};
  const size_t smem = (size_t)(rank + rd) * sizeof(float);
  const bool vec = rank % 4 == 0 && rd % 4 == 0 && hd % 4 == 0 && src_row % 4 == 0 && col0 % 4 == 0 && (partial_stride & 3) == 0 &&
                   ((((uintptr_t)src) | ((uintptr_t)kv_step) | ((uintptr_t)cache) | ((uintptr_t)c_rows)) & 15) == 0;
  int threads = ((vec ? hd / 4 : hd) + 31) / 32 * 32;
  if (threads > 512) threads = 512;
#define CALL(T, V)                                                                                        \
  launch_pdl(latent_store_kernel<T, V>, dim3(n_tokens), dim3(threads), smem, stream, s, c_norm, eps, rot, \
             sq, (T*)kv_step, (T*)cache, (T*)c_rows, rank, hd, capacity, write_cache, page_table,         \
             pages_per_slot, n_pages)
  YALM_BY_TYPE_VEC(dtype, vec, CALL);
#undef CALL
  YALM_LAUNCH_CHECK();
  return 0;
}

// q_out [tokens][H][dim + rd] in `dtype` = q with the last rd features of every head rotated
extern "C" int yalm_latent_rotate_q(const float* q, int n_partials, long long partial_stride, int q_row, int col0,
                                    const float* freq, int halves, float mult, const int* token_seq,
                                    const int* q_start, const int* seq_slot, const int* slot_pos, void* q_out,
                                    int dtype, int n_tokens, int H, int dim, int rd, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || dim <= 0 || rd < 0 || rd % 2 || rd > 8192) return -2;
  const Cols s = {q + col0, n_partials, partial_stride, q_row};
  const Rotation rot = {freq, rd, halves, mult};
  const Seqs sq = {token_seq, q_start, seq_slot, slot_pos};
  const bool vec = dim % 4 == 0 && rd % 8 == 0 && q_row % 4 == 0 && col0 % 4 == 0 && (partial_stride & 3) == 0 &&
                   ((((uintptr_t)q) | ((uintptr_t)q_out)) & 15) == 0;
  int per = H;                                           // heads per block: about 2,048 features
  while (per > 1 && (per - 1) * (dim + rd) >= 2048) --per;
  const dim3 grid(n_tokens, (H + per - 1) / per), block(256);
#define CALL(T, V)                                                                                        \
  launch_pdl(latent_rotate_q_kernel<T, V>, grid, block, (size_t)(rd + 1) * sizeof(float), stream, s, rot, \
             sq, (T*)q_out, H, dim, per)
  YALM_BY_TYPE_VEC(dtype, vec, CALL);
#undef CALL
  YALM_LAUNCH_CHECK();
  return 0;
}

extern "C" int yalm_latent_absorb_q(const float* q, int n_partials, long long partial_stride, int q_row, int col0,
                                    const void* w_uk, const float* freq, int halves, float mult,
                                    const int* token_seq, const int* q_start, const int* seq_slot,
                                    const int* slot_pos, void* q_out, int dtype, int n_tokens, int H, int dim,
                                    int rd, int rank, int hd, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || H > 65535 || dim <= 0 || rd < 0 || rd % 2 || rank <= 0 || hd < rank + rd) return -2;
  const Cols s = {q + col0, n_partials, partial_stride, q_row};
  const Rotation rot = {freq, rd, halves, mult};
  const Seqs sq = {token_seq, q_start, seq_slot, slot_pos};
  const dim3 block(256);
  const int tok = n_tokens <= LT_ONE ? 1 : LT_TOK;
  const size_t smem = ((size_t)(dim + rd) * tok + 64 * tok * LT_CT_Q) * sizeof(float);
  if ((n_tokens > HP_MANY && dtype != DT_F32) || smem > 160 * 1024) {
    const dim3 grid((n_tokens + HP_BM - 1) / HP_BM, H, (rank + HP_BN - 1) / HP_BN);
#define CALL(T)                                                                                     \
  launch_pdl(latent_absorb_q_tiled_kernel<T>, grid, block, 0, stream, s, (const T*)w_uk, rot, sq,   \
             (T*)q_out, n_tokens, H, dim, rank, hd)
    YALM_BY_TYPE(dtype, CALL);
#undef CALL
    YALM_LAUNCH_CHECK();
    return 0;
  }
  const bool vec = rank % 8 == 0 && (((uintptr_t)w_uk) & 15) == 0;
  const dim3 grid((n_tokens + tok - 1) / tok, H, (rank + 8 * LT_CT_Q - 1) / (8 * LT_CT_Q));
#define CALL1(T, V, K)                                                                                  \
  YALM_LT_SMEM((latent_absorb_q_kernel<T, V, K>), smem);                                                \
  launch_pdl(latent_absorb_q_kernel<T, V, K>, grid, block, smem, stream, s, (const T*)w_uk, rot, sq,    \
             (T*)q_out, n_tokens, H, dim, rank, hd)
#define CALL(T, V) if (tok == 1) { CALL1(T, V, 1); } else { CALL1(T, V, LT_TOK); }
  YALM_BY_TYPE_VEC(dtype, vec, CALL);
#undef CALL
#undef CALL1
  YALM_LAUNCH_CHECK();
  return 0;
}

// o [tokens][H][hd] in `dtype`, or with nsplit > 1 the partial results part_o / part_ml (see Parts);
// gate: float32 slices, gate_mode 0 none, 1 one logit per head, 2 one per feature
extern "C" int yalm_latent_expand(const void* o, const float* part_o, const float* part_ml, int nsplit,
                                  const void* w_uv, const float* gate, int gate_mode, int n_partials,
                                  long long partial_stride, int gate_row, int col0, void* out, int dtype,
                                  int n_tokens, int H, int rank, int vdim, int hd, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || H > 65535 || rank <= 0 || vdim <= 0 || hd < rank || gate_mode < 0 || gate_mode > 2) return -2;
  if (nsplit > LT_MAX_SPLIT || (nsplit > 1 && n_tokens > HP_MANY)) return -5;
  const Gate g = {{gate == nullptr ? nullptr : gate + col0, n_partials, partial_stride, gate_row},
                  gate == nullptr ? 0 : gate_mode};
  const Parts parts = {part_o, part_ml, nsplit};
  const dim3 block(256);
  const int tok = n_tokens <= LT_ONE ? 1 : LT_TOK;
  const size_t smem = ((size_t)rank * tok + 64 * tok * LT_CT_V) * sizeof(float);
  if (nsplit <= 1 && ((n_tokens > HP_MANY && dtype != DT_F32) || smem > 160 * 1024)) {
    const dim3 grid((n_tokens + HP_BM - 1) / HP_BM, H, (vdim + HP_BN - 1) / HP_BN);
#define CALL(T)                                                                                        \
  launch_pdl(latent_expand_tiled_kernel<T>, grid, block, 0, stream, (const T*)o, (const T*)w_uv, g,    \
             (T*)out, n_tokens, H, rank, vdim, hd)
    YALM_BY_TYPE(dtype, CALL);
#undef CALL
    YALM_LAUNCH_CHECK();
    return 0;
  }
  if (smem > 160 * 1024) return -2;
  const bool vec = vdim % 8 == 0 && (((uintptr_t)w_uv) & 15) == 0;
  const dim3 grid((n_tokens + tok - 1) / tok, H, (vdim + 8 * LT_CT_V - 1) / (8 * LT_CT_V));
#define CALL1(T, V, K)                                                                                 \
  YALM_LT_SMEM((latent_expand_kernel<T, V, K>), smem);                                                 \
  launch_pdl(latent_expand_kernel<T, V, K>, grid, block, smem, stream, (const T*)o, parts,             \
             (const T*)w_uv, g, (T*)out, n_tokens, H, rank, vdim, hd)
#define CALL(T, V) if (tok == 1) { CALL1(T, V, 1); } else { CALL1(T, V, LT_TOK); }
  YALM_BY_TYPE_VEC(dtype, vec, CALL);
#undef CALL
#undef CALL1
  YALM_LAUNCH_CHECK();
  return 0;
}
