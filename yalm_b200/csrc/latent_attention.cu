// The attention of a latent mixer (latent.cu), scores, softmax weights and weighted sums in 32 bits.
// A query sees the last `window` positions (0: every earlier one); a sink adds exp(sink_h) to the
// softmax's denominator (no key, no value, not scaled, counted once).  Three kernels:
//
//  * attn_latent_mma (16-bit): the absorbed form, a decode step's or a portion's queries over the
//    cached rows.  A block takes 16 heads of one token over one run of its keys; the rows -- keys
//    and values at once -- come in tiles of 32 through two cp.async buffers, small enough for two
//    blocks to share an SM: one's softmax and barriers run under the other's products.  S = q K^T by
//    mma.sync (the 16 heads are the rows of a tile; a warp takes 8 keys and half of the features),
//    softmax by 16 threads per head, O += P C with every weight as three 16-bit terms (all its bits), a
//    warp per part of the columns.  A row is read from memory once for all heads of the group.
//  * attn_latent_fma: the same with 32-bit FMA on any storage type: the 32-bit path, and row sizes
//    that the kernel above does not take.
//  * attn_latent_prefill (16-bit): the expanded form for whole prompts: per head keys
//    [Wuk c | kr] and values Wuv c of this step, made by one product; 64 queries of one head per
//    block, key blocks of 64, weights as three 16-bit terms as in attention_exact.cu.  The output
//    gate is applied to the 32-bit results.
// With several blocks per query the partial results are merged by latent_expand.
#include "api.h"
#include "common.cuh"

namespace yalm {

template <typename T> __device__ __forceinline__ void mma16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1);
template <> __device__ __forceinline__ void mma16<__nv_bfloat16>(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
template <> __device__ __forceinline__ void mma16<__half>(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// 16 bytes to shared memory, or zeros when `bytes` is 0
__device__ __forceinline__ void cp16(const void* dst, const void* src, uint32_t bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// (a, b) as three packed pairs of the 16-bit type whose sum is (a, b)
template <typename T>
__device__ __forceinline__ void three_terms(float a, float b, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  const float ah = to_float(from_float<T>(a)), bh = to_float(from_float<T>(b));
  const float ar = a - ah, br = b - bh;
  const float am = to_float(from_float<T>(ar)), bm = to_float(from_float<T>(br));
  hi = pack2<T>(ah, bh);
  mid = pack2<T>(am, bm);
  lo = pack2<T>(ar - am, br - bm);
}

constexpr float LOG2E = 1.4426950408889634f;

// Where the rows of a latent layer live: positions of this step in kv_step [tokens][2][hd], earlier
// ones in the cache ring (see kv_row_offset).
struct LatentRows {
  const void *kv_step, *cache;
  const int *token_seq, *q_start, *seq_slot, *slot_pos;
  const int* page_table;
  int pps, n_pages, capacity, hd, rank, H, window, nsplit, per;      // per: keys of a split
  float scale_log2;
  const float* sink;         // [H] or null
};
struct LatentOut {
  void* out;                 // [tokens][H][hd] in the storage type, with nsplit == 1
  float *part_o, *part_ml;   // else [tokens][H][nsplit][rank] and [tokens][H][nsplit][2] (maximum in log2 units, sum)
};

// the run of keys of one split; the last split takes whatever is left
__device__ __forceinline__ void split_range(const LatentRows& a, int lo, int pos, int split, int& k0, int& k1) {
  k0 = lo + split * a.per;
  k1 = split == a.nsplit - 1 ? pos + 1 : min(k0 + a.per, pos + 1);
}
template <typename T>
__device__ __forceinline__ const T* latent_row(const LatentRows& a, int key, int past, int qs, int slot) {
  if (key >= past) return reinterpret_cast<const T*>(a.kv_step) + (size_t)(qs + key - past) * 2 * a.hd;
  return reinterpret_cast<const T*>(a.cache) +
         kv_row_offset(a.page_table, a.pps, a.n_pages, slot, 0, 1, a.capacity, key % a.capacity, a.hd);
}

constexpr int LA_HEADS = 16, LA_KEYS = 32, LA_WARPS = 8;
constexpr int LA_SP = LA_KEYS + 4;                     // pitch of the scores (floats)
constexpr int LA_PP = LA_KEYS + 8;                     // pitch of the weights (16-bit)

// NT: 8-column tiles per warp; rank <= 64 NT.  grid (splits, head groups, tokens)
template <typename T, int NT>
__global__ void __launch_bounds__(LA_WARPS * 32, 2)
attn_latent_mma_kernel(const T* __restrict__ q, LatentRows a, LatentOut o_) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t la_smem[];
  const int hd = a.hd, lds = hd + 8;
  T* qs_ = reinterpret_cast<T*>(la_smem);              // [16][lds]
  T* rows = qs_ + LA_HEADS * lds;                      // two tiles [32][lds]
  T* ps = rows + 2 * LA_KEYS * lds + 32;               // weights, three terms [3][16][LA_PP]
  float* ss = reinterpret_cast<float*>(ps + 3 * LA_HEADS * LA_PP);        // scores of either half [2][16][LA_SP]
  __shared__ float corr_s[LA_HEADS], l_s[LA_HEADS];
  const int t = blockIdx.z, h0 = blockIdx.y * LA_HEADS, split = blockIdx.x;
  const int nh = min(LA_HEADS, a.H - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = a.token_seq[t], slot = a.seq_slot[b], qs = a.q_start[b];
  const int past = a.slot_pos[slot], pos = past + (t - qs);
  const int lo = first_visible(pos, a.window);
  int k0, k1;
  split_range(a, lo, pos, split, k0, k1);
  pdl_wait();
  if (k0 >= k1 && a.nsplit > 1) {                      // a split without keys (the first always has one)
    if (threadIdx.x < nh) {
      float* ml = o_.part_ml + (((size_t)t * a.H + h0 + threadIdx.x) * a.nsplit + split) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  const int pieces = hd / 8;
  auto issue = [&](int base, int buf) {
    const int r = threadIdx.x >> 3, key = base + r;
    const bool on = key < k1;
    const T* src = on ? latent_row<T>(a, key, past, qs, slot) : q;
    T* dst = rows + (size_t)buf * LA_KEYS * lds + r * lds;
    for (int c = threadIdx.x & 7; c < pieces; c += 8) cp16(dst + c * 8, src + (on ? c * 8 : 0), on ? 16 : 0);
    cp_commit();
  };
  for (int i = threadIdx.x; i < LA_HEADS * pieces; i += blockDim.x) {
    const int r = i / pieces, c = i - r * pieces;
    const bool on = r < nh;
    cp16(qs_ + r * lds + c * 8, q + ((size_t)t * a.H + h0 + (on ? r : 0)) * hd + c * 8, on ? 16 : 0);
  }
  issue(k0, 0);
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  // softmax: 16 threads per head, two keys each
  const int sh = threadIdx.x >> 4, sk = threadIdx.x & 15;
  float m = -INFINITY, l = 0.f;
  if (a.sink != nullptr && split == 0 && sh < nh) {
    m = a.sink[h0 + sh] * LOG2E;
    l = sk == 0 ? 1.f : 0.f;
  }
  const int g = lane >> 2, t4 = lane & 3;
  const int n_tiles = (k1 - k0 + LA_KEYS - 1) / LA_KEYS;
  const int nk = hd / 16, nk_half = ((nk + 3) / 4) * 2;            // the first half has an even number of steps
  const int kh = warp >> 2, kt = warp & 3;             // this warp's half of the features and its 8 keys
  const int kk0 = kh ? nk_half : 0, kk1 = kh ? nk : min(nk_half, nk);
  for (int it = 0; it < n_tiles; ++it) {
    const int base = k0 + it * LA_KEYS;
    cp_wait<0>();
    __syncthreads();                                   // the tile has landed; the other buffer is no longer read
    if (it + 1 < n_tiles) issue(base + LA_KEYS, (it + 1) & 1);
    const T* tile = rows + (size_t)(it & 1) * LA_KEYS * lds;
    {
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t qa = smem_u32(qs_ + (lane & 15) * lds + (lane >> 4) * 8);
      const uint32_t kb = smem_u32(tile + (kt * 8 + (lane & 7)) * lds + (lane >> 3) * 8);
      int kk = kk0;
#pragma unroll 4
      for (; kk + 2 <= kk1; kk += 2) {
        uint32_t qf[4], qg[4], kf[4];
        ldsm_x4(kf, kb + kk * 32);
        ldsm_x4(qf, qa + kk * 32);
        ldsm_x4(qg, qa + kk * 32 + 32);
        mma16<T>(s0, qf, kf[0], kf[1]);
        mma16<T>(s1, qg, kf[2], kf[3]);
      }
      if (kk < kk1) {
        uint32_t qf[4], kf[4];
        ldsm_x4(kf, kb + kk * 32);                     // the upper half lies in the pad and is not used
        ldsm_x4(qf, qa + kk * 32);
        mma16<T>(s0, qf, kf[0], kf[1]);
      }
      float* sd = ss + kh * LA_HEADS * LA_SP + kt * 8 + 2 * t4;
      *reinterpret_cast<float2*>(sd + g * LA_SP) = make_float2(s0[0] + s1[0], s0[1] + s1[1]);
      *reinterpret_cast<float2*>(sd + (g + 8) * LA_SP) = make_float2(s0[2] + s1[2], s0[3] + s1[3]);
    }
    __syncthreads();
    {
      const float2 u = *reinterpret_cast<const float2*>(ss + sh * LA_SP + sk * 2);
      const float2 w = *reinterpret_cast<const float2*>(ss + (LA_HEADS + sh) * LA_SP + sk * 2);
      const int key = base + sk * 2;
      const float x0 = key < k1 ? (u.x + w.x) * a.scale_log2 : -INFINITY;
      const float x1 = key + 1 < k1 ? (u.y + w.y) * a.scale_log2 : -INFINITY;
      float mx = fmaxf(x0, x1);
#pragma unroll
      for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float mn = fmaxf(m, mx);                   // a tile has at least one key
      const float corr = exp2f(m - mn);                // exp2(-inf) = 0 on the first
      m = mn;
      const float p0 = exp2f(x0 - mn), p1 = exp2f(x1 - mn);
      l = l * corr + (p0 + p1);
      if (sk == 0) corr_s[sh] = corr;
      uint32_t hi, mid, low;
      three_terms<T>(p0, p1, hi, mid, low);
      uint32_t* p = reinterpret_cast<uint32_t*>(ps + sh * LA_PP + sk * 2);
      p[0] = hi;
      p[LA_HEADS * LA_PP / 2] = mid;
      p[LA_HEADS * LA_PP] = low;
    }
    __syncthreads();
    {
      const float c0 = corr_s[g], c1 = corr_s[g + 8];
      if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
        for (int i = 0; i < NT; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
      }
      const uint32_t pa = smem_u32(ps + (lane & 15) * LA_PP + (lane >> 4) * 8);
      const uint32_t va = smem_u32(tile + ((lane >> 3 & 1) * 8 + (lane & 7)) * lds + (lane >> 4) * 8);
#pragma unroll
      for (int kk = 0; kk < LA_KEYS / 16; ++kk) {
        uint32_t p[3][4], r[NT / 2][4];                // the small terms first
        ldsm_x4(p[2], pa + kk * 32);
        ldsm_x4(p[1], pa + kk * 32 + LA_HEADS * LA_PP * 2);
        ldsm_x4(p[0], pa + kk * 32 + 2 * LA_HEADS * LA_PP * 2);
#pragma unroll
        for (int n2 = 0; n2 < NT / 2; ++n2) {
          const int col = warp * NT * 8 + n2 * 16;     // rank <= hd and hd is a multiple of 16: in bounds
          if (col < a.rank) ldsm_x4_trans(r[n2], va + (uint32_t)(kk * 16 * lds + col) * 2);
        }
#pragma unroll
        for (int term = 0; term < 3; ++term)
#pragma unroll
          for (int n2 = 0; n2 < NT / 2; ++n2)
            if (warp * NT * 8 + n2 * 16 < a.rank) {
              mma16<T>(o[2 * n2], p[term], r[n2][0], r[n2][1]);
              mma16<T>(o[2 * n2 + 1], p[term], r[n2][2], r[n2][3]);
            }
      }
    }
  }
#pragma unroll
  for (int off = 8; off > 0; off >>= 1) l += __shfl_xor_sync(0xffffffffu, l, off);
  if (sk == 0) {
    l_s[sh] = l;
    if (a.nsplit > 1 && sh < nh) {
      float* ml = o_.part_ml + (((size_t)t * a.H + h0 + sh) * a.nsplit + split) * 2;
      ml[0] = m;
      ml[1] = l;
    }
  }
  __syncthreads();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int head = g + 8 * half;
    if (head >= nh) continue;
    const float inv = 1.0f / l_s[head];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int col = (warp * NT + i) * 8 + 2 * t4;
      if (col >= a.rank) continue;
      const float x = o[i][2 * half], y = o[i][2 * half + 1];
      if (a.nsplit > 1) {
        float* dst = o_.part_o + (((size_t)t * a.H + h0 + head) * a.nsplit + split) * a.rank + col;
        if ((a.rank & 1) == 0) {
          *reinterpret_cast<float2*>(dst) = make_float2(x, y);
        } else {
          dst[0] = x;
          if (col + 1 < a.rank) dst[1] = y;
        }
      } else {                                         // hd is a multiple of 16: col + 1 < hd
        *reinterpret_cast<uint32_t*>(reinterpret_cast<T*>(o_.out) + ((size_t)t * a.H + h0 + head) * hd + col) =
            pack2<T>(x * inv, y * inv);
      }
    }
  }
}

constexpr int LF_HEADS = 4, LF_KEYS = 64, LF_MAX_COLS = 4;         // rank <= 256 LF_MAX_COLS

template <typename T>
__global__ void __launch_bounds__(256)
attn_latent_fma_kernel(const T* __restrict__ q, LatentRows a, LatentOut o_) {
  pdl_launch_dependents();
  extern __shared__ float lf_q[];                      // [LF_HEADS][hd]
  __shared__ float s_s[LF_HEADS][LF_KEYS];
  __shared__ float corr_s[LF_HEADS], l_s[LF_HEADS];
  __shared__ const T* row_s[LF_KEYS];
  const int t = blockIdx.z, h0 = blockIdx.y * LF_HEADS, split = blockIdx.x, hd = a.hd;
  const int nh = min(LF_HEADS, a.H - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = a.token_seq[t], slot = a.seq_slot[b], qs = a.q_start[b];
  const int past = a.slot_pos[slot], pos = past + (t - qs);
  const int lo = first_visible(pos, a.window);
  int k0, k1;
  split_range(a, lo, pos, split, k0, k1);
  pdl_wait();
  if (k0 >= k1 && a.nsplit > 1) {
    if (threadIdx.x < nh) {
      float* ml = o_.part_ml + (((size_t)t * a.H + h0 + threadIdx.x) * a.nsplit + split) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  for (int i = threadIdx.x; i < LF_HEADS * hd; i += blockDim.x) {
    const int r = i / hd;
    lf_q[i] = r < nh ? to_float(q[((size_t)t * a.H + h0) * hd + i]) : 0.f;
  }
  float acc[LF_HEADS][LF_MAX_COLS];
#pragma unroll
  for (int r = 0; r < LF_HEADS; ++r)
#pragma unroll
    for (int c = 0; c < LF_MAX_COLS; ++c) acc[r][c] = 0.f;
  float m = -INFINITY, l = 0.f;                        // warp r < LF_HEADS: head r
  if (a.sink != nullptr && split == 0 && warp < nh) {
    m = a.sink[h0 + warp] * LOG2E;
    l = 1.f;
  }
  for (int base = k0; base < k1; base += LF_KEYS) {
    const int n = min(LF_KEYS, k1 - base);
    __syncthreads();                                   // the last tile's weights and rows are no longer read
    if (threadIdx.x < n) row_s[threadIdx.x] = latent_row<T>(a, base + threadIdx.x, past, qs, slot);
    __syncthreads();
    for (int k = warp; k < n; k += 8) {
      const T* row = row_s[k];
      float d[LF_HEADS] = {0.f, 0.f, 0.f, 0.f};
      for (int f = lane; f < hd; f += 32) {
        const float v = to_float(row[f]);
#pragma unroll
        for (int r = 0; r < LF_HEADS; ++r) d[r] = fmaf(lf_q[r * hd + f], v, d[r]);
      }
#pragma unroll
      for (int r = 0; r < LF_HEADS; ++r) {
        d[r] = warp_sum(d[r]);
        if (lane == 0) s_s[r][k] = d[r] * a.scale_log2;
      }
    }
    __syncthreads();
    if (warp < LF_HEADS) {
      const float v0 = lane < n ? s_s[warp][lane] : -INFINITY, v1 = lane + 32 < n ? s_s[warp][lane + 32] : -INFINITY;
      const float mn = fmaxf(m, warp_max(fmaxf(v0, v1)));
      const float corr = exp2f(m - mn);
      const float p0 = exp2f(v0 - mn), p1 = exp2f(v1 - mn);
      m = mn;
      l = l * corr + warp_sum(p0 + p1);
      s_s[warp][lane] = p0;
      s_s[warp][lane + 32] = p1;
      if (lane == 0) corr_s[warp] = corr;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < LF_HEADS; ++r)
#pragma unroll
      for (int c = 0; c < LF_MAX_COLS; ++c) acc[r][c] *= corr_s[r];
#pragma unroll
    for (int c = 0; c < LF_MAX_COLS; ++c) {
      const int f = threadIdx.x + 256 * c;
      if (f < a.rank)
        for (int k = 0; k < n; ++k) {
          const float v = to_float(row_s[k][f]);
#pragma unroll
          for (int r = 0; r < LF_HEADS; ++r) acc[r][c] = fmaf(s_s[r][k], v, acc[r][c]);
        }
    }
  }
  if (warp < LF_HEADS && lane == 0) {
    l_s[warp] = l;
    if (a.nsplit > 1 && warp < nh) {
      float* ml = o_.part_ml + (((size_t)t * a.H + h0 + warp) * a.nsplit + split) * 2;
      ml[0] = m;
      ml[1] = l;
    }
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < LF_HEADS; ++r)
#pragma unroll
    for (int c = 0; c < LF_MAX_COLS; ++c) {
      const int f = threadIdx.x + 256 * c;
      if (r >= nh || f >= a.rank) continue;
      if (a.nsplit > 1)
        o_.part_o[(((size_t)t * a.H + h0 + r) * a.nsplit + split) * a.rank + f] = acc[r][c];
      else
        reinterpret_cast<T*>(o_.out)[((size_t)t * a.H + h0 + r) * hd + f] = from_float<T>(acc[r][c] / l_s[r]);
    }
}

// ---- the expanded form: whole prompts ------------------------------------------------------------
struct PromptArgs {
  const void *q, *kv, *kv_step;      // [tokens][H][dim + rd]; [tokens][H][dim + vdim]; rows [tokens][2][hd]
  const int* q_start;
  void* out;                         // [tokens][H][vdim]
  const float* gate;                 // slices [gate_n][tokens][gate_row] from the gate's first column on, or null
  long long gate_stride;
  int gate_n, gate_row, gate_mode;   // 1 one logit per head, 2 one per feature
  const float* sink;
  int H, dim, rd, vdim, rank, hd, window;
  float scale_log2;
};
constexpr int LP_BQ = 64, LP_BK = 32;

// NV: 16-column groups of the values (vdim <= 16 NV)
template <typename T, int NV>
__global__ void __launch_bounds__(128, NV <= 8 ? 3 : 1)
attn_latent_prefill_kernel(PromptArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t lp_smem[];
  const int qd = a.dim + a.rd;
  const int nk = (qd + 15) / 16;
  const int ldk = nk * 16 + 8;
  constexpr int LDV = NV * 16 + 8;
  T* qt = reinterpret_cast<T*>(lp_smem);               // [64][ldk]
  T* kt = qt + LP_BQ * ldk;                            // two key blocks [64][ldk]
  T* vt = kt + 2 * LP_BK * ldk;                        // two value blocks [64][LDV]
  const int b = blockIdx.z, h = blockIdx.x, tile = gridDim.y - 1 - blockIdx.y;      // longest query tiles first
  const int qs = a.q_start[b], ql = a.q_start[b + 1] - qs;
  if (tile * LP_BQ >= ql) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int r0 = tile * LP_BQ + warp * 16 + g, r1 = r0 + 8;        // this thread's two query rows (= positions)
  const int p_first = tile * LP_BQ, p_last = min(p_first + LP_BQ, ql) - 1;
  const int j_lo = first_visible(p_first, a.window);
  const int n_blocks = (p_last - j_lo + LP_BK) / LP_BK;
  if (qd < nk * 16 || a.vdim < NV * 16) {              // columns that are never copied read as zero
    const int total = (LP_BQ + 2 * LP_BK) * ldk + 2 * LP_BK * LDV;
    for (int i = threadIdx.x; i < total / 8; i += blockDim.x) reinterpret_cast<uint4*>(lp_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
  }
  pdl_wait();
  const T* q = reinterpret_cast<const T*>(a.q);
  const T* kv = reinterpret_cast<const T*>(a.kv);
  const T* rows = reinterpret_cast<const T*>(a.kv_step);
  constexpr int TPR = 128 / LP_BK;                                 // threads that copy a key's row
  const int cr = threadIdx.x / TPR, ch = threadIdx.x % TPR;
  const int kvd = a.dim + a.vdim;
  {
    const int r = threadIdx.x >> 1, row = p_first + r;
    const bool on = row < ql;
    const T* src = q + ((size_t)(qs + (on ? row : 0)) * a.H + h) * qd;
    for (int c = threadIdx.x & 1; c < qd / 8; c += 2) cp16(qt + r * ldk + c * 8, src + c * 8, on ? 16 : 0);
  }
  auto issue = [&](int kb) {
    const int key = j_lo + kb * LP_BK + cr;
    const bool on = key <= p_last;
    const size_t tok = qs + (on ? key : 0);
    const T* src = kv + (tok * a.H + h) * kvd;
    const T* rope = rows + tok * 2 * a.hd + a.rank;
    T* kd = kt + (size_t)(kb & 1) * LP_BK * ldk + cr * ldk;
    T* vd = vt + (size_t)(kb & 1) * LP_BK * LDV + cr * LDV;
    const uint32_t bytes = on ? 16 : 0;
    for (int c = ch; c < a.dim / 8; c += TPR) cp16(kd + c * 8, src + c * 8, bytes);
    for (int c = ch; c < a.rd / 8; c += TPR) cp16(kd + a.dim + c * 8, rope + c * 8, bytes);
    for (int c = ch; c < a.vdim / 8; c += TPR) cp16(vd + c * 8, src + a.dim + c * 8, bytes);
    cp_commit();
  };
  float o[2 * NV][4];
#pragma unroll
  for (int i = 0; i < 2 * NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  if (a.sink != nullptr) {
    m[0] = m[1] = a.sink[h] * LOG2E;
    l[0] = l[1] = t4 == 0 ? 1.f : 0.f;
  }
  issue(0);
  const int mi = lane >> 3, mr = lane & 7;
  const uint32_t qaddr = smem_u32(qt + (warp * 16 + (lane & 15)) * ldk + (lane >> 4) * 8);
  for (int kb = 0; kb < n_blocks; ++kb) {
    const int base = j_lo + kb * LP_BK;
    if (kb + 1 < n_blocks) {                           // the next block's copies run under this block's products
      issue(kb + 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const T* ks = kt + (size_t)(kb & 1) * LP_BK * ldk;
    const T* vs = vt + (size_t)(kb & 1) * LP_BK * LDV;
    float s[LP_BK / 8][4];
#pragma unroll
    for (int i = 0; i < LP_BK / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    const uint32_t kaddr = smem_u32(ks + ((mi >> 1) * 8 + mr) * ldk + (mi & 1) * 8);
#pragma unroll 2
    for (int kk = 0; kk < nk; ++kk) {
      uint32_t qf[4];
      ldsm_x4(qf, qaddr + kk * 32);
#pragma unroll
      for (int n2 = 0; n2 < LP_BK / 16; ++n2) {
        uint32_t r[4];
        ldsm_x4(r, kaddr + (uint32_t)(n2 * 16 * ldk + kk * 16) * 2);
        mma16<T>(s[2 * n2], qf, r[0], r[1]);
        mma16<T>(s[2 * n2 + 1], qf, r[2], r[3]);
      }
    }
    // masks only where the block reaches a diagonal or a window's edge
    const bool edge = base + LP_BK - 1 > p_first + warp * 16 || base < first_visible(p_first + warp * 16 + 15, a.window) ||
                      base + LP_BK - 1 > p_last;
    const int lo0 = first_visible(r0, a.window), lo1 = first_visible(r1, a.window);
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < LP_BK / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int rr = e >> 1;
        float v = s[nt][e] * a.scale_log2;
        if (edge) {
          const int key = base + nt * 8 + 2 * t4 + (e & 1);
          if (key > (rr ? r1 : r0) || key < (rr ? lo1 : lo0)) v = -INFINITY;
        }
        s[nt][e] = v;
        mx[rr] = fmaxf(mx[rr], v);
      }
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 1));
      mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 2));
      const float mn = fmaxf(m[rr], mx[rr]);
      const float sub = mn > -INFINITY ? mn : 0.f;     // a row that has seen no key yet: exp2(-inf) = 0
      const float corr = exp2f(m[rr] - sub);
      m[rr] = mn;
      l[rr] *= corr;
      if (__any_sync(0xffffffffu, corr != 1.f)) {        // most blocks raise no maximum
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) { o[i][2 * rr] *= corr; o[i][2 * rr + 1] *= corr; }
      }
      float sum = 0.f;
#pragma unroll
      for (int nt = 0; nt < LP_BK / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float p = exp2f(s[nt][2 * rr + e] - sub);
          s[nt][2 * rr + e] = p;
          sum += p;
        }
      l[rr] += sum;
    }
    const uint32_t vaddr = smem_u32(vs + ((mi & 1) * 8 + mr) * LDV + (mi >> 1) * 8);
#pragma unroll
    for (int kk = 0; kk < LP_BK / 16; ++kk) {
      uint32_t hi[4], mid[4], low[4];
      three_terms<T>(s[2 * kk][0], s[2 * kk][1], hi[0], mid[0], low[0]);
      three_terms<T>(s[2 * kk][2], s[2 * kk][3], hi[1], mid[1], low[1]);
      three_terms<T>(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], mid[2], low[2]);
      three_terms<T>(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], mid[3], low[3]);
#pragma unroll
      for (int n2 = 0; n2 < NV; ++n2) {
        uint32_t r[4];
        ldsm_x4_trans(r, vaddr + (uint32_t)(kk * 16 * LDV + n2 * 16) * 2);
        mma16<T>(o[2 * n2], low, r[0], r[1]);
        mma16<T>(o[2 * n2 + 1], low, r[2], r[3]);
        mma16<T>(o[2 * n2], mid, r[0], r[1]);
        mma16<T>(o[2 * n2 + 1], mid, r[2], r[3]);
        mma16<T>(o[2 * n2], hi, r[0], r[1]);
        mma16<T>(o[2 * n2 + 1], hi, r[2], r[3]);
      }
    }
    __syncthreads();                                   // this buffer is copied into again two blocks on
  }
#pragma unroll
  for (int rr = 0; rr < 2; ++rr) {
    l[rr] += __shfl_xor_sync(0xffffffffu, l[rr], 1);
    l[rr] += __shfl_xor_sync(0xffffffffu, l[rr], 2);
    const int r = rr ? r1 : r0;
    if (r >= ql) continue;
    const float inv = 1.0f / l[rr];
    const float* gz = a.gate_mode ? a.gate + (size_t)(qs + r) * a.gate_row + (a.gate_mode == 1 ? h : h * a.vdim) : nullptr;
    const float hg = a.gate_mode == 1 ? 1.0f / (1.0f + expf(-sum_slices(gz, a.gate_n, a.gate_stride))) : 1.0f;
    T* dst = reinterpret_cast<T*>(a.out) + ((size_t)(qs + r) * a.H + h) * a.vdim;
#pragma unroll
    for (int i = 0; i < 2 * NV; ++i) {
      const int c = i * 8 + 2 * t4;
      if (c >= a.vdim) continue;                       // vdim is a multiple of 8
      float x = o[i][2 * rr] * inv * hg, y = o[i][2 * rr + 1] * inv * hg;
      if (a.gate_mode == 2) {
        x /= 1.0f + expf(-sum_slices(gz + c, a.gate_n, a.gate_stride));
        y /= 1.0f + expf(-sum_slices(gz + c + 1, a.gate_n, a.gate_stride));
      }
      *reinterpret_cast<uint32_t*>(dst + c) = pack2<T>(x, y);
    }
  }
}

}  // namespace yalm

using namespace yalm;

#define YALM_LA_LAUNCH(KERNEL, grid, threads, smem, ...)                                                       \
  do {                                                                                                         \
    static size_t attr = 48 * 1024;                                                                            \
    if ((smem) > attr) {                                                                                       \
      cudaError_t e = cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem));  \
      if (e != cudaSuccess) return (int)e;                                                                     \
      attr = (smem);                                                                                           \
    }                                                                                                          \
    launch_pdl(KERNEL, grid, dim3(threads), smem, stream, __VA_ARGS__);                                        \
  } while (0)

static size_t latent_mma_smem(int hd) {
  return ((size_t)(LA_HEADS + 2 * LA_KEYS) * (hd + 8) + 32 + 3 * LA_HEADS * LA_PP) * 2 + (size_t)2 * LA_HEADS * LA_SP * 4;
}

// whether yalm_latent_attention runs on tensor cores for these sizes
extern "C" int yalm_latent_attention_mma_usable(int dtype, int rank, int hd) {
  return (dtype == DT_BF16 || dtype == DT_F16) && rank > 0 && rank <= 512 && hd % 16 == 0 && hd >= rank &&
         latent_mma_smem(hd) <= 227 * 1024;
}

// The absorbed form.  q, out [tokens][H][hd]; kv_step [tokens][2][hd]; cache [slots][1][capacity][hd] or
// pages; with nsplit > 1 part_o [tokens][H][nsplit][rank] and part_ml [tokens][H][nsplit][2] instead of
// out, split s the keys from per_split s on (those of a query that sees fewer keys stay empty).  sink [H] float32 or null.  mma: 0 runs the FMA kernel whatever the type.
extern "C" int yalm_latent_attention(const void* q, const void* kv_step, const void* cache, const int* token_seq,
                                     const int* q_start, const int* seq_slot, const int* slot_pos, void* out,
                                     float* part_o, float* part_ml, int dtype, int n_tokens, int H, int rank,
                                     int hd, int capacity, int window, float scale, const float* sink, int nsplit,
                                     int per_split, int mma, const int* page_table, int pages_per_slot, int n_pages,
                                     cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || rank <= 0 || rank > 256 * LF_MAX_COLS || hd < rank || hd > 2048 || capacity <= 0 || window < 0) return -2;
  if (nsplit < 1 || nsplit > 64 || per_split < 0 || (nsplit > 1 && per_split <= 0) || !(scale > 0.f)) return -5;
  if (n_tokens > 65535 || (H + LF_HEADS - 1) / LF_HEADS > 65535) return -4;
  const LatentRows a = {kv_step, cache, token_seq, q_start, seq_slot, slot_pos, page_table, pages_per_slot, n_pages,
                        capacity, hd, rank, H, window, nsplit, per_split, scale * LOG2E, sink};
  const LatentOut o = {out, part_o, part_ml};
  if (mma && yalm_latent_attention_mma_usable(dtype, rank, hd)) {
    const dim3 grid(nsplit, (H + LA_HEADS - 1) / LA_HEADS, n_tokens);
    const size_t smem = latent_mma_smem(hd);
#define YALM_LA(T)                                                                                              \
  do {                                                                                                          \
    if (rank <= 128) YALM_LA_LAUNCH((attn_latent_mma_kernel<T, 2>), grid, LA_WARPS * 32, smem, (const T*)q, a, o);      \
    else if (rank <= 256) YALM_LA_LAUNCH((attn_latent_mma_kernel<T, 4>), grid, LA_WARPS * 32, smem, (const T*)q, a, o); \
    else YALM_LA_LAUNCH((attn_latent_mma_kernel<T, 8>), grid, LA_WARPS * 32, smem, (const T*)q, a, o);                  \
  } while (0)
    if (dtype == DT_BF16) YALM_LA(__nv_bfloat16);
    else YALM_LA(__half);
#undef YALM_LA
    YALM_LAUNCH_CHECK();
    return 0;
  }
  const dim3 grid(nsplit, (H + LF_HEADS - 1) / LF_HEADS, n_tokens);
  const size_t smem = (size_t)LF_HEADS * hd * sizeof(float);
  if (dtype == DT_F32) YALM_LA_LAUNCH(attn_latent_fma_kernel<float>, grid, 256, smem, (const float*)q, a, o);
  else if (dtype == DT_BF16) YALM_LA_LAUNCH(attn_latent_fma_kernel<__nv_bfloat16>, grid, 256, smem, (const __nv_bfloat16*)q, a, o);
  else if (dtype == DT_F16) YALM_LA_LAUNCH(attn_latent_fma_kernel<__half>, grid, 256, smem, (const __half*)q, a, o);
  else return -3;
  YALM_LAUNCH_CHECK();
  return 0;
}

static size_t latent_prefill_smem(int qd, int vdim) {
  const int nv = vdim <= 32 ? 2 : vdim <= 64 ? 4 : vdim <= 128 ? 8 : 16;
  const int ldk = (qd + 15) / 16 * 16 + 8;
  return ((size_t)(LP_BQ + 2 * LP_BK) * ldk + (size_t)2 * LP_BK * (nv * 16 + 8)) * 2;
}

// whether yalm_latent_prefill takes these sizes: 16-byte pieces, one block's tiles in shared memory
extern "C" int yalm_latent_prefill_usable(int dtype, int dim, int rd, int vdim, int rank, int hd) {
  return (dtype == DT_BF16 || dtype == DT_F16) && dim > 0 && dim % 8 == 0 && rd % 8 == 0 && vdim > 0 && vdim % 8 == 0 &&
         vdim <= 256 && rank % 8 == 0 && hd % 8 == 0 && latent_prefill_smem(dim + rd, vdim) <= 227 * 1024;
}

// The expanded form over sequences that start with this step: q [tokens][H][dim + rd] (rotated), kv
// [tokens][H][dim + vdim] = (key | value) per head, kv_step [tokens][2][hd] whose features rank ..
// rank + rd are the shared rotated key part; out [tokens][H][vdim], times the sigmoid of the gate
// (gate_mode 0 none, 1 one logit per head, 2 one per feature; float32 slices).
extern "C" int yalm_latent_prefill(const void* q, const void* kv, const void* kv_step, const int* q_start, void* out,
                                   int dtype, int n_seqs, int max_q_len, int H, int dim, int rd, int vdim, int rank,
                                   int hd, int window, float scale, const float* sink, const float* gate,
                                   int gate_mode, int gate_n, long long gate_stride, int gate_row, int gate_col0,
                                   cudaStream_t stream) {
  if (n_seqs <= 0 || max_q_len <= 0) return 0;
  if (!yalm_latent_prefill_usable(dtype, dim, rd, vdim, rank, hd) || window < 0 || H <= 0) return -2;
  if ((((uintptr_t)q | (uintptr_t)kv | (uintptr_t)kv_step) & 15) != 0) return -6;
  const dim3 grid(H, (max_q_len + LP_BQ - 1) / LP_BQ, n_seqs);
  if (grid.y > 65535 || grid.z > 65535) return -4;
  const PromptArgs a = {q, kv, kv_step, q_start, out, gate == nullptr ? nullptr : gate + gate_col0, gate_stride,
                        gate_n, gate_row, gate == nullptr ? 0 : gate_mode, sink, H, dim, rd, vdim, rank, hd, window,
                        scale * LOG2E};
  const size_t smem = latent_prefill_smem(dim + rd, vdim);
#define YALM_LP(T)                                                                                      \
  do {                                                                                                  \
    if (vdim <= 32) YALM_LA_LAUNCH((attn_latent_prefill_kernel<T, 2>), grid, 128, smem, a);             \
    else if (vdim <= 64) YALM_LA_LAUNCH((attn_latent_prefill_kernel<T, 4>), grid, 128, smem, a);        \
    else if (vdim <= 128) YALM_LA_LAUNCH((attn_latent_prefill_kernel<T, 8>), grid, 128, smem, a);       \
    else YALM_LA_LAUNCH((attn_latent_prefill_kernel<T, 16>), grid, 128, smem, a);                       \
  } while (0)
  if (dtype == DT_BF16) YALM_LP(__nv_bfloat16);
  else YALM_LP(__half);
#undef YALM_LP
  YALM_LAUNCH_CHECK();
  return 0;
}
