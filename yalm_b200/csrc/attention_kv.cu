// Causal grouped-query attention whose keys and values have sizes of their own, with an optional learned
// bias per distance and head, score = scale q.k + bias[head][min(i - j, last)], and an optional sink, a
// number per head whose exponential joins the softmax's denominator alone.  Scores, softmax weights and
// weighted sums are 32-bit.  Three kernels:
//
//  * attn_kv_prefill (16-bit): 64 queries of one head per block, keys 32 at a time through two cp.async
//    buffers, S = Q K^T and O += P V by mma.sync with every weight as three 16-bit terms (all its bits).  Keys of
//    this step come from its own buffer, earlier ones from the cache.
//  * attn_kv_decode (16-bit): one query per sequence, every key in the cache.  Transposed, S^T = K Q^T and
//    O^T = V^T P^T: the 16 rows of a tile are keys (or features of a value) and its 8 columns the query heads
//    that share a key head.  A warp walks through its own units of 16 keys with two cp.async buffers of its own, so
//    nothing but the end is a block's business, and two or three blocks share an SM; weights go from accumulators to operands in registers
//    (movmatrix), three terms each.  Long sequences are split over blocks; the block that ends last merges.
//  * attn_kv_fma: the same with 32-bit FMA on any storage type, any number of queries: the 32-bit path.
//
// kv_step [tokens][G dk + G dv]; caches [slots][G][capacity][dk] and [..][dv], or pages (see kv_row_offset).
#include "api.h"
#include "common.cuh"

namespace yalm {

namespace {

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
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// the transpose of an 8 x 8 matrix of 16-bit elements that the warp holds as a fragment
__device__ __forceinline__ uint32_t mov_trans(uint32_t v) {
  uint32_t r;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
  return r;
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

struct KvArgs {
  const void *q, *kv_step, *k_cache, *v_cache;
  const int *token_seq, *q_start, *seq_slot, *slot_pos;
  const int* page_table;
  int pps, n_pages, capacity, H, G, dk, dv;
  const float* bias;           // [H][n_bias], or null
  int n_bias;
  const float* sink;           // [H], or null
  float scale_log2;
  void* out;                   // [tokens][H][dv]
  int nsplit;                  // > 1: part_o [tokens][H][nsplit][dv], part_ml [..][2] (maximum in log2 units, sum)
  float *part_o, *part_ml;
  int* counters;
  int max_keys;
  int* status;
};

__device__ __forceinline__ float distance_bias(const KvArgs& a, int h, int back) {
  return __ldg(a.bias + (size_t)h * a.n_bias + min(max(back, 0), a.n_bias - 1)) * LOG2E;
}
template <typename T>
__device__ __forceinline__ void kv_rows(const KvArgs& a, int key, int past, int qs, int slot, int g, const T*& k, const T*& v) {
  if (key >= past) {
    const T* row = reinterpret_cast<const T*>(a.kv_step) + (size_t)(qs + key - past) * a.G * (a.dk + a.dv);
    k = row + g * a.dk;
    v = row + a.G * a.dk + g * a.dv;
  } else {
    const int r = key % a.capacity;
    const size_t at = kv_row_offset(a.page_table, a.pps, a.n_pages, slot, g, a.G, a.capacity, r, 1);    // rows before it
    k = reinterpret_cast<const T*>(a.k_cache) + at * a.dk;
    v = reinterpret_cast<const T*>(a.v_cache) + at * a.dv;
  }
}

// The last of a query's nsplit blocks (for `nh` heads from h0 on) adds their partial results up; every block
// calls it with its own already in part_o and part_ml.
template <typename T>
__device__ __forceinline__ void merge_splits(const KvArgs& a, int t, int h0, int nh, int* counter) {
  __shared__ int last_s;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) last_s = atomicAdd(counter, 1) == a.nsplit - 1;
  __syncthreads();
  if (!last_s) return;
  __threadfence();
  if (threadIdx.x == 0) *counter = 0;
  for (int i = threadIdx.x; i < nh * a.dv; i += blockDim.x) {
    const int r = i / a.dv, d = i - r * a.dv;
    const size_t first = ((size_t)t * a.H + h0 + r) * a.nsplit;
    float M = -INFINITY;
    for (int s = 0; s < a.nsplit; ++s) M = fmaxf(M, __ldcg(a.part_ml + (first + s) * 2));
    float L = 0.f, O = 0.f;
    for (int s = 0; s < a.nsplit; ++s) {
      const float m = __ldcg(a.part_ml + (first + s) * 2);
      if (m > -INFINITY) {                               // an empty part has written no output
        const float w = exp2f(m - M);
        L = fmaf(__ldcg(a.part_ml + (first + s) * 2 + 1), w, L);
        O = fmaf(__ldcg(a.part_o + (first + s) * a.dv + d), w, O);
      }
    }
    reinterpret_cast<T*>(a.out)[((size_t)t * a.H + h0 + r) * a.dv + d] = from_float<T>(O / L);
  }
}

// ---- prompts ------------------------------------------------------------------------------------------
constexpr int KP_BQ = 64, KP_BK = 32;

// NV: 16-column groups of the values (dv <= 16 NV)
template <typename T, int NV>
__global__ void __launch_bounds__(128, NV <= 8 ? 3 : 2)
attn_kv_prefill_kernel(KvArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t kp_smem[];
  const int nk = (a.dk + 15) / 16;
  const int ldk = nk * 16 + 8;
  constexpr int LDV = NV * 16 + 8;
  T* qt = reinterpret_cast<T*>(kp_smem);               // [64][ldk]
  T* kt = qt + KP_BQ * ldk;                            // two key blocks [32][ldk]
  T* vt = kt + 2 * KP_BK * ldk;                        // two value blocks [32][LDV]
  const int b = blockIdx.z, h = blockIdx.x, tile = gridDim.y - 1 - blockIdx.y;      // longest query tiles first
  const int qs = a.q_start[b], ql = a.q_start[b + 1] - qs;
  if (tile * KP_BQ >= ql) return;
  const int slot = a.seq_slot[b], past = a.slot_pos[slot], gkv = h / (a.H / a.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int r0 = tile * KP_BQ + warp * 16 + g, r1 = r0 + 8;        // this thread's two query rows
  const int p_first = past + tile * KP_BQ, p_last = past + min(tile * KP_BQ + KP_BQ, ql) - 1;
  const int n_blocks = p_last / KP_BK + 1;
  if (a.dk < nk * 16 || a.dv < NV * 16) {              // columns that are never copied read as zero
    const int total = (KP_BQ + 2 * KP_BK) * ldk + 2 * KP_BK * LDV;
    for (int i = threadIdx.x; i < total / 8; i += blockDim.x) reinterpret_cast<uint4*>(kp_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
  }
  pdl_wait();
  const T* q = reinterpret_cast<const T*>(a.q);
  constexpr int TPR = 128 / KP_BK;                                 // threads that copy a key's row
  const int cr = threadIdx.x / TPR, ch = threadIdx.x % TPR;
  {
    const int r = threadIdx.x >> 1, row = tile * KP_BQ + r;
    const bool on = row < ql;
    const T* src = q + ((size_t)(qs + (on ? row : 0)) * a.H + h) * a.dk;
    for (int c = threadIdx.x & 1; c < a.dk / 8; c += 2) cp16(qt + r * ldk + c * 8, src + c * 8, on ? 16 : 0);
  }
  auto issue = [&](int kb) {
    const int key = kb * KP_BK + cr;
    const bool on = key <= p_last;
    const T *ks = q, *vs = q;
    if (on) kv_rows<T>(a, key, past, qs, slot, gkv, ks, vs);
    T* kd = kt + (size_t)(kb & 1) * KP_BK * ldk + cr * ldk;
    T* vd = vt + (size_t)(kb & 1) * KP_BK * LDV + cr * LDV;
    const uint32_t bytes = on ? 16 : 0;
    for (int c = ch; c < a.dk / 8; c += TPR) cp16(kd + c * 8, ks + (on ? c * 8 : 0), bytes);
    for (int c = ch; c < a.dv / 8; c += TPR) cp16(vd + c * 8, vs + (on ? c * 8 : 0), bytes);
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
  const float far_bias = a.bias != nullptr ? distance_bias(a, h, a.n_bias) : 0.f;
  issue(0);
  const int mi = lane >> 3, mr = lane & 7;
  const uint32_t qaddr = smem_u32(qt + (warp * 16 + (lane & 15)) * ldk + (lane >> 4) * 8);
  const int w_first = p_first + warp * 16;             // this warp's first query position
  for (int kb = 0; kb < n_blocks; ++kb) {
    const int base = kb * KP_BK;
    if (kb + 1 < n_blocks) {                           // the next block's copies run under this block's products
      issue(kb + 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const T* ks = kt + (size_t)(kb & 1) * KP_BK * ldk;
    const T* vs = vt + (size_t)(kb & 1) * KP_BK * LDV;
    if (base <= w_first + 15) {                        // else no query of this warp sees any of these keys
    float s[KP_BK / 8][4];
#pragma unroll
    for (int i = 0; i < KP_BK / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    const uint32_t kaddr = smem_u32(ks + ((mi >> 1) * 8 + mr) * ldk + (mi & 1) * 8);
#pragma unroll 2
    for (int kk = 0; kk < nk; ++kk) {
      uint32_t qf[4];
      ldsm_x4(qf, qaddr + kk * 32);
#pragma unroll
      for (int n2 = 0; n2 < KP_BK / 16; ++n2) {
        uint32_t r[4];
        ldsm_x4(r, kaddr + (uint32_t)(n2 * 16 * ldk + kk * 16) * 2);
        mma16<T>(s[2 * n2], qf, r[0], r[1]);
        mma16<T>(s[2 * n2 + 1], qf, r[2], r[3]);
      }
    }
    // the mask only where the block reaches the diagonal; a table look-up only where distances are near
    const bool edge = base + KP_BK - 1 > w_first || base + KP_BK - 1 > p_last;
    const bool near = a.bias != nullptr && w_first - (base + KP_BK - 1) < a.n_bias - 1;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < KP_BK / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int rr = e >> 1;
        const int key = base + nt * 8 + 2 * t4 + (e & 1), pos = past + (rr ? r1 : r0);
        float v = fmaf(s[nt][e], a.scale_log2, near ? distance_bias(a, h, pos - key) : far_bias);
        if (edge && key > pos) v = -INFINITY;
        s[nt][e] = v;
        mx[rr] = fmaxf(mx[rr], v);
      }
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 1));
      mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 2));
      const float mn = fmaxf(m[rr], mx[rr]);           // position 0 is visible to every query
      const float corr = exp2f(m[rr] - mn);
      m[rr] = mn;
      l[rr] *= corr;
      if (__any_sync(0xffffffffu, corr != 1.f)) {        // most blocks raise no maximum
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) { o[i][2 * rr] *= corr; o[i][2 * rr + 1] *= corr; }
      }
      float sum = 0.f;
#pragma unroll
      for (int nt = 0; nt < KP_BK / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float p = exp2f(s[nt][2 * rr + e] - mn);
          s[nt][2 * rr + e] = p;
          sum += p;
        }
      l[rr] += sum;
    }
    const uint32_t vaddr = smem_u32(vs + ((mi & 1) * 8 + mr) * LDV + (mi >> 1) * 8);
#pragma unroll
    for (int kk = 0; kk < KP_BK / 16; ++kk) {
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
    T* dst = reinterpret_cast<T*>(a.out) + ((size_t)(qs + r) * a.H + h) * a.dv;
#pragma unroll
    for (int i = 0; i < 2 * NV; ++i) {
      const int c = i * 8 + 2 * t4;
      if (c < a.dv) *reinterpret_cast<uint32_t*>(dst + c) = pack2<T>(o[i][2 * rr] * inv, o[i][2 * rr + 1] * inv);
    }
  }
}

// ---- one query per sequence ---------------------------------------------------------------------------
constexpr int KD_HEADS = 8, KD_KEYS = 16, KD_WARPS = 4, KD_STAGES = 2;

// NK, NV: 16-feature groups of keys and values (dk <= 16 NK, dv <= 16 NV).  grid (splits, G * tiles of 8 query
// heads, sequences)
template <typename T, int NK, int NV>
__global__ void __launch_bounds__(KD_WARPS * 32)
attn_kv_decode_kernel(KvArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t kd_smem[];
  constexpr int LDK = NK * 16 + 8, LDV = NV * 16 + 8;              // row pitches: ldmatrix without bank conflicts
  constexpr int UNIT = KD_KEYS * (LDK + LDV);                      // one unit of 16 keys and values
  __shared__ float ml_s[KD_WARPS][KD_HEADS][2];
  const int R = a.H / a.G, tiles = (R + KD_HEADS - 1) / KD_HEADS;
  const int gkv = blockIdx.y / tiles, h0 = gkv * R + (blockIdx.y % tiles) * KD_HEADS;
  const int nh = min(KD_HEADS, (gkv + 1) * R - h0);
  const int b = blockIdx.z, split = blockIdx.x;
  const int slot = a.seq_slot[b], pos = a.slot_pos[slot], n_keys = pos + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int per = ((n_keys + a.nsplit - 1) / a.nsplit + KD_KEYS - 1) / KD_KEYS * KD_KEYS;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  T* ring = reinterpret_cast<T*>(kd_smem) + (size_t)warp * KD_STAGES * UNIT;
  if (a.dk < NK * 16 || a.dv < NV * 16)                            // columns that are never copied read as zero
    for (int i = lane; i < KD_STAGES * UNIT / 8; i += 32) reinterpret_cast<uint4*>(ring)[i] = make_uint4(0u, 0u, 0u, 0u);
  __syncwarp();
  pdl_wait();
  if (n_keys > a.max_keys && split == 0 && threadIdx.x == 0) atomicOr(a.status, ERR_CONTEXT_RANGE);
  const T* q = reinterpret_cast<const T*>(a.q) + ((size_t)b * a.H + h0) * a.dk;
  const int n_units = k1 > k0 ? (k1 - k0 + KD_KEYS - 1) / KD_KEYS : 0;
  const int mine = n_units > warp ? (n_units - warp + KD_WARPS - 1) / KD_WARPS : 0;      // units warp, warp + 4, ..
  // two lanes copy a key: its row of K and of V in 16-byte pieces
  const int cr = lane >> 1, ch = lane & 1;
  auto issue = [&](int u) {
    if (u < mine) {
      const int key = k0 + (warp + u * KD_WARPS) * KD_KEYS + cr;
      const bool on = key < k1;
      const size_t at = on ? kv_row_offset(a.page_table, a.pps, a.n_pages, slot, gkv, a.G, a.capacity, key % a.capacity, 1) : 0;
      const T* ks = reinterpret_cast<const T*>(a.k_cache) + at * a.dk;
      const T* vs = reinterpret_cast<const T*>(a.v_cache) + at * a.dv;
      T* kd = ring + (size_t)(u % KD_STAGES) * UNIT + cr * LDK;
      T* vd = ring + (size_t)(u % KD_STAGES) * UNIT + KD_KEYS * LDK + cr * LDV;
      const uint32_t bytes = on ? 16 : 0;
      for (int c = ch; c < a.dk / 8; c += 2) cp16(kd + c * 8, ks + c * 8, bytes);
      for (int c = ch; c < a.dv / 8; c += 2) cp16(vd + c * 8, vs + c * 8, bytes);
    }
    cp_commit();
  };
  issue(0);
  issue(1);
  // the queries as the products' second operand: head g, features 2 t4 ..
  uint32_t qf[NK][2];
#pragma unroll
  for (int kk = 0; kk < NK; ++kk)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int f = kk * 16 + e * 8 + 2 * t4;
      qf[kk][e] = g < nh && f < a.dk ? *reinterpret_cast<const uint32_t*>(q + (size_t)g * a.dk + f) : 0u;
    }
  float o[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  // heads 2 t4 and 2 t4 + 1: maxima are the warp's, sums this lane's own part
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, far[2] = {0.f, 0.f};
  const int hd[2] = {h0 + min(2 * t4, nh - 1), h0 + min(2 * t4 + 1, nh - 1)};
#pragma unroll
  for (int c = 0; c < 2; ++c) {
    if (a.sink != nullptr && split == 0 && warp == 0) {
      m[c] = a.sink[hd[c]] * LOG2E;
      l[c] = g == 0 ? 1.f : 0.f;
    }
    if (a.bias != nullptr) far[c] = distance_bias(a, hd[c], a.n_bias);
  }
  const int mi = lane >> 3, mr = lane & 7;
  for (int u = 0; u < mine; ++u) {
    const int base = k0 + (warp + u * KD_WARPS) * KD_KEYS;
    float bias[4] = {far[0], far[1], far[0], far[1]};
    if (a.bias != nullptr && pos - (base + KD_KEYS - 1) < a.n_bias - 1) {
#pragma unroll
      for (int e = 0; e < 4; ++e) bias[e] = distance_bias(a, hd[e & 1], pos - (base + g + 8 * (e >> 1)));
    }
    cp_wait<KD_STAGES - 1>();
    __syncwarp();
    const T* ks = ring + (size_t)(u % KD_STAGES) * UNIT;
    const T* vs = ks + KD_KEYS * LDK;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const uint32_t ka = smem_u32(ks + ((mi & 1) * 8 + mr) * LDK + (mi >> 1) * 8);
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      uint32_t r[4];
      ldsm_x4(r, ka + kk * 32);
      mma16<T>(s[kk & 1], r, qf[kk][0], qf[kk][1]);
    }
    float x[4], mx[2];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      x[e] = fmaf(s[0][e] + s[1][e], a.scale_log2, bias[e]);
      if (base + g + 8 * (e >> 1) >= k1) x[e] = -INFINITY;
    }
    bool moved = false;
    float corr[2];
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      mx[c] = fmaxf(x[c], x[c + 2]);
      mx[c] = fmaxf(mx[c], __shfl_xor_sync(0xffffffffu, mx[c], 4));
      mx[c] = fmaxf(mx[c], __shfl_xor_sync(0xffffffffu, mx[c], 8));
      mx[c] = fmaxf(mx[c], __shfl_xor_sync(0xffffffffu, mx[c], 16));
      const float mn = fmaxf(m[c], mx[c]);               // a unit has at least one key
      corr[c] = exp2f(m[c] - mn);
      moved |= corr[c] != 1.f;
      m[c] = mn;
      x[c] = exp2f(x[c] - mn);
      x[c + 2] = exp2f(x[c + 2] - mn);
      l[c] = fmaf(l[c], corr[c], x[c] + x[c + 2]);
    }
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int i = 0; i < NV; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[1]; o[i][2] *= corr[0]; o[i][3] *= corr[1]; }
    }
    uint32_t p[3][2];                                    // [term][keys 0-7, 8-15]
    three_terms<T>(x[0], x[1], p[0][0], p[1][0], p[2][0]);
    three_terms<T>(x[2], x[3], p[0][1], p[1][1], p[2][1]);
#pragma unroll
    for (int term = 0; term < 3; ++term) {
      p[term][0] = mov_trans(p[term][0]);
      p[term][1] = mov_trans(p[term][1]);
    }
    const uint32_t va = smem_u32(vs + ((mi >> 1) * 8 + mr) * LDV + (mi & 1) * 8);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      uint32_t r[4];
      ldsm_x4_trans(r, va + i * 32);
      mma16<T>(o[i], r, p[2][0], p[2][1]);               // the small terms first
      mma16<T>(o[i], r, p[1][0], p[1][1]);
      mma16<T>(o[i], r, p[0][0], p[0][1]);
    }
    __syncwarp();                                        // this unit's buffer may be copied into again
    issue(u + 2);
  }
  cp_wait<0>();
#pragma unroll
  for (int c = 0; c < 2; ++c) {
    l[c] += __shfl_xor_sync(0xffffffffu, l[c], 4);
    l[c] += __shfl_xor_sync(0xffffffffu, l[c], 8);
    l[c] += __shfl_xor_sync(0xffffffffu, l[c], 16);
    if (g == 0) {
      ml_s[warp][2 * t4 + c][0] = m[c];
      ml_s[warp][2 * t4 + c][1] = l[c];
    }
  }
  __syncthreads();                                       // every warp is done with its ring
  float* os = reinterpret_cast<float*>(kd_smem);         // [warps][8 heads][NV 16 + 4]
  constexpr int LDO = NV * 16 + 4;
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      os[((size_t)warp * KD_HEADS + 2 * t4 + (e & 1)) * LDO + i * 16 + g + 8 * (e >> 1)] = o[i][e];
  __syncthreads();
  for (int i = threadIdx.x; i < nh * a.dv; i += blockDim.x) {
    const int r = i / a.dv, d = i - r * a.dv;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < KD_WARPS; ++w) M = fmaxf(M, ml_s[w][r][0]);
    float L = 0.f, O = 0.f;
    if (M > -INFINITY) {
#pragma unroll
      for (int w = 0; w < KD_WARPS; ++w) {
        const float f = exp2f(ml_s[w][r][0] - M);
        L = fmaf(ml_s[w][r][1], f, L);
        O = fmaf(os[((size_t)w * KD_HEADS + r) * LDO + d], f, O);
      }
    }
    const size_t th = (size_t)b * a.H + h0 + r;
    if (a.nsplit == 1) {
      reinterpret_cast<T*>(a.out)[th * a.dv + d] = from_float<T>(O / L);
    } else {
      const size_t at = th * a.nsplit + split;
      a.part_o[at * a.dv + d] = O;
      if (d == 0) {
        a.part_ml[at * 2] = M;
        a.part_ml[at * 2 + 1] = L;
      }
    }
  }
  if (a.nsplit > 1) merge_splits<T>(a, b, h0, nh, a.counters + (size_t)b * gridDim.y + blockIdx.y);
}

// ---- 32-bit FMA on any storage type -------------------------------------------------------------------
constexpr int KF_HEADS = 4, KF_KEYS = 64;

// grid (splits, G * tiles of 4 query heads, tokens); a thread owns one value column
template <typename T>
__global__ void __launch_bounds__(256)
attn_kv_fma_kernel(KvArgs a, int t_first) {
  pdl_launch_dependents();
  extern __shared__ float kf_q[];                        // [KF_HEADS][dk]
  __shared__ float s_s[KF_HEADS][KF_KEYS];
  __shared__ float corr_s[KF_HEADS], l_s[KF_HEADS];
  __shared__ const T *k_s[KF_KEYS], *v_s[KF_KEYS];
  const int R = a.H / a.G, tiles = (R + KF_HEADS - 1) / KF_HEADS;
  const int gkv = blockIdx.y / tiles, h0 = gkv * R + (blockIdx.y % tiles) * KF_HEADS;
  const int nh = min(KF_HEADS, (gkv + 1) * R - h0);
  const int t = t_first + blockIdx.z, split = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = a.token_seq[t], slot = a.seq_slot[b], qs = a.q_start[b];
  const int past = a.slot_pos[slot], pos = past + (t - qs), n_keys = pos + 1;
  const int per = (n_keys + a.nsplit - 1) / a.nsplit;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  pdl_wait();
  for (int i = threadIdx.x; i < KF_HEADS * a.dk; i += blockDim.x)
    kf_q[i] = i / a.dk < nh ? to_float(reinterpret_cast<const T*>(a.q)[((size_t)t * a.H + h0) * a.dk + i]) : 0.f;
  float acc[KF_HEADS] = {0.f, 0.f, 0.f, 0.f};
  const int f = threadIdx.x;
  float m = -INFINITY, l = 0.f;                          // warp r < KF_HEADS: head r
  if (a.sink != nullptr && split == 0 && warp < nh) {
    m = a.sink[h0 + warp] * LOG2E;
    l = 1.f;
  }
  for (int base = k0; base < k1; base += KF_KEYS) {
    const int n = min(KF_KEYS, k1 - base);
    __syncthreads();                                     // the last tile's weights and rows are no longer read
    if (threadIdx.x < n) kv_rows<T>(a, base + threadIdx.x, past, qs, slot, gkv, k_s[threadIdx.x], v_s[threadIdx.x]);
    __syncthreads();
    for (int k = warp; k < n; k += 8) {
      const T* row = k_s[k];
      float d[KF_HEADS] = {0.f, 0.f, 0.f, 0.f};
      for (int i = lane; i < a.dk; i += 32) {
        const float v = to_float(row[i]);
#pragma unroll
        for (int r = 0; r < KF_HEADS; ++r) d[r] = fmaf(kf_q[r * a.dk + i], v, d[r]);
      }
#pragma unroll
      for (int r = 0; r < KF_HEADS; ++r) {
        d[r] = warp_sum(d[r]) * a.scale_log2;
        if (lane == r) s_s[r][k] = d[r] + (a.bias != nullptr && r < nh ? distance_bias(a, h0 + r, pos - (base + k)) : 0.f);
      }
    }
    __syncthreads();
    if (warp < KF_HEADS) {
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
    for (int r = 0; r < KF_HEADS; ++r) acc[r] *= corr_s[r];
    if (f < a.dv)
      for (int k = 0; k < n; ++k) {
        const float v = to_float(v_s[k][f]);
#pragma unroll
        for (int r = 0; r < KF_HEADS; ++r) acc[r] = fmaf(s_s[r][k], v, acc[r]);
      }
  }
  if (warp < nh && lane == 0) {
    l_s[warp] = l;
    if (a.nsplit > 1) {
      float* ml = a.part_ml + (((size_t)t * a.H + h0 + warp) * a.nsplit + split) * 2;
      ml[0] = m;
      ml[1] = l;
    }
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < KF_HEADS; ++r) {
    if (r >= nh || f >= a.dv) continue;
    const size_t th = (size_t)t * a.H + h0 + r;
    if (a.nsplit > 1) a.part_o[(th * a.nsplit + split) * a.dv + f] = acc[r];
    else reinterpret_cast<T*>(a.out)[th * a.dv + f] = from_float<T>(acc[r] / l_s[r]);
  }
  if (a.nsplit > 1) merge_splits<T>(a, t, h0, nh, a.counters + (size_t)t * gridDim.y + blockIdx.y);
}

}  // namespace
}  // namespace yalm

using namespace yalm;

#define YALM_KV_LAUNCH(KERNEL, grid, threads, smem, ...)                                                       \
  do {                                                                                                         \
    static size_t attr = 0;                                                                                    \
    if ((smem) > attr) {                                                                                       \
      cudaError_t e = cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem));  \
      if (e != cudaSuccess) return (int)e;                                                                     \
      attr = (smem);                                                                                           \
    }                                                                                                          \
    launch_pdl(KERNEL, grid, dim3(threads), smem, stream, __VA_ARGS__);                                        \
  } while (0)

// q [tokens][H][dk], out [tokens][H][dv]; kv_step [tokens][G dk + G dv]; dk and dv up to 256 (16-bit: multiples of
// 8).  bias float32 [H][n_bias] or null, sink float32 [H] or null.  decode: every sequence brings one token whose
// row is in the caches already, no position is beyond max_keys - 1.  mma: 0 runs the FMA kernel whatever the type.
// nsplit > 1 (with decode, or the FMA kernel): part_o [tokens][H][nsplit][dv], part_ml [tokens][H][nsplit][2]
// float32 scratch, counters int32 [tokens][G * ceil(H / G / 4)], zero before the first call and after each.
extern "C" int yalm_attention_kv(const void* q, const void* kv_step, const void* k_cache, const void* v_cache,
                                 const int* token_seq, const int* q_start, const int* seq_slot, const int* slot_pos,
                                 void* out, int dtype, int n_tokens, int n_seqs, int max_q_len, int H, int G, int dk,
                                 int dv, int capacity, float scale, const float* bias, int n_bias, const float* sink,
                                 int decode, int mma, int nsplit, float* part_o, float* part_ml, int* counters,
                                 int max_keys, int* status, const int* page_table, int pages_per_slot, int n_pages,
                                 cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || dk > 256 || dv > 256 || capacity <= 0 || !(scale > 0.f)) return -2;
  if ((bias != nullptr && n_bias <= 0) || nsplit < 1 || nsplit > 1024 || (decode && n_tokens != n_seqs)) return -3;
  if (nsplit > 1 && (part_o == nullptr || part_ml == nullptr || counters == nullptr)) return -3;
  const KvArgs a = {q, kv_step, k_cache, v_cache, token_seq, q_start, seq_slot, slot_pos, page_table, pages_per_slot,
                    n_pages, capacity, H, G, dk, dv, bias, n_bias, sink, scale * LOG2E, out, nsplit, part_o, part_ml,
                    counters, max_keys, status};
  const bool half = dtype == DT_BF16 || dtype == DT_F16;
  if (half && mma) {
    if (dk % 8 || dv % 8) return -2;
    if ((((uintptr_t)q | (uintptr_t)kv_step | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)out) & 15) != 0) return -6;
  }
  if (half && mma && decode) {
    const dim3 grid(nsplit, G * ((H / G + KD_HEADS - 1) / KD_HEADS), n_seqs);
    if (grid.y > 65535 || grid.z > 65535) return -4;
#define YALM_KD1(T, K, V)                                                                                     \
  do {                                                                                                        \
    const size_t ring = (size_t)KD_WARPS * KD_STAGES * KD_KEYS * (K * 16 + 8 + V * 16 + 8) * 2;               \
    const size_t sums = (size_t)KD_WARPS * KD_HEADS * (V * 16 + 4) * 4;                                       \
    const size_t smem = ring > sums ? ring : sums;                                                            \
    YALM_KV_LAUNCH((attn_kv_decode_kernel<T, K, V>), grid, KD_WARPS * 32, smem, a);                           \
  } while (0)
#define YALM_KD2(T, K)                   \
  do {                                   \
    if (dv <= 64) YALM_KD1(T, K, 4);     \
    else if (dv <= 128) YALM_KD1(T, K, 8); \
    else if (dv <= 192) YALM_KD1(T, K, 12); \
    else YALM_KD1(T, K, 16);             \
  } while (0)
#define YALM_KD(T)                       \
  do {                                   \
    if (dk <= 64) YALM_KD2(T, 4);        \
    else if (dk <= 128) YALM_KD2(T, 8);  \
    else YALM_KD2(T, 16);                \
  } while (0)
    if (dtype == DT_BF16) YALM_KD(__nv_bfloat16);
    else YALM_KD(__half);
#undef YALM_KD
#undef YALM_KD2
#undef YALM_KD1
    YALM_LAUNCH_CHECK();
    return 0;
  }
  if (half && mma) {
    if (nsplit != 1) return -3;
    const dim3 grid(H, (max_q_len + KP_BQ - 1) / KP_BQ, n_seqs);
    if (grid.y > 65535 || grid.z > 65535) return -4;
    const int ldk = (dk + 15) / 16 * 16 + 8;
#define YALM_KP1(T, NV)                                                                                   \
  do {                                                                                                    \
    const size_t smem = ((size_t)(KP_BQ + 2 * KP_BK) * ldk + (size_t)2 * KP_BK * (NV * 16 + 8)) * 2;      \
    YALM_KV_LAUNCH((attn_kv_prefill_kernel<T, NV>), grid, 128, smem, a);                                  \
  } while (0)
#define YALM_KP(T)                       \
  do {                                   \
    if (dv <= 32) YALM_KP1(T, 2);        \
    else if (dv <= 64) YALM_KP1(T, 4);   \
    else if (dv <= 96) YALM_KP1(T, 6);   \
    else if (dv <= 128) YALM_KP1(T, 8);  \
    else if (dv <= 192) YALM_KP1(T, 12); \
    else YALM_KP1(T, 16);                \
  } while (0)
    if (dtype == DT_BF16) YALM_KP(__nv_bfloat16);
    else YALM_KP(__half);
#undef YALM_KP
#undef YALM_KP1
    YALM_LAUNCH_CHECK();
    return 0;
  }
  const int groups = G * ((H / G + KF_HEADS - 1) / KF_HEADS);
  if (groups > 65535) return -4;
  const size_t smem = (size_t)KF_HEADS * dk * sizeof(float);
  for (int t0 = 0; t0 < n_tokens; t0 += 65535) {         // gridDim.z is limited
    const dim3 grid(nsplit, groups, n_tokens - t0 < 65535 ? n_tokens - t0 : 65535);
    if (dtype == DT_F32) YALM_KV_LAUNCH(attn_kv_fma_kernel<float>, grid, 256, smem, a, t0);
    else if (dtype == DT_BF16) YALM_KV_LAUNCH(attn_kv_fma_kernel<__nv_bfloat16>, grid, 256, smem, a, t0);
    else if (dtype == DT_F16) YALM_KV_LAUNCH(attn_kv_fma_kernel<__half>, grid, 256, smem, a, t0);
    else return -3;
    YALM_LAUNCH_CHECK();
  }
  return 0;
}
