// What the scans over a state in packed pairs of floats share (ssd.cu, gla.cu): packed arithmetic, the
// form in which a decay is applied, asynchronous copies, and the cut of a ragged step into runs.
#pragma once
#include "common.cuh"

namespace yalm {

// tokens per stage of the ring and stages, tokens per run; a lane group of 16 owns CPL = 4 columns of the state (2
// where blocks of half as many columns fill the device better), a block of four warps 8 CPL
constexpr int SS_TOK = 16, SS_STAGES = 3, SS_RUN = 8;

typedef unsigned long long f2;                           // two packed floats
__device__ __forceinline__ f2 pack_f2(float lo, float hi) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void unpack_f2(f2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f2 fma_f2(f2 a, f2 b, f2 c) {
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f2 mul_f2(f2 a, f2 b) {
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f2 add_f2(f2 a, f2 b) {
  f2 r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ float sum_f2(f2 a, f2 b) {    // the sum of all four
  float lo, hi;
  unpack_f2(add_f2(a, b), lo, hi);
  return lo + hi;
}
template <int BYTES>
__device__ __forceinline__ void ss_copy(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(dst)), "l"(src), "n"(BYTES) : "memory");
}

// the same columns of nt <= SS_TOK tokens: a whole stage's copies go out without a test or a loop between them
template <int BYTES>
__device__ __forceinline__ void ss_copy_tokens(float* dst, int dst_pitch, const float* src, int src_pitch, int nt) {
  if (nt == SS_TOK) {
#pragma unroll
    for (int tt = 0; tt < SS_TOK; ++tt) ss_copy<BYTES>(dst + tt * dst_pitch, src + (size_t)tt * src_pitch);
  } else {
    for (int tt = 0; tt < nt; ++tt) ss_copy<BYTES>(dst + tt * dst_pitch, src + (size_t)tt * src_pitch);
  }
}

__device__ __forceinline__ float softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// A factor exp(a) as it is applied: S <- coef S + keep S, with keep 1 where coef = exp(a) - 1 (its sign bit is
// set, also for a = 0) and 0 where coef = exp(a): a below -0.69, or above 0 (what rounding leaves of a
// logarithm that is 0)
__device__ __forceinline__ float decay_coef(float a) { return a > -0.69f && a <= 0.f ? copysignf(expm1f(a), -1.f) : expf(a); }
__device__ __forceinline__ float decay_keep(float coef) { return signbit(coef) ? 1.f : 0.f; }

// The step's sequences are cut into runs of RUN tokens, each sequence from its own first token on.  Run
// number `index`: its sequence and its first token within that; false beyond the last.  Every lane of a
// warp calls it.
template <int RUN>
__device__ __forceinline__ bool find_run(const int* __restrict__ q_start, int n_seqs, int index, int& seq, int& first) {
  const int lane = threadIdx.x & 31;
  for (int base = 0; base < n_seqs; base += 32) {
    const int b = base + lane;
    const int count = b < n_seqs ? (q_start[b + 1] - q_start[b] + RUN - 1) / RUN : 0;
    int upto = count;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, upto, o);
      if (lane >= o) upto += v;
    }
    const int total = __shfl_sync(0xffffffffu, upto, 31);
    if (index < total) {
      const int who = __ffs(__ballot_sync(0xffffffffu, upto > index)) - 1;
      seq = base + who;
      first = (index - (__shfl_sync(0xffffffffu, upto, who) - __shfl_sync(0xffffffffu, count, who))) * RUN;
      return true;
    }
    index -= total;
  }
  return false;
}

// 8 CPL sums over 16 lanes, value number CPL tt + c of each lane's o: in every round a lane hands half of its values
// over and adds the other half of its partner's; lane `sub` of the 16 ends with the whole sums from number
// sub CPL / 2 on, CPL / 2 of them (token sub / 2, columns (sub % 2) CPL / 2 ..)
template <int CPL>
__device__ __forceinline__ void run_sums(float* o, int lane) {
  static_assert(CPL == 4 || CPL == 2, "two outputs or one per lane");
#pragma unroll
  for (int bit = 8, half = 4 * CPL; bit >= 1; bit >>= 1, half >>= 1) {
    const bool upper = (lane & bit) != 0;
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float send = upper ? o[i] : o[i + half];
      const float keep = upper ? o[i + half] : o[i];
      o[i] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
    }
  }
}
// CPL neighbouring values, from shared memory
template <int CPL>
__device__ __forceinline__ void load_columns(const float* p, float* x) {
  if constexpr (CPL == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
  } else {
    const float2 v = *reinterpret_cast<const float2*>(p);
    x[0] = v.x; x[1] = v.y;
  }
}
// What one token brings to a lane: its rows of two vectors (C read, B written) and its columns' values.  A run's
// tokens are fetched one ahead of their use, so that a warp alone on its scheduler does not wait for shared memory.
template <int K4, int CPL>
struct RunToken {
  ulonglong2 C[K4], B[K4];
  float x[CPL];
  __device__ __forceinline__ void fetch(const float* c, const float* b, const float* v) {
#pragma unroll
    for (int k = 0; k < K4; ++k) {
      B[k] = *reinterpret_cast<const ulonglong2*>(b + 64 * k);
      C[k] = *reinterpret_cast<const ulonglong2*>(c + 64 * k);
    }
    load_columns<CPL>(v, x);
  }
  // S += B x^T, then o[c] = this lane's part of S^T C
  __device__ __forceinline__ void apply(f2 (*S)[2 * K4], float* o) const {
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      const f2 xd = pack_f2(x[c], x[c]);
#pragma unroll
      for (int k = 0; k < K4; ++k) {
        S[c][2 * k] = fma_f2(B[k].x, xd, S[c][2 * k]);
        S[c][2 * k + 1] = fma_f2(B[k].y, xd, S[c][2 * k + 1]);
      }
    }
    f2 lo[CPL], hi[CPL];
#pragma unroll
    for (int k = 0; k < K4; ++k)
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        lo[c] = k == 0 ? mul_f2(S[c][0], C[0].x) : fma_f2(S[c][2 * k], C[k].x, lo[c]);
        hi[c] = k == 0 ? mul_f2(S[c][1], C[0].y) : fma_f2(S[c][2 * k + 1], C[k].y, hi[c]);
      }
#pragma unroll
    for (int c = 0; c < CPL; ++c) o[c] = sum_f2(lo[c], hi[c]);
  }
};
// whether blocks of half as many columns (CPL 2) are worth it: the usual ones leave a third of the SMs idle
inline bool narrow_blocks(long long blocks) { return blocks <= 96; }

// The lane's rows of one state column (K4 groups of four: rows 64 k + 4 sub + j), N rows in memory
template <int K4, bool VEC>
__device__ __forceinline__ void load_column(const float* __restrict__ col, int N, int sub, bool on, f2* S) {
#pragma unroll
  for (int k = 0; k < K4; ++k) {
    const int i = 64 * k + 4 * sub;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on) {
      if constexpr (VEC) {
        if (i < N) v = *reinterpret_cast<const float4*>(col + i);
      } else {
        if (i < N) v.x = col[i];
        if (i + 1 < N) v.y = col[i + 1];
        if (i + 2 < N) v.z = col[i + 2];
        if (i + 3 < N) v.w = col[i + 3];
      }
    }
    S[2 * k] = pack_f2(v.x, v.y);
    S[2 * k + 1] = pack_f2(v.z, v.w);
  }
}
template <int K4, bool VEC>
__device__ __forceinline__ void store_column(float* __restrict__ col, int N, int sub, const f2* S) {
#pragma unroll
  for (int k = 0; k < K4; ++k) {
    const int i = 64 * k + 4 * sub;
    float4 v;
    unpack_f2(S[2 * k], v.x, v.y);
    unpack_f2(S[2 * k + 1], v.z, v.w);
    if constexpr (VEC) {
      if (i < N) *reinterpret_cast<float4*>(col + i) = v;
    } else {
      if (i < N) col[i] = v.x;
      if (i + 1 < N) col[i + 1] = v.y;
      if (i + 2 < N) col[i + 2] = v.z;
      if (i + 3 < N) col[i + 3] = v.w;
    }
  }
}

}  // namespace yalm
