// Gated linear attention with a decay per key channel, per head with key size dk and value size dv:
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,
//   log alpha_t = logsigmoid(z_t) / tau,   z_t = W2 l_t + b      (l_t: a few values per token, rank of them)
// so the read-out sees the current token.  Everything here is 32-bit.  Three kernels:
//
//  * gla_prep: what the scan reads.  A block takes one run of GL_RUN tokens of one head, a thread one key
//    channel: it forms z (rank multiply-adds per token), the logarithms of the decays and, with c_t their
//    sum from the run's first token on, writes q e^(c_t) and k e^(-c_t) and the run's whole decay: within
//    the run
//        T_t = T_(t-1) + (k e^(-c)) v^T,   o_t = T_t^T (q e^(c)),
//    needs no decay per element, and S = diag(e^(c_last)) T at the run's end.  A run in which some channel
//    forgets more than e^(-GL_SPAN) is marked instead: q and k stay as they are and every token has its
//    own decays.  Decays are kept in the form of decay_coef (scan.cuh).
//  * gla_scan: the recurrence.  As in ssd_scan a block owns 32 (or 16) value columns of one (sequence, head), 16
//    lanes own four (or two) of them, four warps compute and a fifth brings the tokens through a cp.async ring.
//  * gla_step: one token per sequence, the state streamed once: a warp per eight columns.
//
// A token's row, float32: [q: H dk | k: H dk | decays: H dk | v: H dv]; a product in one slice keeps its v columns
// where they are.  State [slots][H][dv][dk].
#include "api.h"
#include "scan.cuh"

namespace yalm {

constexpr int GL_RUN = SS_RUN;
constexpr float GL_SPAN = 30.f;

struct GlaPrep {
  const float* proj;           // slices [n_partials][tokens][proj_row]; q, k, v, l at their columns
  int n_partials, proj_row, col_q, col_k, col_v, col_low, rank;
  long long partial_stride;
  const float* w2;             // [rank][H dk]
  const float* bias;           // [H dk]
  float* act;
  int* marks;                  // [tokens][H], at a run's first token
  const int* q_start;
  int n_seqs, H, dk, dv, per_token, copy_v;
  float inv_tau, q_scale;
};

// grid (runs, heads); one thread per key channel.  ONE: the product came in one slice, so that an element is one
// load and all of a thread's are in flight at once
template <bool ONE>
__global__ void __launch_bounds__(256) gla_prep_kernel(GlaPrep a) {
  pdl_launch_dependents();
  extern __shared__ float low_s[];                       // [GL_RUN][rank]
  int b, first;
  if (!find_run<GL_RUN>(a.q_start, a.n_seqs, blockIdx.x, b, first)) return;
  const int h = blockIdx.y, qs = a.q_start[b];
  const int nt = min(GL_RUN, a.q_start[b + 1] - qs - first);
  const int t0 = qs + first, n_k = a.H * a.dk, row = 3 * n_k + a.H * a.dv;
  pdl_wait();
  const float* p = a.proj + (size_t)t0 * a.proj_row;
  auto get = [&](const float* e) { return ONE ? *e : sum_slices(e, a.n_partials, a.partial_stride); };
  const int c = threadIdx.x, ch = h * a.dk + c;
  const bool on = c < a.dk;
  float q[GL_RUN], k[GL_RUN];
  if (on) {
#pragma unroll
    for (int tt = 0; tt < GL_RUN; ++tt)
      if (tt < nt) {
        q[tt] = get(p + (size_t)tt * a.proj_row + a.col_q + ch) * a.q_scale;
        k[tt] = get(p + (size_t)tt * a.proj_row + a.col_k + ch);
      }
  }
  for (int e = threadIdx.x; e < nt * a.rank; e += blockDim.x) {
    const int tt = e / a.rank, r = e - tt * a.rank;
    low_s[e] = get(p + (size_t)tt * a.proj_row + a.col_low + r);
  }
  __syncthreads();
  float la[GL_RUN], sum = -0.f;
  if (on) {
    const float bias = a.bias[ch];
#pragma unroll
    for (int tt = 0; tt < GL_RUN; ++tt) la[tt] = bias;
    for (int r = 0; r < a.rank; ++r) {
      const float w = a.w2[(size_t)r * n_k + ch];
#pragma unroll
      for (int tt = 0; tt < GL_RUN; ++tt)
        if (tt < nt) la[tt] = fmaf(w, low_s[tt * a.rank + r], la[tt]);
    }
#pragma unroll
    for (int tt = 0; tt < GL_RUN; ++tt) {
      la[tt] = tt < nt ? -softplus(-la[tt]) * a.inv_tau : -0.f;
      sum += la[tt];
    }
  }
  const bool marked = __syncthreads_or((on && sum < -GL_SPAN) || a.per_token) != 0;
  if (threadIdx.x == 0) a.marks[(size_t)t0 * a.H + h] = marked ? 1 : 0;
  float* out = a.act + (size_t)t0 * row;
  if (on) {
    float cum = -0.f;
#pragma unroll
    for (int tt = 0; tt < GL_RUN; ++tt)
      if (tt < nt) {
        cum += la[tt];
        float* o = out + (size_t)tt * row;
        o[ch] = marked ? q[tt] : q[tt] * expf(cum);
        o[n_k + ch] = marked ? k[tt] : k[tt] * expf(-cum);
        if (marked || tt == nt - 1) o[2 * n_k + ch] = decay_coef(marked ? la[tt] : cum);
      }
  }
  if (a.copy_v)
    for (int e = threadIdx.x; e < nt * a.dv; e += blockDim.x) {
      const int tt = e / a.dv, i = h * a.dv + e - tt * a.dv;
      out[(size_t)tt * row + 3 * n_k + i] = get(p + (size_t)tt * a.proj_row + a.col_v + i);
    }
}

struct GlaArgs {
  const float* act;
  const float* v;              // the first token's values, rows of v_row
  int v_row;
  const int* marks;
  const int *q_start, *seq_slot;
  float* state;                // [slots][H][dv][dk]
  float* out;                  // [tokens][H dv]
  int H, dk, dv;
};

// the decay of a lane's four rows on their column pairs: S <- keep S + coef S (+ kv)
__device__ __forceinline__ void decay_pairs(const float4& d, f2& c0, f2& c1, f2& k0, f2& k1) {
  c0 = pack_f2(d.x, d.y);
  c1 = pack_f2(d.z, d.w);
  k0 = pack_f2(decay_keep(d.x), decay_keep(d.y));
  k1 = pack_f2(decay_keep(d.z), decay_keep(d.w));
}

// K4: groups of four rows per lane (64 K4 >= dk); VEC: sizes and pointers allow 16-byte accesses
template <int K4, bool VEC, int CPL>
__global__ void __launch_bounds__(160, 1)
gla_scan_kernel(GlaArgs a) {
  pdl_launch_dependents();
  constexpr int COLS = 8 * CPL;
  constexpr int NP = 64 * K4;                            // rows, padded
  constexpr int PER_TOK = 3 * NP + COLS;              // q, k, decays, then this block's v columns
  extern __shared__ __align__(16) float gl_stage[];      // [SS_STAGES][SS_TOK][PER_TOK]
  __shared__ int mark_s[SS_STAGES][SS_TOK / SS_RUN];
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * COLS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int slot = a.seq_slot[b];
  const int t0 = a.q_start[b], t1 = a.q_start[b + 1];
  const int dk = a.dk, dv = a.dv, n_k = a.H * dk, inner = a.H * dv;
  // rows beyond dk and columns beyond dv: never copied over, zero for ever
  if (dk < NP || c0 + COLS > dv) {
    for (int i = threadIdx.x; i < SS_STAGES * SS_TOK * PER_TOK; i += blockDim.x) gl_stage[i] = 0.f;
    __syncthreads();
  }
  pdl_wait();
  const int n_groups = (t1 - t0 + SS_TOK - 1) / SS_TOK;
  if (warp == 4) {                                       // the warp that feeds the others
    const int row = 3 * n_k + inner;
    constexpr int W = VEC ? 4 : 1;
    const int per = (2 * dk + min(COLS, dv - c0)) / W, per_d = dk / W;
    auto load_mark = [&](int gi) {
      const int t = t0 + gi * SS_TOK + lane * SS_RUN;
      return lane < SS_TOK / SS_RUN && t < t1 ? a.marks[(size_t)t * a.H + h] : 0;
    };
    auto issue = [&](int gi, int mark) {
      const int m0 = __shfl_sync(0xffffffffu, mark, 0), m1 = __shfl_sync(0xffffffffu, mark, 1);
      if (gi < n_groups) {
        const int base = t0 + gi * SS_TOK;
        const int nt = min(SS_TOK, t1 - base);
        float* dst = gl_stage + (size_t)(gi % SS_STAGES) * SS_TOK * PER_TOK;
        if (lane < SS_TOK / SS_RUN) mark_s[gi % SS_STAGES][lane] = mark;
        for (int e = lane; e < per; e += 32) {
          const int f = e * W;
          const float* src = a.act + (size_t)base * row + h * dk;
          int pitch = row, d;
          if (f < dk) { src += f; d = f; }
          else if (f < 2 * dk) { src += n_k + (f - dk); d = NP + (f - dk); }
          else {
            src = a.v + (size_t)base * a.v_row + h * dv + c0 + (f - 2 * dk);
            pitch = a.v_row;
            d = 3 * NP + (f - 2 * dk);
          }
          ss_copy_tokens<4 * W>(dst + d, PER_TOK, src, pitch, nt);
        }
        // decays: of every token of a marked run, else of the run's last token
        for (int e = lane; e < per_d; e += 32) {
          const int f = e * W;
          const float* src = a.act + (size_t)base * row + 2 * n_k + h * dk + f;
          for (int r = 0; r < SS_TOK && r < nt; r += SS_RUN) {
            const int end = min(r + SS_RUN, nt);
            for (int tt = (r ? m1 : m0) ? r : end - 1; tt < end; ++tt)
              ss_copy<4 * W>(dst + tt * PER_TOK + 2 * NP + f, src + (size_t)tt * row);
          }
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int mark0 = load_mark(0), mark1 = load_mark(1);
    issue(0, mark0);
    issue(1, mark1);
    int mark = load_mark(2);
    for (int gi = 0; gi < n_groups; ++gi) {
      asm volatile("cp.async.wait_group %0;" ::"n"(SS_STAGES - 2) : "memory");
      __syncthreads();                                   // stage gi has landed; stage gi - 1 is no longer read
      issue(gi + 2, mark);
      mark = load_mark(gi + 3);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    return;
  }
  const int sub = lane & 15, lc = (warp * 2 + (lane >> 4)) * CPL;       // the lane's rows; its first column in the block
  f2 S[CPL][2 * K4];
  float* st = a.state + ((size_t)slot * a.H + h) * dv * dk;
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int col = c0 + lc + c;
    load_column<K4, VEC>(st + (size_t)col * dk, dk, sub, col < dv, S[c]);
  }
  for (int gi = 0; gi < n_groups; ++gi) {
    __syncthreads();
    const int base = t0 + gi * SS_TOK;
    const int nt = min(SS_TOK, t1 - base);
    const float* sg = gl_stage + (size_t)(gi % SS_STAGES) * SS_TOK * PER_TOK;
#pragma unroll 1
    for (int r = 0; r < SS_TOK / SS_RUN; ++r) {
      const int first = r * SS_RUN, here = min(SS_RUN, nt - first);
      if (here <= 0) break;
      float o[SS_RUN * CPL];
      RunToken<K4, CPL> buf[2];
      auto fetch = [&](int tt) {
        const float* p = sg + (first + tt) * PER_TOK;
        buf[tt & 1].fetch(p + 4 * sub, p + NP + 4 * sub, p + 3 * NP + lc);
      };
      auto token = [&](int tt) { buf[tt & 1].apply(S, o + CPL * tt); };     // the write and the read-out, without a decay
      auto decay = [&](int tt) {
        const float* p = sg + (first + tt) * PER_TOK + 2 * NP;
#pragma unroll
        for (int k = 0; k < K4; ++k) {
          f2 e0, e1, k0, k1;
          decay_pairs(*reinterpret_cast<const float4*>(p + 64 * k + 4 * sub), e0, e1, k0, k1);
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            S[c][2 * k] = fma_f2(e0, S[c][2 * k], mul_f2(k0, S[c][2 * k]));
            S[c][2 * k + 1] = fma_f2(e1, S[c][2 * k + 1], mul_f2(k1, S[c][2 * k + 1]));
          }
        }
      };
      if (mark_s[gi % SS_STAGES][r]) {
#pragma unroll
        for (int tt = 0; tt < SS_RUN; ++tt) {
          if (tt < here) {
            fetch(tt);
            decay(tt);
            token(tt);
          } else {
#pragma unroll
            for (int c = 0; c < CPL; ++c) o[CPL * tt + c] = 0.f;
          }
        }
      } else if (here == SS_RUN) {
#pragma unroll
        for (int tt = 0; tt < SS_RUN; ++tt) {
          if (tt == 0) fetch(0);
          if (tt + 1 < SS_RUN) fetch(tt + 1);
          token(tt);
        }
        decay(SS_RUN - 1);
      } else {
#pragma unroll
        for (int tt = 0; tt < SS_RUN; ++tt) {
          if (tt < here) {
            fetch(tt);
            token(tt);
          } else {
#pragma unroll
            for (int c = 0; c < CPL; ++c) o[CPL * tt + c] = 0.f;
          }
        }
        decay(here - 1);
      }
      run_sums<CPL>(o, lane);
      const int tt = first + (sub >> 1), col = c0 + lc + (sub & 1) * (CPL / 2);
      if (tt < nt && col < dv) {
        float* dst = a.out + (size_t)(base + tt) * inner + h * dv + col;
        if constexpr (VEC && CPL == 4) {
          *reinterpret_cast<float2*>(dst) = make_float2(o[0], o[1]);
        } else {
#pragma unroll
          for (int c = 0; c < CPL / 2; ++c)
            if (col + c < dv) dst[c] = o[c];
        }
      }
    }
  }
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int col = c0 + lc + c;
    if (col < dv) store_column<K4, VEC>(st + (size_t)col * dk, dk, sub, S[c]);
  }
}

constexpr int GS_COLS = 8;                               // columns per warp of gla_step

// One token per sequence, every token with decays of its own.  grid (column tiles of 8 GS_COLS, heads,
// sequences), eight warps
template <bool VEC>
__global__ void __launch_bounds__(256, 3)
gla_step_kernel(GlaArgs a) {
  pdl_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c0 = (blockIdx.x * 8 + warp) * GS_COLS;
  const int slot = a.seq_slot[b], t = a.q_start[b];
  const int dk = a.dk, dv = a.dv, n_k = a.H * dk, inner = a.H * dv;
  if (c0 >= dv) return;
  float* st = a.state + ((size_t)slot * a.H + h) * dv * dk;
  const float* row = a.act + (size_t)t * (3 * n_k + inner);
  pdl_wait();
  float x[GS_COLS], y[GS_COLS];
#pragma unroll
  for (int c = 0; c < GS_COLS; ++c) {
    x[c] = c0 + c < dv ? a.v[(size_t)t * a.v_row + h * dv + c0 + c] : 0.f;
    y[c] = 0.f;
  }
  constexpr int W = VEC ? 4 : 1;
  for (int i = lane * W; i < dk; i += 32 * W) {
    float Q[W], K[W], D[W], S[GS_COLS][W];
    const float* qp = row + h * dk + i;
    if constexpr (VEC) {
#pragma unroll
      for (int c = 0; c < GS_COLS; ++c) {
        const float4 v = c0 + c < dv ? *reinterpret_cast<const float4*>(st + (size_t)(c0 + c) * dk + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[c][0] = v.x; S[c][1] = v.y; S[c][2] = v.z; S[c][3] = v.w;
      }
      const float4 q4 = *reinterpret_cast<const float4*>(qp);
      const float4 k4 = *reinterpret_cast<const float4*>(qp + n_k);
      const float4 d4 = *reinterpret_cast<const float4*>(qp + 2 * n_k);
      Q[0] = q4.x; Q[1] = q4.y; Q[2] = q4.z; Q[3] = q4.w;
      K[0] = k4.x; K[1] = k4.y; K[2] = k4.z; K[3] = k4.w;
      D[0] = d4.x; D[1] = d4.y; D[2] = d4.z; D[3] = d4.w;
    } else {
#pragma unroll
      for (int c = 0; c < GS_COLS; ++c) S[c][0] = c0 + c < dv ? st[(size_t)(c0 + c) * dk + i] : 0.f;
      Q[0] = qp[0]; K[0] = qp[n_k]; D[0] = qp[2 * n_k];
    }
#pragma unroll
    for (int c = 0; c < GS_COLS; ++c) {
#pragma unroll
      for (int j = 0; j < W; ++j) {
        S[c][j] = fmaf(decay_keep(D[j]), S[c][j], fmaf(D[j], S[c][j], K[j] * x[c]));
        y[c] = fmaf(S[c][j], Q[j], y[c]);
      }
      if (c0 + c < dv) {
        if constexpr (VEC) *reinterpret_cast<float4*>(st + (size_t)(c0 + c) * dk + i) = make_float4(S[c][0], S[c][1], S[c][2], S[c][3]);
        else st[(size_t)(c0 + c) * dk + i] = S[c][0];
      }
    }
  }
  // eight sums over 32 lanes: three rounds leave one value per lane, two more add up the quarters
#pragma unroll
  for (int half = 4; half >= 1; half >>= 1) {
    const bool upper = (lane & half) != 0;
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float send = upper ? y[i] : y[i + half];
      const float keep = upper ? y[i + half] : y[i];
      y[i] = keep + __shfl_xor_sync(0xffffffffu, send, half);
    }
  }
  y[0] += __shfl_xor_sync(0xffffffffu, y[0], 8);
  y[0] += __shfl_xor_sync(0xffffffffu, y[0], 16);
  if (lane < GS_COLS && c0 + lane < dv) a.out[(size_t)t * inner + h * dv + c0 + lane] = y[0];
}

}  // namespace yalm

using namespace yalm;

// proj: float32 slices [n_partials][tokens][proj_row] with q (H dk columns) at col_q, k at col_k, v (H dv) at
// col_v and the low-rank values at col_low; w2 [rank][H dk], bias [H dk]; act: float32 scratch [tokens][3 H dk +
// H dv]; marks: int32 scratch [tokens][H]; state float32 [slots][H][dv][dk], read at the step's start and written
// at its end; out float32 [tokens][H dv].  dk up to 256, rank up to 1,024.
extern "C" int yalm_gla(const float* proj, int n_partials, long long partial_stride, int proj_row, int col_q,
                        int col_k, int col_v, int col_low, int rank, const float* w2, const float* bias, float inv_tau,
                        float q_scale, float* act, int* marks, const int* q_start, const int* seq_slot, float* state,
                        float* out, int n_tokens, int n_seqs, int H, int dk, int dv, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (H <= 0 || dk <= 0 || dk > 256 || dv <= 0 || rank <= 0 || rank > 1024 || !(inv_tau > 0.f)) return -2;
  if (n_seqs > 65535 || H > 65535) return -4;
  const bool step = n_tokens == n_seqs;                  // every sequence brings one token
  const int row = 3 * H * dk + H * dv;
  const bool one = n_partials == 1;
  const GlaPrep p = {proj, n_partials, proj_row, col_q, col_k, col_v, col_low, rank, partial_stride, w2, bias, act,
                     marks, q_start, n_seqs, H, dk, dv, step ? 1 : 0, one ? 0 : 1, inv_tau, q_scale};
  const dim3 pgrid(step ? n_tokens : n_tokens / GL_RUN + n_seqs, H), pblock((dk + 31) / 32 * 32);
  const size_t psmem = (size_t)GL_RUN * rank * sizeof(float);
  if (one) launch_pdl(gla_prep_kernel<true>, pgrid, pblock, psmem, stream, p);
  else launch_pdl(gla_prep_kernel<false>, pgrid, pblock, psmem, stream, p);
  YALM_LAUNCH_CHECK();
  const GlaArgs a = {act, one ? proj + col_v : act + 3 * H * dk, one ? proj_row : row, marks, q_start, seq_slot, state, out,
                     H, dk, dv};
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && a.v_row % 4 == 0 &&
                   ((((uintptr_t)act) | ((uintptr_t)a.v) | ((uintptr_t)state) | ((uintptr_t)out)) & 15) == 0;
  if (step) {
    const dim3 grid((dv + 8 * GS_COLS - 1) / (8 * GS_COLS), H, n_seqs), block(256);
    if (vec) launch_pdl(gla_step_kernel<true>, grid, block, 0, stream, a);
    else launch_pdl(gla_step_kernel<false>, grid, block, 0, stream, a);
    YALM_LAUNCH_CHECK();
    return 0;
  }
  const bool narrow = narrow_blocks((long long)((dv + 31) / 32) * H * n_seqs);
  const int cols = narrow ? 16 : 32;
  const dim3 grid((dv + cols - 1) / cols, H, n_seqs), block(160);
#define YALM_GLA1(K, V, C)                                                                                    \
  do {                                                                                                        \
    const size_t smem = (size_t)SS_STAGES * SS_TOK * (3 * 64 * K + 8 * C) * sizeof(float);                    \
    static bool set = false;                                                                                  \
    if (!set) {                                                                                               \
      cudaError_t e = cudaFuncSetAttribute(gla_scan_kernel<K, V, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           (int)smem);                                                        \
      if (e != cudaSuccess) return (int)e;                                                                    \
      set = true;                                                                                             \
    }                                                                                                         \
    launch_pdl(gla_scan_kernel<K, V, C>, grid, block, smem, stream, a);                                       \
  } while (0)
#define YALM_GLA(K)                              \
  do {                                           \
    if (vec && narrow) YALM_GLA1(K, true, 2);    \
    else if (vec) YALM_GLA1(K, true, 4);         \
    else if (narrow) YALM_GLA1(K, false, 2);     \
    else YALM_GLA1(K, false, 4);                 \
  } while (0)
  if (dk <= 64) YALM_GLA(1);
  else if (dk <= 128) YALM_GLA(2);
  else YALM_GLA(4);
#undef YALM_GLA
#undef YALM_GLA1
  YALM_LAUNCH_CHECK();
  return 0;
}
