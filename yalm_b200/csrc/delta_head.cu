// The gated delta rule with ONE decay per head, per head with key size dk and value size dv:
//   S <- e^(a_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t,   a_t <= 0
// (delta_rule.cu has the form with a decay per key channel).  32-bit throughout, the state carried from step to
// step as [slots][H][dv][dk]: a column's rows are neighbours.
//
// Tokens go in groups of 16.  With A_t = e^(a_first + .. + a_t) over a group and T = S / A the decay leaves the
// elements, and the group's writes w_t (T <- T + k_t w_t^T) solve a triangular system whose matrix does not depend
// on the state:
//   w_t = beta_t (v_t / A_t - T_0^T k_t - sum_(s<t) (k_s.k_t) w_s),   o_t = A_t (T_0^T q_t + sum_(s<=t) (k_s.q_t) w_s)
//   (I + L) w = beta r,  L_ts = beta_t (k_s.k_t) for s < t,  r_t = v_t / A_t - T_0^T k_t;   w = M r,  M = (I + L)^-1 beta
// (the delta rule in this form: Yang et al., "Parallelizing Linear Transformers with the Delta Rule over Sequence
// Length").  A group's reductions over the key channels are then made together, none waits for another's write.
//
//  * delta_head_prep: a block takes one group of one q/k head: q and k of every token become unit vectors
//    (x / sqrt(sum x^2 + 1e-6)), q times 1/sqrt(dk); beta = sigmoid(.) and a = -exp(A_h) softplus(. + dt_h) for the
//    heads that read it; and, for whole groups, the products k_s.q_t and every head's M.
//  * delta_head_scan: a block owns 16 value columns of one (sequence, head), eight lanes own a column, a lane
//    RPL of its rows in packed pairs; tokens come through a three-stage cp.async ring of 16.  Three multiply-adds
//    per element and token.  A group that forgets more than e^(-DH_SPAN), and a sequence's last tokens, take the
//    recurrence as it stands, one all-reduce over the eight lanes per token.
//  * delta_head_step: one token per sequence, the state streamed once: a warp per DS_COLS columns.
//
// A token's row, float32: [q: G dk | k: G dk | v: H dv | beta: H padded to 4 | a: H padded to 4 | k_s.q_t: 16 G |
// M's row: 16 H].
#include "api.h"
#include "scan.cuh"

namespace yalm {

constexpr int DH_TOK = SS_TOK, DH_STAGES = 3, DH_WARPS = 4, DH_COLS = 4 * DH_WARPS;
constexpr float DH_SPAN = 30.f;

struct DeltaHeadPrep {
  float* act;
  const float* proj;           // slices [n_partials][tokens][proj_row]: beta's logits at col_b, the decays' at col_a
  int n_partials, proj_row, col_b, col_a;
  long long partial_stride;
  const float *dt_bias, *a_log;        // [H]
  const int* q_start;
  int n_seqs, row, H, G, dk, dv;
};

__device__ __forceinline__ int dh_tail(int H, int G, int dk, int dv) { return 2 * G * dk + H * dv + 2 * ((H + 3) & ~3); }

constexpr int DP_THREADS = 128;

// grid (groups of 16 tokens, q/k heads)
__global__ void __launch_bounds__(DP_THREADS) delta_head_prep_kernel(DeltaHeadPrep a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float dp_s[];         // q, k [16][pitch]; then betas [16][R], k.k [16][17]
  int b, first;
  if (!find_run<DH_TOK>(a.q_start, a.n_seqs, blockIdx.x, b, first)) return;
  const int g = blockIdx.y, R = a.H / a.G, qs = a.q_start[b];
  const int nt = min(DH_TOK, a.q_start[b + 1] - qs - first), t0 = qs + first;
  const int pitch = ((a.dk + 3) & ~3) + 4, dkp = (a.dk + 3) & ~3;
  float *q_s = dp_s, *k_s = q_s + DH_TOK * pitch, *beta_s = k_s + DH_TOK * pitch, *kk_s = beta_s + DH_TOK * R;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int beta0 = 2 * a.G * a.dk + a.H * a.dv, hp = (a.H + 3) & ~3, tail = dh_tail(a.H, a.G, a.dk, a.dv);
  pdl_wait();
  // 2 x 16 vectors over four warps, four of a warp's at a time so that their loads are in flight together: unit
  // vectors, in memory and here
  constexpr int NW = DP_THREADS / 32, AT_ONCE = 4;
  for (int i0 = warp; i0 < 2 * nt; i0 += NW * AT_ONCE) {
    float x[AT_ONCE][8], ss[AT_ONCE];                   // dk up to 256
#pragma unroll
    for (int u = 0; u < AT_ONCE; ++u) {
      const int i = i0 + u * NW, tt = i >> 1, is_k = i & 1;
      const float* v = a.act + (size_t)(t0 + tt) * a.row + (is_k * a.G + g) * a.dk;
#pragma unroll
      for (int j = 0; j < 8; ++j) x[u][j] = i < 2 * nt && lane + 32 * j < a.dk ? v[lane + 32 * j] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < AT_ONCE; ++u) {
      ss[u] = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) ss[u] += x[u][j] * x[u][j];
      ss[u] = warp_sum(ss[u]);
    }
#pragma unroll
    for (int u = 0; u < AT_ONCE; ++u) {
      const int i = i0 + u * NW, tt = i >> 1, is_k = i & 1;
      if (i >= 2 * nt) continue;
      float* v = a.act + (size_t)(t0 + tt) * a.row + (is_k * a.G + g) * a.dk;
      float* d = (is_k ? k_s : q_s) + tt * pitch;
      const float r = (1.0f / sqrtf(ss[u] + 1e-6f)) * (is_k ? 1.0f : 1.0f / sqrtf((float)a.dk));
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int c = lane + 32 * j;
        if (c < a.dk) v[c] = x[u][j] * r;
        if (c < dkp) d[c] = x[u][j] * r;                // zero beyond dk
      }
    }
  }
  for (int i = threadIdx.x; i < nt * R; i += DP_THREADS) {
    const int tt = i / R, r = i - tt * R, h = g * R + r;
    const float* p = a.proj + (size_t)(t0 + tt) * a.proj_row + h;
    float* o = a.act + (size_t)(t0 + tt) * a.row + beta0 + h;
    const float beta = 1.0f / (1.0f + expf(-sum_slices(p + a.col_b, a.n_partials, a.partial_stride)));
    const float z = sum_slices(p + a.col_a, a.n_partials, a.partial_stride) + a.dt_bias[h];
    beta_s[tt * R + r] = beta;
    o[0] = beta;
    o[hp] = -expf(a.a_log[h]) * softplus(z);
  }
  if (nt < DH_TOK) return;                              // these tokens take the recurrence as it stands
  __syncthreads();
  {                                                     // token t = thread / 8 against s = 2 (thread % 8) and the next
    const int t = threadIdx.x >> 3, s0 = (threadIdx.x & 7) * 2;
    float kq[2] = {0.f, 0.f}, kk[2] = {0.f, 0.f};
    for (int c = 0; c < dkp; c += 4) {
      const float4 qt = *reinterpret_cast<const float4*>(q_s + t * pitch + c);
      const float4 kt = *reinterpret_cast<const float4*>(k_s + t * pitch + c);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const float4 ks = *reinterpret_cast<const float4*>(k_s + (s0 + j) * pitch + c);
        kq[j] = fmaf(ks.x, qt.x, fmaf(ks.y, qt.y, fmaf(ks.z, qt.z, fmaf(ks.w, qt.w, kq[j]))));
        kk[j] = fmaf(ks.x, kt.x, fmaf(ks.y, kt.y, fmaf(ks.z, kt.z, fmaf(ks.w, kt.w, kk[j]))));
      }
    }
    float* o = a.act + (size_t)(t0 + t) * a.row + tail + g * DH_TOK + s0;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      o[j] = s0 + j <= t ? kq[j] : 0.f;
      kk_s[t * 17 + s0 + j] = kk[j];
    }
  }
  __syncthreads();
  // a thread per (head, column s) of M
  for (int i = threadIdx.x; i < R * DH_TOK; i += DP_THREADS) {
    const int r = i / DH_TOK, s = i - r * DH_TOK;
    float m[DH_TOK];
    float* o = a.act + (size_t)t0 * a.row + tail + (a.G + g * R + r) * DH_TOK + s;
    const float bs = beta_s[s * R + r];
#pragma unroll
    for (int t = 0; t < DH_TOK; ++t) {
      float sum = 0.f;
#pragma unroll
      for (int u = 0; u < t; ++u) sum = fmaf(kk_s[t * 17 + u], m[u], sum);      // m[u] is 0 above the diagonal
      m[t] = t < s ? 0.f : t == s ? 1.f : -beta_s[t * R + r] * sum;
      o[(size_t)t * a.row] = m[t] * bs;
    }
  }
}

struct DeltaHead {
  const float* act;
  const int *q_start, *seq_slot;
  float* state;                // [slots][H][dv][dk]
  float* out;                  // [tokens][H dv]
  int row, H, G, dk, dv;
};

// The eight lanes' partial sums of a column's 16 values: in every round a lane hands half of its values to its
// partner and adds the partner's other half to its own; lane `sub` is left with the whole sums number 2 sub and
// 2 sub + 1 in v[0] and v[1]
__device__ __forceinline__ void column_sums(float* v, int sub) {
  static_assert(DH_TOK == 16, "two values per lane");
#pragma unroll
  for (int half = 4, n = 8; half >= 1; half >>= 1, n >>= 1) {
    const bool upper = (sub & half) != 0;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float send = upper ? v[i] : v[i + n];
      const float keep = upper ? v[i + n] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, half);
    }
  }
}
// a row of 16 numbers in shared memory times 16 in registers
__device__ __forceinline__ float row_times(const float* row, const float* x) {
  float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < DH_TOK; i += 4) {
    const float4 m = *reinterpret_cast<const float4*>(row + i);
    s[0] = fmaf(m.x, x[i], s[0]); s[1] = fmaf(m.y, x[i + 1], s[1]);
    s[2] = fmaf(m.z, x[i + 2], s[2]); s[3] = fmaf(m.w, x[i + 3], s[3]);
  }
  return (s[0] + s[1]) + (s[2] + s[3]);
}

template <int RPL, int VEC>
__global__ void __launch_bounds__(32 * DH_WARPS, 1) delta_head_scan_kernel(DeltaHead a) {
  pdl_launch_dependents();
  constexpr int DKP = 8 * RPL;                          // rows, padded
  // q, k, this block's v columns, beta, a (+ padding), k_s.q_t, M's row
  constexpr int OFF_S = 2 * DKP + DH_COLS, OFF_G = OFF_S + 4, PER_TOK = OFF_G + 2 * DH_TOK;
  constexpr int NT = 32 * DH_WARPS, NF = RPL / 2;
  extern __shared__ __align__(16) float dh_stage[];     // [DH_STAGES][DH_TOK][PER_TOK]
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * DH_COLS;
  const int dk = a.dk, dv = a.dv, H = a.H, G = a.G, row = a.row;
  const int hq = h / (H / G);
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
  const int sub = lane & 7, lc = w * 4 + (lane >> 3), col = c0 + lc;
  const int slot = a.seq_slot[b];
  const int t0 = a.q_start[b], t1 = a.q_start[b + 1];
  if (dk < DKP || c0 + DH_COLS > dv) {                  // rows beyond dk, columns beyond dv: zero for ever
    for (int i = threadIdx.x; i < DH_STAGES * DH_TOK * PER_TOK; i += NT) dh_stage[i] = 0.f;
    __syncthreads();
  }
  const int n_v = min(DH_COLS, dv - c0), per = (2 * dk + n_v + 2 * DH_TOK) / VEC;
  const int tail = dh_tail(H, G, dk, dv);
  const int beta_off = 2 * G * dk + H * dv + h, hp = (H + 3) & ~3;
  pdl_wait();
  // register pair 2 j + e holds rows 4 (sub + 8 j) + 2 e and the next
  f2 S[NF];
  float* st = a.state + ((size_t)slot * H + h) * dv * dk + (size_t)col * dk;
#pragma unroll
  for (int j = 0; j < RPL / 4; ++j) {
    const int i = 4 * (sub + 8 * j);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col < dv) {
      if constexpr (VEC == 4) {
        if (i < dk) v = *reinterpret_cast<const float4*>(st + i);
      } else {
        if (i < dk) v.x = st[i];
        if (i + 1 < dk) v.y = st[i + 1];
        if (i + 2 < dk) v.z = st[i + 2];
        if (i + 3 < dk) v.w = st[i + 3];
      }
    }
    S[2 * j] = pack_f2(v.x, v.y);
    S[2 * j + 1] = pack_f2(v.z, v.w);
  }
  const int n_groups = (t1 - t0 + DH_TOK - 1) / DH_TOK;
  auto issue = [&](int g) {
    if (g < n_groups) {
      const int base = t0 + g * DH_TOK;
      const int nt = min(DH_TOK, t1 - base);
      float* dst = dh_stage + (size_t)(g % DH_STAGES) * DH_TOK * PER_TOK;
      const float* src = a.act + (size_t)base * row;
      for (int e = threadIdx.x; e < per; e += NT) {
        const int f = e * VEC;
        int so, d;
        if (f < dk) { so = hq * dk + f; d = f; }
        else if (f < 2 * dk) { so = G * dk + hq * dk + (f - dk); d = DKP + (f - dk); }
        else if (f < 2 * dk + n_v) { so = 2 * G * dk + h * dv + c0 + (f - 2 * dk); d = 2 * DKP + (f - 2 * dk); }
        else {
          const int e2 = f - 2 * dk - n_v;
          so = tail + (e2 < DH_TOK ? hq * DH_TOK + e2 : (G + h) * DH_TOK + (e2 - DH_TOK));
          d = OFF_G + e2;
        }
        ss_copy_tokens<4 * VEC>(dst + d, PER_TOK, src + so, row, nt);
      }
      if (threadIdx.x < nt) ss_copy<4>(dst + threadIdx.x * PER_TOK + OFF_S, src + (size_t)threadIdx.x * row + beta_off);
      else if (threadIdx.x >= 32 && threadIdx.x < 32 + nt)
        ss_copy<4>(dst + (threadIdx.x - 32) * PER_TOK + OFF_S + 1, src + (size_t)(threadIdx.x - 32) * row + beta_off + hp);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(0);
  issue(1);
  for (int g = 0; g < n_groups; ++g) {
    asm volatile("cp.async.wait_group %0;" ::"n"(DH_STAGES - 2) : "memory");
    __syncthreads();                                    // stage g has landed; stage g - 1 is no longer read
    issue(g + 2);
    const int base = t0 + g * DH_TOK;
    const int nt = min(DH_TOK, t1 - base);
    const float* sg = dh_stage + (size_t)(g % DH_STAGES) * DH_TOK * PER_TOK;
    // lane tt and lane 16 + tt of every warp: token tt's a and the sum up to it
    const int mine = lane & (DH_TOK - 1);
    const float la = mine < nt ? sg[mine * PER_TOK + OFF_S + 1] : -0.f;
    float cum = la;
#pragma unroll
    for (int o = 1; o < DH_TOK; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, cum, o, DH_TOK);
      if (mine >= o) cum += v;
    }
    const float total = __shfl_sync(0xffffffffu, cum, DH_TOK - 1);
    const bool whole = total >= -DH_SPAN;
    // whole groups: A and 1 / A; others: the token's own decay as decay_coef gives it
    const float f_a = whole ? expf(cum) : decay_coef(la), f_inv = expf(whole ? -cum : 0.f);
    float o[DH_TOK];
    auto token = [&](int tt, bool scaled) {
      const float* qq = sg + tt * PER_TOK + 4 * sub;
      f2 qr[NF], kr[NF];
#pragma unroll
      for (int j = 0; j < RPL / 4; ++j) {               // the eight lanes of a column read 128 neighbouring bytes
        const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(qq + 32 * j);
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(qq + DKP + 32 * j);
        qr[2 * j] = q2.x; qr[2 * j + 1] = q2.y;
        kr[2 * j] = k2.x; kr[2 * j + 1] = k2.y;
      }
      const float beta = sg[tt * PER_TOK + OFF_S];
      float vj = sg[tt * PER_TOK + 2 * DKP + lc];
      const float fa = __shfl_sync(0xffffffffu, f_a, tt);
      if (scaled) {
        vj *= __shfl_sync(0xffffffffu, f_inv, tt);
      } else {
        const float keep = decay_keep(fa);
        const f2 e = pack_f2(fa, fa), kp = pack_f2(keep, keep);
#pragma unroll
        for (int r = 0; r < NF; ++r) S[r] = fma_f2(e, S[r], mul_f2(kp, S[r]));
      }
      f2 k0 = mul_f2(kr[0], S[0]), k1 = mul_f2(kr[1], S[1]);
#pragma unroll
      for (int r = 2; r < NF; r += 2) {
        k0 = fma_f2(kr[r], S[r], k0);
        k1 = fma_f2(kr[r + 1], S[r + 1], k1);
      }
      float x0, x1, x2, x3;
      unpack_f2(k0, x0, x1);
      unpack_f2(k1, x2, x3);
      float kdot = (x0 + x1) + (x2 + x3);
      kdot += __shfl_xor_sync(0xffffffffu, kdot, 4);
      kdot += __shfl_xor_sync(0xffffffffu, kdot, 2);
      kdot += __shfl_xor_sync(0xffffffffu, kdot, 1);
      const float u = beta * (vj - kdot);
      const f2 uu = pack_f2(u, u);
#pragma unroll
      for (int r = 0; r < NF; ++r) S[r] = fma_f2(kr[r], uu, S[r]);
      f2 o0 = mul_f2(qr[0], S[0]), o1 = mul_f2(qr[1], S[1]);
#pragma unroll
      for (int r = 2; r < NF; r += 2) {
        o0 = fma_f2(qr[r], S[r], o0);
        o1 = fma_f2(qr[r + 1], S[r + 1], o1);
      }
      unpack_f2(o0, x0, x1);
      unpack_f2(o1, x2, x3);
      o[tt] = (x0 + x1) + (x2 + x3);
      if (scaled) o[tt] *= fa;
    };
    if (nt == DH_TOK && whole) {                        // the usual group
      // T_0^T k_t and T_0^T q_t for all of its tokens, rows fetched one token ahead of their use
      float kd[DH_TOK];
      constexpr int NB = RPL <= 16 ? 2 : 1;
      ulonglong2 qb[NB][RPL / 4], kb[NB][RPL / 4];
      auto fetch = [&](int tt, bool q) {
        const float* p = sg + tt * PER_TOK + 4 * sub;
#pragma unroll
        for (int j = 0; j < RPL / 4; ++j) {
          kb[tt % NB][j] = *reinterpret_cast<const ulonglong2*>(p + DKP + 32 * j);
          if (q) qb[tt % NB][j] = *reinterpret_cast<const ulonglong2*>(p + 32 * j);
        }
      };
      if (NB == 2) fetch(0, true);
#pragma unroll
      for (int tt = 0; tt < DH_TOK; ++tt) {
        if (NB == 1) fetch(tt, true);
        else if (tt + 1 < DH_TOK) fetch(tt + 1, true);
        const ulonglong2 *q2 = qb[tt % NB], *k2 = kb[tt % NB];
        f2 k0 = mul_f2(k2[0].x, S[0]), k1 = mul_f2(k2[0].y, S[1]), q0 = mul_f2(q2[0].x, S[0]), q1 = mul_f2(q2[0].y, S[1]);
#pragma unroll
        for (int j = 1; j < RPL / 4; ++j) {
          k0 = fma_f2(k2[j].x, S[2 * j], k0); k1 = fma_f2(k2[j].y, S[2 * j + 1], k1);
          q0 = fma_f2(q2[j].x, S[2 * j], q0); q1 = fma_f2(q2[j].y, S[2 * j + 1], q1);
        }
        kd[tt] = sum_f2(k0, k1);
        o[tt] = sum_f2(q0, q1);
      }
      // over the eight lanes; lane `sub` keeps those of tokens 2 sub and 2 sub + 1
      column_sums(kd, sub);
      column_sums(o, sub);
      const float* mine_s = sg + (2 * sub) * PER_TOK;
      float w[2], rr[DH_TOK];
#pragma unroll
      for (int i = 0; i < 2; ++i)
        w[i] = fmaf(mine_s[i * PER_TOK + 2 * DKP + lc], __shfl_sync(0xffffffffu, f_inv, 2 * sub + i), -kd[i]);
#pragma unroll
      for (int tt = 0; tt < DH_TOK; ++tt) rr[tt] = __shfl_sync(0xffffffffu, w[tt & 1], (lane & 24) | (tt >> 1));
#pragma unroll
      for (int i = 0; i < 2; ++i) w[i] = row_times(mine_s + i * PER_TOK + OFF_G + DH_TOK, rr);
#pragma unroll
      for (int tt = 0; tt < DH_TOK; ++tt) rr[tt] = __shfl_sync(0xffffffffu, w[tt & 1], (lane & 24) | (tt >> 1));
      // the outputs of this lane's two tokens, then the writes
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float A = __shfl_sync(0xffffffffu, f_a, 2 * sub + i);
        const float y = A * (o[i] + row_times(mine_s + i * PER_TOK + OFF_G, rr));
        if (col < dv) a.out[((size_t)(base + 2 * sub + i) * H + h) * dv + col] = y;
      }
      __syncwarp();                                     // the keys are loaded again, not kept in registers
      if (NB == 2) fetch(0, false);
#pragma unroll
      for (int tt = 0; tt < DH_TOK; ++tt) {
        if (NB == 1) fetch(tt, false);
        else if (tt + 1 < DH_TOK) fetch(tt + 1, false);
        const f2 ww = pack_f2(rr[tt], rr[tt]);
#pragma unroll
        for (int j = 0; j < RPL / 4; ++j) {
          S[2 * j] = fma_f2(kb[tt % NB][j].x, ww, S[2 * j]);
          S[2 * j + 1] = fma_f2(kb[tt % NB][j].y, ww, S[2 * j + 1]);
        }
      }
    } else if (whole) {
#pragma unroll
      for (int tt = 0; tt < DH_TOK; ++tt) {
        o[tt] = 0.f;
        if (tt < nt) token(tt, true);
      }
    } else {
#pragma unroll
      for (int tt = 0; tt < DH_TOK; ++tt) {
        o[tt] = 0.f;
        if (tt < nt) token(tt, false);
      }
    }
    if (whole) {
      const float c = decay_coef(total), keep = decay_keep(c);
      const f2 e = pack_f2(c, c), kp = pack_f2(keep, keep);
#pragma unroll
      for (int r = 0; r < NF; ++r) S[r] = fma_f2(e, S[r], mul_f2(kp, S[r]));
    }
    if (nt == DH_TOK && whole) continue;
    column_sums(o, sub);
    if (col < dv) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int tt = 2 * sub + i;
        if (tt < nt) a.out[((size_t)(base + tt) * H + h) * dv + col] = o[i];
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (col < dv) {
#pragma unroll
    for (int j = 0; j < RPL / 4; ++j) {
      const int i = 4 * (sub + 8 * j);
      float4 v;
      unpack_f2(S[2 * j], v.x, v.y);
      unpack_f2(S[2 * j + 1], v.z, v.w);
      if constexpr (VEC == 4) {
        if (i < dk) *reinterpret_cast<float4*>(st + i) = v;
      } else {
        if (i < dk) st[i] = v.x;
        if (i + 1 < dk) st[i + 1] = v.y;
        if (i + 2 < dk) st[i + 2] = v.z;
        if (i + 3 < dk) st[i + 3] = v.w;
      }
    }
  }
}

constexpr int DS_COLS = 4;                               // columns per warp of delta_head_step

// One token per sequence.  grid (column tiles of 8 DS_COLS, heads, sequences), eight warps; a lane holds C
// groups of W rows of each of the warp's columns (32 C W >= dk)
template <int C, int W>
__global__ void __launch_bounds__(256) delta_head_step_kernel(DeltaHead a) {
  pdl_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c0 = (blockIdx.x * 8 + warp) * DS_COLS;
  const int dk = a.dk, dv = a.dv, H = a.H, G = a.G;
  const int slot = a.seq_slot[b], t = a.q_start[b];
  if (c0 >= dv) return;
  float* st = a.state + ((size_t)slot * H + h) * dv * dk;
  const float* row = a.act + (size_t)t * a.row;
  const int hq = h / (H / G), beta_off = 2 * G * dk + H * dv + h, hp = (H + 3) & ~3;
  pdl_wait();
  float S[DS_COLS][C][W], k[C][W], kd[DS_COLS];
#pragma unroll
  for (int g = 0; g < C; ++g) {
    const int i = (g * 32 + lane) * W;
#pragma unroll
    for (int c = 0; c < DS_COLS; ++c) {
      const bool on = i < dk && c0 + c < dv;
      const float* p = st + (size_t)(c0 + c) * dk + i;
      if constexpr (W == 4) {
        const float4 v = on ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[c][g][0] = v.x; S[c][g][1] = v.y; S[c][g][2] = v.z; S[c][g][3] = v.w;
      } else {
        S[c][g][0] = on ? p[0] : 0.f;
      }
    }
    const float* kp = row + (G + hq) * dk + i;
#pragma unroll
    for (int j = 0; j < W; ++j) k[g][j] = i < dk ? kp[j] : 0.f;
  }
  const float beta = row[beta_off], coef = decay_coef(row[beta_off + hp]), keep = decay_keep(coef);
#pragma unroll
  for (int c = 0; c < DS_COLS; ++c) {
    kd[c] = 0.f;
#pragma unroll
    for (int g = 0; g < C; ++g)
#pragma unroll
      for (int j = 0; j < W; ++j) {
        S[c][g][j] = fmaf(coef, S[c][g][j], keep * S[c][g][j]);
        kd[c] = fmaf(k[g][j], S[c][g][j], kd[c]);
      }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int c = 0; c < DS_COLS; ++c) kd[c] += __shfl_xor_sync(0xffffffffu, kd[c], o);
  float y[DS_COLS];
#pragma unroll
  for (int c = 0; c < DS_COLS; ++c) {
    const float v = c0 + c < dv ? row[2 * G * dk + h * dv + c0 + c] : 0.f;
    kd[c] = beta * (v - kd[c]);
    y[c] = 0.f;
  }
#pragma unroll
  for (int g = 0; g < C; ++g) {
    const int i = (g * 32 + lane) * W;
    const float* qp = row + hq * dk + i;
    float q[W];
#pragma unroll
    for (int j = 0; j < W; ++j) q[j] = i < dk ? qp[j] : 0.f;
#pragma unroll
    for (int c = 0; c < DS_COLS; ++c) {
#pragma unroll
      for (int j = 0; j < W; ++j) {
        S[c][g][j] = fmaf(k[g][j], kd[c], S[c][g][j]);
        y[c] = fmaf(q[j], S[c][g][j], y[c]);
      }
      if (i < dk && c0 + c < dv) {
        float* p = st + (size_t)(c0 + c) * dk + i;
        if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(S[c][g][0], S[c][g][1], S[c][g][2], S[c][g][3]);
        else p[0] = S[c][g][0];
      }
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int c = 0; c < DS_COLS; ++c) y[c] += __shfl_xor_sync(0xffffffffu, y[c], o);
#pragma unroll
  for (int c = 0; c < DS_COLS; ++c)
    if (lane == c && c0 + c < dv) a.out[((size_t)t * H + h) * dv + c0 + c] = y[c];
}

}  // namespace yalm

using namespace yalm;

// The length of a token's row (see the head of this file)
extern "C" int yalm_delta_head_row(int H, int G, int dk, int dv) {
  return 2 * G * dk + H * dv + 2 * ((H + 3) & ~3) + DH_TOK * (G + H);
}

// act float32 [tokens][yalm_delta_head_row], whose first 2 G dk + H dv columns hold q | k | v after their convolution
// and activation; proj: float32 slices [n_partials][tokens][proj_row] with the H beta logits at col_b and the H decay
// logits at col_a; dt_bias, a_log [H].  dk up to 256.
extern "C" int yalm_delta_head_prep(float* act, const float* proj, int n_partials, long long partial_stride, int proj_row,
                                    int col_b, int col_a, const float* dt_bias, const float* a_log, const int* q_start,
                                    int n_tokens, int n_seqs, int H, int G, int dk, int dv, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || dk > 256) return -2;
  if (G > 65535) return -4;
  const DeltaHeadPrep a = {act, proj, n_partials, proj_row, col_b, col_a, partial_stride, dt_bias, a_log, q_start, n_seqs,
                           yalm_delta_head_row(H, G, dk, dv), H, G, dk, dv};
  const size_t smem = ((size_t)DH_TOK * 2 * (((dk + 3) & ~3) + 4) + (size_t)DH_TOK * (H / G) + DH_TOK * 17) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  static size_t attr = 48 * 1024;
  if (smem > attr) {
    cudaError_t e = cudaFuncSetAttribute(delta_head_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    attr = smem;
  }
  const int runs = n_tokens == n_seqs ? n_tokens : n_tokens / DH_TOK + n_seqs;
  launch_pdl(delta_head_prep_kernel, dim3(runs, G), dim3(DP_THREADS), smem, stream, a);
  YALM_LAUNCH_CHECK();
  return 0;
}

// act as delta_head_prep leaves it; state float32 [slots][H][dv][dk], read at the step's start and
// written at its end; out float32 [tokens][H dv].  dk up to 256.
extern "C" int yalm_delta_head_scan(const float* act, const int* q_start, const int* seq_slot, float* state, float* out,
                                    int n_tokens, int n_seqs, int H, int G, int dk, int dv, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || dk > 256) return -2;
  if (n_seqs > 65535 || H > 65535) return -4;
  const DeltaHead a = {act, q_start, seq_slot, state, out, yalm_delta_head_row(H, G, dk, dv), H, G, dk, dv};
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && ((((uintptr_t)act) | ((uintptr_t)state)) & 15) == 0;
  if (n_tokens == n_seqs) {                              // every sequence brings one token
    const dim3 grid((dv + 8 * DS_COLS - 1) / (8 * DS_COLS), H, n_seqs), block(256);
    if (vec && dk <= 128) launch_pdl(delta_head_step_kernel<1, 4>, grid, block, 0, stream, a);
    else if (vec) launch_pdl(delta_head_step_kernel<2, 4>, grid, block, 0, stream, a);
    else if (dk <= 64) launch_pdl(delta_head_step_kernel<2, 1>, grid, block, 0, stream, a);
    else launch_pdl(delta_head_step_kernel<8, 1>, grid, block, 0, stream, a);
    YALM_LAUNCH_CHECK();
    return 0;
  }
  const dim3 grid((dv + DH_COLS - 1) / DH_COLS, H, n_seqs), block(32 * DH_WARPS);
#define YALM_DH1(R, V)                                                                                             \
  do {                                                                                                             \
    const size_t smem = (size_t)DH_STAGES * DH_TOK * (2 * 8 * R + DH_COLS + 4 + 2 * DH_TOK) * sizeof(float);                    \
    static bool set = false;                                                                                       \
    if (!set && smem > 48 * 1024) {                                                                                \
      cudaError_t e = cudaFuncSetAttribute(delta_head_scan_kernel<R, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           (int)smem);                                                             \
      if (e != cudaSuccess) return (int)e;                                                                         \
      set = true;                                                                                                  \
    }                                                                                                              \
    launch_pdl(delta_head_scan_kernel<R, V>, grid, block, smem, stream, a);                                        \
  } while (0)
#define YALM_DH(R)            \
  do {                        \
    if (vec) YALM_DH1(R, 4);  \
    else YALM_DH1(R, 1);      \
  } while (0)
  if (dk <= 32) YALM_DH(4);
  else if (dk <= 64) YALM_DH(8);
  else if (dk <= 128) YALM_DH(16);
  else YALM_DH(32);
#undef YALM_DH
#undef YALM_DH1
  YALM_LAUNCH_CHECK();
  return 0;
}
