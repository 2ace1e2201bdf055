// The gated delta rule with ONE decay per head, per head with key size dk and value size dv:
//   S <- e^(a_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t,   a_t <= 0
// (delta_rule.cu has the form with a decay per key channel, and delta_prep, which makes the unit vectors, the
// betas and the a_t).  32-bit throughout, the state carried from step to step as [slots][H][dv][dk]: a
// column's rows are neighbours.
//
//  * delta_head_scan: a block owns 16 value columns of one (sequence, head), eight lanes own a column, a lane
//    RPL of its rows in packed pairs; tokens come through a three-stage cp.async ring of 16.  With A_t =
//    e^(a_first + .. + a_t) over a group of 16 tokens and T = S / A the decay leaves the elements:
//        T <- T + k_t w^T,   w = beta_t (v_t / A_t - T^T k_t),   o_t = A_t T^T q_t,
//    three multiply-adds per element and token, and S = A T at the group's end.  A group that forgets more
//    than e^(-DH_SPAN) applies every token's own decay instead.  Every token needs one all-reduce over the
//    eight lanes before its write; the outputs' sums are formed for 16 tokens at once.
//  * delta_head_step: one token per sequence, the state streamed once: a warp per DS_COLS columns.
//
// A token's row, float32: [q: G dk | k: G dk | v: H dv | beta: H padded to 4 | a: H padded to 4].
#include "api.h"
#include "scan.cuh"

namespace yalm {

constexpr int DH_TOK = 16, DH_STAGES = 3, DH_WARPS = 4, DH_COLS = 4 * DH_WARPS;
constexpr float DH_SPAN = 30.f;

struct DeltaHead {
  const float* act;
  const int *q_start, *seq_slot;
  float* state;                // [slots][H][dv][dk]
  float* out;                  // [tokens][H dv]
  int row, H, G, dk, dv;
};

template <int RPL, int VEC>
__global__ void __launch_bounds__(32 * DH_WARPS) delta_head_scan_kernel(DeltaHead a) {
  pdl_launch_dependents();
  constexpr int DKP = 8 * RPL;                          // rows, padded
  constexpr int PER_TOK = 2 * DKP + DH_COLS + 4;        // q, k, this block's v columns, beta, a (+ padding)
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
  const int per = (2 * dk + min(DH_COLS, dv - c0)) / VEC;
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
        else { so = 2 * G * dk + h * dv + c0 + (f - 2 * dk); d = 2 * DKP + (f - 2 * dk); }
        for (int tt = 0; tt < nt; ++tt) ss_copy<4 * VEC>(dst + tt * PER_TOK + d, src + (size_t)tt * row + so);
      }
      if (threadIdx.x < nt) ss_copy<4>(dst + threadIdx.x * PER_TOK + 2 * DKP + DH_COLS, src + (size_t)threadIdx.x * row + beta_off);
      else if (threadIdx.x >= 32 && threadIdx.x < 32 + nt)
        ss_copy<4>(dst + (threadIdx.x - 32) * PER_TOK + 2 * DKP + DH_COLS + 1, src + (size_t)(threadIdx.x - 32) * row + beta_off + hp);
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
    const float la = mine < nt ? sg[mine * PER_TOK + 2 * DKP + DH_COLS + 1] : -0.f;
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
      const float beta = sg[tt * PER_TOK + 2 * DKP + DH_COLS];
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
    if (nt == DH_TOK && whole) {                        // the usual group: no test between the tokens
#pragma unroll
      for (int tt = 0; tt < DH_TOK; ++tt) token(tt, true);
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
    // the eight lanes' partial sums of the column's 16 outputs: in every round a lane hands half of its values to
    // its partner and adds the partner's other half to its own; two whole sums are left per lane
    static_assert(DH_TOK == 16, "two outputs per lane");
#pragma unroll
    for (int half = 4, n = 8; half >= 1; half >>= 1, n >>= 1) {
      const bool upper = (sub & half) != 0;
#pragma unroll
      for (int i = 0; i < n; ++i) {
        const float send = upper ? o[i] : o[i + n];
        const float keep = upper ? o[i + n] : o[i];
        o[i] = keep + __shfl_xor_sync(0xffffffffu, send, half);
      }
    }
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
extern "C" int yalm_delta_head_row(int H, int G, int dk, int dv) { return 2 * G * dk + H * dv + 2 * ((H + 3) & ~3); }

// act float32 [tokens][yalm_delta_head_row]; state float32 [slots][H][dv][dk], read at the step's start and
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
    const size_t smem = (size_t)DH_STAGES * DH_TOK * (2 * 8 * R + DH_COLS + 4) * sizeof(float);                    \
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
