// A state-space recurrence with one decay per head ("state-space duality"), per head with state
// size N and value size P:
//   S_t = exp(a_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,
//   dt_t = softplus(raw_t + bias),   a_t = -exp(A_log) dt_t,
// B and C shared by the heads of a group.  Everything here is 32-bit.  Three kernels:
//
//  * ssd_scan: a block owns 32 (or 16) value columns of one (sequence, head).  The columns of S are
//    independent; 16 lanes own CPL = 4 (or 2) of them, a lane 4 K4 rows of those, in packed pairs (two FP32
//    operations per instruction).  Four warps compute; a fifth feeds them: it brings the tokens (B | C |
//    the block's x) through a three-stage cp.async ring of SS_TOK and turns their raw steps into dt and
//    decays.  The sums over the 16 lanes are formed for SS_RUN tokens at once.  Runs of SS_RUN whole
//    tokens whose decays multiply to no less than exp(-SS_SPAN) go without a decay per element: with
//    A_t = exp(a_first + .. + a_t) and T_t = S_t / A_t,
//        T_t = T_(t-1) + B_t (dt_t / A_t) x_t^T,   y_t = A_t T_t^T C_t,
//    two multiply-adds per element and token, and S = A T at the run's end.  Other tokens take
//    exp(a) S + dt B x.  A decay above one half is applied as S + (exp(a) - 1) S with exp(a) - 1 = expm1(a),
//    so that one close to one is not rounded to a float near one each time; a smaller one as it is, so
//    that what it leaves is not the difference of two nearly equal numbers.
//  * ssd_step: the same for steps of one token per sequence (bound by the state's bytes): a warp per
//    eight columns, the 32 lanes along a column's rows.
//  * gated_group_norm: y silu(z), every one of `groups` equal parts of a row over its own root mean
//    square, times a weight per feature, into the storage type.
//
// The state is kept as [slots][H][P][N]: a column's rows are neighbours, which is how lanes own them.
#include "api.h"
#include "scan.cuh"

namespace yalm {

constexpr float SS_SPAN = 16.f;

struct SsdArgs {
  const float* act;            // [tokens][H P + 2 G N] = (x | B | C), after the convolution
  const float* dt;             // slices [dt_n][tokens][dt_row], one raw step per head
  int dt_n, dt_row;
  long long dt_stride;
  const float *dt_bias, *a_log, *d_skip;       // [H]; d_skip may be null
  const float *log_decay, *put;                // [tokens][H]: a_t and dt_t as they are, in place of the four above
  const int *q_start, *seq_slot;
  float* state;                // [slots][H][P][N]
  float* out;                  // [tokens][H P]
  int H, G, P, N;
};

// K4: groups of four rows per lane (64 K4 >= N); VEC: N, P and the pointers allow 16-byte accesses
template <int K4, bool VEC, int CPL>
__global__ void __launch_bounds__(160, 1)
ssd_scan_kernel(SsdArgs a) {
  pdl_launch_dependents();
  constexpr int COLS = 8 * CPL;
  constexpr int NP = 64 * K4;                            // rows, padded
  constexpr int PER_TOK = 2 * NP + COLS;              // B, C, then this block's x columns
  extern __shared__ __align__(16) float ss_stage[];      // [SS_STAGES][SS_TOK][PER_TOK]
  // per token: the decay's coefficient, dt, and for whole runs A_t and dt / A_t
  __shared__ __align__(16) float4 step_s[SS_STAGES][SS_TOK];
  __shared__ float2 run_s[SS_STAGES][SS_TOK / SS_RUN];   // a run's sum of a, its decay's coefficient
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * COLS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int slot = a.seq_slot[b];
  const int t0 = a.q_start[b], t1 = a.q_start[b + 1];
  const int N = a.N, P = a.P, inner = a.H * P;
  // rows beyond N and columns beyond P: never copied over, zero for ever
  if (N < NP || c0 + COLS > P) {
    for (int i = threadIdx.x; i < SS_STAGES * SS_TOK * PER_TOK; i += blockDim.x) ss_stage[i] = 0.f;
    __syncthreads();
  }
  pdl_wait();
  const int n_groups = (t1 - t0 + SS_TOK - 1) / SS_TOK;
  if (warp == 4) {                                       // the warp that feeds the others
    const int row = inner + 2 * a.G * N, g = h / (a.H / a.G);
    const bool given = a.put != nullptr;
    const float neg_a = given ? 0.f : -expf(a.a_log[h]), bias = given ? 0.f : a.dt_bias[h];
    constexpr int W = VEC ? 4 : 1;
    const int per = (2 * N + min(COLS, P - c0)) / W;  // copies per token
    auto issue = [&](int gi) {
      if (gi < n_groups) {
        const int base = t0 + gi * SS_TOK;
        const int nt = min(SS_TOK, t1 - base);
        float* dst = ss_stage + (size_t)(gi % SS_STAGES) * SS_TOK * PER_TOK;
        for (int e = lane; e < per; e += 32) {
          const int f = e * W;
          int so, d;
          if (f < N) { so = inner + g * N + f; d = f; }
          else if (f < 2 * N) { so = inner + (a.G + g) * N + (f - N); d = NP + (f - N); }
          else { so = h * P + c0 + (f - 2 * N); d = 2 * NP + (f - 2 * N); }
          const float* src = a.act + (size_t)base * row + so;
          ss_copy_tokens<4 * W>(dst + d, PER_TOK, src, row, nt);
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto load_dt = [&](int gi) {
      const int t = t0 + gi * SS_TOK + lane;
      if (lane >= SS_TOK || t >= t1) return make_float2(0.f, -0.f);
      if (given) return make_float2(a.put[(size_t)t * a.H + h], a.log_decay[(size_t)t * a.H + h]);
      return make_float2(sum_slices(a.dt + (size_t)t * a.dt_row + h, a.dt_n, a.dt_stride), 0.f);
    };
    auto put_dt = [&](int gi, float2 raw) {
      const float dt = given ? raw.x : softplus(raw.x + bias);
      const float la = given ? raw.y : neg_a * dt;
      float cum = la;                                    // the run's inclusive sum
#pragma unroll
      for (int o = 1; o < SS_RUN; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, cum, o, SS_RUN);
        if ((lane & (SS_RUN - 1)) >= o) cum += v;
      }
      if (lane < SS_TOK) {
        const float A = expf(cum);
        step_s[gi % SS_STAGES][lane] = make_float4(decay_coef(la), dt, A, dt / A);     // dt / A is read for short spans only
        if ((lane & (SS_RUN - 1)) == SS_RUN - 1) run_s[gi % SS_STAGES][lane / SS_RUN] = make_float2(cum, decay_coef(cum));
      }
    };
    float2 raw0 = load_dt(0), raw1 = load_dt(1);
    issue(0);
    issue(1);
    put_dt(0, raw0);
    put_dt(1, raw1);
    float2 raw = load_dt(2);
    for (int gi = 0; gi < n_groups; ++gi) {
      asm volatile("cp.async.wait_group %0;" ::"n"(SS_STAGES - 2) : "memory");
      __syncthreads();                                   // stage gi has landed; stage gi - 1 is no longer read
      issue(gi + 2);
      put_dt(gi + 2, raw);
      raw = load_dt(gi + 3);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    return;
  }
  const int sub = lane & 15, lc = (warp * 2 + (lane >> 4)) * CPL;       // the lane's rows; its first column in the block
  const float skip = a.d_skip != nullptr ? a.d_skip[h] : 0.f;
  // the state: rows 64 k + 4 sub + j of the lane's columns, in packed pairs
  f2 S[CPL][2 * K4];
  float* st = a.state + ((size_t)slot * a.H + h) * P * N;
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int col = c0 + lc + c;
    load_column<K4, VEC>(st + (size_t)col * N, N, sub, col < P, S[c]);
  }
  for (int gi = 0; gi < n_groups; ++gi) {
    __syncthreads();
    const int base = t0 + gi * SS_TOK;
    const int nt = min(SS_TOK, t1 - base);
    const float* sg = ss_stage + (size_t)(gi % SS_STAGES) * SS_TOK * PER_TOK;
    const float4* steps = step_s[gi % SS_STAGES];
#pragma unroll 1
    for (int r = 0; r < SS_TOK / SS_RUN; ++r) {
      const int first = r * SS_RUN;
      if (first >= nt) break;
      const float2 run = run_s[gi % SS_STAGES][r];
      float o[SS_RUN * CPL];
      if (nt >= first + SS_RUN && run.x >= -SS_SPAN) {
        RunToken<K4, CPL> buf[2];
        auto fetch = [&](int tt) {
          const float* p = sg + (first + tt) * PER_TOK;
          buf[tt & 1].fetch(p + NP + 4 * sub, p + 4 * sub, p + 2 * NP + lc);
        };
        fetch(0);
#pragma unroll
        for (int tt = 0; tt < SS_RUN; ++tt) {
          const float4 sv = steps[first + tt];
          if (tt + 1 < SS_RUN) fetch(tt + 1);
#pragma unroll
          for (int c = 0; c < CPL; ++c) buf[tt & 1].x[c] *= sv.w;
          buf[tt & 1].apply(S, o + CPL * tt);
#pragma unroll
          for (int c = 0; c < CPL; ++c) o[CPL * tt + c] *= sv.z;
        }
        const float keep = decay_keep(run.y);
        const f2 e = pack_f2(run.y, run.y), kp = pack_f2(keep, keep);
#pragma unroll
        for (int c = 0; c < CPL; ++c)
#pragma unroll
          for (int k = 0; k < 2 * K4; ++k) S[c][k] = fma_f2(e, S[c][k], mul_f2(kp, S[c][k]));
      } else {
#pragma unroll
        for (int tt = 0; tt < SS_RUN; ++tt) {
#pragma unroll
          for (int c = 0; c < CPL; ++c) o[CPL * tt + c] = 0.f;
          if (first + tt < nt) {
            const float* p = sg + (first + tt) * PER_TOK;
            const float4 sv = steps[first + tt];
            const float keep = decay_keep(sv.x);
            const f2 am = pack_f2(sv.x, sv.x), kp = pack_f2(keep, keep);
            float x[CPL];
            load_columns<CPL>(p + 2 * NP + lc, x);
#pragma unroll
            for (int c = 0; c < CPL; ++c) x[c] *= sv.y;
            f2 oc[CPL];
#pragma unroll
            for (int k = 0; k < K4; ++k) {
              const ulonglong2 B = *reinterpret_cast<const ulonglong2*>(p + 64 * k + 4 * sub);
              const ulonglong2 C = *reinterpret_cast<const ulonglong2*>(p + NP + 64 * k + 4 * sub);
#pragma unroll
              for (int c = 0; c < CPL; ++c) {
                const f2 xd = pack_f2(x[c], x[c]);
                S[c][2 * k] = fma_f2(kp, S[c][2 * k], fma_f2(am, S[c][2 * k], mul_f2(B.x, xd)));
                S[c][2 * k + 1] = fma_f2(kp, S[c][2 * k + 1], fma_f2(am, S[c][2 * k + 1], mul_f2(B.y, xd)));
                oc[c] = k == 0 ? mul_f2(S[c][0], C.x) : fma_f2(S[c][2 * k], C.x, oc[c]);
                oc[c] = fma_f2(S[c][2 * k + 1], C.y, oc[c]);
              }
            }
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
              float lo, hi;
              unpack_f2(oc[c], lo, hi);
              o[CPL * tt + c] = lo + hi;
            }
          }
        }
      }
      // the run's outputs of these columns: lane `sub` gets CPL / 2 of token sub / 2's
      run_sums<CPL>(o, lane);
      const int tt = first + (sub >> 1), lcc = lc + (sub & 1) * (CPL / 2), col = c0 + lcc;
      if (tt < nt && col < P) {
        const float* x = sg + tt * PER_TOK + 2 * NP + lcc;
        float* dst = a.out + (size_t)(base + tt) * inner + h * P + col;
        if constexpr (VEC && CPL == 4) {
          *reinterpret_cast<float2*>(dst) = make_float2(fmaf(skip, x[0], o[0]), fmaf(skip, x[1], o[1]));
        } else {
#pragma unroll
          for (int c = 0; c < CPL / 2; ++c)
            if (col + c < P) dst[c] = fmaf(skip, x[c], o[c]);
        }
      }
    }
  }
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int col = c0 + lc + c;
    if (col < P) store_column<K4, VEC>(st + (size_t)col * N, N, sub, S[c]);
  }
}

constexpr int SD_COLS = 8;                               // columns per warp of ssd_step

// One token per sequence.  grid (column tiles of 8 SD_COLS, heads, sequences), eight warps
template <bool VEC>
__global__ void __launch_bounds__(256, 3)
ssd_step_kernel(SsdArgs a) {
  pdl_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c0 = (blockIdx.x * 8 + warp) * SD_COLS;
  const int slot = a.seq_slot[b], t = a.q_start[b];
  const int N = a.N, P = a.P, inner = a.H * P;
  if (c0 >= P) return;
  const int g = h / (a.H / a.G);
  float* st = a.state + ((size_t)slot * a.H + h) * P * N;
  const float* row = a.act + (size_t)t * (inner + 2 * a.G * N);
  pdl_wait();
  const bool given = a.put != nullptr;
  const float dt = given ? a.put[(size_t)t * a.H + h]
                         : softplus(sum_slices(a.dt + (size_t)t * a.dt_row + h, a.dt_n, a.dt_stride) + a.dt_bias[h]);
  const float coef = decay_coef(given ? a.log_decay[(size_t)t * a.H + h] : -expf(a.a_log[h]) * dt), keep = decay_keep(coef);
  float x[SD_COLS], y[SD_COLS];
#pragma unroll
  for (int c = 0; c < SD_COLS; ++c) {
    x[c] = c0 + c < P ? row[h * P + c0 + c] : 0.f;
    y[c] = 0.f;
  }
  constexpr int W = VEC ? 4 : 1;
  for (int i = lane * W; i < N; i += 32 * W) {
    float B[W], C[W], S[SD_COLS][W];
    if constexpr (VEC) {
#pragma unroll
      for (int c = 0; c < SD_COLS; ++c) {
        const float4 v = c0 + c < P ? *reinterpret_cast<const float4*>(st + (size_t)(c0 + c) * N + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[c][0] = v.x; S[c][1] = v.y; S[c][2] = v.z; S[c][3] = v.w;
      }
      const float4 u = *reinterpret_cast<const float4*>(row + inner + g * N + i);
      const float4 w = *reinterpret_cast<const float4*>(row + inner + (a.G + g) * N + i);
      B[0] = u.x; B[1] = u.y; B[2] = u.z; B[3] = u.w;
      C[0] = w.x; C[1] = w.y; C[2] = w.z; C[3] = w.w;
    } else {
#pragma unroll
      for (int c = 0; c < SD_COLS; ++c) S[c][0] = c0 + c < P ? st[(size_t)(c0 + c) * N + i] : 0.f;
      B[0] = row[inner + g * N + i];
      C[0] = row[inner + (a.G + g) * N + i];
    }
#pragma unroll
    for (int c = 0; c < SD_COLS; ++c) {
#pragma unroll
      for (int j = 0; j < W; ++j) {
        S[c][j] = fmaf(keep, S[c][j], fmaf(coef, S[c][j], B[j] * (dt * x[c])));
        y[c] = fmaf(S[c][j], C[j], y[c]);
      }
      if (c0 + c < P) {
        if constexpr (VEC) *reinterpret_cast<float4*>(st + (size_t)(c0 + c) * N + i) = make_float4(S[c][0], S[c][1], S[c][2], S[c][3]);
        else st[(size_t)(c0 + c) * N + i] = S[c][0];
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
  if (lane < SD_COLS && c0 + lane < P)
    a.out[(size_t)t * inner + h * P + c0 + lane] = fmaf(a.d_skip != nullptr ? a.d_skip[h] : 0.f, row[h * P + c0 + lane], y[0]);
}

// grid (tokens, groups); y [tokens][inner]; z slices [z_n][tokens][z_row]; out [tokens][inner]
template <typename T, bool VEC>
__global__ void gated_group_norm_kernel(const float* __restrict__ y, const float* __restrict__ z, int z_n,
                                        long long z_stride, int z_row, const float* __restrict__ w,
                                        T* __restrict__ out, int inner, int size, float eps) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float gg_row[];
  __shared__ float scratch[33];
  const size_t t = blockIdx.x;
  const int f0 = blockIdx.y * size;
  pdl_wait();
  const float* yr = y + t * inner + f0;
  const float* zr = z + t * z_row + f0;
  constexpr int W = VEC ? 4 : 1;
  float ss = 0.f;
  for (int i = threadIdx.x * W; i < size; i += blockDim.x * W) {
    float v[W], u[W];
    if constexpr (VEC) {
      const float4 a = *reinterpret_cast<const float4*>(yr + i);
      v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
      float4 s = *reinterpret_cast<const float4*>(zr + i);
      for (int k = 1; k < z_n; ++k) {
        const float4 e = *reinterpret_cast<const float4*>(zr + (size_t)k * z_stride + i);
        s.x += e.x; s.y += e.y; s.z += e.z; s.w += e.w;
      }
      u[0] = s.x; u[1] = s.y; u[2] = s.z; u[3] = s.w;
    } else {
      v[0] = yr[i];
      u[0] = sum_slices(zr + i, z_n, z_stride);
    }
#pragma unroll
    for (int j = 0; j < W; ++j) {
      const float r = v[j] * (u[j] / (1.0f + expf(-u[j])));
      gg_row[i + j] = r;
      ss += r * r;
    }
  }
  const float r = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + eps);
  T* dst = out + t * inner + f0;
  for (int i = threadIdx.x * W; i < size; i += blockDim.x * W) {
    if constexpr (VEC && sizeof(T) == 2) {
      uint2 u;
      u.x = pack2<T>(gg_row[i] * r * w[f0 + i], gg_row[i + 1] * r * w[f0 + i + 1]);
      u.y = pack2<T>(gg_row[i + 2] * r * w[f0 + i + 2], gg_row[i + 3] * r * w[f0 + i + 3]);
      *reinterpret_cast<uint2*>(dst + i) = u;
    } else {
#pragma unroll
      for (int j = 0; j < W; ++j) dst[i + j] = from_float<T>(gg_row[i + j] * r * w[f0 + i + j]);
    }
  }
}

}  // namespace yalm

using namespace yalm;

// act float32 [tokens][H P + 2 G N] = (x | B | C); dt: float32 slices whose column col0 + h is head h's raw
// step; state float32 [slots][H][P][N], read at the step's start and written at its end; out float32
// [tokens][H P].  N up to 256.  With put and log_decay float32 [tokens][H] those are dt_t and a_t themselves
// (a_t <= 0), and dt, dt_bias, a_log are not read.  d_skip may be null.
extern "C" int yalm_ssd_scan(const float* act, const float* dt, int dt_n, long long dt_stride, int dt_row, int col0,
                             const float* dt_bias, const float* a_log, const float* d_skip, const float* log_decay,
                             const float* put, const int* q_start,
                             const int* seq_slot, float* state, float* out, int n_tokens, int n_seqs, int H, int G,
                             int P, int N, cudaStream_t stream) {
  if (n_seqs <= 0 || n_tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || P <= 0 || N <= 0 || N > 256) return -2;
  if ((put == nullptr) != (log_decay == nullptr) || (put == nullptr && (dt == nullptr || dt_bias == nullptr || a_log == nullptr))) return -3;
  if (n_seqs > 65535 || H > 65535) return -4;
  const SsdArgs a = {act, dt + col0, dt_n, dt_row, dt_stride, dt_bias, a_log, d_skip, log_decay, put, q_start, seq_slot, state, out, H, G, P, N};
  const bool vec = N % 4 == 0 && P % 4 == 0 && ((((uintptr_t)act) | ((uintptr_t)state) | ((uintptr_t)out)) & 15) == 0;
  if (n_tokens == n_seqs) {                              // every sequence brings one token
    const dim3 sgrid((P + 8 * SD_COLS - 1) / (8 * SD_COLS), H, n_seqs), sblock(256);
    if (vec) launch_pdl(ssd_step_kernel<true>, sgrid, sblock, 0, stream, a);
    else launch_pdl(ssd_step_kernel<false>, sgrid, sblock, 0, stream, a);
    YALM_LAUNCH_CHECK();
    return 0;
  }
  const bool narrow = narrow_blocks((long long)((P + 31) / 32) * H * n_seqs);
  const int cols = narrow ? 16 : 32;
  const dim3 grid((P + cols - 1) / cols, H, n_seqs), block(160);
#define YALM_SSD1(K, V, C)                                                                                    \
  do {                                                                                                        \
    const size_t smem = (size_t)SS_STAGES * SS_TOK * (2 * 64 * K + 8 * C) * sizeof(float);                    \
    static bool set = false;                                                                                  \
    if (!set && smem > 40 * 1024) {                                                                           \
      cudaError_t e = cudaFuncSetAttribute(ssd_scan_kernel<K, V, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           (int)smem);                                                        \
      if (e != cudaSuccess) return (int)e;                                                                    \
      set = true;                                                                                             \
    }                                                                                                         \
    launch_pdl(ssd_scan_kernel<K, V, C>, grid, block, smem, stream, a);                                       \
  } while (0)
#define YALM_SSD(K)                              \
  do {                                           \
    if (vec && narrow) YALM_SSD1(K, true, 2);    \
    else if (vec) YALM_SSD1(K, true, 4);         \
    else if (narrow) YALM_SSD1(K, false, 2);     \
    else YALM_SSD1(K, false, 4);                 \
  } while (0)
  if (N <= 64) YALM_SSD(1);
  else if (N <= 128) YALM_SSD(2);
  else YALM_SSD(4);
#undef YALM_SSD
#undef YALM_SSD1
  YALM_LAUNCH_CHECK();
  return 0;
}

// out [rows][inner] (out_dtype) = n(y silu(z)) w, the norm over each of `groups` equal parts of a row; y
// float32 [rows][inner], z float32 slices whose columns col0 .. col0 + inner are the gate's logits
extern "C" int yalm_gated_group_norm(const float* y, const float* z, int z_n, long long z_stride, int z_row, int col0,
                                     const float* w, void* out, int out_dtype, int rows, int inner, int groups,
                                     float eps, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (inner <= 0 || groups <= 0 || inner % groups || groups > 65535) return -2;
  const int size = inner / groups;
  if (size > 12000) return -2;
  const float* zc = z + col0;
  const bool vec = size % 4 == 0 && z_row % 4 == 0 && (z_stride & 3) == 0 &&
                   ((((uintptr_t)y) | ((uintptr_t)zc) | ((uintptr_t)out)) & 15) == 0;
  int threads = ((vec ? size / 4 : size) + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const dim3 grid(rows, groups), block(threads);
  const size_t smem = (size_t)size * sizeof(float);
#define YALM_GG(T, V)                                                                                     \
  launch_pdl(gated_group_norm_kernel<T, V>, grid, block, smem, stream, y, zc, z_n, z_stride, z_row, w,    \
             (T*)out, inner, size, eps)
  if (out_dtype == DT_F32) { if (vec) YALM_GG(float, true); else YALM_GG(float, false); }
  else if (out_dtype == DT_BF16) { if (vec) YALM_GG(__nv_bfloat16, true); else YALM_GG(__nv_bfloat16, false); }
  else if (out_dtype == DT_F16) { if (vec) YALM_GG(__half, true); else YALM_GG(__half, false); }
  else return -3;
#undef YALM_GG
  YALM_LAUNCH_CHECK();
  return 0;
}
