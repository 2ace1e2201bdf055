// A state-space recurrence with one decay per head ("state-space duality"), per head with state
// size N and value size P:
//   S_t = exp(a_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,
//   dt_t = softplus(raw_t + bias),   a_t = -exp(A_log) dt_t,
// B and C shared by the heads of a group.  Everything here is 32-bit.  Two kernels:
//
//  * ssd_scan: a block of four warps owns SS_COLS = 32 value columns of one (sequence, head).  The
//    columns of S are independent; a group of eight lanes owns two of them, a lane RPT rows of
//    those, in packed pairs, so that a token costs a lane 2 RPT updates and 2 RPT multiply-adds
//    (half as many instructions) and the sums over the eight lanes are formed for SS_TOK tokens at
//    once.  Tokens (B | C | the block's x) come through a three-stage cp.async ring; the steps dt
//    and decays of a group are formed one stage ahead.  The update is S + (exp(a) - 1) S + dt B x:
//    exp(a) - 1 as expm1, so that a decay close to one is not rounded to a float near one each time.
//  * gated_group_norm: y silu(z), every one of `groups` equal parts of a row over its own root mean
//    square, times a weight per feature, into the storage type.
//
// The state is kept as [slots][H][P][N]: a column's rows are neighbours, which is how lanes own them.
#include "api.h"
#include "common.cuh"

namespace yalm {

constexpr int SS_COLS = 32, SS_TOK = 16, SS_STAGES = 3;

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

template <int BYTES>
__device__ __forceinline__ void ss_copy(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(dst)), "l"(src), "n"(BYTES) : "memory");
}

struct SsdArgs {
  const float* act;            // [tokens][H P + 2 G N] = (x | B | C), after the convolution
  const float* dt;             // slices [dt_n][tokens][dt_row], one raw step per head
  int dt_n, dt_row;
  long long dt_stride;
  const float *dt_bias, *a_log, *d_skip;       // [H]
  const int *q_start, *seq_slot;
  float* state;                // [slots][H][P][N]
  float* out;                  // [tokens][H P]
  int H, G, P, N;
};

// RPT rows per lane (8 RPT >= N); VEC: N, P and the pointers allow 16-byte accesses
template <int RPT, bool VEC>
__global__ void __launch_bounds__(128)
ssd_scan_kernel(SsdArgs a) {
  pdl_launch_dependents();
  constexpr int NP = 8 * RPT;                            // rows, padded
  constexpr int PER_TOK = 2 * NP + SS_COLS;              // B, C, then this block's x columns
  constexpr int K4 = RPT / 4;
  extern __shared__ __align__(16) float ss_stage[];      // [SS_STAGES][SS_TOK][PER_TOK]
  __shared__ float dt_s[SS_STAGES][SS_TOK], am1_s[SS_STAGES][SS_TOK];
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * SS_COLS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int sub = lane & 7, lc = warp * 8 + (lane >> 3) * 2;       // the lane's rows; its two columns in the block
  const int slot = a.seq_slot[b];
  const int t0 = a.q_start[b], t1 = a.q_start[b + 1];
  const int N = a.N, P = a.P, inner = a.H * P, row = inner + 2 * a.G * N;
  const int g = h / (a.H / a.G);
  const float neg_a = -expf(a.a_log[h]), bias = a.dt_bias[h], skip = a.d_skip[h];
  // rows beyond N and columns beyond P: never copied over, zero for ever
  if (N < NP || c0 + SS_COLS > P) {
    for (int i = threadIdx.x; i < SS_STAGES * SS_TOK * PER_TOK; i += blockDim.x) ss_stage[i] = 0.f;
    __syncthreads();
  }
  pdl_wait();
  const int cols = min(SS_COLS, P - c0);
  const int n_groups = (t1 - t0 + SS_TOK - 1) / SS_TOK;
  constexpr int W = VEC ? 4 : 1;
  const int per = (2 * N + cols) / W;                    // copies per token
  auto issue = [&](int gi) {
    if (gi < n_groups) {
      const int base = t0 + gi * SS_TOK;
      const int nt = min(SS_TOK, t1 - base);
      float* dst = ss_stage + (size_t)(gi % SS_STAGES) * SS_TOK * PER_TOK;
      for (int e = threadIdx.x; e < per; e += blockDim.x) {
        const int f = e * W;
        int so, d;
        if (f < N) { so = inner + g * N + f; d = f; }
        else if (f < 2 * N) { so = inner + (a.G + g) * N + (f - N); d = NP + (f - N); }
        else { so = h * P + c0 + (f - 2 * N); d = 2 * NP + (f - 2 * N); }
        const float* src = a.act + (size_t)base * row + so;
        for (int tt = 0; tt < nt; ++tt) ss_copy<4 * W>(dst + tt * PER_TOK + d, src + (size_t)tt * row);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // a group's raw steps are loaded by threads 0 .. SS_TOK - 1 when its copies are issued, and turned into
  // dt and exp(a) - 1 one group later
  auto load_dt = [&](int gi) {
    const int t = t0 + gi * SS_TOK + threadIdx.x;
    return (threadIdx.x < SS_TOK && t < t1) ? sum_slices(a.dt + (size_t)t * a.dt_row + h, a.dt_n, a.dt_stride) : 0.f;
  };
  auto put_dt = [&](int gi, float raw) {
    if (threadIdx.x < SS_TOK) {
      const float z = raw + bias;
      const float dt = z > 20.f ? z : log1pf(expf(z));
      dt_s[gi % SS_STAGES][threadIdx.x] = dt;
      am1_s[gi % SS_STAGES][threadIdx.x] = expm1f(neg_a * dt);
    }
  };
  issue(0);
  issue(1);
  put_dt(0, load_dt(0));
  float raw_next = load_dt(1);
  // the state: rows 32 k + 4 sub + j of the lane's two columns, in packed pairs
  f2 S[2][RPT / 2];
  float* st = a.state + ((size_t)slot * a.H + h) * P * N;
#pragma unroll
  for (int c = 0; c < 2; ++c) {
    const int col = c0 + lc + c;
    float* sc = st + (size_t)col * N;
#pragma unroll
    for (int k = 0; k < K4; ++k) {
      const int i = 32 * k + 4 * sub;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (col < P) {
        if constexpr (VEC) {
          if (i < N) v = *reinterpret_cast<const float4*>(sc + i);
        } else {
          if (i < N) v.x = sc[i];
          if (i + 1 < N) v.y = sc[i + 1];
          if (i + 2 < N) v.z = sc[i + 2];
          if (i + 3 < N) v.w = sc[i + 3];
        }
      }
      S[c][2 * k] = pack_f2(v.x, v.y);
      S[c][2 * k + 1] = pack_f2(v.z, v.w);
    }
  }
  for (int gi = 0; gi < n_groups; ++gi) {
    asm volatile("cp.async.wait_group %0;" ::"n"(SS_STAGES - 2) : "memory");
    __syncthreads();                                     // stage gi has landed; stage gi - 1 is no longer read
    issue(gi + 2);
    put_dt(gi + 1, raw_next);                            // read after the next barrier
    raw_next = load_dt(gi + 2);
    const int base = t0 + gi * SS_TOK;
    const int nt = min(SS_TOK, t1 - base);
    const float* sg = ss_stage + (size_t)(gi % SS_STAGES) * SS_TOK * PER_TOK;
    const float* dts = dt_s[gi % SS_STAGES];
    const float* ams = am1_s[gi % SS_STAGES];
    float o[SS_TOK * 2];
#pragma unroll
    for (int tt = 0; tt < SS_TOK; ++tt) {
      o[2 * tt] = o[2 * tt + 1] = 0.f;
      if (tt < nt) {
        const float* p = sg + tt * PER_TOK;
        const float2 x = *reinterpret_cast<const float2*>(p + 2 * NP + lc);
        const float dt = dts[tt], am1 = ams[tt];
        const f2 am = pack_f2(am1, am1);
        const f2 xd0 = pack_f2(dt * x.x, dt * x.x), xd1 = pack_f2(dt * x.y, dt * x.y);
        f2 o0 = 0ull, o1 = 0ull;                         // two zeros
#pragma unroll
        for (int k = 0; k < K4; ++k) {
          const ulonglong2 B = *reinterpret_cast<const ulonglong2*>(p + 32 * k + 4 * sub);
          const ulonglong2 C = *reinterpret_cast<const ulonglong2*>(p + NP + 32 * k + 4 * sub);
          S[0][2 * k] = add_f2(S[0][2 * k], fma_f2(am, S[0][2 * k], mul_f2(B.x, xd0)));
          S[1][2 * k] = add_f2(S[1][2 * k], fma_f2(am, S[1][2 * k], mul_f2(B.x, xd1)));
          S[0][2 * k + 1] = add_f2(S[0][2 * k + 1], fma_f2(am, S[0][2 * k + 1], mul_f2(B.y, xd0)));
          S[1][2 * k + 1] = add_f2(S[1][2 * k + 1], fma_f2(am, S[1][2 * k + 1], mul_f2(B.y, xd1)));
          o0 = fma_f2(S[0][2 * k], C.x, o0);
          o1 = fma_f2(S[1][2 * k], C.x, o1);
          o0 = fma_f2(S[0][2 * k + 1], C.y, o0);
          o1 = fma_f2(S[1][2 * k + 1], C.y, o1);
        }
        float lo, hi;
        unpack_f2(o0, lo, hi);
        o[2 * tt] = lo + hi;
        unpack_f2(o1, lo, hi);
        o[2 * tt + 1] = lo + hi;
      }
    }
    // the group's 2 SS_TOK outputs of these columns, each the sum of eight lanes' parts: in every round a
    // lane hands half of its values over and adds the other half of its partner's, so that lane `sub`
    // ends with the whole sums of values 4 s .. 4 s + 3 (two tokens), s = its bits from 4 down to 1
#pragma unroll
    for (int half = SS_TOK; half >= SS_TOK / 4; half >>= 1) {
      const int bit = half * 4 / SS_TOK;                 // lane bits 4, 2, 1
      const bool upper = (lane & bit) != 0;
#pragma unroll
      for (int i = 0; i < half; ++i) {
        const float send = upper ? o[i] : o[i + half];
        const float keep = upper ? o[i + half] : o[i];
        o[i] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int tt = sub * 2 + i, col = c0 + lc;
      if (tt < nt && col < P) {
        const float* x = sg + tt * PER_TOK + 2 * NP + lc;
        float* dst = a.out + (size_t)(base + tt) * inner + h * P + col;
        const float y0 = fmaf(skip, x[0], o[2 * i]), y1 = fmaf(skip, x[1], o[2 * i + 1]);
        if (VEC) {
          *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
        } else {
          dst[0] = y0;
          if (col + 1 < P) dst[1] = y1;
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int c = 0; c < 2; ++c) {
    const int col = c0 + lc + c;
    if (col >= P) continue;
    float* sc = st + (size_t)col * N;
#pragma unroll
    for (int k = 0; k < K4; ++k) {
      const int i = 32 * k + 4 * sub;
      float4 v;
      unpack_f2(S[c][2 * k], v.x, v.y);
      unpack_f2(S[c][2 * k + 1], v.z, v.w);
      if constexpr (VEC) {
        if (i < N) *reinterpret_cast<float4*>(sc + i) = v;
      } else {
        if (i < N) sc[i] = v.x;
        if (i + 1 < N) sc[i + 1] = v.y;
        if (i + 2 < N) sc[i + 2] = v.z;
        if (i + 3 < N) sc[i + 3] = v.w;
      }
    }
  }
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
// [tokens][H P].  N up to 256.
extern "C" int yalm_ssd_scan(const float* act, const float* dt, int dt_n, long long dt_stride, int dt_row, int col0,
                             const float* dt_bias, const float* a_log, const float* d_skip, const int* q_start,
                             const int* seq_slot, float* state, float* out, int n_tokens, int n_seqs, int H, int G,
                             int P, int N, cudaStream_t stream) {
  if (n_seqs <= 0 || n_tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || P <= 0 || N <= 0 || N > 256) return -2;
  if (n_seqs > 65535 || H > 65535) return -4;
  const SsdArgs a = {act, dt + col0, dt_n, dt_row, dt_stride, dt_bias, a_log, d_skip, q_start, seq_slot, state, out, H, G, P, N};
  const dim3 grid((P + SS_COLS - 1) / SS_COLS, H, n_seqs), block(128);
  const bool vec = N % 4 == 0 && P % 4 == 0 && ((((uintptr_t)act) | ((uintptr_t)state) | ((uintptr_t)out)) & 15) == 0;
#define YALM_SSD1(R, V)                                                                                       \
  do {                                                                                                        \
    const size_t smem = (size_t)SS_STAGES * SS_TOK * (2 * 8 * R + SS_COLS) * sizeof(float);                   \
    static bool set = false;                                                                                  \
    if (!set && smem > 40 * 1024) {                                                                           \
      cudaError_t e = cudaFuncSetAttribute(ssd_scan_kernel<R, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           (int)smem);                                                        \
      if (e != cudaSuccess) return (int)e;                                                                    \
      set = true;                                                                                             \
    }                                                                                                         \
    launch_pdl(ssd_scan_kernel<R, V>, grid, block, smem, stream, a);                                          \
  } while (0)
#define YALM_SSD(R)              \
  do {                           \
    if (vec) YALM_SSD1(R, true); \
    else YALM_SSD1(R, false);    \
  } while (0)
  if (N <= 32) YALM_SSD(4);
  else if (N <= 64) YALM_SSD(8);
  else if (N <= 128) YALM_SSD(16);
  else YALM_SSD(32);
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
