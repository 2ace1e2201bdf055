// The matrix memory of xLSTM (Beck et al., "xLSTM: Extended Long Short-Term Memory") as the state-space scan of
// ssd.cu runs it, and the output step that the recurrences of this library's later designs share.
//
//  * mlstm_prep: per head, with i = cap tanh((z_i + b_i) / cap) and f = logsigmoid(cap tanh((z_f + b_f) / cap)),
//        m_t = max(f_t + m_(t-1), i_t),
//        S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T,   n_t likewise with k_t alone.
//    It writes log decays f + (m_(t-1) - m_t), inputs e^(i - m) and floors e^(-m) per token and head, and the
//    rows (x | B | C) = (v, 1, 0.. | k | q): n is one more column of the state, the one whose value is 1, and
//    n.q that column's output.  The running maximum is a scan over the step's tokens (x -> max(f + x, i)
//    composes as (f1 + f2, max(i1 + f2, i2))) and is carried in the sequence's state.  How m is rounded does not
//    matter to S: the logarithms are formed from the m's that are kept, and m_(t-1) - m_t is exact for
//    neighbours of a size, so what rounding leaves of m goes into the decay (which may be 1 + an ulp).
//  * gated_heads: every head's `size` values of y, divided by max(|y_size|, floor) + 1e-6 where the caller has a
//    floor (y_size: the value after the head's own), over their root mean square, times a weight, times a gate
//    (sigmoid or SiLU of a product's columns), into the storage type.
// All arithmetic is 32-bit.
#include "api.h"
#include "scan.cuh"

namespace yalm {

struct MlstmPrep {
  const float* proj;           // slices [n_partials][tokens][proj_row]
  int n_partials, proj_row, col_q, col_k, col_v, col_i, col_f;
  long long partial_stride;
  const float *i_bias, *f_bias;        // [H]
  float* act;                  // [tokens][H P + 2 H dk]
  float *log_decay, *put, *floor;      // [tokens][H]
  float* maxima;               // [slots][H]
  const int *q_start, *seq_slot;
  int n_tokens, n_seqs, H, dk, dv, P;
  float cap, q_scale;
};

constexpr int ML_THREADS = 256;

__device__ __forceinline__ float4 four_of(const float* p, int n, long long stride) {
  float4 v = *reinterpret_cast<const float4*>(p);
  for (int k = 1; k < n; ++k) {
    const float4 u = *reinterpret_cast<const float4*>(p + (size_t)k * stride);
    v.x += u.x; v.y += u.y; v.z += u.z; v.w += u.w;
  }
  return v;
}

// blocks 0 .. n_seqs H - 1: a (sequence, head)'s gates; the others: ML_PART elements of one token's row.  VEC: sizes,
// columns and pointers allow 16-byte accesses
constexpr int ML_PART = 2048;
template <bool VEC>
__global__ void __launch_bounds__(ML_THREADS) mlstm_prep_kernel(MlstmPrep a, int parts) {
  pdl_launch_dependents();
  const int n_gate = a.n_seqs * a.H;
  if ((int)blockIdx.x >= n_gate) {
    const int idx = blockIdx.x - n_gate, t = idx / parts, part = idx - t * parts;
    const int n_x = a.H * a.P, n_k = a.H * a.dk, row = n_x + 2 * n_k;
    pdl_wait();
    const float* p = a.proj + (size_t)t * a.proj_row;
    float* o = a.act + (size_t)t * row;
    const int end = min(row, (part + 1) * ML_PART);
    if constexpr (VEC) {
#pragma unroll
      for (int u = 0; u < ML_PART / (4 * ML_THREADS); ++u) {
        const int e = part * ML_PART + (u * ML_THREADS + threadIdx.x) * 4;
        if (e >= end) continue;
        float4 v;
        if (e < n_x) {
          const int h = e / a.P, c = e - h * a.P;
          v = c < a.dv ? four_of(p + a.col_v + h * a.dv + c, a.n_partials, a.partial_stride)
                       : make_float4(c == a.dv ? 1.f : 0.f, 0.f, 0.f, 0.f);
        } else if (e < n_x + n_k) {
          v = four_of(p + a.col_k + (e - n_x), a.n_partials, a.partial_stride);
        } else {
          v = four_of(p + a.col_q + (e - n_x - n_k), a.n_partials, a.partial_stride);
          v.x *= a.q_scale; v.y *= a.q_scale; v.z *= a.q_scale; v.w *= a.q_scale;
        }
        *reinterpret_cast<float4*>(o + e) = v;
      }
    } else {
      for (int e = part * ML_PART + threadIdx.x; e < end; e += ML_THREADS) {
        float v;
        if (e < n_x) {
          const int h = e / a.P, c = e - h * a.P;
          v = c < a.dv ? sum_slices(p + a.col_v + h * a.dv + c, a.n_partials, a.partial_stride) : (c == a.dv ? 1.f : 0.f);
        } else if (e < n_x + n_k) {
          v = sum_slices(p + a.col_k + (e - n_x), a.n_partials, a.partial_stride);
        } else {
          v = sum_slices(p + a.col_q + (e - n_x - n_k), a.n_partials, a.partial_stride) * a.q_scale;
        }
        o[e] = v;
      }
    }
    return;
  }
  __shared__ float sum_s[ML_THREADS / 32], top_s[ML_THREADS / 32], m_s[ML_THREADS];
  const int b = blockIdx.x / a.H, h = blockIdx.x - b * a.H;
  const int t0 = a.q_start[b], t1 = a.q_start[b + 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* kept = a.maxima + (size_t)a.seq_slot[b] * a.H + h;
  const float bi = a.i_bias[h], bf = a.f_bias[h];
  pdl_wait();
  float carry = *kept;
  __syncthreads();                                       // every thread has read it
  for (int base = t0; base < t1; base += ML_THREADS) {
    const int t = base + threadIdx.x;
    const bool on = t < t1;
    float li = -INFINITY, lf = 0.f;
    if (on) {
      const float* p = a.proj + (size_t)t * a.proj_row;
      li = a.cap * tanhf((sum_slices(p + a.col_i + h, a.n_partials, a.partial_stride) + bi) / a.cap);
      lf = -softplus(-a.cap * tanhf((sum_slices(p + a.col_f + h, a.n_partials, a.partial_stride) + bf) / a.cap));
    }
    float s = lf, m = li;                                // x -> max(s + x, m) from the chunk's first token to this one
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float s1 = __shfl_up_sync(0xffffffffu, s, o), m1 = __shfl_up_sync(0xffffffffu, m, o);
      if (lane >= o) {
        m = fmaxf(m1 + s, m);
        s += s1;
      }
    }
    if (lane == 31) { sum_s[warp] = s; top_s[warp] = m; }
    __syncthreads();
    float before = carry;
    for (int w = 0; w < warp; ++w) before = fmaxf(sum_s[w] + before, top_s[w]);
    m = fmaxf(s + before, m);
    m_s[threadIdx.x] = m;
    __syncthreads();
    if (on) {
      const float prev = threadIdx.x ? m_s[threadIdx.x - 1] : carry;
      const size_t at = (size_t)t * a.H + h;
      a.log_decay[at] = lf + (prev - m);
      a.put[at] = expf(li - m);
      a.floor[at] = expf(-m);
    }
    carry = m_s[min(ML_THREADS, t1 - base) - 1];
    __syncthreads();                                     // m_s and the warps' sums are written again
  }
  if (threadIdx.x == 0) *kept = carry;
}

struct GatedHeads {
  const float* y;              // [tokens][heads * pitch]
  const float* floor;          // [tokens][heads] or null
  const float* w;              // [heads * size]
  const float* gate;           // slices from the gate's first column on, rows of gate_row
  int gate_n, gate_row, silu;
  long long gate_stride;
  long long n_heads_total;
  int heads, size, pitch;
  float eps;
};

// LPH lanes per (token, head); W: neighbouring features per access; E accesses per lane kept in registers
template <typename T, int LPH, int W, int E>
__global__ void __launch_bounds__(256) gated_heads_kernel(GatedHeads a, T* __restrict__ out) {
  pdl_launch_dependents();
  const long long head = (long long)blockIdx.x * (256 / LPH) + threadIdx.x / LPH;
  const bool on = head < a.n_heads_total;
  const int lane = threadIdx.x & (LPH - 1);
  const long long hh = on ? head : 0;
  const long long t = hh / a.heads;
  const int h = (int)(hh - t * a.heads);
  pdl_wait();
  const float* y = a.y + hh * a.pitch;
  float v[E][W], ss = 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = (e * LPH + lane) * W;
#pragma unroll
    for (int j = 0; j < W; ++j) v[e][j] = 0.f;
    if (i < a.size) {
      if constexpr (W == 4) {
        const float4 u = *reinterpret_cast<const float4*>(y + i);
        v[e][0] = u.x; v[e][1] = u.y; v[e][2] = u.z; v[e][3] = u.w;
      } else {
        v[e][0] = y[i];
      }
    }
  }
  if (a.floor != nullptr) {
    const float den = fmaxf(fabsf(y[a.size]), a.floor[hh]) + 1e-6f;
#pragma unroll
    for (int e = 0; e < E; ++e)
#pragma unroll
      for (int j = 0; j < W; ++j) v[e][j] /= den;
  }
#pragma unroll
  for (int e = 0; e < E; ++e)
#pragma unroll
    for (int j = 0; j < W; ++j) ss += v[e][j] * v[e][j];
#pragma unroll
  for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!on) return;
  const float r = 1.0f / sqrtf(ss / (float)a.size + a.eps);
  const float* gp = a.gate + t * a.gate_row + (size_t)h * a.size;
  const float* w = a.w + (size_t)h * a.size;
  T* dst = out + hh * a.size;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = (e * LPH + lane) * W;
    if (i >= a.size) continue;
    float g[W];
    if constexpr (W == 4) {
      float4 s = *reinterpret_cast<const float4*>(gp + i);
      for (int k = 1; k < a.gate_n; ++k) {
        const float4 u = *reinterpret_cast<const float4*>(gp + (size_t)k * a.gate_stride + i);
        s.x += u.x; s.y += u.y; s.z += u.z; s.w += u.w;
      }
      g[0] = s.x; g[1] = s.y; g[2] = s.z; g[3] = s.w;
    } else {
      g[0] = sum_slices(gp + i, a.gate_n, a.gate_stride);
    }
    float o[W];
#pragma unroll
    for (int j = 0; j < W; ++j) o[j] = v[e][j] * r * w[i + j] * ((a.silu ? g[j] : 1.0f) / (1.0f + expf(-g[j])));
    if constexpr (W == 4 && sizeof(T) == 2) {
      *reinterpret_cast<uint2*>(dst + i) = make_uint2(pack2<T>(o[0], o[1]), pack2<T>(o[2], o[3]));
    } else {
#pragma unroll
      for (int j = 0; j < W; ++j) dst[i + j] = from_float<T>(o[j]);
    }
  }
}

}  // namespace yalm

using namespace yalm;

// proj: float32 slices [n_partials][tokens][proj_row] with q, k (H dk columns), v (H dv), i and f (H) at their
// columns; act float32 [tokens][H P + 2 H dk], P > dv; log_decay, put, floor float32 [tokens][H]; maxima float32
// [slots][H], read at the step's start and written at its end.
extern "C" int yalm_mlstm_prep(const float* proj, int n_partials, long long partial_stride, int proj_row, int col_q,
                               int col_k, int col_v, int col_i, int col_f, const float* i_bias, const float* f_bias,
                               float cap, float q_scale, float* act, float* log_decay, float* put, float* floor,
                               float* maxima, const int* q_start, const int* seq_slot, int n_tokens, int n_seqs, int H,
                               int dk, int dv, int P, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (H <= 0 || dk <= 0 || dv <= 0 || P <= dv || !(cap > 0.f)) return -2;
  const int parts = (H * P + 2 * H * dk + ML_PART - 1) / ML_PART;
  const long long blocks = (long long)n_seqs * H + (long long)n_tokens * parts;
  if (blocks > 0x7fffffffLL) return -4;
  const MlstmPrep a = {proj, n_partials, proj_row, col_q, col_k, col_v, col_i, col_f, partial_stride, i_bias, f_bias,
                       act, log_decay, put, floor, maxima, q_start, seq_slot, n_tokens, n_seqs, H, dk, dv, P, cap, q_scale};
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && P % 4 == 0 && proj_row % 4 == 0 && col_q % 4 == 0 && col_k % 4 == 0 &&
                   col_v % 4 == 0 && (partial_stride & 3) == 0 && ((((uintptr_t)proj) | ((uintptr_t)act)) & 15) == 0;
  if (vec) launch_pdl(mlstm_prep_kernel<true>, dim3((unsigned)blocks), dim3(ML_THREADS), 0, stream, a, parts);
  else launch_pdl(mlstm_prep_kernel<false>, dim3((unsigned)blocks), dim3(ML_THREADS), 0, stream, a, parts);
  YALM_LAUNCH_CHECK();
  return 0;
}

// y float32 [rows][heads pitch]; floor float32 [rows][heads] or null (with it pitch > size); w float32 [heads
// size]; gate: float32 slices whose columns col0 .. col0 + heads size are the gate's logits; out [rows][heads
// size] in out_dtype.  silu: the gate is SiLU instead of the sigmoid.  size up to 1,024.
extern "C" int yalm_gated_heads(const float* y, const float* floor, const float* w, const float* gate, int gate_n,
                                long long gate_stride, int gate_row, int col0, int silu, void* out, int out_dtype,
                                int rows, int heads, int size, int pitch, float eps, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (heads <= 0 || size <= 0 || size > 1024 || pitch < size || (floor != nullptr && pitch <= size)) return -2;
  const float* gc = gate + col0;
  const GatedHeads a = {y, floor, w, gc, gate_n, gate_row, silu, gate_stride, (long long)rows * heads, heads, size, pitch, eps};
  const bool vec = size % 4 == 0 && pitch % 4 == 0 && gate_row % 4 == 0 && (gate_stride & 3) == 0 &&
                   ((((uintptr_t)y) | ((uintptr_t)gc) | ((uintptr_t)out)) & 15) == 0;
  const int lph = vec && size <= 64 ? 16 : 32;
  const long long blocks = (a.n_heads_total + 256 / lph - 1) / (256 / lph);
  if (blocks > 0x7fffffffLL) return -4;
#define YALM_GH1(T, L, W, E) launch_pdl(gated_heads_kernel<T, L, W, E>, dim3((unsigned)blocks), dim3(256), 0, stream, a, (T*)out)
#define YALM_GH(T)                                \
  do {                                            \
    if (vec && size <= 64) YALM_GH1(T, 16, 4, 1); \
    else if (vec && size <= 128) YALM_GH1(T, 32, 4, 1); \
    else if (vec && size <= 512) YALM_GH1(T, 32, 4, 4); \
    else if (vec) YALM_GH1(T, 32, 4, 8);          \
    else if (size <= 128) YALM_GH1(T, 32, 1, 4);  \
    else YALM_GH1(T, 32, 1, 32);                  \
  } while (0)
  if (out_dtype == DT_F32) YALM_GH(float);
  else if (out_dtype == DT_BF16) YALM_GH(__nv_bfloat16);
  else if (out_dtype == DT_F16) YALM_GH(__half);
  else return -3;
#undef YALM_GH
#undef YALM_GH1
  YALM_LAUNCH_CHECK();
  return 0;
}
