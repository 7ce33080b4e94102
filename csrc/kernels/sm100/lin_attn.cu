// build: precise
// Linear attention whose state decays per key channel, token by token, with what goes around it (lin_attn_chunk.cu holds
// the form for prompts). Per (sequence, head), with k_t, alpha_t over dk key channels and v_t over dv columns:
//     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T
//     o_t = S_t^T q_t                                     (no bonus)
//     o_t = (S_(t-1) + diag(u) k_t v_t^T)^T q_t           (bonus u: the current token is read with its own weight)
// and o, normed per head, times a weight, times silu(gate), is the mixer's output before its projection.
//   kern_token_shift_<act>      every row mixed with the row before it, once per target
//   kern_shift_state_<act>      the last row of each sequence into its state line
//   kern_decay_<in>             alpha = sigmoid(z)^(1/tau) or exp(-exp(z)), z = W act(a) + bias from a low-rank row
//   kern_lin_rule_<act>_*       the recurrence; `fused` also norms, weighs and gates
//   kern_lin_norm_gate_<act>    the same behind the chunk kernel
// A state line holds [previous row: f32, when the mixer shifts][S: H x dk x dv f32]; line 0 is the null line (padding rows
// use it and nothing is written to it). Decays, state and norms are f32; q, k, v, gates and outputs are activations.
#include "act.cuh"

using namespace kern;

namespace {

KERN_DEVICE int checked_line(const uint8_t* state, int line, long long line_bytes) {
  return line > 0 && KERN_CHECK(state + (size_t)line * line_bytes, (size_t)line_bytes, SITE_STATE_SLOT) ? line : 0;
}

KERN_DEVICE int seq_of_row(const int* cu, int seqs, int r) {      // the last s with cu[s] <= r
  int lo = 0, hi = seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= r) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// ---- token shift ------------------------------------------------------------------------------------------------
// grid [rows, column blocks]; out [rows][targets][width] = h + (before - h) mu[target]. Without cu (one row per sequence)
// the row also goes into the line; of a ragged call kern_shift_state does that afterwards.
template <typename T, int V>
KERN_DEVICE void shift_body(const T* h, const __nv_bfloat16* mu, T* out, uint8_t* state, const int* lines, const int* cu,
                            int seqs, int width, int targets, long long line_bytes) {
  const int r = blockIdx.x;
  if (r >= (cu ? cu[seqs] : seqs)) return;
  const int s = cu ? seq_of_row(cu, seqs, r) : r;
  const bool first = !cu || r == cu[s];
  const int line = first ? checked_line(state, lines[s], line_bytes) : 0;
  float* kept = reinterpret_cast<float*>(state + (size_t)line * line_bytes);
  for (int c = (blockIdx.y * 256 + threadIdx.x) * V; c < width; c += gridDim.y * 256 * V) {
    const Vec<V> x = ldv<V>(h + (size_t)r * width + c);
    Vec<V> b = {};
    if (!first) b = ldv<V>(h + (size_t)(r - 1) * width + c);
    else if (line > 0) b = ldv<V>(kept + c);
    if (!cu && line > 0) stv<V>(kept + c, x);
    for (int m = 0; m < targets; ++m) {
      const Vec<V> w = ldv<V>(mu + (size_t)m * width + c);
      Vec<V> o;
#pragma unroll
      for (int e = 0; e < V; ++e) o.v[e] = x.v[e] + (b.v[e] - x.v[e]) * w.v[e];
      stv<V>(out + ((size_t)r * targets + m) * width + c, o);
    }
  }
}

template <typename T>
KERN_DEVICE void shift_state_body(const T* h, uint8_t* state, const int* lines, const int* cu, int seqs, int width,
                                  long long line_bytes) {
  const int s = blockIdx.x;
  if (s >= seqs || cu[s + 1] <= cu[s]) return;
  const int line = checked_line(state, lines[s], line_bytes);
  if (line <= 0) return;
  float* kept = reinterpret_cast<float*>(state + (size_t)line * line_bytes);
  for (int c = blockIdx.y * 256 + threadIdx.x; c < width; c += gridDim.y * 256) kept[c] = ldf(h + (size_t)(cu[s + 1] - 1) * width + c);
}

// ---- the decays ---------------------------------------------------------------------------------------------------
// One 64 x 64 tile of alpha [rows, n] per block: z = act(a) . W^T + bias in f32, then the decay. mode 0: act(a) = a,
// alpha = sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau); mode 1: act = tanh, alpha = exp(-exp(z)).
constexpr int DB = 64, DK = 64;
template <typename T>
KERN_DEVICE void decay_body(const T* a, const __nv_bfloat16* W, const __nv_bfloat16* bias, float* alpha, int rows, int n, int rank,
                            int lda, int mode, float inv_tau) {
  __shared__ __align__(16) float as[DK][DB + 4], ws[DK][DB + 4];
  const int m0 = blockIdx.y * DB, n0 = blockIdx.x * DB;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < rank; k0 += DK) {
    // a warp moves 8 columns of 4 rows at a time: whole sectors in, no two lanes on one bank
    const int kb = threadIdx.x & 7, rb = (threadIdx.x >> 3) & 3, warp = threadIdx.x >> 5;
#pragma unroll 4
    for (int i = warp; i < (DB / 4) * (DK / 8); i += 8) {
      const int r = (i / (DK / 8)) * 4 + rb, k = (i % (DK / 8)) * 8 + kb;
      const float v = (k0 + k < rank && m0 + r < rows) ? ldf(a + (size_t)(m0 + r) * lda + k0 + k) : 0.f;
      as[k][r] = mode && v != 0.f ? tanhf(v) : v;
      ws[k][r] = (k0 + k < rank && n0 + r < n) ? __bfloat162float(W[(size_t)(n0 + r) * rank + k0 + k]) : 0.f;
    }
    __syncthreads();
    const int kn = min(DK, (rank - k0 + 3) & ~3);      // what is past the rank is zero
#pragma unroll 4
    for (int k = 0; k < kn; ++k) {
      const Vec<4> x = ldv<4>(&as[k][ty * 4]), w = ldv<4>(&ws[k][tx * 4]);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += x.v[i] * w.v[j];
    }
    __syncthreads();
  }
  const int c = n0 + tx * 4;
  float b[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) b[j] = c + j < n ? __bfloat162float(bias[c + j]) : 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = m0 + ty * 4 + i;
    if (r >= rows) continue;
    Vec<4> o;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float z = acc[i][j] + b[j];
      o.v[j] = expf(mode ? -expf(z) : -(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau);
    }
    float* dst = alpha + (size_t)r * n + c;
    if (n % 4 == 0) {
      if (c < n) stv<4>(dst, o);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < n) dst[j] = o.v[j];
    }
  }
}

// ---- the recurrence ------------------------------------------------------------------------------------------------
struct RuleArgs {
  const void *q, *k, *v, *gate;
  const float* alpha;
  const __nv_bfloat16 *u, *norm;      // u null: no bonus
  void* out;                          // fused: T [.., out_stride]; else f32 [rows, H dv]
  uint8_t* state;
  const int *lines, *cu;
  int seqs, H, dk, dv, stride, norm_step, out_stride, s_off, fused, tb, max_rows;
  long long line_bytes;
  float q_scale, out_scale, eps;
};

// A block owns a head's columns [c0, c0 + 32 V) of one sequence: a lane V of them, a warp the key channels warp, + 8, ..
// (RK of them at most, so S is RK x V registers). V: columns of a lane, contiguous.
template <typename T, int RK, int V>
KERN_DEVICE void rule_body(const RuleArgs& a) {
  extern __shared__ __align__(16) float rule_sm[];
  __shared__ float part[2][8][32 * V];
  const int tiles = (a.dv + 32 * V - 1) / (32 * V);
  const int h = blockIdx.x / tiles, c0 = (blockIdx.x % tiles) * 32 * V, s = blockIdx.y;
  if (s >= a.seqs) return;
  const int r0 = a.cu ? a.cu[s] : s, r1 = a.cu ? a.cu[s + 1] : s + 1;
  if (r1 <= r0 || r1 - r0 > a.max_rows) return;      // longer sequences belong to the chunk kernel
  const int line = checked_line(a.state, a.lines[s], a.line_bytes);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c = c0 + lane * V;
  const int dk = a.dk, dv = a.dv, tb = a.tb;
  const bool vec = V > 1 && dv % V == 0;
  float* qs = rule_sm;                    // [tb][dk] each
  float* ks = qs + tb * dk;
  float* as = ks + tb * dk;
  float* us = as + tb * dk;               // [dk], with a bonus
  float* Sg = reinterpret_cast<float*>(a.state + (size_t)line * a.line_bytes + a.s_off) + (size_t)h * dk * dv;
  float S[RK][V];
#pragma unroll
  for (int i = 0; i < RK; ++i) {
    const int kk = i * 8 + warp;
#pragma unroll
    for (int e = 0; e < V; ++e) S[i][e] = 0.f;
    if (line > 0 && kk < dk && c < dv) {
      if (vec) {
        if constexpr (V == 4) {
          const float4 f = *reinterpret_cast<const float4*>(Sg + (size_t)kk * dv + c);
          S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
        } else if constexpr (V == 2) {
          const float2 f = *reinterpret_cast<const float2*>(Sg + (size_t)kk * dv + c);
          S[i][0] = f.x; S[i][1] = f.y;
        }
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e)
          if (c + e < dv) S[i][e] = Sg[(size_t)kk * dv + c + e];
      }
    }
  }
  const T* q = reinterpret_cast<const T*>(a.q) + (size_t)h * dk;
  const T* k = reinterpret_cast<const T*>(a.k) + (size_t)h * dk;
  const T* v = reinterpret_cast<const T*>(a.v) + (size_t)h * dv;
  const bool bonus = a.u != nullptr;
  if (bonus)
    for (int i = threadIdx.x; i < dk; i += 256) us[i] = __bfloat162float(a.u[(size_t)h * dk + i]);
  int par = 0;
  for (int base = r0; base < r1; base += tb) {
    const int nb = min(tb, r1 - base);
    __syncthreads();
    for (int i = threadIdx.x; i < nb * dk; i += 256) {
      const int t = i / dk, kk = i - t * dk;
      const size_t at = (size_t)(base + t) * a.stride + kk;
      qs[i] = ldf(q + at) * a.q_scale;
      ks[i] = ldf(k + at);
      as[i] = a.alpha[(size_t)(base + t) * a.H * dk + (size_t)h * dk + kk];
    }
    __syncthreads();
    for (int t = 0; t < nb; ++t, par ^= 1) {
      float vv[V], o[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        vv[e] = c + e < dv ? ldf(v + (size_t)(base + t) * a.stride + c + e) : 0.f;
        o[e] = 0.f;
      }
#pragma unroll
      for (int i = 0; i < RK; ++i) {
        const int kk = i * 8 + warp;
        if (kk >= dk) continue;
        const float qk = qs[t * dk + kk], kv = ks[t * dk + kk], al = as[t * dk + kk];
        const float b = bonus ? us[kk] * kv : 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          if (bonus) o[e] += qk * (S[i][e] + b * vv[e]);
          S[i][e] = al * S[i][e] + kv * vv[e];
          if (!bonus) o[e] += qk * S[i][e];
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) part[par][warp][lane * V + e] = o[e];
      __syncthreads();      // the next token writes the other half of `part`
      if (warp == (t & 7)) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          o[e] = 0.f;
#pragma unroll
          for (int w = 0; w < 8; ++w) o[e] += part[par][w][lane * V + e];
          ss += o[e] * o[e];
        }
        const int row = base + t;
        if (a.fused) {
          const float inv = a.out_scale / sqrtf(warp_sum(ss) / (float)dv + a.eps);
          const T* g = reinterpret_cast<const T*>(a.gate) + (size_t)row * a.stride + (size_t)h * dv;
          T* dst = reinterpret_cast<T*>(a.out) + (size_t)row * a.out_stride + (size_t)h * dv;
#pragma unroll
          for (int e = 0; e < V; ++e)
            if (c + e < dv) {
              const float gv = ldf(g + c + e);
              stf(dst + c + e, o[e] * inv * __bfloat162float(a.norm[(size_t)h * a.norm_step + c + e]) * (gv / (1.f + expf(-gv))));
            }
        } else {
          float* dst = reinterpret_cast<float*>(a.out) + ((size_t)row * a.H + h) * dv;
#pragma unroll
          for (int e = 0; e < V; ++e)
            if (c + e < dv) dst[c + e] = o[e];
        }
      }
    }
  }
  if (line > 0 && c < dv) {
#pragma unroll
    for (int i = 0; i < RK; ++i) {
      const int kk = i * 8 + warp;
      if (kk >= dk) continue;
      if (vec) {
        if constexpr (V == 4) *reinterpret_cast<float4*>(Sg + (size_t)kk * dv + c) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        else if constexpr (V == 2) *reinterpret_cast<float2*>(Sg + (size_t)kk * dv + c) = make_float2(S[i][0], S[i][1]);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e)
          if (c + e < dv) Sg[(size_t)kk * dv + c + e] = S[i][e];
      }
    }
  }
}

// ---- norm, weight, gate ------------------------------------------------------------------------------------------------
// A warp per (row, head); grid [rows, ceil(H / 8)].
template <typename T, int V>
KERN_DEVICE void norm_gate_body(const float* o, const T* gate, const __nv_bfloat16* norm, T* out, int H, int dv, int g_stride,
                                int norm_step, int out_stride, float out_scale, float eps) {
  const int row = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= H) return;
  const float* x = o + ((size_t)row * H + h) * dv;
  float ss = 0.f;
  for (int c = lane * V; c < dv; c += 32 * V) {
    const Vec<V> a = ldv<V>(x + c);
#pragma unroll
    for (int e = 0; e < V; ++e) ss += a.v[e] * a.v[e];
  }
  const float inv = out_scale / sqrtf(warp_sum(ss) / (float)dv + eps);
  for (int c = lane * V; c < dv; c += 32 * V) {
    const Vec<V> a = ldv<V>(x + c), w = ldv<V>(norm + (size_t)h * norm_step + c), g = ldv<V>(gate + (size_t)row * g_stride + (size_t)h * dv + c);
    Vec<V> r;
#pragma unroll
    for (int e = 0; e < V; ++e) r.v[e] = a.v[e] * inv * w.v[e] * (g.v[e] / (1.f + expf(-g.v[e])));
    stv<V>(out + (size_t)row * out_stride + (size_t)h * dv + c, r);
  }
}

KERN_DEVICE bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

// shift: grid [rows, any]; shift_state: grid [seqs, any]; decay: grid [ceil(n / 64), ceil(rows / 64)]; all block 256.
#define LIN_ENTRIES(T, SFX)                                                                                               \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_token_shift_##SFX(const T* h, const __nv_bfloat16* mu, T* out, uint8_t* state, const int* lines, const int* cu, \
                             int seqs, int width, int targets, long long line_bytes) {                                    \
    pdl_wait();                                                                                                           \
    if (width % 4 == 0) shift_body<T, 4>(h, mu, out, state, lines, cu, seqs, width, targets, line_bytes);                 \
    else shift_body<T, 1>(h, mu, out, state, lines, cu, seqs, width, targets, line_bytes);                                \
    pdl_launch_dependents();                                                                                              \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_shift_state_##SFX(const T* h, uint8_t* state, const int* lines, const int* cu, int seqs, int width,            \
                             long long line_bytes) {                                                                      \
    pdl_wait();                                                                                                           \
    shift_state_body<T>(h, state, lines, cu, seqs, width, line_bytes);                                                    \
    pdl_launch_dependents();                                                                                              \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256, 4)                                                                    \
      kern_decay_##SFX(const T* a, const __nv_bfloat16* W, const __nv_bfloat16* bias, float* alpha, int rows, int n,      \
                       int rank, int lda, int mode, float inv_tau) {                                                      \
    pdl_wait();                                                                                                           \
    decay_body<T>(a, W, bias, alpha, rows, n, rank, lda, mode, inv_tau);                                                  \
    pdl_launch_dependents();                                                                                              \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_lin_norm_gate_##SFX(const float* o, const T* gate, const __nv_bfloat16* norm, T* out, int H, int dv,           \
                               int g_stride, int norm_step, int out_stride, float out_scale, float eps) {                 \
    pdl_wait();                                                                                                           \
    if ((dv | g_stride | norm_step | out_stride) % 4 == 0 && aligned16(o) && aligned16(gate) && aligned16(norm) && aligned16(out)) \
      norm_gate_body<T, 4>(o, gate, norm, out, H, dv, g_stride, norm_step, out_stride, out_scale, eps);                   \
    else                                                                                                                  \
      norm_gate_body<T, 1>(o, gate, norm, out, H, dv, g_stride, norm_step, out_stride, out_scale, eps);                   \
    pdl_launch_dependents();                                                                                              \
  }
// rule: grid [H ceil(dv / (32 V)), seqs], block 256, (3 tb + 1) dk floats of shared memory; RK >= ceil(dk / 8)
#define LIN_RULE(T, SFX, RK, V)                                                                                           \
  extern "C" __global__ void __launch_bounds__(256, RK <= 8 ? (V <= 2 ? 5 : 3) : (RK == 16 ? 2 : 1))                      \
      kern_lin_rule_##SFX##_r##RK##_v##V(const T* q, const T* k, const T* v, const T* gate, const float* alpha,           \
                                         const __nv_bfloat16* u, const __nv_bfloat16* norm, void* out, uint8_t* state,    \
                                         const int* lines, const int* cu, int seqs, int H, int dk, int dv, int stride,    \
                                         int norm_step, int out_stride, long long line_bytes, int s_off, int fused,       \
                                         int tb, int max_rows, float q_scale, float out_scale, float eps) {               \
    pdl_wait();                                                                                                           \
    const RuleArgs a{q, k, v, gate, alpha, u, norm, out, state, lines, cu, seqs, H, dk, dv, stride, norm_step, out_stride, \
                     s_off, fused, tb, max_rows, line_bytes, q_scale, out_scale, eps};                                    \
    rule_body<T, RK, V>(a);                                                                                               \
    pdl_launch_dependents();                                                                                              \
  }
#define LIN_RULES(T, SFX)   \
  LIN_RULE(T, SFX, 4, 1)    \
  LIN_RULE(T, SFX, 4, 2)    \
  LIN_RULE(T, SFX, 4, 4)    \
  LIN_RULE(T, SFX, 8, 1)    \
  LIN_RULE(T, SFX, 8, 2)    \
  LIN_RULE(T, SFX, 8, 4)    \
  LIN_RULE(T, SFX, 16, 1)   \
  LIN_RULE(T, SFX, 16, 2)   \
  LIN_RULE(T, SFX, 16, 4)   \
  LIN_RULE(T, SFX, 32, 1)   \
  LIN_RULE(T, SFX, 32, 2)   \
  LIN_RULE(T, SFX, 32, 4)

LIN_ENTRIES(__nv_bfloat16, bf16)
LIN_ENTRIES(float, f32)
LIN_RULES(__nv_bfloat16, bf16)
LIN_RULES(float, f32)
