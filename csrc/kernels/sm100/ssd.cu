// build: precise
// Mamba-2 (state-space duality): the short causal convolution for any number of taps and channels, the recurrence, and
// the gated group norm behind it. One per-sequence state line per layer:
//     [conv window: (taps - 1) x channels, the activations' type][S: H x P x N f32]
// line 0 is the null line (padding rows use it and nothing is written to it).
//
// Per (sequence, head h of group g = h / (H / G)), per token:
//   dt' = softplus(dt + dt_bias[h]);  S = exp(-exp(A_log[h]) dt') S + dt' x B^T;  y = S C + D[h] x
// Everything inside the recurrence is f32; x, B, C and dt come from the projection and the convolution as activations.
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

template <typename T>
KERN_DEVICE void conv_body(const T* x, T* y, const uint8_t* state, const int* lines, const int* cu, const __nv_bfloat16* w,
                           const __nv_bfloat16* bias, int seqs, int rows, int channels, int taps, int x_stride,
                           long long line_bytes) {
  const int r = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  const int total = cu ? min(rows, cu[seqs]) : min(rows, seqs);
  if (r >= total || c >= channels) return;
  const int s = cu ? seq_of_row(cu, seqs, r) : r, r0 = cu ? cu[s] : s;
  const int line = checked_line(state, lines[s], line_bytes);
  const T* win = reinterpret_cast<const T*>(state + (size_t)line * line_bytes);
  float acc = __bfloat162float(bias[c]);
  for (int j = 0; j < taps; ++j) {
    const int rr = r - (taps - 1) + j;
    float v = 0.f;
    if (rr >= r0) v = ldf(x + (size_t)rr * x_stride + c);
    else if (line > 0) v = ldf(win + (size_t)(taps - 1 + rr - r0) * channels + c);
    acc += __bfloat162float(w[(size_t)c * taps + j]) * v;
  }
  stf(y + (size_t)r * channels + c, acc / (1.f + expf(-acc)));
}

template <typename T>
KERN_DEVICE void conv_state_body(const T* x, uint8_t* state, const int* lines, const int* cu, int seqs, int channels, int taps,
                                 int x_stride, long long line_bytes) {
  const int s = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  if (s >= seqs || c >= channels) return;
  const int line = checked_line(state, lines[s], line_bytes);
  const int r0 = cu ? cu[s] : s, n = (cu ? cu[s + 1] : s + 1) - r0, keep = taps - 1;
  if (line <= 0 || n <= 0) return;
  T* win = reinterpret_cast<T*>(state + (size_t)line * line_bytes);
  // ascending: row j takes old row j + n, which no earlier j has overwritten
  for (int j = 0; j < keep; ++j) {
    const int src = n + j - keep;
    win[(size_t)j * channels + c] = src >= 0 ? x[(size_t)(r0 + src) * x_stride + c] : win[(size_t)(j + n) * channels + c];
  }
}

KERN_DEVICE float softplus(float v) { return v > 30.f ? v : log1pf(expf(v)); }

// A warp keeps two rows of S (two values p of one head) in registers, lane l the columns n = 32 i + l; a block of eight
// warps is sixteen rows. Tokens are staged `tb` at a time in shared memory.
template <typename T, int NL>
KERN_DEVICE void rule_body(const T* xbc, const T* dt, float* y, uint8_t* state, const int* lines, const int* cu,
                           const __nv_bfloat16* A_log, const __nv_bfloat16* dt_bias, const __nv_bfloat16* D, int seqs, int H,
                           int P, int N, int G, int dt_stride, long long line_bytes, int s_off, int tb, int max_rows) {
  extern __shared__ __align__(16) float ssd_sm[];
  const int parts = (P + 15) / 16;
  const int h = blockIdx.x / parts, p0 = (blockIdx.x % parts) * 16, s = blockIdx.y;
  if (s >= seqs) return;
  const int line = checked_line(state, lines[s], line_bytes);
  const int r0 = cu ? cu[s] : s, r1 = cu ? cu[s + 1] : s + 1;
  if (r1 <= r0 || r1 - r0 > max_rows) return;      // longer sequences belong to ssd_chunk.cu
  float* Bs = ssd_sm;
  float* Cs = Bs + (size_t)tb * N;
  float* xs = Cs + (size_t)tb * N;
  float* ms = xs + (size_t)tb * 16;          // [tb] decays, then [tb] steps
  const int inner = H * P, channels = inner + 2 * G * N, g = h / (H / G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pa = p0 + warp * 2, pb = pa + 1;
  float* Sg = reinterpret_cast<float*>(state + (size_t)line * line_bytes + s_off) + (size_t)h * P * N;
  float Sa[NL], Sb[NL];
#pragma unroll
  for (int i = 0; i < NL; ++i) {
    const int n = i * 32 + lane;
    Sa[i] = (line > 0 && n < N && pa < P) ? Sg[(size_t)pa * N + n] : 0.f;
    Sb[i] = (line > 0 && n < N && pb < P) ? Sg[(size_t)pb * N + n] : 0.f;
  }
  const float a = -expf(__bfloat162float(A_log[h])), bias = __bfloat162float(dt_bias[h]), skip = __bfloat162float(D[h]);
  for (int base = r0; base < r1; base += tb) {
    const int nb = min(tb, r1 - base);
    __syncthreads();
    for (int i = threadIdx.x; i < nb * N; i += 256) {
      const int t = i / N, n = i % N;
      const T* row = xbc + (size_t)(base + t) * channels + inner + g * N + n;
      Bs[i] = ldf(row);
      Cs[i] = ldf(row + G * N);
    }
    for (int i = threadIdx.x; i < nb * 16; i += 256) {
      const int t = i / 16, p = p0 + i % 16;
      xs[i] = p < P ? ldf(xbc + (size_t)(base + t) * channels + h * P + p) : 0.f;
    }
    for (int t = threadIdx.x; t < nb; t += 256) {
      const float d = softplus(ldf(dt + (size_t)(base + t) * dt_stride + h) + bias);
      ms[t] = expf(a * d);
      ms[tb + t] = d;
    }
    __syncthreads();
#pragma unroll 4
    for (int t = 0; t < nb; ++t) {
      const float decay = ms[t], step = ms[tb + t];
      const float xa = xs[t * 16 + warp * 2], xb = xs[t * 16 + warp * 2 + 1];
      const float da = step * xa, db = step * xb;
      float ya = 0.f, yb = 0.f;
#pragma unroll
      for (int i = 0; i < NL; ++i) {
        const int n = i * 32 + lane;
        const float b = n < N ? Bs[t * N + n] : 0.f, c = n < N ? Cs[t * N + n] : 0.f;
        Sa[i] = decay * Sa[i] + da * b;
        Sb[i] = decay * Sb[i] + db * b;
        ya += Sa[i] * c;
        yb += Sb[i] * c;
      }
      ya = warp_sum(ya);
      yb = warp_sum(yb);
      float* yr = y + (size_t)(base + t) * inner + h * P;
      if (lane == 0 && pa < P) yr[pa] = ya + skip * xa;
      if (lane == 1 && pb < P) yr[pb] = yb + skip * xb;
    }
  }
  if (line > 0) {
#pragma unroll
    for (int i = 0; i < NL; ++i) {
      const int n = i * 32 + lane;
      if (n < N && pa < P) Sg[(size_t)pa * N + n] = Sa[i];
      if (n < N && pb < P) Sg[(size_t)pb * N + n] = Sb[i];
    }
  }
}

template <typename T, int V>
KERN_DEVICE void gate_norm_body(const float* y, const T* z, const __nv_bfloat16* w, T* out, int inner, int parts, int z_stride,
                                float eps) {
  extern __shared__ __align__(16) float ssd_sm[];
  __shared__ float part[8];
  const int t = blockIdx.x, width = inner / parts, c0 = blockIdx.y * width, warps = blockDim.x >> 5;
  const float* yr = y + (size_t)t * inner + c0;
  const T* zr = z + (size_t)t * z_stride + c0;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    const Vec<V> g = ldv<V>(zr + i);
    Vec<V> v = ldv<V>(yr + i);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      v.v[e] *= g.v[e] / (1.f + expf(-g.v[e]));
      ss += v.v[e] * v.v[e];
    }
    stv<V>(ssd_sm + i, v);
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < warps; ++i) ss += part[i];
  const float inv = 1.f / sqrtf(ss / (float)width + eps);
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    const Vec<V> v = ldv<V>(ssd_sm + i), g = ldv<V>(w + c0 + i);
    Vec<V> o;
#pragma unroll
    for (int e = 0; e < V; ++e) o.v[e] = v.v[e] * inv * g.v[e];
    stv<V>(out + (size_t)t * inner + c0 + i, o);
  }
}

}  // namespace

#define SSD_RULE(T, SFX, NL)                                                                                               \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_ssd_rule_##SFX##_n##NL(const T* xbc, const T* dt, float* y, uint8_t* state, const int* lines, const int* cu,    \
                                  const __nv_bfloat16* A_log, const __nv_bfloat16* dt_bias, const __nv_bfloat16* D,        \
                                  int seqs, int H, int P, int N, int G, int dt_stride, long long line_bytes, int s_off,    \
                                  int tb, int max_rows) {                                                                  \
    pdl_wait();                                                                                                            \
    rule_body<T, NL / 32>(xbc, dt, y, state, lines, cu, A_log, dt_bias, D, seqs, H, P, N, G, dt_stride, line_bytes, s_off, \
                          tb, max_rows);                                                                                   \
    pdl_launch_dependents();                                                                                               \
  }
// conv: grid [rows, ceil(channels / 256)]; conv_state: grid [seqs, ceil(channels / 256)]; rule: grid [H ceil(P / 16), seqs];
// gate_norm: grid [tokens, parts], block a multiple of 32 up to 256; block 256 elsewhere.
#define SSD_ENTRIES(T, SFX)                                                                                                \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_ssd_conv_##SFX(const T* x, T* y, const uint8_t* state, const int* lines, const int* cu, const __nv_bfloat16* w, \
                          const __nv_bfloat16* bias, int seqs, int rows, int channels, int taps, int x_stride,             \
                          long long line_bytes) {                                                                          \
    pdl_wait();                                                                                                            \
    conv_body<T>(x, y, state, lines, cu, w, bias, seqs, rows, channels, taps, x_stride, line_bytes);                       \
  }                                                                                                                        \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_ssd_conv_state_##SFX(const T* x, uint8_t* state, const int* lines, const int* cu, int seqs, int channels,       \
                                int taps, int x_stride, long long line_bytes) {                                            \
    pdl_wait();                                                                                                            \
    conv_state_body<T>(x, state, lines, cu, seqs, channels, taps, x_stride, line_bytes);                                   \
  }                                                                                                                        \
  SSD_RULE(T, SFX, 32)                                                                                                     \
  SSD_RULE(T, SFX, 64)                                                                                                     \
  SSD_RULE(T, SFX, 128)                                                                                                    \
  SSD_RULE(T, SFX, 256)                                                                                                    \
  SSD_RULE(T, SFX, 512)                                                                                                    \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_ssd_gate_norm_##SFX(const float* y, const T* z, const __nv_bfloat16* w, T* out, int inner, int parts,           \
                               int z_stride, float eps) {                                                                  \
    pdl_wait();                                                                                                            \
    if ((inner / parts | z_stride) % 4 == 0 && (reinterpret_cast<uintptr_t>(z) & 15) == 0)                                 \
      gate_norm_body<T, 4>(y, z, w, out, inner, parts, z_stride, eps);                                                     \
    else                                                                                                                   \
      gate_norm_body<T, 1>(y, z, w, out, inner, parts, z_stride, eps);                                                     \
    pdl_launch_dependents();                                                                                               \
  }

SSD_ENTRIES(__nv_bfloat16, bf16)
SSD_ENTRIES(float, f32)
