// build: precise
// The residual of a decoder that norms a sublayer's result before adding it as well as the next sublayer's input:
//     x <- x + rms(y) w_post;   xn = rms(x) w_next
// x is f32 (one row per token), y the sublayer's result: a row of a plain buffer, or the weighted sum of a token's k
// expert rows, summed here. Without `w_post` y is added as it is. A gated result is first multiplied, element by element, by
// sigmoid(gate + gate_b). Where the next sublayer reads its input plus a short convolution of it over time, one row per sequence
// (decode) is convolved here too (prompts: conv_add.cu).
// or, in a decoder that only scales a sublayer's result, element by element:
//     x <- x + s (y + bias + w_id h + sigmoid(gate) shared);   xn = rms(x) w_next
// where h is the sublayer's own input, w_id the weight of the experts that hand it back, and `shared` an expert for every token.
// kern_resid_embed  token row, times a factor, into x, and the first sublayer's normed input; kern_resid_embed_conv also convolves it
// kern_resid_scale  the second form; kern_resid_mix the first, kern_resid_gate the first with a gate, kern_resid_gate_conv that and
// the next input convolved; with `hidden` the sum goes there instead and nothing is normed (the last sublayer)
// Residual, sums and norms are f32; activations are T (bf16, or f32 in the 32-bit form of a model).
#include "act.cuh"

using namespace kern;

namespace {

KERN_DEVICE float block_sum(float v) {      // block of 256
  __shared__ float part[8];
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) s += part[i];
  __syncthreads();
  return s;
}

KERN_DEVICE float inv_rms(float ss, int width, float eps) { return 1.f / sqrtf(block_sum(ss) / (float)width + eps); }

// u (shared, each thread reads what it wrote) -> xn = u inv w
template <typename T, int V>
KERN_DEVICE void norm_out(const float* u, float inv, const __nv_bfloat16* w, T* xn, int width) {
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    const Vec<V> a = ldv<V>(u + i), b = ldv<V>(w + i);
    Vec<V> o;
#pragma unroll
    for (int e = 0; e < V; ++e) o.v[e] = a.v[e] * inv * b.v[e];
    stv<V>(xn + i, o);
  }
}

// what a later pass over the row reads, on its way from memory while the first sums are made
KERN_DEVICE void fetch(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// out = h + conv(h) of one row per sequence, conv_t = sum_j w[c][j] h_(t - taps + 1 + j). `state` holds lines of the last
// taps - 1 rows, which move on by one; line 0 is nobody's (zeros, and nothing is kept).
template <typename T>
struct ConvStep {
  const __nv_bfloat16* w = nullptr;
  T* out = nullptr;
  uint8_t* state = nullptr;
  const int* lines = nullptr;
  int taps = 0;
  long long line_bytes = 0;
};

// columns i .. of row t; h as the activations' type holds it
template <typename T, int V>
KERN_DEVICE void conv_step(const ConvStep<T>& cv, int line, int t, int i, const Vec<V>& h, int width) {
  const int keep = cv.taps - 1;
  T* win = reinterpret_cast<T*>(cv.state + (size_t)line * cv.line_bytes) + i;
  const __nv_bfloat16* w = cv.w + (size_t)i * cv.taps;
  Vec<V> acc = h;
#pragma unroll
  for (int e = 0; e < V; ++e) acc.v[e] += __bfloat162float(w[e * cv.taps + keep]) * h.v[e];
  if (line > 0) {
    Vec<V> past[3];      // the usual few taps: all rows in flight at once
    const int few = min(keep, 3);
#pragma unroll
    for (int j = 0; j < 3; ++j)
      if (j < few) past[j] = ldv<V>(win + (size_t)j * width);
#pragma unroll
    for (int j = 0; j < 3; ++j) {
      if (j >= few) continue;
#pragma unroll
      for (int e = 0; e < V; ++e) acc.v[e] += __bfloat162float(w[e * cv.taps + j]) * past[j].v[e];
      if (j > 0) stv<V>(win + (size_t)(j - 1) * width, past[j]);
    }
    for (int j = 3; j < keep; ++j) {
      const Vec<V> v = ldv<V>(win + (size_t)j * width);
#pragma unroll
      for (int e = 0; e < V; ++e) acc.v[e] += __bfloat162float(w[e * cv.taps + j]) * v.v[e];
      stv<V>(win + (size_t)(j - 1) * width, v);
    }
    if (keep > 0) stv<V>(win + (size_t)(keep - 1) * width, h);
  }
  stv<V>(cv.out + (size_t)t * width + i, acc);
}

template <typename T>
KERN_DEVICE int conv_line(const ConvStep<T>& cv, int t) {
  const int line = cv.lines[t];
  return line > 0 && KERN_CHECK(cv.state + (size_t)line * cv.line_bytes, (size_t)cv.line_bytes, SITE_STATE_SLOT) ? line : 0;
}

// the row's past and the norm's and the convolution's weights, 128 bytes a thread and step
template <typename T>
KERN_DEVICE void fetch_conv(const ConvStep<T>& cv, const __nv_bfloat16* w_post, const __nv_bfloat16* w_next, int width) {
  const int line = conv_line(cv, blockIdx.x), step = threadIdx.x * 128;
  auto span = [&](const void* p, int bytes) {
    for (int i = step; i < bytes; i += 256 * 128) fetch(reinterpret_cast<const uint8_t*>(p) + i);
  };
  span(cv.w, width * cv.taps * 2);
  span(w_next, width * 2);
  if (w_post) span(w_post, width * 2);
  if (line > 0) span(cv.state + (size_t)line * cv.line_bytes, (cv.taps - 1) * width * (int)sizeof(T));
}

// As norm_out, and the row's convolution
template <typename T, int V>
KERN_DEVICE void norm_conv_out(const float* u, float inv, const __nv_bfloat16* w, T* xn, const ConvStep<T>& cv, int width) {
  const int t = blockIdx.x, line = conv_line(cv, t);
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    const Vec<V> a = ldv<V>(u + i), b = ldv<V>(w + i);
    T held[V];
    Vec<V> o;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      stf(held + e, a.v[e] * inv * b.v[e]);
      o.v[e] = ldf(held + e);
    }
    stv<V>(xn + i, o);
    conv_step<T, V>(cv, line, t, i, o, width);
  }
}

template <typename T, int V, bool CONV>
KERN_DEVICE void embed_body(const long long* ids, const __nv_bfloat16* table, const __nv_bfloat16* w_norm, float* x, T* xn,
                            int width, int vocab, float scale, float eps, int* err, const ConvStep<T>& cv) {
  extern __shared__ __align__(16) float resid_sm[];
  const int t = blockIdx.x;
  long long id = ids[t];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) set_error(err, ERR_BOUNDS);
    id = 0;
  }
  if constexpr (CONV) fetch_conv(cv, nullptr, w_norm, width);
  const __nv_bfloat16* a = table + (size_t)id * width;
  const bool ok = KERN_CHECK(a, (size_t)width * 2, SITE_EMBED_ROW);
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    Vec<V> v = {};
    if (ok) v = ldv<V>(a + i);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      v.v[j] *= scale;
      ss += v.v[j] * v.v[j];
    }
    stv<V>(x + (size_t)t * width + i, v);
    stv<V>(resid_sm + i, v);
  }
  const float inv = inv_rms(ss, width, eps);
  if constexpr (CONV) norm_conv_out<T, V>(resid_sm, inv, w_norm, xn + (size_t)t * width, cv, width);
  else norm_out<T, V>(resid_sm, inv, w_norm, xn + (size_t)t * width, width);
}

template <typename T, int V, bool GATED, bool CONV>
KERN_DEVICE void mix_body(float* x, const T* y, const int* perm, const float* topw, const T* gate, const __nv_bfloat16* gate_b,
                          const __nv_bfloat16* w_post, const __nv_bfloat16* w_next, T* xn, float* hidden, int width, int k,
                          float eps, const ConvStep<T>& cv) {
  extern __shared__ __align__(16) float resid_sm[];
  __shared__ float tw[32];
  __shared__ int tr[32];
  const int t = blockIdx.x;
  if constexpr (CONV) fetch_conv(cv, w_post, w_next, width);
  if (perm) {
    if (threadIdx.x < k) {
      const int r = perm[(size_t)t * k + threadIdx.x];
      const bool ok = r >= 0 && KERN_CHECK(y + (size_t)r * width, (size_t)width * sizeof(T), SITE_MOE_COMBINE);
      tr[threadIdx.x] = ok ? r : -1;
      tw[threadIdx.x] = topw[(size_t)t * k + threadIdx.x];
    }
    __syncthreads();
  }
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    Vec<V> v = {};
    if (perm) {
      for (int j = 0; j < k; ++j) {
        if (tr[j] < 0) continue;
        const Vec<V> r = ldv<V>(y + (size_t)tr[j] * width + i);
#pragma unroll
        for (int e = 0; e < V; ++e) v.v[e] += tw[j] * r.v[e];
      }
    } else {
      v = ldv<V>(y + (size_t)t * width + i);
    }
    if constexpr (GATED) {
      const Vec<V> g = ldv<V>(gate + (size_t)t * width + i), b = ldv<V>(gate_b + i);
#pragma unroll
      for (int e = 0; e < V; ++e) v.v[e] /= 1.f + expf(-(g.v[e] + b.v[e]));
    }
#pragma unroll
    for (int e = 0; e < V; ++e) ss += v.v[e] * v.v[e];
    stv<V>(resid_sm + i, v);
  }
  const float inv = w_post ? inv_rms(ss, width, eps) : 1.f;
  float* xt = x + (size_t)t * width;
  ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    const Vec<V> v = ldv<V>(resid_sm + i);
    Vec<V> s = ldv<V>(xt + i), w;
    if (w_post) w = ldv<V>(w_post + i);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      s.v[e] += w_post ? v.v[e] * inv * w.v[e] : v.v[e];
      ss += s.v[e] * s.v[e];
    }
    if (hidden) {
      stv<V>(hidden + (size_t)t * width + i, s);
    } else {
      stv<V>(xt + i, s);
      stv<V>(resid_sm + i, s);
    }
  }
  if (hidden) return;
  const float next = inv_rms(ss, width, eps);
  if constexpr (CONV) norm_conv_out<T, V>(resid_sm, next, w_next, xn + (size_t)t * width, cv, width);
  else norm_out<T, V>(resid_sm, next, w_next, xn + (size_t)t * width, width);
}

// A sublayer's result: y, or with `perm` the weighted sum of a token's expert rows; choices without a row (perm < 0) are the
// experts that hand back the input, xn as it is on entry. `shared` [rows][width] is weighed by sigmoid(gate[t gate_stride]).
template <typename T, int V, bool ROUTED>
KERN_DEVICE void scale_body(float* x, const T* y, const int* perm, const float* topw, const T* shared, const float* gate,
                            const __nv_bfloat16* bias, const __nv_bfloat16* scale, const __nv_bfloat16* w_next, T* xn, float* hidden,
                            int width, int k, int gate_stride, float eps) {
  extern __shared__ __align__(16) float resid_sm[];
  __shared__ float tw[32];
  __shared__ int tr[32], n_rows;
  __shared__ float own_w;
  const int t = blockIdx.x;
  float self = 0.f;
  if constexpr (ROUTED) {
    if (threadIdx.x < 32) {      // the choices with a row to the front, then nothing
      const int j = threadIdx.x;
      int r = j < k ? perm[(size_t)t * k + j] : -1;
      const float w = j < k ? topw[(size_t)t * k + j] : 0.f;
      if (r >= 0 && !KERN_CHECK(y + (size_t)r * width, (size_t)width * sizeof(T), SITE_MOE_COMBINE)) r = -1;
      const unsigned have = __ballot_sync(0xffffffffu, r >= 0);
      if (r >= 0) { tr[__popc(have & ((1u << j) - 1))] = r; tw[__popc(have & ((1u << j) - 1))] = w; }
      const float own = warp_sum(r < 0 ? w : 0.f);
      if (j == 0) { n_rows = __popc(have); own_w = own; }
    }
    __syncthreads();
    self = own_w;
  }
  const float g = shared ? 1.f / (1.f + expf(-gate[(size_t)t * gate_stride])) : 0.f;
  float* xt = x + (size_t)t * width;
  T* xnt = xn + (size_t)t * width;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    Vec<V> v = {};
    if constexpr (ROUTED) {
      const int n = n_rows;
      int j = 0;
      for (; j + 4 <= n; j += 4) {      // four rows in flight
        const RawOf<T, V> r0 = raw<V>(y + (size_t)tr[j] * width + i), r1 = raw<V>(y + (size_t)tr[j + 1] * width + i),
                          r2 = raw<V>(y + (size_t)tr[j + 2] * width + i), r3 = raw<V>(y + (size_t)tr[j + 3] * width + i);
        add(v, r0, tw[j]); add(v, r1, tw[j + 1]); add(v, r2, tw[j + 2]); add(v, r3, tw[j + 3]);
      }
      for (; j < n; ++j) add(v, raw<V>(y + (size_t)tr[j] * width + i), tw[j]);
      if (self != 0.f) add(v, raw<V>(xnt + i), self);
    } else {
      v = ldv<V>(y + (size_t)t * width + i);
    }
    if (shared) {
      add(v, raw<V>(shared + (size_t)t * width + i), g);
    }
    if (bias) {
      const Vec<V> r = ldv<V>(bias + i);
#pragma unroll
      for (int e = 0; e < V; ++e) v.v[e] += r.v[e];
    }
    Vec<V> s = ldv<V>(xt + i);
    const Vec<V> w = ldv<V>(scale + i);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      s.v[e] += v.v[e] * w.v[e];
      ss += s.v[e] * s.v[e];
    }
    if (hidden) {
      stv<V>(hidden + (size_t)t * width + i, s);
    } else {
      stv<V>(xt + i, s);
      stv<V>(resid_sm + i, s);
    }
  }
  if (!hidden) norm_out<T, V>(resid_sm, inv_rms(ss, width, eps), w_next, xnt, width);
}

}  // namespace

// grid = rows, block 256, `width` floats of shared memory
#define RESID_WIDTHS(call4, call1)                                                                                        \
  pdl_wait();                                                                                                             \
  if (width % 4 == 0) call4; else call1;                                                                                  \
  pdl_launch_dependents();
#define RESID_ENTRIES(T, SFX)                                                                                             \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_resid_embed_##SFX(const long long* ids, const __nv_bfloat16* table, const __nv_bfloat16* w_norm, float* x,     \
                             T* xn, int width, int vocab, float scale, float eps, int* err) {                             \
    RESID_WIDTHS((embed_body<T, 4, false>(ids, table, w_norm, x, xn, width, vocab, scale, eps, err, {})),                 \
                 (embed_body<T, 1, false>(ids, table, w_norm, x, xn, width, vocab, scale, eps, err, {})))                 \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_resid_embed_conv_##SFX(const long long* ids, const __nv_bfloat16* table, const __nv_bfloat16* w_norm,          \
                                  float* x, T* xn, int width, int vocab, float scale, float eps, int* err,                \
                                  const __nv_bfloat16* conv_w, T* conv_out, uint8_t* state, const int* lines, int taps,   \
                                  long long line_bytes) {                                                                 \
    const ConvStep<T> cv{conv_w, conv_out, state, lines, taps, line_bytes};                                               \
    RESID_WIDTHS((embed_body<T, 4, true>(ids, table, w_norm, x, xn, width, vocab, scale, eps, err, cv)),                  \
                 (embed_body<T, 1, true>(ids, table, w_norm, x, xn, width, vocab, scale, eps, err, cv)))                  \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_resid_mix_##SFX(float* x, const T* y, const int* perm, const float* topw, const __nv_bfloat16* w_post,         \
                           const __nv_bfloat16* w_next, T* xn, float* hidden, int width, int k, float eps) {              \
    RESID_WIDTHS((mix_body<T, 4, false, false>(x, y, perm, topw, nullptr, nullptr, w_post, w_next, xn, hidden, width, k, eps, {})), \
                 (mix_body<T, 1, false, false>(x, y, perm, topw, nullptr, nullptr, w_post, w_next, xn, hidden, width, k, eps, {}))) \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_resid_gate_##SFX(float* x, const T* y, const int* perm, const float* topw, const __nv_bfloat16* w_post,        \
                            const __nv_bfloat16* w_next, T* xn, float* hidden, int width, int k, float eps,               \
                            const T* gate, const __nv_bfloat16* gate_b) {                                                 \
    RESID_WIDTHS((mix_body<T, 4, true, false>(x, y, perm, topw, gate, gate_b, w_post, w_next, xn, hidden, width, k, eps, {})), \
                 (mix_body<T, 1, true, false>(x, y, perm, topw, gate, gate_b, w_post, w_next, xn, hidden, width, k, eps, {}))) \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_resid_gate_conv_##SFX(float* x, const T* y, const int* perm, const float* topw, const __nv_bfloat16* w_post,   \
                                 const __nv_bfloat16* w_next, T* xn, int width, int k, float eps, const T* gate,          \
                                 const __nv_bfloat16* gate_b, const __nv_bfloat16* conv_w, T* conv_out, uint8_t* state,   \
                                 const int* lines, int taps, long long line_bytes) {                                      \
    const ConvStep<T> cv{conv_w, conv_out, state, lines, taps, line_bytes};                                               \
    RESID_WIDTHS((mix_body<T, 4, true, true>(x, y, perm, topw, gate, gate_b, w_post, w_next, xn, nullptr, width, k, eps, cv)), \
                 (mix_body<T, 1, true, true>(x, y, perm, topw, gate, gate_b, w_post, w_next, xn, nullptr, width, k, eps, cv))) \
  }

RESID_ENTRIES(__nv_bfloat16, bf16)
RESID_ENTRIES(float, f32)

// the routed form has an entry of its own: its rows in flight would cost the plain one registers
#define RESID_SCALE(NAME, T, ROUTED)                                                                                      \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      NAME(float* x, const T* y, const int* perm, const float* topw, const T* shared, const float* gate,                  \
           const __nv_bfloat16* bias, const __nv_bfloat16* scale, const __nv_bfloat16* w_next, T* xn, float* hidden,      \
           int width, int k, int gate_stride, float eps) {                                                                \
    pdl_wait();                                                                                                           \
    if (width % 4 == 0)                                                                                                   \
      scale_body<T, 4, ROUTED>(x, y, perm, topw, shared, gate, bias, scale, w_next, xn, hidden, width, k, gate_stride, eps); \
    else                                                                                                                  \
      scale_body<T, 1, ROUTED>(x, y, perm, topw, shared, gate, bias, scale, w_next, xn, hidden, width, k, gate_stride, eps); \
    pdl_launch_dependents();                                                                                              \
  }
RESID_SCALE(kern_resid_scale_bf16, __nv_bfloat16, false)
RESID_SCALE(kern_resid_scale_f32, float, false)
RESID_SCALE(kern_resid_scale_routed_bf16, __nv_bfloat16, true)
RESID_SCALE(kern_resid_scale_routed_f32, float, true)
