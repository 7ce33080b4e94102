// build: precise
// Hyper-connections: a token's residual is `streams` f32 rows instead of one. A sublayer reads one weighted sum of
// them (u = sum_s in[s] x_s, then an RMS norm) and writes back into all of them at once:
//     x_t <- sum_s mix[s, t] x_s + out[t] y          (mix is indexed [from, to]; the right side uses the old streams)
// kern_hyper_embed  token row + position row, RMS norm, copied into every stream, and the first sublayer's input
// kern_hyper_mix    one sublayer's result into the streams and the next sublayer's normed input, in one pass over the
//                   residual; y may be a row of a plain buffer or the weighted sum of a token's k expert rows
// kern_hyper_last   the last sublayer: only the sum of the new streams is wanted
// kern_row_norm_f32 RMS norm of picked f32 rows (the last row of every sequence, or rows named by the host)
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

// u (shared, `width` floats, each thread reads what it wrote) -> xn = u / rms(u) * w
template <typename T, int V>
KERN_DEVICE void norm_out(const float* u, float ss, const __nv_bfloat16* w, T* xn, int width, float eps) {
  const float inv = 1.f / sqrtf(block_sum(ss) / (float)width + eps);
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    const Vec<V> a = ldv<V>(u + i), b = ldv<V>(w + i);
    Vec<V> o;
#pragma unroll
    for (int e = 0; e < V; ++e) o.v[e] = a.v[e] * inv * b.v[e];
    stv<V>(xn + i, o);
  }
}

template <typename T, int V>
KERN_DEVICE void embed_body(const long long* ids, const long long* positions, const __nv_bfloat16* table,
                            const __nv_bfloat16* pos_table, const __nv_bfloat16* w_embed, const __nv_bfloat16* w_in,
                            const __nv_bfloat16* w_norm, float* x, T* xn, int width, int streams, int vocab, int max_pos,
                            float eps, int* err) {
  extern __shared__ __align__(16) float hyper_sm[];
  float* e = hyper_sm;
  const int t = blockIdx.x;
  long long id = ids[t], pos = positions[t];
  if (id < 0 || id >= vocab || pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0) set_error(err, ERR_BOUNDS);
    if (id < 0 || id >= vocab) id = 0;
    if (pos < 0 || pos >= max_pos) pos = 0;
  }
  const __nv_bfloat16* a = table + (size_t)id * width;
  const __nv_bfloat16* b = pos_table + (size_t)pos * width;
  const bool ok = KERN_CHECK(a, (size_t)width * 2, SITE_EMBED_ROW) && KERN_CHECK(b, (size_t)width * 2, SITE_EMBED_ROW);
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    Vec<V> va = {}, vb = {};
    if (ok) { va = ldv<V>(a + i); vb = ldv<V>(b + i); }
#pragma unroll
    for (int j = 0; j < V; ++j) { va.v[j] += vb.v[j]; ss += va.v[j] * va.v[j]; }
    stv<V>(e + i, va);
  }
  float in_sum = 0.f;
  for (int s = 0; s < streams; ++s) in_sum += __bfloat162float(w_in[s]);
  const float inv = 1.f / sqrtf(block_sum(ss) / (float)width + eps);
  ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    Vec<V> v = ldv<V>(e + i);
    const Vec<V> w = ldv<V>(w_embed + i);
#pragma unroll
    for (int j = 0; j < V; ++j) v.v[j] = v.v[j] * inv * w.v[j];
    for (int s = 0; s < streams; ++s) stv<V>(x + ((size_t)t * streams + s) * width + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) { v.v[j] *= in_sum; ss += v.v[j] * v.v[j]; }
    stv<V>(e + i, v);
  }
  norm_out<T, V>(e, ss, w_norm, xn + (size_t)t * width, width, eps);
}

constexpr int MAX_STREAMS = 16;

// S: the number of streams when it is one of the compiled counts, else 0 (up to MAX_STREAMS, read from `streams`).
template <typename T, int V, int S>
KERN_DEVICE void mix_body(float* x, const T* y, const int* perm, const float* topw, const __nv_bfloat16* w_mix,
                          const __nv_bfloat16* w_out, const __nv_bfloat16* w_in, const __nv_bfloat16* w_norm, T* xn,
                          float* hidden, int width, int streams, int k, float eps) {
  extern __shared__ __align__(16) float hyper_sm[];
  __shared__ float mix[MAX_STREAMS * MAX_STREAMS], out[MAX_STREAMS], in[MAX_STREAMS], tw[32];
  __shared__ int tr[32];
  constexpr int SM = S > 0 ? S : MAX_STREAMS;
  const int n = S > 0 ? S : streams;
  const int t = blockIdx.x;
  for (int i = threadIdx.x; i < n * n; i += 256) mix[i] = __bfloat162float(w_mix[i]);
  if (threadIdx.x < n) {
    out[threadIdx.x] = __bfloat162float(w_out[threadIdx.x]);
    in[threadIdx.x] = w_in ? __bfloat162float(w_in[threadIdx.x]) : 1.f;
  }
  if (perm && threadIdx.x < k) {
    const int r = perm[(size_t)t * k + threadIdx.x];
    const bool ok = r >= 0 && KERN_CHECK(y + (size_t)r * width, (size_t)width * sizeof(T), SITE_MOE_COMBINE);
    tr[threadIdx.x] = ok ? r : -1;
    tw[threadIdx.x] = topw[(size_t)t * k + threadIdx.x];
  }
  __syncthreads();
  float* xt = x + (size_t)t * n * width;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    Vec<V> xs[SM], yv = {};
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < n) xs[s] = ldv<V>(xt + (size_t)s * width + i);
    if (perm) {
      for (int j = 0; j < k; ++j) {
        if (tr[j] < 0) continue;
        const Vec<V> r = ldv<V>(y + (size_t)tr[j] * width + i);
#pragma unroll
        for (int e = 0; e < V; ++e) yv.v[e] += tw[j] * r.v[e];
      }
    } else {
      yv = ldv<V>(y + (size_t)t * width + i);
    }
    Vec<V> u = {};
#pragma unroll
    for (int o = 0; o < SM; ++o) {
      if (o >= n) continue;
      Vec<V> v;
#pragma unroll
      for (int e = 0; e < V; ++e) v.v[e] = out[o] * yv.v[e];
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < n) {
          const float m = mix[s * n + o];
#pragma unroll
          for (int e = 0; e < V; ++e) v.v[e] += m * xs[s].v[e];
        }
      if (!hidden) stv<V>(xt + (size_t)o * width + i, v);
#pragma unroll
      for (int e = 0; e < V; ++e) u.v[e] += in[o] * v.v[e];
    }
    if (hidden) {
      stv<V>(hidden + (size_t)t * width + i, u);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) ss += u.v[e] * u.v[e];
      stv<V>(hyper_sm + i, u);
    }
  }
  if (!hidden) norm_out<T, V>(hyper_sm, ss, w_norm, xn + (size_t)t * width, width, eps);
}

// any other stream count runs one column per thread: sixteen streams of four columns would not fit the registers
template <typename T, int S>
KERN_DEVICE void mix_any(float* x, const T* y, const int* perm, const float* topw, const __nv_bfloat16* w_mix,
                         const __nv_bfloat16* w_out, const __nv_bfloat16* w_in, const __nv_bfloat16* w_norm, T* xn,
                         float* hidden, int width, int streams, int k, float eps) {
  if constexpr (S > 0) {
    if (width % 4 == 0) {
      mix_body<T, 4, S>(x, y, perm, topw, w_mix, w_out, w_in, w_norm, xn, hidden, width, streams, k, eps);
      return;
    }
  }
  mix_body<T, 1, S>(x, y, perm, topw, w_mix, w_out, w_in, w_norm, xn, hidden, width, streams, k, eps);
}

template <typename T, int V>
KERN_DEVICE void row_norm_body(const float* src, const int* cu, const int* rows, const __nv_bfloat16* w, T* y, int src_rows,
                               int width, float eps) {
  extern __shared__ __align__(16) float hyper_sm[];
  const int r = blockIdx.x;
  int from = cu ? cu[r + 1] - 1 : (rows ? rows[r] : r);
  from = max(0, min(from, src_rows - 1));
  const float* x = src + (size_t)from * width;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += 256 * V) {
    const Vec<V> v = ldv<V>(x + i);
#pragma unroll
    for (int e = 0; e < V; ++e) ss += v.v[e] * v.v[e];
    stv<V>(hyper_sm + i, v);
  }
  norm_out<T, V>(hyper_sm, ss, w, y + (size_t)r * width, width, eps);
}

}  // namespace

// grid = rows, block 256, `width` floats of shared memory (none for kern_hyper_last)
#define HYPER_ENTRIES(T, SFX)                                                                                              \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_hyper_embed_##SFX(const long long* ids, const long long* positions, const __nv_bfloat16* table,                 \
                             const __nv_bfloat16* pos_table, const __nv_bfloat16* w_embed, const __nv_bfloat16* w_in,      \
                             const __nv_bfloat16* w_norm, float* x, T* xn, int width, int streams, int vocab, int max_pos, \
                             float eps, int* err) {                                                                        \
    pdl_wait();                                                                                                            \
    if (width % 4 == 0)                                                                                                    \
      embed_body<T, 4>(ids, positions, table, pos_table, w_embed, w_in, w_norm, x, xn, width, streams, vocab, max_pos,     \
                       eps, err);                                                                                          \
    else                                                                                                                   \
      embed_body<T, 1>(ids, positions, table, pos_table, w_embed, w_in, w_norm, x, xn, width, streams, vocab, max_pos,     \
                       eps, err);                                                                                          \
    pdl_launch_dependents();                                                                                               \
  }                                                                                                                        \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_row_norm_f32_##SFX(const float* src, const int* cu, const int* rows, const __nv_bfloat16* w, T* y,              \
                              int src_rows, int width, float eps) {                                                        \
    pdl_wait();                                                                                                            \
    if (width % 4 == 0) row_norm_body<T, 4>(src, cu, rows, w, y, src_rows, width, eps);                                    \
    else row_norm_body<T, 1>(src, cu, rows, w, y, src_rows, width, eps);                                                   \
    pdl_launch_dependents();                                                                                               \
  }
// one entry per compiled stream count; _s0 takes any count up to MAX_STREAMS
#define HYPER_MIX(T, SFX, S)                                                                                               \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_hyper_mix_##SFX##_s##S(float* x, const T* y, const int* perm, const float* topw, const __nv_bfloat16* w_mix,    \
                                  const __nv_bfloat16* w_out, const __nv_bfloat16* w_in, const __nv_bfloat16* w_norm,      \
                                  T* xn, int width, int streams, int k, float eps) {                                       \
    pdl_wait();                                                                                                            \
    mix_any<T, S>(x, y, perm, topw, w_mix, w_out, w_in, w_norm, xn, nullptr, width, streams, k, eps);                      \
    pdl_launch_dependents();                                                                                               \
  }                                                                                                                        \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_hyper_last_##SFX##_s##S(const float* x, const T* y, const int* perm, const float* topw,                         \
                                   const __nv_bfloat16* w_mix, const __nv_bfloat16* w_out, float* hidden, int width,       \
                                   int streams, int k) {                                                                   \
    pdl_wait();                                                                                                            \
    mix_any<T, S>(const_cast<float*>(x), y, perm, topw, w_mix, w_out, nullptr, nullptr, nullptr, hidden, width, streams,   \
                  k, 0.f);                                                                                                 \
    pdl_launch_dependents();                                                                                               \
  }

HYPER_ENTRIES(__nv_bfloat16, bf16)
HYPER_ENTRIES(float, f32)
HYPER_MIX(__nv_bfloat16, bf16, 0)
HYPER_MIX(__nv_bfloat16, bf16, 1)
HYPER_MIX(__nv_bfloat16, bf16, 2)
HYPER_MIX(__nv_bfloat16, bf16, 3)
HYPER_MIX(__nv_bfloat16, bf16, 4)
HYPER_MIX(float, f32, 0)
HYPER_MIX(float, f32, 1)
HYPER_MIX(float, f32, 2)
HYPER_MIX(float, f32, 3)
HYPER_MIX(float, f32, 4)
