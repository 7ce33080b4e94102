// build: precise
// A row plus a short causal convolution of it over time, channel by channel, for prompts and any ragged call:
//     out_t = h_t + sum_j w[c][j] h_(t - taps + 1 + j)      (zeros before a sequence's first row)
// The last taps - 1 rows of a sequence are its state line (the activations' type); line 0 is nobody's. One row per sequence
// (decode) is done by the kernel that makes h (resid.cu).
#include "act.cuh"

using namespace kern;

namespace {

constexpr int kRun = 4;      // rows a thread does

KERN_DEVICE int seq_of_row(const int* cu, int seqs, int r) {      // the last s with cu[s] <= r
  int lo = 0, hi = seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= r) lo = mid; else hi = mid - 1;
  }
  return lo;
}

KERN_DEVICE int checked_line(const uint8_t* state, int line, long long line_bytes) {
  return line > 0 && KERN_CHECK(state + (size_t)line * line_bytes, (size_t)line_bytes, SITE_STATE_SLOT) ? line : 0;
}

// grid [ceil(rows / 4), ceil(width / 256 V)]. KEEP > 0: taps - 1, known. Rows that reach back to the line, a sequence's first
// taps - 1, are all done by the threads whose run holds its first row; these then move the line on, so nobody sees it half-moved.
template <typename T, int V, int KEEP>
KERN_DEVICE void conv_body(const T* h, T* out, uint8_t* state, const int* lines, const int* cu, const __nv_bfloat16* w, int seqs,
                           int rows, int width, int taps, long long line_bytes) {
  const int c = (blockIdx.y * 256 + threadIdx.x) * V, keep = KEEP > 0 ? KEEP : taps - 1;
  const int ra = blockIdx.x * kRun, rb = min(min(rows, cu[seqs]), ra + kRun);
  if (c >= width || ra >= rb) return;
  int s = seq_of_row(cu, seqs, ra), r0 = cu[s], r1 = cu[s + 1];
  const T* hc = h + c;
  const __nv_bfloat16* wc = w + (size_t)c * taps;
  if constexpr (KEEP > 0) {
    if (rb - ra == kRun && ra - r0 >= KEEP && rb <= r1) {      // inside one sequence: every row in flight at once
      RawOf<T, V> x[KEEP + kRun];
#pragma unroll
      for (int j = 0; j < KEEP + kRun; ++j) x[j] = raw<V>(hc + (size_t)(ra - KEEP + j) * width);
      float wt[V][KEEP + 1];      // the taps of V neighbouring channels lie side by side
      static_assert(V == 4 && (KEEP + 1) % 4 == 0, "whole vectors of weights");
#pragma unroll
      for (int i = 0; i < V * (KEEP + 1); i += 4) {
        const Vec<4> v = ldv<4>(wc + i);
#pragma unroll
        for (int e = 0; e < 4; ++e) wt[(i + e) / (KEEP + 1)][(i + e) % (KEEP + 1)] = v.v[e];
      }
#pragma unroll
      for (int t = 0; t < kRun; ++t) {
        Vec<V> acc = {};
        add(acc, x[KEEP + t], 1.f);
#pragma unroll
        for (int j = 0; j <= KEEP; ++j) {
          const Vec<V> v = ldv<V>(reinterpret_cast<const T*>(&x[t + j]));
#pragma unroll
          for (int e = 0; e < V; ++e) acc.v[e] += wt[e][j] * v.v[e];
        }
        stv<V>(out + (size_t)(ra + t) * width + c, acc);
      }
      return;
    }
  }
  for (int r = ra; r < rb; ++r) {
    while (r >= r1) { ++s; r0 = cu[s]; r1 = cu[s + 1]; }      // empty sequences are skipped
    if (r - r0 >= keep) {
      Vec<V> acc = ldv<V>(hc + (size_t)r * width);
      for (int j = 0; j <= keep; ++j) {
        const Vec<V> v = ldv<V>(hc + (size_t)(r - keep + j) * width);
#pragma unroll
        for (int e = 0; e < V; ++e) acc.v[e] += __bfloat162float(wc[e * taps + j]) * v.v[e];
      }
      stv<V>(out + (size_t)r * width + c, acc);
    } else if (r == r0) {
      const int line = checked_line(state, lines[s], line_bytes), n = r1 - r0;
      T* win = reinterpret_cast<T*>(state + (size_t)line * line_bytes) + c;
      for (int q = 0; q < min(keep, n); ++q) {
        Vec<V> acc = ldv<V>(hc + (size_t)(r0 + q) * width);
        for (int j = 0; j <= keep; ++j) {
          const int at = q + j - keep;      // a row of this call, of the line, or nothing
          Vec<V> v = {};
          if (at >= 0) v = ldv<V>(hc + (size_t)(r0 + at) * width);
          else if (line > 0) v = ldv<V>(win + (size_t)(q + j) * width);
#pragma unroll
          for (int e = 0; e < V; ++e) acc.v[e] += __bfloat162float(wc[e * taps + j]) * v.v[e];
        }
        stv<V>(out + (size_t)(r0 + q) * width + c, acc);
      }
      for (int j = 0; line > 0 && j < keep; ++j) {      // ascending: row j takes old row j + n, which no earlier j has overwritten
        const int at = n + j - keep;
        stv<V>(win + (size_t)j * width, at >= 0 ? ldv<V>(hc + (size_t)(r0 + at) * width) : ldv<V>(win + (size_t)(j + n) * width));
      }
    }
  }
}

}  // namespace

#define CONV_ADD(T, SFX)                                                                                                  \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_conv_add_##SFX(const T* h, T* out, uint8_t* state, const int* lines, const int* cu, const __nv_bfloat16* w,    \
                          int seqs, int rows, int width, int taps, long long line_bytes) {                                \
    pdl_wait();                                                                                                           \
    if (width % 4 == 0) {                                                                                                 \
      if (taps == 4) conv_body<T, 4, 3>(h, out, state, lines, cu, w, seqs, rows, width, taps, line_bytes);                \
      else conv_body<T, 4, 0>(h, out, state, lines, cu, w, seqs, rows, width, taps, line_bytes);                          \
    } else {                                                                                                              \
      conv_body<T, 1, 0>(h, out, state, lines, cu, w, seqs, rows, width, taps, line_bytes);                               \
    }                                                                                                                     \
    pdl_launch_dependents();                                                                                              \
  }
CONV_ADD(__nv_bfloat16, bf16)
CONV_ADD(float, f32)
