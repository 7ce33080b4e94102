// build: precise
// A row plus a short causal convolution of it over time, channel by channel, for prompts and any ragged call:
//     out_t = h_t + sum_j w[c][j] h_(t - taps + 1 + j)      (zeros before a sequence's first row)
// The last taps - 1 rows of a sequence are its state line (the activations' type); line 0 is nobody's. One row per sequence
// (decode) is done by the kernel that makes h (resid.cu).
//   kern_conv_add_<act>        the rows
//   kern_conv_add_state_<act>  the lines move on, in a launch of their own: no row may see one half-moved
#include "act.cuh"

using namespace kern;

namespace {

constexpr int kRun = 16;      // rows a thread walks

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

// grid [ceil(rows / 16), ceil(width / 256 V)]. KEEP > 0: that many past rows (taps - 1) stay in registers.
template <typename T, int V, int KEEP>
KERN_DEVICE void conv_body(const T* h, T* out, const uint8_t* state, const int* lines, const int* cu, const __nv_bfloat16* w,
                           int seqs, int rows, int width, int taps, long long line_bytes) {
  const int c = (blockIdx.y * 256 + threadIdx.x) * V, keep = KEEP > 0 ? KEEP : taps - 1;
  const int ra = blockIdx.x * kRun, rb = min(min(rows, cu[seqs]), ra + kRun);
  if (c >= width || ra >= rb) return;
  int s = seq_of_row(cu, seqs, ra), r0 = cu[s], r1 = cu[s + 1], line = 0;
  const T* win = nullptr;
  auto enter = [&]() {
    line = checked_line(state, lines[s], line_bytes);
    win = reinterpret_cast<const T*>(state + (size_t)line * line_bytes) + c;
  };
  auto row = [&](int rr) {      // a row of this call, of the line, or nothing
    Vec<V> v = {};
    if (rr >= r0) v = ldv<V>(h + (size_t)rr * width + c);
    else if (line > 0) v = ldv<V>(win + (size_t)(keep + rr - r0) * width);
    return v;
  };
  enter();
  if constexpr (KEEP > 0) {
    float wt[KEEP + 1][V];
#pragma unroll
    for (int j = 0; j <= KEEP; ++j)
#pragma unroll
      for (int e = 0; e < V; ++e) wt[j][e] = __bfloat162float(w[(size_t)(c + e) * (KEEP + 1) + j]);
    Vec<V> past[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) past[j] = row(ra - KEEP + j);
    for (int r = ra; r < rb; ++r) {
      if (r >= r1) {
        while (r >= r1) { ++s; r1 = cu[s + 1]; }      // empty sequences are skipped
        r0 = cu[s];
        enter();
#pragma unroll
        for (int j = 0; j < KEEP; ++j) past[j] = row(r - KEEP + j);
      }
      const Vec<V> cur = ldv<V>(h + (size_t)r * width + c);
      Vec<V> acc = cur;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        acc.v[e] += wt[KEEP][e] * cur.v[e];
#pragma unroll
        for (int j = 0; j < KEEP; ++j) acc.v[e] += wt[j][e] * past[j].v[e];
      }
#pragma unroll
      for (int j = 0; j + 1 < KEEP; ++j) past[j] = past[j + 1];
      past[KEEP - 1] = cur;
      stv<V>(out + (size_t)r * width + c, acc);
    }
  } else {
    for (int r = ra; r < rb; ++r) {
      if (r >= r1) {
        while (r >= r1) { ++s; r1 = cu[s + 1]; }
        r0 = cu[s];
        enter();
      }
      Vec<V> acc = ldv<V>(h + (size_t)r * width + c);
      for (int j = keep; j >= 0; --j) {
        const Vec<V> v = row(r - keep + j);
#pragma unroll
        for (int e = 0; e < V; ++e) acc.v[e] += __bfloat162float(w[(size_t)(c + e) * taps + j]) * v.v[e];
      }
      stv<V>(out + (size_t)r * width + c, acc);
    }
  }
}

// grid [seqs, ceil(width / 256)]
template <typename T>
KERN_DEVICE void state_body(const T* h, uint8_t* state, const int* lines, const int* cu, int width, int taps, long long line_bytes) {
  const int s = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  if (c >= width) return;
  const int line = checked_line(state, lines[s], line_bytes);
  const int r0 = cu[s], n = cu[s + 1] - r0, keep = taps - 1;
  if (line <= 0 || n <= 0) return;
  T* win = reinterpret_cast<T*>(state + (size_t)line * line_bytes) + c;
  for (int j = 0; j < keep; ++j) {      // ascending: row j takes old row j + n, which no earlier j has overwritten
    const int src = n + j - keep;
    win[(size_t)j * width] = src >= 0 ? h[(size_t)(r0 + src) * width + c] : win[(size_t)(j + n) * width];
  }
}

}  // namespace

#define CONV_ADD(T, SFX)                                                                                                  \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_conv_add_##SFX(const T* h, T* out, const uint8_t* state, const int* lines, const int* cu,                      \
                          const __nv_bfloat16* w, int seqs, int rows, int width, int taps, long long line_bytes) {        \
    pdl_wait();                                                                                                           \
    if (width % 4 == 0) {                                                                                                 \
      if (taps == 4) conv_body<T, 4, 3>(h, out, state, lines, cu, w, seqs, rows, width, taps, line_bytes);                \
      else conv_body<T, 4, 0>(h, out, state, lines, cu, w, seqs, rows, width, taps, line_bytes);                          \
    } else {                                                                                                              \
      conv_body<T, 1, 0>(h, out, state, lines, cu, w, seqs, rows, width, taps, line_bytes);                               \
    }                                                                                                                     \
    pdl_launch_dependents();                                                                                              \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_conv_add_state_##SFX(const T* h, uint8_t* state, const int* lines, const int* cu, int width, int taps,         \
                                long long line_bytes) {                                                                   \
    pdl_wait();                                                                                                           \
    state_body<T>(h, state, lines, cu, width, taps, line_bytes);                                                          \
    pdl_launch_dependents();                                                                                              \
  }
CONV_ADD(__nv_bfloat16, bf16)
CONV_ADD(float, f32)
