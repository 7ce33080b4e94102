// build: precise
// Latent attention whose keys and values are both linear maps of one cached row per token, in the absorbed form: per head,
// score = (W_uk^T q) . c, and the weighted sum of the rows c goes through W_uv afterwards. A row may hold rotated key columns
// behind the latent, one part for all heads; then a sink per head may join the denominator, a window may end a row's reach and a
// gate per head may multiply its result. These kernels take any latent width
// and either activation type; mla_decode.cu holds the tensor-core form.
//   kern_latent_append_<act>   RMS norm of a token's latent, written to its row of the paged cache
//   kern_latent_prep_<act>     the same with the rotated columns behind it, and the RMS norm of a low-rank query row
//   kern_latent_attn_<act>     one (row, head) per block: softmax over the row's causal reach, f32 throughout
//   kern_latent_rot_attn_<act> the same with rotated columns (turning the query's), a sink, a window, a gate
#include "act.cuh"

using namespace kern;

namespace {

// x [n] -> out = x / rms w, by a block of 128
template <typename T>
KERN_DEVICE void norm_row(const T* x, const __nv_bfloat16* w, T* out, int n, float eps) {
  __shared__ float part[4];
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += 128) { const float v = ldf(x + i); ss += v * v; }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float inv = 1.f / sqrtf((part[0] + part[1] + part[2] + part[3]) / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += 128) stf(out + i, ldf(x + i) * inv * __bfloat162float(w[i]));
}

template <typename T>
KERN_DEVICE void append_body(const T* lat, uint8_t* cache, const long long* slots, const __nv_bfloat16* w, int rank, int stride,
                             float eps) {
  const int t = blockIdx.x;
  const long long slot = slots[t];
  if (slot < 0) return;
  T* dst = reinterpret_cast<T*>(cache) + (size_t)slot * rank;
  if (!KERN_CHECK(dst, (size_t)rank * sizeof(T), SITE_KV_APPEND)) return;
  norm_row(lat + (size_t)t * stride, w, dst, rank, eps);
}

// Row [query latent | latent | rot columns]: the first normed to q_low, the second normed and the third turned by the token's
// position (pairs i, i + rot / 2, or neighbours) to the token's cached row. Block 256, (q_rank + rank) floats of shared memory, V columns per
// thread and step.
template <typename T, int V>
KERN_DEVICE void prep_body(const T* rows, uint8_t* cache, T* q_low, const long long* positions, const long long* slots,
                           const float* cos_tab, const float* sin_tab, const __nv_bfloat16* w, const __nv_bfloat16* wq, int rank,
                           int rot, int halves, int q_rank, int stride, int q_stride, int max_pos, float eps, int* err) {
  extern __shared__ __align__(16) float lat_sm[];
  __shared__ float part[2][8];
  const int t = blockIdx.x, n = q_rank + rank, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* x = rows + (size_t)t * stride;
  const long long slot = slots[t];
  long long pos = positions[t];
  float sq = 0.f, sc = 0.f;
  for (int c = threadIdx.x * V; c < n; c += 256 * V) {
    const Vec<V> a = ldv<V>(x + c);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s += a.v[e] * a.v[e];
    if (c < q_rank) sq += s; else sc += s;
    stv<V>(lat_sm + c, a);
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if (lane == 0) { part[0][warp] = sq; part[1][warp] = sc; }
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) { sq += part[0][i]; sc += part[1][i]; }
  const float inv_q = 1.f / sqrtf(sq / (float)q_rank + eps), inv_c = 1.f / sqrtf(sc / (float)rank + eps);
  T* dst = reinterpret_cast<T*>(cache) + (size_t)(slot < 0 ? 0 : slot) * (rank + rot);
  const bool store = slot >= 0 && KERN_CHECK(dst, (size_t)(rank + rot) * sizeof(T), SITE_KV_APPEND);
  for (int c = threadIdx.x * V; c < n; c += 256 * V) {
    const bool is_q = c < q_rank;
    if (!is_q && !store) break;
    const Vec<V> a = ldv<V>(lat_sm + c), b = ldv<V>(is_q ? wq + c : w + (c - q_rank));
    const float inv = is_q ? inv_q : inv_c;
    Vec<V> o;
#pragma unroll
    for (int e = 0; e < V; ++e) o.v[e] = a.v[e] * inv * b.v[e];
    stv<V>(is_q ? q_low + (size_t)t * q_stride + c : dst + (c - q_rank), o);
  }
  if (pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0) set_error(err, ERR_BOUNDS);
    pos = 0;
  }
  const int half = rot >> 1;
  if (store)
    for (int i = threadIdx.x; i < half; i += 256) {
      const int lo = halves ? i : 2 * i, hi = halves ? half + i : 2 * i + 1;
      const float a = ldf(x + n + lo), b = ldf(x + n + hi), c = cos_tab[pos * half + i], s = sin_tab[pos * half + i];
      stf(dst + rank + lo, a * c - b * s);
      stf(dst + rank + hi, b * c + a * s);
    }
}

template <typename T>
struct RotArgs {      // as LatentExtra in mla_decode.cu
  const T* q_rot = nullptr;
  int stride = 0, rot = 0, max_pos = 0;
  const float* cos_tab = nullptr;
  const float* sin_tab = nullptr;
  const __nv_bfloat16* sink = nullptr;
  int halves = 1, window = 0x7fffffff;
  const T* gate = nullptr;
  int gate_stride = 0;
};

// Four warps walk the keys (key j belongs to warp j % 4); a lane holds the columns i * 32 + lane of the query and of the
// warp's running sum. RL = columns per lane. The rotated columns of the query are turned into shared memory first (ROT).
template <typename T, int RL, bool ROT = false>
KERN_DEVICE void attn_body(const T* q, const uint8_t* cache, T* out, const int* table, const int* lens, const int* row_seq,
                           int heads, int rank, int max_pages, int page, float scale, int* err, const RotArgs<T>& ex = RotArgs<T>()) {
  extern __shared__ __align__(16) float lat_sm[];      // [4][rank] partial sums, then [4] maxima, [4] weights, [rot] turned query
  const int h = blockIdx.x, r = blockIdx.y;
  const int L = lens[r];
  if (L <= 0) return;
  if (L > max_pages * page && threadIdx.x == 0) set_error(err, ERR_BOUNDS);     // keys past the table row are left out
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* pages = table + (size_t)(row_seq ? row_seq[r] : r) * max_pages;
  const T* rows = reinterpret_cast<const T*>(cache);
  const T* qr = q + ((size_t)r * heads + h) * rank;
  const int cols = rank + (ROT ? ex.rot : 0);
  float* turned = lat_sm + 4 * rank + 8;
  if constexpr (ROT) {
    if (L > ex.max_pos && threadIdx.x == 0) set_error(err, ERR_BOUNDS);
    const int half = ex.rot >> 1, pos = min(L, ex.max_pos) - 1;
    const T* x = ex.q_rot + (size_t)r * ex.stride + (size_t)h * ex.rot;
    for (int i = threadIdx.x; i < half; i += 128) {
      const int lo = ex.halves ? i : 2 * i, hi = ex.halves ? half + i : 2 * i + 1;
      const float a = ldf(x + lo), b = ldf(x + hi), c = ex.cos_tab[(size_t)pos * half + i], s = ex.sin_tab[(size_t)pos * half + i];
      turned[lo] = a * c - b * s;
      turned[hi] = b * c + a * s;
    }
    __syncthreads();
  }
  float qv[RL], o[RL];
#pragma unroll
  for (int i = 0; i < RL; ++i) {
    const int c = i * 32 + lane;
    qv[i] = c < rank ? ldf(qr + c) : 0.f;
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int j = (ROT ? max(0, L - ex.window) : 0) + warp; j < L; j += 4) {
    const int pi = j / page;
    if (pi >= max_pages) break;
    const T* row = rows + ((size_t)pages[pi] * page + j % page) * cols;
    if (!KERN_CHECK(row, (size_t)cols * sizeof(T), SITE_LATENT_ROW)) continue;
    float c[RL], s = 0.f;
#pragma unroll
    for (int i = 0; i < RL; ++i) {
      const int k = i * 32 + lane;
      c[i] = k < rank ? ldf(row + k) : 0.f;
      s += qv[i] * c[i];
    }
    if constexpr (ROT)
      for (int k = lane; k < ex.rot; k += 32) s += turned[k] * ldf(row + rank + k);
    s = warp_sum(s) * scale;
    const float mn = fmaxf(m, s), f = expf(m - mn), e = expf(s - mn);
    m = mn;
    l = l * f + e;
#pragma unroll
    for (int i = 0; i < RL; ++i) o[i] = o[i] * f + e * c[i];
  }
  float* acc = lat_sm;
  float* ms = lat_sm + 4 * rank;
  float* ls = ms + 4;
  if (lane == 0) { ms[warp] = m; ls[warp] = l; }
#pragma unroll
  for (int i = 0; i < RL; ++i)
    if (i * 32 + lane < rank) acc[warp * rank + i * 32 + lane] = o[i];
  __syncthreads();
  float mx = fmaxf(fmaxf(ms[0], ms[1]), fmaxf(ms[2], ms[3]));
  float f[4], den = 0.f, den_gate = 1.f;
  if constexpr (ROT) {
    if (ex.gate) den_gate = 1.f + expf(-ldf(ex.gate + (size_t)r * ex.gate_stride + h));
    if (ex.sink) {
      const float sk = __bfloat162float(ex.sink[h]);
      mx = fmaxf(mx, sk);
      den = expf(sk - mx);
    }
  }
#pragma unroll
  for (int w = 0; w < 4; ++w) { f[w] = expf(ms[w] - mx); den += f[w] * ls[w]; }
  for (int c = threadIdx.x; c < rank; c += 128) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += f[w] * acc[w * rank + c];
    stf(out + ((size_t)r * heads + h) * rank + c, v / (den * den_gate));
  }
}

}  // namespace

// append: grid = tokens, block 128. prep: grid = tokens. attn: grid [heads, rows], block 128, (4 rank + 8 + rot) floats of shared memory.
#define LATENT_ATTN(T, SFX, W)                                                                                            \
  extern "C" __global__ void __launch_bounds__(128)                                                                       \
      kern_latent_attn_##SFX##_w##W(const T* q, const uint8_t* cache, T* out, const int* table, const int* lens,          \
                                    const int* row_seq, int heads, int rank, int max_pages, int page, float scale,        \
                                    int* err) {                                                                           \
    pdl_wait();                                                                                                           \
    attn_body<T, W / 32>(q, cache, out, table, lens, row_seq, heads, rank, max_pages, page, scale, err);                  \
  }
#define LATENT_ROT_ATTN(T, SFX, W)                                                                                        \
  extern "C" __global__ void __launch_bounds__(128)                                                                       \
      kern_latent_rot_attn_##SFX##_w##W(const T* q, const uint8_t* cache, T* out, const int* table, const int* lens,      \
                                        const int* row_seq, int heads, int rank, int max_pages, int page, float scale,    \
                                        int* err, const T* q_rot, const float* cos_tab, const float* sin_tab,             \
                                        const __nv_bfloat16* sink, const T* gate, int rot_stride, int rot, int max_pos,   \
                                        int halves, int window, int gate_stride) {                                        \
    pdl_wait();                                                                                                           \
    const RotArgs<T> ex{q_rot, rot_stride, rot, max_pos, cos_tab, sin_tab, sink, halves, window, gate, gate_stride};      \
    attn_body<T, W / 32, true>(q, cache, out, table, lens, row_seq, heads, rank, max_pages, page, scale, err, ex);        \
  }
#define LATENT_ENTRIES(T, SFX)                                                                                            \
  extern "C" __global__ void __launch_bounds__(128)                                                                       \
      kern_latent_append_##SFX(const T* lat, uint8_t* cache, const long long* slots, const __nv_bfloat16* w, int rank,    \
                               int stride, float eps) {                                                                   \
    pdl_wait();                                                                                                           \
    append_body<T>(lat, cache, slots, w, rank, stride, eps);                                                              \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_latent_prep_##SFX(const T* rows, uint8_t* cache, T* q_low, const long long* positions, const long long* slots, \
                             const float* cos_tab, const float* sin_tab, const __nv_bfloat16* w, const __nv_bfloat16* wq, \
                             int rank, int rot, int halves, int q_rank, int stride, int q_stride, int max_pos, float eps, \
                             int* err) {                                                                                  \
    pdl_wait();                                                                                                           \
    const bool vec = (rank | rot | q_rank | stride | q_stride) % 4 == 0 &&                                                \
                     ((reinterpret_cast<uintptr_t>(rows) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(q_low) | \
                       reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(wq)) & 15) == 0;                      \
    if (vec)                                                                                                              \
      prep_body<T, 4>(rows, cache, q_low, positions, slots, cos_tab, sin_tab, w, wq, rank, rot, halves, q_rank, stride, q_stride, \
                      max_pos, eps, err);                                                                                 \
    else                                                                                                                  \
      prep_body<T, 1>(rows, cache, q_low, positions, slots, cos_tab, sin_tab, w, wq, rank, rot, halves, q_rank, stride, q_stride, \
                      max_pos, eps, err);                                                                                 \
    pdl_launch_dependents();                                                                                              \
  }                                                                                                                       \
  LATENT_ATTN(T, SFX, 64)                                                                                                 \
  LATENT_ATTN(T, SFX, 128)                                                                                                \
  LATENT_ATTN(T, SFX, 256)                                                                                                \
  LATENT_ATTN(T, SFX, 512)                                                                                                \
  LATENT_ATTN(T, SFX, 1024)                                                                                               \
  LATENT_ROT_ATTN(T, SFX, 64)                                                                                             \
  LATENT_ROT_ATTN(T, SFX, 128)                                                                                            \
  LATENT_ROT_ATTN(T, SFX, 256)                                                                                            \
  LATENT_ROT_ATTN(T, SFX, 512)                                                                                            \
  LATENT_ROT_ATTN(T, SFX, 1024)

LATENT_ENTRIES(__nv_bfloat16, bf16)
LATENT_ENTRIES(float, f32)
