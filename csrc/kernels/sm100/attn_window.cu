// build: precise
// Attention over a paged cache in a sliding window, with capped scores and a learned sink per query head:
//     score = cap tanh(q.k scale / cap);  weight_j = exp(score_j) / (exp(sink_h) + sum over the window of exp(score))
// attention over the whole causal reach with a sink (learned, or a score of 0) and an output gate, attention in a window beside the
// mean keys and values of the blocks before it, and what prepares their rows.
//   kern_qk_prep_<act>          per head: RMS norm of q and k with a weight of their own (or none), rotary positions on the first
//                               columns (pairs (2i, 2i + 1), or halves), k and v into their rows of the paged cache
//   kern_qk_prep_pool_<act>     the same for one row per sequence, and the mean row of the block that it completes, if it does
//   kern_pool_blocks_<act>      the mean rows of the blocks that end in a ragged call
//   kern_qk_prep_whole_<act>    the same with a norm over all heads' columns at once, and values from any columns of the row (the
//                               keys' own, as projected, in a mixer whose keys are its values)
//   kern_window_attn_<act>_w*   one (row, query head) per block, any sizes, either activation type
//   kern_attn_window_*_d*       bf16 with equal head dims 64 / 128 / 256: the bodies of attn_paged.cu (decode rows with split
//                               keys, prompt rows, both lists of a ragged call in one launch)
//   kern_pooled_attn_<act>_w*   the same in a window beside pooled rows, without cap and sink
//   kern_attn_sink_*_d*         the same bodies without window and cap
//   kern_attn_pooled_*_d*       the same bodies in a window beside pooled rows
//   kern_attn_window_merge      the partials of split keys, where the sink joins the denominator
// Cache of one layer: [page][k: head, offset, dim | v: head, offset, vdim]; with equal dims that is attn_prep.cu's layout. Pooled
// rows are a second cache on the same pages: block b of P tokens lies in the page of its last token, at slot b minus the first
// block that ends in that page; [page][k: head, slot, dim | v: head, slot, vdim], ceil(page / P) slots.
// Norms, angles, scores, weights and sums are f32.
#define KERN_ATTN_NO_ENTRIES
#include "attn_paged.cu"
#include "act.cuh"

using namespace kern;

namespace {

// grid = rows, block 256: a warp per head, heads dealt to the eight warps; 8 max(d, dv) floats of shared memory. N > 0: pairs of
// neighbours, heads of up to 128 N whole vectors, norms on both or (NORM false) on neither.
template <typename T, int N, bool NORM = true>
KERN_DEVICE void prep_body(T* qkv, uint8_t* cache, const long long* positions, const long long* slots, const float* cos_tab,
                           const float* sin_tab, const __nv_bfloat16* q_norm, const __nv_bfloat16* k_norm, int hq, int hk, int d,
                           int dv, int rot, int halves, int page_size, int row_stride, int max_pos, float eps, int* err) {
  extern __shared__ __align__(16) float prep_sm[];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* row = prep_sm + warp * max(d, dv);
  long long pos = positions[t];
  const long long slot = slots[t];
  if (pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0) set_error(err, ERR_BOUNDS);
    pos = 0;
  }
  const int half = rot >> 1;
  const float* cs = cos_tab + (size_t)pos * half;
  const float* sn = sin_tab + (size_t)pos * half;
  T* base = qkv + (size_t)t * row_stride;
  T* page = reinterpret_cast<T*>(cache) + (size_t)(slot < 0 ? 0 : slot / page_size) * hk * page_size * (d + dv);
  const int off = slot < 0 ? 0 : (int)(slot % page_size);
  if constexpr (N > 0) {
    // four neighbouring columns per lane and step, both columns of a pair in the lane: nothing leaves the registers
    Vec<4> w[2][N], c2[N];
    bool turned[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * 32 + lane) * 4;
      turned[i] = c < rot;
      if (NORM && c < d) { w[0][i] = ldv<4>(q_norm + c); w[1][i] = ldv<4>(k_norm + c); }
      if (turned[i]) {
        const float2 a = *reinterpret_cast<const float2*>(cs + c / 2), b = *reinterpret_cast<const float2*>(sn + c / 2);
        c2[i].v[0] = a.x; c2[i].v[1] = b.x; c2[i].v[2] = a.y; c2[i].v[3] = b.y;
      }
    }
#pragma unroll 4
    for (int h = warp; h < hq + hk; h += 8) {
      const bool is_q = h < hq;
      T* src = base + (size_t)h * d;
      T* dst = is_q ? src : page + ((size_t)(h - hq) * page_size + off) * d;
      const bool store = is_q || (slot >= 0 && KERN_CHECK(dst, (size_t)d * sizeof(T), SITE_KV_APPEND));
      Vec<4> x[N];
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int c = (i * 32 + lane) * 4;
        if (c >= d) continue;
        x[i] = ldv<4>(src + c);
#pragma unroll
        for (int e = 0; e < 4; ++e) ss += x[i].v[e] * x[i].v[e];
      }
      const float inv = NORM ? 1.f / sqrtf(warp_sum(ss) / (float)d + eps) : 1.f;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int c = (i * 32 + lane) * 4;
        if (c >= d || !store) continue;
        if constexpr (NORM) {
#pragma unroll
          for (int e = 0; e < 4; ++e) x[i].v[e] *= inv * (is_q ? w[0][i].v[e] : w[1][i].v[e]);
        }
        if (turned[i]) {
          Vec<4> o;
          o.v[0] = x[i].v[0] * c2[i].v[0] - x[i].v[1] * c2[i].v[1]; o.v[1] = x[i].v[1] * c2[i].v[0] + x[i].v[0] * c2[i].v[1];
          o.v[2] = x[i].v[2] * c2[i].v[2] - x[i].v[3] * c2[i].v[3]; o.v[3] = x[i].v[3] * c2[i].v[2] + x[i].v[2] * c2[i].v[3];
          x[i] = o;
        }
        stv<4>(dst + c, x[i]);
      }
    }
  }
  for (int h = (N > 0 ? hq + hk : 0) + warp; h < hq + 2 * hk; h += 8) {
    const bool is_q = h < hq, is_v = h >= hq + hk;
    if (!is_q && slot < 0) continue;
    if (is_v) {
      const int kh = h - hq - hk;
      const T* src = base + (size_t)(hq + hk) * d + (size_t)kh * dv;
      T* dst = page + (size_t)hk * page_size * d + ((size_t)kh * page_size + off) * dv;
      if (!KERN_CHECK(dst, (size_t)dv * sizeof(T), SITE_KV_APPEND)) continue;
      for (int i = lane; i < dv; i += 32) dst[i] = src[i];
      continue;
    }
    T* src = base + (size_t)h * d;
    T* dst = is_q ? src : page + ((size_t)(h - hq) * page_size + off) * d;
    if (!is_q && !KERN_CHECK(dst, (size_t)d * sizeof(T), SITE_KV_APPEND)) continue;
    const __nv_bfloat16* w = is_q ? q_norm : k_norm;
    float ss = 0.f;
    for (int i = lane; i < d; i += 32) {
      const float v = ldf(src + i);
      row[i] = v;
      ss += v * v;
    }
    const float inv = w ? 1.f / sqrtf(warp_sum(ss) / (float)d + eps) : 1.f;
    __syncwarp();
    if (w)
      for (int i = lane; i < d; i += 32) row[i] *= inv * __bfloat162float(w[i]);
    __syncwarp();
    for (int i = lane; i < d; i += 32) {
      float o = row[i];
      if (i < rot) {
        const int j = halves ? (i < half ? i : i - half) : i >> 1;
        const bool lo = halves ? i < half : !(i & 1);
        const int other = halves ? (lo ? i + half : i - half) : i ^ 1;
        o = lo ? o * cs[j] - row[other] * sn[j] : o * cs[j] + row[other] * sn[j];
      }
      stf(dst + i, o);
    }
    __syncwarp();
  }
}

template <typename T>
KERN_DEVICE void prep_rows(T* qkv, uint8_t* cache, const long long* positions, const long long* slots, const float* cos_tab,
                           const float* sin_tab, const __nv_bfloat16* q_norm, const __nv_bfloat16* k_norm, int hq, int hk, int d,
                           int dv, int rot, int halves, int page_size, int row_stride, int max_pos, float eps, int* err) {
  const bool vec = !halves && (d | dv | rot | row_stride) % 4 == 0 && d <= 256 && !q_norm == !k_norm &&
                   ((reinterpret_cast<uintptr_t>(qkv) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(q_norm) |
                     reinterpret_cast<uintptr_t>(k_norm)) & 15) == 0;
#define PREP_BODY(...) \
  prep_body<T, __VA_ARGS__>(qkv, cache, positions, slots, cos_tab, sin_tab, q_norm, k_norm, hq, hk, d, dv, rot, halves, page_size, row_stride, max_pos, eps, err)
  if (vec && q_norm && d <= 128) PREP_BODY(1);
  else if (vec && q_norm) PREP_BODY(2);
  else if (vec && d <= 128) PREP_BODY(1, false);
  else if (vec) PREP_BODY(2, false);
  else PREP_BODY(0);
#undef PREP_BODY
}

// The block of `pool` tokens that the row at `pos` ends: the mean of its keys and of its values as the cache holds them, by a block
// of 256. `pages`: the table row of the sequence; `slot`: where the row itself lies. V columns per thread and step.
template <typename T, int V>
KERN_DEVICE void pool_body(const T* cache, T* pooled, const int* pages, long long pos, long long slot, int hk, int d, int dv,
                           int pool, int slots, long long pooled_stride, int page, int max_pages, int* err) {
  const int b = (int)(pos / pool), first = b * pool, kcols = hk * d;
  const int at = b - (int)(pos / page) * page / pool;
  T* out = reinterpret_cast<T*>(reinterpret_cast<uint8_t*>(pooled) + (slot / page) * pooled_stride);
  if (pos / page >= max_pages) {      // the table row does not reach that far
    if (threadIdx.x == 0) set_error(err, ERR_BOUNDS);
    return;
  }
  for (int c = threadIdx.x * V; c < hk * (d + dv); c += 256 * V) {
    const bool is_k = c < kcols;
    const int cols = is_k ? d : dv, h = (is_k ? c : c - kcols) / cols, i = (is_k ? c : c - kcols) - h * cols;
    const size_t base = (is_k ? 0 : (size_t)kcols * page) + (size_t)h * page * cols + i;
    T* dst = out + (is_k ? 0 : (size_t)kcols * slots) + ((size_t)h * slots + at) * cols + i;
    Vec<V> acc = {};
    for (int left = pool, pi = first / page, off = first % page; left > 0; ++pi, off = 0) {      // page by page
      const int run = min(left, page - off);
      const T* src = cache + (size_t)pages[pi] * hk * page * (d + dv) + base + (size_t)off * cols;
      left -= run;
      if (!KERN_CHECK(src, (size_t)run * cols * sizeof(T), SITE_KV_ROW)) continue;
#pragma unroll 8
      for (int j = 0; j < run; ++j) {
        const Vec<V> a = ldv<V>(src + (size_t)j * cols);
#pragma unroll
        for (int e = 0; e < V; ++e) acc.v[e] += a.v[e];
      }
    }
    if (!KERN_CHECK(dst, V * sizeof(T), SITE_KV_APPEND)) continue;
#pragma unroll
    for (int e = 0; e < V; ++e) acc.v[e] /= (float)pool;
    stv<V>(dst, acc);
  }
}

KERN_DEVICE int seq_of_row(const int* cu, int seqs, int r) {      // the last s with cu[s] <= r
  int lo = 0, hi = seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= r) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// Row t ends a block, or nothing happens. `cu`: a ragged call's row starts; without it row t is sequence t's.
template <typename T>
KERN_DEVICE void pool_row(int t, const uint8_t* cache, uint8_t* pooled, const long long* positions, const long long* slots,
                          const int* table, const int* cu, int seqs, int hk, int d, int dv, int pool, int n_slots,
                          long long pooled_stride, int page, int max_pages, int* err) {
  const long long pos = positions[t], slot = slots[t];
  if (slot < 0 || pos < 0 || (pos + 1) % pool != 0) return;
  const int* pages = table + (size_t)(cu ? seq_of_row(cu, seqs, t) : t) * max_pages;
  const T* src = reinterpret_cast<const T*>(cache);
  T* dst = reinterpret_cast<T*>(pooled);
  if ((d | dv) % 4 == 0 && pooled_stride % 16 == 0)
    pool_body<T, 4>(src, dst, pages, pos, slot, hk, d, dv, pool, n_slots, pooled_stride, page, max_pages, err);
  else
    pool_body<T, 1>(src, dst, pages, pos, slot, hk, d, dv, pool, n_slots, pooled_stride, page, max_pages, err);
}

// grid = rows, block 256; (hq + hk) d floats of shared memory. V columns per thread and step.
template <typename T, int V>
KERN_DEVICE void prep_whole_body(T* qkv, uint8_t* cache, const long long* positions, const long long* slots, const float* cos_tab,
                                 const float* sin_tab, const __nv_bfloat16* q_norm, const __nv_bfloat16* k_norm, int hq, int hk,
                                 int d, int dv, int v_col, int rot, int halves, int page_size, int row_stride, int max_pos,
                                 float eps, int* err) {
  extern __shared__ __align__(16) float prep_sm[];      // q and k as projected
  __shared__ float part[2][8];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nq = hq * d, n = (hq + hk) * d;
  long long pos = positions[t];
  const long long slot = slots[t];
  if (pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0) set_error(err, ERR_BOUNDS);
    pos = 0;
  }
  const int half = rot >> 1;
  const float* cs = cos_tab + (size_t)pos * half;
  const float* sn = sin_tab + (size_t)pos * half;
  T* row = qkv + (size_t)t * row_stride;
  float ssq = 0.f, ssk = 0.f;
  for (int c = threadIdx.x * V; c < n; c += 256 * V) {
    const Vec<V> a = ldv<V>(row + c);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s += a.v[e] * a.v[e];
    if (c < nq) ssq += s; else ssk += s;
    stv<V>(prep_sm + c, a);
  }
  ssq = warp_sum(ssq);
  ssk = warp_sum(ssk);
  if (lane == 0) { part[0][warp] = ssq; part[1][warp] = ssk; }
  __syncthreads();
  ssq = ssk = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) { ssq += part[0][i]; ssk += part[1][i]; }
  const float inv_q = 1.f / sqrtf(ssq / (float)nq + eps), inv_k = 1.f / sqrtf(ssk / (float)(n - nq) + eps);
  T* page = reinterpret_cast<T*>(cache) + (size_t)(slot < 0 ? 0 : slot / page_size) * hk * page_size * (d + dv);
  const int off = slot < 0 ? 0 : (int)(slot % page_size);
  for (int c = threadIdx.x * V; c < n; c += 256 * V) {
    const bool is_q = c < nq;
    if (!is_q && slot < 0) break;
    const __nv_bfloat16* w = is_q ? q_norm : k_norm - nq;
    const float inv = is_q ? inv_q : inv_k;
    const int h = c / d, i = c - h * d;
    T* dst = is_q ? row + c : page + ((size_t)(h - hq) * page_size + off) * d + i;
    if (!is_q && !KERN_CHECK(dst, V * sizeof(T), SITE_KV_APPEND)) continue;
    const Vec<V> a = ldv<V>(prep_sm + c), b = ldv<V>(w + c);
    Vec<V> o;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      o.v[e] = a.v[e] * inv * b.v[e];
      if (i + e < rot) {
        const int j = halves ? (i + e < half ? i + e : i + e - half) : (i + e) >> 1;
        const bool lo = halves ? i + e < half : !((i + e) & 1);
        const int other = c + e + (halves ? (lo ? half : -half) : (lo ? 1 : -1));
        const float x = prep_sm[other] * inv * __bfloat162float(w[other]);
        o.v[e] = lo ? o.v[e] * cs[j] - x * sn[j] : o.v[e] * cs[j] + x * sn[j];
      }
    }
    stv<V>(dst, o);
  }
  if (slot < 0) return;
  // the values, as they are: k above went to the cache only, so these may be its columns
  for (int c = threadIdx.x * V; c < hk * dv; c += 256 * V) {
    const int h = c / dv, i = c - h * dv;
    T* dst = page + (size_t)hk * page_size * d + ((size_t)h * page_size + off) * dv + i;
    if (!KERN_CHECK(dst, V * sizeof(T), SITE_KV_APPEND)) continue;
    stv<V>(dst, ldv<V>(row + v_col + c));
  }
}

// Four warps walk the keys of the row's window (key j belongs to warp j % 4); a lane holds the columns i * 32 + lane of the
// query and of the warp's running sum. RL = columns per lane. cap 0: scores as they are; no sink pointer: a score of 0; gate:
// sigmoid of it multiplies the finished row. POOL: before the window come the pooled rows that the row sees, and there is no sink.
struct PooledRows {
  const uint8_t* rows = nullptr;
  int pool = 1, slots = 1;
  long long page_stride = 0;
};
template <typename T, int RL, bool POOL = false>
KERN_DEVICE void attn_any_body(const T* q, const uint8_t* cache, T* out, const int* table, const int* lens, const int* row_seq,
                               const __nv_bfloat16* sink, const T* gate, int hq, int hk, int d, int dv, int q_stride, int out_stride,
                               int gate_stride, int max_pages, int page, int window, float scale, float cap, float out_scale, int* err,
                               const PooledRows& pr = PooledRows()) {
  extern __shared__ __align__(16) float win_sm[];      // [4][dv] partial sums, then [4] maxima, [4] weights
  const int h = blockIdx.x, r = blockIdx.y;
  const int L = lens[r];
  if (L <= 0) return;
  if (L > max_pages * page && threadIdx.x == 0) set_error(err, ERR_BOUNDS);     // keys past the table row are left out
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kh = h / (hq / hk);
  const int* pages = table + (size_t)(row_seq ? row_seq[r] : r) * max_pages;
  const T* rows = reinterpret_cast<const T*>(cache);
  const T* qr = q + (size_t)r * q_stride + (size_t)h * d;
  float qv[RL], o[RL];
#pragma unroll
  for (int i = 0; i < RL; ++i) {
    const int c = i * 32 + lane;
    qv[i] = c < d ? ldf(qr + c) : 0.f;
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  auto see = [&](const T* kr, const T* vr) {
    if (!KERN_CHECK(kr, (size_t)d * sizeof(T), SITE_KV_ROW) || !KERN_CHECK(vr, (size_t)dv * sizeof(T), SITE_KV_ROW)) return;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < RL; ++i) {
      const int c = i * 32 + lane;
      if (c < d) s += qv[i] * ldf(kr + c);
    }
    s = warp_sum(s) * scale;
    if (cap > 0.f) s = cap * tanhf(s / cap);
    const float mn = fmaxf(m, s), f = expf(m - mn), e = expf(s - mn);
    m = mn;
    l = l * f + e;
#pragma unroll
    for (int i = 0; i < RL; ++i) {
      const int c = i * 32 + lane;
      o[i] = o[i] * f + e * (c < dv ? ldf(vr + c) : 0.f);
    }
  };
  if constexpr (POOL) {
    const int seen = L - window > 0 ? (L - window) / pr.pool : 0;
    for (int b = warp; b < seen; b += 4) {
      const int pi = (b * pr.pool + pr.pool - 1) / page, at = b - pi * page / pr.pool;
      if (pi >= max_pages) break;
      const T* pg = reinterpret_cast<const T*>(pr.rows + (size_t)pages[pi] * pr.page_stride);
      see(pg + ((size_t)kh * pr.slots + at) * d, pg + (size_t)hk * pr.slots * d + ((size_t)kh * pr.slots + at) * dv);
    }
  }
  for (int j = max(0, L - window) + warp; j < L; j += 4) {
    const int pi = j / page;
    if (pi >= max_pages) break;
    const T* pg = rows + (size_t)pages[pi] * hk * page * (d + dv);
    see(pg + ((size_t)kh * page + j % page) * d, pg + (size_t)hk * page * d + ((size_t)kh * page + j % page) * dv);
  }
  float* acc = win_sm;
  float* ms = win_sm + 4 * dv;
  float* ls = ms + 4;
  if (lane == 0) { ms[warp] = m; ls[warp] = l; }
#pragma unroll
  for (int i = 0; i < RL; ++i)
    if (i * 32 + lane < dv) acc[warp * dv + i * 32 + lane] = o[i];
  __syncthreads();
  const float sk = POOL ? -INFINITY : (sink ? __bfloat162float(sink[h]) : 0.f);
  const float mx = fmaxf(sk, fmaxf(fmaxf(ms[0], ms[1]), fmaxf(ms[2], ms[3])));
  float f[4], den = expf(sk - mx);
#pragma unroll
  for (int w = 0; w < 4; ++w) { f[w] = expf(ms[w] - mx); den += f[w] * ls[w]; }
  for (int c = threadIdx.x; c < dv; c += 128) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += f[w] * acc[w * dv + c];
    v = v / den * out_scale;
    if (gate) v /= 1.f + expf(-ldf(gate + (size_t)r * gate_stride + (size_t)h * dv + c));
    stf(out + (size_t)r * out_stride + (size_t)h * dv + c, v);
  }
}

}  // namespace

// attn: grid [heads, rows], block 128, (4 dv + 8) floats of shared memory
#define WINDOW_ATTN(T, SFX, W)                                                                                             \
  extern "C" __global__ void __launch_bounds__(128)                                                                        \
      kern_window_attn_##SFX##_w##W(const T* q, const uint8_t* cache, T* out, const int* table, const int* lens,           \
                                    const int* row_seq, const __nv_bfloat16* sink, const T* gate, int hq, int hk, int d,   \
                                    int dv, int q_stride, int out_stride, int gate_stride, int max_pages, int page,        \
                                    int window, float scale, float cap, float out_scale, int* err) {                       \
    pdl_wait();                                                                                                            \
    attn_any_body<T, W / 32>(q, cache, out, table, lens, row_seq, sink, gate, hq, hk, d, dv, q_stride, out_stride,         \
                             gate_stride, max_pages, page, window, scale, cap, out_scale, err);                            \
  }
#define POOLED_ATTN(T, SFX, W)                                                                                             \
  extern "C" __global__ void __launch_bounds__(128)                                                                        \
      kern_pooled_attn_##SFX##_w##W(const T* q, const uint8_t* cache, const uint8_t* pooled, T* out, const int* table,     \
                                    const int* lens, const int* row_seq, int hq, int hk, int d, int dv, int q_stride,      \
                                    int out_stride, int max_pages, int page, int window, int pool, int n_slots,            \
                                    long long pooled_stride, float scale, int* err) {                                      \
    pdl_wait();                                                                                                            \
    attn_any_body<T, W / 32, true>(q, cache, out, table, lens, row_seq, nullptr, nullptr, hq, hk, d, dv, q_stride,         \
                                   out_stride, 0, max_pages, page, window, scale, 0.f, 1.f, err,                           \
                                   PooledRows{pooled, pool, n_slots, pooled_stride});                                      \
  }
#define WINDOW_ENTRIES(T, SFX)                                                                                             \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_qk_prep_##SFX(T* qkv, uint8_t* cache, const long long* positions, const long long* slots, const float* cos_tab, \
                         const float* sin_tab, const __nv_bfloat16* q_norm, const __nv_bfloat16* k_norm, int hq, int hk,   \
                         int d, int dv, int rot, int halves, int page_size, int row_stride, int max_pos, float eps,        \
                         int* err) {                                                                                       \
    pdl_wait();                                                                                                            \
    prep_rows<T>(qkv, cache, positions, slots, cos_tab, sin_tab, q_norm, k_norm, hq, hk, d, dv, rot, halves, page_size,    \
                 row_stride, max_pos, eps, err);                                                                           \
    pdl_launch_dependents();                                                                                               \
  }                                                                                                                        \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_qk_prep_pool_##SFX(T* qkv, uint8_t* cache, uint8_t* pooled, const long long* positions, const long long* slots, \
                              const int* table, const float* cos_tab, const float* sin_tab, int hq, int hk, int d, int dv, \
                              int rot, int halves, int page_size, int row_stride, int max_pos, int pool, int n_slots,      \
                              long long pooled_stride, int max_pages, int* err) {                                          \
    pdl_wait();                                                                                                            \
    prep_rows<T>(qkv, cache, positions, slots, cos_tab, sin_tab, nullptr, nullptr, hq, hk, d, dv, rot, halves, page_size,  \
                 row_stride, max_pos, 0.f, err);                                                                           \
    __syncthreads();      /* the row that ends a block is part of it */                                                    \
    pool_row<T>(blockIdx.x, cache, pooled, positions, slots, table, nullptr, 0, hk, d, dv, pool, n_slots, pooled_stride,   \
                page_size, max_pages, err);                                                                                \
    pdl_launch_dependents();                                                                                               \
  }                                                                                                                        \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_pool_blocks_##SFX(const uint8_t* cache, uint8_t* pooled, const long long* positions, const long long* slots,    \
                             const int* table, const int* cu, int seqs, int rows, int hk, int d, int dv, int page_size,    \
                             int pool, int n_slots, long long pooled_stride, int max_pages, int* err) {                    \
    pdl_wait();                                                                                                            \
    if (blockIdx.x < min(rows, cu[seqs]))                                                                                  \
      pool_row<T>(blockIdx.x, cache, pooled, positions, slots, table, cu, seqs, hk, d, dv, pool, n_slots, pooled_stride,   \
                  page_size, max_pages, err);                                                                              \
    pdl_launch_dependents();                                                                                               \
  }                                                                                                                        \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_qk_prep_whole_##SFX(T* qkv, uint8_t* cache, const long long* positions, const long long* slots,                 \
                               const float* cos_tab, const float* sin_tab, const __nv_bfloat16* q_norm,                    \
                               const __nv_bfloat16* k_norm, int hq, int hk, int d, int dv, int v_col, int rot, int halves, \
                               int page_size, int row_stride, int max_pos, float eps, int* err) {                          \
    pdl_wait();                                                                                                            \
    const bool vec = (d | dv | v_col | row_stride) % 4 == 0 &&                                                             \
                     ((reinterpret_cast<uintptr_t>(qkv) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(q_norm) | \
                       reinterpret_cast<uintptr_t>(k_norm)) & 15) == 0;                                                    \
    if (vec)                                                                                                               \
      prep_whole_body<T, 4>(qkv, cache, positions, slots, cos_tab, sin_tab, q_norm, k_norm, hq, hk, d, dv, v_col, rot,     \
                            halves, page_size, row_stride, max_pos, eps, err);                                             \
    else                                                                                                                   \
      prep_whole_body<T, 1>(qkv, cache, positions, slots, cos_tab, sin_tab, q_norm, k_norm, hq, hk, d, dv, v_col, rot,     \
                            halves, page_size, row_stride, max_pos, eps, err);                                             \
    pdl_launch_dependents();                                                                                               \
  }                                                                                                                        \
  WINDOW_ATTN(T, SFX, 64)                                                                                                  \
  WINDOW_ATTN(T, SFX, 128)                                                                                                 \
  WINDOW_ATTN(T, SFX, 256)                                                                                                 \
  WINDOW_ATTN(T, SFX, 512)                                                                                                 \
  POOLED_ATTN(T, SFX, 64)                                                                                                  \
  POOLED_ATTN(T, SFX, 128)                                                                                                 \
  POOLED_ATTN(T, SFX, 256)                                                                                                 \
  POOLED_ATTN(T, SFX, 512)

WINDOW_ENTRIES(__nv_bfloat16, bf16)
WINDOW_ENTRIES(float, f32)

// ---- the tensor-core bodies ------------------------------------------------------------------------------------------
#define WINDOW_TC(name, D, PREFILL)                                                                                        \
  extern "C" __global__ void __launch_bounds__(160, (PREFILL && D <= 128) ? 2 : 1)                                         \
      name(const __grid_constant__ CUtensorMap kv_map, const __nv_bfloat16* q, __nv_bfloat16* out, float* ws_o,            \
           float* ws_ml, const int* block_table, const int* seq_lens, const int* cu_q, const int* work,                    \
           const int* work_count, int hq, int hk, int q_stride, int out_stride, int max_pages, int page_size, int splits,  \
           int pool_pages, int* err, const __nv_bfloat16* sink, int window, float c1, float c2, float out_scale) {         \
    AttnArgs a{q, out, ws_o, ws_ml, block_table, seq_lens, cu_q, work, work_count, err, 0x7fffffff, hq, hk, q_stride,      \
               out_stride, max_pages, page_size, 1, splits, pool_pages, 1.f, {window, c1, c2, out_scale, sink}};           \
    attn_body<D, PREFILL, 0, kAttnWindow>(&kv_map, a, (int)blockIdx.y);                                                           \
  }
WINDOW_TC(kern_attn_window_decode_d64, 64, false)
WINDOW_TC(kern_attn_window_decode_d128, 128, false)
WINDOW_TC(kern_attn_window_decode_d256, 256, false)
WINDOW_TC(kern_attn_window_prefill_d64, 64, true)
WINDOW_TC(kern_attn_window_prefill_d128, 128, true)
WINDOW_TC(kern_attn_window_prefill_d256, 256, true)

// Both lists of a ragged call in one launch, as in attn_paged.cu: two CTAs per SM with a two-stage ring each.
#define WINDOW_RAGGED(name, D)                                                                                             \
  extern "C" __global__ void __launch_bounds__(160, 2)                                                                     \
      name(const __grid_constant__ CUtensorMap kv_map, const __nv_bfloat16* q, __nv_bfloat16* out, const int* block_table, \
           const int* seq_lens, const int* cu_q, const int* work_p, const int* count_p, const int* work_d,                 \
           const int* count_d, int hq, int hk, int q_stride, int out_stride, int max_pages, int page_size, int pool_pages, \
           int* err, const __nv_bfloat16* sink, int window, float c1, float c2, float out_scale) {                         \
    const int np = *count_p, nd = *count_d, m = np < nd ? np : nd;                                                         \
    const int y = blockIdx.y;                                                                                              \
    if (y >= np + nd) return;                                                                                              \
    const bool is_p = y < 2 * m ? !(y & 1) : np > nd;                                                                      \
    AttnArgs a{q, out, nullptr, nullptr, block_table, seq_lens, cu_q, is_p ? work_p : work_d, is_p ? count_p : count_d,    \
               err, 0x7fffffff, hq, hk, q_stride, out_stride, max_pages, page_size, 1, 1, pool_pages, 1.f,                 \
               {window, c1, c2, out_scale, sink}};                                                                         \
    const int idx = y < 2 * m ? (y >> 1) : y - m;                                                                          \
    if (is_p) attn_body<D, true, 2, kAttnWindow>(&kv_map, a, idx);                                                                \
    else attn_body<D, false, 2, kAttnWindow>(&kv_map, a, idx);                                                                    \
  }
WINDOW_RAGGED(kern_attn_window_ragged_d64, 64)
WINDOW_RAGGED(kern_attn_window_ragged_d128, 128)

// ---- the same over the whole causal reach ------------------------------------------------------------------------------
#define SINK_TC(name, D, PREFILL)                                                                                          \
  extern "C" __global__ void __launch_bounds__(160, (PREFILL && D <= 128) ? 2 : 1)                                         \
      name(const __grid_constant__ CUtensorMap kv_map, const __nv_bfloat16* q, __nv_bfloat16* out, float* ws_o,            \
           float* ws_ml, const int* block_table, const int* seq_lens, const int* cu_q, const int* work,                    \
           const int* work_count, int hq, int hk, int q_stride, int out_stride, int max_pages, int page_size, int splits,  \
           int pool_pages, int* err, const __nv_bfloat16* sink, const __nv_bfloat16* gate, int gate_stride,                \
           float scale_log2) {                                                                                             \
    AttnArgs a{q, out, ws_o, ws_ml, block_table, seq_lens, cu_q, work, work_count, err, 0x7fffffff, hq, hk, q_stride,      \
               out_stride, max_pages, page_size, 1, splits, pool_pages, scale_log2, {0, 0.f, 0.f, 1.f, sink, gate, gate_stride}}; \
    attn_body<D, PREFILL, 0, kAttnSink>(&kv_map, a, (int)blockIdx.y);                                                      \
  }
SINK_TC(kern_attn_sink_decode_d64, 64, false)
SINK_TC(kern_attn_sink_decode_d128, 128, false)
SINK_TC(kern_attn_sink_decode_d256, 256, false)
SINK_TC(kern_attn_sink_prefill_d64, 64, true)
SINK_TC(kern_attn_sink_prefill_d128, 128, true)
SINK_TC(kern_attn_sink_prefill_d256, 256, true)

#define SINK_RAGGED(name, D)                                                                                               \
  extern "C" __global__ void __launch_bounds__(160, 2)                                                                     \
      name(const __grid_constant__ CUtensorMap kv_map, const __nv_bfloat16* q, __nv_bfloat16* out, const int* block_table, \
           const int* seq_lens, const int* cu_q, const int* work_p, const int* count_p, const int* work_d,                 \
           const int* count_d, int hq, int hk, int q_stride, int out_stride, int max_pages, int page_size, int pool_pages, \
           int* err, const __nv_bfloat16* sink, const __nv_bfloat16* gate, int gate_stride, float scale_log2) {            \
    const int np = *count_p, nd = *count_d, m = np < nd ? np : nd;                                                         \
    const int y = blockIdx.y;                                                                                              \
    if (y >= np + nd) return;                                                                                              \
    const bool is_p = y < 2 * m ? !(y & 1) : np > nd;                                                                      \
    AttnArgs a{q, out, nullptr, nullptr, block_table, seq_lens, cu_q, is_p ? work_p : work_d, is_p ? count_p : count_d,    \
               err, 0x7fffffff, hq, hk, q_stride, out_stride, max_pages, page_size, 1, 1, pool_pages, scale_log2,          \
               {0, 0.f, 0.f, 1.f, sink, gate, gate_stride}};                                                               \
    const int idx = y < 2 * m ? (y >> 1) : y - m;                                                                          \
    if (is_p) attn_body<D, true, 2, kAttnSink>(&kv_map, a, idx);                                                           \
    else attn_body<D, false, 2, kAttnSink>(&kv_map, a, idx);                                                               \
  }
SINK_RAGGED(kern_attn_sink_ragged_d64, 64)
SINK_RAGGED(kern_attn_sink_ragged_d128, 128)

// ---- in a window beside the pooled rows before it ------------------------------------------------------------------------
#define POOLED_TC(name, D, PREFILL)                                                                                        \
  extern "C" __global__ void __launch_bounds__(160, (PREFILL && D <= 128) ? 2 : 1)                                         \
      name(const __grid_constant__ CUtensorMap kv_map, const __grid_constant__ CUtensorMap pool_map, const __nv_bfloat16* q, \
           __nv_bfloat16* out, float* ws_o, float* ws_ml, const int* block_table, const int* seq_lens, const int* cu_q,    \
           const int* work, const int* work_count, int hq, int hk, int q_stride, int out_stride, int max_pages,            \
           int page_size, int splits, int pool_pages, int* err, int window, int pool, int slots, float scale_log2) {       \
    AttnArgs a{q, out, ws_o, ws_ml, block_table, seq_lens, cu_q, work, work_count, err, 0x7fffffff, hq, hk, q_stride,      \
               out_stride, max_pages, page_size, 1, splits, pool_pages, scale_log2,                                        \
               {window, 0.f, 0.f, 1.f, nullptr, nullptr, 0, &pool_map, pool, slots}};                                      \
    attn_body<D, PREFILL, 0, kAttnPooled>(&kv_map, a, (int)blockIdx.y);                                                    \
  }
POOLED_TC(kern_attn_pooled_decode_d64, 64, false)
POOLED_TC(kern_attn_pooled_decode_d128, 128, false)
POOLED_TC(kern_attn_pooled_decode_d256, 256, false)
POOLED_TC(kern_attn_pooled_prefill_d64, 64, true)
POOLED_TC(kern_attn_pooled_prefill_d128, 128, true)
POOLED_TC(kern_attn_pooled_prefill_d256, 256, true)

#define POOLED_RAGGED(name, D)                                                                                             \
  extern "C" __global__ void __launch_bounds__(160, 2)                                                                     \
      name(const __grid_constant__ CUtensorMap kv_map, const __grid_constant__ CUtensorMap pool_map, const __nv_bfloat16* q, \
           __nv_bfloat16* out, const int* block_table, const int* seq_lens, const int* cu_q, const int* work_p,            \
           const int* count_p, const int* work_d, const int* count_d, int hq, int hk, int q_stride, int out_stride,        \
           int max_pages, int page_size, int pool_pages, int* err, int window, int pool, int slots, float scale_log2) {    \
    const int np = *count_p, nd = *count_d, m = np < nd ? np : nd;                                                         \
    const int y = blockIdx.y;                                                                                              \
    if (y >= np + nd) return;                                                                                              \
    const bool is_p = y < 2 * m ? !(y & 1) : np > nd;                                                                      \
    AttnArgs a{q, out, nullptr, nullptr, block_table, seq_lens, cu_q, is_p ? work_p : work_d, is_p ? count_p : count_d,    \
               err, 0x7fffffff, hq, hk, q_stride, out_stride, max_pages, page_size, 1, 1, pool_pages, scale_log2,          \
               {window, 0.f, 0.f, 1.f, nullptr, nullptr, 0, &pool_map, pool, slots}};                                      \
    const int idx = y < 2 * m ? (y >> 1) : y - m;                                                                          \
    if (is_p) attn_body<D, true, 2, kAttnPooled>(&kv_map, a, idx);                                                         \
    else attn_body<D, false, 2, kAttnPooled>(&kv_map, a, idx);                                                             \
  }
POOLED_RAGGED(kern_attn_pooled_ragged_d64, 64)
POOLED_RAGGED(kern_attn_pooled_ragged_d128, 128)

// Split keys without a sink, the finished rows times sigmoid of a gate per head, [row][gate_stride]. grid = rows x hq, block
// min(256, d).
extern "C" __global__ void kern_attn_gated_merge(const float* ws_o, const float* ws_ml, __nv_bfloat16* out,
                                                 const __nv_bfloat16* gate, int gate_stride, int rows, int hq, int d, int splits,
                                                 int out_stride) {
  pdl_wait();
  const int row = blockIdx.x;  // row * hq + head
  if (row >= rows) return;
  const int tk = row / hq, head = row % hq;
  float m = -INFINITY;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, ws_ml[((size_t)row * splits + s) * 2]);
  const float m_use = m == -INFINITY ? 0.f : m;
  float l = 0.f;
  for (int s = 0; s < splits; ++s) {
    const size_t b = (size_t)row * splits + s;
    l += ws_ml[b * 2 + 1] * exp2f(ws_ml[b * 2] - m_use);
  }
  const float f = l > 0.f ? gate_factor(__bfloat162float(gate[(size_t)tk * gate_stride + head])) / l : 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < splits; ++s) {
      const size_t b = (size_t)row * splits + s;
      acc += ws_o[b * d + c] * exp2f(ws_ml[b * 2] - m_use);
    }
    out[(size_t)tk * out_stride + (size_t)head * d + c] = __float2bfloat16(acc * f);
  }
}

// grid = rows x hq, block min(256, d); sink and gate as in AttnWindow
extern "C" __global__ void kern_attn_window_merge(const float* ws_o, const float* ws_ml, __nv_bfloat16* out,
                                                  const __nv_bfloat16* sink, const __nv_bfloat16* gate, int gate_stride, int rows,
                                                  int hq, int d, int splits, int out_stride, float out_scale) {
  pdl_wait();
  const int row = blockIdx.x;  // row * hq + head
  if (row >= rows) return;
  const int tk = row / hq, head = row % hq;
  float m = -INFINITY;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, ws_ml[((size_t)row * splits + s) * 2]);
  const float m_use = m == -INFINITY ? 0.f : m;
  float l = 0.f;
  for (int s = 0; s < splits; ++s) {
    const size_t b = (size_t)row * splits + s;
    l += ws_ml[b * 2 + 1] * exp2f(ws_ml[b * 2] - m_use);
  }
  const float f = sink_factor(m, l, sink ? __bfloat162float(sink[head]) : 0.f, out_scale);
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < splits; ++s) {
      const size_t b = (size_t)row * splits + s;
      acc += ws_o[b * d + c] * exp2f(ws_ml[b * 2] - m_use);
    }
    acc *= f;
    if (gate) acc *= gate_factor(__bfloat162float(gate[(size_t)tk * gate_stride + (size_t)head * d + c]));
    out[(size_t)tk * out_stride + (size_t)head * d + c] = __float2bfloat16(acc);
  }
}
