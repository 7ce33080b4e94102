// build: precise
// Latent attention whose keys and values are both linear maps of one cached row per token (no rotated part), in the
// absorbed form: per head, score = (W_uk^T q) . c, and the weighted sum of the rows c goes through W_uv afterwards. These
// kernels take any latent width and either activation type; mla_decode.cu holds the tensor-core form.
//   kern_latent_append_<act>   RMS norm of a token's latent, written to its row of the paged cache
//   kern_latent_attn_<act>     one (row, head) per block: softmax over the row's causal reach, f32 throughout
#include "act.cuh"

using namespace kern;

namespace {

template <typename T>
KERN_DEVICE void append_body(const T* lat, uint8_t* cache, const long long* slots, const __nv_bfloat16* w, int rank, int stride,
                             float eps) {
  __shared__ float part[4];
  const int t = blockIdx.x;
  const long long slot = slots[t];
  if (slot < 0) return;
  const T* x = lat + (size_t)t * stride;
  float ss = 0.f;
  for (int i = threadIdx.x; i < rank; i += 128) { const float v = ldf(x + i); ss += v * v; }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float inv = 1.f / sqrtf((part[0] + part[1] + part[2] + part[3]) / (float)rank + eps);
  T* dst = reinterpret_cast<T*>(cache) + (size_t)slot * rank;
  if (!KERN_CHECK(dst, (size_t)rank * sizeof(T), SITE_KV_APPEND)) return;
  for (int i = threadIdx.x; i < rank; i += 128) stf(dst + i, ldf(x + i) * inv * __bfloat162float(w[i]));
}

// Four warps walk the keys (key j belongs to warp j % 4); a lane holds the columns i * 32 + lane of the query and of the
// warp's running sum. RL = columns per lane.
template <typename T, int RL>
KERN_DEVICE void attn_body(const T* q, const uint8_t* cache, T* out, const int* table, const int* lens, const int* row_seq,
                           int heads, int rank, int max_pages, int page, float scale, int* err) {
  extern __shared__ __align__(16) float lat_sm[];      // [4][rank] partial sums, then [4] maxima, [4] weights
  const int h = blockIdx.x, r = blockIdx.y;
  const int L = lens[r];
  if (L <= 0) return;
  if (L > max_pages * page && threadIdx.x == 0) set_error(err, ERR_BOUNDS);     // keys past the table row are left out
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* pages = table + (size_t)(row_seq ? row_seq[r] : r) * max_pages;
  const T* rows = reinterpret_cast<const T*>(cache);
  const T* qr = q + ((size_t)r * heads + h) * rank;
  float qv[RL], o[RL];
#pragma unroll
  for (int i = 0; i < RL; ++i) {
    const int c = i * 32 + lane;
    qv[i] = c < rank ? ldf(qr + c) : 0.f;
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int j = warp; j < L; j += 4) {
    const int pi = j / page;
    if (pi >= max_pages) break;
    const T* row = rows + ((size_t)pages[pi] * page + j % page) * rank;
    if (!KERN_CHECK(row, (size_t)rank * sizeof(T), SITE_LATENT_ROW)) continue;
    float c[RL], s = 0.f;
#pragma unroll
    for (int i = 0; i < RL; ++i) {
      const int k = i * 32 + lane;
      c[i] = k < rank ? ldf(row + k) : 0.f;
      s += qv[i] * c[i];
    }
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
  const float mx = fmaxf(fmaxf(ms[0], ms[1]), fmaxf(ms[2], ms[3]));
  float f[4], den = 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) { f[w] = expf(ms[w] - mx); den += f[w] * ls[w]; }
  for (int c = threadIdx.x; c < rank; c += 128) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += f[w] * acc[w * rank + c];
    stf(out + ((size_t)r * heads + h) * rank + c, v / den);
  }
}

}  // namespace

// append: grid = tokens, block 128. attn: grid [heads, rows], block 128, (4 rank + 8) floats of shared memory.
#define LATENT_ATTN(T, SFX, W)                                                                                            \
  extern "C" __global__ void __launch_bounds__(128)                                                                       \
      kern_latent_attn_##SFX##_w##W(const T* q, const uint8_t* cache, T* out, const int* table, const int* lens,          \
                                    const int* row_seq, int heads, int rank, int max_pages, int page, float scale,        \
                                    int* err) {                                                                           \
    pdl_wait();                                                                                                           \
    attn_body<T, W / 32>(q, cache, out, table, lens, row_seq, heads, rank, max_pages, page, scale, err);                  \
  }
#define LATENT_ENTRIES(T, SFX)                                                                                            \
  extern "C" __global__ void __launch_bounds__(128)                                                                       \
      kern_latent_append_##SFX(const T* lat, uint8_t* cache, const long long* slots, const __nv_bfloat16* w, int rank,    \
                               int stride, float eps) {                                                                   \
    pdl_wait();                                                                                                           \
    append_body<T>(lat, cache, slots, w, rank, stride, eps);                                                              \
  }                                                                                                                       \
  LATENT_ATTN(T, SFX, 64)                                                                                                 \
  LATENT_ATTN(T, SFX, 128)                                                                                                \
  LATENT_ATTN(T, SFX, 256)                                                                                                \
  LATENT_ATTN(T, SFX, 512)                                                                                                \
  LATENT_ATTN(T, SFX, 1024)

LATENT_ENTRIES(__nv_bfloat16, bf16)
LATENT_ENTRIES(float, f32)
