// build: precise
// Matrix products for what the tensor-core tiles do not take: 32-bit activations (a model's exact form), and sizes whose
// rows are not whole 16-byte vectors. C[M, N] = A[M, K] . W^T with W bf16 read through two strides (so a transposed view
// needs no copy), one 64 x 64 tile per block, f32 products and sums.
//   kern_linear_<act>[_f32 | _swiglu | _geglu | _clamped]   plain; blockIdx.z walks a batch (one weight, one column range of A and C per head)
//   kern_linear_grouped_<act>[_<gated unit>]           rows sorted by expert, the planner's tile table (tiles of at most 64 rows)
//   kern_rows_scatter_<act>                    x_perm[perm[i]] = x[i / k]
//   kern_gate_mul_<act>                        out = x * sigmoid(gate)
//   kern_transpose_heads_bf16                  [H][R][C] -> [H][C][R]
//   kern_copy_cols_bf16                        [R][C] into columns of wider rows
#include "act.cuh"

using namespace kern;

namespace {

constexpr int LB = 64, LK = 16;

// the gated units of common.cuh without the fast exponential; ACT < 0: none
template <int ACT>
KERN_DEVICE float glu_exact(float g, float u, float limit) {
  if constexpr (ACT == kGeglu) return g / (1.f + expf(-1.5957691216057308f * (g + 0.044715f * g * g * g))) * u;
  if constexpr (ACT == kClampedGlu) {
    g = fminf(g, limit);
    return g / (1.f + expf(-1.702f * g)) * (fmaxf(-limit, fminf(u, limit)) + 1.f);
  }
  return g / (1.f + expf(-g)) * u;
}

// rows [m0, m_end) of A, columns [n0, ..) of C; with a gated unit W holds N gate rows, then N up rows. `bias`: one per row of W
template <typename AT, typename OT, int ACT>
KERN_DEVICE void tile_body(const AT* A, const __nv_bfloat16* W, OT* C, int m0, int m_end, int n0, int N, int K, int lda,
                           int ldc, long long wsn, long long wsk, float limit = 0.f, const __nv_bfloat16* bias = nullptr) {
  constexpr bool SWIGLU = ACT >= 0;
  __shared__ float as[LK][LB + 4], ws[LK][LB + 4], us[SWIGLU ? LK : 1][LB + 4];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {}, acu[SWIGLU ? 4 : 1][4] = {};
  for (int k0 = 0; k0 < K; k0 += LK) {
    for (int i = threadIdx.x; i < LB * LK; i += 256) {
      const int r = i / LK, k = i % LK;
      as[k][r] = (k0 + k < K && m0 + r < m_end) ? ldf(A + (size_t)(m0 + r) * lda + k0 + k) : 0.f;
    }
    for (int i = threadIdx.x; i < LB * LK; i += 256) {
      const int r = wsk == 1 ? i / LK : i % LB, k = wsk == 1 ? i % LK : i / LB;
      const bool in = k0 + k < K && n0 + r < N;
      ws[k][r] = in ? __bfloat162float(W[(long long)(n0 + r) * wsn + (long long)(k0 + k) * wsk]) : 0.f;
      if constexpr (SWIGLU) us[k][r] = in ? __bfloat162float(W[(long long)(N + n0 + r) * wsn + (long long)(k0 + k) * wsk]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < LK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = as[k][ty * 4 + i]; b[i] = ws[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
      if constexpr (SWIGLU) {
#pragma unroll
        for (int j = 0; j < 4; ++j) b[j] = us[k][tx * 4 + j];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acu[i][j] += a[i] * b[j];
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= m_end || n >= N) continue;
      float v = acc[i][j];
      if (bias) v += __bfloat162float(bias[n]);
      if constexpr (SWIGLU) v = glu_exact<ACT>(v, acu[i][j] + (bias ? __bfloat162float(bias[N + n]) : 0.f), limit);
      stf(C + (size_t)m * ldc + n, v);
    }
}

// grid [columns / (256 V), rows]: a thread walks the rows blockIdx.y, + gridDim.y, .. of its columns
template <typename T, int V>
KERN_DEVICE void gate_mul_body(const T* x, const T* gate, T* out, int tokens, int d, int x_stride, int g_stride, int o_stride) {
  for (int t = blockIdx.y; t < tokens; t += gridDim.y)
    for (int c = (blockIdx.x * 256 + threadIdx.x) * V; c < d; c += gridDim.x * 256 * V) {
      const Vec<V> a = ldv<V>(x + (size_t)t * x_stride + c), g = ldv<V>(gate + (size_t)t * g_stride + c);
      Vec<V> o;
#pragma unroll
      for (int e = 0; e < V; ++e) o.v[e] = a.v[e] / (1.f + expf(-g.v[e]));
      stv<V>(out + (size_t)t * o_stride + c, o);
    }
}

}  // namespace

// grid [ceil(N / 64), ceil(M / 64), batch], block 256. Batch z: A + z a_z, W + z w_z, C + z c_z (elements).
#define LINEAR_ENTRY(NAME, AT, OT, ACT)                                                                                     \
  extern "C" __global__ void __launch_bounds__(256)                                                                         \
      NAME(const AT* A, const __nv_bfloat16* W, OT* C, int M, int N, int K, int lda, int ldc, long long wsn, long long wsk, \
           long long a_z, long long w_z, long long c_z, int* err, float limit, const __nv_bfloat16* bias) {                 \
    pdl_wait();                                                                                                             \
    if (M > (int)gridDim.y * LB && threadIdx.x == 0) set_error(err, ERR_BOUNDS);   /* rows the grid does not cover */       \
    const int z = blockIdx.z;                                                                                               \
    tile_body<AT, OT, ACT>(A + z * a_z, W + z * w_z, C + z * c_z, blockIdx.y * LB, M, blockIdx.x * LB, N, K, lda, ldc, wsn, \
                           wsk, limit, bias);                                                                               \
  }
// grid [ceil(N / 64), blocks], block 256; `tiles` int4 {expert, first row, rows, -}.
#define LINEAR_GROUPED_ENTRY(NAME, T, ACT)                                                                                  \
  extern "C" __global__ void __launch_bounds__(256)                                                                         \
      NAME(const T* A, const __nv_bfloat16* W, T* C, const int* tiles, const int* tile_count, int rows, int N, int K,       \
           long long w_z, int* err, float limit) {                                                                          \
    pdl_wait();                                                                                                             \
    const int n = *tile_count;                                                                                              \
    for (int i = blockIdx.y; i < n; i += gridDim.y) {                                                                       \
      const int4 e = reinterpret_cast<const int4*>(tiles)[i];                                                               \
      if (e.y + e.z > rows || e.z > LB) { if (threadIdx.x == 0) set_error(err, ERR_BOUNDS); continue; }                     \
      tile_body<T, T, ACT>(A, W + e.x * w_z, C, e.y, e.y + e.z, blockIdx.x * LB, N, K, K, N, K, 1, limit);                  \
    }                                                                                                                       \
  }
#define LINEAR_MISC(T, SFX)                                                                                                 \
  extern "C" __global__ void __launch_bounds__(256)                                                                         \
      kern_rows_scatter_##SFX(const T* x, const int* perm, T* x_perm, int entries, int k, int width) {                      \
    pdl_wait();                                                                                                             \
    const int i = blockIdx.x;                                                                                               \
    if (i >= entries) return;                                                                                               \
    const int r = perm[i];                                                                                                  \
    if (r < 0 || !KERN_CHECK(x_perm + (size_t)r * width, (size_t)width * sizeof(T), SITE_MOE_GATHER)) return;               \
    for (int c = threadIdx.x; c < width; c += 256) x_perm[(size_t)r * width + c] = x[(size_t)(i / k) * width + c];          \
  }                                                                                                                         \
  extern "C" __global__ void __launch_bounds__(256)                                                                         \
      kern_gate_mul_##SFX(const T* x, const T* gate, T* out, int tokens, int d, int x_stride, int g_stride, int o_stride) { \
    pdl_wait();                                                                                                             \
    const bool vec = (d | x_stride | g_stride | o_stride) % 4 == 0 &&                                                       \
                     ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) & 15) == 0; \
    if (vec) gate_mul_body<T, 4>(x, gate, out, tokens, d, x_stride, g_stride, o_stride);                                    \
    else gate_mul_body<T, 1>(x, gate, out, tokens, d, x_stride, g_stride, o_stride);                                        \
  }

LINEAR_ENTRY(kern_linear_bf16, __nv_bfloat16, __nv_bfloat16, -1)
LINEAR_ENTRY(kern_linear_bf16_f32, __nv_bfloat16, float, -1)
LINEAR_ENTRY(kern_linear_f32, float, float, -1)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_bf16, __nv_bfloat16, -1)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_f32, float, -1)
#define LINEAR_GLU(SFX, ACT)                                                            \
  LINEAR_ENTRY(kern_linear_bf16_##SFX, __nv_bfloat16, __nv_bfloat16, ACT)               \
  LINEAR_ENTRY(kern_linear_f32_##SFX, float, float, ACT)
LINEAR_GLU(swiglu, kSwiglu)
LINEAR_GLU(geglu, kGeglu)
LINEAR_GLU(clamped, kClampedGlu)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_bf16_swiglu, __nv_bfloat16, kSwiglu)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_f32_swiglu, float, kSwiglu)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_bf16_geglu, __nv_bfloat16, kGeglu)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_f32_geglu, float, kGeglu)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_bf16_clamped, __nv_bfloat16, kClampedGlu)
LINEAR_GROUPED_ENTRY(kern_linear_grouped_f32_clamped, float, kClampedGlu)
LINEAR_MISC(__nv_bfloat16, bf16)
LINEAR_MISC(float, f32)

// grid [ceil(C / 32), ceil(R / 32), H], block 256.
extern "C" __global__ void __launch_bounds__(256)
    kern_transpose_heads_bf16(const __nv_bfloat16* src, __nv_bfloat16* dst, int R, int C) {
  __shared__ __nv_bfloat16 tile[32][33];
  pdl_wait();
  const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5;
  const size_t base = (size_t)blockIdx.z * R * C;
  for (int j = ty; j < 32; j += 8) {
    const int r = blockIdx.y * 32 + j, c = blockIdx.x * 32 + tx;
    if (r < R && c < C) tile[j][tx] = src[base + (size_t)r * C + c];
  }
  __syncthreads();
  for (int j = ty; j < 32; j += 8) {
    const int c = blockIdx.x * 32 + j, r = blockIdx.y * 32 + tx;
    if (r < R && c < C) dst[base + (size_t)c * R + r] = tile[tx][j];
  }
}

// dst[r, 0 .. C) of rows `stride` elements apart. grid [rows], block 256.
extern "C" __global__ void __launch_bounds__(256)
    kern_copy_cols_bf16(const __nv_bfloat16* src, __nv_bfloat16* dst, int C, int stride) {
  pdl_wait();
  for (int c = threadIdx.x; c < C; c += 256) dst[(size_t)blockIdx.x * stride + c] = src[(size_t)blockIdx.x * C + c];
}
