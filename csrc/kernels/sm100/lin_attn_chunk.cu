// build: precise
// Linear attention with a decay per key channel over prompts, sixteen tokens at a time on the tensor cores (lin_attn.cu
// holds the token-by-token form, the equations and the state line's layout). Inside a chunk, with P_i = alpha_1 .. alpha_i
// per key channel:
//     o_i = S^T (P_i q_i) + sum_{j <= i} A_ij v_j,   A_ij = sum_c q_i[c] k_j[c] alpha_(j+1) .. alpha_i
//     S  <- diag(P_16) S + sum_j (alpha_(j+1) .. alpha_16 k_j) v_j^T
// and with a bonus u the same with P_(i-1), the product of A_ij ending at i - 1, and A_ii = sum_c q_i[c] u[c] k_i[c]. Every
// decay enters as a running product of at most sixteen factors <= 1: no logarithm, no quotient, nothing that can overflow.
//
// A CTA owns 64 value columns of one head of one sequence and walks its chunks in order. Warps 4..7 prepare chunk i + 1
// (the scaled q and k, the pair matrix A, all from shared memory) while warps 0..3 run the MMAs of chunk i; each MMA warp
// holds S^T for its 16 value columns as f32 accumulators over the whole prompt. v is bf16 and enters exactly; a factor
// that is f32 enters as bf16 terms: the state's update and A as three (24 bits), the state's read as two times two (the
// product of the low parts left out). Raw q, k, alpha and v of chunk i + 2 are in flight (cp.async) meanwhile.
// NP: key channels padded to 32 / 64 / 128 / 256. Sequences with fewer than `min_rows` rows are left to lin_attn.cu.
#include "act.cuh"

using namespace kern;

namespace {

constexpr int Q = 16, VT = 64, VS = VT + 8, AS = Q + 8;

KERN_DEVICE void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
KERN_DEVICE void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
KERN_DEVICE void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
KERN_DEVICE void cp16(uint32_t dst, const void* src, bool in) {      // 16 bytes, zeros when `in` is false
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
// (u, v) as two bf16 pairs; the remainder is left out
KERN_DEVICE void split2(float u, float v, uint32_t& a, uint32_t& b) {
  a = pack_bf16x2(u, v);
  const float2 h = unpack_bf16x2(a);
  b = pack_bf16x2(u - h.x, v - h.y);
}
KERN_DEVICE void put2(__nv_bfloat16* hi, __nv_bfloat16* lo, float u) {
  *hi = __float2bfloat16(u);
  *lo = __float2bfloat16(u - __bfloat162float(*hi));
}

template <int NP>
struct LinCfg {
  static constexpr int KS = NP + 8;                                         // row stride of the prepared q and k
  static constexpr int kPrep = 5 * Q * KS * 2 + 3 * Q * AS * 2 + NP * 4;    // q hi, lo; k 3 terms; A 3 terms; P_16
  static constexpr int kRaw = Q * NP * (2 + 2 + 4);                         // q, k bf16, alpha f32
  static constexpr int kV = Q * VS * 2;
  static constexpr int kBytes = 2 * kPrep + 2 * kRaw + 3 * kV + NP * 4;     // + u
  static_assert(kBytes <= 227 * 1024, "shared memory of one CTA");
};

struct ChunkArgs {
  const __nv_bfloat16 *q, *k, *v;
  const float* alpha;
  const __nv_bfloat16* u;
  float* out;
  uint8_t* state;
  const int *lines, *cu;
  int seqs, H, dk, dv, stride, s_off, min_rows;
  long long line_bytes;
  float q_scale;
};

template <int NP, bool BONUS>
KERN_DEVICE void chunk_body(const ChunkArgs& a) {
  using Cfg = LinCfg<NP>;
  constexpr int KS = Cfg::KS, NT = NP / 8;
  extern __shared__ __align__(16) uint8_t lin_sm[];
  uint8_t* prep0 = lin_sm;
  uint8_t* raw0 = prep0 + 2 * Cfg::kPrep;
  __nv_bfloat16* v0s = reinterpret_cast<__nv_bfloat16*>(raw0 + 2 * Cfg::kRaw);
  float* us = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(v0s) + 3 * Cfg::kV);
  const int tiles = (a.dv + VT - 1) / VT;
  const int h = blockIdx.x / tiles, c0 = (blockIdx.x % tiles) * VT, s = blockIdx.y;
  if (s >= a.seqs) return;
  const int r0 = a.cu[s], r1 = a.cu[s + 1], dk = a.dk, dv = a.dv;
  if (r1 - r0 < a.min_rows) return;
  int line = a.lines[s];
  if (line > 0 && !KERN_CHECK(a.state + (size_t)line * a.line_bytes, (size_t)a.line_bytes, SITE_STATE_SLOT)) line = 0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const __nv_bfloat16* qg = a.q + (size_t)h * dk;
  const __nv_bfloat16* kg = a.k + (size_t)h * dk;
  const __nv_bfloat16* vg = a.v + (size_t)h * dv + c0;
  const float* ag = a.alpha + (size_t)h * dk;
  const size_t a_stride = (size_t)a.H * dk;
  const bool vec = (dk | dv | a.stride) % 8 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k) | reinterpret_cast<uintptr_t>(a.v) |
                     reinterpret_cast<uintptr_t>(a.alpha)) & 15) == 0;
  const int chunks = (r1 - r0 + Q - 1) / Q;

  // q, k, alpha, v of chunk i; tokens and channels past the end are zeros (alpha is set to 1 when it is used)
  auto load = [&](int i) {
    const int base = r0 + i * Q, nb = min(Q, r1 - base);
    uint8_t* raw = raw0 + (i & 1) * Cfg::kRaw;
    __nv_bfloat16* rq = reinterpret_cast<__nv_bfloat16*>(raw);
    __nv_bfloat16* rk = rq + Q * NP;
    float* ra = reinterpret_cast<float*>(rk + Q * NP);
    __nv_bfloat16* rv = v0s + (i % 3) * (Q * VS);
    if (vec) {
      for (int x = tid; x < Q * (NP / 8); x += 256) {
        const int t = x / (NP / 8), c = (x % (NP / 8)) * 8;
        const bool in = t < nb && c < dk;
        const size_t at = (size_t)(in ? base + t : base) * a.stride + (in ? c : 0);
        cp16(smem_u32(rq + t * NP + c), qg + at, in);
        cp16(smem_u32(rk + t * NP + c), kg + at, in);
      }
      for (int x = tid; x < Q * (NP / 4); x += 256) {
        const int t = x / (NP / 4), c = (x % (NP / 4)) * 4;
        const bool in = t < nb && c < dk;
        cp16(smem_u32(ra + t * NP + c), ag + (size_t)(in ? base + t : base) * a_stride + (in ? c : 0), in);
      }
      if (tid < Q * (VT / 8)) {
        const int t = tid / (VT / 8), c = (tid % (VT / 8)) * 8;
        const bool in = t < nb && c0 + c < dv;
        cp16(smem_u32(rv + t * VS + c), vg + (size_t)(in ? base + t : base) * a.stride + (in ? c : 0), in);
      }
    } else {
      const __nv_bfloat16 zero = __float2bfloat16(0.f);
      for (int x = tid; x < Q * NP; x += 256) {
        const int t = x / NP, c = x % NP;
        const bool in = t < nb && c < dk;
        rq[x] = in ? qg[(size_t)(base + t) * a.stride + c] : zero;
        rk[x] = in ? kg[(size_t)(base + t) * a.stride + c] : zero;
        ra[x] = in ? ag[(size_t)(base + t) * a_stride + c] : 0.f;
      }
      for (int x = tid; x < Q * VT; x += 256) {
        const int t = x / VT, c = x % VT;
        rv[t * VS + c] = (t < nb && c0 + c < dv) ? vg[(size_t)(base + t) * a.stride + c] : zero;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // ---- warps 4..7: chunk i from its raw rows into its prepared stage ----
  auto prepare = [&](int i) {
    const int nb = min(Q, r1 - (r0 + i * Q)), p = tid - 128;
    const uint8_t* raw = raw0 + (i & 1) * Cfg::kRaw;
    const __nv_bfloat16* rq = reinterpret_cast<const __nv_bfloat16*>(raw);
    const __nv_bfloat16* rk = rq + Q * NP;
    const float* ra = reinterpret_cast<const float*>(rk + Q * NP);
    uint8_t* st = prep0 + (i & 1) * Cfg::kPrep;
    __nv_bfloat16* pq = reinterpret_cast<__nv_bfloat16*>(st);      // [2][Q][KS]
    __nv_bfloat16* pk = pq + 2 * Q * KS;                           // [3][Q][KS]
    __nv_bfloat16* pa = pk + 3 * Q * KS;                           // [3][Q][AS]
    float* dec = reinterpret_cast<float*>(pa + 3 * Q * AS);        // [NP]
    for (int c = p; c < NP; c += 128) {
      float run = 1.f;
#pragma unroll
      for (int t = 0; t < Q; ++t) {
        const float al = t < nb ? ra[t * NP + c] : 1.f;
        const float x = __bfloat162float(rq[t * NP + c]) * a.q_scale;
        if constexpr (!BONUS) run *= al;
        put2(pq + t * KS + c, pq + Q * KS + t * KS + c, x * run);
        if constexpr (BONUS) run *= al;
      }
      dec[c] = run;
      run = 1.f;
#pragma unroll
      for (int t = Q - 1; t >= 0; --t) {
        const float al = t < nb ? ra[t * NP + c] : 1.f;
        const float x = __bfloat162float(rk[t * NP + c]) * run;
        const __nv_bfloat16 hi = __float2bfloat16(x);
        const float rest = x - __bfloat162float(hi);
        pk[t * KS + c] = hi;
        put2(pk + Q * KS + t * KS + c, pk + 2 * Q * KS + t * KS + c, rest);
        run *= al;
      }
    }
    // the pair matrix: a warp takes the tokens j = w, 7 - w, 8 + w, 15 - w; a lane the channel pairs 2 lane + 64 m (or one
    // channel each of 32)
    const int w = warp - 4;
#pragma unroll 1
    for (int jj = 0; jj < 4; ++jj) {
      const int j = jj == 0 ? w : (jj == 1 ? 7 - w : (jj == 2 ? 8 + w : 15 - w));
      float acc[Q];
#pragma unroll
      for (int t = 0; t < Q; ++t) acc[t] = 0.f;
#pragma unroll
      for (int m = 0; m < (NP + 63) / 64; ++m) {
        float2 kr;
        const int c = NP >= 64 ? 2 * lane + 64 * m : lane;
        if constexpr (NP >= 64) kr = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(rk + j * NP + c));
        else kr = make_float2(__bfloat162float(rk[j * NP + c]), 0.f);
        float2 run = kr;
#pragma unroll
        for (int t = 0; t < Q; ++t) {
          if (t < j) continue;
          float2 x, al;
          if constexpr (NP >= 64) {
            x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(rq + t * NP + c));
            al = *reinterpret_cast<const float2*>(ra + t * NP + c);
          } else {
            x = make_float2(__bfloat162float(rq[t * NP + c]), 0.f);
            al = make_float2(ra[t * NP + c], 0.f);
          }
          if (t >= nb) al = make_float2(1.f, 1.f);
          if constexpr (BONUS) {
            if (t == j) {
              acc[t] += x.x * us[c] * kr.x + (NP >= 64 ? x.y * us[NP >= 64 ? c + 1 : c] * kr.y : 0.f);
            } else {
              acc[t] += x.x * run.x + x.y * run.y;
              run.x *= al.x; run.y *= al.y;
            }
          } else {
            if (t > j) { run.x *= al.x; run.y *= al.y; }
            acc[t] += x.x * run.x + x.y * run.y;
          }
        }
      }
      // sixteen sums over 32 lanes: halve the values a lane carries at every step; lane l ends with token (l >> 1)'s sum
#pragma unroll
      for (int o = 16, n = 8; n >= 1; o >>= 1, n >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int t = 0; t < n; ++t) {
          const float send = up ? acc[t] : acc[t + n];
          const float keep = up ? acc[t + n] : acc[t];
          acc[t] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
      }
      const float sum = (acc[0] + __shfl_xor_sync(0xffffffffu, acc[0], 1)) * a.q_scale;
      if ((lane & 1) == 0) {
        const int t = lane >> 1;      // A[t][j]; zero above the diagonal
        const __nv_bfloat16 hi = __float2bfloat16(sum);
        pa[t * AS + j] = hi;
        put2(pa + Q * AS + t * AS + j, pa + 2 * Q * AS + t * AS + j, sum - __bfloat162float(hi));
      }
    }
  };

  // ---- warps 0..3: S^T of 16 value columns, rows v = lane / 4 (+ 8), columns 8 i + 2 (lane % 4) (+ 1) ----
  const int vw = (warp & 3) * 16;
  float S[NT][4];
  float* Sg = reinterpret_cast<float*>(a.state + (size_t)line * a.line_bytes + a.s_off) + (size_t)h * dk * dv + c0;
  auto s_at = [&](int i, int e, int& c, int& v) {
    v = vw + (lane >> 2) + (e >> 1) * 8;
    c = i * 8 + 2 * (lane & 3) + (e & 1);
    return c < dk && c0 + v < dv;
  };
  auto run = [&](int i) {
    const int base = r0 + i * Q, nb = min(Q, r1 - base);
    const uint8_t* st = prep0 + (i & 1) * Cfg::kPrep;
    const __nv_bfloat16* pq = reinterpret_cast<const __nv_bfloat16*>(st);
    const __nv_bfloat16* pk = pq + 2 * Q * KS;
    const __nv_bfloat16* pa = pk + 3 * Q * KS;
    const float* dec = reinterpret_cast<const float*>(pa + 3 * Q * AS);
    const __nv_bfloat16* rv = v0s + (i % 3) * (Q * VS);
    float O[2][4] = {}, X[2][4] = {};      // hi x hi, and the cross terms
    const uint32_t q_addr = smem_u32(pq + ((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk) {
      uint32_t sh[4], sl[4], qh[4], ql[4];
      split2(S[2 * kk][0], S[2 * kk][1], sh[0], sl[0]);
      split2(S[2 * kk][2], S[2 * kk][3], sh[1], sl[1]);
      split2(S[2 * kk + 1][0], S[2 * kk + 1][1], sh[2], sl[2]);
      split2(S[2 * kk + 1][2], S[2 * kk + 1][3], sh[3], sl[3]);
      ldsm4(q_addr + kk * 32, qh);
      ldsm4(q_addr + kk * 32 + Q * KS * 2, ql);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        mma(O[n], sh, qh[2 * n], qh[2 * n + 1]);
        mma(X[n], sl, qh[2 * n], qh[2 * n + 1]);
        mma(X[n], sh, ql[2 * n], ql[2 * n + 1]);
      }
    }
    uint32_t vt[4];
    ldsm4_t(smem_u32(rv + ((lane & 7) + (lane >> 4) * 8) * VS + vw + ((lane >> 3) & 1) * 8), vt);
    const uint32_t a_addr = smem_u32(pa + ((lane & 7) + (lane >> 4) * 8) * AS + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int z = 2; z >= 0; --z) {
      uint32_t b[4];
      ldsm4(a_addr + z * Q * AS * 2, b);
      mma(z ? X[0] : O[0], vt, b[0], b[1]);
      mma(z ? X[1] : O[1], vt, b[2], b[3]);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = vw + (lane >> 2) + (e >> 1) * 8, t = n * 8 + 2 * (lane & 3) + (e & 1);
        if (t < nb && c0 + v < dv) a.out[((size_t)(base + t) * a.H + h) * dv + c0 + v] = O[n][e] + X[n][e];
      }
    // the state after the chunk
    const uint32_t k_addr = smem_u32(pk + ((lane & 7) + ((lane >> 3) & 1) * 8) * KS + (lane >> 4) * 8);
#pragma unroll
    for (int i2 = 0; i2 < NT; i2 += 2) {
      const float2 d0 = *reinterpret_cast<const float2*>(dec + i2 * 8 + 2 * (lane & 3));
      const float2 d1 = *reinterpret_cast<const float2*>(dec + i2 * 8 + 8 + 2 * (lane & 3));
      S[i2][0] *= d0.x; S[i2][1] *= d0.y; S[i2][2] *= d0.x; S[i2][3] *= d0.y;
      S[i2 + 1][0] *= d1.x; S[i2 + 1][1] *= d1.y; S[i2 + 1][2] *= d1.x; S[i2 + 1][3] *= d1.y;
#pragma unroll
      for (int z = 2; z >= 0; --z) {
        uint32_t b[4];
        ldsm4_t(k_addr + (z * Q * KS + i2 * 8) * 2, b);
        mma(S[i2], vt, b[0], b[1]);
        mma(S[i2 + 1], vt, b[2], b[3]);
      }
    }
  };

  for (int c = tid; c < NP; c += 256) us[c] = (BONUS && c < dk) ? __bfloat162float(a.u[(size_t)h * dk + c]) : 0.f;
  load(0);
  if (chunks > 1) {
    load(1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
  } else {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
  }
  __syncthreads();
  if (warp >= 4) {
    prepare(0);
  } else {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int c, v;
        S[i][e] = (s_at(i, e, c, v) && line > 0) ? Sg[(size_t)c * dv + v] : 0.f;
      }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();      // chunk 0 is prepared, chunk 1 is here
#pragma unroll 1
  for (int i = 0; i < chunks; ++i) {
    if (i + 2 < chunks) load(i + 2);      // into the raw rows of chunk i, which nobody reads any more, and a third v stage
    if (warp >= 4) {
      if (i + 1 < chunks) prepare(i + 1);
    } else {
      run(i);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
  }
  if (warp < 4 && line > 0) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int c, v;
        if (s_at(i, e, c, v)) Sg[(size_t)c * dv + v] = S[i][e];
      }
  }
}

}  // namespace

// grid [H ceil(dv / 64), seqs], block 256, LinCfg<NP>::kBytes of shared memory.
#define LIN_CHUNK(NP)                                                                                                     \
  extern "C" __global__ void __launch_bounds__(256)                                                                       \
      kern_lin_chunk_n##NP(const __nv_bfloat16* q, const __nv_bfloat16* k, const __nv_bfloat16* v, const float* alpha,    \
                           const __nv_bfloat16* u, float* out, uint8_t* state, const int* lines, const int* cu, int seqs, \
                           int H, int dk, int dv, int stride, long long line_bytes, int s_off, int min_rows,              \
                           float q_scale) {                                                                               \
    pdl_wait();                                                                                                           \
    const ChunkArgs a{q, k, v, alpha, u, out, state, lines, cu, seqs, H, dk, dv, stride, s_off, min_rows, line_bytes, q_scale}; \
    if (u) chunk_body<NP, true>(a);                                                                                       \
    else chunk_body<NP, false>(a);                                                                                        \
    pdl_launch_dependents();                                                                                              \
  }

LIN_CHUNK(32)
LIN_CHUNK(64)
LIN_CHUNK(128)
LIN_CHUNK(256)
