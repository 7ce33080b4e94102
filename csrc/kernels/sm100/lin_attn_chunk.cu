// build: precise
// Linear attention with a decay per key channel over prompts, sixteen tokens at a time on the tensor cores (lin_attn.cu
// holds the token-by-token form, the equations and the state line's layout). Inside a chunk, with P_i = alpha_1 .. alpha_i
// per key channel:
//     o_i = S^T (P_i q_i) + sum_{j <= i} A_ij v_j,   A_ij = sum_c q_i[c] k_j[c] alpha_(j+1) .. alpha_i
//     S  <- diag(P_16) S + sum_j (alpha_(j+1) .. alpha_16 k_j) v_j^T
// and with a bonus u the same with P_(i-1), the product of A_ij ending at i - 1, and A_ii = sum_c q_i[c] u[c] k_i[c]. Every
// decay enters as a running product of at most sixteen factors <= 1: no logarithm, no quotient, nothing that can overflow.
//
// kern_lin_prep_*   a CTA per (chunk, head): the scaled q and k and the pair matrix A, as the bf16 terms the MMAs take, one
//                   block of kPrep bytes per chunk and head. Chunk i of sequence s is slot cu[s] / 16 + s + i: distinct for all
//                   chunks of a call, without a scan over the sequences.
// kern_lin_chunk_*  a CTA owns 64 value columns of one head of one sequence and walks its chunks in order; each of its four
//                   warps holds S^T for 16 value columns as f32 accumulators over the whole prompt. The next three chunks are in
//                   flight (cp.async) meanwhile.
// v is bf16 and enters exactly; a factor that is f32 enters as bf16 terms: the state's update and A as three (24 bits), the
// state's read as two times two (the product of the low parts left out).
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
KERN_DEVICE void split3(float u, float v, uint32_t& a, uint32_t& b, uint32_t& c) {      // as three, with all of their 24 bits
  a = pack_bf16x2(u, v);
  const float2 h = unpack_bf16x2(a);
  split2(u - h.x, v - h.y, b, c);
}

template <int NP>
struct LinCfg {
  static constexpr int KS = NP + 8;                                         // row stride of the prepared q and k
  static constexpr int kPrep = 5 * Q * KS * 2 + 3 * Q * AS * 2 + NP * 4;    // q hi, lo; k 3 terms; A 3 terms; P_16
  static constexpr int kV = Q * VS * 2;
  static constexpr int kStages = 4;
  static constexpr int kRaw = Q * NP * (2 + 2 + 4) + NP * 4;                // q, k bf16, alpha f32; u
  static_assert(kRaw <= 48 * 1024 && kStages * (kPrep + kV) <= 227 * 1024, "shared memory of one CTA");
};

struct ChunkArgs {
  const __nv_bfloat16 *q, *k, *v;
  const float* alpha;
  const __nv_bfloat16* u;
  uint8_t* prep;
  float* out;
  uint8_t* state;
  const int *lines, *cu;
  int seqs, H, dk, dv, stride, s_off, min_rows, slots;
  long long line_bytes;
  float q_scale;
};

KERN_DEVICE int slot_of(const int* cu, int s) { return cu[s] / Q + s; }

// block 128, kRaw bytes of shared memory
template <int NP, bool BONUS>
KERN_DEVICE void prep_body(const ChunkArgs& a) {
  using Cfg = LinCfg<NP>;
  constexpr int KS = Cfg::KS;
  extern __shared__ __align__(16) uint8_t lin_sm[];
  const int slot = blockIdx.x, h = blockIdx.y, p = threadIdx.x, dk = a.dk;
  int s = 0;
  {      // the last sequence whose slots start at or before this one
    int hi = a.seqs - 1;
    while (s < hi) {
      const int mid = (s + hi + 1) >> 1;
      if (slot_of(a.cu, mid) <= slot) s = mid; else hi = mid - 1;
    }
  }
  const int r0 = a.cu[s], r1 = a.cu[s + 1], base = r0 + (slot - slot_of(a.cu, s)) * Q;
  if (slot < slot_of(a.cu, s) || base >= r1 || r1 - r0 < a.min_rows) return;
  const int nb = min(Q, r1 - base);
  __nv_bfloat16* rq = reinterpret_cast<__nv_bfloat16*>(lin_sm);
  __nv_bfloat16* rk = rq + Q * NP;
  float* ra = reinterpret_cast<float*>(rk + Q * NP);
  float* us = ra + Q * NP;
  const __nv_bfloat16* qg = a.q + (size_t)h * dk;
  const __nv_bfloat16* kg = a.k + (size_t)h * dk;
  const float* ag = a.alpha + (size_t)h * dk;
  const size_t a_stride = (size_t)a.H * dk;
  const bool vec = (dk | a.stride) % 8 == 0 && ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k) |
                                                 reinterpret_cast<uintptr_t>(a.alpha)) & 15) == 0;
  // tokens past the end: q = k = 0, alpha = 1; channels past the end: zeros
  if (vec) {
    const uint4 zero = make_uint4(0, 0, 0, 0);
    for (int x = p; x < Q * (NP / 8); x += 128) {
      const int t = x / (NP / 8), c = (x % (NP / 8)) * 8;
      const bool in = t < nb && c < dk;
      const size_t at = (size_t)(base + t) * a.stride + c;
      reinterpret_cast<uint4*>(rq)[x] = in ? *reinterpret_cast<const uint4*>(qg + at) : zero;
      reinterpret_cast<uint4*>(rk)[x] = in ? *reinterpret_cast<const uint4*>(kg + at) : zero;
    }
    for (int x = p; x < Q * (NP / 4); x += 128) {
      const int t = x / (NP / 4), c = (x % (NP / 4)) * 4;
      const float e = t < nb ? 0.f : 1.f;
      reinterpret_cast<float4*>(ra)[x] = (t < nb && c < dk) ? *reinterpret_cast<const float4*>(ag + (size_t)(base + t) * a_stride + c) : make_float4(e, e, e, e);
    }
  } else {
    const __nv_bfloat16 zero = __float2bfloat16(0.f);
    for (int x = p; x < Q * NP; x += 128) {
      const int t = x / NP, c = x % NP;
      const bool in = t < nb && c < dk;
      rq[x] = in ? qg[(size_t)(base + t) * a.stride + c] : zero;
      rk[x] = in ? kg[(size_t)(base + t) * a.stride + c] : zero;
      ra[x] = in ? ag[(size_t)(base + t) * a_stride + c] : (t < nb ? 0.f : 1.f);
    }
  }
  if constexpr (BONUS)
    for (int c = p; c < NP; c += 128) us[c] = c < dk ? __bfloat162float(a.u[(size_t)h * dk + c]) : 0.f;
  __syncthreads();
  uint8_t* st = a.prep + ((size_t)slot * a.H + h) * Cfg::kPrep;
  uint32_t* pq = reinterpret_cast<uint32_t*>(st);                       // [2][Q][KS] bf16, read and written in pairs
  uint32_t* pk = pq + Q * KS;                                           // [3][Q][KS]
  __nv_bfloat16* pa = reinterpret_cast<__nv_bfloat16*>(st) + 5 * Q * KS;      // [3][Q][AS]
  float* dec = reinterpret_cast<float*>(pa + 3 * Q * AS);               // [NP]
  // a thread takes two channels, of q from the front or of k from the back
  for (int x = p; x < NP; x += 128) {
    const int c = (x % (NP / 2)) * 2;
    const bool is_k = x >= NP / 2;
    float2 run = make_float2(1.f, 1.f);
#pragma unroll
    for (int n = 0; n < Q; ++n) {
      const int t = is_k ? Q - 1 - n : n;
      const float2 al = *reinterpret_cast<const float2*>(ra + t * NP + c);
      float2 v = unpack_bf16x2(*reinterpret_cast<const uint32_t*>((is_k ? rk : rq) + t * NP + c));
      if (!is_k) {
        if constexpr (!BONUS) { run.x *= al.x; run.y *= al.y; }
        v.x *= a.q_scale; v.y *= a.q_scale;
      }
      uint32_t w0, w1, w2;
      split3(v.x * run.x, v.y * run.y, w0, w1, w2);
      const int at = (t * KS + c) / 2;
      if (is_k) {
        pk[at] = w0; pk[Q * KS / 2 + at] = w1; pk[Q * KS + at] = w2;
      } else {
        pq[at] = w0; pq[Q * KS / 2 + at] = w1;
      }
      if (BONUS || is_k) { run.x *= al.x; run.y *= al.y; }
    }
    if (!is_k) *reinterpret_cast<float2*>(dec + c) = run;
  }
  // the pair matrix: a warp takes the tokens j = w, 7 - w, 8 + w, 15 - w; a lane the channel pairs 2 lane + 64 m (or one
  // channel each of 32)
  const int w = p >> 5, lane = p & 31;
#pragma unroll 1
  for (int jj = 0; jj < 4; ++jj) {
    const int j = jj == 0 ? w : (jj == 1 ? 7 - w : (jj == 2 ? 8 + w : 15 - w));
    float acc[Q];
#pragma unroll
    for (int t = 0; t < Q; ++t) acc[t] = 0.f;
#pragma unroll
    for (int m = 0; m < (NP + 63) / 64; ++m) {
      const int c = NP >= 64 ? 2 * lane + 64 * m : lane;
      auto pair = [&](const __nv_bfloat16* r, int t) {
        if constexpr (NP >= 64) return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(r + t * NP + c));
        else return make_float2(__bfloat162float(r[t * NP + c]), 0.f);
      };
      float2 run = pair(rk, j);
      float2 own = run;      // what the token itself is read with
      if constexpr (BONUS) { own.x *= us[c]; own.y *= NP >= 64 ? us[c + (NP >= 64)] : 0.f; }
#pragma unroll
      for (int t = 0; t < Q; ++t) {      // tokens before j: nothing is added and nothing decays
        const float2 x = pair(rq, t);
        float2 al;
        if constexpr (NP >= 64) al = *reinterpret_cast<const float2*>(ra + t * NP + c);
        else al = make_float2(ra[t * NP + c], 0.f);
        const bool after = t > j;
        if constexpr (!BONUS) { run.x = after ? run.x * al.x : run.x; run.y = after ? run.y * al.y : run.y; }
        const float2 f = t == j ? own : run;
        acc[t] += t >= j ? x.x * f.x + x.y * f.y : 0.f;
        if constexpr (BONUS) { run.x = after ? run.x * al.x : run.x; run.y = after ? run.y * al.y : run.y; }
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
      const int at = (lane >> 1) * AS + j;      // A[t][j]; zero above the diagonal
      uint32_t w0, w1, w2;
      split3(sum, 0.f, w0, w1, w2);
      reinterpret_cast<uint16_t*>(pa)[at] = (uint16_t)w0;
      reinterpret_cast<uint16_t*>(pa)[Q * AS + at] = (uint16_t)w1;
      reinterpret_cast<uint16_t*>(pa)[2 * Q * AS + at] = (uint16_t)w2;
    }
  }
}

template <int NP>
KERN_DEVICE void chunk_body(const ChunkArgs& a) {
  using Cfg = LinCfg<NP>;
  constexpr int KS = Cfg::KS, NT = NP / 8, ST = Cfg::kStages;
  extern __shared__ __align__(16) uint8_t lin_sm[];
  const int tiles = (a.dv + VT - 1) / VT;
  const int h = blockIdx.x / tiles, c0 = (blockIdx.x % tiles) * VT, s = blockIdx.y;
  if (s >= a.seqs) return;
  const int r0 = a.cu[s], r1 = a.cu[s + 1], dk = a.dk, dv = a.dv;
  if (r1 - r0 < a.min_rows) return;
  int line = a.lines[s];
  if (line > 0 && !KERN_CHECK(a.state + (size_t)line * a.line_bytes, (size_t)a.line_bytes, SITE_STATE_SLOT)) line = 0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const __nv_bfloat16* vg = a.v + (size_t)h * dv + c0;
  const bool vec = (dv | a.stride) % 8 == 0 && (reinterpret_cast<uintptr_t>(a.v) & 15) == 0;
  const int chunks = (r1 - r0 + Q - 1) / Q;
  const uint8_t* blocks = a.prep + ((size_t)slot_of(a.cu, s) * a.H + h) * Cfg::kPrep;

  auto stage = [&](int i) { return lin_sm + (i % ST) * (Cfg::kPrep + Cfg::kV); };
  auto load = [&](int i) {      // the prepared block and v of chunk i; one group even where there is nothing to load
    if (i < chunks) {
      uint8_t* st = stage(i);
      const uint8_t* src = blocks + (size_t)i * a.H * Cfg::kPrep;
      for (int x = tid; x < Cfg::kPrep / 16; x += 128) cp16(smem_u32(st + x * 16), src + x * 16, true);
      __nv_bfloat16* rv = reinterpret_cast<__nv_bfloat16*>(st + Cfg::kPrep);
      const int base = r0 + i * Q, nb = min(Q, r1 - base);
      if (vec) {
        const int t = tid / (VT / 8), c = (tid % (VT / 8)) * 8;
        const bool in = t < nb && c0 + c < dv;
        cp16(smem_u32(rv + t * VS + c), vg + (size_t)(in ? base + t : base) * a.stride + (in ? c : 0), in);
      } else {
        for (int x = tid; x < Q * VT; x += 128) {
          const int t = x / VT, c = x % VT;
          rv[t * VS + c] = (t < nb && c0 + c < dv) ? vg[(size_t)(base + t) * a.stride + c] : __float2bfloat16(0.f);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // ---- S^T of a warp's 16 value columns: rows v = lane / 4 (+ 8), columns 8 i + 2 (lane % 4) (+ 1) ----
  const int vw = warp * 16;
  float S[NT][4];
  float* Sg = reinterpret_cast<float*>(a.state + (size_t)line * a.line_bytes + a.s_off) + (size_t)h * dk * dv + c0;
  auto s_at = [&](int i, int e, int& c, int& v) {
    v = vw + (lane >> 2) + (e >> 1) * 8;
    c = i * 8 + 2 * (lane & 3) + (e & 1);
    return c < dk && c0 + v < dv;
  };
  auto run = [&](int i) {
    const int base = r0 + i * Q, nb = min(Q, r1 - base);
    const uint8_t* st = stage(i);
    const __nv_bfloat16* pq = reinterpret_cast<const __nv_bfloat16*>(st);
    const __nv_bfloat16* pk = pq + 2 * Q * KS;
    const __nv_bfloat16* pa = pk + 3 * Q * KS;
    const float* dec = reinterpret_cast<const float*>(pa + 3 * Q * AS);
    const __nv_bfloat16* rv = reinterpret_cast<const __nv_bfloat16*>(st + Cfg::kPrep);
    float O[2][4] = {}, X[2][4] = {}, Y[2][4] = {};      // hi x hi, and the cross terms
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
        mma(Y[n], sh, ql[2 * n], ql[2 * n + 1]);
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
        if (t < nb && c0 + v < dv) a.out[((size_t)(base + t) * a.H + h) * dv + c0 + v] = O[n][e] + (X[n][e] + Y[n][e]);
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

#pragma unroll
  for (int i = 0; i < ST - 1; ++i) load(i);
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      int c, v;
      S[i][e] = (s_at(i, e, c, v) && line > 0) ? Sg[(size_t)c * dv + v] : 0.f;
    }
#pragma unroll 1
  for (int i = 0; i < chunks; ++i) {
    asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
    __syncthreads();      // chunk i is here, and nobody reads chunk i - 1 any more
    load(i + ST - 1);
    run(i);
  }
  if (line > 0) {
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

// prep: grid [slots, H], block 128, LinCfg<NP>::kRaw bytes of shared memory; chunk: grid [H ceil(dv / 64), seqs], block 128,
// kStages (kPrep + kV) bytes. `slots`: blocks of the prepared buffer per head.
#define LIN_CHUNK(NP)                                                                                                     \
  extern "C" __global__ void __launch_bounds__(128)                                                                       \
      kern_lin_prep_n##NP(const __nv_bfloat16* q, const __nv_bfloat16* k, const float* alpha, const __nv_bfloat16* u,     \
                          uint8_t* prep, const int* cu, int seqs, int H, int dk, int stride, int min_rows, int slots,     \
                          float q_scale) {                                                                                \
    pdl_wait();                                                                                                           \
    if ((int)blockIdx.x >= slots) return;                                                                                 \
    ChunkArgs a{};                                                                                                        \
    a.q = q; a.k = k; a.alpha = alpha; a.u = u; a.prep = prep; a.cu = cu; a.seqs = seqs; a.H = H; a.dk = dk;              \
    a.stride = stride; a.min_rows = min_rows; a.q_scale = q_scale;                                                        \
    if (u) prep_body<NP, true>(a);                                                                                        \
    else prep_body<NP, false>(a);                                                                                         \
    pdl_launch_dependents();                                                                                              \
  }                                                                                                                       \
  extern "C" __global__ void __launch_bounds__(128)                                                                       \
      kern_lin_chunk_n##NP(const __nv_bfloat16* v, const uint8_t* prep, float* out, uint8_t* state, const int* lines,     \
                           const int* cu, int seqs, int H, int dk, int dv, int stride, long long line_bytes, int s_off,   \
                           int min_rows) {                                                                                \
    pdl_wait();                                                                                                           \
    ChunkArgs a{};                                                                                                        \
    a.v = v; a.prep = const_cast<uint8_t*>(prep); a.out = out; a.state = state; a.lines = lines; a.cu = cu; a.seqs = seqs; \
    a.H = H; a.dk = dk; a.dv = dv; a.stride = stride; a.line_bytes = line_bytes; a.s_off = s_off; a.min_rows = min_rows;  \
    chunk_body<NP>(a);                                                                                                    \
    pdl_launch_dependents();                                                                                              \
  }

LIN_CHUNK(32)
LIN_CHUNK(64)
LIN_CHUNK(128)
LIN_CHUNK(256)
