// build: precise
// The Mamba-2 recurrence over prompts in its chunked (state-space dual) form on the tensor cores; ssd.cu holds the
// token-by-token form and the state line's layout. Per head and chunk of 64 tokens, with a_t = -exp(A_log) dt'_t and
// c_t = a_1 + .. + a_t inside the chunk:
//     y_i = sum_{j <= i} (C_i . B_j) exp(c_i - c_j) dt'_j x_j  +  exp(c_i) S C_i  +  D x_i
//     S  <- exp(c_64) S + sum_j exp(c_64 - c_j) dt'_j x_j B_j^T
// A CTA owns 32 value columns of one head of one sequence and walks its chunks in order; S stays in registers as f32 MMA
// accumulators for the whole prompt. B, C and x are bf16 already and enter the products exactly; every factor that is f32
// (decay-weighted scores, the state, decay-weighted inputs) enters as the sum of three bf16 numbers, which carries all of
// its 24 bits, so the products are those of f32 arithmetic with f32 sums. Exponents are differences of a sum kept in two
// floats. The next chunk's B, C and x are copied (cp.async) while this one is computed.
// NP: state columns padded to 32 / 64 / 128 / 256 (zeros). Sequences with fewer than `min_rows` rows are left to ssd.cu.
#include "act.cuh"

using namespace kern;

namespace {

constexpr int Q = 64, PT = 32, XS = PT + 8;

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
// the pair (u, v) as three bf16 pairs whose sums are u and v
KERN_DEVICE void split3(float u, float v, uint32_t& a, uint32_t& b, uint32_t& c) {
  a = pack_bf16x2(u, v);
  const float2 h = unpack_bf16x2(a);
  u -= h.x; v -= h.y;
  b = pack_bf16x2(u, v);
  const float2 m = unpack_bf16x2(b);
  c = pack_bf16x2(u - m.x, v - m.y);
}
KERN_DEVICE float softplus(float v) { return v > 30.f ? v : log1pf(expf(v)); }

template <int NP>
struct ChunkCfg {
  static constexpr int BS = NP + 8;                                  // row stride of B, C and S in shared memory
  static constexpr int kBC = Q * BS, kX = Q * XS, kS = PT * BS;      // elements
  static constexpr int kStage = 2 * kBC + kX;
  static constexpr int kBytes = 2 * kStage * 2 + 3 * kS * 2 + Q * PT * 4 + 5 * Q * 4;
};

template <int NP>
KERN_DEVICE void chunk_body(const __nv_bfloat16* xbc, const __nv_bfloat16* dt, float* y, uint8_t* state, const int* lines,
                            const int* cu, const __nv_bfloat16* A_log, const __nv_bfloat16* dt_bias, const __nv_bfloat16* D,
                            int seqs, int H, int P, int N, int G, int dt_stride, long long line_bytes, int s_off, int min_rows) {
  using Cfg = ChunkCfg<NP>;
  constexpr int BS = Cfg::BS, NT = NP / 32;
  extern __shared__ __align__(16) uint8_t chunk_sm[];
  __nv_bfloat16* stage0 = reinterpret_cast<__nv_bfloat16*>(chunk_sm);
  __nv_bfloat16* Ss = stage0 + 2 * Cfg::kStage;                       // [3][PT][BS]
  float* Ys = reinterpret_cast<float*>(Ss + 3 * Cfg::kS);             // [Q][PT]
  float* ch = Ys + Q * PT;                                            // c_t: high part, then low part
  float* cl = ch + Q;
  float* step = cl + Q;                                               // dt'_t
  float* ws = step + Q;                                               // exp(c_64 - c_t) dt'_t
  float* ec = ws + Q;                                                 // exp(c_t)
  const int parts = (P + PT - 1) / PT;
  const int h = blockIdx.x / parts, p0 = (blockIdx.x % parts) * PT, s = blockIdx.y;
  if (s >= seqs) return;
  const int r0 = cu[s], r1 = cu[s + 1];
  if (r1 - r0 < min_rows) return;
  int line = lines[s];
  if (line > 0 && !KERN_CHECK(state + (size_t)line * line_bytes, (size_t)line_bytes, SITE_STATE_SLOT)) line = 0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int inner = H * P, channels = inner + 2 * G * N, g = h / (H / G);
  const __nv_bfloat16* xb = xbc + h * P + p0;
  const __nv_bfloat16* bb = xbc + inner + g * N;
  const bool vec = channels % 8 == 0 && inner % 8 == 0 && N % 8 == 0 && P % 8 == 0 && (reinterpret_cast<uintptr_t>(xbc) & 15) == 0;

  auto load = [&](int base, __nv_bfloat16* st) {
    __nv_bfloat16* Bs = st;
    __nv_bfloat16* Cs = st + Cfg::kBC;
    __nv_bfloat16* Xs = st + 2 * Cfg::kBC;
    const int nb = min(Q, r1 - base);
    if (vec) {
      for (int i = tid; i < Q * (NP / 8); i += 256) {
        const int t = i / (NP / 8), c = (i % (NP / 8)) * 8;
        const bool in = t < nb && c < N;
        const __nv_bfloat16* src = bb + (size_t)(in ? base + t : base) * channels + (in ? c : 0);
        cp16(smem_u32(Bs + t * BS + c), src, in);
        cp16(smem_u32(Cs + t * BS + c), src + (in ? G * N : 0), in);
      }
      {
        const int t = tid / (PT / 8), c = (tid % (PT / 8)) * 8;
        const bool in = t < nb && p0 + c < P;
        cp16(smem_u32(Xs + t * XS + c), xb + (size_t)(in ? base + t : base) * channels + (in ? c : 0), in);
      }
    } else {
      const __nv_bfloat16 zero = __float2bfloat16(0.f);
      for (int i = tid; i < Q * NP; i += 256) {
        const int t = i / NP, c = i % NP;
        const bool in = t < nb && c < N;
        const __nv_bfloat16* src = bb + (size_t)(base + t) * channels + c;
        Bs[t * BS + c] = in ? src[0] : zero;
        Cs[t * BS + c] = in ? src[G * N] : zero;
      }
      for (int i = tid; i < Q * PT; i += 256) {
        const int t = i / PT, c = i % PT;
        Xs[t * XS + c] = (t < nb && p0 + c < P) ? xb[(size_t)(base + t) * channels + c] : zero;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // ---- the state: warp (mt, ng) holds rows 16 mt .. + 15, columns 8 (ng NT + i) .. + 7 ----
  const int mt = warp & 1, ng = warp >> 1;
  float* Sg = reinterpret_cast<float*>(state + (size_t)line * line_bytes + s_off) + ((size_t)h * P + p0) * N;
  float S[NT][4];
  auto s_at = [&](int i, int e, int& p, int& n) {
    p = mt * 16 + (lane >> 2) + (e >> 1) * 8;
    n = (ng * NT + i) * 8 + 2 * (lane & 3) + (e & 1);
    return p0 + p < P && n < N;
  };
  auto publish = [&]() {      // S as three bf16 terms in shared memory
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int p = mt * 16 + (lane >> 2) + (e >> 1) * 8, n = (ng * NT + i) * 8 + 2 * (lane & 3);
        uint32_t a, b, c;
        split3(S[i][e], S[i][e + 1], a, b, c);
        *reinterpret_cast<uint32_t*>(Ss + p * BS + n) = a;
        *reinterpret_cast<uint32_t*>(Ss + Cfg::kS + p * BS + n) = b;
        *reinterpret_cast<uint32_t*>(Ss + 2 * Cfg::kS + p * BS + n) = c;
      }
  };
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      int p, n;
      S[i][e] = (s_at(i, e, p, n) && line > 0) ? Sg[(size_t)p * N + n] : 0.f;
    }
  publish();
  const float a = -expf(__bfloat162float(A_log[h])), bias = __bfloat162float(dt_bias[h]), skip = __bfloat162float(D[h]);
  const int wm = warp & 3, wn = warp >> 2;
  const int rowA = wm * 16 + (lane >> 2), rowB = rowA + 8;

  int cur = 0;
  load(r0, stage0);
  for (int base = r0; base < r1; base += Q) {
    const int nb = min(Q, r1 - base);
    __nv_bfloat16* Bs = stage0 + cur * Cfg::kStage;
    __nv_bfloat16* Cs = Bs + Cfg::kBC;
    __nv_bfloat16* Xs = Bs + 2 * Cfg::kBC;
    // steps and running sums of the chunk: one warp, two tokens per lane
    if (warp == 0) {
      float d[2];
      double c[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = lane * 2 + i;
        d[i] = t < nb ? softplus(__bfloat162float(dt[(size_t)(base + t) * dt_stride + h]) + bias) : 0.f;
        c[i] = (double)(a * d[i]);
      }
      double run = c[0] + c[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      const double total = __shfl_sync(0xffffffffu, run, 31);
      const double at[2] = {run - c[1], run};
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = lane * 2 + i;
        ch[t] = (float)at[i];
        cl[t] = (float)(at[i] - (double)ch[t]);
        step[t] = d[i];
        ws[t] = expf((float)(total - at[i])) * d[i];
        ec[t] = expf((float)at[i]);
      }
    }
    if (base + Q < r1) {
      load(base + Q, stage0 + (cur ^ 1) * Cfg::kStage);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();      // this chunk's rows, sums, and the published state

    // ---- scores of rows 16 wm .. against tokens 32 wn .. + 31, decayed, and their product with x ----
    float Y[PT / 8][4];
#pragma unroll
    for (int i = 0; i < PT / 8; ++i) Y[i][0] = Y[i][1] = Y[i][2] = Y[i][3] = 0.f;
    const uint32_t c_addr = smem_u32(Cs + (wm * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * BS + (lane >> 4) * 8);
    if (wn * 32 <= wm * 16 + 15) {
      float Gt[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) Gt[i][0] = Gt[i][1] = Gt[i][2] = Gt[i][3] = 0.f;
      const uint32_t b_addr = smem_u32(Bs + (wn * 32 + (lane & 7)) * BS + (lane >> 3) * 8);
#pragma unroll
      for (int k = 0; k < NP; k += 32) {
        uint32_t c0[4], c1[4];
        ldsm4(c_addr + k * 2, c0);
        ldsm4(c_addr + k * 2 + 32, c1);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          uint32_t b[4];
          ldsm4(b_addr + i * 8 * BS * 2 + k * 2, b);
          mma(Gt[i], c0, b[0], b[1]);
          mma(Gt[i], c1, b[2], b[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = e < 2 ? rowA : rowB, j = wn * 32 + i * 8 + 2 * (lane & 3) + (e & 1);
          Gt[i][e] = j <= r ? Gt[i][e] * expf((ch[r] - ch[j]) + (cl[r] - cl[j])) * step[j] : 0.f;
        }
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        uint32_t m[3][4];
        split3(Gt[2 * k][0], Gt[2 * k][1], m[0][0], m[1][0], m[2][0]);
        split3(Gt[2 * k][2], Gt[2 * k][3], m[0][1], m[1][1], m[2][1]);
        split3(Gt[2 * k + 1][0], Gt[2 * k + 1][1], m[0][2], m[1][2], m[2][2]);
        split3(Gt[2 * k + 1][2], Gt[2 * k + 1][3], m[0][3], m[1][3], m[2][3]);
        const uint32_t x_addr = smem_u32(Xs + (wn * 32 + k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * XS + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < PT / 16; ++i) {
          uint32_t b[4];
          ldsm4_t(x_addr + i * 32, b);
#pragma unroll
          for (int z = 2; z >= 0; --z) {
            mma(Y[2 * i], m[z], b[0], b[1]);
            mma(Y[2 * i + 1], m[z], b[2], b[3]);
          }
        }
      }
    }
    // ---- what the earlier chunks left: exp(c_i) C_i S, this warp's half of the state columns ----
    {
      float E[PT / 8][4];
#pragma unroll
      for (int i = 0; i < PT / 8; ++i) E[i][0] = E[i][1] = E[i][2] = E[i][3] = 0.f;
      const uint32_t s_addr = smem_u32(Ss + (lane & 7) * BS + (lane >> 3) * 8);
      // NP = 32 is one step of 32 columns: only the first half-group of warps takes it
#pragma unroll
      for (int kk = 0; kk < (NP >= 64 ? NP / 2 : 32); kk += 32) {
        const int k = NP >= 64 ? wn * (NP / 2) + kk : 0;
        if (NP < 64 && wn != 0) break;
        uint32_t c0[4], c1[4];
        ldsm4(c_addr + k * 2, c0);
        ldsm4(c_addr + k * 2 + 32, c1);
#pragma unroll
        for (int z = 2; z >= 0; --z)
#pragma unroll
          for (int i = 0; i < PT / 8; ++i) {
            uint32_t b[4];
            ldsm4(s_addr + (z * Cfg::kS + i * 8 * BS + k) * 2, b);
            mma(E[i], c0, b[0], b[1]);
            mma(E[i], c1, b[2], b[3]);
          }
      }
      const float fa = ec[rowA], fb = ec[rowB];
#pragma unroll
      for (int i = 0; i < PT / 8; ++i) {
        Y[i][0] += fa * E[i][0]; Y[i][1] += fa * E[i][1];
        Y[i][2] += fb * E[i][2]; Y[i][3] += fb * E[i][3];
      }
    }
    if (wn == 1) {
#pragma unroll
      for (int i = 0; i < PT / 8; ++i) {
        const int c = i * 8 + 2 * (lane & 3);
        *reinterpret_cast<float2*>(Ys + rowA * PT + c) = make_float2(Y[i][0], Y[i][1]);
        *reinterpret_cast<float2*>(Ys + rowB * PT + c) = make_float2(Y[i][2], Y[i][3]);
      }
    }
    __syncthreads();      // the other half's sums are in; nobody reads the published state any more
    if (wn == 0) {
#pragma unroll
      for (int i = 0; i < PT / 8; ++i)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int t = hh ? rowB : rowA, c = i * 8 + 2 * (lane & 3);
          if (t >= nb) continue;
          const float2 o = *reinterpret_cast<const float2*>(Ys + t * PT + c);
          const float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(Xs + t * XS + c));
          float* dst = y + (size_t)(base + t) * inner + h * P + p0 + c;
          if (p0 + c < P) dst[0] = Y[i][2 * hh] + o.x + skip * x.x;
          if (p0 + c + 1 < P) dst[1] = Y[i][2 * hh + 1] + o.y + skip * x.y;
        }
    }
    // ---- the state after the chunk ----
    const float keep = ec[Q - 1];      // tokens past the end have step 0, so the last sum is the chunk's
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] *= keep;
#pragma unroll
    for (int k = 0; k < Q / 16; ++k) {
      uint32_t xr[4], m[3][4];
      ldsm4_t(smem_u32(Xs + (k * 16 + (lane & 7) + (lane >> 4) * 8) * XS + mt * 16 + ((lane >> 3) & 1) * 8), xr);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int t = k * 16 + (q >> 1) * 8 + 2 * (lane & 3);
        const float2 x = unpack_bf16x2(xr[q]);
        split3(x.x * ws[t], x.y * ws[t + 1], m[0][q], m[1][q], m[2][q]);
      }
      const uint32_t b_addr = smem_u32(Bs + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * BS);
#pragma unroll
      for (int i = 0; i < NT; i += 2) {
        uint32_t b[4];
        const int tile = ng * NT + i + (NT > 1 ? (lane >> 4) : 0);
        ldsm4_t(b_addr + tile * 16, b);
#pragma unroll
        for (int z = 2; z >= 0; --z) {
          mma(S[i], m[z], b[0], b[1]);
          if constexpr (NT > 1) mma(S[i + 1], m[z], b[2], b[3]);
        }
      }
    }
    publish();
    __syncthreads();      // sums and this stage may be overwritten
    cur ^= 1;
  }
  if (line > 0) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int p, n;
        if (s_at(i, e, p, n)) Sg[(size_t)p * N + n] = S[i][e];
      }
  }
}

}  // namespace

// grid [H ceil(P / 32), seqs], block 256.
#define SSD_CHUNK(NP)                                                                                                      \
  extern "C" __global__ void __launch_bounds__(256)                                                                        \
      kern_ssd_chunk_n##NP(const __nv_bfloat16* xbc, const __nv_bfloat16* dt, float* y, uint8_t* state, const int* lines,  \
                           const int* cu, const __nv_bfloat16* A_log, const __nv_bfloat16* dt_bias,                        \
                           const __nv_bfloat16* D, int seqs, int H, int P, int N, int G, int dt_stride,                    \
                           long long line_bytes, int s_off, int min_rows) {                                                \
    pdl_wait();                                                                                                            \
    chunk_body<NP>(xbc, dt, y, state, lines, cu, A_log, dt_bias, D, seqs, H, P, N, G, dt_stride, line_bytes, s_off,        \
                   min_rows);                                                                                              \
    pdl_launch_dependents();                                                                                               \
  }

SSD_CHUNK(32)
SSD_CHUNK(64)
SSD_CHUNK(128)
SSD_CHUNK(256)
