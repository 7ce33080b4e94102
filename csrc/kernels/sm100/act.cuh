// Loads and stores of activations whose type is a template parameter (bf16, or f32 in a model's 32-bit form), one value or
// four at a time.
#pragma once
#include "common.cuh"

namespace kern {

KERN_DEVICE float ldf(const float* p) { return *p; }
KERN_DEVICE float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
KERN_DEVICE void stf(float* p, float v) { *p = v; }
KERN_DEVICE void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <int V> struct Vec { float v[V]; };
template <int V> KERN_DEVICE Vec<V> ldv(const float* p) {
  Vec<V> r;
  if constexpr (V == 4) { const float4 a = *reinterpret_cast<const float4*>(p); r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w; }
  else r.v[0] = *p;
  return r;
}
template <int V> KERN_DEVICE Vec<V> ldv(const __nv_bfloat16* p) {
  Vec<V> r;
  if constexpr (V == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = unpack_bf16x2(a.x), hi = unpack_bf16x2(a.y);
    r.v[0] = lo.x; r.v[1] = lo.y; r.v[2] = hi.x; r.v[3] = hi.y;
  } else r.v[0] = __bfloat162float(*p);
  return r;
}
template <int V> KERN_DEVICE void stv(float* p, const Vec<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int V> KERN_DEVICE void stv(__nv_bfloat16* p, const Vec<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(r.v[0], r.v[1]), pack_bf16x2(r.v[2], r.v[3]));
  else *p = __float2bfloat16(r.v[0]);
}

// V values as they lie in memory: what waits for its turn takes no more registers than that
template <typename T, int V> struct RawOf { T v[V]; };
template <> struct __align__(8) RawOf<__nv_bfloat16, 4> { uint2 v; };
template <> struct __align__(16) RawOf<float, 4> { float4 v; };
template <int V, typename T> KERN_DEVICE RawOf<T, V> raw(const T* p) { return *reinterpret_cast<const RawOf<T, V>*>(p); }
template <typename T, int V> KERN_DEVICE void add(Vec<V>& a, const RawOf<T, V>& r, float w) {
  const Vec<V> b = ldv<V>(reinterpret_cast<const T*>(&r));
#pragma unroll
  for (int e = 0; e < V; ++e) a.v[e] += w * b.v[e];
}

}  // namespace kern
