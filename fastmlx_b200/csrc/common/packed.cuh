// What the recurrences share: four neighbouring values in one access, pairs of floats in one 64-bit register, and sums
// over neighbouring lanes of several values together.
#pragma once
#include "common.cuh"

namespace {
// four neighbouring values of any element type in one access
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<unsigned*>(&a);
  u.y = *reinterpret_cast<unsigned*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

// ---- pairs of floats in one 64-bit register: the packed multiply-add of sm_100
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pair_of(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float pair_sum(f32x2 a) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(a));
  return lo + hi;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// NV values of every lane added up across L lanes (NV <= L, both powers of two): each round halves what a lane holds,
// and lane `sub` is left with the sum of value sub * NV / L.  The pairs of lanes that meet are the same for every value.
template <int NV, int L> __device__ __forceinline__ float reduce_scatter(float (&v)[NV], int sub) {
  int d = L / 2;
#pragma unroll
  for (int w = NV / 2; w >= 1; w >>= 1, d >>= 1) {
    const bool upper = (sub & d) != 0;
#pragma unroll
    for (int i = 0; i < w; ++i) {
      const float give = upper ? v[i] : v[i + w], keep = upper ? v[i + w] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, d);
    }
  }
#pragma unroll
  for (int e = L / NV / 2; e >= 1; e >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], e);
  return v[0];
}
// The same, and every lane gets all the sums.
template <int NV, int L> __device__ __forceinline__ void all_reduce(float (&v)[NV], int sub) {
  const float mine = reduce_scatter<NV, L>(v, sub);
  const int base = (threadIdx.x & 31) - sub;
#pragma unroll
  for (int i = 0; i < NV; ++i) v[i] = __shfl_sync(0xffffffffu, mine, base + i * (L / NV));
}
}  // namespace
