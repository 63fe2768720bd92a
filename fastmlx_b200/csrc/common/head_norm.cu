// The read-out of a recurrence's heads: each head's o, optionally over a normaliser, divided by its root mean square, times a
// weight (shared by the heads or one per head), times sigmoid or silu of a gate of its own type.  32-bit but for the gate that
// comes in and the activations that go out.
#include <math.h>
#include "common.cuh"
#include "packed.cuh"

namespace {
// What a head's read-out is divided by first, where a recurrence has a normaliser: max(|nq|, floor) + 1e-6 (floor: the third of
// four gate values per token and head).
__device__ __forceinline__ float over_normaliser(const float* nq, const float4* gates, long long item) {
  return nq == nullptr ? 1.0f : 1.0f / (fmaxf(fabsf(nq[item]), gates[item].z) + 1e-6f);
}

// One warp per (token, head): out[t, h, :] = o / sqrt(mean(o^2) + eps) * w[h * w_stride ...] * act(gate[t, h, :]), act sigmoid or
// silu.
template <typename TG, typename T>
__global__ void __launch_bounds__(128)
head_norm_gate_kernel(const float* o, const TG* gate, long long gate_stride, const float* __restrict__ w, T* out,
                      long long out_stride, long long n_items, int H, int Dv, float eps, int silu, int w_stride, const float* nq, const float4* gates) {
  pdl_wait();
  pdl_trigger();
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= n_items) return;
  const long long t = item / H;
  const int h = (int)(item - t * H);
  const float* op = o + item * Dv;
  const TG* gp = gate + t * gate_stride + (long long)h * Dv;
  T* dst = out + t * out_stride + (long long)h * Dv;
  const float mul = over_normaliser(nq, gates, item);
  const float* wp = w + (long long)h * w_stride;
  float ss = 0.f;
  for (int e = lane; e < Dv; e += 32) ss = fmaf(op[e] * mul, op[e] * mul, ss);
  const float rstd = mul / sqrtf(warp_sum(ss) / (float)Dv + eps);
  for (int e = lane; e < Dv; e += 32) {
    const float x = to_f(gp[e]), sg = 1.0f / (1.0f + expf(-x));
    dst[e] = from_f<T>(op[e] * rstd * wp[e] * (silu ? x * sg : sg));
  }
}

// The same with four neighbouring values per lane: LG = Dv / 4 lanes (8, 16 or 32) per (token, head).
template <typename TG, typename T, int LG>
__global__ void __launch_bounds__(128)
head_norm_gate_vec_kernel(const float* o, const TG* gate, long long gate_stride, const float* __restrict__ w, T* out,
                          long long out_stride, long long n_items, int H, float eps, int silu, int w_stride, const float* nq, const float4* gates) {
  pdl_wait();
  pdl_trigger();
  const long long item = (long long)blockIdx.x * (128 / LG) + threadIdx.x / LG;
  const int e = 4 * (threadIdx.x % LG), Dv = 4 * LG;
  const bool live = item < n_items;                // (every lane takes part in the exchange)
  const long long t = live ? item / H : 0;
  const int h = live ? (int)(item - t * H) : 0;
  float4 x = live ? load4(o + item * Dv + e) : make_float4(0.f, 0.f, 0.f, 0.f);
  if (live && nq != nullptr) {
    const float mul = over_normaliser(nq, gates, item);
    x = make_float4(x.x * mul, x.y * mul, x.z * mul, x.w * mul);
  }
  float ss = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w)));
#pragma unroll
  for (int d = LG / 2; d >= 1; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  if (!live) return;
  const float rstd = 1.0f / sqrtf(ss / (float)Dv + eps);
  const float4 g = load4(gate + t * gate_stride + (long long)h * Dv + e), ww = load4(w + (long long)h * w_stride + e);
  auto act = [&](float v) { const float sg = 1.0f / (1.0f + expf(-v)); return silu ? v * sg : sg; };
  store4(out + t * out_stride + (long long)h * Dv + e, make_float4(x.x * rstd * ww.x * act(g.x), x.y * rstd * ww.y * act(g.y),
                                                                  x.z * rstd * ww.z * act(g.z), x.w * rstd * ww.w * act(g.w)));
}
}  // namespace

// o [T, H*Dv] 32-bit; gate rows of gate_stride elements of type g_dtype; out rows of out_stride elements of type dtype; head h's
// weights start at w + h * w_stride (0: one weight of Dv values for all heads).  nq [T, H] and gates [T, H, 4], or both null: o is first
// divided by max(|nq|, gates[.., 2]) + 1e-6.
FMX_EXPORT int fmx_head_norm_gate(const float* o, const void* gate, long long gate_stride, int g_dtype, const float* w, void* out,
                                  long long out_stride, int dtype, int T, int H, int Dv, float eps, int silu, int w_stride, const float* nq,
                                  const float* gates, cudaStream_t stream) {
  if (T == 0) return 0;
  if (T < 0 || H <= 0 || Dv <= 0 || gate_stride < (long long)H * Dv || out_stride < (long long)H * Dv)
    return fmx_fail("fmx_head_norm_gate: bad sizes T=%d H=%d Dv=%d", T, H, Dv);
  if ((nq == nullptr) != (gates == nullptr) || ((uintptr_t)gates & 15)) return fmx_fail("fmx_head_norm_gate: a normaliser and its floors come together");
  const long long items = (long long)T * H, grid = (items + 3) / 4;
  if (grid > 2147483647LL) return fmx_fail("fmx_head_norm_gate: batch too large");
  const bool vec = (Dv == 32 || Dv == 64 || Dv == 128) && gate_stride % 4 == 0 && out_stride % 4 == 0 && ((uintptr_t)o & 15) == 0 &&
                   ((uintptr_t)w & 15) == 0 && w_stride % 4 == 0 && ((uintptr_t)gate & (g_dtype == FMX_F32 ? 15 : 7)) == 0 &&
                   ((uintptr_t)out & (dtype == FMX_F32 ? 15 : 7)) == 0;
#define FMX_HNG_V(TG, TO, LG)                                                                                          \
  fmx_launch(head_norm_gate_vec_kernel<TG, TO, LG>, dim3((unsigned)((items + 128 / (LG) - 1) / (128 / (LG)))), dim3(128), 0, stream, o, \
             (const TG*)gate, gate_stride, w, (TO*)out, out_stride, items, H, eps, silu, w_stride, nq, (const float4*)gates)
#define FMX_HNG_VEC(TG, TO)                                                                                            \
  do {                                                                                                                 \
    if (Dv == 32) FMX_HNG_V(TG, TO, 8);                                                                                \
    else if (Dv == 64) FMX_HNG_V(TG, TO, 16);                                                                          \
    else FMX_HNG_V(TG, TO, 32);                                                                                        \
  } while (0)
  if (vec) {
    if (g_dtype == FMX_F32 && dtype == FMX_F32) FMX_HNG_VEC(float, float);
    else if (g_dtype == FMX_F32 && dtype == FMX_BF16) FMX_HNG_VEC(float, bf16);
    else if (g_dtype == FMX_BF16 && dtype == FMX_BF16) FMX_HNG_VEC(bf16, bf16);
    else return fmx_fail("fmx_head_norm_gate: unknown dtypes %d, %d", g_dtype, dtype);
    FMX_LAUNCH_CHECK();
    return 0;
  }
#undef FMX_HNG_VEC
#undef FMX_HNG_V
#define FMX_HNG(TG, TO)                                                                                                \
  fmx_launch(head_norm_gate_kernel<TG, TO>, dim3((unsigned)grid), dim3(128), 0, stream, o, (const TG*)gate, gate_stride, w, (TO*)out, \
             out_stride, items, H, Dv, eps, silu, w_stride, nq, (const float4*)gates)
  if (g_dtype == FMX_F32 && dtype == FMX_F32) FMX_HNG(float, float);
  else if (g_dtype == FMX_F32 && dtype == FMX_BF16) FMX_HNG(float, bf16);
  else if (g_dtype == FMX_BF16 && dtype == FMX_BF16) FMX_HNG(bf16, bf16);
  else return fmx_fail("fmx_head_norm_gate: unknown dtypes %d, %d", g_dtype, dtype);
#undef FMX_HNG
  FMX_LAUNCH_CHECK();
  return 0;
}
