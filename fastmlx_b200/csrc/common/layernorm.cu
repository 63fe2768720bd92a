// Layer norm behind a sublayer, fused with the sum into the residual stream and with the norm that may follow it.
// Per row, with L_w(v) = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps) * w:
//
//     r  = residual (or 0 where the stream starts here) + mult * post(y)      post = L_w, or the identity
//     residual = r                                                             (32-bit, in place or into a stream of its own)
//     out = pre(r)                                                             pre = another L_w, or the identity
//
// One block per row holds the row in registers (or, for long or unaligned rows, in shared memory).  Everything is
// 32-bit; the variance is the mean of the squared deviations; the order of a row's sums depends on its width alone.
#include <math.h>
#include "common.cuh"

namespace {
constexpr int LN_BLOCK = 256;

__device__ __forceinline__ float4 ln_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ln_load4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void ln_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ln_store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<unsigned*>(&a);
  u.y = *reinterpret_cast<unsigned*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

// the row's values v (four neighbouring columns per thread and pass) normalised in place
template <int NV>
__device__ __forceinline__ void ln_row(float4 (&v)[NV], int cols, float eps, const float* __restrict__ w) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);          // columns beyond the row hold zeros
  const float mean = block_sum<LN_BLOCK>(s) / (float)cols;
  s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = 4 * (threadIdx.x + i * LN_BLOCK);
    if (c < cols) {
      v[i] = make_float4(v[i].x - mean, v[i].y - mean, v[i].z - mean, v[i].w - mean);
      s = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, s))));
    }
  }
  const float rstd = 1.0f / sqrtf(block_sum<LN_BLOCK>(s) / (float)cols + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = 4 * (threadIdx.x + i * LN_BLOCK);
    if (c < cols) {
      const float4 g = ln_load4(w + c);
      v[i] = make_float4(v[i].x * rstd * g.x, v[i].y * rstd * g.y, v[i].z * rstd * g.z, v[i].w * rstd * g.w);
    }
  }
}

template <typename TY, typename TO, int NV>
__global__ void __launch_bounds__(LN_BLOCK)
layernorm_step_kernel(const TY* y, long long y_stride, const float* __restrict__ post_w, float post_eps, float mult,
                      const float* res_in, float* res_out, const float* __restrict__ pre_w, float pre_eps, TO* out,
                      long long out_stride, int cols) {
  pdl_wait();
  pdl_trigger();
  const long long r = blockIdx.x;
  float4 s[NV], v[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = 4 * (threadIdx.x + i * LN_BLOCK);
    const bool in = c < cols;
    s[i] = (in && res_in != nullptr) ? ln_load4(res_in + r * cols + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    v[i] = (in && y != nullptr) ? ln_load4(y + r * y_stride + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (y != nullptr) {
    if (post_w != nullptr) ln_row<NV>(v, cols, post_eps, post_w);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      s[i] = make_float4(fmaf(mult, v[i].x, s[i].x), fmaf(mult, v[i].y, s[i].y), fmaf(mult, v[i].z, s[i].z), fmaf(mult, v[i].w, s[i].w));
  }
  if (res_out != nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = 4 * (threadIdx.x + i * LN_BLOCK);
      if (c < cols) ln_store4(res_out + r * cols + c, s[i]);
    }
  }
  if (out == nullptr) return;
  if (pre_w != nullptr) ln_row<NV>(s, cols, pre_eps, pre_w);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = 4 * (threadIdx.x + i * LN_BLOCK);
    if (c < cols) ln_store4(out + r * out_stride + c, s[i]);
  }
}

// The same for rows of any width and alignment, a column per thread and pass, the row in shared memory (a thread reads
// back its own columns only).
__device__ __forceinline__ void ln_row_any(float* v, int cols, float eps, const float* __restrict__ w) {
  float s = 0.f;
  for (int c = threadIdx.x; c < cols; c += LN_BLOCK) s += v[c];
  const float mean = block_sum<LN_BLOCK>(s) / (float)cols;
  s = 0.f;
  for (int c = threadIdx.x; c < cols; c += LN_BLOCK) {
    const float d = v[c] - mean;
    v[c] = d;
    s = fmaf(d, d, s);
  }
  const float rstd = 1.0f / sqrtf(block_sum<LN_BLOCK>(s) / (float)cols + eps);
  for (int c = threadIdx.x; c < cols; c += LN_BLOCK) v[c] = v[c] * rstd * w[c];
}

template <typename TY, typename TO>
__global__ void __launch_bounds__(LN_BLOCK)
layernorm_step_any_kernel(const TY* y, long long y_stride, const float* __restrict__ post_w, float post_eps, float mult,
                          const float* res_in, float* res_out, const float* __restrict__ pre_w, float pre_eps, TO* out,
                          long long out_stride, int cols) {
  extern __shared__ float row[];
  pdl_wait();
  pdl_trigger();
  const long long r = blockIdx.x;
  for (int c = threadIdx.x; c < cols; c += LN_BLOCK) row[c] = y != nullptr ? to_f(y[r * y_stride + c]) : 0.f;
  if (y != nullptr && post_w != nullptr) ln_row_any(row, cols, post_eps, post_w);
  for (int c = threadIdx.x; c < cols; c += LN_BLOCK) {
    const float s = fmaf(mult, row[c], res_in != nullptr ? res_in[r * cols + c] : 0.f);
    if (res_out != nullptr) res_out[r * cols + c] = s;
    row[c] = s;
  }
  if (out == nullptr) return;
  if (pre_w != nullptr) ln_row_any(row, cols, pre_eps, pre_w);
  for (int c = threadIdx.x; c < cols; c += LN_BLOCK) out[r * out_stride + c] = from_f<TO>(row[c]);
}
}  // namespace

// y (of y_dtype, rows of y_stride) may be null; post_w null: y is added as it is; res_in null: the stream starts at zero;
// res_out null: the stream is not written (res_in and res_out may be the same array); pre_w null: out = the stream; out
// null: nothing is written there.
FMX_EXPORT int fmx_layernorm_step(const void* y, long long y_stride, int y_dtype, const float* post_w, float post_eps, float mult,
                                  const float* res_in, float* res_out, const float* pre_w, float pre_eps, void* out,
                                  long long out_stride, int out_dtype, int rows, int cols, cudaStream_t stream) {
  if (rows == 0 || cols == 0) return 0;
  if (rows < 0 || cols < 0 || (y != nullptr && y_stride < cols) || (out != nullptr && out_stride < cols))
    return fmx_fail("fmx_layernorm_step: bad sizes rows=%d cols=%d", rows, cols);
  if ((size_t)cols * sizeof(float) > 200 * 1024) return fmx_fail("fmx_layernorm_step: rows of %d columns are too long", cols);
  auto a16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = cols % 4 == 0 && cols <= 8 * 4 * LN_BLOCK && y_stride % 4 == 0 && out_stride % 4 == 0 && a16(y) && a16(out) &&
                   a16(res_in) && a16(res_out) && a16(post_w) && a16(pre_w);
  const int passes = (cols + 4 * LN_BLOCK - 1) / (4 * LN_BLOCK);
  const size_t smem = (size_t)cols * sizeof(float);
#define FMX_LN_V(TY, TO, NV)                                                                                           \
  fmx_launch(layernorm_step_kernel<TY, TO, NV>, dim3(rows), dim3(LN_BLOCK), 0, stream, (const TY*)y, y_stride, post_w, post_eps, mult, \
             res_in, res_out, pre_w, pre_eps, (TO*)out, out_stride, cols)
#define FMX_LN(TY, TO)                                                                                                 \
  do {                                                                                                                 \
    if (vec && passes <= 1) FMX_LN_V(TY, TO, 1);                                                                       \
    else if (vec && passes <= 2) FMX_LN_V(TY, TO, 2);                                                                  \
    else if (vec && passes <= 4) FMX_LN_V(TY, TO, 4);                                                                  \
    else if (vec) FMX_LN_V(TY, TO, 8);                                                                                 \
    else {                                                                                                             \
      if (smem > 48 * 1024)                                                                                            \
        cudaFuncSetAttribute(layernorm_step_any_kernel<TY, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      fmx_launch(layernorm_step_any_kernel<TY, TO>, dim3(rows), dim3(LN_BLOCK), smem, stream, (const TY*)y, y_stride, post_w, \
                 post_eps, mult, res_in, res_out, pre_w, pre_eps, (TO*)out, out_stride, cols);                         \
    }                                                                                                                  \
  } while (0)
  const int yd = y != nullptr ? y_dtype : FMX_F32, od = out != nullptr ? out_dtype : FMX_F32;
  if (yd == FMX_F32 && od == FMX_F32) FMX_LN(float, float);
  else if (yd == FMX_F32 && od == FMX_BF16) FMX_LN(float, bf16);
  else if (yd == FMX_BF16 && od == FMX_F32) FMX_LN(bf16, float);
  else if (yd == FMX_BF16 && od == FMX_BF16) FMX_LN(bf16, bf16);
  else return fmx_fail("fmx_layernorm_step: unknown dtypes %d, %d", y_dtype, out_dtype);
#undef FMX_LN
#undef FMX_LN_V
  FMX_LAUNCH_CHECK();
  return 0;
}
