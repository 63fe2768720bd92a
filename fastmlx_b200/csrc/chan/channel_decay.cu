// Linear attention whose state decays by key channel: every row of a head's matrix of state has a decay of its own.
//
// Per head, with key k, query q (size D), value v (size Dv) and a decay g in (0, 1) per key channel, a token does
//     gated linear attention:   S <- diag(g) S + k v^T;                                     o = S^T q
//     delta rule:               S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;     o = S^T q
// so the read-out sees the token's own write.  S [D, Dv] lives in 32-bit in a state slot of the request and is carried
// from step to step (S^T of every head, [H, Dv, D], at the head of a slot).
//
//   channel_delta_prepare   per token: a short causal convolution per channel + SiLU of the projected q | k | v channels
//                           (inputs before the portion's start come from the slot's convolution state), q and k made unit
//                           vectors per head (q also times D^-1/2), beta = sigmoid(b), g = exp(-exp(A_log) softplus(z +
//                           bias)).  A warp per (token, head); in steps of single tokens the warp that read a channel's
//                           state also moves it on, else conv_state_update does.
//   channel_gla_prepare     per token: q scaled, k, v in 32-bit, g = sigmoid(z + bias)^(1/tau).
//   channel_scan            the recurrence, see there.
//
// Everything is 32-bit but the projections that come in and the activations that go out.
#include <math.h>
#include "common.cuh"
#include "conv_state.cuh"
#include "packed.cuh"

namespace {
__device__ __forceinline__ float softplus_f(float a) { return fmaxf(a, 0.f) + log1pf(expf(-fabsf(a))); }

// proj [T, stride]: q (G*D) | k (G*D) | v (H*Dv) | ...; b [T, b_stride] the write strengths' pre-activations; z [T, z_stride]
// 32-bit: the decays' pre-activations (H*D).  out_qkv [T, C], out_g [T, H*D], out_beta [T, H], 32-bit.
// MAXI: values of a q or k head that a lane holds (D <= 32 MAXI).  W: neighbouring channels that a lane takes at a time (2
// where D, Dv and the rows' starts allow it).
template <typename T> __device__ __forceinline__ float2 load2(const T* p);
template <> __device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 load2<bf16>(const bf16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}

template <typename T, int MAXI, int W>
__global__ void __launch_bounds__(128)
channel_delta_prepare_kernel(const T* proj, long long stride, const T* b, long long b_stride, const float* z, long long z_stride,
                             const float* __restrict__ conv_w, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                             const int* token_row, const int* row_start, const int* row_slot, float* state, long long slot_stride,
                             long long conv_off, float* out_qkv, float* out_g, float* out_beta, int H, int G, int D, int Dv,
                             int taps, int R, int max_slots, int single, int* status) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const int item = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (item >= 2 * G + 2 * H) return;
  const int C = 2 * G * D + H * Dv;
  if (item >= 2 * G + H) {                        // a head's decays and its write strength
    const int h = item - 2 * G - H;
    const float rate = expf(a_log[h]);
    for (int e = W * lane; e < D; e += 32 * W) {
      const long long c = (long long)h * D + e;
      if (W == 2) {
        const float2 x = load2(z + (long long)t * z_stride + c), b2 = load2(dt_bias + c);
        *reinterpret_cast<float2*>(out_g + (long long)t * H * D + c) =
            make_float2(expf(-rate * softplus_f(x.x + b2.x)), expf(-rate * softplus_f(x.y + b2.y)));
      } else {
        out_g[(long long)t * H * D + c] = expf(-rate * softplus_f(z[(long long)t * z_stride + c] + dt_bias[c]));
      }
    }
    if (lane == 0) out_beta[(long long)t * H + h] = 1.0f / (1.0f + expf(-to_f(b[(long long)t * b_stride + h])));
    return;
  }
  const int r = token_row[t];
  const int slot = (r >= 0 && r < R) ? row_slot[r] : -1;
  const int c0 = item < 2 * G ? item * D : 2 * G * D + (item - 2 * G) * Dv, n_c = item < 2 * G ? D : Dv;
  float* dst = out_qkv + (long long)t * C + c0;
  if (slot < 0 || slot >= max_slots) {            // a padding row of a captured step, or a bad row: nothing to do
    if (lane == 0 && item == 0) {
      if (r < 0 || r >= R) fmx_set_status(status, FMX_BAD_ROW, r, t);
      else if (slot >= max_slots) fmx_set_status(status, FMX_BAD_SLOT, slot, t);
    }
    for (int e = lane; e < n_c; e += 32) dst[e] = 0.f;
    return;
  }
  const int first = row_start[r], i = t - first;  // the token's place in its portion
  float* cs = state + (long long)slot * slot_stride + conv_off;                // [taps-1, C]
  auto channel = [&](int e) -> float {
    const int c = c0 + e;
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int n = i - (taps - 1) + j;
      const float x = n >= 0 ? to_f(proj[(long long)(first + n) * stride + c]) : cs[(long long)(taps - 1 + n) * C + c];
      acc = fmaf(conv_w[(long long)c * taps + j], x, acc);
      if (single && j > 0) cs[(long long)(j - 1) * C + c] = x;                 // the state moves on by one token
    }
    return silu_f(acc);
  };
  auto channels = [&](int e) -> float2 {          // channels e and e + 1
    const int c = c0 + e;
    float2 acc = make_float2(0.f, 0.f);
    for (int j = 0; j < taps; ++j) {
      const int n = i - (taps - 1) + j;
      const float2 x = n >= 0 ? load2(proj + (long long)(first + n) * stride + c) : load2(cs + (long long)(taps - 1 + n) * C + c);
      acc.x = fmaf(conv_w[(long long)c * taps + j], x.x, acc.x);
      acc.y = fmaf(conv_w[(long long)(c + 1) * taps + j], x.y, acc.y);
      if (single && j > 0) *reinterpret_cast<float2*>(cs + (long long)(j - 1) * C + c) = x;
    }
    return make_float2(silu_f(acc.x), silu_f(acc.y));
  };
  if (item >= 2 * G) {
    for (int e = W * lane; e < n_c; e += 32 * W) {
      if (W == 2) *reinterpret_cast<float2*>(dst + e) = channels(e);
      else dst[e] = channel(e);
    }
    return;
  }
  if (W == 2) {
    float2 v[MAXI / 2];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < MAXI / 2; ++k) {
      const int e = 2 * lane + 64 * k;
      v[k] = e < D ? channels(e) : make_float2(0.f, 0.f);
      ss = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, ss));
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
    const float mul = item < G ? inv * (1.0f / sqrtf((float)D)) : inv;         // q heads come first
#pragma unroll
    for (int k = 0; k < MAXI / 2; ++k) {
      const int e = 2 * lane + 64 * k;
      if (e < D) *reinterpret_cast<float2*>(dst + e) = make_float2(v[k].x * mul, v[k].y * mul);
    }
    return;
  }
  float v[MAXI], ss = 0.f;
#pragma unroll
  for (int k = 0; k < MAXI; ++k) {
    const int e = lane + 32 * k;
    v[k] = e < D ? channel(e) : 0.f;
    ss = fmaf(v[k], v[k], ss);
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
  const float mul = item < G ? inv * (1.0f / sqrtf((float)D)) : inv;           // q heads come first
#pragma unroll
  for (int k = 0; k < MAXI; ++k) {
    const int e = lane + 32 * k;
    if (e < D) dst[e] = v[k] * mul;
  }
}

// proj [T, stride]: q (H*D) | k (H*D) | v (H*Dv) | ...; z [T, z_stride] 32-bit; out_qkv [T, 2*H*D + H*Dv], out_g [T, H*D].
// A block takes 512 columns of a token (those of out_qkv, then those of out_g), four neighbouring ones per thread and pass.
template <typename T>
__global__ void __launch_bounds__(128)
channel_gla_prepare_kernel(const T* proj, long long stride, const float* z, long long z_stride, const float* __restrict__ bias,
                           float* out_qkv, float* out_g, int HD, int C, float q_scale, float inv_tau) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int N = C + HD;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int c = blockIdx.y * 512 + k * 128 + threadIdx.x;
    if (c >= N) return;
    if (c < C) {
      const float x = to_f(proj[t * stride + c]);
      out_qkv[t * C + c] = c < HD ? x * q_scale : x;
    } else {
      const int e = c - C;
      const float x = z[t * z_stride + e] + (bias != nullptr ? bias[e] : 0.f);
      out_g[t * HD + e] = expf(-softplus_f(-x) * inv_tau);                     // sigmoid(x)^(1/tau)
    }
  }
}

// The same with four neighbouring columns per access (HD, C and every row start multiples of four).
template <typename T>
__global__ void __launch_bounds__(128)
channel_gla_prepare_vec_kernel(const T* proj, long long stride, const float* z, long long z_stride, const float* __restrict__ bias,
                               float* out_qkv, float* out_g, int HD, int C, float q_scale, float inv_tau) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int c = (blockIdx.y * 128 + threadIdx.x) * 4;
  if (c < C) {
    float4 x = load4(proj + t * stride + c);
    if (c < HD) x = make_float4(x.x * q_scale, x.y * q_scale, x.z * q_scale, x.w * q_scale);
    store4(out_qkv + t * C + c, x);
  } else if (c < C + HD) {
    const int e = c - C;
    float4 x = load4(z + t * z_stride + e);
    if (bias != nullptr) {
      const float4 b = load4(bias + e);
      x = make_float4(x.x + b.x, x.y + b.y, x.z + b.z, x.w + b.w);
    }
    store4(out_g + t * HD + e, make_float4(expf(-softplus_f(-x.x) * inv_tau), expf(-softplus_f(-x.y) * inv_tau),
                                           expf(-softplus_f(-x.z) * inv_tau), expf(-softplus_f(-x.w) * inv_tau)));
  }
}

// The recurrence over every row's tokens of a step, in order, from and into the rows' state slots.
//
// Columns of S are independent (column j needs v_j only).  grid (ceil(Dv / COLS), H, R), 128 threads: L adjacent lanes hold
// CPT neighbouring columns, lane `sub` the rows 4 (sub + L i) .. + 3, i < RPL / 4 (D <= RPL L), in registers.  A token's
// operands (k and q of the head's group, the decays, the block's values, beta) come through shared memory in runs of
// TB tokens, the next run copied (cp.async) while the current one is walked.
//
// The delta rule's chain from token to token is a sum over the column's lanes.  GT = 4 tokens are therefore taken
// together: with S_0 the state in front of them and P_j = g_1 ... g_j (per channel), the sum that token j needs is
//     S'_j^T k_j = S_0^T (P_j k_j) + sum_{i < j} u_i  k_i . (g_{i+1} ... g_j k_j),      S'_j = diag(g_j) S_{j-1},
// so one exchange between the lanes gives all four sums with S_0, the dot products of keys are numbers that no state
// enters (worked out per run, a warp per group of four), and u_1 .. u_4 follow one from another without an exchange.
// Only products of decays occur, never a quotient.  GT = 1 (steps of single tokens) is the rule as it stands.
template <bool DELTA, int RPL, int L, int CPT, int GT, int TB>
__global__ void __launch_bounds__(128)
channel_scan_kernel(const float* qkv, const float* decay, const float* beta, const int* row_start, const int* row_slot,
                    float* state, long long slot_stride, float* out, int H, int G, int D, int Dv, int max_slots) {
  constexpr int COLS = 128 / L * CPT, DP = RPL * L, NP = RPL / 2, NV = GT * CPT;
  constexpr int ROWF = 3 * DP + COLS + 4;         // floats of one token: k | q | g | values | beta, 3 key dot products
  static_assert(NV <= L && TB % GT == 0 && COLS % 4 == 0, "sizes");
  extern __shared__ __align__(16) float runs[];   // two runs of TB tokens
  const int r = blockIdx.z, h = blockIdx.y;
  const int c0 = blockIdx.x * COLS;
  const int cg = threadIdx.x / L, sub = threadIdx.x % L;
  const int col0 = c0 + cg * CPT;
  for (int i = threadIdx.x; i < 2 * TB * 3 * (DP - D); i += 128) {             // rows d >= D are zero and stay so
    const int s = i / (3 * (DP - D)), e = i - s * 3 * (DP - D), which = e / (DP - D);
    runs[s * ROWF + which * DP + D + e - which * (DP - D)] = 0.f;
  }
  pdl_wait();
  pdl_trigger();
  const int slot = row_slot[r];
  if (slot < 0 || slot >= max_slots) return;
  const int first = row_start[r], n = row_start[r + 1] - first;
  const int C = 2 * G * D + H * Dv;
  const int g = h / (H / G);
  float* sp[CPT];
#pragma unroll
  for (int c = 0; c < CPT; ++c)                   // lanes beyond the last column follow it and write nothing
    sp[c] = state + (long long)slot * slot_stride + ((long long)h * Dv + min(col0 + c, Dv - 1)) * D;
  f32x2 S[CPT][NP];
  const bool vec = (D & 3) == 0 && (slot_stride & 3) == 0 && (((uintptr_t)state) & 15) == 0;
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int i = 0; i < RPL / 4; ++i) {
      const int d = 4 * (sub + L * i);
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (vec) {
        if (d < D) x = *reinterpret_cast<const float4*>(sp[c] + d);
      } else {
        if (d < D) x.x = sp[c][d];
        if (d + 1 < D) x.y = sp[c][d + 1];
        if (d + 2 < D) x.z = sp[c][d + 2];
        if (d + 3 < D) x.w = sp[c][d + 3];
      }
      S[c][2 * i] = pair_of(x.x, x.y);
      S[c][2 * i + 1] = pair_of(x.z, x.w);
    }
  const long long qoff = (long long)g * D, koff = (long long)(G + g) * D, voff = (long long)2 * G * D + (long long)h * Dv;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // 16-byte copies where a token's k, q and decays start on 16 bytes in global memory, else 4-byte ones
  const bool wide = (D & 3) == 0 && (C & 3) == 0 && (((uintptr_t)qkv) & 15) == 0 && (((uintptr_t)decay) & 15) == 0;
  const bool wide_v = wide && c0 + COLS <= Dv && (Dv & 3) == 0;
  auto cp = [](float* dst, const float* src, int bytes) {
    const unsigned sa = (unsigned)__cvta_generic_to_shared(dst);
    if (bytes == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(sa), "l"(src));
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(sa), "l"(src));
  };
  auto copy_run = [&](int run) {                  // tokens [run * TB, ...) of the row into buffer run & 1: a warp per token
    float* dst0 = runs + (run & 1) * TB * ROWF;
    const int t0 = run * TB, cnt = min(TB, n - t0);
    for (int s = warp; s < (cnt + GT - 1) / GT * GT; s += 4) {
      float* dst = dst0 + s * ROWF;
      if (s >= cnt) {                             // the last group's missing tokens change nothing: k = q = 0, g = 1, beta = 0
        for (int d = lane; d < DP; d += 32) {
          dst[d] = dst[DP + d] = 0.f;
          dst[2 * DP + d] = 1.f;
        }
        for (int e = lane; e < COLS + 4; e += 32) dst[3 * DP + e] = 0.f;
        continue;
      }
      const long long t = first + t0 + s;
      const float* row = qkv + t * C;
      const float* dec = decay + (t * H + h) * D;
      if (wide) {
        for (int d = 4 * lane; d < D; d += 128) {
          cp(dst + d, row + koff + d, 16);
          cp(dst + DP + d, row + qoff + d, 16);
          cp(dst + 2 * DP + d, dec + d, 16);
        }
      } else {
        for (int d = lane; d < D; d += 32) {
          cp(dst + d, row + koff + d, 4);
          cp(dst + DP + d, row + qoff + d, 4);
          cp(dst + 2 * DP + d, dec + d, 4);
        }
      }
      if (wide_v) {
        for (int e = 4 * lane; e < COLS; e += 128) cp(dst + 3 * DP + e, row + voff + c0 + e, 16);
      } else {
        for (int e = lane; e < COLS; e += 32) cp(dst + 3 * DP + e, row + voff + min(c0 + e, Dv - 1), 4);
      }
      if (DELTA && lane == 0) cp(dst + 3 * DP + COLS, beta + t * H + h, 4);
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  const int n_runs = (n + TB - 1) / TB;
  __syncthreads();                                // the zeros are written before any copy lands
  if (n_runs > 0) copy_run(0);
  for (int run = 0; run < n_runs; ++run) {
    if (run + 1 < n_runs) {
      copy_run(run + 1);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    float* buf = runs + (run & 1) * TB * ROWF;
    const int cnt = min(TB, n - run * TB);
    if (DELTA && GT == 4) {                       // the keys' dot products of the run's groups, a warp per group
      for (int s = 4 * warp; s < cnt; s += 16) {
        float* p0 = buf + s * ROWF;
        float a[6] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        for (int d = lane; d < DP; d += 32) {
          const float k0 = p0[d], k1 = p0[ROWF + d], k2 = p0[2 * ROWF + d], k3 = p0[3 * ROWF + d];
          const float g1 = p0[ROWF + 2 * DP + d], g2 = p0[2 * ROWF + 2 * DP + d], g3 = p0[3 * ROWF + 2 * DP + d];
          const float t1 = g1 * k1, t2 = g2 * k2, t3 = g3 * k3, w2 = g1 * t2, w3 = g2 * t3;
          a[0] = fmaf(k0, t1, a[0]);              // tokens 1, 0
          a[1] = fmaf(k1, t2, a[1]);              // 2, 1
          a[2] = fmaf(k0, w2, a[2]);              // 2, 0
          a[3] = fmaf(k2, t3, a[3]);              // 3, 2
          a[4] = fmaf(k1, w3, a[4]);              // 3, 1
          a[5] = fmaf(k0, g1 * w3, a[5]);         // 3, 0
        }
#pragma unroll
        for (int i = 0; i < 6; ++i) a[i] = warp_sum(a[i]);
        if (lane == 0) {
          p0[ROWF + 3 * DP + COLS + 1] = a[0];
          p0[2 * ROWF + 3 * DP + COLS + 1] = a[1];
          p0[2 * ROWF + 3 * DP + COLS + 2] = a[2];
          p0[3 * ROWF + 3 * DP + COLS + 1] = a[3];
          p0[3 * ROWF + 3 * DP + COLS + 2] = a[4];
          p0[3 * ROWF + 3 * DP + COLS + 3] = a[5];
        }
      }
      __syncthreads();
    }
    for (int s = 0; s < cnt; s += GT) {
      const float* p0 = buf + s * ROWF;
      auto fetch = [&](f32x2 (&x)[NP], int j, int which) {
#pragma unroll
        for (int i = 0; i < RPL / 4; ++i) {
          const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(p0 + j * ROWF + which * DP + 4 * (sub + L * i));
          x[2 * i] = w.x;
          x[2 * i + 1] = w.y;
        }
      };
      f32x2 k[GT][NP], gd[GT][NP];
#pragma unroll
      for (int j = 0; j < GT; ++j) {
        fetch(k[j], j, 0);
        fetch(gd[j], j, 2);
      }
      float u[NV];                                // what is written: u of token j, column c at [j * CPT + c]
#pragma unroll
      for (int j = 0; j < GT; ++j)
#pragma unroll
        for (int c = 0; c < CPT; ++c) u[j * CPT + c] = p0[j * ROWF + 3 * DP + cg * CPT + c];
      if (DELTA) {
        float dot[NV];
        f32x2 P[NP];
#pragma unroll
        for (int j = 0; j < GT; ++j) {
          f32x2 kt[NP];
#pragma unroll
          for (int i = 0; i < NP; ++i) {
            P[i] = j == 0 ? gd[0][i] : mul2(P[i], gd[j][i]);
            kt[i] = mul2(P[i], k[j][i]);
          }
#pragma unroll
          for (int c = 0; c < CPT; ++c) {
            f32x2 a = mul2(S[c][0], kt[0]), b = mul2(S[c][1], kt[1]);
#pragma unroll
            for (int i = 2; i < NP; i += 2) {
              a = fma2(S[c][i], kt[i], a);
              b = fma2(S[c][i + 1], kt[i + 1], b);
            }
            dot[j * CPT + c] = pair_sum(a) + pair_sum(b);
          }
        }
        all_reduce<NV, L>(dot, sub);
#pragma unroll
        for (int j = 0; j < GT; ++j) {
          const float4 x = *reinterpret_cast<const float4*>(p0 + j * ROWF + 3 * DP + COLS);       // beta, dot products
#pragma unroll
          for (int c = 0; c < CPT; ++c) {
            float v = u[j * CPT + c] - dot[j * CPT + c];
            if (j >= 1) v = fmaf(-x.y, u[(j - 1) * CPT + c], v);
            if (j >= 2) v = fmaf(-x.z, u[(j - 2) * CPT + c], v);
            if (j >= 3) v = fmaf(-x.w, u[(j - 3) * CPT + c], v);
            u[j * CPT + c] = x.x * v;
          }
        }
      }
      float o[NV];
#pragma unroll
      for (int j = 0; j < GT; ++j) {
        f32x2 q[NP];
        fetch(q, j, 1);
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          const f32x2 uu = pair_of(u[j * CPT + c], u[j * CPT + c]);
#pragma unroll
          for (int i = 0; i < NP; ++i) S[c][i] = fma2(k[j][i], uu, mul2(gd[j][i], S[c][i]));
          f32x2 a = mul2(S[c][0], q[0]), b = mul2(S[c][1], q[1]);
#pragma unroll
          for (int i = 2; i < NP; i += 2) {
            a = fma2(S[c][i], q[i], a);
            b = fma2(S[c][i + 1], q[i + 1], b);
          }
          o[j * CPT + c] = pair_sum(a) + pair_sum(b);
        }
      }
      const float mine = reduce_scatter<NV, L>(o, sub);
      const int at = sub * NV / L, j = at / CPT, c = at % CPT;
      if (sub % (L / NV) == 0 && s + j < cnt && col0 + c < Dv)
        out[(long long)(first + run * TB + s + j) * H * Dv + (long long)h * Dv + col0 + c] = mine;
    }
    __syncthreads();                              // the run is walked: its buffer may take the run after the next
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    if (col0 + c >= Dv) continue;
#pragma unroll
    for (int i = 0; i < RPL / 4; ++i) {
      const int d = 4 * (sub + L * i);
      float4 x;
      asm("mov.b64 {%0, %1}, %2;" : "=f"(x.x), "=f"(x.y) : "l"(S[c][2 * i]));
      asm("mov.b64 {%0, %1}, %2;" : "=f"(x.z), "=f"(x.w) : "l"(S[c][2 * i + 1]));
      if (vec) {
        if (d < D) *reinterpret_cast<float4*>(sp[c] + d) = x;
      } else {
        if (d < D) sp[c][d] = x.x;
        if (d + 1 < D) sp[c][d + 1] = x.y;
        if (d + 2 < D) sp[c][d + 2] = x.z;
        if (d + 3 < D) sp[c][d + 3] = x.w;
      }
    }
  }
}

}  // namespace

// single: every row of the step brings one token; the convolution state then moves on inside the kernel.
FMX_EXPORT int fmx_channel_delta_prepare(const void* proj, long long stride, const void* b, long long b_stride, const float* z,
                                         long long z_stride, const float* conv_w, const float* a_log, const float* dt_bias,
                                         const int* token_row, const int* row_start, const int* row_slot, float* state,
                                         long long slot_stride, long long conv_off, float* out_qkv, float* out_g, float* out_beta,
                                         int T, int R, int H, int G, int D, int Dv, int taps, int max_slots, int single,
                                         int dtype, int* status, cudaStream_t stream) {
  if (T == 0) return 0;
  if (T < 0 || R <= 0 || H <= 0 || G <= 0 || H % G || D <= 0 || D > 512 || Dv <= 0 || taps < 1 || taps > MAX_TAPS)
    return fmx_fail("fmx_channel_delta_prepare: bad sizes T=%d R=%d H=%d G=%d D=%d Dv=%d taps=%d", T, R, H, G, D, Dv, taps);
  const int C = 2 * G * D + H * Dv;
  if (stride < C || b_stride < H || z_stride < (long long)H * D) return fmx_fail("fmx_channel_delta_prepare: rows too narrow");
  // two channels at a time: every head, row and slot starts on a pair
  const bool two = D % 2 == 0 && Dv % 2 == 0 && stride % 2 == 0 && z_stride % 2 == 0 && slot_stride % 2 == 0 && conv_off % 2 == 0 &&
                   ((uintptr_t)z & 7) == 0 && ((uintptr_t)dt_bias & 7) == 0 && ((uintptr_t)state & 7) == 0 &&
                   ((uintptr_t)out_qkv & 7) == 0 && ((uintptr_t)out_g & 7) == 0 && ((uintptr_t)proj & (dtype == FMX_F32 ? 7 : 3)) == 0;
#define FMX_CDP(TT, MAXI)                                                                                              \
  do {                                                                                                                 \
    if (two) FMX_CDP_W(TT, MAXI, 2);                                                                                   \
    else FMX_CDP_W(TT, MAXI, 1);                                                                                       \
  } while (0)
#define FMX_CDP_W(TT, MAXI, W)                                                                                         \
  fmx_launch(channel_delta_prepare_kernel<TT, MAXI, W>, dim3(T, (2 * G + 2 * H + 3) / 4), dim3(128), 0, stream, (const TT*)proj, stride, \
             (const TT*)b, b_stride, z, z_stride, conv_w, a_log, dt_bias, token_row, row_start, row_slot, state, slot_stride, \
             conv_off, out_qkv, out_g, out_beta, H, G, D, Dv, taps, R, max_slots, single, status)
#define FMX_CDP_T(TT)                                                                                                  \
  do {                                                                                                                 \
    if (D <= 64) FMX_CDP(TT, 2);                                                                                       \
    else if (D <= 128) FMX_CDP(TT, 4);                                                                                 \
    else FMX_CDP(TT, 16);                                                                                              \
    if (!single && taps > 1)                                                                                           \
      fmx_launch(conv_state_update_kernel<TT>, dim3((C + 127) / 128, R), dim3(128), 0, stream, (const TT*)proj, stride, \
                 row_start, row_slot, state, slot_stride, conv_off, C, taps, max_slots);                               \
  } while (0)
  if (dtype == FMX_F32) FMX_CDP_T(float);
  else if (dtype == FMX_BF16) FMX_CDP_T(bf16);
  else return fmx_fail("fmx_channel_delta_prepare: unknown dtype %d", dtype);
#undef FMX_CDP_T
#undef FMX_CDP_W
#undef FMX_CDP
  FMX_LAUNCH_CHECK();
  return 0;
}

FMX_EXPORT int fmx_channel_gla_prepare(const void* proj, long long stride, const float* z, long long z_stride, const float* bias,
                                       float* out_qkv, float* out_g, int T, int H, int D, int Dv, float q_scale, float inv_tau,
                                       int dtype, cudaStream_t stream) {
  if (T == 0) return 0;
  const int HD = H * D, C = 2 * HD + H * Dv;
  if (T < 0 || H <= 0 || D <= 0 || Dv <= 0 || stride < C || z_stride < HD)
    return fmx_fail("fmx_channel_gla_prepare: bad sizes T=%d H=%d D=%d Dv=%d", T, H, D, Dv);
  const dim3 grid(T, (C + HD + 511) / 512);
  auto a16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (HD % 4 == 0 && C % 4 == 0 && stride % 4 == 0 && z_stride % 4 == 0 && a16(z) && a16(bias) && a16(out_qkv) && a16(out_g) &&
      ((uintptr_t)proj & (dtype == FMX_F32 ? 15 : 7)) == 0 && (dtype == FMX_F32 || dtype == FMX_BF16)) {
    if (dtype == FMX_F32)
      fmx_launch(channel_gla_prepare_vec_kernel<float>, grid, dim3(128), 0, stream, (const float*)proj, stride, z, z_stride, bias,
                 out_qkv, out_g, HD, C, q_scale, inv_tau);
    else
      fmx_launch(channel_gla_prepare_vec_kernel<bf16>, grid, dim3(128), 0, stream, (const bf16*)proj, stride, z, z_stride, bias,
                 out_qkv, out_g, HD, C, q_scale, inv_tau);
    FMX_LAUNCH_CHECK();
    return 0;
  }
  if (dtype == FMX_F32)
    fmx_launch(channel_gla_prepare_kernel<float>, grid, dim3(128), 0, stream, (const float*)proj, stride, z, z_stride, bias, out_qkv,
               out_g, HD, C, q_scale, inv_tau);
  else if (dtype == FMX_BF16)
    fmx_launch(channel_gla_prepare_kernel<bf16>, grid, dim3(128), 0, stream, (const bf16*)proj, stride, z, z_stride, bias, out_qkv,
               out_g, HD, C, q_scale, inv_tau);
  else
    return fmx_fail("fmx_channel_gla_prepare: unknown dtype %d", dtype);
  FMX_LAUNCH_CHECK();
  return 0;
}

// beta null: gated linear attention; else the delta rule.  single: every row brings one token.  lanes (8, 16, 32): lanes that
// share a column, cpt (1, 2, 4): columns that they hold; 0: the choice is made here.
FMX_EXPORT int fmx_channel_scan(const float* qkv, const float* decay, const float* beta, const int* row_start,
                                const int* row_slot, float* state, long long slot_stride, float* out, int R, int H, int G, int D,
                                int Dv, int max_slots, int single, int lanes, int cpt, cudaStream_t stream) {
  if (R == 0) return 0;
  if (R < 0 || H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 || D > 512)
    return fmx_fail("fmx_channel_scan: bad sizes R=%d H=%d G=%d D=%d Dv=%d", R, H, G, D, Dv);
  if (H > 65535 || R > 65535) return fmx_fail("fmx_channel_scan: batch too large");
  // Measured (us for 2,048 tokens of one request, 32 heads; delta rule / gated linear attention): 64 x 64 state: 8 lanes with one
  // column 418 / 291, with two 461 / 318, 16 lanes with two 389 / 265; 128 x 128: 16 lanes with one column 820 / 610, two
  // 630 / 453, four 747 / 358.  64 single tokens: 64 x 64: 8 lanes with two columns 23 / 23, 16 with two 31 / 29; 128 x 128: 16
  // lanes with one column 88 / 66, with four 68 / 59.
  const long long heads = (long long)R * H;
  const bool few = !single && heads * ((Dv + 15) / 16) < fmx_num_sms() * 3 / 2;           // one warp per scheduler at most
  if (lanes == 0) lanes = D <= 64 ? (few && D > 32 ? 16 : 8) : D <= 128 ? 16 : 32;
  if (lanes == 8 && D > 64) lanes = 16;
  if (lanes == 16 && D > 128) lanes = 32;
  if (lanes == 32 && D <= 128) lanes = 16;
  if (lanes != 8 && lanes != 16 && lanes != 32) return fmx_fail("fmx_channel_scan: 8, 16 or 32 lanes per column, not %d", lanes);
  const int most = D > 256 ? 1 : lanes == 8 ? 2 : 4;                          // four tokens' sums of a lane's columns fit its lanes
  if (cpt == 0) {                                 // as many columns per group of lanes as leave every multiprocessor a block
    cpt = most;
    while (cpt > 1 && heads * ((Dv + 128 / lanes * cpt - 1) / (128 / lanes * cpt)) < fmx_num_sms() * 3 / 4) cpt /= 2;
    if (beta != nullptr && !single && cpt == 4 && heads * ((Dv + 512 / lanes - 1) / (512 / lanes)) < fmx_num_sms()) cpt = 2;
    if (few && D <= 64 && lanes == 16) cpt = 2;
  }
  if (cpt != 1 && cpt != 2 && cpt != 4) return fmx_fail("fmx_channel_scan: 1, 2 or 4 columns per group of lanes, not %d", cpt);
  if (cpt > most) cpt = most;
#define FMX_CS(DELTA, RPL, L, CPT, GT, TB)                                                                             \
  do {                                                                                                                 \
    constexpr int cols = 128 / (L) * (CPT);                                                                            \
    constexpr size_t smem = (size_t)2 * (TB) * (3 * (RPL) * (L) + cols + 4) * sizeof(float);                           \
    if (smem > 48 * 1024)                                                                                              \
      cudaFuncSetAttribute(channel_scan_kernel<DELTA, RPL, L, CPT, GT, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    fmx_launch(channel_scan_kernel<DELTA, RPL, L, CPT, GT, TB>, dim3((Dv + cols - 1) / cols, H, R), dim3(128), smem, stream, qkv, \
               decay, beta, row_start, row_slot, state, slot_stride, out, H, G, D, Dv, max_slots);                     \
  } while (0)
#define FMX_CS_G(RPL, L, CPT, TB)                                                                                      \
  do {                                                                                                                 \
    if (beta != nullptr && single) FMX_CS(true, RPL, L, CPT, 1, 4);                                                    \
    else if (beta != nullptr) FMX_CS(true, RPL, L, CPT, 4, TB);                                                        \
    else if (single) FMX_CS(false, RPL, L, CPT, 1, 4);                                                                 \
    else FMX_CS(false, RPL, L, CPT, 4, TB);                                                                            \
  } while (0)
#define FMX_CS_C(RPL, L, TB)                                                                                          \
  do {                                                                                                                 \
    if (cpt == 1) FMX_CS_G(RPL, L, 1, TB);                                                                             \
    else if (cpt == 2) FMX_CS_G(RPL, L, 2, TB);                                                                        \
    else FMX_CS_G(RPL, L, 4, TB);                                                                                      \
  } while (0)
  if (lanes == 8) {
    if (D <= 32) { if (cpt == 1) FMX_CS_G(4, 8, 1, 16); else FMX_CS_G(4, 8, 2, 16); }
    else { if (cpt == 1) FMX_CS_G(8, 8, 1, 16); else FMX_CS_G(8, 8, 2, 16); }
  } else if (lanes == 16) {
    if (D <= 64) FMX_CS_C(4, 16, 16);
    else FMX_CS_C(8, 16, 16);
  } else if (D <= 256) FMX_CS_C(8, 32, 16);
  else FMX_CS_G(16, 32, 1, 8);
#undef FMX_CS_C
#undef FMX_CS_G
#undef FMX_CS
  FMX_LAUNCH_CHECK();
  return 0;
}
