// A matrix memory with exponential gates.
//
// Per head, with key k, query q (size D), value v (size Dv), log gates i and f, and the state S [D, Dv], n [D], m (all zero at a
// request's start), a token does
//     m' = max(f + m, i);   S <- exp(f + m - m') S + exp(i - m') k v^T;   n <- exp(f + m - m') n + exp(i - m') k;   m <- m'
//     o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
// n is one more column of S whose value is 1.  A slot's state is one run of 32-bit floats: S^T and n of every head, [H, Dv + 1, D], and
// then m of every head, [H].
//
//   mlstm_gates   steps with portions: the log gates of every token, capped, and the running maxima.  A token maps m to max(a + m, b)
//                 (a = f, b = i), and such maps compose; a block per (row, head) gives every thread a run of tokens, scans
//                 the runs' maps over its threads, and walks each run once more from the maximum in front of it.  Sums are
//                 taken along each path itself, never as differences of running totals.
//   mlstm_scan    steps with portions: the recurrence over every row's tokens, from the factors that mlstm_gates left, token by token.
//   mlstm_chunks  the same in runs of 64 tokens as matrix products, for bfloat16 projections: see there.
//   mlstm_step    rows of one token each: gates, recurrence, division, norm per head and output gate in one kernel, a block per
//                 (row, head): the state is read once and written once, and nothing else of its size is touched.
//
// Everything is 32-bit but the projections that come in and the activations that go out.  No sum's order depends on what else is in
// the batch.
#include <math.h>
#include "common.cuh"
#include "packed.cuh"

namespace {
__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// z [T, z_stride] 32-bit: input gates (H) | forget gates (H); bias [2 H]; out [T, H]: (kept by, put in by, exp(-m), log of kept by).
template <int GATE_THREADS>
__global__ void __launch_bounds__(GATE_THREADS)
mlstm_gates_kernel(const float* z, long long z_stride, const float* __restrict__ bias, float cap, const int* row_start,
                   const int* row_slot, float* state, long long slot_stride, long long m_off, float4* out, int H, int max_slots) {
  __shared__ float wa[GATE_THREADS / 32], wb[GATE_THREADS / 32];
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, r = blockIdx.y;
  const int slot = row_slot[r];
  if (slot < 0 || slot >= max_slots) return;
  const int first = row_start[r], n = row_start[r + 1] - first;
  if (n <= 0) return;
  float* mp = state + (long long)slot * slot_stride + m_off + h;
  const float m0 = *mp;
  const float bi = bias[h], bf = bias[H + h];
  const int per = (n + GATE_THREADS - 1) / GATE_THREADS;
  const int t0 = threadIdx.x * per, t1 = min(n, t0 + per);
  float a = 0.f, b = -INFINITY;                    // this thread's tokens as one map m -> max(a + m, b)
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    const float* zr = z + (long long)(first + t) * z_stride;
    const float i = capped(zr[h] + bi, cap), f = log_sigmoid(capped(zr[H + h] + bf, cap));
    out[(long long)(first + t) * H + h] = make_float4(f, i, 0.f, 0.f);         // read again below by this same thread
    b = fmaxf(b + f, i);
    a += f;
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
  for (int d = 1; d < 32; d <<= 1) {
    const float pa = __shfl_up_sync(0xffffffffu, a, d), pb = __shfl_up_sync(0xffffffffu, b, d);
    if (lane >= d) {                               // the earlier tokens' map first, then this one
      b = fmaxf(pb + a, b);
      a += pa;
    }
  }
  if (lane == 31) { wa[warp] = a; wb[warp] = b; }
  float xa = __shfl_up_sync(0xffffffffu, a, 1), xb = __shfl_up_sync(0xffffffffu, b, 1);
  __syncthreads();
  float m = m0;
  for (int w = 0; w < warp; ++w) m = fmaxf(wa[w] + m, wb[w]);
  if (lane > 0) m = fmaxf(xa + m, xb);
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    float4* g = out + (long long)(first + t) * H + h;
    const float4 x = *g;
    const float mn = fmaxf(x.x + m, x.y);
    const float lk = x.x + m - mn;
    *g = make_float4(expf(lk), expf(x.y - mn), expf(-mn), lk);
    m = mn;
  }
  if (t0 < n && t1 == n) *mp = m;                  // (every thread has read the old one: the barrier above)
}

// Four neighbouring values of which `have` exist (the others are zero); `vec`, the same for all threads: their starts are aligned
// for one access and `have` is four or more, or none.  Selects and not branches: the lanes stay together.
template <typename T> __device__ __forceinline__ float4 some4(const T* p, int have, bool vec) {
  float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
  if (vec) {
    if (have >= 4) x = load4(p);
  } else {
    x.x = have > 0 ? to_f(p[0]) : 0.f;
    x.y = have > 1 ? to_f(p[1]) : 0.f;
    x.z = have > 2 ? to_f(p[2]) : 0.f;
    x.w = have > 3 ? to_f(p[3]) : 0.f;
  }
  return x;
}

// Columns of S are independent; column Dv is n.  grid (ceil((Dv + 1) / COLS), H, R), 128 threads: L adjacent lanes hold CPT
// neighbouring columns, lane `sub` the rows 4 (sub + L i) .. + 3, i < RPL / 4 (D <= RPL L), in registers.  A token's k, q and the block's
// values go through registers into shared memory as 32-bit floats in runs of TB tokens: a run is fetched while the one before
// it is walked.  Four tokens' read-outs are summed over the lanes together.  proj [T, stride]: q (H*D) | k (H*D) | v (H*Dv) | ...; out [T, H*Dv]
// and nq [T, H]: S^T q and n . q with q scaled by D^-1/2, not divided yet.
template <typename T, int RPL, int L, int CPT, int TB>
__global__ void __launch_bounds__(128)
mlstm_scan_kernel(const T* proj, long long stride, const float4* gates, const int* row_start, const int* row_slot, float* state,
                  long long slot_stride, float* out, float* nq, int H, int D, int Dv, int max_slots, int vec_in) {
  constexpr int COLS = 128 / L * CPT, DP = RPL * L, NP = RPL / 2, GT = 4, NV = GT * CPT;
  constexpr int ROWF = 2 * DP + COLS + 4;          // floats of one token: k | q | values | kept by, put in by
  constexpr int CH = (2 * DP + COLS) / 4;          // pieces of four of one token
  constexpr int NIT = (TB * CH + 127) / 128;
  static_assert(NV <= L && TB % GT == 0 && COLS % 4 == 0 && DP % 4 == 0 && TB <= 128, "sizes");
  extern __shared__ __align__(16) float runs[];    // two runs of TB tokens
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.z, h = blockIdx.y;
  const int slot = row_slot[r];
  if (slot < 0 || slot >= max_slots) return;
  const int c0 = blockIdx.x * COLS;
  const int cg = threadIdx.x / L, sub = threadIdx.x % L;
  const int col0 = c0 + cg * CPT;
  const int first = row_start[r], n = row_start[r + 1] - first;
  float* sp[CPT];
#pragma unroll
  for (int c = 0; c < CPT; ++c)                    // lanes beyond n's column follow it and write nothing
    sp[c] = state + (long long)slot * slot_stride + ((long long)h * (Dv + 1) + min(col0 + c, Dv)) * D;
  f32x2 S[CPT][NP];
  const bool vec = (D & 3) == 0 && (slot_stride & 3) == 0 && (((uintptr_t)state) & 15) == 0;
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int i = 0; i < RPL / 4; ++i) {
      const int d = 4 * (sub + L * i);
      const float4 x = some4(sp[c] + d, D - d, vec);
      S[c][2 * i] = pair_of(x.x, x.y);
      S[c][2 * i + 1] = pair_of(x.z, x.w);
    }
  const long long qoff = (long long)h * D, koff = (long long)(H + h) * D, voff = (long long)2 * H * D + (long long)h * Dv;
  const float q_scale = 1.0f / sqrtf((float)D);
  float4 ahead[NIT];
  float2 ahead_gate = make_float2(1.f, 0.f);
  auto fetch_run = [&](int run) {                  // what this thread brings of tokens [run * TB, ...)
    const int t0 = run * TB, cnt = min(TB, n - t0);
#pragma unroll
    for (int it = 0; it < NIT; ++it) {
      const int item = threadIdx.x + it * 128;
      const int s = item / CH, e = 4 * (item - s * CH);
      // one source per piece of four: k, q or the values (a run's missing tokens have none: k = q = v = 0)
      const T* row = proj + (long long)(first + t0 + min(s, cnt - 1)) * stride;
      const bool is_k = e < DP, is_q = !is_k && e < 2 * DP;
      const int d = is_k ? e : is_q ? e - DP : c0 + e - 2 * DP;
      const T* src = row + (is_k ? koff : is_q ? qoff : voff) + d;
      const int have = s < cnt ? (is_k || is_q ? D : Dv) - d : 0;
      float4 x = some4(src, have, vec_in);
      const int one = is_k || is_q || s >= cnt ? -1 : Dv - d;          // n's column has the value 1
      x.x = one == 0 ? 1.f : x.x;
      x.y = one == 1 ? 1.f : x.y;
      x.z = one == 2 ? 1.f : x.z;
      x.w = one == 3 ? 1.f : x.w;
      ahead[it] = x;
    }
    if (threadIdx.x < TB) {
      ahead_gate = make_float2(1.f, 0.f);          // a missing token changes nothing
      if (threadIdx.x < cnt) {
        const float4 g = gates[(long long)(first + t0 + threadIdx.x) * H + h];
        ahead_gate = make_float2(g.x, g.y);
      }
    }
  };
  const int n_runs = (n + TB - 1) / TB;
  if (n_runs > 0) fetch_run(0);
  for (int run = 0; run < n_runs; ++run) {
    float* buf = runs + (run & 1) * TB * ROWF;     // walked last two runs ago, behind the barrier of the run before this one
#pragma unroll
    for (int it = 0; it < NIT; ++it) {
      const int item = threadIdx.x + it * 128;
      const int s = item / CH, e = 4 * (item - s * CH);
      if (TB * CH % 128 == 0 || s < TB) *reinterpret_cast<float4*>(buf + s * ROWF + e) = ahead[it];
    }
    if (threadIdx.x < TB) *reinterpret_cast<float2*>(buf + threadIdx.x * ROWF + 2 * DP + COLS) = ahead_gate;
    __syncwarp();
    __syncthreads();
    if (run + 1 < n_runs) fetch_run(run + 1);
    const int cnt = min(TB, n - run * TB);
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
      float o[NV];
#pragma unroll
      for (int j = 0; j < GT; ++j) {
        f32x2 k[NP], q[NP];
        fetch(k, j, 0);
        fetch(q, j, 1);
        const float2 g = *reinterpret_cast<const float2*>(p0 + j * ROWF + 2 * DP + COLS);
        const f32x2 keep = pair_of(g.x, g.x);
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          const float u = g.y * p0[j * ROWF + 2 * DP + cg * CPT + c];
          const f32x2 uu = pair_of(u, u);
#pragma unroll
          for (int i = 0; i < NP; ++i) S[c][i] = fma2(k[i], uu, mul2(keep, S[c][i]));
          f32x2 a = mul2(S[c][0], q[0]), b = mul2(S[c][1], q[1]);
#pragma unroll
          for (int i = 2; i < NP; i += 2) {
            a = fma2(S[c][i], q[i], a);
            b = fma2(S[c][i + 1], q[i + 1], b);
          }
          o[j * CPT + c] = pair_sum(a) + pair_sum(b);
        }
      }
      __syncwarp();
      const float mine = reduce_scatter<NV, L>(o, sub) * q_scale;
      const int at = sub * NV / L, j = at / CPT, col = col0 + at % CPT;
      if (sub % (L / NV) == 0 && s + j < cnt && col <= Dv) {
        const long long t = first + run * TB + s + j;
        if (col < Dv) out[t * H * Dv + (long long)h * Dv + col] = mine;
        else nq[t * H + h] = mine;
      }
    }
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    if (col0 + c > Dv) continue;
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

// ---- the recurrence in runs of 64 tokens as matrix products
//
// Inside a run, with a_t = what token t keeps the state by, p_t = what it is put in by, G_t = log a_1 + .. + log a_t from the run's start,
// and S_0, n_0 in front of it,
//     S_t^T q_t = exp(G_t) S_0^T q_t + sum_{s <= t} (q_t . k_s) exp(G_t - G_s) p_s v_s,
//     n_t . q_t = exp(G_t) n_0 . q_t + sum_{s <= t} (q_t . k_s) exp(G_t - G_s) p_s,
//     S_64 = exp(G_64) S_0 + sum_s exp(G_64 - G_s) p_s k_s v_s^T      (n_64 with k_s alone).
// q, k and v are bfloat16 as projected, so q . k^T is exact up to its 32-bit sums; what is 32-bit enters its product as two bfloat16
// terms (x = hi + lo to 2^-17 of x): the weights of a run's own tokens against v, S_0 against q, and the weighed values against k.
// S itself stays in 32-bit accumulators.  G is summed in 64-bit and kept as two floats, so that a difference of two of them
// is as good as a sum over the tokens between (they are held as logarithms of base 2).  A request's runs start where its portion does.
//
// grid (ceil(Dv / VB), H, R), four warps; a block owns VB columns of S (the first one n as well).  Warp w takes tokens 16 w .. + 15 of a run
// for the read-out, and a 16-row strip of S^T [VB, D] by NT tiles of eight columns for its update.  q, k, v of the next run are
// copied (cp.async) while the present one is worked on.
constexpr int CHUNK = 64;
template <int KD, int VB> struct ChunkSize {
  static constexpr int D = 16 * KD, QP = D + 8, VP = VB + 8;        // rows of 16 bytes more than their width: no bank conflicts
  static constexpr int STAGE = 2 * CHUNK * QP + CHUNK * VP;         // q, k, v of a run
  static constexpr size_t SMEM = (size_t)(2 * STAGE + 2 * CHUNK * VP + 2 * VB * QP) * sizeof(bf16) + (4 * CHUNK * 4 + D) * sizeof(float);
};

__device__ __forceinline__ void ldsm4(unsigned (&r)[4], const bf16* p) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldsm4t(unsigned (&r)[4], const bf16* p) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as two pairs of bfloat16: hi = their roundings, lo = the roundings of what is left
__device__ __forceinline__ void two_terms(float x, float y, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 hf = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - hf.x, y - hf.y);
  hi = *reinterpret_cast<const unsigned*>(&h);
  lo = *reinterpret_cast<const unsigned*>(&l);
}

template <int KD, int VB>
__global__ void __launch_bounds__(128)
mlstm_chunk_kernel(const bf16* proj, long long stride, const float4* gates, const int* row_start, const int* row_slot, float* state,
                   long long slot_stride, float* out, float* nq, int H, int Dv, int max_slots) {
  using Z = ChunkSize<KD, VB>;
  constexpr int D = Z::D, QP = Z::QP, VP = Z::VP, NV = VB / 8;
  constexpr int MW = VB / 16, NW = 4 / MW, NT = D / 8 / NW;        // warps along S^T's rows and columns; tiles of eight columns per warp
  static_assert(NT % 2 == 0 && NV % 2 == 0, "tiles are fetched in pairs");
  extern __shared__ __align__(16) unsigned char chunk_smem[];
  bf16* stages = reinterpret_cast<bf16*>(chunk_smem);
  bf16* vh = stages + 2 * Z::STAGE;                // weighed values, two terms
  bf16* vl = vh + CHUNK * VP;
  bf16* sh = vl + CHUNK * VP;                      // S^T in front of the run, two terms
  bf16* sl = sh + VB * QP;
  float4* gs = reinterpret_cast<float4*>(sl + VB * QP);            // per warp and token: G in two floats, p, exp(G_64 - G) p
  float* n_s = reinterpret_cast<float*>(gs + 4 * CHUNK);
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * VB;
  const int slot = row_slot[r];
  if (slot < 0 || slot >= max_slots) return;
  const int first = row_start[r], n = row_start[r + 1] - first;
  if (n <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
  const bool with_n = blockIdx.x == 0;
  float* st = state + (long long)slot * slot_stride + (long long)h * (Dv + 1) * D;
  const bf16* qp = proj + (long long)first * stride + (long long)h * D;
  const bf16* kp = qp + (long long)H * D;
  const bf16* vp = proj + (long long)first * stride + 2LL * H * D + (long long)h * Dv + v0;
  const float q_scale = 1.0f / sqrtf((float)D);
  const int mi = warp % MW, d0 = (warp / MW) * NT * 8;             // this warp's strip of S^T: rows 16 mi, columns d0
  float s[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int v = 16 * mi + g + 8 * x;
      float2 y = make_float2(0.f, 0.f);
      if (v0 + v < Dv) y = *reinterpret_cast<const float2*>(st + (long long)(v0 + v) * D + d0 + 8 * i + 2 * q4);
      s[i][2 * x] = y.x;
      s[i][2 * x + 1] = y.y;
    }
  if (with_n && tid < D) n_s[tid] = st[(long long)Dv * D + tid];
  auto put_state = [&]() {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        unsigned hi, lo;
        two_terms(s[i][2 * x], s[i][2 * x + 1], hi, lo);
        const int at = (16 * mi + g + 8 * x) * QP + d0 + 8 * i + 2 * q4;
        *reinterpret_cast<unsigned*>(sh + at) = hi;
        *reinterpret_cast<unsigned*>(sl + at) = lo;
      }
  };
  put_state();
  auto cp16 = [](bf16* dst, const bf16* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0));
  };
  auto copy_run = [&](int run) {                   // what is missing (tokens behind the row's end, columns behind Dv) is zero
    bf16* qs = stages + (run & 1) * Z::STAGE;
    const int t0 = run * CHUNK;
#pragma unroll
    for (int i = tid; i < CHUNK * 2 * KD; i += 128) {
      const int t = i / (2 * KD), c = 8 * (i - t * 2 * KD);
      const bool ok = t0 + t < n;
      const long long off = ok ? (long long)(t0 + t) * stride + c : 0;
      cp16(qs + t * QP + c, qp + off, ok);
      cp16(qs + CHUNK * QP + t * QP + c, kp + off, ok);
    }
#pragma unroll
    for (int i = tid; i < CHUNK * NV; i += 128) {
      const int t = i / NV, c = 8 * (i - t * NV);
      const bool ok = t0 + t < n && v0 + c < Dv;
      cp16(qs + 2 * CHUNK * QP + t * VP + c, ok ? vp + (long long)(t0 + t) * stride + c : vp, ok);
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  float2 ga[2];                                    // (put in by, log of kept by) of this lane's two tokens of a run
  auto fetch_gates = [&](int run) {
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int t = run * CHUNK + 2 * lane + x;
      const float4 y = gates[(long long)(first + min(t, n - 1)) * H + h];
      ga[x] = t < n ? make_float2(y.y, y.w) : make_float2(0.f, 0.f);
    }
  };
  const int runs = (n + CHUNK - 1) / CHUNK;
  copy_run(0);
  fetch_gates(0);
  for (int run = 0; run < runs; ++run) {
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();                               // the run's operands and S are there, and the other stage is no longer read
    const bf16* qs = stages + (run & 1) * Z::STAGE;
    const bf16* ks = qs + CHUNK * QP;
    const bf16* vs = ks + CHUNK * QP;
    if (run + 1 < runs) copy_run(run + 1);
    // ---- G: every warp for itself, two tokens per lane
    double total;
    {
      const double log2e = 1.4426950408889634074;
      const double a = (double)ga[0].y * log2e, b = a + (double)ga[1].y * log2e;
      double inc = b;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, inc, d);
        inc += lane >= d ? up : 0.0;
      }
      total = __shfl_sync(0xffffffffu, inc, 31);
      const double G[2] = {inc - b + a, inc};
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const float hi = (float)G[x];
        gs[warp * CHUNK + 2 * lane + x] = make_float4(hi, (float)(G[x] - (double)hi), ga[x].x, exp2f((float)(total - G[x])) * ga[x].x);
      }
    }
    const float keep_all = exp2f((float)total);
    if (run + 1 < runs) fetch_gates(run + 1);
    __syncwarp();
    const float4* gw = gs + warp * CHUNK;
    // ---- the weighed values in two terms
#pragma unroll
    for (int i = tid; i < CHUNK * VB / 2; i += 128) {
      const int t = i / (VB / 2), c = 2 * (i - t * (VB / 2));
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vs + t * VP + c));
      const float w = gw[t].w;
      unsigned hi, lo;
      two_terms(v.x * w, v.y * w, hi, lo);
      *reinterpret_cast<unsigned*>(vh + t * VP + c) = hi;
      *reinterpret_cast<unsigned*>(vl + t * VP + c) = lo;
    }
    // ---- read-out of this warp's 16 tokens
    const int t_lo = 16 * warp + g;
    const float4 g_lo = gw[t_lo], g_hi = gw[t_lo + 8];
    unsigned aq[KD][4];
#pragma unroll
    for (int kd = 0; kd < KD; ++kd) ldsm4(aq[kd], qs + (16 * warp + (lane & 7) + ((lane >> 3) & 1) * 8) * QP + 16 * kd + (lane >> 4) * 8);
    float o[NV][4];
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const int bn = (lane & 7) + (lane >> 4) * 8, bk = ((lane >> 3) & 1) * 8;          // operands in rows of k
    const int tk = (lane & 7) + ((lane >> 3) & 1) * 8, tn = (lane >> 4) * 8;          // operands in rows of n, transposed on their way
#pragma unroll
    for (int kd = 0; kd < KD; ++kd)
#pragma unroll
      for (int p = 0; p < NV / 2; ++p) {
        unsigned b[4];
        ldsm4(b, sh + (16 * p + bn) * QP + 16 * kd + bk);
        mma16816(o[2 * p], aq[kd], b[0], b[1]);
        mma16816(o[2 * p + 1], aq[kd], b[2], b[3]);
        ldsm4(b, sl + (16 * p + bn) * QP + 16 * kd + bk);
        mma16816(o[2 * p], aq[kd], b[0], b[1]);
        mma16816(o[2 * p + 1], aq[kd], b[2], b[3]);
      }
    const float e_lo = exp2f(g_lo.x), e_hi = exp2f(g_hi.x);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      o[i][0] *= e_lo; o[i][1] *= e_lo;
      o[i][2] *= e_hi; o[i][3] *= e_hi;
    }
    float sum_lo = 0.f, sum_hi = 0.f;
    // 32 keys at a time: the scores of all of them before any exponential, so that the products' latencies overlap (keys behind
    // a token weigh nothing; every warp takes the same time)
#pragma unroll
    for (int kp = 0; kp < 2; ++kp) {
      float c[4][4];
#pragma unroll
      for (int x = 0; x < 4; ++x) c[x][0] = c[x][1] = c[x][2] = c[x][3] = 0.f;
#pragma unroll
      for (int kd = 0; kd < KD; ++kd)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          unsigned b[4];
          ldsm4(b, ks + (32 * kp + 16 * y + bn) * QP + 16 * kd + bk);
          mma16816(c[2 * y], aq[kd], b[0], b[1]);
          mma16816(c[2 * y + 1], aq[kd], b[2], b[3]);
        }
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = 32 * kp + 8 * x + 2 * q4 + e;              // the token whose key and value this is
          const float4 y = gw[t];
          const float w_lo = (g_lo.x - y.x) + (g_lo.y - y.y), w_hi = (g_hi.x - y.x) + (g_hi.y - y.y);
          c[x][e] *= exp2f(t <= t_lo ? w_lo : -INFINITY) * y.z;
          c[x][2 + e] *= exp2f(t <= t_lo + 8 ? w_hi : -INFINITY) * y.z;
          sum_lo += c[x][e];
          sum_hi += c[x][2 + e];
        }
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        unsigned ah[4], al[4];
        two_terms(c[2 * y][0], c[2 * y][1], ah[0], al[0]);
        two_terms(c[2 * y][2], c[2 * y][3], ah[1], al[1]);
        two_terms(c[2 * y + 1][0], c[2 * y + 1][1], ah[2], al[2]);
        two_terms(c[2 * y + 1][2], c[2 * y + 1][3], ah[3], al[3]);
#pragma unroll
        for (int p = 0; p < NV / 2; ++p) {
          unsigned b[4];
          ldsm4t(b, vs + (32 * kp + 16 * y + tk) * VP + 16 * p + tn);
          mma16816(o[2 * p], ah, b[0], b[1]);
          mma16816(o[2 * p + 1], ah, b[2], b[3]);
          mma16816(o[2 * p], al, b[0], b[1]);
          mma16816(o[2 * p + 1], al, b[2], b[3]);
        }
      }
    }
    const long long tok = first + (long long)run * CHUNK + t_lo;
    const int left = n - run * CHUNK - t_lo;       // tokens from t_lo to the row's end
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = v0 + 8 * i + 2 * q4;
      if (c >= Dv) continue;
      if (left > 0) *reinterpret_cast<float2*>(out + tok * H * Dv + (long long)h * Dv + c) = make_float2(o[i][0] * q_scale, o[i][1] * q_scale);
      if (left > 8) *reinterpret_cast<float2*>(out + (tok + 8) * H * Dv + (long long)h * Dv + c) = make_float2(o[i][2] * q_scale, o[i][3] * q_scale);
    }
    if (with_n) {                                  // n . q: two lanes per token for n_0 . q, then the sums of the weights
      const bf16* qr = qs + (16 * warp + (lane >> 1)) * QP + (lane & 1) * (D / 2);
      const float* nr = n_s + (lane & 1) * (D / 2);
      float dot = 0.f;
#pragma unroll 8
      for (int d = 0; d < D / 2; d += 2) {
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(qr + d));
        dot = fmaf(x.x, nr[d], fmaf(x.y, nr[d + 1], dot));
      }
      dot += __shfl_xor_sync(0xffffffffu, dot, 1);
      const float n_lo = __shfl_sync(0xffffffffu, dot, 2 * g), n_hi = __shfl_sync(0xffffffffu, dot, 2 * g + 16);
#pragma unroll
      for (int d = 1; d < 4; d <<= 1) {
        sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, d);
        sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, d);
      }
      if (q4 == 0 && left > 0) nq[tok * H + h] = fmaf(e_lo, n_lo, sum_lo) * q_scale;
      if (q4 == 0 && left > 8) nq[(tok + 8) * H + h] = fmaf(e_hi, n_hi, sum_hi) * q_scale;
    }
    __syncthreads();                               // the weighed values are there, and S and n of the run's start are no longer read
    // ---- S and n behind the run
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[i][e] *= keep_all;
    const int ak = (lane & 7) + (lane >> 4) * 8, am = ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      unsigned ah[4], al[4];
      ldsm4t(ah, vh + (16 * kk + ak) * VP + 16 * mi + am);
      ldsm4t(al, vl + (16 * kk + ak) * VP + 16 * mi + am);
#pragma unroll
      for (int p = 0; p < NT / 2; ++p) {
        unsigned b[4];
        ldsm4t(b, ks + (16 * kk + tk) * QP + d0 + 16 * p + tn);
        mma16816(s[2 * p], ah, b[0], b[1]);
        mma16816(s[2 * p + 1], ah, b[2], b[3]);
        mma16816(s[2 * p], al, b[0], b[1]);
        mma16816(s[2 * p + 1], al, b[2], b[3]);
      }
    }
    if (with_n && tid < D) {
      float a[4] = {keep_all * n_s[tid], 0.f, 0.f, 0.f};
#pragma unroll 4
      for (int t = 0; t < CHUNK; t += 4)
#pragma unroll
        for (int x = 0; x < 4; ++x) a[x] = fmaf(gw[t + x].w, __bfloat162float(ks[(t + x) * QP + tid]), a[x]);
      n_s[tid] = (a[0] + a[1]) + (a[2] + a[3]);
    }
    put_state();
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int v = v0 + 16 * mi + g + 8 * x;
      if (v < Dv) *reinterpret_cast<float2*>(st + (long long)v * D + d0 + 8 * i + 2 * q4) = make_float2(s[i][2 * x], s[i][2 * x + 1]);
    }
  if (with_n && tid < D) st[(long long)Dv * D + tid] = n_s[tid];
}

// Rows of one token.  grid (H, R), STEP_THREADS threads: LN neighbouring lanes take a row of S^T, each NI pieces of four of its D
// values; U rows per group of lanes are in flight at a time, and the first group's lanes hold n beside them.  proj row: q | k | v | output gate; z: as in mlstm_gates.
constexpr int STEP_THREADS = 256;
template <typename TP, typename TO, int LN, int NI>
__global__ void __launch_bounds__(STEP_THREADS, NI == 1 ? 4 : 1)
mlstm_step_kernel(const TP* proj, long long stride, const float* z, long long z_stride, const float* __restrict__ bias, float cap,
                  const int* row_start, const int* row_slot, float* state, long long slot_stride, long long m_off,
                  const float* __restrict__ w, float eps, TO* out, long long out_stride, int H, int D, int Dv, int max_slots, int vec_in) {
  constexpr int GROUPS = STEP_THREADS / LN, U = NI >= 4 ? 2 : 4;
  extern __shared__ float o_s[];                   // Dv + 1 read-outs
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, r = blockIdx.y;
  const int slot = row_slot[r];
  const long long t = row_start[r];
  if (slot < 0 || slot >= max_slots) {             // a padding row of a captured step
    if (row_start[r + 1] > t)
      for (int e = threadIdx.x; e < Dv; e += STEP_THREADS) out[t * out_stride + (long long)h * Dv + e] = from_f<TO>(0.f);
    return;
  }
  float* sp = state + (long long)slot * slot_stride + (long long)h * (Dv + 1) * D;
  float* mp = state + (long long)slot * slot_stride + m_off + h;
  const int sub = threadIdx.x % LN, grp = threadIdx.x / LN;
  const bool vec = (D & 3) == 0 && (slot_stride & 3) == 0 && (((uintptr_t)state) & 15) == 0;
  const TP* row = proj + t * stride;
  float4 S[U][NI];
  auto load_rows = [&](int j0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int j = j0 + u * GROUPS;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = 4 * (sub + LN * i);
        S[u][i] = some4(sp + (long long)j * D + d, j < Dv ? D - d : 0, vec);
      }
    }
  };
  load_rows(grp);
  float4 N[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = 4 * (sub + LN * i);
    N[i] = some4(sp + (long long)Dv * D + d, grp == 0 ? D - d : 0, vec);
  }
  const float m0 = *mp;
  const float gi = capped(z[t * z_stride + h] + bias[h], cap);
  const float gf = log_sigmoid(capped(z[t * z_stride + H + h] + bias[H + h], cap));
  const float m = fmaxf(gf + m0, gi);
  const float keep = expf(gf + m0 - m), put = expf(gi - m);
  const float q_scale = 1.0f / sqrtf((float)D);
  float4 k[NI], q[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = 4 * (sub + LN * i);
    q[i] = some4(row + (long long)h * D + d, D - d, vec_in);
    k[i] = some4(row + (long long)(H + h) * D + d, D - d, vec_in);
  }
  const TP* vrow = row + (long long)2 * H * D + (long long)h * Dv;
  // one row's step: S <- keep S + x k, written back; -> this lane's part of S . q
  auto advance = [&](float4 (&y)[NI], float x, float* dst, bool live) {
    float dot = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      float4& v = y[i];
      v.x = fmaf(k[i].x, x, keep * v.x);
      v.y = fmaf(k[i].y, x, keep * v.y);
      v.z = fmaf(k[i].z, x, keep * v.z);
      v.w = fmaf(k[i].w, x, keep * v.w);
      dot = fmaf(v.x, q[i].x, fmaf(v.y, q[i].y, fmaf(v.z, q[i].z, fmaf(v.w, q[i].w, dot))));
      const int d = 4 * (sub + LN * i), have = live ? D - d : 0;
      if (vec) {
        if (have > 0) *reinterpret_cast<float4*>(dst + d) = v;
      } else {
        if (have > 0) dst[d] = v.x;
        if (have > 1) dst[d + 1] = v.y;
        if (have > 2) dst[d + 2] = v.z;
        if (have > 3) dst[d + 3] = v.w;
      }
    }
    return dot;
  };
  for (int j0 = grp; j0 - grp < Dv; j0 += U * GROUPS) {        // (the same number of passes for every group of lanes)
    float dot[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int j = j0 + u * GROUPS;
      dot[u] = advance(S[u], put * (j < Dv ? to_f(vrow[j]) : 0.f), sp + (long long)j * D, j < Dv);
    }
    if (j0 - grp + U * GROUPS < Dv) load_rows(j0 + U * GROUPS);
    __syncwarp();
#pragma unroll
    for (int u = 0; u < U; ++u) {
#pragma unroll
      for (int e = LN / 2; e >= 1; e >>= 1) dot[u] += __shfl_xor_sync(0xffffffffu, dot[u], e);
      const int j = j0 + u * GROUPS;
      if (sub == 0 && j < Dv) o_s[j] = dot[u] * q_scale;
    }
  }
  if (threadIdx.x < 32) {                          // n, by the first group of lanes
    float dot = advance(N, put, sp + (long long)Dv * D, grp == 0);
    __syncwarp();
#pragma unroll
    for (int e = LN / 2; e >= 1; e >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, e);
    if (threadIdx.x == 0) o_s[Dv] = dot * q_scale;
  }
  __syncthreads();
  if (threadIdx.x == 0) *mp = m;
  const float mul = 1.0f / (fmaxf(fabsf(o_s[Dv]), expf(-m)) + 1e-6f);
  float ss = 0.f;
  for (int e = threadIdx.x; e < Dv; e += STEP_THREADS) ss = fmaf(o_s[e] * mul, o_s[e] * mul, ss);
  const float rstd = mul / sqrtf(block_sum<STEP_THREADS>(ss) / (float)Dv + eps);
  const TP* grow = vrow - (long long)h * Dv + (long long)H * Dv + (long long)h * Dv;
  for (int e = threadIdx.x; e < Dv; e += STEP_THREADS)
    out[t * out_stride + (long long)h * Dv + e] =
        from_f<TO>(o_s[e] * rstd * w[(long long)h * Dv + e] * (1.0f / (1.0f + expf(-to_f(grow[e])))));
}
}  // namespace

FMX_EXPORT int fmx_mlstm_gates(const float* z, long long z_stride, const float* bias, float cap, const int* row_start,
                               const int* row_slot, float* state, long long slot_stride, long long m_off, float* gates, int R, int H,
                               int max_slots, int longest, cudaStream_t stream) {
  if (R == 0) return 0;
  if (R < 0 || R > 65535 || H <= 0 || z_stride < 2LL * H || !(cap > 0.f) || ((uintptr_t)gates & 15))
    return fmx_fail("fmx_mlstm_gates: bad arguments R=%d H=%d cap=%g", R, H, (double)cap);
  // a row's tokens are shared out over the block's threads: more of them for long portions (longest: the longest row's tokens)
  if (longest > 256)
    fmx_launch(mlstm_gates_kernel<512>, dim3(H, R), dim3(512), 0, stream, z, z_stride, bias, cap, row_start, row_slot, state, slot_stride,
               m_off, (float4*)gates, H, max_slots);
  else
    fmx_launch(mlstm_gates_kernel<128>, dim3(H, R), dim3(128), 0, stream, z, z_stride, bias, cap, row_start, row_slot, state, slot_stride,
               m_off, (float4*)gates, H, max_slots);
  FMX_LAUNCH_CHECK();
  return 0;
}

// lanes (8, 16, 32): lanes that share a column, cpt (1, 2, 4): columns that they hold; 0: the choice is made here.
FMX_EXPORT int fmx_mlstm_scan(const void* proj, long long stride, const float* gates, const int* row_start, const int* row_slot,
                              float* state, long long slot_stride, float* out, float* nq, int R, int H, int D, int Dv, int max_slots,
                              int dtype, int lanes, int cpt, cudaStream_t stream) {
  if (R == 0) return 0;
  if (R < 0 || H <= 0 || D <= 0 || Dv <= 0 || D > 512 || stride < 2LL * H * D + (long long)H * Dv)
    return fmx_fail("fmx_mlstm_scan: bad sizes R=%d H=%d D=%d Dv=%d", R, H, D, Dv);
  if (H > 65535 || R > 65535) return fmx_fail("fmx_mlstm_scan: batch too large");
  if (dtype != FMX_F32 && dtype != FMX_BF16) return fmx_fail("fmx_mlstm_scan: unknown dtype %d", dtype);
  const long long heads = (long long)R * H;
  if (lanes == 0) lanes = D <= 32 ? 8 : D <= 128 ? 16 : 32;
  if (lanes == 8 && D > 64) lanes = 16;
  if (lanes == 16 && D > 128) lanes = 32;
  if (lanes == 32 && D <= 128) lanes = 16;
  if (lanes != 8 && lanes != 16 && lanes != 32) return fmx_fail("fmx_mlstm_scan: 8, 16 or 32 lanes per column, not %d", lanes);
  const int most = D > 256 ? 1 : lanes == 8 ? 2 : 4;           // four tokens' sums of a lane's columns fit its lanes
  if (cpt == 0) {                                              // as many columns per group of lanes as leave every multiprocessor a block
    cpt = most;
    while (cpt > 1 && heads * ((Dv + 128 / lanes * cpt) / (128 / lanes * cpt)) < fmx_num_sms() * 3 / 4) cpt /= 2;
  }
  if (cpt != 1 && cpt != 2 && cpt != 4) return fmx_fail("fmx_mlstm_scan: 1, 2 or 4 columns per group of lanes, not %d", cpt);
  if (cpt > most) cpt = most;
  const int vec_in = D % 4 == 0 && Dv % 4 == 0 && stride % 4 == 0 && ((uintptr_t)proj & (dtype == FMX_F32 ? 15 : 7)) == 0;
#define FMX_MS_T(T, RPL, L, CPT, TB)                                                                                   \
  do {                                                                                                                 \
    constexpr int cols = 128 / (L) * (CPT);                                                                            \
    constexpr size_t smem = (size_t)2 * (TB) * (2 * (RPL) * (L) + cols + 4) * sizeof(float);                           \
    if (smem > 48 * 1024)                                                                                              \
      cudaFuncSetAttribute(mlstm_scan_kernel<T, RPL, L, CPT, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    fmx_launch(mlstm_scan_kernel<T, RPL, L, CPT, TB>, dim3((Dv + cols) / cols, H, R), dim3(128), smem, stream, (const T*)proj, stride, \
               (const float4*)gates, row_start, row_slot, state, slot_stride, out, nq, H, D, Dv, max_slots, vec_in);   \
  } while (0)
#define FMX_MS(RPL, L, CPT, TB)                                                                                        \
  do {                                                                                                                 \
    if (dtype == FMX_F32) FMX_MS_T(float, RPL, L, CPT, TB);                                                            \
    else FMX_MS_T(bf16, RPL, L, CPT, TB);                                                                              \
  } while (0)
#define FMX_MS_C(RPL, L, TB)                                                                                           \
  do {                                                                                                                 \
    if (cpt == 1) FMX_MS(RPL, L, 1, TB);                                                                               \
    else if (cpt == 2) FMX_MS(RPL, L, 2, TB);                                                                          \
    else FMX_MS(RPL, L, 4, TB);                                                                                        \
  } while (0)
  if (lanes == 8) {
    if (D <= 32) { if (cpt == 1) FMX_MS(4, 8, 1, 16); else FMX_MS(4, 8, 2, 16); }
    else { if (cpt == 1) FMX_MS(8, 8, 1, 16); else FMX_MS(8, 8, 2, 16); }
  } else if (lanes == 16) {
    if (D <= 64) FMX_MS_C(4, 16, 16);
    else FMX_MS_C(8, 16, 16);
  } else if (D <= 256) FMX_MS_C(8, 32, 16);
  else FMX_MS(16, 32, 1, 8);
#undef FMX_MS_C
#undef FMX_MS
#undef FMX_MS_T
  FMX_LAUNCH_CHECK();
  return 0;
}

// The same as fmx_mlstm_scan for bfloat16 projections, in runs of 64 tokens as matrix products: D of 32, 64, 96 or 128, Dv a multiple of
// 8, rows of 16 bytes.  columns (16, 32; 0: the choice is made here): columns of S per block (16 with D of 64 or 128).
FMX_EXPORT int fmx_mlstm_chunks(const void* proj, long long stride, const float* gates, const int* row_start, const int* row_slot,
                                float* state, long long slot_stride, float* out, float* nq, int R, int H, int D, int Dv, int max_slots,
                                int columns, cudaStream_t stream) {
  if (R == 0) return 0;
  if (R < 0 || H <= 0 || (D != 32 && D != 64 && D != 96 && D != 128) || Dv <= 0 || Dv % 8 || stride % 8 || slot_stride % 2 ||
      stride < 2LL * H * D + (long long)H * Dv || ((uintptr_t)proj & 15) || ((uintptr_t)state & 7) || ((uintptr_t)out & 7) || ((uintptr_t)gates & 15))
    return fmx_fail("fmx_mlstm_chunks: bad sizes R=%d H=%d D=%d Dv=%d stride=%lld", R, H, D, Dv, stride);
  if (H > 65535 || R > 65535) return fmx_fail("fmx_mlstm_chunks: batch too large");
  if (columns == 0) columns = (D == 64 || D == 128) && (long long)R * H * ((Dv + 31) / 32) < fmx_num_sms() * 3 / 4 ? 16 : 32;
  if (columns != 32 && !(columns == 16 && (D == 64 || D == 128))) return fmx_fail("fmx_mlstm_chunks: %d columns per block with D=%d", columns, D);
  cudaError_t err = cudaSuccess;
#define FMX_MC(KD, VB)                                                                                                 \
  do {                                                                                                                 \
    using Z = ChunkSize<KD, VB>;                                                                                       \
    static const cudaError_t set = cudaFuncSetAttribute(mlstm_chunk_kernel<KD, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Z::SMEM); \
    err = set;                                                                                                         \
    if (err == cudaSuccess)                                                                                            \
      fmx_launch(mlstm_chunk_kernel<KD, VB>, dim3((Dv + VB - 1) / VB, H, R), dim3(128), Z::SMEM, stream, (const bf16*)proj, stride, \
                 (const float4*)gates, row_start, row_slot, state, slot_stride, out, nq, H, Dv, max_slots);            \
  } while (0)
  if (D == 32) FMX_MC(2, 32);
  else if (D == 64) { if (columns == 16) FMX_MC(4, 16); else FMX_MC(4, 32); }
  else if (D == 96) FMX_MC(6, 32);
  else { if (columns == 16) FMX_MC(8, 16); else FMX_MC(8, 32); }
#undef FMX_MC
  if (err != cudaSuccess) return fmx_fail("fmx_mlstm_chunks: shared memory refused: %s", cudaGetErrorString(err));
  FMX_LAUNCH_CHECK();
  return 0;
}

// proj [T, stride] of p_dtype (q | k | v | output gate), out rows of out_stride elements of o_dtype.
FMX_EXPORT int fmx_mlstm_step(const void* proj, long long stride, int p_dtype, const float* z, long long z_stride, const float* bias,
                              float cap, const int* row_start, const int* row_slot, float* state, long long slot_stride,
                              long long m_off, const float* w, float eps, void* out, long long out_stride, int o_dtype, int R, int H,
                              int D, int Dv, int max_slots, cudaStream_t stream) {
  if (R == 0) return 0;
  if (R < 0 || R > 65535 || H <= 0 || D <= 0 || Dv <= 0 || D > 512 || Dv > 8192 || stride < 2LL * H * D + 2LL * H * Dv ||
      z_stride < 2LL * H || out_stride < (long long)H * Dv || !(cap > 0.f))
    return fmx_fail("fmx_mlstm_step: bad sizes R=%d H=%d D=%d Dv=%d", R, H, D, Dv);
  const int vec_in = D % 4 == 0 && stride % 4 == 0 && ((uintptr_t)proj & (p_dtype == FMX_F32 ? 15 : 7)) == 0;
  const size_t smem = (size_t)(Dv + 1) * sizeof(float);
#define FMX_MST(TP, TO, LN, NI)                                                                                        \
  fmx_launch(mlstm_step_kernel<TP, TO, LN, NI>, dim3(H, R), dim3(STEP_THREADS), smem, stream, (const TP*)proj, stride, z, z_stride, bias, cap, \
             row_start, row_slot, state, slot_stride, m_off, w, eps, (TO*)out, out_stride, H, D, Dv, max_slots, vec_in)
#define FMX_MST_D(TP, TO)                                                                                              \
  do {                                                                                                                 \
    if (D <= 32) FMX_MST(TP, TO, 8, 1);                                                                                \
    else if (D <= 64) FMX_MST(TP, TO, 16, 1);                                                                          \
    else if (D <= 128) FMX_MST(TP, TO, 32, 1);                                                                         \
    else if (D <= 256) FMX_MST(TP, TO, 32, 2);                                                                         \
    else FMX_MST(TP, TO, 32, 4);                                                                                       \
  } while (0)
  if (p_dtype == FMX_F32 && o_dtype == FMX_F32) FMX_MST_D(float, float);
  else if (p_dtype == FMX_F32 && o_dtype == FMX_BF16) FMX_MST_D(float, bf16);
  else if (p_dtype == FMX_BF16 && o_dtype == FMX_BF16) FMX_MST_D(bf16, bf16);
  else return fmx_fail("fmx_mlstm_step: unknown dtypes %d, %d", p_dtype, o_dtype);
#undef FMX_MST_D
#undef FMX_MST
  FMX_LAUNCH_CHECK();
  return 0;
}
