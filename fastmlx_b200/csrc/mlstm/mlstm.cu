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
//   mlstm_scan    steps with portions: the recurrence over every row's tokens, from the factors that mlstm_gates left.
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

constexpr int GATE_THREADS = 128;

// z [T, z_stride] 32-bit: input gates (H) | forget gates (H); bias [2 H]; out [T, H]: (kept by, put in by, exp(-m), 0).
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
    *g = make_float4(expf(x.x + m - mn), expf(x.y - mn), expf(-mn), 0.f);
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

// Rows of one token.  grid (H, R), STEP_THREADS threads: LN neighbouring lanes take a row of S^T (or n), each NI pieces of four of its D
// values; U rows per group of lanes are in flight at a time.  proj row: q | k | v | output gate; z: as in mlstm_gates.
constexpr int STEP_THREADS = 256;
template <typename TP, typename TO, int LN, int NI>
__global__ void __launch_bounds__(STEP_THREADS)
mlstm_step_kernel(const TP* proj, long long stride, const float* z, long long z_stride, const float* __restrict__ bias, float cap,
                  const int* row_start, const int* row_slot, float* state, long long slot_stride, long long m_off,
                  const float* __restrict__ w, float eps, TO* out, long long out_stride, int H, int D, int Dv, int max_slots, int vec_in) {
  constexpr int GROUPS = STEP_THREADS / LN, U = NI >= 4 ? 2 : NI == 2 ? 4 : 4;
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
        S[u][i] = j <= Dv ? some4(sp + (long long)j * D + d, D - d, vec) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
  };
  load_rows(grp);
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
  for (int j0 = grp; j0 - grp <= Dv; j0 += U * GROUPS) {       // (the same number of passes for every group of lanes)
    float dot[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int j = j0 + u * GROUPS;
      const float x = put * (j < Dv ? to_f(vrow[j]) : 1.0f);
      dot[u] = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        float4& s = S[u][i];
        s.x = fmaf(k[i].x, x, keep * s.x);
        s.y = fmaf(k[i].y, x, keep * s.y);
        s.z = fmaf(k[i].z, x, keep * s.z);
        s.w = fmaf(k[i].w, x, keep * s.w);
        dot[u] = fmaf(s.x, q[i].x, fmaf(s.y, q[i].y, fmaf(s.z, q[i].z, fmaf(s.w, q[i].w, dot[u]))));
        const int d = 4 * (sub + LN * i);
        if (j <= Dv) {
          float* dst = sp + (long long)j * D + d;
          if (vec) {
            if (d < D) *reinterpret_cast<float4*>(dst) = s;
          } else {
            if (d < D) dst[0] = s.x;
            if (d + 1 < D) dst[1] = s.y;
            if (d + 2 < D) dst[2] = s.z;
            if (d + 3 < D) dst[3] = s.w;
          }
        }
      }
    }
    if (j0 - grp + U * GROUPS <= Dv) load_rows(j0 + U * GROUPS);
    __syncwarp();
#pragma unroll
    for (int u = 0; u < U; ++u) {
#pragma unroll
      for (int e = LN / 2; e >= 1; e >>= 1) dot[u] += __shfl_xor_sync(0xffffffffu, dot[u], e);
      const int j = j0 + u * GROUPS;
      if (sub == 0 && j <= Dv) o_s[j] = dot[u] * q_scale;
    }
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
                               int max_slots, cudaStream_t stream) {
  if (R == 0) return 0;
  if (R < 0 || R > 65535 || H <= 0 || z_stride < 2LL * H || !(cap > 0.f) || ((uintptr_t)gates & 15))
    return fmx_fail("fmx_mlstm_gates: bad arguments R=%d H=%d cap=%g", R, H, (double)cap);
  fmx_launch(mlstm_gates_kernel, dim3(H, R), dim3(GATE_THREADS), 0, stream, z, z_stride, bias, cap, row_start, row_slot, state, slot_stride,
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
