// The delta rule with one decay a key channel: a linear recurrence over a matrix state per head,
//     S <- g S (row c of S times g[c]);  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// (S: dim x vdim, float32), with q and k unit vectors per head (q also times dim^(-1/2)), beta in (0, 1)
// and g = exp(-exp(A) softplus(pre + dt_bias)) in (0, 1) per head and key channel; all of it 32-bit.  In
// front of it q, k and v pass a short causal convolution over time, channel by channel, and silu.
//
// Per request the state slot holds, in float32: the heads' matrices TRANSPOSED and padded,
// [heads, vdim, dim_padded] (a thread owns consecutive rows of a column), and behind them the convolution's
// last taps - 1 inputs, [taps - 1, channels], oldest first.  A request's rows of a step are consecutive
// (q_start[r] .. q_start[r + 1]).
//
// A portion is worked through in runs of four tokens, counted from the portion's start.  With P_t the product
// of the run's decays up to and with token t (per channel) and S0 the matrix before the run, the rule unrolls,
// column by column, to
//     w_t = beta_t (v_t - S0^T (P_t k_t))
//     u_t = w_t - sum_{s<t} beta_t A[t][s] u_s,        A[t][s] = sum_c k_t[c] k_s[c] g_{s+1}[c] .. g_t[c]
//     o_t = S0^T (P_t q_t) + sum_{s<=t} B[t][s] u_s,   B[t][s] = sum_c q_t[c] k_s[c] g_{s+1}[c] .. g_t[c]
//     S4  = P_3 S0 + sum_s (g_{s+1} .. g_3 k_s) u_s^T
// Only products of decays occur, never quotients, so nothing can overflow.  The triangular solve is the same
// for all columns: u = M w with M the inverse of the unit triangle (I + beta A), and o = S0^T (P q) + (B M) w.
//
//   cdr_prepare   a block a (run, head): convolution, silu, unit vectors, decays; the run's 13 vectors (P_t k_t,
//                 P_t q_t, P_3, the four decayed keys), the 8 x 4 coefficients, beta and v as one record
//   cdr_scan      the recurrence over the runs.  A warp owns four columns, P lanes a column, a thread DPL
//                 rows of P / 8 columns: the run's 8 sums of its columns are exactly P numbers a thread, and
//                 one butterfly over the P lanes leaves lane p with number p.  Records are staged through shared memory by
//                 cp.async, a few runs ahead
//   cdr_step      a step of single tokens in one kernel: a block a (row, head) with convolution, the decay's and
//                 the gate's second low-rank products, unit vectors, the token's recurrence, output norm and gate
//   take_columns  a column range of a float32 product in the compute type (the low-rank products' operand)
#include "common.cuh"

#define CDR_RUN 4
#define CDR_WARPS 4
#define CDR_COLS (CDR_WARPS * 4)         // columns of a scan block
#define CDR_STAGES 4
#define CDR_MAX_TAPS 16
#define CDR_MAX_DIM 512
#define CDR_COEFF 40                     // 8 x 4 coefficients, 4 beta, 4 unused

__device__ __forceinline__ float cdr_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float cdr_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// two 32-bit lanes in one 64-bit register
typedef unsigned long long cdr2;
__device__ __forceinline__ cdr2 cdr_pack(float a, float b) {
  cdr2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void cdr_unpack(cdr2 v, float& a, float& b) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
}
__device__ __forceinline__ cdr2 cdr_fma2(cdr2 a, cdr2 b, cdr2 c) {
  cdr2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ cdr2 cdr_mul2(cdr2 a, cdr2 b) {
  cdr2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// The runs of the requests lie one behind the other: request r's first run, by a scan over the requests' lengths.
__device__ __forceinline__ int cdr_runs_of(const int* q_start, int r) { return (q_start[r + 1] - q_start[r] + CDR_RUN - 1) / CDR_RUN; }

// The runs before request r (called by whole warps).
__device__ __forceinline__ int cdr_first_run(const int* q_start, int r, int lane) {
  int sum = 0;
  for (int i = lane; i < r; i += 32) sum += cdr_runs_of(q_start, i);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  return sum;
}

// The request that run c belongs to and the run's place in it; r = -1 behind the last run (called by whole warps).
__device__ __forceinline__ void cdr_find_run(const int* q_start, int n_requests, int c, int lane, int& r, int& place) {
  int before = 0;
  r = -1;
  place = 0;
  for (int r0 = 0; r0 < n_requests; r0 += 32) {
    const int n = r0 + lane < n_requests ? cdr_runs_of(q_start, r0 + lane) : 0;
    int upto = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int other = __shfl_up_sync(0xffffffffu, upto, o);
      if (lane >= o) upto += other;
    }
    const unsigned beyond = __ballot_sync(0xffffffffu, before + upto > c);
    if (beyond) {
      const int at = __ffs(beyond) - 1;
      r = r0 + at;
      place = c - before - __shfl_sync(0xffffffffu, upto - n, at);
      return;
    }
    before += __shfl_sync(0xffffffffu, upto, 31);
  }
}

// ---- the run's record ---------------------------------------------------------------------------------
// proj: the stacked input product [T, ld] in float32; columns qkv_at .. + channels are q (groups * dim), k (groups * dim),
// v (heads * vdim), b_at .. + heads the projection behind beta.  pre: [T, pre_ld], columns 0 .. heads * dim
// the decay's pre-activations.
__global__ void __launch_bounds__(128)
cdr_prepare_kernel(const float* __restrict__ proj, int ld, int qkv_at, int b_at, const float* __restrict__ pre,
                   int pre_ld, int groups, int heads, int dim, int vdim, int taps, const float* __restrict__ conv_w,
                   const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                   const float* __restrict__ state, long long state_stride, int conv_off,
                   const int* __restrict__ q_start, int n_requests, const int* __restrict__ state_slot, float q_scale,
                   int dim_p, int vdim_p, float* __restrict__ records) {
  extern __shared__ float cdr_s[];          // q, k, g: [4][dim_p] each
  __shared__ float dots[2 * CDR_RUN * CDR_RUN], beta_s[CDR_RUN];
  const int c = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int r, place;
  cdr_find_run(q_start, n_requests, c, lane, r, place);
  pdl_wait();
  pdl_launch();
  if (r < 0) return;
  const int at0 = place * CDR_RUN;                     // the run's first token's place in its portion
  const int t0 = q_start[r] + at0;
  const int n_here = min(CDR_RUN, q_start[r + 1] - t0);
  const int g = h / (heads / groups);
  const int channels = 2 * groups * dim + heads * vdim;
  const float* kept = state + (size_t)state_slot[r] * state_stride + conv_off;
  float* q_s = cdr_s;
  float* k_s = q_s + CDR_RUN * dim_p;
  float* g_s = k_s + CDR_RUN * dim_p;
  float* rec = records + ((size_t)c * heads + h) * (13 * dim_p + CDR_COEFF + CDR_RUN * vdim_p);
  float* v_out = rec + 13 * dim_p + CDR_COEFF;

  for (int i = threadIdx.x; i < 2 * dim_p + vdim_p; i += blockDim.x) {
    const int which = i < dim_p ? 0 : i < 2 * dim_p ? 1 : 2;
    const int l = i - which * dim_p;
    float* dst = which == 0 ? q_s + l : which == 1 ? k_s + l : v_out + l;
    const int step = which == 2 ? vdim_p : dim_p;
    if (l >= (which == 2 ? vdim : dim)) {
#pragma unroll
      for (int t = 0; t < CDR_RUN; ++t) dst[t * step] = 0.f;
      continue;
    }
    const int ch = which == 0 ? g * dim + l : which == 1 ? (groups + g) * dim + l : 2 * groups * dim + h * vdim + l;
    const float* in = proj + qkv_at + ch;
    const float* w = conv_w + (size_t)ch * taps;
    // an input `back` places before the portion's start is the kept one that many from the end
    auto input = [&](int place_in) {
      return place_in >= 0 ? in[(size_t)(q_start[r] + place_in) * ld] : kept[(size_t)(taps - 1 + place_in) * channels + ch];
    };
    float acc[CDR_RUN] = {0.f, 0.f, 0.f, 0.f};
    if (taps == 4) {
      float x[CDR_RUN + 3], tap[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) tap[j] = w[j];
#pragma unroll
      for (int j = 0; j < CDR_RUN + 3; ++j) x[j] = j - 3 < n_here ? input(at0 + j - 3) : 0.f;
#pragma unroll
      for (int t = 0; t < CDR_RUN; ++t) {
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[t] = fmaf(tap[j], x[t + j], acc[t]);
      }
    } else {
      for (int t = 0; t < n_here; ++t)
        for (int j = 0; j < taps; ++j) acc[t] = fmaf(w[j], input(at0 + t - (taps - 1 - j)), acc[t]);
    }
#pragma unroll
    for (int t = 0; t < CDR_RUN; ++t) dst[t * step] = t < n_here ? acc[t] * cdr_sigmoid(acc[t]) : 0.f;
  }
  const float a = expf(a_log[h]);
  for (int i = threadIdx.x; i < CDR_RUN * dim_p; i += blockDim.x) {
    const int t = i / dim_p, l = i - t * dim_p;
    float decay = 1.f;
    if (t < n_here && l < dim)
      decay = expf(-a * cdr_softplus(pre[(size_t)(t0 + t) * pre_ld + h * dim + l] + dt_bias[h * dim + l]));
    g_s[i] = decay;
  }
  if (threadIdx.x < CDR_RUN)
    beta_s[threadIdx.x] = threadIdx.x < n_here ? cdr_sigmoid(proj[(size_t)(t0 + threadIdx.x) * ld + b_at + h]) : 0.f;
  __syncthreads();
  {                                          // warp t: token t's unit vectors
    float* qt = q_s + warp * dim_p;
    float* kt = k_s + warp * dim_p;
    float qq = 0.f, kk = 0.f;
    for (int l = lane; l < dim; l += 32) {
      qq = fmaf(qt[l], qt[l], qq);
      kk = fmaf(kt[l], kt[l], kk);
    }
    const float q_unit = 1.0f / sqrtf(warp_sum(qq) + 1e-6f) * q_scale, k_unit = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
    for (int l = lane; l < dim; l += 32) {
      qt[l] *= q_unit;
      kt[l] *= k_unit;
    }
  }
  __syncthreads();
  {                                          // warp t: A[t][s], s < t, and B[t][s], s <= t
    const int t = warp;
    float da[CDR_RUN] = {0.f, 0.f, 0.f, 0.f}, db[CDR_RUN] = {0.f, 0.f, 0.f, 0.f};
    for (int l = lane; l < dim; l += 32) {
      const float kt = k_s[t * dim_p + l], qt = q_s[t * dim_p + l];
      float between = 1.f;                   // g_{s+1} .. g_t
#pragma unroll
      for (int s = CDR_RUN - 1; s >= 0; --s) {
        if (s > t) continue;
        const float ks = k_s[s * dim_p + l] * between;
        db[s] = fmaf(qt, ks, db[s]);
        if (s < t) da[s] = fmaf(kt, ks, da[s]);
        between *= g_s[s * dim_p + l];
      }
    }
#pragma unroll
    for (int s = 0; s < CDR_RUN; ++s) {
      da[s] = warp_sum(da[s]);
      db[s] = warp_sum(db[s]);
      if (lane == 0) {
        dots[t * CDR_RUN + s] = da[s];
        dots[CDR_RUN * CDR_RUN + t * CDR_RUN + s] = db[s];
      }
    }
  }
  // the 13 vectors
  for (int l = threadIdx.x; l < dim_p; l += blockDim.x) {
    float k[CDR_RUN], q[CDR_RUN], d[CDR_RUN];
#pragma unroll
    for (int t = 0; t < CDR_RUN; ++t) {
      k[t] = k_s[t * dim_p + l];
      q[t] = q_s[t * dim_p + l];
      d[t] = g_s[t * dim_p + l];
    }
    float upto = 1.f;
#pragma unroll
    for (int t = 0; t < CDR_RUN; ++t) {
      upto *= d[t];
      rec[t * dim_p + l] = upto * k[t];
      rec[(CDR_RUN + t) * dim_p + l] = upto * q[t];
    }
    rec[8 * dim_p + l] = upto;
    float behind = 1.f;
#pragma unroll
    for (int t = CDR_RUN - 1; t >= 0; --t) {
      rec[(9 + t) * dim_p + l] = behind * k[t];
      behind *= d[t];
    }
  }
  __syncthreads();
  // row i of M (the inverse of the unit triangle I + beta A) and of B M: thread i, column j of M by substitution
  if (threadIdx.x < 8) {
    float m[CDR_RUN][CDR_RUN];
#pragma unroll
    for (int s = 0; s < CDR_RUN; ++s) {
#pragma unroll
      for (int t = 0; t < CDR_RUN; ++t) {
        float v = t == s ? 1.f : 0.f;
        if (t > s) {
          float sum = 0.f;
#pragma unroll
          for (int i = 0; i < CDR_RUN; ++i)
            if (i >= s && i < t) sum = fmaf(dots[t * CDR_RUN + i], m[i][s], sum);
          v = -beta_s[t] * sum;
        }
        m[t][s] = v;
      }
    }
    const int row = threadIdx.x & 3;
    float* coeff = rec + 13 * dim_p;
#pragma unroll
    for (int s = 0; s < CDR_RUN; ++s) {
      float v = 0.f;
#pragma unroll
      for (int t = 0; t < CDR_RUN; ++t) {
        if (threadIdx.x < 4) {
          if (t == row) v = m[t][s];
        } else if (t <= row) {
          v = fmaf(dots[CDR_RUN * CDR_RUN + row * CDR_RUN + t], m[t][s], v);
        }
      }
      coeff[threadIdx.x * CDR_RUN + s] = v;
    }
    coeff[32 + threadIdx.x] = threadIdx.x < CDR_RUN ? beta_s[threadIdx.x] : 0.f;
  }
}

// ---- the recurrence ------------------------------------------------------------------------------------
__device__ __forceinline__ void cdr_copy16(float* dst, const float* src) {
  const unsigned to = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to), "l"(src) : "memory");
}

template <int P, int DPL>
__global__ void __launch_bounds__(CDR_WARPS * 32)
cdr_scan_kernel(const float* __restrict__ records, int heads, int vdim, int vdim_p, float* __restrict__ state,
                long long state_stride, const int* __restrict__ q_start, const int* __restrict__ state_slot,
                float* __restrict__ o_out) {
  constexpr int dim_p = P * DPL, CPT = P / 8, PAIRS = DPL / 2;
  constexpr int kShared = 13 * dim_p + CDR_COEFF, kStage = kShared + CDR_RUN * CDR_COLS;
  extern __shared__ __align__(16) float cdr_stage[];
  const int r = blockIdx.z, h = blockIdx.y, block_col = blockIdx.x * CDR_COLS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane % P, group = lane / P;
  const int first = q_start[r], n = q_start[r + 1] - first;
  const int run0 = cdr_first_run(q_start, r, lane);
  const int my_col = warp * 4 + group * CPT;           // the thread's first column inside the block
  const bool any = n > 0;
  // the matrices were last written by an earlier step: asked for before the wait on the predecessor
  cdr2 S[CPT][PAIRS];
  float* mine[CPT];
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    const int col = block_col + my_col + j;
    const bool live = any && col < vdim;
    mine[j] = state + (size_t)(any ? state_slot[r] : 0) * state_stride + ((size_t)h * vdim + (live ? col : 0)) * dim_p + part * DPL;
#pragma unroll
    for (int e = 0; e < PAIRS; e += 2) {
      const ulonglong2 v = live ? *reinterpret_cast<const ulonglong2*>(mine[j] + 2 * e) : make_ulonglong2(0ull, 0ull);
      S[j][e] = v.x;
      S[j][e + 1] = v.y;
    }
  }
  pdl_wait();
  pdl_launch();
  if (!any) return;
  const int n_runs = (n + CDR_RUN - 1) / CDR_RUN;
  const size_t record = (size_t)kShared + CDR_RUN * vdim_p;
  const float* base = records + ((size_t)run0 * heads + h) * record;
  auto fetch = [&](int c) {
    if (c < n_runs) {
      const float* src = base + (size_t)c * heads * record;
      float* dst = cdr_stage + (c % CDR_STAGES) * kStage;
      for (int i = threadIdx.x; i < kShared / 4; i += CDR_WARPS * 32) cdr_copy16(dst + i * 4, src + i * 4);
      if (threadIdx.x < CDR_RUN * CDR_COLS / 4) {
        const int t = threadIdx.x / (CDR_COLS / 4), piece = (threadIdx.x % (CDR_COLS / 4)) * 4;
        if (block_col + piece < vdim_p)
          cdr_copy16(dst + kShared + t * CDR_COLS + piece, src + kShared + t * vdim_p + block_col + piece);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int c = 0; c < CDR_STAGES - 1; ++c) fetch(c);
  const int row = part & 7, tok = part & 3, out_col = block_col + my_col + (part >> 3);
  const bool reads_out = row >= 4;                     // this lane ends up with an output (else with a u)
  float* o_mine = o_out + (size_t)(first + tok) * heads * vdim + (size_t)h * vdim + out_col;
  const bool writes = reads_out && out_col < vdim;
  for (int c = 0; c < n_runs; ++c) {
    asm volatile("cp.async.wait_group %0;" ::"n"(CDR_STAGES - 2) : "memory");
    __syncthreads();                                   // run c has landed for all; run c - 1 is no longer read
    fetch(c + CDR_STAGES - 1);
    const float* stage = cdr_stage + (c % CDR_STAGES) * kStage;
    const float* vectors = stage + part * DPL;
    float sum[P];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      cdr2 x[PAIRS];
#pragma unroll
      for (int e = 0; e < PAIRS; e += 2) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(vectors + i * dim_p + 2 * e);
        x[e] = v.x;
        x[e + 1] = v.y;
      }
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        cdr2 acc = cdr_mul2(S[j][0], x[0]);
#pragma unroll
        for (int e = 1; e < PAIRS; ++e) acc = cdr_fma2(S[j][e], x[e], acc);
        float lo, hi;
        cdr_unpack(acc, lo, hi);
        sum[j * 8 + i] = lo + hi;
      }
    }
    // lane p of a column group's P lanes ends with the whole sum number p
#pragma unroll
    for (int o = P / 2; o > 0; o >>= 1) {
      const bool upper = part & o;
#pragma unroll
      for (int i = 0; i < o; ++i) {
        const float got = __shfl_xor_sync(0xffffffffu, upper ? sum[i] : sum[i + o], o);
        sum[i] = (upper ? sum[i + o] : sum[i]) + got;
      }
    }
    const float4 m = *reinterpret_cast<const float4*>(stage + 13 * dim_p + row * 4);
    const float v = stage[kShared + tok * CDR_COLS + my_col + (part >> 3)];
    const float w = stage[13 * dim_p + 32 + tok] * (v - sum[0]);
    const float w0 = __shfl_sync(0xffffffffu, w, 0, 8), w1 = __shfl_sync(0xffffffffu, w, 1, 8);
    const float w2 = __shfl_sync(0xffffffffu, w, 2, 8), w3 = __shfl_sync(0xffffffffu, w, 3, 8);
    float val = reads_out ? sum[0] : 0.f;
    val = fmaf(m.x, w0, val);
    val = fmaf(m.y, w1, val);
    val = fmaf(m.z, w2, val);
    val = fmaf(m.w, w3, val);
    if (writes && c * CDR_RUN + tok < n) o_mine[(size_t)c * CDR_RUN * heads * vdim] = val;
    cdr2 u[CPT][CDR_RUN];
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
#pragma unroll
      for (int t = 0; t < CDR_RUN; ++t) {
        const float x = __shfl_sync(0xffffffffu, val, j * 8 + t, P);
        u[j][t] = cdr_pack(x, x);
      }
    }
#pragma unroll
    for (int i = 8; i < 13; ++i) {                     // the run's decay, then the four decayed keys
#pragma unroll
      for (int e = 0; e < PAIRS; e += 2) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(vectors + i * dim_p + 2 * e);
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          S[j][e] = i == 8 ? cdr_mul2(x.x, S[j][e]) : cdr_fma2(x.x, u[j][i < 9 ? 0 : i - 9], S[j][e]);
          S[j][e + 1] = i == 8 ? cdr_mul2(x.y, S[j][e + 1]) : cdr_fma2(x.y, u[j][i < 9 ? 0 : i - 9], S[j][e + 1]);
        }
      }
    }
  }
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    if (block_col + my_col + j < vdim) {
#pragma unroll
      for (int e = 0; e < PAIRS; e += 2)
        *reinterpret_cast<ulonglong2*>(mine[j] + 2 * e) = make_ulonglong2(S[j][e], S[j][e + 1]);
    }
  }
}

// ---- a step of single tokens ---------------------------------------------------------------------------
// `low_at` .. + ra + rg: columns of proj with the low-rank activations of the decay (ra) and of the gate (rg);
// w2: [heads * dim + heads * vdim, ra + rg], the second products' rows (the decay's read the first ra columns, the
// gate's the last rg).  With `pre` given ([T, heads * (dim + vdim)]) those products are done already.  `shift`:
// every head has q and k channels of its own, so the block moves its channels' kept inputs on itself.
template <typename TW> struct CdrPiece;               // a lane's piece of a weight row: four elements
template <> struct CdrPiece<float> {
  typedef float4 Raw;
  static __device__ __forceinline__ Raw raw(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ float4 wide(Raw v) { return v; }
};
template <> struct CdrPiece<__nv_bfloat16> {
  typedef uint2 Raw;
  static __device__ __forceinline__ Raw raw(const __nv_bfloat16* p) { return *reinterpret_cast<const uint2*>(p); }
  static __device__ __forceinline__ float4 wide(Raw v) {
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
  }
};

// threads of a block: fewer where a thread keeps more of the matrix
constexpr int cdr_step_warps(int dpl) { return dpl <= 4 ? 32 : dpl <= 8 ? 16 : 8; }

template <int P, int DPL, typename TW, typename TO>
__global__ void __launch_bounds__(cdr_step_warps(DPL) * 32)
cdr_step_kernel(const float* __restrict__ proj, int ld, int qkv_at, int b_at, int low_at, int ra, int rg,
                const TW* __restrict__ w2, const float* __restrict__ pre, int groups, int heads, int dim, int vdim,
                int taps, const float* __restrict__ conv_w, const float* __restrict__ a_log,
                const float* __restrict__ dt_bias, const float* __restrict__ gain, float eps, float q_scale,
                float* __restrict__ state, long long state_stride, int conv_off, const int* __restrict__ row_req,
                const int* __restrict__ state_slot, int shift, TO* __restrict__ out) {
  constexpr int dim_p = P * DPL, CPT = P / 8;
  // q, k [dim_p] each, v [vdim], decays [dim_p], o, gate [vdim] each; low-rank activations [ra + rg]
  extern __shared__ __align__(16) float cdr_one[];
  __shared__ float scratch[33], misc[4];
  const int t = blockIdx.x, h = blockIdx.y;
  const int r = row_req[t];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int part = lane % P, group = lane / P;
  float* q_s = cdr_one;
  float* k_s = q_s + dim_p;
  float* v_s = k_s + dim_p;
  float* g_s = v_s + vdim;
  float* o_s = g_s + dim_p;
  float* gate_s = o_s + vdim;
  float* low_s = gate_s + (vdim + (-(3 * vdim) & 3));         // on 16 bytes
  float* slot = state + (size_t)(r < 0 ? 0 : state_slot[r]) * state_stride;
  // the first columns' matrix rows, last written by an earlier step: asked for before the wait
  float S[CPT][DPL];
  auto load_columns = [&](int col0) {
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      const int col = col0 + j;
      const float* mine = slot + ((size_t)h * vdim + (col < vdim ? col : 0)) * dim_p + part * DPL;
#pragma unroll
      for (int e = 0; e < DPL; e += 4) {
        const float4 m = *reinterpret_cast<const float4*>(mine + e);
        S[j][e] = m.x; S[j][e + 1] = m.y; S[j][e + 2] = m.z; S[j][e + 3] = m.w;
      }
    }
  };
  const int my_col = warp * 4 + group * CPT;
  const int g = h / (heads / groups);
  const int channels = 2 * groups * dim + heads * vdim;
  float* kept = slot + conv_off;
  // ... and so are the thread's first channel's taps and kept inputs, and the warp's first rows of the second
  // products (a lane's first four elements of each), which nothing of this step writes
  constexpr int kAhead = 8;
  const int outputs = dim_p + vdim;
  auto second_row = [&](int i) {               // the weight row of output i and where its inputs start; null: none
    const bool decay = i < dim_p;
    const int l = decay ? i : i - dim_p;
    return decay && l >= dim ? (const TW*)nullptr
                             : w2 + (size_t)(decay ? h * dim + l : heads * dim + h * vdim + l) * (ra + rg) + (decay ? 0 : ra);
  };
  auto channel_of = [&](int i) {               // the channel of item i of q, k, v; -1: a padded lane
    if (i >= 2 * dim_p) return 2 * groups * dim + h * vdim + i - 2 * dim_p;
    const int l = i < dim_p ? i : i - dim_p;
    return l < dim ? (i < dim_p ? g : groups + g) * dim + l : -1;
  };
  float tap[4], old[3];
  typename CdrPiece<TW>::Raw ahead[kAhead];
  const int first_channel = (int)threadIdx.x < 2 * dim_p + vdim ? channel_of(threadIdx.x) : -1;
  const bool quick = taps == 4 && first_channel >= 0;
  if (r >= 0) {
    load_columns(my_col);
    if (quick) {
#pragma unroll
      for (int j = 0; j < 4; ++j) tap[j] = conv_w[(size_t)first_channel * 4 + j];
#pragma unroll
      for (int j = 0; j < 3; ++j) old[j] = kept[(size_t)j * channels + first_channel];
    }
    if (pre == nullptr) {
#pragma unroll
      for (int k = 0; k < kAhead; ++k) {
        const int i = warp + k * warps;
        const TW* w = i < outputs ? second_row(i) : nullptr;
        if (w != nullptr && lane * 4 < (i < dim_p ? ra : rg)) ahead[k] = CdrPiece<TW>::raw(w + lane * 4);
      }
    }
  }
  pdl_wait();
  pdl_launch();
  if (r < 0) return;
  const float* row = proj + (size_t)t * ld;
  for (int i = threadIdx.x; i < 2 * dim_p + vdim; i += blockDim.x) {
    const int c = channel_of(i);
    float value = 0.f;
    if (c >= 0) {
      const float newest = row[qkv_at + c];
      float acc;
      if (quick && i == (int)threadIdx.x) {
        acc = tap[3] * newest;
#pragma unroll
        for (int j = 0; j < 3; ++j) acc = fmaf(tap[j], old[j], acc);
        if (shift) {
          kept[c] = old[1];
          kept[(size_t)channels + c] = old[2];
        }
      } else {
        acc = conv_w[(size_t)c * taps + taps - 1] * newest;
        for (int j = 0; j + 1 < taps; ++j) {                // kept inputs move on one place as they are read
          const float in = kept[(size_t)j * channels + c];
          acc = fmaf(conv_w[(size_t)c * taps + j], in, acc);
          if (shift && j > 0) kept[(size_t)(j - 1) * channels + c] = in;
        }
      }
      if (shift && taps > 1) kept[(size_t)(taps - 2) * channels + c] = newest;
      value = acc * cdr_sigmoid(acc);
    }
    q_s[i] = value;                            // q, k and v lie one behind the other
  }
  if (pre == nullptr)
    for (int i = threadIdx.x; i < ra + rg; i += blockDim.x) low_s[i] = row[low_at + i];
  __syncthreads();
  // the decay's and the gate's second products (a warp an output), and the token's unit vectors
  const float a = expf(a_log[h]);
  if (pre == nullptr) {
    // kAhead outputs a warp at a time, so that their sums cross the lanes side by side; lane k finishes output k
    for (int base = warp; base < outputs; base += kAhead * warps) {
      float acc[kAhead];
#pragma unroll
      for (int k = 0; k < kAhead; ++k) {
        const int i = base + k * warps;
        const TW* w = i < outputs ? second_row(i) : nullptr;
        const int from = i < dim_p ? 0 : ra, n = w == nullptr ? 0 : i < dim_p ? ra : rg;
        acc[k] = 0.f;
        for (int j = lane * 4; j < n; j += 128) {        // ranks and their sum are whole 8s
          const float4 x = CdrPiece<TW>::wide(base == warp && j < 128 ? ahead[k] : CdrPiece<TW>::raw(w + j));
          const float4 y = *reinterpret_cast<const float4*>(low_s + from + j);
          acc[k] = fmaf(x.x, y.x, acc[k]);
          acc[k] = fmaf(x.y, y.y, acc[k]);
          acc[k] = fmaf(x.z, y.z, acc[k]);
          acc[k] = fmaf(x.w, y.w, acc[k]);
        }
      }
      float mine = 0.f;
#pragma unroll
      for (int k = 0; k < kAhead; ++k) {
        acc[k] = warp_sum(acc[k]);
        if (lane == k) mine = acc[k];
      }
      const int i = base + lane * warps;
      if (lane < kAhead && i < outputs) {
        if (i >= dim_p) gate_s[i - dim_p] = cdr_sigmoid(mine);
        else g_s[i] = i < dim ? expf(-a * cdr_softplus(mine + dt_bias[h * dim + i])) : 1.f;
      }
    }
  } else {
    const float* p = pre + (size_t)t * heads * (dim + vdim);
    for (int i = threadIdx.x; i < outputs; i += blockDim.x) {
      if (i < dim_p) g_s[i] = i < dim ? expf(-a * cdr_softplus(p[h * dim + i] + dt_bias[h * dim + i])) : 1.f;
      else gate_s[i - dim_p] = cdr_sigmoid(p[heads * dim + h * vdim + i - dim_p]);
    }
  }
  for (int which = warp; which < 3; which += warps) {
    const float* x = which == 1 ? k_s : q_s;
    const float* y = which == 0 ? q_s : k_s;
    float sum = 0.f;
    for (int l = lane; l < dim; l += 32) sum = fmaf(x[l], y[l], sum);
    sum = warp_sum(sum);
    if (lane == 0) misc[which] = which == 2 ? sum : 1.0f / sqrtf(sum + 1e-6f);     // |q|, |k| inverted, q . k (raw)
  }
  if (threadIdx.x == 0) misc[3] = cdr_sigmoid(row[b_at + h]);
  __syncthreads();
  const float q_unit = misc[0] * q_scale, k_unit = misc[1], kq = misc[2] * q_unit * k_unit, beta = misc[3];
  float squares = 0.f;
  for (int col0 = my_col; col0 - group * CPT < vdim; col0 += warps * 4) {
    if (col0 != my_col) load_columns(col0);
    float kk[DPL], dk[CPT], dq[CPT];
#pragma unroll
    for (int j = 0; j < CPT; ++j) dk[j] = dq[j] = 0.f;
#pragma unroll
    for (int e = 0; e < DPL; ++e) {
      const int c = part * DPL + e;
      const float decay = g_s[c], q = q_s[c] * q_unit;
      kk[e] = k_s[c] * k_unit;
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        S[j][e] *= decay;
        dk[j] = fmaf(S[j][e], kk[e], dk[j]);
        dq[j] = fmaf(S[j][e], q, dq[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
#pragma unroll
      for (int o = P / 2; o > 0; o >>= 1) {
        dk[j] += __shfl_xor_sync(0xffffffffu, dk[j], o);
        dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], o);
      }
      const int col = col0 + j;
      if (col < vdim) {
        const float u = beta * (v_s[col] - dk[j]);
        float* mine = slot + ((size_t)h * vdim + col) * dim_p + part * DPL;
#pragma unroll
        for (int e = 0; e < DPL; e += 4)
          *reinterpret_cast<float4*>(mine + e) =
              make_float4(fmaf(kk[e], u, S[j][e]), fmaf(kk[e + 1], u, S[j][e + 1]),
                          fmaf(kk[e + 2], u, S[j][e + 2]), fmaf(kk[e + 3], u, S[j][e + 3]));
        if (part == 0) {
          const float o = fmaf(kq, u, dq[j]);
          o_s[col] = o;
          squares = fmaf(o, o, squares);
        }
      }
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)vdim + eps);       // publishes o_s too
  for (int l = threadIdx.x; l < vdim; l += blockDim.x)
    out[((size_t)t * heads + h) * vdim + l] = from_float<TO>(o_s[l] * inv * gain[l] * gate_s[l]);
}

template <typename TO>
__global__ void take_columns_kernel(const float* __restrict__ proj, int ld, int at, int n, TO* __restrict__ out,
                                    size_t total) {
  pdl_wait();
  pdl_launch();
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride)
    out[i] = from_float<TO>(proj[(i / n) * ld + at + i % n]);
}

// columns and rows in whole 8s, everything on 16 bytes: eight consecutive columns a thread
__device__ __forceinline__ void take_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void take_store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(h);
}
template <typename TO>
__global__ void take_columns8_kernel(const float* __restrict__ proj, int ld, int at, int n8, TO* __restrict__ out, int n_rows) {
  pdl_wait();
  pdl_launch();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n_rows * n8) return;
  const int t = i / n8, c = (i - t * n8) * 8;
  const float* in = proj + (size_t)t * ld + at + c;
  const float4 a = *reinterpret_cast<const float4*>(in), b = *reinterpret_cast<const float4*>(in + 4);
  TO* o = out + (size_t)t * n8 * 8 + c;
  take_store4(o, a);
  take_store4(o + 4, b);
}

// ---- launchers -----------------------------------------------------------------------------------------
static inline int cdr_parts(int dim) { return dim <= 32 ? 8 : dim <= 64 ? 16 : 32; }
static inline int cdr_rows(int dim) { return dim <= 128 ? 4 : dim <= 256 ? 8 : 16; }

// Rows of a head's padded state column; 0: a size the rule's kernels do not take.
TOKB200_API int tokb200_cdr_padded_dim(int dim) {
  return dim <= 0 || dim > CDR_MAX_DIM ? 0 : cdr_parts(dim) * cdr_rows(dim);
}

// Floats of one run's record of one head.
TOKB200_API int tokb200_cdr_record(int dim, int vdim) {
  return 13 * tokb200_cdr_padded_dim(dim) + CDR_COEFF + CDR_RUN * ((vdim + 3) / 4 * 4);
}

static inline bool cdr_sizes_ok(int groups, int heads, int dim, int vdim, int taps, const float* state,
                                long long state_stride) {
  return groups > 0 && heads > 0 && heads % groups == 0 && heads <= 65535 && dim > 0 && dim <= CDR_MAX_DIM && vdim > 0 &&
         taps >= 1 && taps <= CDR_MAX_TAPS && ((uintptr_t)state & 15) == 0 && state_stride % 4 == 0;
}

// records: n_rows / 4 + n_requests of them, tokb200_cdr_record() floats each and head.
TOKB200_API int tokb200_cdr_prepare(const float* proj, int ld, int qkv_at, int b_at, const float* pre, int pre_ld,
                                    int groups, int heads, int dim, int vdim, int taps, const float* conv_w,
                                    const float* a_log, const float* dt_bias, const float* state,
                                    long long state_stride, int conv_off, const int* q_start, const int* state_slot,
                                    int n_rows, int n_requests, float* records, cudaStream_t stream) {
  if (n_rows <= 0 || n_requests <= 0) return TOKB200_OK;
  if (!cdr_sizes_ok(groups, heads, dim, vdim, taps, state, state_stride)) return TOKB200_BAD_SIZE;
  const int dim_p = tokb200_cdr_padded_dim(dim);
  const size_t smem = (size_t)3 * CDR_RUN * dim_p * sizeof(float);
  return launch_dependent(cdr_prepare_kernel, dim3(n_rows / CDR_RUN + n_requests, heads), dim3(128), smem, stream, proj,
                          ld, qkv_at, b_at, pre, pre_ld, groups, heads, dim, vdim, taps, conv_w, a_log, dt_bias, state,
                          state_stride, conv_off, q_start, n_requests, state_slot, 1.0f / sqrtf((float)dim), dim_p,
                          (vdim + 3) / 4 * 4, records);
}

#define CDR_BY_SIZE(CALL)                     \
  switch (tokb200_cdr_padded_dim(dim)) {      \
    case 32: CALL(8, 4); break;               \
    case 64: CALL(16, 4); break;              \
    case 128: CALL(32, 4); break;             \
    case 256: CALL(32, 8); break;             \
    default: CALL(32, 16); break;             \
  }

template <int P, int DPL>
static int cdr_launch_scan(const float* records, int heads, int vdim, float* state, long long state_stride,
                           const int* q_start, const int* state_slot, int n_requests, float* o_out,
                           cudaStream_t stream) {
  constexpr size_t smem = (size_t)CDR_STAGES * (13 * P * DPL + CDR_COEFF + CDR_RUN * CDR_COLS) * sizeof(float);
  if (smem > 48 * 1024) {
    static bool configured[64] = {};
    int device = 0;
    if (cudaGetDevice(&device) != cudaSuccess || device < 0 || device >= 64) return TOKB200_BAD_SIZE;
    if (!configured[device]) {
      cudaError_t err = cudaFuncSetAttribute(cdr_scan_kernel<P, DPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (err != cudaSuccess) return (int)err;
      configured[device] = true;
    }
  }
  dim3 grid((vdim + CDR_COLS - 1) / CDR_COLS, heads, n_requests);
  return launch_dependent(cdr_scan_kernel<P, DPL>, grid, dim3(CDR_WARPS * 32), smem, stream, records, heads, vdim,
                          (vdim + 3) / 4 * 4, state, state_stride, q_start, state_slot, o_out);
}

TOKB200_API int tokb200_cdr_scan(const float* records, int heads, int dim, int vdim, float* state,
                                 long long state_stride, const int* q_start, const int* state_slot, int n_requests,
                                 float* o_out, cudaStream_t stream) {
  if (n_requests <= 0) return TOKB200_OK;
  if (!cdr_sizes_ok(heads, heads, dim, vdim, 1, state, state_stride) || n_requests > 65535 || ((uintptr_t)records & 15))
    return TOKB200_BAD_SIZE;
  int status = TOKB200_BAD_SIZE;
#define CALL(P, DPL) status = cdr_launch_scan<P, DPL>(records, heads, vdim, state, state_stride, q_start, state_slot, n_requests, o_out, stream)
  CDR_BY_SIZE(CALL)
#undef CALL
  return status;
}

// One token a request (row t belongs to request row_req[t], whose state lies in state_slot[row_req[t]]).
TOKB200_API int tokb200_cdr_step(const float* proj, int ld, int qkv_at, int b_at, int low_at, int ra, int rg,
                                 const void* w2, int w2_dtype, const float* pre, int groups, int heads, int dim, int vdim,
                                 int taps, const float* conv_w, const float* a_log, const float* dt_bias,
                                 const float* gain, float eps, float* state, long long state_stride, int conv_off,
                                 const int* row_req, const int* state_slot, int n_rows, int shift, void* out,
                                 int out_dtype, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (!cdr_sizes_ok(groups, heads, dim, vdim, taps, state, state_stride) || ra < 0 || rg < 0 || ra % 8 || rg % 8 ||
      (shift && heads != groups) || (pre == nullptr && (w2 == nullptr || ((uintptr_t)w2 & 15))))
    return TOKB200_BAD_SIZE;
  const size_t smem = (size_t)(3 * tokb200_cdr_padded_dim(dim) + 3 * vdim + 4 + ra + rg) * sizeof(float);
  if (smem > 48 * 1024) return TOKB200_BAD_SIZE;
  const int most = cdr_step_warps(cdr_rows(dim));
  const int warps = (vdim + 3) / 4 < most ? (vdim + 3) / 4 : most;
  const float q_scale = 1.0f / sqrtf((float)dim);
  dim3 grid(n_rows, heads), block(warps * 32);
  int status = TOKB200_BAD_DTYPE;
#define LAUNCH(P, DPL, TW, TO)                                                                                         \
  status = launch_dependent(cdr_step_kernel<P, DPL, TW, TO>, grid, block, smem, stream, proj, ld, qkv_at, b_at, low_at, \
                            ra, rg, (const TW*)w2, pre, groups, heads, dim, vdim, taps, conv_w, a_log, dt_bias, gain,  \
                            eps, q_scale, state, state_stride, conv_off, row_req, state_slot, shift, (TO*)out)
#define CALL_F32(P, DPL) LAUNCH(P, DPL, float, float)
#define CALL_BF16(P, DPL) LAUNCH(P, DPL, __nv_bfloat16, __nv_bfloat16)
  if (w2_dtype == TOKB200_F32 && out_dtype == TOKB200_F32) { CDR_BY_SIZE(CALL_F32) }
  else if (w2_dtype == TOKB200_BF16 && out_dtype == TOKB200_BF16) { CDR_BY_SIZE(CALL_BF16) }
#undef CALL_F32
#undef CALL_BF16
#undef LAUNCH
  return status;
}

TOKB200_API int tokb200_take_columns(const float* proj, int ld, int at, int n, void* out, int out_dtype, int n_rows,
                                     cudaStream_t stream) {
  if (n_rows <= 0 || n <= 0) return TOKB200_OK;
  if (at < 0 || at + n > ld) return TOKB200_BAD_SIZE;
  const size_t total = (size_t)n_rows * n, blocks = (total + 255) / 256;
  if (n % 8 == 0 && at % 4 == 0 && ld % 4 == 0 && ((((uintptr_t)proj) | ((uintptr_t)out)) & 15) == 0 &&
      total / 8 < (1u << 30)) {
    const dim3 wide((unsigned)((total / 8 + 255) / 256));
    if (out_dtype == TOKB200_F32)
      return launch_dependent(take_columns8_kernel<float>, wide, dim3(256), 0, stream, proj, ld, at, n / 8, (float*)out, n_rows);
    if (out_dtype == TOKB200_BF16)
      return launch_dependent(take_columns8_kernel<__nv_bfloat16>, wide, dim3(256), 0, stream, proj, ld, at, n / 8,
                              (__nv_bfloat16*)out, n_rows);
  }
  const dim3 grid((unsigned)(blocks < 8192 ? blocks : 8192));
  if (out_dtype == TOKB200_F32)
    return launch_dependent(take_columns_kernel<float>, grid, dim3(256), 0, stream, proj, ld, at, n, (float*)out, total);
  if (out_dtype == TOKB200_BF16)
    return launch_dependent(take_columns_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, proj, ld, at, n,
                            (__nv_bfloat16*)out, total);
  return TOKB200_BAD_DTYPE;
}
