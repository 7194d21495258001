// A matrix memory with exponential gates (the mLSTM form), in 32-bit.
//
// Per head a matrix S (dim x vdim), a vector n (dim) and a number m, all float32 and a request's state, from zero.
// Per token, with i the logarithm of the input gate and f that of the forget gate:
//     m' = max(f + m, i);  keep = exp(f + m - m');  add = exp(i - m')
//     S <- keep S + add k v^T;  n <- keep n + add k;  m <- m'
//     o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
// i = cap tanh(z_i / cap), f = logsigmoid(cap tanh(z_f / cap)), z the gates' pre-activations with their biases.  Every
// head's o is then divided by its root mean square over vdim (eps inside the root), times a gain a lane and the
// sigmoid of one more projection.
//
//   mlstm_gates     m over every request's rows, side by side (max-plus is associative), and from it keep, add and
//                   exp(-m), one of each a token and head; the rest of the recurrence is then linear in (S, n)
//   mlstm_scan      that recurrence on the scan that matrix recurrences share (matrix_scan.cuh): n is the column
//                   of ones, its product with q comes back as one number a token and head
//   mlstm_out_norm  the division, the norm, the gain and the gate: a warp a (token, head), or a few of them
//   mlstm_step      all of it for a step of single tokens, a block a (row, head)
// (In bfloat16 long portions take the scan and the norm in chunks on tensor cores instead: mlstm_chunks.cu.)
//
// A slot: [heads, vdim + 1, dim] (S transposed, n behind the last column), then m [heads].
#include "matrix_scan.cuh"

#define ML_EPS 1e-6f          // added to the normaliser

__device__ __forceinline__ float ml_capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ml_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// What a run of tokens does to m: m -> max(m + a, b).
struct MlStep {
  float a, b;
};
__device__ __forceinline__ MlStep ml_then(MlStep first, MlStep second) {
  return {first.a + second.a, fmaxf(first.b + second.a, second.b)};
}

// proj: [T, ld]; columns i_at .. + heads and f_at .. + heads are the gates' products.  A block a (head, request).  With
// `start` (float32 [requests, heads]) the three numbers a token and head are f, i and m themselves instead, and `start`
// receives the m in front of the step's rows: what the form in chunks works from.
__global__ void mlstm_gates_kernel(const float* __restrict__ proj, int ld, int i_at, int f_at,
                                   const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap,
                                   float* __restrict__ state, long long stride, int m_off, const int* __restrict__ q_start,
                                   const int* __restrict__ state_slot, float* __restrict__ keep,
                                   float* __restrict__ add, float* __restrict__ floor_out, long long gate_ld,
                                   float* __restrict__ start_out) {
  __shared__ float warp_a[32], warp_b[32];
  __shared__ float tops[1024];
  const int head = blockIdx.x, r = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const float ib = i_bias[head], fb = f_bias[head];
  pdl_wait();
  pdl_launch();
  const int first = q_start[r], n = q_start[r + 1] - first;
  if (n <= 0) return;
  float* m_state = state + (size_t)state_slot[r] * stride + m_off + head;
  float carry = *m_state;
  if (start_out && threadIdx.x == 0) start_out[(size_t)r * gridDim.x + head] = carry;
  for (int base = 0; base < n; base += blockDim.x) {
    const int at = base + threadIdx.x;
    const bool live = at < n;
    float li = 0.f, lf = 0.f;
    MlStep mine = {0.f, -INFINITY};                       // leaves m as it is
    if (live) {
      const float* row = proj + (size_t)(first + at) * ld;
      li = ml_capped(row[i_at + head] + ib, cap);
      lf = ml_log_sigmoid(ml_capped(row[f_at + head] + fb, cap));
      mine = {lf, li};
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const MlStep before = {__shfl_up_sync(0xffffffffu, mine.a, o), __shfl_up_sync(0xffffffffu, mine.b, o)};
      if (lane >= o) mine = ml_then(before, mine);
    }
    if (lane == 31) {
      warp_a[warp] = mine.a;
      warp_b[warp] = mine.b;
    }
    __syncthreads();
    float start = carry;                                  // m in front of this warp's first token
    for (int w = 0; w < warp; ++w) start = fmaxf(start + warp_a[w], warp_b[w]);
    const float top = fmaxf(start + mine.a, mine.b);
    tops[threadIdx.x] = top;
    __syncthreads();
    if (live) {
      // the neighbour's own number: what one token's S is divided by is what the next token's keep starts from
      const float before = threadIdx.x == 0 ? carry : tops[threadIdx.x - 1];
      const size_t o = (size_t)head * gate_ld + first + at;
      keep[o] = start_out ? lf : expf(lf + before - top);
      add[o] = start_out ? li : expf(li - top);
      floor_out[o] = start_out ? top : expf(-top);
    }
    carry = tops[warps * 32 - 1];                         // idle threads behind the last token carry its m on
    __syncthreads();                                      // tops and the warps' sums are written again by the next run
  }
  if (threadIdx.x == 0) *m_state = carry;
}

TOKB200_API int tokb200_mlstm_gates(const float* proj, int ld, int i_at, int f_at, const float* i_bias,
                                    const float* f_bias, float cap, int heads, float* state, long long stride, int m_off,
                                    const int* q_start, const int* state_slot, int n_requests, int n_rows, float* keep,
                                    float* add, float* floor_out, long long gate_ld, float* start, cudaStream_t stream) {
  if (n_requests <= 0 || n_rows <= 0) return TOKB200_OK;
  if (heads <= 0 || n_requests > 65535 || cap <= 0.f || i_at + heads > ld || f_at + heads > ld || gate_ld < n_rows ||
      m_off + heads > stride)
    return TOKB200_BAD_SIZE;
  const int threads = n_rows >= 1024 ? 1024 : n_rows >= 256 ? 256 : 64;
  return launch_dependent(mlstm_gates_kernel, dim3(heads, n_requests), dim3(threads), 0, stream, proj, ld, i_at, f_at,
                          i_bias, f_bias, cap, state, stride, m_off, q_start, state_slot, keep, add, floor_out, gate_ld,
                          start);
}

// proj: float32 [T, ld]: q (heads * dim), k (heads * dim) and v (heads * vdim) at their columns.  y [T, heads, vdim]
// receives S^T q * scale, yn [T, heads] n . q * scale.
TOKB200_API int tokb200_mlstm_scan(const float* proj, int ld, int q_at, int k_at, int v_at, int heads, int dim, int vdim,
                                   float scale, const float* keep, const float* add, long long gate_ld, float* state,
                                   long long stride, const int* q_start, const int* state_slot, int n_requests, float* y,
                                   float* yn, float* scratch, int segments, cudaStream_t stream) {
  if (heads <= 0 || dim <= 0 || vdim <= 0 || q_at + heads * dim > ld || k_at + heads * dim > ld || v_at + heads * vdim > ld)
    return TOKB200_BAD_SIZE;
  MatrixScanArgs a = {};
  a.x = proj + v_at; a.x_ld = ld; a.x_head = vdim;
  a.b = proj + k_at; a.b_ld = ld; a.b_group = dim;
  a.c = proj + q_at; a.c_ld = ld; a.c_group = dim;
  a.heads = heads; a.groups = heads; a.P = vdim + 1; a.copied = vdim; a.N = dim; a.scale = scale;
  a.state = state; a.stride = stride; a.q_start = q_start; a.state_slot = state_slot; a.y = y; a.y_ones = yn;
  a.keep = keep; a.add = add; a.gate_ld = gate_ld; a.scratch = scratch; a.segments = segments; a.n_requests = n_requests;
  return launch_matrix_scan<float, MS_GATES_GIVEN>(a, stream);
}

// y [T, heads, vdim], yn [T, heads], floors [heads, gate_ld]; the gate's products at columns g_at .. of proj.
// SPAN > 0: heads of up to 128 SPAN lanes in whole 4s with everything on 16 bytes: a warp takes 4 / SPAN of them, every
// load asked for before the first is used.
#define ML_NORM_WARPS 8
template <typename TO, int SPAN>
__global__ void __launch_bounds__(ML_NORM_WARPS * 32)
mlstm_out_norm_kernel(const float* __restrict__ y, const float* __restrict__ yn, const float* __restrict__ floors,
                      long long gate_ld, const float* __restrict__ proj, int ld, int g_at,
                      const float* __restrict__ gain, float eps, int heads, int vdim, const int* __restrict__ row_req,
                      TO* __restrict__ out, int n_rows) {
  constexpr int ITEMS = SPAN ? 4 / SPAN : 1;
  const int lane = threadIdx.x & 31;
  const int first = (blockIdx.x * ML_NORM_WARPS + (threadIdx.x >> 5)) * ITEMS;
  pdl_wait();
  pdl_launch();
  if (SPAN) {
    constexpr int WIDE = SPAN ? SPAN : 1;
    float4 kept[ITEMS][WIDE], gate[ITEMS][WIDE];
    float den[ITEMS];
    int token[ITEMS];
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
      const int t = (first + k) / heads, head = first + k - t * heads;
      const bool on = t < n_rows && row_req[t] >= 0;
      token[k] = on ? t : -1;
      den[k] = on ? fmaxf(fabsf(yn[(size_t)t * heads + head]), floors[(size_t)head * gate_ld + t]) : 1.f;
#pragma unroll
      for (int j = 0; j < WIDE; ++j) {
        const int l = (lane + 32 * j) * 4;
        kept[k][j] = gate[k][j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (on && l < vdim) {
          kept[k][j] = *reinterpret_cast<const float4*>(y + ((size_t)t * heads + head) * vdim + l);
          gate[k][j] = *reinterpret_cast<const float4*>(proj + (size_t)t * ld + g_at + head * vdim + l);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
      if (token[k] < 0) continue;             // the same for the whole warp
      const int head = first + k - token[k] * heads;
      const float inv_den = 1.0f / (den[k] + ML_EPS);
      float squares = 0.f;
#pragma unroll
      for (int j = 0; j < WIDE; ++j) {
        float4& v = kept[k][j];
        v.x *= inv_den; v.y *= inv_den; v.z *= inv_den; v.w *= inv_den;
        squares += fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
      }
      const float inv = 1.0f / sqrtf(warp_sum(squares) / (float)vdim + eps);
#pragma unroll
      for (int j = 0; j < WIDE; ++j) {
        const int l = (lane + 32 * j) * 4;
        if (l >= vdim) continue;
        const float4 w = *reinterpret_cast<const float4*>(gain + head * vdim + l), v = kept[k][j], g = gate[k][j];
        const float r[4] = {v.x * inv * w.x * ml_sigmoid(g.x), v.y * inv * w.y * ml_sigmoid(g.y),
                            v.z * inv * w.z * ml_sigmoid(g.z), v.w * inv * w.w * ml_sigmoid(g.w)};
        TO* o = out + ((size_t)token[k] * heads + head) * vdim + l;
        if (sizeof(TO) == 4) {
          *reinterpret_cast<float4*>(o) = make_float4(r[0], r[1], r[2], r[3]);
        } else {
          __nv_bfloat162 h[2] = {__floats2bfloat162_rn(r[0], r[1]), __floats2bfloat162_rn(r[2], r[3])};
          *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(h);
        }
      }
    }
    return;
  }
  const int t = first / heads, head = first % heads;
  if (t >= n_rows || row_req[t] < 0) return;
  const float* yr = y + ((size_t)t * heads + head) * vdim;
  const float* gr = proj + (size_t)t * ld + g_at + head * vdim;
  TO* o = out + ((size_t)t * heads + head) * vdim;
  const float inv_den = 1.0f / (fmaxf(fabsf(yn[(size_t)t * heads + head]), floors[(size_t)head * gate_ld + t]) + ML_EPS);
  float squares = 0.f;
  for (int l = lane; l < vdim; l += 32) {
    const float v = yr[l] * inv_den;
    squares = fmaf(v, v, squares);
  }
  const float inv = 1.0f / sqrtf(warp_sum(squares) / (float)vdim + eps);
  for (int l = lane; l < vdim; l += 32) o[l] = from_float<TO>(yr[l] * inv_den * inv * gain[head * vdim + l] * ml_sigmoid(gr[l]));
}

TOKB200_API int tokb200_mlstm_out_norm(const float* y, const float* yn, const float* floors, long long gate_ld,
                                       const float* proj, int ld, int g_at, const float* gain, float eps, int heads,
                                       int vdim, const int* row_req, void* out, int out_dtype, int n_rows,
                                       cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (heads <= 0 || vdim <= 0 || g_at + heads * vdim > ld || gate_ld < n_rows) return TOKB200_BAD_SIZE;
  const bool quads = vdim % 4 == 0 && vdim <= 512 && ld % 4 == 0 && g_at % 4 == 0 &&
                     (((uintptr_t)y | (uintptr_t)proj | (uintptr_t)gain | (uintptr_t)out) & 15) == 0;
  const int span = !quads ? 0 : vdim <= 128 ? 1 : vdim <= 256 ? 2 : 4;
  const size_t items = (size_t)n_rows * heads, a_block = (size_t)ML_NORM_WARPS * (span ? 4 / span : 1);
  const dim3 grid((unsigned)((items + a_block - 1) / a_block)), block(ML_NORM_WARPS * 32);
#define LAUNCH(TO, SPAN)                                                                                               \
  return launch_dependent(mlstm_out_norm_kernel<TO, SPAN>, grid, block, 0, stream, y, yn, floors, gate_ld, proj, ld, g_at, \
                          gain, eps, heads, vdim, row_req, (TO*)out, n_rows)
#define BY_SPAN(TO)             \
  if (span == 0) LAUNCH(TO, 0); \
  if (span == 1) LAUNCH(TO, 1); \
  if (span == 2) LAUNCH(TO, 2); \
  LAUNCH(TO, 4)
  if (out_dtype == TOKB200_F32) { BY_SPAN(float); }
  if (out_dtype == TOKB200_BF16) { BY_SPAN(__nv_bfloat16); }
#undef BY_SPAN
#undef LAUNCH
  return TOKB200_BAD_DTYPE;
}

// ---- a step of single tokens ---------------------------------------------------------------
// A block a (head, row).  A warp takes ML_COLS columns of the head's matrix at a time (n is the one behind the last),
// VEC lanes of dim a thread and load, PIECES of them; what a warp takes first is asked for before the wait on the
// input product (the matrices were written a step ago).
#define ML_STEP_WARPS 8
#define ML_COLS 4
template <int VEC, int PIECES, typename TO>
__global__ void __launch_bounds__(ML_STEP_WARPS * 32)
mlstm_step_kernel(const float* __restrict__ proj, int ld, int q_at, int k_at, int v_at, int g_at, int i_at, int f_at,
                  const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap, int heads, int dim, int vdim,
                  float scale, const float* __restrict__ gain, float eps, float* __restrict__ state, long long stride, int m_off,
                  const int* __restrict__ row_req, const int* __restrict__ state_slot, TO* __restrict__ out) {
  extern __shared__ float shared[];
  __shared__ float scratch[33];
  float* num = shared;                                    // [vdim + 1]
  const int head = blockIdx.x, t = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int r = row_req[t];
  if (r < 0) {
    pdl_wait();
    pdl_launch();
    return;
  }
  float* slot = state + (size_t)state_slot[r] * stride;
  float* mats = slot + (size_t)head * (vdim + 1) * dim;
  const float ib = i_bias[head], fb = f_bias[head];
  float S[ML_COLS][PIECES][VEC];
  auto load = [&](int col0) {
#pragma unroll
    for (int c = 0; c < ML_COLS; ++c)
#pragma unroll
      for (int p = 0; p < PIECES; ++p) {
        const int l = (lane + 32 * p) * VEC, col = col0 + c;
        const bool on = col <= vdim && l < dim;
        const float* from = mats + (size_t)col * dim + l;
        if (VEC == 4) {
          const float4 v = on ? *reinterpret_cast<const float4*>(from) : make_float4(0.f, 0.f, 0.f, 0.f);
          S[c][p][0] = v.x; S[c][p][1 % VEC] = v.y; S[c][p][2 % VEC] = v.z; S[c][p][3 % VEC] = v.w;
        } else {
          S[c][p][0] = on ? *from : 0.f;
        }
      }
  };
  load(warp * ML_COLS);
  const float m_old = slot[m_off + head];
  pdl_wait();
  pdl_launch();
  const float* row = proj + (size_t)t * ld;
  const float li = ml_capped(row[i_at + head] + ib, cap);
  const float lf = ml_log_sigmoid(ml_capped(row[f_at + head] + fb, cap));
  const float top = fmaxf(lf + m_old, li);
  const float keep = expf(lf + m_old - top), add = expf(li - top);
  float q[PIECES][VEC], k[PIECES][VEC];
#pragma unroll
  for (int p = 0; p < PIECES; ++p)
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      const int l = (lane + 32 * p) * VEC + e;
      q[p][e] = l < dim ? row[q_at + head * dim + l] * scale : 0.f;
      k[p][e] = l < dim ? row[k_at + head * dim + l] * add : 0.f;
    }
  for (int col0 = warp * ML_COLS; col0 <= vdim; col0 += ML_STEP_WARPS * ML_COLS) {
    if (col0 != warp * ML_COLS) load(col0);
    float sum[ML_COLS];
#pragma unroll
    for (int c = 0; c < ML_COLS; ++c) {
      const int col = col0 + c;
      const float v = col < vdim ? row[v_at + head * vdim + col] : 1.f;
      sum[c] = 0.f;
#pragma unroll
      for (int p = 0; p < PIECES; ++p)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          S[c][p][e] = fmaf(keep, S[c][p][e], k[p][e] * v);
          sum[c] = fmaf(S[c][p][e], q[p][e], sum[c]);
        }
    }
#pragma unroll
    for (int c = 0; c < ML_COLS; ++c) {
      const int col = col0 + c;
      if (col <= vdim) {
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
          const int l = (lane + 32 * p) * VEC;
          if (l < dim) {
            float* to = mats + (size_t)col * dim + l;
            if (VEC == 4)
              *reinterpret_cast<float4*>(to) = make_float4(S[c][p][0], S[c][p][1 % VEC], S[c][p][2 % VEC], S[c][p][3 % VEC]);
            else
              *to = S[c][p][0];
          }
        }
      }
    }
#pragma unroll
    for (int c = 0; c < ML_COLS; ++c) {
      const float whole = warp_sum(sum[c]);
      if (lane == 0 && col0 + c <= vdim) num[col0 + c] = whole;
    }
  }
  __syncthreads();
  if (threadIdx.x == 0) slot[m_off + head] = top;
  const float inv_den = 1.0f / (fmaxf(fabsf(num[vdim]), expf(-top)) + ML_EPS);
  float squares = 0.f;
  for (int l = threadIdx.x; l < vdim; l += blockDim.x) {
    const float v = num[l] * inv_den;
    squares = fmaf(v, v, squares);
  }
  const float inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)vdim + eps);
  for (int l = threadIdx.x; l < vdim; l += blockDim.x)
    out[((size_t)t * heads + head) * vdim + l] =
        from_float<TO>(num[l] * inv_den * inv * gain[head * vdim + l] * ml_sigmoid(row[g_at + head * vdim + l]));
}

TOKB200_API int tokb200_mlstm_step(const float* proj, int ld, int q_at, int k_at, int v_at, int g_at, int i_at, int f_at,
                                   const float* i_bias, const float* f_bias, float cap, int heads, int dim, int vdim,
                                   float scale, const float* gain, float eps, float* state, long long stride, int m_off,
                                   const int* row_req, const int* state_slot, int n_rows, void* out, int out_dtype,
                                   cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (heads <= 0 || dim <= 0 || dim > 256 || vdim <= 0 || vdim > 8192 || n_rows > 65535 || cap <= 0.f ||
      q_at + heads * dim > ld || k_at + heads * dim > ld || v_at + heads * vdim > ld || g_at + heads * vdim > ld ||
      i_at + heads > ld || f_at + heads > ld || (long long)heads * (vdim + 1) * dim > m_off || m_off + heads > stride)
    return TOKB200_BAD_SIZE;
  const dim3 grid(heads, n_rows), block(ML_STEP_WARPS * 32);
  const size_t smem = (size_t)(vdim + 1) * sizeof(float);
  const bool quads = dim % 4 == 0 && stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
#define LAUNCH(VEC, PIECES, TO)                                                                                          \
  return launch_dependent(mlstm_step_kernel<VEC, PIECES, TO>, grid, block, smem, stream, proj, ld, q_at, k_at, v_at, g_at, \
                          i_at, f_at, i_bias, f_bias, cap, heads, dim, vdim, scale, gain, eps, state, stride, m_off,     \
                          row_req, state_slot, (TO*)out)
#define BY_SIZE(TO)                       \
  if (quads && dim <= 128) LAUNCH(4, 1, TO); \
  if (quads) LAUNCH(4, 2, TO);            \
  LAUNCH(1, 8, TO)
  if (out_dtype == TOKB200_F32) { BY_SIZE(float); }
  if (out_dtype == TOKB200_BF16) { BY_SIZE(__nv_bfloat16); }
#undef BY_SIZE
#undef LAUNCH
  return TOKB200_BAD_DTYPE;
}
