// A norm without statistics, and the residual stream's steps around it.
//
//   stream_update   x <- (x or base) + y + share * carried;  optionally out = tanh(alpha x) * gain + bias of the
//                   new x (alpha one number, gain and bias over the width), or the new x as it is in the compute
//                   type, and beside it a second matrix (`beside`) in the same row
//
// y is a sublayer's output: [T, H] in float32 or bfloat16, or float32 partial sums [S, T, H] of a product cut
// along k, added in index order.  carried [T, H] with one number a row (`share`): what an identity expert
// hands through.  base: a vector over the width that x is started from instead of its own value.  rows: only
// those rows of x are read (then nothing is added and x stays).  Everything is 32-bit but y, carried and out.
// Nothing crosses elements, so the work is cut evenly over the device whatever the number of rows.
#include "common.cuh"

struct SuArgs {
  float* x;
  const void* y;
  int y_bf16, y_partials;
  long long y_stride;
  const float* base;
  const void* carried;
  int carried_bf16, share_ld;
  const float* share;
  int norm;                  // 1: out = tanh(alpha x) gain + bias; 0: out = x
  float alpha;
  const float* gain;
  const float* bias;
  const float* beside;
  int out_ld;
  const int* rows;
  int n_rows, hidden;
};

__device__ __forceinline__ float su_norm(float v, float alpha, float gain, float bias) {
  return fmaf(tanhf(alpha * v), gain, bias);
}

template <typename TO>
__global__ void stream_update_kernel(SuArgs a, TO* __restrict__ out) {
  pdl_wait();
  pdl_launch();
  const size_t n = (size_t)a.n_rows * a.hidden, stride = (size_t)gridDim.x * blockDim.x;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride) {
    const int t = (int)(i / a.hidden), c = (int)(i % a.hidden);
    const size_t at = (size_t)(a.rows ? a.rows[t] : t) * a.hidden + c;
    float v = a.base ? a.base[c] : a.x[at];
    bool changed = a.base != nullptr;
    if (a.y) {
      float y = 0.f;
      if (a.y_bf16) y = __bfloat162float(((const __nv_bfloat16*)a.y)[at]);
      else
        for (int s = 0; s < a.y_partials; ++s) y += ((const float*)a.y)[(size_t)s * a.y_stride + at];
      v += y;
      changed = true;
    }
    if (a.carried) {
      const float h = a.carried_bf16 ? __bfloat162float(((const __nv_bfloat16*)a.carried)[at]) : ((const float*)a.carried)[at];
      v = fmaf(a.share[(size_t)t * a.share_ld], h, v);
      changed = true;
    }
    if (changed) a.x[at] = v;
    if (out) {
      TO* o = out + (size_t)t * a.out_ld;
      o[c] = from_float<TO>(a.norm ? su_norm(v, a.alpha, a.gain[c], a.bias[c]) : v);
      if (a.beside) o[a.hidden + c] = from_float<TO>(a.beside[at]);
    }
  }
}

// ---- widths in whole 8s, everything on 16 bytes: eight consecutive elements a thread ----
__device__ __forceinline__ void su_load8(const float* p, float v[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void su_load8(const __nv_bfloat16* p, float v[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x;
    v[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void su_store8(float* p, const float v[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void su_store8(__nv_bfloat16* p, const float v[8]) {
  __nv_bfloat162 h[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(h);
}

template <typename TO>
__global__ void __launch_bounds__(256) stream_update_rows8_kernel(SuArgs a, TO* __restrict__ out) {
  const int per_row = a.hidden / 8;
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const bool on = i < (size_t)a.n_rows * per_row;
  const int t = on ? (int)(i / per_row) : 0, c = on ? (int)(i % per_row) * 8 : 0;
  // gain and bias are weights: asked for before the wait on the predecessor
  float gain[8], bias[8];
  if (on && a.norm) {
    su_load8(a.gain + c, gain);
    su_load8(a.bias + c, bias);
  }
  pdl_wait();
  pdl_launch();
  if (!on) return;
  const size_t at = (size_t)(a.rows ? a.rows[t] : t) * a.hidden + c;
  float v[8];
  su_load8(a.base ? a.base + c : a.x + at, v);
  bool changed = a.base != nullptr;
  if (a.y) {
    float y[8];
    if (a.y_bf16) su_load8((const __nv_bfloat16*)a.y + at, y);
    else {
      su_load8((const float*)a.y + at, y);
      for (int s = 1; s < a.y_partials; ++s) {
        float part[8];
        su_load8((const float*)a.y + (size_t)s * a.y_stride + at, part);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] += part[e];
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] += y[e];
    changed = true;
  }
  if (a.carried) {
    float h[8];
    const float share = a.share[(size_t)t * a.share_ld];
    if (a.carried_bf16) su_load8((const __nv_bfloat16*)a.carried + at, h);
    else su_load8((const float*)a.carried + at, h);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = fmaf(share, h[e], v[e]);
    changed = true;
  }
  if (changed) su_store8(a.x + at, v);
  if (out == nullptr) return;
  if (a.norm) {
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = su_norm(v[e], a.alpha, gain[e], bias[e]);
  }
  TO* o = out + (size_t)t * a.out_ld + c;
  su_store8(o, v);
  if (a.beside) {
    su_load8(a.beside + at, v);
    su_store8(o + a.hidden, v);
  }
}

// y, base, carried, beside, rows and out may be null; out rows are out_ld elements apart (2 * hidden with `beside`).
TOKB200_API int tokb200_stream_update(float* x, const void* y, int y_dtype, int y_partials, long long y_stride,
                                      const float* base, const void* carried, int carried_dtype, const float* share,
                                      int share_ld, int norm, float alpha, const float* gain, const float* bias,
                                      const float* beside, void* out, int out_dtype, int out_ld, const int* rows,
                                      int n_rows, int hidden, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (hidden <= 0 || (y && y_partials < 1) || (rows && (y || base || carried)) || (carried && share == nullptr) ||
      (norm && (gain == nullptr || bias == nullptr || out == nullptr)) || (out && out_ld < (beside ? 2 * hidden : hidden)))
    return TOKB200_BAD_SIZE;
  if (y && y_dtype == TOKB200_BF16 && y_partials != 1) return TOKB200_BAD_DTYPE;
  SuArgs a = {x, y, y_dtype == TOKB200_BF16, y_partials, y_stride, base, carried, carried_dtype == TOKB200_BF16, share_ld,
              share, norm, alpha, gain, bias, beside, out_ld, rows, n_rows, hidden};
  const uintptr_t all = (uintptr_t)x | (uintptr_t)y | (uintptr_t)base | (uintptr_t)carried | (uintptr_t)gain |
                        (uintptr_t)bias | (uintptr_t)beside | (uintptr_t)out;
  const bool wide = hidden % 8 == 0 && (all & 15) == 0 && y_stride % 4 == 0 && out_ld % 8 == 0;
  const bool bf16 = out != nullptr && out_dtype == TOKB200_BF16;
  const size_t n = (size_t)n_rows * hidden / (wide ? 8 : 1);
  const int threads = 256;
  const size_t blocks = (n + threads - 1) / threads;
  if (wide) {
    const dim3 grid((unsigned)blocks);
    if (bf16)
      return launch_dependent(stream_update_rows8_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, a, (__nv_bfloat16*)out);
    return launch_dependent(stream_update_rows8_kernel<float>, grid, dim3(threads), 0, stream, a, (float*)out);
  }
  const dim3 grid((unsigned)(blocks < 8192 ? blocks : 8192));
  if (bf16) return launch_dependent(stream_update_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, a, (__nv_bfloat16*)out);
  return launch_dependent(stream_update_kernel<float>, grid, dim3(threads), 0, stream, a, (float*)out);
}
