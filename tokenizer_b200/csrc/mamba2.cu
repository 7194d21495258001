// The selective state-space recurrence with a scalar decay a head (the Mamba-2 form), in 32-bit.
//
// Per head a matrix S (N x P, float32, a request's state) and per token t of that head:
//     dt = softplus(raw_dt + dt_bias);  S <- exp(-exp(A_log) dt) S + dt B x^T;  y = S^T C + D x
// with x (P lanes of the head), B and C (N lanes of the head's group) the convolved and activated
// inputs.
//
//   mamba2_scan      the recurrence over every request's rows of the step, token by token, on the scan that
//                    matrix recurrences share (matrix_scan.cuh).  State: [slots, stride], a slot's
//                    matrices [heads, P, N] at its start.
//   mamba2_out_norm  y * silu(z), divided by its root mean square inside each of `parts` equal parts
//                    of the row, times a gain: a block a (row, part).
#include "matrix_scan.cuh"

// xbc: float32 [T, channels]: x (heads * P), B (groups * N), C (groups * N).  proj: the input product
// [T, ld] whose columns dt_at .. + heads are the raw step sizes.
TOKB200_API int tokb200_mamba2_scan(const float* xbc, int channels, const void* proj, int proj_dtype, int ld, int dt_at,
                                    const float* dt_bias, const float* a_log, const float* skip, int heads, int groups,
                                    int P, int N, float* state, long long stride, const int* q_start,
                                    const int* state_slot, int n_requests, float* y, float* scratch, int segments,
                                    cudaStream_t stream) {
  if (n_requests <= 0) return TOKB200_OK;
  if (channels != heads * P + 2 * groups * N) return TOKB200_BAD_SIZE;
  MatrixScanArgs a = {};
  a.x = xbc; a.x_ld = channels; a.x_head = P;
  a.b = xbc + (size_t)heads * P; a.b_ld = channels; a.b_group = N;
  a.c = a.b + (size_t)groups * N; a.c_ld = channels; a.c_group = N;
  a.heads = heads; a.groups = groups; a.P = P; a.copied = P; a.N = N; a.scale = 1.f; a.skip = skip;
  a.state = state; a.stride = stride; a.q_start = q_start; a.state_slot = state_slot; a.y = y;
  a.raw_ld = ld; a.bias = dt_bias; a.a_log = a_log; a.scratch = scratch; a.segments = segments; a.n_requests = n_requests;
  if (proj_dtype == TOKB200_F32) {
    a.raw = (const float*)proj + dt_at;
    return launch_matrix_scan<float, MS_GATES_STEP>(a, stream);
  }
  if (proj_dtype == TOKB200_BF16) {
    a.raw = (const __nv_bfloat16*)proj + dt_at;
    return launch_matrix_scan<__nv_bfloat16, MS_GATES_STEP>(a, stream);
  }
  return TOKB200_BAD_DTYPE;
}

// y: float32 [T, inner]; z: the gate's pre-activation, columns z_at .. + inner of `proj` [T, ld].
#define M2_NORM_PER_THREAD 8
template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
mamba2_out_norm_kernel(const float* __restrict__ y, const TI* __restrict__ proj, int ld, int z_at,
                       const float* __restrict__ gain, float eps, int inner, int parts,
                       const int* __restrict__ row_req, TO* __restrict__ out) {
  __shared__ float scratch[33];
  const int t = blockIdx.x, g = blockIdx.y;
  const int width = inner / parts;
  pdl_wait();
  pdl_launch();
  if (row_req[t] < 0) return;
  const float* yr = y + (size_t)t * inner + (size_t)g * width;
  const TI* zr = proj + (size_t)t * ld + z_at + (size_t)g * width;
  float kept[M2_NORM_PER_THREAD];
  float squares = 0.f;
#pragma unroll
  for (int k = 0; k < M2_NORM_PER_THREAD; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    kept[k] = 0.f;
    if (i < width) {
      const float z = to_float(zr[i]);
      const float v = yr[i] * (z / (1.0f + expf(-z)));
      kept[k] = v;
      squares = fmaf(v, v, squares);
    }
  }
  for (int i = threadIdx.x + M2_NORM_PER_THREAD * blockDim.x; i < width; i += blockDim.x) {
    const float z = to_float(zr[i]);
    const float v = yr[i] * (z / (1.0f + expf(-z)));
    squares = fmaf(v, v, squares);
  }
  const float inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)width + eps);
  TO* o = out + (size_t)t * inner + (size_t)g * width;
  const float* gr = gain + (size_t)g * width;
#pragma unroll
  for (int k = 0; k < M2_NORM_PER_THREAD; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < width) o[i] = from_float<TO>(kept[k] * inv * gr[i]);
  }
  for (int i = threadIdx.x + M2_NORM_PER_THREAD * blockDim.x; i < width; i += blockDim.x) {
    const float z = to_float(zr[i]);
    o[i] = from_float<TO>(yr[i] * (z / (1.0f + expf(-z))) * inv * gr[i]);
  }
}


// Four neighbouring lanes of the gate's pre-activation.
__device__ __forceinline__ float4 m2_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 m2_load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void m2_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void m2_store4(__nv_bfloat16* p, float4 v) {
  uint2 raw;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
  h[0] = __floats2bfloat162_rn(v.x, v.y);
  h[1] = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ float m2_silu(float z) { return z / (1.0f + expf(-z)); }

// The same for parts of whole 4s up to 2,048 lanes, everything aligned: four lanes a load, the part kept in
// registers between the sum and the scaling.
template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
mamba2_out_norm4_kernel(const float* __restrict__ y, const TI* __restrict__ proj, int ld, int z_at,
                        const float* __restrict__ gain, float eps, int inner, int parts,
                        const int* __restrict__ row_req, TO* __restrict__ out) {
  __shared__ float scratch[33];
  const int t = blockIdx.x, g = blockIdx.y;
  const int width = inner / parts;
  pdl_wait();
  pdl_launch();
  if (row_req[t] < 0) return;
  const float* yr = y + (size_t)t * inner + (size_t)g * width;
  const TI* zr = proj + (size_t)t * ld + z_at + (size_t)g * width;
  float4 kept[2];
  float squares = 0.f;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int i = (threadIdx.x + k * blockDim.x) * 4;
    kept[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < width) {
      const float4 v = m2_load4(yr + i), z = m2_load4(zr + i);
      kept[k] = make_float4(v.x * m2_silu(z.x), v.y * m2_silu(z.y), v.z * m2_silu(z.z), v.w * m2_silu(z.w));
      squares = fmaf(kept[k].x, kept[k].x, squares);
      squares = fmaf(kept[k].y, kept[k].y, squares);
      squares = fmaf(kept[k].z, kept[k].z, squares);
      squares = fmaf(kept[k].w, kept[k].w, squares);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)width + eps);
  TO* o = out + (size_t)t * inner + (size_t)g * width;
  const float* gr = gain + (size_t)g * width;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int i = (threadIdx.x + k * blockDim.x) * 4;
    if (i < width) {
      const float4 w = m2_load4(gr + i);
      m2_store4(o + i, make_float4(kept[k].x * inv * w.x, kept[k].y * inv * w.y, kept[k].z * inv * w.z, kept[k].w * inv * w.w));
    }
  }
}

TOKB200_API int tokb200_mamba2_out_norm(const float* y, const void* proj, int proj_dtype, int ld, int z_at,
                                        const float* gain, float eps, int inner, int parts, const int* row_req,
                                        void* out, int out_dtype, int n_rows, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (inner <= 0 || parts <= 0 || inner % parts || parts > 65535) return TOKB200_BAD_SIZE;
  const int width = inner / parts;
  const dim3 grid(n_rows, parts);
  const int z_size = proj_dtype == TOKB200_BF16 ? 2 : 4, o_size = out_dtype == TOKB200_BF16 ? 2 : 4;
  if (width % 4 == 0 && width <= 2048 && ld % 4 == 0 && z_at % 4 == 0 && (((uintptr_t)y | (uintptr_t)gain) & 15) == 0 &&
      ((uintptr_t)proj % (4 * z_size)) == 0 && ((uintptr_t)out % (4 * o_size)) == 0) {
    int threads4 = (width / 4 + 31) / 32 * 32;
    threads4 = threads4 > 256 ? 256 : threads4;
#define LAUNCH4(TI, TO)                                                                                              \
    return launch_dependent(mamba2_out_norm4_kernel<TI, TO>, grid, dim3(threads4), 0, stream, y, (const TI*)proj, ld, \
                            z_at, gain, eps, inner, parts, row_req, (TO*)out)
    if (proj_dtype == TOKB200_F32 && out_dtype == TOKB200_F32) LAUNCH4(float, float);
    if (proj_dtype == TOKB200_F32 && out_dtype == TOKB200_BF16) LAUNCH4(float, __nv_bfloat16);
    if (proj_dtype == TOKB200_BF16 && out_dtype == TOKB200_BF16) LAUNCH4(__nv_bfloat16, __nv_bfloat16);
    if (proj_dtype == TOKB200_BF16 && out_dtype == TOKB200_F32) LAUNCH4(__nv_bfloat16, float);
#undef LAUNCH4
  }
  int threads = (width + 31) / 32 * 32;
  threads = threads > 256 ? 256 : threads;
#define LAUNCH(TI, TO)                                                                                           \
  return launch_dependent(mamba2_out_norm_kernel<TI, TO>, grid, dim3(threads), 0, stream, y, (const TI*)proj, ld, \
                          z_at, gain, eps, inner, parts, row_req, (TO*)out)
  if (proj_dtype == TOKB200_F32 && out_dtype == TOKB200_F32) LAUNCH(float, float);
  if (proj_dtype == TOKB200_F32 && out_dtype == TOKB200_BF16) LAUNCH(float, __nv_bfloat16);
  if (proj_dtype == TOKB200_BF16 && out_dtype == TOKB200_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  if (proj_dtype == TOKB200_BF16 && out_dtype == TOKB200_F32) LAUNCH(__nv_bfloat16, float);
#undef LAUNCH
  return TOKB200_BAD_DTYPE;
}
