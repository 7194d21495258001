// The small kernels around attention over a cached latent.
//
// latent_prepare: one projection's output row holds, side by side, a query latent (q_rank
// lanes), a key/value latent (kv_rank lanes) and a key part that carries the position (rot_dim
// lanes, possibly none).  Per token: the query latent is RMS-normed with its gain and written
// out dense; the key/value latent is RMS-normed with its gain and written to the token's cache
// row; the positional key part is rotated at the token's position and written behind it in the
// same cache row.  Norm statistics, angles, sines and cosines are 32-bit.
//
// rotate_interleaved: rotary encoding with lane 2i paired with lane 2i + 1, on `dims` lanes
// starting at `lane0` of every head's vector, in place; angle = position * inv_freq[i].
#include "common.cuh"

// a warp a token: the row's two sums by shuffles, no barrier; the second pass over the row hits L1
#define LAT_WARPS 8
template <typename TI, typename TO>
__global__ void __launch_bounds__(LAT_WARPS * 32)
latent_prepare_kernel(const TI* __restrict__ proj, int ld, int q_at, int q_rank, int c_at,
                      int kv_rank, int rot_dim, int rot_dims, const float* __restrict__ q_gain,
                      const float* __restrict__ c_gain, float eps,
                      const float* __restrict__ inv_freq, const int* __restrict__ pos,
                      const int* __restrict__ row_req, const int* __restrict__ slot,
                      TO* __restrict__ q_latent, TO* __restrict__ pool, int pool_row, int n_rows) {
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x * LAT_WARPS + (threadIdx.x >> 5);
  const bool have = t < n_rows;
  const int r = have ? row_req[t] : -1;
  const int p = have ? pos[t] : 0;
  const int where = (have && slot) ? slot[t] : -1;
  pdl_wait();
  pdl_launch();
  if (r < 0) return;
  const TI* row = proj + (size_t)t * ld;
  float sq = 0.f, sc = 0.f;
  for (int i = lane; i < q_rank; i += 32) {
    const float v = to_float(row[q_at + i]);
    sq += v * v;
  }
  for (int i = lane; i < kv_rank; i += 32) {
    const float v = to_float(row[c_at + i]);
    sc += v * v;
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  const float inv_q = 1.0f / sqrtf(sq / (float)q_rank + eps);
  const float inv_c = 1.0f / sqrtf(sc / (float)kv_rank + eps);
  TO* q_dst = q_latent + (size_t)t * q_rank;
  for (int i = lane; i < q_rank; i += 32)
    q_dst[i] = from_float<TO>(to_float(row[q_at + i]) * inv_q * q_gain[i]);
  if (where < 0) return;
  TO* c_dst = pool + (size_t)where * pool_row;
  for (int i = lane; i < kv_rank; i += 32)
    c_dst[i] = from_float<TO>(to_float(row[c_at + i]) * inv_c * c_gain[i]);
  const TI* k_rot = row + c_at + kv_rank;
  for (int i = lane; i < rot_dim; i += 32) {
    float value = to_float(k_rot[i]);
    if (i < rot_dims) {          // lane 2j pairs with lane 2j + 1; the lanes behind rot_dims pass
      float s, c;
      sincosf((float)p * inv_freq[i >> 1], &s, &c);
      const float other = to_float(k_rot[i ^ 1]);
      value = (i & 1) ? value * c + other * s : value * c - other * s;
    }
    c_dst[kv_rank + i] = from_float<TO>(value);
  }
}

TOKB200_API int tokb200_latent_prepare(const void* proj, int proj_dtype, int ld, int q_at, int q_rank,
                                       int c_at, int kv_rank, int rot_dim, int rot_dims,
                                       const float* q_gain, const float* c_gain, float eps,
                                       const float* inv_freq, const int* pos, const int* row_req,
                                       const int* slot, void* q_latent, void* pool, int pool_row,
                                       int out_dtype, int n_rows, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (q_rank <= 0 || kv_rank <= 0 || rot_dim < 0 || rot_dims < 0 || rot_dims > rot_dim || (rot_dims & 1) ||
      pool_row < kv_rank + rot_dim || q_at + q_rank > ld || c_at + kv_rank + rot_dim > ld)
    return TOKB200_BAD_SIZE;
#define LAUNCH(TI, TO)                                                                           \
  return launch_dependent(latent_prepare_kernel<TI, TO>, dim3((n_rows + LAT_WARPS - 1) / LAT_WARPS),  \
                          dim3(LAT_WARPS * 32), 0, stream,                                        \
                          (const TI*)proj, ld, q_at, q_rank, c_at, kv_rank, rot_dim, rot_dims,   \
                          q_gain, c_gain, eps, inv_freq, pos, row_req, slot, (TO*)q_latent,      \
                          (TO*)pool, pool_row, n_rows)
  if (proj_dtype == TOKB200_F32 && out_dtype == TOKB200_F32) LAUNCH(float, float);
  if (proj_dtype == TOKB200_F32 && out_dtype == TOKB200_BF16) LAUNCH(float, __nv_bfloat16);
  if (proj_dtype == TOKB200_BF16 && out_dtype == TOKB200_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
#undef LAUNCH
  return TOKB200_BAD_DTYPE;
}

// x: [rows, heads, head_row]; pairs (lane0 + 2i, lane0 + 2i + 1), i < dims / 2, are rotated
template <typename T>
__global__ void __launch_bounds__(256)
rotate_interleaved_kernel(T* __restrict__ x, int heads, int head_row, int lane0, int dims,
                          const float* __restrict__ inv_freq, const int* __restrict__ pos,
                          const int* __restrict__ row_req, int n_rows) {
  pdl_wait();
  pdl_launch();
  const int half = dims / 2;
  const size_t total = (size_t)n_rows * heads * half;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total;
       i += (size_t)gridDim.x * blockDim.x) {
    const int pair = (int)(i % half);
    const size_t th = i / half;
    const int t = (int)(th / heads);
    if (row_req[t] < 0) continue;
    float s, c;
    sincosf((float)pos[t] * inv_freq[pair], &s, &c);
    T* at = x + th * head_row + lane0 + 2 * pair;
    const float u = to_float(at[0]), v = to_float(at[1]);
    at[0] = from_float<T>(u * c - v * s);
    at[1] = from_float<T>(v * c + u * s);
  }
}

// bfloat16, 8 lanes (four pairs, 16 bytes) a thread: for rotated ranges that start and end on 16 bytes
__global__ void __launch_bounds__(256)
rotate_interleaved_vec_kernel(__nv_bfloat16* __restrict__ x, int heads, int head_row, int lane0, int dims,
                              const float* __restrict__ inv_freq, const int* __restrict__ pos,
                              const int* __restrict__ row_req, int n_rows) {
  pdl_wait();
  pdl_launch();
  const int pieces = dims / 8;
  const size_t total = (size_t)n_rows * heads * pieces;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total;
       i += (size_t)gridDim.x * blockDim.x) {
    const int piece = (int)(i % pieces);
    const size_t th = i / pieces;
    const int t = (int)(th / heads);
    if (row_req[t] < 0) continue;
    const float p = (float)pos[t];
    uint4* at = reinterpret_cast<uint4*>(x + th * head_row + lane0 + 8 * piece);
    uint4 v = *at;
    __nv_bfloat162* pairs = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      float s, c;
      sincosf(p * inv_freq[4 * piece + k], &s, &c);
      const float u = __low2float(pairs[k]), w = __high2float(pairs[k]);
      pairs[k] = __floats2bfloat162_rn(u * c - w * s, w * c + u * s);
    }
    *at = v;
  }
}

TOKB200_API int tokb200_rotate_interleaved(void* x, int dtype, int heads, int head_row, int lane0, int dims,
                                           const float* inv_freq, const int* pos, const int* row_req,
                                           int n_rows, cudaStream_t stream) {
  if (n_rows <= 0 || dims <= 0) return TOKB200_OK;
  if (heads <= 0 || (dims & 1) || lane0 < 0 || lane0 + dims > head_row) return TOKB200_BAD_SIZE;
  if (dtype == TOKB200_BF16 && dims % 8 == 0 && lane0 % 8 == 0 && head_row % 8 == 0 && ((uintptr_t)x & 15) == 0) {
    const size_t pieces = (size_t)n_rows * heads * (dims / 8);
    const unsigned vec_blocks = (unsigned)((pieces + 255) / 256 > 148 * 16 ? 148 * 16 : (pieces + 255) / 256);
    return launch_dependent(rotate_interleaved_vec_kernel, dim3(vec_blocks), dim3(256), 0, stream, (__nv_bfloat16*)x,
                            heads, head_row, lane0, dims, inv_freq, pos, row_req, n_rows);
  }
  const size_t total = (size_t)n_rows * heads * (dims / 2);
  const unsigned blocks = (unsigned)((total + 255) / 256 > 148 * 16 ? 148 * 16 : (total + 255) / 256);
  if (dtype == TOKB200_F32)
    return launch_dependent(rotate_interleaved_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)x,
                            heads, head_row, lane0, dims, inv_freq, pos, row_req, n_rows);
  if (dtype == TOKB200_BF16)
    return launch_dependent(rotate_interleaved_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream,
                            (__nv_bfloat16*)x, heads, head_row, lane0, dims, inv_freq, pos, row_req, n_rows);
  return TOKB200_BAD_DTYPE;
}

// ---- queries straight from the mixer's input, and values that pass a gate -------------------
//
// latent_rotate_store: one projection's output row holds the key/value latent with its positional key part (c_at ..)
// and, for every head, a query in the cache row's own lanes (q_at .., `row` a head: kv_rank lanes without position,
// rot_dim with, the rest zero).  The latent is RMS-normed with its gain, the positional parts of the key and of every
// query are rotated (lane 2i with lane 2i + 1), the key row goes to the cache, the queries to q_out.  A block a token;
// the angles are formed in 64-bit and brought into one turn before sine and cosine, once a token.  The key row is one
// warp's; the queries are a warp's each, or, where everything comes in whole 4s on 16 bytes (QUADS), four lanes a
// thread wherever they lie, asked for before the angles are waited for.
template <typename TO, bool QUADS>
__global__ void __launch_bounds__(256)
latent_rotate_store_kernel(const float* __restrict__ proj, int ld, int c_at, int q_at, int heads, int kv_rank, int rot_dim,
                           int rot_dims, int row, const float* __restrict__ c_gain, float eps,
                           const double* __restrict__ inv_freq, const int* __restrict__ pos,
                           const int* __restrict__ row_req, const int* __restrict__ slot, TO* __restrict__ q_out,
                           TO* __restrict__ pool) {
  extern __shared__ float angles[];          // cosines, then sines, one a frequency
  const int half = rot_dims >> 1;
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int r = row_req[t], p = pos[t];
  const int where = slot ? slot[t] : -1;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    double a = (double)p * inv_freq[i];
    a -= 6.283185307179586476925 * rint(a * 0.15915494309189533577);
    float sn, cs;
    sincosf((float)a, &sn, &cs);
    angles[i] = cs;
    angles[half + i] = sn;
  }
  pdl_wait();
  pdl_launch();
  if (r < 0) return;
  const float* in = proj + (size_t)t * ld;
  if (QUADS) {
    constexpr int DEEP = 4;
    const int n = heads * row;
    for (int base = threadIdx.x * 4; base < n; base += blockDim.x * 4 * DEEP) {
      float4 v[DEEP];
#pragma unroll
      for (int d = 0; d < DEEP; ++d) {
        const int i = base + d * blockDim.x * 4;
        if (i < n) v[d] = *reinterpret_cast<const float4*>(in + q_at + i);
      }
      if (base == threadIdx.x * 4) __syncthreads();      // the angles (every thread comes by once: n is at least a thread's 4 lanes)
#pragma unroll
      for (int d = 0; d < DEEP; ++d) {
        const int i = base + d * blockDim.x * 4;
        if (i >= n) continue;
        const int l = i % row - kv_rank;                 // inside the rotated part: 0 .. rot_dims - 1
        if (l >= 0 && l < rot_dims) {
          const float c0 = angles[l >> 1], s0 = angles[half + (l >> 1)], c1 = angles[(l >> 1) + 1], s1 = angles[half + (l >> 1) + 1];
          v[d] = make_float4(v[d].x * c0 - v[d].y * s0, v[d].y * c0 + v[d].x * s0, v[d].z * c1 - v[d].w * s1,
                             v[d].w * c1 + v[d].z * s1);
        }
        TO* dst = q_out + (size_t)t * n + i;
        if (sizeof(TO) == 4) {
          *reinterpret_cast<float4*>(dst) = v[d];
        } else {
          __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v[d].x, v[d].y), __floats2bfloat162_rn(v[d].z, v[d].w)};
          *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(h);
        }
      }
    }
  } else {
    __syncthreads();
  }
  // lane l of a rotated part that starts at `part`
  auto rotated = [&](const float* part, int l) {
    const float own = part[l];
    if (l >= rot_dims) return own;
    const float other = part[l ^ 1], c = angles[l >> 1], s = angles[half + (l >> 1)];
    return (l & 1) ? own * c + other * s : own * c - other * s;
  };
  for (int item = QUADS ? (warp == warps - 1 ? 0 : 1) : warp; item <= (QUADS ? 0 : heads); item += warps) {
    if (item == 0) {                          // the latent and the shared key part
      if (where < 0) continue;
      const float* c = in + c_at;
      float squares = 0.f;
      for (int l = lane; l < kv_rank; l += 32) squares = fmaf(c[l], c[l], squares);
      const float inv = 1.0f / sqrtf(warp_sum(squares) / (float)kv_rank + eps);
      TO* dst = pool + (size_t)where * row;
      for (int l = lane; l < row; l += 32) {
        float v = 0.f;
        if (l < kv_rank) v = c[l] * inv * c_gain[l];
        else if (l < kv_rank + rot_dim) v = rotated(c + kv_rank, l - kv_rank);
        dst[l] = from_float<TO>(v);
      }
    } else {
      const float* q = in + q_at + (size_t)(item - 1) * row;
      TO* dst = q_out + ((size_t)t * heads + item - 1) * row;
      for (int l = lane; l < row; l += 32)
        dst[l] = from_float<TO>((l < kv_rank || l >= kv_rank + rot_dim) ? q[l] : rotated(q + kv_rank, l - kv_rank));
    }
  }
}

TOKB200_API int tokb200_latent_rotate_store(const float* proj, int ld, int c_at, int q_at, int heads, int kv_rank,
                                            int rot_dim, int rot_dims, int row, const float* c_gain, float eps,
                                            const double* inv_freq, const int* pos, const int* row_req, const int* slot,
                                            void* q_out, void* pool, int out_dtype, int n_rows, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (heads <= 0 || kv_rank <= 0 || rot_dim < 0 || rot_dims < 0 || rot_dims > rot_dim || (rot_dims & 1) ||
      row < kv_rank + rot_dim || c_at + kv_rank + rot_dim > ld || q_at + heads * row > ld || rot_dims > 8192 ||
      (rot_dims > 0 && inv_freq == nullptr))
    return TOKB200_BAD_SIZE;
  const bool quads = heads * row >= 128 && ((row | kv_rank | rot_dims | q_at | ld) & 3) == 0 && (((uintptr_t)proj | (uintptr_t)q_out) & 15) == 0;
  // QUADS: no more threads than there are quads of query lanes
  const int warps = quads ? (heads * row / 128 < 8 ? heads * row / 128 : 8) : heads + 1 < 8 ? heads + 1 : 8;
  const size_t smem = (size_t)rot_dims * sizeof(float);
#define LAUNCH(TO, QUADS)                                                                                              \
  return launch_dependent(latent_rotate_store_kernel<TO, QUADS>, dim3(n_rows), dim3(warps * 32), smem, stream, proj, ld, c_at, \
                          q_at, heads, kv_rank, rot_dim, rot_dims, row, c_gain, eps, inv_freq, pos, row_req, slot,      \
                          (TO*)q_out, (TO*)pool)
  if (out_dtype == TOKB200_F32) {
    if (quads) LAUNCH(float, true);
    LAUNCH(float, false);
  }
  if (out_dtype == TOKB200_BF16) {
    if (quads) LAUNCH(__nv_bfloat16, true);
    LAUNCH(__nv_bfloat16, false);
  }
#undef LAUNCH
  return TOKB200_BAD_DTYPE;
}

// latent_values: the heads' values from their weighted latents, through a gate:
//     out[t, h, l] = (sum_c w[h, l, c] mixed[t, h, c]) * sigmoid(gate[t, g_at + h vdim + l])
// mixed [T, heads, row], w per head.  In bfloat16 (w [heads, vdim, row], row in whole 16s) a product on tensor cores
// whose epilogue applies the gate: it is bound by reading mixed and gate, not by its arithmetic (row and vdim are a
// hundred or so).  A tile is 64 lanes of a head by 64 rows (a warp 16 rows), or, with few rows, by 16 (a warp 16 lanes);
// k goes through shared memory in pieces of 128, every load of a piece in flight at once, and the gate is asked for with
// the first piece.
#define LV_K 128
#define LV_PITCH (LV_K + 8)
template <bool FEW>
__global__ void __launch_bounds__(128)
latent_values_mma_kernel(const __nv_bfloat16* __restrict__ mixed, const __nv_bfloat16* __restrict__ w,
                         const float* __restrict__ gate, int ld, int g_at, int heads, int vdim, int row,
                         __nv_bfloat16* __restrict__ out, int n_rows) {
  constexpr int ROWS = FEW ? 16 : 64, TILES = FEW ? 2 : 8;      // TILES: pieces of 8 lanes a warp
  __shared__ __align__(16) __nv_bfloat16 a_s[ROWS][LV_PITCH];
  __shared__ __align__(16) __nv_bfloat16 w_s[64][LV_PITCH];
  const int t0 = blockIdx.x * ROWS, head = blockIdx.y, l0 = blockIdx.z * 64;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int row_in = FEW ? 0 : warp * 16, lane_in = FEW ? warp * 16 : 0;
  const __nv_bfloat16* wh = w + (size_t)head * vdim * row;
  auto copy16 = [](__nv_bfloat16* dst, const __nv_bfloat16* src, bool ok) {      // zeros where there is nothing
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src),
                 "r"(ok ? 16 : 0) : "memory");
  };
  auto stage_w = [&](int k0) {
    for (int i = threadIdx.x; i < 64 * (LV_K / 8); i += 128) {
      const int l = i / (LV_K / 8), k = (i % (LV_K / 8)) * 8;
      const bool ok = l0 + l < vdim && k0 + k < row;
      copy16(&w_s[l][k], ok ? wh + (size_t)(l0 + l) * row + k0 + k : wh, ok);
    }
  };
  auto stage_a = [&](int k0) {
    for (int i = threadIdx.x; i < ROWS * (LV_K / 8); i += 128) {
      const int m = i / (LV_K / 8), k = (i % (LV_K / 8)) * 8;
      const bool ok = t0 + m < n_rows && k0 + k < row;
      copy16(&a_s[m][k], ok ? mixed + ((size_t)(t0 + m) * heads + head) * row + k0 + k : mixed, ok);
    }
  };
  stage_w(0);                                 // weights are written by no kernel of the step
  pdl_wait();
  pdl_launch();
  stage_a(0);
  const int g = lane >> 2, q = lane & 3;
  const bool pairs = (vdim & 1) == 0 && (g_at & 1) == 0 && (ld & 1) == 0;
  float2 z[TILES][2];                         // the gate's numbers for this thread's results
#pragma unroll
  for (int j = 0; j < TILES; ++j)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = t0 + row_in + g + 8 * h, l = l0 + lane_in + 8 * j + 2 * q;
      z[j][h] = make_float2(0.f, 0.f);
      if (t >= n_rows || l >= vdim) continue;
      const float* from = gate + (size_t)t * ld + g_at + head * vdim + l;
      if (pairs) z[j][h] = *reinterpret_cast<const float2*>(from);
      else z[j][h] = make_float2(from[0], l + 1 < vdim ? from[1] : 0.f);
    }
  float acc[TILES][4];
#pragma unroll
  for (int j = 0; j < TILES; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  for (int k0 = 0; k0 < row; k0 += LV_K) {
    if (k0) {
      __syncthreads();                        // the piece before has been read
      stage_w(k0);
      stage_a(k0);
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    const int k_end = row - k0 < LV_K ? row - k0 : LV_K;      // rows come in whole 16s
#pragma unroll
    for (int k = 0; k < LV_K; k += 16) {
      if (k >= k_end) break;
      unsigned a[4];
      const unsigned from = (unsigned)__cvta_generic_to_shared(&a_s[row_in + (lane & 15)][k + (lane >> 4) * 8]);
      asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                   : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"(from));
#pragma unroll
      for (int j = 0; j < TILES; j += 2) {    // two pieces of 8 lanes a load
        unsigned b[4];
        const int l = lane_in + 8 * j + (lane & 7) + ((lane >> 4) << 3);
        const unsigned at = (unsigned)__cvta_generic_to_shared(&w_s[l][k + ((lane >> 3) & 1) * 8]);
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                     : "=r"(b[0]), "=r"(b[1]), "=r"(b[2]), "=r"(b[3]) : "r"(at));
#pragma unroll
        for (int h = 0; h < 2; ++h)
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                       : "+f"(acc[j + h][0]), "+f"(acc[j + h][1]), "+f"(acc[j + h][2]), "+f"(acc[j + h][3])
                       : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[2 * h]), "r"(b[2 * h + 1]));
      }
    }
  }
#pragma unroll
  for (int j = 0; j < TILES; ++j)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = t0 + row_in + g + 8 * h, l = l0 + lane_in + 8 * j + 2 * q;
      if (t >= n_rows || l >= vdim) continue;
      __nv_bfloat16* o = out + ((size_t)t * heads + head) * vdim + l;
      const float v0 = acc[j][2 * h] / (1.0f + expf(-z[j][h].x)), v1 = acc[j][2 * h + 1] / (1.0f + expf(-z[j][h].y));
      if ((vdim & 1) == 0) {
        *reinterpret_cast<__nv_bfloat162*>(o) = __floats2bfloat162_rn(v0, v1);
      } else {
        o[0] = __float2bfloat16_rn(v0);
        if (l + 1 < vdim) o[1] = __float2bfloat16_rn(v1);
      }
    }
}

// The 32-bit form (w [heads, row, vdim]: neighbouring threads on neighbouring lanes), k in index order: a block a
// (row, head), the weighted latent in shared memory.
__global__ void __launch_bounds__(128)
latent_values_f32_kernel(const float* __restrict__ mixed, const float* __restrict__ w, const float* __restrict__ gate,
                         int ld, int g_at, int heads, int vdim, int row, float* __restrict__ out) {
  extern __shared__ float latent_s[];
  const int t = blockIdx.x, head = blockIdx.y;
  pdl_wait();
  pdl_launch();
  const float* in = mixed + ((size_t)t * heads + head) * row;
  for (int c = threadIdx.x; c < row; c += blockDim.x) latent_s[c] = in[c];
  __syncthreads();
  const float* wh = w + (size_t)head * row * vdim;
  for (int l = threadIdx.x; l < vdim; l += blockDim.x) {
    float sum = 0.f;
    for (int c = 0; c < row; ++c) sum = fmaf(wh[(size_t)c * vdim + l], latent_s[c], sum);
    out[((size_t)t * heads + head) * vdim + l] = sum / (1.0f + expf(-gate[(size_t)t * ld + g_at + head * vdim + l]));
  }
}

// w: [heads, vdim, row] in bfloat16, [heads, row, vdim] in float32.
TOKB200_API int tokb200_latent_values(const void* mixed, const void* w, const float* gate, int ld, int g_at, int heads,
                                      int vdim, int row, void* out, int dtype, int n_rows, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (heads <= 0 || heads > 65535 || vdim <= 0 || row <= 0 || row > 8192 || g_at + heads * vdim > ld) return TOKB200_BAD_SIZE;
  if (dtype == TOKB200_F32)
    return launch_dependent(latent_values_f32_kernel, dim3(n_rows, heads), dim3(vdim <= 32 ? 32 : vdim <= 64 ? 64 : 128),
                            (size_t)row * sizeof(float), stream, (const float*)mixed, (const float*)w, gate, ld, g_at, heads,
                            vdim, row, (float*)out);
  if (dtype != TOKB200_BF16) return TOKB200_BAD_DTYPE;
  if (row % 16 || (((uintptr_t)mixed | (uintptr_t)w) & 15) || ((uintptr_t)out & 3) || ((uintptr_t)gate & 7)) return TOKB200_BAD_ALIGNMENT;
  const bool few = n_rows <= 64;
  const dim3 grid((n_rows + (few ? 15 : 63)) / (few ? 16 : 64), heads, (vdim + 63) / 64);
#define LAUNCH(FEW)                                                                                              \
  return launch_dependent(latent_values_mma_kernel<FEW>, grid, dim3(128), 0, stream, (const __nv_bfloat16*)mixed, \
                          (const __nv_bfloat16*)w, gate, ld, g_at, heads, vdim, row, (__nv_bfloat16*)out, n_rows)
  if (few) LAUNCH(true);
  LAUNCH(false);
#undef LAUNCH
}
