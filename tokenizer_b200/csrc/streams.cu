// Several residual streams side by side, float32 [T, streams, H], and the step between two sublayers:
//
//   streams_step   what is pending:  x_t <- sum_s mix[s, t] x_s + share[t] y     (all streams at once, from the old ones)
//                  what comes next:  u = sum_s read[s] x_s of the new streams, and out = u / sqrt(mean(u^2) + eps) * gain
//
// y is a sublayer's output: [T, H] in float32 or bfloat16, or float32 partial sums [S, T, H] of a product cut along k,
// added in index order.  Before the first sublayer's output is added the streams are equal and x is one of them,
// [T, H]: every stream reads it, and the kernel writes the streams to `x_out`.  Without y nothing is written.  Without
// gain, out is u itself.  `rows`: only those rows are read, and nothing is written but out (dense).  Everything is
// 32-bit but y and out.  A block a row; an element's streams lie in one thread.
#include "common.cuh"

#define ST_MAX 8
#define ST_PLANES 4
#define ST_CHUNKS 2            // pieces of a row whose u stays in registers between the sum and the scaling

struct StArgs {
  const float* x;
  long long x_row, x_stream;   // elements between rows and between streams (0: one stream that stands for all)
  float* x_out;                // [T, streams, H]; may be x
  const void* y;
  int y_bf16, y_partials;
  long long y_stride;
  const float* mix;            // [streams, streams], from the row to the column
  const float* share;          // [streams]
  const float* read;           // [streams], or null: all one
  const float* gain;           // [H], or null
  float eps;
  const int* rows;
  int n_rows, hidden;
};

template <int V> struct StVec { float v[V]; };
template <int V>
__device__ __forceinline__ StVec<V> st_load(const float* p) {
  StVec<V> o;
  if (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    o.v[0] = a.x; o.v[1 % V] = a.y; o.v[2 % V] = a.z; o.v[3 % V] = a.w;
  } else {
    o.v[0] = *p;
  }
  return o;
}
template <int V>
__device__ __forceinline__ StVec<V> st_load(const __nv_bfloat16* p) {
  StVec<V> o;
  if (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
    const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
    o.v[0] = a.x; o.v[1 % V] = a.y; o.v[2 % V] = b.x; o.v[3 % V] = b.y;
  } else {
    o.v[0] = __bfloat162float(*p);
  }
  return o;
}
template <int V>
__device__ __forceinline__ void st_store(float* p, const StVec<V>& a) {
  if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1 % V], a.v[2 % V], a.v[3 % V]);
  else *p = a.v[0];
}
template <int V>
__device__ __forceinline__ void st_store(__nv_bfloat16* p, const StVec<V>& a) {
  if (V == 4) {
    __nv_bfloat162 h[2] = {__floats2bfloat162_rn(a.v[0], a.v[1 % V]), __floats2bfloat162_rn(a.v[2 % V], a.v[3 % V])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(h);
  } else {
    *p = __float2bfloat16_rn(a.v[0]);
  }
}

// CUT: y comes as partial sums, of which a few planes are asked for at once (steps of few rows; a whole y keeps the
// registers that those take for more blocks a multiprocessor).
template <int STREAMS, int V, bool CUT, typename TO>
__global__ void __launch_bounds__(512) streams_step_kernel(const StArgs a, TO* __restrict__ out) {
  __shared__ float scratch[33];
  // the weights are written by no kernel of the step: asked for before the wait on the predecessor
  float mix[STREAMS][STREAMS], share[STREAMS], read[STREAMS];
#pragma unroll
  for (int s = 0; s < STREAMS; ++s) {
    read[s] = a.read ? a.read[s] : 1.f;
    share[s] = a.y ? a.share[s] : 0.f;
#pragma unroll
    for (int t = 0; t < STREAMS; ++t) mix[s][t] = a.y ? a.mix[s * STREAMS + t] : 0.f;
  }
  const int item = blockIdx.x;
  pdl_wait();
  pdl_launch();
  const int t = a.rows ? a.rows[item] : item;
  const float* x = a.x + (size_t)t * a.x_row;
  const int H = a.hidden, step = blockDim.x * V;
  // one place of the row: the new streams (written back where they stay) and their weighted sum
  auto place = [&](int i) {
    StVec<V> old[STREAMS];
#pragma unroll
    for (int s = 0; s < STREAMS; ++s)
      old[s] = (s > 0 && a.x_stream == 0) ? old[0] : st_load<V>(x + (size_t)s * a.x_stream + i);
    StVec<V> u;
#pragma unroll
    for (int e = 0; e < V; ++e) u.v[e] = 0.f;
    if (a.y) {
      StVec<V> y;
      if (a.y_bf16) {
        y = st_load<V>((const __nv_bfloat16*)a.y + (size_t)t * H + i);
      } else {
        y = st_load<V>((const float*)a.y + (size_t)t * H + i);
        for (int k = 1; CUT && k < a.y_partials; k += ST_PLANES) {      // a few planes asked for at once, added in index order
          StVec<V> part[ST_PLANES];
#pragma unroll
          for (int d = 0; d < ST_PLANES; ++d)
            if (k + d < a.y_partials) part[d] = st_load<V>((const float*)a.y + (size_t)(k + d) * a.y_stride + (size_t)t * H + i);
#pragma unroll
          for (int d = 0; d < ST_PLANES; ++d) {
            if (k + d >= a.y_partials) continue;
#pragma unroll
            for (int e = 0; e < V; ++e) y.v[e] += part[d].v[e];
          }
        }
      }
#pragma unroll
      for (int to = 0; to < STREAMS; ++to) {
        StVec<V> now;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          float sum = mix[0][to] * old[0].v[e];
#pragma unroll
          for (int s = 1; s < STREAMS; ++s) sum = fmaf(mix[s][to], old[s].v[e], sum);
          now.v[e] = fmaf(share[to], y.v[e], sum);
          u.v[e] = fmaf(read[to], now.v[e], u.v[e]);
        }
        if (a.x_out) st_store<V>(a.x_out + ((size_t)t * STREAMS + to) * H + i, now);
      }
    } else {
#pragma unroll
      for (int s = 0; s < STREAMS; ++s)
#pragma unroll
        for (int e = 0; e < V; ++e) u.v[e] = fmaf(read[s], old[s].v[e], u.v[e]);
    }
    return u;
  };
  TO* o = out ? out + (size_t)item * H : nullptr;
  StVec<V> kept[ST_CHUNKS];
  float squares = 0.f;
#pragma unroll
  for (int c = 0; c < ST_CHUNKS; ++c) {
    const int i = threadIdx.x * V + c * step;
    if (i < H) {
      kept[c] = place(i);
#pragma unroll
      for (int e = 0; e < V; ++e) squares = fmaf(kept[c].v[e], kept[c].v[e], squares);
    }
  }
  // a row longer than the registers hold: without a gain its u goes straight out, else it is summed up again below
  // from the streams this thread has just written
  for (int i = threadIdx.x * V + ST_CHUNKS * step; i < H; i += step) {
    const StVec<V> u = place(i);
#pragma unroll
    for (int e = 0; e < V; ++e) squares = fmaf(u.v[e], u.v[e], squares);
    if (a.gain == nullptr && o) st_store<V>(o + i, u);
  }
  if (o == nullptr) return;
  const float inv = a.gain ? 1.0f / sqrtf(block_sum(squares, scratch) / (float)H + a.eps) : 1.f;
#pragma unroll
  for (int c = 0; c < ST_CHUNKS; ++c) {
    const int i = threadIdx.x * V + c * step;
    if (i < H) {
      if (a.gain) {
        const StVec<V> g = st_load<V>(a.gain + i);
#pragma unroll
        for (int e = 0; e < V; ++e) kept[c].v[e] = kept[c].v[e] * inv * g.v[e];
      }
      st_store<V>(o + i, kept[c]);
    }
  }
  if (a.gain == nullptr) return;
  for (int i = threadIdx.x * V + ST_CHUNKS * step; i < H; i += step) {
    StVec<V> u;
#pragma unroll
    for (int e = 0; e < V; ++e) u.v[e] = 0.f;
    if (a.y && a.x_out) {
#pragma unroll
      for (int s = 0; s < STREAMS; ++s) {
        const StVec<V> now = st_load<V>(a.x_out + ((size_t)t * STREAMS + s) * H + i);
#pragma unroll
        for (int e = 0; e < V; ++e) u.v[e] = fmaf(read[s], now.v[e], u.v[e]);
      }
    } else {
      u = place(i);
    }
    const StVec<V> g = st_load<V>(a.gain + i);
#pragma unroll
    for (int e = 0; e < V; ++e) u.v[e] = u.v[e] * inv * g.v[e];
    st_store<V>(o + i, u);
  }
}

template <int STREAMS, typename TO>
static int st_launch(const StArgs& a, void* out, bool quads, cudaStream_t stream) {
  const int items = quads ? a.hidden / 4 : a.hidden;
  int threads = (items + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  const dim3 grid(a.n_rows), block(threads);
  if (quads && a.y && a.y_partials > 1)
    return launch_dependent(streams_step_kernel<STREAMS, 4, true, TO>, grid, block, 0, stream, a, (TO*)out);
  if (quads) return launch_dependent(streams_step_kernel<STREAMS, 4, false, TO>, grid, block, 0, stream, a, (TO*)out);
  return launch_dependent(streams_step_kernel<STREAMS, 1, true, TO>, grid, block, 0, stream, a, (TO*)out);
}

// x: [T, H] (`equal` not 0: all streams are this one) or [T, streams, H].  y, x_out, read, gain, out and rows may be null
// (x_out must not with y and without rows).
TOKB200_API int tokb200_streams_step(const float* x, int equal, float* x_out, int streams, const void* y, int y_dtype,
                                     int y_partials, long long y_stride, const float* mix, const float* share,
                                     const float* read, const float* gain, float eps, void* out, int out_dtype,
                                     const int* rows, int n_rows, int hidden, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (hidden <= 0 || streams < 1 || streams > ST_MAX || (y && (y_partials < 1 || mix == nullptr || share == nullptr)) ||
      (y && rows == nullptr && x_out == nullptr) || (rows && x_out) || (gain && out == nullptr))
    return TOKB200_BAD_SIZE;
  if (y && y_dtype == TOKB200_BF16 && y_partials != 1) return TOKB200_BAD_DTYPE;
  StArgs a = {x, equal ? (long long)hidden : (long long)streams * hidden, equal ? 0 : (long long)hidden, x_out, y,
              y_dtype == TOKB200_BF16, y_partials, y_stride, mix, share, read, gain, eps, rows, n_rows, hidden};
  const uintptr_t all = (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)y | (uintptr_t)gain | (uintptr_t)out;
  const bool quads = hidden % 4 == 0 && (all & 15) == 0 && y_stride % 4 == 0;
  const bool bf16 = out != nullptr && out_dtype == TOKB200_BF16;
#define CASE(S) \
  case S: return bf16 ? st_launch<S, __nv_bfloat16>(a, out, quads, stream) : st_launch<S, float>(a, out, quads, stream);
  switch (streams) {
    CASE(1) CASE(2) CASE(3) CASE(4) CASE(5) CASE(6) CASE(7) CASE(8)
  }
#undef CASE
  return TOKB200_BAD_SIZE;
}
