// The matrix memory with exponential gates (see mlstm.cu) over prompt portions, in chunks of 64 tokens on tensor cores.
//
// With the running maximum m known for every token the recurrence is linear, so a chunk's outputs and its contribution to
// the state are products of matrices.  F_t is the sum of the logarithms of the forget gates from the chunk's start to
// token t, m_0 the maximum in front of the chunk:
//     A_t = F_t - m_t,  G_s = i_s - F_s,  D[t][s] = exp(A_t + G_s) for s <= t (never above one)
//     S^T q of token t:  exp(A_t + m_0) S_0^T q_t + sum_s D[t][s] (k_s . q_t) v_s;      n . q alike with v = 1
//     the chunk's end:   exp(A_L + m_0) S_0 + sum_s exp(A_L + G_s) k_s v_s^T
//
//   mlstm_chunk_states   sum_s exp(A_L + G_s) k_s v_s^T of every chunk and head from zero, side by side
//   mlstm_chunk_carry    what is in front of every chunk: the sums carried on from chunk to chunk, element by element;
//                        the last goes to the request's slot
//   mlstm_chunk_outputs  the outputs with everything behind them (normaliser, root mean square, gain, gate)
//
// q, k and v, the projections, are bfloat16 operands.  Everything else that meets them in a product is 32-bit: the state,
// the weighted keys and the weights of the scores are taken as three bfloat16 pieces each (8 + 8 + 8 bits of the
// mantissa), so that a product of a piece and a bfloat16 number is exact and only the 32-bit sums round.  F, A and G are
// formed in 64-bit and handed over as pairs of 32-bit numbers (hundreds of closed gates cancel inside a chunk).
// Heads of up to 128 lanes and 128 values; chunks are counted from a portion's start, so another cut rounds
// differently and does nothing else.
#include "common.cuh"

#define MC_L 64                 // tokens a chunk
#define MC_PITCH 136            // elements between rows in shared memory: 16 bytes off whole 128s
#define MC_EPS 1e-6f

struct McArgs {
  const float* proj;            // [T, ld]: q, k, v and the gate at their columns
  int ld, q_at, k_at, v_at, g_at;
  int heads, dim, vdim;
  float scale;
  const float* log_f;           // [heads, gate_ld]: logarithms of the forget and input gates, the running maxima
  const float* log_i;
  const float* top;
  long long gate_ld;
  const float* start;           // [requests, heads]: the maxima in front of the step's rows
  const int* q_start;
  const int* state_slot;
  int n_requests;
  float* state;                 // [slots, stride], a slot starts with [heads, vdim + 1, dim]
  long long stride;
  float* sums;                  // [chunks, heads, vdim + 1, dim]
  float* decay;                 // [chunks, heads]
  const float* gain;            // [heads * vdim]
  float eps;
  __nv_bfloat16* out;           // [T, heads * vdim]
  int quads;                    // rows and columns come in whole 4s on 16 bytes
};

// Chunk c of request r has the place q_start[r] / 64 + r + c: distinct, without a list.
__device__ __forceinline__ int mc_base(const McArgs& a, int r) { return a.q_start[r] / MC_L + r; }

struct McChunk {
  int request, first, rows, index;      // request -1: nothing here
};

// Which chunk a place holds (every thread of the block asks).
__device__ __forceinline__ McChunk mc_find(const McArgs& a, int place, int* found) {
  if (threadIdx.x == 0) *found = -1;
  __syncthreads();
  for (int r = threadIdx.x; r < a.n_requests; r += blockDim.x) {
    const int c = place - mc_base(a, r), n = a.q_start[r + 1] - a.q_start[r];
    if (c >= 0 && c * MC_L < n) *found = r;
  }
  __syncthreads();
  McChunk m = {*found, 0, 0, 0};
  if (m.request >= 0) {
    const int n = a.q_start[m.request + 1] - a.q_start[m.request];
    m.index = place - mc_base(a, m.request);
    m.first = a.q_start[m.request] + m.index * MC_L;
    m.rows = n - m.index * MC_L < MC_L ? n - m.index * MC_L : MC_L;
  }
  return m;
}

// A sum of two 32-bit numbers that stands for one of more digits.
struct McPair {
  float hi, lo;
};
__device__ __forceinline__ McPair mc_pair(double v) {
  const float hi = (float)v;
  return {hi, (float)(v - (double)hi)};
}
__device__ __forceinline__ float mc_exp(McPair a, McPair b) { return expf((a.hi + b.hi) + (a.lo + b.lo)); }

// A and G of a chunk's tokens into shared memory, by the first warp: lane l has tokens 2l and 2l + 1.  Rows behind the
// chunk's end repeat nothing: their G is minus infinity (no weight).
__device__ __forceinline__ void mc_gates(const McArgs& a, const McChunk& m, int head, McPair* A, McPair* G) {
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x;
  const size_t at = (size_t)head * a.gate_ld + m.first;
  double f[2];
  float top[2], in[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const bool on = 2 * lane + e < m.rows;
    f[e] = on ? (double)a.log_f[at + 2 * lane + e] : 0.0;
    top[e] = on ? a.top[at + 2 * lane + e] : 0.f;
    in[e] = on ? a.log_i[at + 2 * lane + e] : 0.f;
  }
  f[1] += f[0];
  double sum = f[1];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double before = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += before;
  }
  const double base = sum - f[1];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int t = 2 * lane + e;
    const double F = base + f[e];
    A[t] = {0.f, 0.f};
    G[t] = {-INFINITY, 0.f};
    if (t < m.rows) {
      A[t] = mc_pair(F - (double)top[e]);
      G[t] = mc_pair((double)in[e] - F);
    }
  }
}

__device__ __forceinline__ float mc_before(const McArgs& a, const McChunk& m, int head) {
  return m.index ? a.top[(size_t)head * a.gate_ld + m.first - 1] : a.start[m.request * a.heads + head];
}

__device__ __forceinline__ void mc_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mc_ldmatrix(unsigned (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((unsigned)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mc_ldmatrix_trans(unsigned (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((unsigned)__cvta_generic_to_shared(p)));
}

// Lane addresses of a 16 x 16 piece for one ldmatrix: of an A operand stored as it is or transposed, and of two B
// operands of 8 columns stored by columns (k runs inside a row) or by rows.
__device__ __forceinline__ const __nv_bfloat16* mc_a(const __nv_bfloat16* s, int row0, int k0, int lane) {
  return s + (row0 + (lane & 15)) * MC_PITCH + k0 + (lane >> 4) * 8;
}
__device__ __forceinline__ const __nv_bfloat16* mc_a_trans(const __nv_bfloat16* s, int row0, int k0, int lane) {
  return s + (k0 + (lane & 7) + (lane >> 4) * 8) * MC_PITCH + row0 + ((lane >> 3) & 1) * 8;
}
__device__ __forceinline__ const __nv_bfloat16* mc_b(const __nv_bfloat16* s, int n0, int k0, int lane) {
  return s + (n0 + (lane & 7) + (lane >> 4) * 8) * MC_PITCH + k0 + ((lane >> 3) & 1) * 8;
}
__device__ __forceinline__ const __nv_bfloat16* mc_b_trans(const __nv_bfloat16* s, int n0, int k0, int lane) {
  return s + (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * MC_PITCH + n0 + (lane >> 4) * 8;
}

// x in three bfloat16 pieces that add up to it.
__device__ __forceinline__ void mc_split(float x, __nv_bfloat16 (&piece)[3]) {
  piece[0] = __float2bfloat16_rn(x);
  const float rest = x - __bfloat162float(piece[0]);
  piece[1] = __float2bfloat16_rn(rest);
  piece[2] = __float2bfloat16_rn(rest - __bfloat162float(piece[1]));
}
__device__ __forceinline__ unsigned mc_two(__nv_bfloat16 a, __nv_bfloat16 b) {
  const __nv_bfloat162 v = __halves2bfloat162(a, b);
  return *reinterpret_cast<const unsigned*>(&v);
}

// Four lanes of a row of the product from column `col` on, zero from `lanes` on.
__device__ __forceinline__ float4 mc_load4(const McArgs& a, size_t row, int col, int l, int lanes, bool on) {
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (!on || l >= lanes) return v;
  const float* p = a.proj + row * a.ld + col + l;
  if (a.quads) return *reinterpret_cast<const float4*>(p);
  v.x = p[0];
  if (l + 1 < lanes) v.y = p[1];
  if (l + 2 < lanes) v.z = p[2];
  if (l + 3 < lanes) v.w = p[3];
  return v;
}
__device__ __forceinline__ void mc_store4(__nv_bfloat16* p, __nv_bfloat16 a, __nv_bfloat16 b, __nv_bfloat16 c, __nv_bfloat16 d) {
  *reinterpret_cast<uint2*>(p) = make_uint2(mc_two(a, b), mc_two(c, d));
}

// A block of 256 threads holds a chunk's rows of one head's columns: thread (warp w, lane l) has lanes 4l .. 4l + 3 of the
// tokens w, w + 8 ...  All of them are asked for before the first is used.
#define MC_EACH (MC_L / 8)
__device__ __forceinline__ void mc_fetch(const McArgs& a, const McChunk& m, int col, int lanes, float4 (&v)[MC_EACH]) {
#pragma unroll
  for (int j = 0; j < MC_EACH; ++j) {
    const int t = (threadIdx.x >> 5) + 8 * j;
    v[j] = mc_load4(a, (size_t)m.first + t, col, (threadIdx.x & 31) * 4, lanes, t < m.rows);
  }
}
// As bfloat16 rows in shared memory, in whole 16s of lanes, zeros behind.
__device__ __forceinline__ void mc_keep(const float4 (&v)[MC_EACH], int lanes, __nv_bfloat16* to) {
  const int l = (threadIdx.x & 31) * 4;
  if (l >= ((lanes + 15) & ~15)) return;
#pragma unroll
  for (int j = 0; j < MC_EACH; ++j)
    mc_store4(to + ((threadIdx.x >> 5) + 8 * j) * MC_PITCH + l, __float2bfloat16_rn(v[j].x), __float2bfloat16_rn(v[j].y),
              __float2bfloat16_rn(v[j].z), __float2bfloat16_rn(v[j].w));
}

// ---- a chunk's contribution to the state ----
#define MC_STATE_THREADS 256
static constexpr size_t MC_STATE_SMEM = (size_t)4 * MC_L * MC_PITCH * 2;
__global__ void __launch_bounds__(MC_STATE_THREADS) mlstm_chunk_states_kernel(const McArgs a) {
  extern __shared__ __align__(16) __nv_bfloat16 mc_raw[];
  __nv_bfloat16* v_s = mc_raw;                          // [token][value]
  __nv_bfloat16* k_s = v_s + MC_L * MC_PITCH;           // three pieces of the weighted keys, [token][lane]
  __shared__ McPair A[MC_L], G[MC_L];
  __shared__ int found;
  const int head = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  pdl_launch();
  const McChunk m = mc_find(a, blockIdx.x, &found);
  if (m.request < 0) return;
  float4 v[MC_EACH], keys[MC_EACH];
  mc_fetch(a, m, a.v_at + head * a.vdim, a.vdim, v);
  mc_fetch(a, m, a.k_at + head * a.dim, a.dim, keys);
  mc_gates(a, m, head, A, G);
  mc_keep(v, a.vdim, v_s);
  __syncthreads();
  const McPair end = A[m.rows - 1];
  const int dk = (a.dim + 15) / 16, dv = (a.vdim + 15) / 16;
  if (lane * 4 < dk * 16) {
#pragma unroll
    for (int j = 0; j < MC_EACH; ++j) {
      const int t = warp + 8 * j;
      const float w = mc_exp(end, G[t]);
      const float x[4] = {keys[j].x, keys[j].y, keys[j].z, keys[j].w};
      __nv_bfloat16 piece[4][3];
#pragma unroll
      for (int e = 0; e < 4; ++e) mc_split(w * __bfloat162float(__float2bfloat16_rn(x[e])), piece[e]);
#pragma unroll
      for (int p = 0; p < 3; ++p)
        mc_store4(k_s + (p * MC_L + t) * MC_PITCH + lane * 4, piece[0][p], piece[1][p], piece[2][p], piece[3][p]);
    }
  }
  __syncthreads();
  const size_t cell = (size_t)blockIdx.x * a.heads + head;
  float* sums = a.sums + cell * (a.vdim + 1) * a.dim;
  if (threadIdx.x == 0) a.decay[cell] = mc_exp(end, {mc_before(a, m, head), 0.f});
  if ((int)threadIdx.x < a.dim) {                       // the normaliser's sum: the weighted keys themselves
    float sum = 0.f;
#pragma unroll 8
    for (int t = 0; t < MC_L; ++t) {                    // (rows behind the chunk's end are zeros)
      float k = 0.f;
#pragma unroll
      for (int p = 2; p >= 0; --p) k += __bfloat162float(k_s[(p * MC_L + t) * MC_PITCH + threadIdx.x]);
      sum += k;
    }
    sums[(size_t)a.vdim * a.dim + threadIdx.x] = sum;
  }
  // a warp 16 lanes of the keys: its operands stay in registers while it walks the values
  for (int n = warp; n < dk; n += MC_STATE_THREADS / 32) {
    unsigned b[MC_L / 16][3][4];
#pragma unroll
    for (int k = 0; k < MC_L / 16; ++k)
#pragma unroll
      for (int p = 0; p < 3; ++p) mc_ldmatrix_trans(b[k][p], mc_b_trans(k_s + p * MC_L * MC_PITCH, n * 16, k * 16, lane));
    for (int r = 0; r < dv; ++r) {
      float acc[2][4] = {};
#pragma unroll
      for (int k = 0; k < MC_L / 16; ++k) {
        unsigned v[4];
        mc_ldmatrix_trans(v, mc_a_trans(v_s, r * 16, k * 16, lane));
#pragma unroll
        for (int p = 0; p < 3; ++p) {
          mc_mma(acc[0], v, b[k][p][0], b[k][p][1]);
          mc_mma(acc[1], v, b[k][p][2], b[k][p][3]);
        }
      }
      const int g = lane >> 2, q = lane & 3;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int row = r * 16 + g + 8 * h, col = n * 16 + 8 * j + 2 * q;
          if (row >= a.vdim || col >= a.dim) continue;
          float* to = sums + (size_t)row * a.dim + col;
          if ((a.dim & 1) == 0) *reinterpret_cast<float2*>(to) = make_float2(acc[j][2 * h], acc[j][2 * h + 1]);
          else {
            to[0] = acc[j][2 * h];
            if (col + 1 < a.dim) to[1] = acc[j][2 * h + 1];
          }
        }
    }
  }
}

// ---- what is in front of every chunk ----
template <int V>
__global__ void __launch_bounds__(256) mlstm_chunk_carry_kernel(const McArgs a) {
  const int head = blockIdx.y, r = blockIdx.z;
  const int size = (a.vdim + 1) * a.dim, i = (blockIdx.x * 256 + threadIdx.x) * V;
  pdl_wait();
  pdl_launch();
  const int n = a.q_start[r + 1] - a.q_start[r];
  if (n <= 0 || i >= size) return;
  const int base = mc_base(a, r), chunks = (n + MC_L - 1) / MC_L;
  float* slot = a.state + (size_t)a.state_slot[r] * a.stride + (size_t)head * size + i;
  const size_t step = (size_t)a.heads * size;
  float* at = a.sums + ((size_t)base * a.heads + head) * size + i;
  const float* decay = a.decay + (size_t)base * a.heads + head;
  constexpr int DEEP = 8;                                // chunks asked for at once, one batch ahead
  float sum[2][DEEP][V], d[2][DEEP];
  auto fetch = [&](int c, int which) {
#pragma unroll
    for (int k = 0; k < DEEP; ++k) {
      if (c + k >= chunks) continue;
      d[which][k] = decay[(size_t)(c + k) * a.heads];
      const float* from = at + (c + k) * step;
      if (V == 2) {
        const float2 v = *reinterpret_cast<const float2*>(from);
        sum[which][k][0] = v.x; sum[which][k][1 % V] = v.y;
      } else {
        sum[which][k][0] = *from;
      }
    }
  };
  fetch(0, 0);
  float S[V];
#pragma unroll
  for (int e = 0; e < V; ++e) S[e] = slot[e];
  auto walk = [&](int c, int which) {
#pragma unroll
    for (int k = 0; k < DEEP; ++k) {
      if (c + k >= chunks) continue;
      float* to = at + (c + k) * step;
      if (V == 2) *reinterpret_cast<float2*>(to) = make_float2(S[0], S[1 % V]);
      else *to = S[0];
#pragma unroll
      for (int e = 0; e < V; ++e) S[e] = fmaf(d[which][k], S[e], sum[which][k][e]);
    }
  };
  for (int c = 0; c < chunks; c += 2 * DEEP) {
    fetch(c + DEEP, 1);
    walk(c, 0);
    fetch(c + 2 * DEEP, 0);
    walk(c + DEEP, 1);
  }
#pragma unroll
  for (int e = 0; e < V; ++e) slot[e] = S[e];
}

// ---- the outputs ----
// Eight warps: warp w has the chunk's token rows 16 (w mod 4) .. and one half of the values, in pieces of 16 lanes.
#define MC_OUT_THREADS 256
#define MC_OUT_TILES 4          // pieces of 16 values a warp, at most
static constexpr size_t MC_OUT_SMEM = (size_t)(3 * MC_L + 3 * 32) * MC_PITCH * 2;
__global__ void __launch_bounds__(MC_OUT_THREADS, 2) mlstm_chunk_outputs_kernel(const McArgs a) {
  extern __shared__ __align__(16) __nv_bfloat16 mc_raw[];
  __nv_bfloat16* q_s = mc_raw;
  __nv_bfloat16* k_s = q_s + MC_L * MC_PITCH;
  __nv_bfloat16* v_s = k_s + MC_L * MC_PITCH;
  __nv_bfloat16* S_s = v_s + MC_L * MC_PITCH;           // three pieces of 32 columns of S: 16 of either half
  __shared__ McPair A[MC_L], G[MC_L];
  __shared__ float norm_s[128], den_s[MC_L], squares_s[2][MC_L];
  __shared__ int found;
  const int head = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int rt = warp & 3, half = warp >> 2, g = lane >> 2, q = lane & 3;
  pdl_wait();
  pdl_launch();
  const McChunk m = mc_find(a, blockIdx.x, &found);
  if (m.request < 0) return;
  const int dk = (a.dim + 15) / 16, dv = (a.vdim + 15) / 16, first_half = (dv + 1) / 2;
  const int my_first = half ? first_half : 0, my_tiles = half ? dv - first_half : first_half;
  const float* S0 = a.sums + ((size_t)blockIdx.x * a.heads + head) * (a.vdim + 1) * a.dim;
  // a piece of 32 columns of S: thread (warp w, lane l) has lanes 4l .. 4l + 3 of the columns w, w + 8 ..
  const bool whole4 = (a.dim & 3) == 0;
  float4 column[4];
  auto fetch_columns = [&](int j) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = warp + 8 * e, l = lane * 4, row = r < 16 ? j * 16 + r : (first_half + j) * 16 + r - 16;
      column[e] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (row >= a.vdim || l >= a.dim) continue;
      const float* from = S0 + (size_t)row * a.dim + l;
      if (whole4) {
        column[e] = *reinterpret_cast<const float4*>(from);
      } else {
        column[e].x = from[0];
        if (l + 1 < a.dim) column[e].y = from[1];
        if (l + 2 < a.dim) column[e].z = from[2];
        if (l + 3 < a.dim) column[e].w = from[3];
      }
    }
  };
  {
    float4 rows[MC_EACH];
    mc_fetch(a, m, a.q_at + head * a.dim, a.dim, rows);
    fetch_columns(0);
    mc_gates(a, m, head, A, G);
    mc_keep(rows, a.dim, q_s);
    mc_fetch(a, m, a.k_at + head * a.dim, a.dim, rows);
    mc_keep(rows, a.dim, k_s);
    mc_fetch(a, m, a.v_at + head * a.vdim, a.vdim, rows);
    mc_keep(rows, a.vdim, v_s);
  }
  if (threadIdx.x < 128) norm_s[threadIdx.x] = (int)threadIdx.x < a.dim ? S0[(size_t)a.vdim * a.dim + threadIdx.x] : 0.f;
  const float m0 = mc_before(a, m, head);
  // ---- S_0^T q ----
  float acc[MC_OUT_TILES][2][4];
#pragma unroll
  for (int j = 0; j < MC_OUT_TILES; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][0][e] = acc[j][1][e] = 0.f;
#pragma unroll
  for (int j = 0; j < MC_OUT_TILES; ++j) {
    if (j >= first_half) break;
    if (j) __syncthreads();                             // the pieces before have been read
    if (lane * 4 < dk * 16) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float x[4] = {column[e].x, column[e].y, column[e].z, column[e].w};
        __nv_bfloat16 piece[4][3];
#pragma unroll
        for (int c = 0; c < 4; ++c) mc_split(x[c], piece[c]);
#pragma unroll
        for (int p = 0; p < 3; ++p)
          mc_store4(S_s + (p * 32 + warp + 8 * e) * MC_PITCH + lane * 4, piece[0][p], piece[1][p], piece[2][p], piece[3][p]);
      }
    }
    if (j + 1 < first_half) fetch_columns(j + 1);
    __syncthreads();
    if (j < my_tiles) {
      for (int k = 0; k < dk; ++k) {
        unsigned aq[4];
        mc_ldmatrix(aq, mc_a(q_s, rt * 16, k * 16, lane));
#pragma unroll
        for (int p = 0; p < 3; ++p) {
          unsigned b[4];
          mc_ldmatrix(b, mc_b(S_s + p * 32 * MC_PITCH, half * 16, k * 16, lane));
          mc_mma(acc[j][0], aq, b[0], b[1]);
          mc_mma(acc[j][1], aq, b[2], b[3]);
        }
      }
    }
  }
  // ---- n_0 . q: four threads a token ----
  {
    const int t = threadIdx.x >> 2;
    float sum = 0.f;
    for (int l = threadIdx.x & 3; l < a.dim; l += 4) sum = fmaf(norm_s[l], __bfloat162float(q_s[t * MC_PITCH + l]), sum);
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    if ((threadIdx.x & 3) == 0) den_s[t] = sum;
  }
  const int t_lo = rt * 16 + g, t_hi = t_lo + 8;
  const McPair a_lo = A[t_lo], a_hi = A[t_hi], from0 = {m0, 0.f};
  const float w_lo = mc_exp(a_lo, from0) * a.scale, w_hi = mc_exp(a_hi, from0) * a.scale;
#pragma unroll
  for (int j = 0; j < MC_OUT_TILES; ++j)
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      acc[j][n][0] *= w_lo; acc[j][n][1] *= w_lo;
      acc[j][n][2] *= w_hi; acc[j][n][3] *= w_hi;
    }
  // ---- the chunk's own keys, 16 at a time, up to this warp's rows ----
  float own_lo = 0.f, own_hi = 0.f;
  for (int st = 0; st <= rt; ++st) {
    float score[2][4] = {};
    for (int k = 0; k < dk; ++k) {
      unsigned aq[4], b[4];
      mc_ldmatrix(aq, mc_a(q_s, rt * 16, k * 16, lane));
      mc_ldmatrix(b, mc_b(k_s, st * 16, k * 16, lane));
      mc_mma(score[0], aq, b[0], b[1]);
      mc_mma(score[1], aq, b[2], b[3]);
    }
    unsigned w[3][4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int s = st * 16 + 8 * n + 2 * q;
      const McPair g0 = G[s], g1 = G[s + 1];
      const float p0 = s <= t_lo ? mc_exp(a_lo, g0) * (score[n][0] * a.scale) : 0.f;
      const float p1 = s + 1 <= t_lo ? mc_exp(a_lo, g1) * (score[n][1] * a.scale) : 0.f;
      const float p2 = s <= t_hi ? mc_exp(a_hi, g0) * (score[n][2] * a.scale) : 0.f;
      const float p3 = s + 1 <= t_hi ? mc_exp(a_hi, g1) * (score[n][3] * a.scale) : 0.f;
      own_lo += p0 + p1;
      own_hi += p2 + p3;
      __nv_bfloat16 c0[3], c1[3], c2[3], c3[3];
      mc_split(p0, c0); mc_split(p1, c1); mc_split(p2, c2); mc_split(p3, c3);
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        w[p][2 * n] = mc_two(c0[p], c1[p]);
        w[p][2 * n + 1] = mc_two(c2[p], c3[p]);
      }
    }
#pragma unroll
    for (int j = 0; j < MC_OUT_TILES; ++j) {
      if (j >= my_tiles) break;
      unsigned b[4];
      mc_ldmatrix_trans(b, mc_b_trans(v_s, (my_first + j) * 16, st * 16, lane));
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        mc_mma(acc[j][0], w[p], b[0], b[1]);
        mc_mma(acc[j][1], w[p], b[2], b[3]);
      }
    }
  }
  own_lo += __shfl_xor_sync(0xffffffffu, own_lo, 1);
  own_lo += __shfl_xor_sync(0xffffffffu, own_lo, 2);
  own_hi += __shfl_xor_sync(0xffffffffu, own_hi, 1);
  own_hi += __shfl_xor_sync(0xffffffffu, own_hi, 2);
  __syncthreads();                                      // den_s is written
  const bool on_lo = t_lo < m.rows, on_hi = t_hi < m.rows;
  const float* tops = a.top + (size_t)head * a.gate_ld + m.first;
  const float inv_lo = on_lo ? 1.0f / (fmaxf(fabsf(fmaf(w_lo, den_s[t_lo], own_lo)), expf(-tops[t_lo])) + MC_EPS) : 0.f;
  const float inv_hi = on_hi ? 1.0f / (fmaxf(fabsf(fmaf(w_hi, den_s[t_hi], own_hi)), expf(-tops[t_hi])) + MC_EPS) : 0.f;
  float2 z[MC_OUT_TILES][2][2];                         // the gate, asked for at once
  const bool even = ((a.vdim | a.ld | a.g_at) & 1) == 0 && ((uintptr_t)a.proj & 7) == 0;
#pragma unroll
  for (int j = 0; j < MC_OUT_TILES; ++j)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int l = (my_first + j) * 16 + 8 * n + 2 * q;
        z[j][n][h] = make_float2(0.f, 0.f);
        if (j < my_tiles && l < a.vdim && (h ? on_hi : on_lo)) {
          const float* from = a.proj + (size_t)(m.first + (h ? t_hi : t_lo)) * a.ld + a.g_at + head * a.vdim + l;
          if (even) z[j][n][h] = *reinterpret_cast<const float2*>(from);
          else z[j][n][h] = make_float2(from[0], l + 1 < a.vdim ? from[1] : 0.f);
        }
      }
  float sq_lo = 0.f, sq_hi = 0.f;
#pragma unroll
  for (int j = 0; j < MC_OUT_TILES; ++j)
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      float(&v)[4] = acc[j][n];
      v[0] *= inv_lo; v[1] *= inv_lo; v[2] *= inv_hi; v[3] *= inv_hi;
      sq_lo = fmaf(v[0], v[0], fmaf(v[1], v[1], sq_lo));
      sq_hi = fmaf(v[2], v[2], fmaf(v[3], v[3], sq_hi));
    }
  sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 1);
  sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 2);
  sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 1);
  sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 2);
  if (q == 0) {
    squares_s[half][t_lo] = sq_lo;
    squares_s[half][t_hi] = sq_hi;
  }
  __syncthreads();
  const float r_lo = 1.0f / sqrtf((squares_s[0][t_lo] + squares_s[1][t_lo]) / (float)a.vdim + a.eps);
  const float r_hi = 1.0f / sqrtf((squares_s[0][t_hi] + squares_s[1][t_hi]) / (float)a.vdim + a.eps);
#pragma unroll
  for (int j = 0; j < MC_OUT_TILES; ++j) {
    if (j >= my_tiles) break;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int l = (my_first + j) * 16 + 8 * n + 2 * q;
      if (l >= a.vdim) continue;
      const bool two = l + 1 < a.vdim;
      const float g0 = a.gain[head * a.vdim + l], g1 = two ? a.gain[head * a.vdim + l + 1] : 0.f;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = h ? t_hi : t_lo;
        if (!(h ? on_hi : on_lo)) continue;
        __nv_bfloat16* o = a.out + ((size_t)(m.first + t) * a.heads + head) * a.vdim + l;
        const float inv = h ? r_hi : r_lo;
        const float v0 = acc[j][n][2 * h] * inv * g0 / (1.0f + expf(-z[j][n][h].x));
        const float v1 = acc[j][n][2 * h + 1] * inv * g1 / (1.0f + expf(-z[j][n][h].y));
        if (two && (a.vdim & 1) == 0) {
          *reinterpret_cast<__nv_bfloat162*>(o) = __floats2bfloat162_rn(v0, v1);
        } else {
          o[0] = __float2bfloat16_rn(v0);
          if (two) o[1] = __float2bfloat16_rn(v1);
        }
      }
    }
  }
}

static int mc_allow(const void* kernel, size_t smem, int which) {
  static bool configured[2][64] = {};
  int device = 0;
  if (cudaGetDevice(&device) != cudaSuccess || device < 0 || device >= 64) return TOKB200_BAD_SIZE;
  if (!configured[which][device]) {
    cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
    configured[which][device] = true;
  }
  return TOKB200_OK;
}

// The places chunks can have in a step of n_rows rows of n_requests requests (see mc_base).
TOKB200_API int tokb200_mlstm_chunk_places(int n_rows, int n_requests) { return n_rows / MC_L + n_requests; }

// 1 where the kernels take the head's sizes.
TOKB200_API int tokb200_mlstm_chunks_supported(int dim, int vdim) { return dim > 0 && vdim > 0 && dim <= 128 && vdim <= 128; }

// log_f, log_i and top [heads, gate_ld] and start [requests, heads] from mlstm_gates; sums float32 [places, heads, vdim + 1,
// dim] and decay [places, heads] are scratch; out bfloat16 [T, heads * vdim].  Three launches.
TOKB200_API int tokb200_mlstm_chunks(const float* proj, int ld, int q_at, int k_at, int v_at, int g_at, int heads, int dim,
                                     int vdim, float scale, const float* log_f, const float* log_i, const float* top,
                                     long long gate_ld, const float* start, const int* q_start, const int* state_slot,
                                     int n_requests, int n_rows, float* state, long long stride, float* sums, float* decay,
                                     const float* gain, float eps, void* out, cudaStream_t stream) {
  if (n_rows <= 0 || n_requests <= 0) return TOKB200_OK;
  if (!tokb200_mlstm_chunks_supported(dim, vdim) || heads <= 0 || heads > 65535 || n_requests > 65535 ||
      q_at + heads * dim > ld || k_at + heads * dim > ld || v_at + heads * vdim > ld || g_at + heads * vdim > ld ||
      gate_ld < n_rows || (long long)heads * (vdim + 1) * dim > stride)
    return TOKB200_BAD_SIZE;
  if (((uintptr_t)sums & 15) || ((uintptr_t)out & 3)) return TOKB200_BAD_ALIGNMENT;
  McArgs a = {proj, ld, q_at, k_at, v_at, g_at, heads, dim, vdim, scale, log_f, log_i, top, gate_ld, start, q_start, state_slot,
              n_requests, state, stride, sums, decay, gain, eps, (__nv_bfloat16*)out, 0};
  a.quads = ((ld | q_at | k_at | v_at | dim | vdim) & 3) == 0 && ((uintptr_t)proj & 15) == 0;
  int status = mc_allow((const void*)mlstm_chunk_states_kernel, MC_STATE_SMEM, 0);
  if (status == TOKB200_OK) status = mc_allow((const void*)mlstm_chunk_outputs_kernel, MC_OUT_SMEM, 1);
  if (status != TOKB200_OK) return status;
  const dim3 grid(tokb200_mlstm_chunk_places(n_rows, n_requests), heads);
  status = launch_dependent(mlstm_chunk_states_kernel, grid, dim3(MC_STATE_THREADS), MC_STATE_SMEM, stream, a);
  if (status != TOKB200_OK) return status;
  const int size = (vdim + 1) * dim;
  if (size % 2 == 0)
    status = launch_dependent(mlstm_chunk_carry_kernel<2>, dim3((size / 2 + 255) / 256, heads, n_requests), dim3(256), 0, stream, a);
  else
    status = launch_dependent(mlstm_chunk_carry_kernel<1>, dim3((size + 255) / 256, heads, n_requests), dim3(256), 0, stream, a);
  if (status != TOKB200_OK) return status;
  return launch_dependent(mlstm_chunk_outputs_kernel, grid, dim3(MC_OUT_THREADS), MC_OUT_SMEM, stream, a);
}
