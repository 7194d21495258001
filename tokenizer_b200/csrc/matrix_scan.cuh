// A linear recurrence over a matrix per head, in 32-bit, token by token:
//     S <- keep S + add b x^T;   y = S^T c + skip x, or scale S^T c
// with S [N, P] (a request's state, kept as [P, N]), b and c the token's vectors over N (of the head's group of
// heads), x its vector over P, `keep` and `add` two numbers a token and head.  The mixers that run on it differ in
// where the two numbers come from and in what their columns are; both are parameters of this kernel.
//
// The columns of S are independent (column p needs x_p only), so a thread keeps NPER neighbouring
// rows (rows j NPER .. (j + 1) NPER - 1 for part j) of TWO neighbouring columns in registers and reads a
// token's b and c once for both; the 8 parts of a column add their shares of S^T c by shuffles, eight
// tokens in 4 + 2 + 1 exchanges.  The rows' arithmetic is packed: two rows an instruction.  Tokens are
// staged through shared memory in runs (cp.async, the next run on its way while
// the current one is computed); a part's rows of b and c lie side by side there,
// padded so that the 16-byte reads of the 8 parts fall on different banks.  Grid:
// (blocks of 32 columns, heads, requests).
//
// GATES STEP: add = softplus(raw step size + bias), keep = exp(-exp(a_log) add).  GATES GIVEN: both come in arrays.
// A column behind the `copied` ones has x = 1 for every token (`ones`): its S is the sum of the b's under the
// same keeps and adds, its y what that sum gives with c; it goes to `y_ones`, one number a token and head.
#pragma once
#include "common.cuh"

#define MS_PARTS 8                 // threads that share a column
#define MS_COLS 32                 // columns a block
#define MS_OWN 2                   // neighbouring columns a thread: b and c are read once for both
#define MS_THREADS (MS_PARTS * MS_COLS / MS_OWN)

enum : int { MS_GATES_STEP = 0, MS_GATES_GIVEN = 1 };

struct MatrixScanArgs {
  const float* x;            // x of token t and head h: x + t * x_ld + h * x_head, `copied` lanes
  int x_ld, x_head;
  const float* b;            // b of token t and group g: b + t * b_ld + g * b_group, N lanes; c alike
  int b_ld, b_group;
  const float* c;
  int c_ld, c_group;
  int heads, groups;
  int P, copied;             // columns, and how many of them x has (P - copied is 0, or 1: the column of ones)
  int N;
  int by16;                  // every row above starts and ends on 16 bytes (set by the launcher)
  float scale;               // GATES GIVEN: y = scale S^T c
  const float* skip;         // GATES STEP: y = S^T c + skip x, one a head
  float* state;              // [slots, stride], a slot's matrices [heads, P, N] at its start
  long long stride;
  const int* q_start;
  const int* state_slot;
  float* y;                  // [T, heads, copied]
  float* y_ones;             // [T, heads]
  // GATES STEP: raw step sizes at raw[t * raw_ld + head]; bias and a_log one a head
  const void* raw;
  int raw_ld;
  const float* bias;
  const float* a_log;
  // GATES GIVEN: [heads, gate_ld], one a token
  const float* keep;
  const float* add;
  long long gate_ld;
  float* scratch;
  int segments, n_requests;
};

__device__ __forceinline__ void ms_copy4(float* dst, const float* src) {
  const unsigned to = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(to), "l"(src) : "memory");
}

__device__ __forceinline__ void ms_copy16(float* dst, const float* src) {
  const unsigned to = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to), "l"(src) : "memory");
}

__device__ __forceinline__ float ms_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// PASS 0 runs a request's rows from first to last.  PASS 1 and 2 together do the same with a request's rows cut
// into up to `segments` equal segments (whole 16s of rows) that run side by side, for steps whose requests are
// too few to fill the device: the recurrence is linear in S, so a segment's end is (product of its decays) *
// (its start) + (its end from a zero start).  PASS 1: segment 0 runs in full from the slot's matrices; every
// other segment but the last runs from zero without reading c or writing y and leaves its end and the product
// of its decays in `scratch`.  PASS 2: every segment from the second on folds the ends before it into its start,
// then runs in full; the last one writes the slot.  (A request with one segment is done in PASS 1.)
// scratch: [requests, segments, heads, P, N] ends, then [requests, segments, heads] products.
template <int NPER, typename TI, int GATES, int PASS>
__global__ void __launch_bounds__(MS_THREADS)
matrix_scan_kernel(const MatrixScanArgs args) {
  const int heads = args.heads, P = args.P, N = args.N, copied = args.copied, segments = args.segments;
  const long long stride = args.stride;
  float* __restrict__ const state = args.state;
  float* __restrict__ const scratch = args.scratch;
  constexpr int RUN = NPER >= 32 ? 8 : 16;            // tokens staged at a time
  constexpr int PADDED = NPER + 4;                    // a part's rows and four idle lanes
  constexpr int NPAD = PADDED * MS_PARTS;
  __shared__ __align__(16) float Bs[2][RUN][NPAD];
  __shared__ __align__(16) float Cs[2][RUN][NPAD];
  __shared__ __align__(16) float xs[2][RUN][MS_COLS];
  __shared__ float dts[2][RUN];
  __shared__ float decs[2][RUN];
  // neither launch of the two has blocks for a segment that is nothing to it (the last one; the first one): blocks that
  // end at once would leave the others unevenly spread over the device
  const int head = blockIdx.y, r = PASS == 0 ? blockIdx.z : blockIdx.z / (segments - 1);
  const int seg = PASS == 0 ? 0 : blockIdx.z % (segments - 1) + (PASS == 2 ? 1 : 0);
  const int col0 = blockIdx.x * MS_COLS;
  const int part = threadIdx.x % MS_PARTS, mine_x = (threadIdx.x / MS_PARTS) * MS_OWN, col = col0 + mine_x;
  const int group = head / (heads / args.groups);
  const float a = GATES == MS_GATES_STEP ? expf(args.a_log[head]) : 0.f, bias = GATES == MS_GATES_STEP ? args.bias[head] : 0.f;
  const float d = GATES == MS_GATES_STEP ? args.skip[head] : 0.f, scale = args.scale;
  // lanes that no copy reaches (rows from N on, columns from P on) stay zero in both halves
  if (N < NPER * MS_PARTS) {
    for (int i = threadIdx.x; i < 2 * RUN * NPAD; i += MS_THREADS) {
      (&Bs[0][0][0])[i] = 0.f;
      (&Cs[0][0][0])[i] = 0.f;
    }
  }
  // (a column of ones is one of those: it is written here once)
  if (copied - col0 < MS_COLS)
    for (int i = threadIdx.x; i < 2 * RUN * MS_COLS; i += MS_THREADS)
      (&xs[0][0][0])[i] = (P > copied && i % MS_COLS == copied - col0) ? 1.f : 0.f;
  pdl_wait();
  // the second launch of the two starts when the first one's blocks end: blocks that came earlier would take whatever
  // places the first has left and lie unevenly (8,192 tokens of a lone request: 1.22 against 1.42 ms)
  if (PASS != 1) pdl_launch();
  int first = args.q_start[r], n = args.q_start[r + 1] - first;
  if (n <= 0) return;
  float* mine = state + (size_t)args.state_slot[r] * stride + ((size_t)head * P + col) * N;
  float2 S[MS_OWN][NPER / 2];              // pairs of neighbouring rows: the arithmetic below is packed, two lanes an instruction
  // a thread's rows are neighbours in the slot: 16-byte loads where the matrix has whole runs of them
  const bool whole = N == NPER * MS_PARTS && col + MS_OWN <= P && (stride & 3) == 0 && ((uintptr_t)state & 15) == 0 &&
                     (PASS == 0 || ((uintptr_t)scratch & 15) == 0);
  auto load = [&](const float* from, float2 (&T)[MS_OWN][NPER / 2]) {
    if (whole) {
#pragma unroll
      for (int o = 0; o < MS_OWN; ++o)
#pragma unroll
        for (int i = 0; i < NPER / 4; ++i) {
          const float4 v = *reinterpret_cast<const float4*>(from + (size_t)o * N + part * NPER + 4 * i);
          T[o][2 * i] = make_float2(v.x, v.y);
          T[o][2 * i + 1] = make_float2(v.z, v.w);
        }
    } else {
#pragma unroll
      for (int o = 0; o < MS_OWN; ++o)
#pragma unroll
        for (int i = 0; i < NPER / 2; ++i) {
          const int row = part * NPER + 2 * i;
          const float* f = from + (size_t)o * N;
          T[o][i] = make_float2((col + o < P && row < N) ? f[row] : 0.f, (col + o < P && row + 1 < N) ? f[row + 1] : 0.f);
        }
    }
  };
  auto store = [&](float* to) {
    if (whole) {
#pragma unroll
      for (int o = 0; o < MS_OWN; ++o)
#pragma unroll
        for (int i = 0; i < NPER / 4; ++i)
          *reinterpret_cast<float4*>(to + (size_t)o * N + part * NPER + 4 * i) =
              make_float4(S[o][2 * i].x, S[o][2 * i].y, S[o][2 * i + 1].x, S[o][2 * i + 1].y);
      return;
    }
#pragma unroll
    for (int o = 0; o < MS_OWN; ++o)
#pragma unroll
      for (int i = 0; i < NPER / 2; ++i) {
        const int row = part * NPER + 2 * i;
        float* t = to + (size_t)o * N;
        if (col + o < P && row < N) t[row] = S[o][i].x;
        if (col + o < P && row + 1 < N) t[row + 1] = S[o][i].y;
      }
  };
  bool full = true;                        // reads c and writes y
  float* end = mine;                       // where the matrices go when the rows are done (nullptr: nowhere)
  float* product = nullptr;                // where the product of the decays goes
  if (PASS == 0) {
    load(mine, S);
  } else {
    const int length = (((n + segments - 1) / segments) + 15) & ~15;
    const int count = (n + length - 1) / length;
    if (seg >= count) return;
    const bool last = seg == count - 1;
    const size_t matrices = (size_t)heads * P * N;
    float* ends = scratch + (size_t)r * segments * matrices + ((size_t)head * P + col) * N;     // + seg * matrices
    float* products = scratch + (size_t)args.n_requests * segments * matrices + (size_t)r * segments * heads + head;
    first += seg * length;
    n = n - seg * length < length ? n - seg * length : length;
    if (PASS == 1) {
      if (seg == 0) {
        load(mine, S);
        end = last ? mine : ends;
      } else {
        if (last) return;
#pragma unroll
        for (int o = 0; o < MS_OWN; ++o)
#pragma unroll
          for (int i = 0; i < NPER / 2; ++i) S[o][i] = make_float2(0.f, 0.f);
        full = false;
        end = ends + (size_t)seg * matrices;
        if (blockIdx.x == 0 && threadIdx.x == 0) product = products + (size_t)seg * heads;
      }
    } else {
      load(ends, S);
      for (int j = 1; j < seg; ++j) {
        float2 local[MS_OWN][NPER / 2];
        load(ends + (size_t)j * matrices, local);
        const float decay = products[(size_t)j * heads];
        const float2 decay2 = make_float2(decay, decay);
#pragma unroll
        for (int o = 0; o < MS_OWN; ++o)
#pragma unroll
          for (int i = 0; i < NPER / 2; ++i) S[o][i] = __ffma2_rn(decay2, S[o][i], local[o][i]);
      }
      end = last ? mine : nullptr;
    }
  }
  __syncthreads();                         // the zeros are written before the first copies land
  // 16 bytes a copy where rows, lanes and channels come in whole 4s (a piece of 4 rows lies inside one part)
  const bool by16 = args.by16 != 0;
  const float* __restrict__ const b_base = args.b + (size_t)group * args.b_group;
  const float* __restrict__ const c_base = args.c + (size_t)group * args.c_group;
  const float* __restrict__ const x_base = args.x + (size_t)head * args.x_head + col0;
  const size_t y_ld = (size_t)heads * copied;
  float* __restrict__ const y_base = args.y + (size_t)first * y_ld + (size_t)head * copied;
  auto stage = [&](int run, int half) {    // the copies of a run's x, b and c, in flight when it returns
    const int here = n - run < RUN ? n - run : RUN;
    const int cols = copied - col0 < MS_COLS ? copied - col0 : MS_COLS;
    if (by16) {
      const int pieces = N >> 2;
      for (int i = threadIdx.x; i < here * pieces; i += MS_THREADS) {
        const int k = i / pieces, row = (i - k * pieces) << 2;
        const size_t t = (size_t)(first + run + k);
        const int at = (row / NPER) * PADDED + row % NPER;
        ms_copy16(&Bs[half][k][at], b_base + t * args.b_ld + row);
        if (full) ms_copy16(&Cs[half][k][at], c_base + t * args.c_ld + row);
      }
      const int across = cols >> 2;
      for (int i = threadIdx.x; i < here * across; i += MS_THREADS) {
        const int k = i / across, c = (i - k * across) << 2;
        ms_copy16(&xs[half][k][c], x_base + (size_t)(first + run + k) * args.x_ld + c);
      }
    } else {
      for (int i = threadIdx.x; i < here * N; i += MS_THREADS) {
        const int k = i / N, row = i - k * N;
        const size_t t = (size_t)(first + run + k);
        const int at = (row / NPER) * PADDED + row % NPER;
        ms_copy4(&Bs[half][k][at], b_base + t * args.b_ld + row);
        if (full) ms_copy4(&Cs[half][k][at], c_base + t * args.c_ld + row);
      }
      for (int i = threadIdx.x; i < here * cols; i += MS_THREADS) {
        const int k = i / cols, c = i - k * cols;
        ms_copy4(&xs[half][k][c], x_base + (size_t)(first + run + k) * args.x_ld + c);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto raw_step = [&](int run) {           // the two numbers of token run + threadIdx.x, or its raw step size (asked for early)
    float2 raw = make_float2(0.f, 0.f);
    if (threadIdx.x < RUN && run + (int)threadIdx.x < n) {
      const size_t t = (size_t)(first + run + threadIdx.x);
      if (GATES == MS_GATES_STEP) {
        raw.x = to_float(((const TI*)args.raw)[t * args.raw_ld + head]);
      } else {
        raw = make_float2(args.add[(size_t)head * args.gate_ld + t], args.keep[(size_t)head * args.gate_ld + t]);
      }
    }
    return raw;
  };
  auto keep_step = [&](float2 raw, int half) {
    if (threadIdx.x < RUN) {
      if (GATES == MS_GATES_STEP) {
        const float dt = ms_softplus(raw.x + bias);
        dts[half][threadIdx.x] = dt;
        decs[half][threadIdx.x] = expf(-a * dt);
      } else {
        dts[half][threadIdx.x] = raw.x;
        decs[half][threadIdx.x] = raw.y;
      }
    }
  };
  auto write = [&](int token, int column, float x, float sum) {
    if (column < copied) y_base[token * y_ld + column] = GATES == MS_GATES_STEP ? fmaf(d, x, sum) : scale * sum;
    else if (GATES == MS_GATES_GIVEN && column < P) args.y_ones[(size_t)(first + token) * heads + head] = scale * sum;
  };
  float decayed = 1.f;                     // the product of the decays of a run from zero
  stage(0, 0);
  keep_step(raw_step(0), 0);
  int half = 0;
  for (int run = 0; run < n; run += RUN, half ^= 1) {
    const int here = n - run < RUN ? n - run : RUN;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                       // this run has landed; the other half has been read to its end
    const bool more = run + RUN < n;
    float2 raw = make_float2(0.f, 0.f);
    if (more) {
      stage(run + RUN, half ^ 1);
      raw = raw_step(run + RUN);
    }
    // one token of this thread's rows: S <- dec S + (dt x) B, and the rows' share of S^T c, for both columns
    // from one read of b and c.  Two rows an instruction (each lane an IEEE multiply or fused multiply-add of
    // its own), two sums of pairs a column so that the chain is half as long.
    auto token = [&](int k, float (&sum)[MS_OWN]) {
      const float dec = decs[half][k], dt = dts[half][k];
      const float4* b4 = reinterpret_cast<const float4*>(&Bs[half][k][part * PADDED]);
      const float4* c4 = reinterpret_cast<const float4*>(&Cs[half][k][part * PADDED]);
      const float2 dec2 = make_float2(dec, dec);
      float2 dtx2[MS_OWN], even[MS_OWN], odd[MS_OWN];
#pragma unroll
      for (int o = 0; o < MS_OWN; ++o) {
        const float dtx = dt * xs[half][k][mine_x + o];
        dtx2[o] = make_float2(dtx, dtx);
        even[o] = odd[o] = make_float2(0.f, 0.f);
      }
#pragma unroll
      for (int i = 0; i < NPER / 4; ++i) {
        const float4 b = b4[i], c = c4[i];
#pragma unroll
        for (int o = 0; o < MS_OWN; ++o) {
          S[o][2 * i] = __ffma2_rn(dec2, S[o][2 * i], __fmul2_rn(dtx2[o], make_float2(b.x, b.y)));
          S[o][2 * i + 1] = __ffma2_rn(dec2, S[o][2 * i + 1], __fmul2_rn(dtx2[o], make_float2(b.z, b.w)));
          even[o] = __ffma2_rn(S[o][2 * i], make_float2(c.x, c.y), even[o]);
          odd[o] = __ffma2_rn(S[o][2 * i + 1], make_float2(c.z, c.w), odd[o]);
        }
      }
#pragma unroll
      for (int o = 0; o < MS_OWN; ++o) {
        const float2 both = __fadd2_rn(even[o], odd[o]);
        sum[o] = both.x + both.y;
      }
    };
    int k = 0;
    if (PASS == 1 && !full) {              // from a zero start: the matrices and the product of the decays alone
      for (; k < here; ++k) {
        const float dec = decs[half][k], dt = dts[half][k];
        const float4* b4 = reinterpret_cast<const float4*>(&Bs[half][k][part * PADDED]);
        const float2 dec2 = make_float2(dec, dec);
        float2 dtx2[MS_OWN];
#pragma unroll
        for (int o = 0; o < MS_OWN; ++o) {
          const float dtx = dt * xs[half][k][mine_x + o];
          dtx2[o] = make_float2(dtx, dtx);
        }
#pragma unroll
        for (int i = 0; i < NPER / 4; ++i) {
          const float4 b = b4[i];
#pragma unroll
          for (int o = 0; o < MS_OWN; ++o) {
            S[o][2 * i] = __ffma2_rn(dec2, S[o][2 * i], __fmul2_rn(dtx2[o], make_float2(b.x, b.y)));
            S[o][2 * i + 1] = __ffma2_rn(dec2, S[o][2 * i + 1], __fmul2_rn(dtx2[o], make_float2(b.z, b.w)));
          }
        }
        decayed *= dec;
      }
    }
    // eight tokens at a time: the eight parts of a column add their shares of all eight in 4 + 2 + 1 exchanges
    // (a part passes on the half of the sums that the other side gathers), after which part j holds token j's
    // sum and writes it.  The pairs are those of the single token's rounds below, so a token's sum does not
    // depend on where in a run it falls.
    for (; k + MS_PARTS <= here; k += MS_PARTS) {
      float acc[MS_PARTS][MS_OWN];
#pragma unroll
      for (int j = 0; j < MS_PARTS; ++j) token(k + j, acc[j]);
#pragma unroll
      for (int width = MS_PARTS / 2; width >= 1; width >>= 1) {
        const bool upper = (part & width) != 0;
#pragma unroll
        for (int j = 0; j < width; ++j)
#pragma unroll
          for (int o = 0; o < MS_OWN; ++o) {
            const float send = upper ? acc[j][o] : acc[j + width][o], keep = upper ? acc[j + width][o] : acc[j][o];
            acc[j][o] = keep + __shfl_xor_sync(0xffffffffu, send, width);
          }
      }
#pragma unroll
      for (int o = 0; o < MS_OWN; ++o)
        write(run + k + part, col + o, xs[half][k + part][mine_x + o], acc[0][o]);
    }
    for (; k < here; ++k) {
      float acc[MS_OWN];
      token(k, acc);
#pragma unroll
      for (int o = 0; o < MS_OWN; ++o) {
        acc[o] += __shfl_xor_sync(0xffffffffu, acc[o], 4);
        acc[o] += __shfl_xor_sync(0xffffffffu, acc[o], 2);
        acc[o] += __shfl_xor_sync(0xffffffffu, acc[o], 1);
        if (part == 0) write(run + k, col + o, xs[half][k][mine_x + o], acc[o]);
      }
    }
    if (more) keep_step(raw, half ^ 1);
  }
  if (end != nullptr) store(end);
  if (product != nullptr) *product = decayed;
}

// `segments` > 1: a request's rows run as that many segments side by side (two launches); `scratch` then has
// n_requests * segments * heads * (P * N + 1) floats.
template <typename TI, int GATES>
static int launch_matrix_scan(MatrixScanArgs a, cudaStream_t stream) {
  if (a.n_requests <= 0) return TOKB200_OK;
  if (a.heads <= 0 || a.groups <= 0 || a.heads % a.groups || a.P <= 0 || a.N <= 0 || a.N > 32 * MS_PARTS || a.heads > 65535 ||
      a.n_requests > 65535 || a.copied < 0 || a.P - a.copied < 0 || a.P - a.copied > 1 ||
      (a.P > a.copied && a.y_ones == nullptr) || (long long)a.heads * a.P * a.N > a.stride ||
      a.segments < 1 || (a.segments > 1 && a.scratch == nullptr) || (long long)a.n_requests * a.segments > 65535)
    return TOKB200_BAD_SIZE;
  a.by16 = ((a.N | a.copied | a.x_ld | a.x_head | a.b_ld | a.b_group | a.c_ld | a.c_group) & 3) == 0 &&
           (((uintptr_t)a.x | (uintptr_t)a.b | (uintptr_t)a.c) & 15) == 0;
  const dim3 grid((a.P + MS_COLS - 1) / MS_COLS, a.heads, a.n_requests * (a.segments > 1 ? a.segments - 1 : 1));
#define MS_LAUNCH_PASS(NPER, PASS) launch_dependent(matrix_scan_kernel<NPER, TI, GATES, PASS>, grid, dim3(MS_THREADS), 0, stream, a)
#define MS_LAUNCH(NPER)                                             \
  {                                                                 \
    if (a.segments == 1) return MS_LAUNCH_PASS(NPER, 0);            \
    const int status = MS_LAUNCH_PASS(NPER, 1);                     \
    return status != TOKB200_OK ? status : MS_LAUNCH_PASS(NPER, 2); \
  }
  if (a.N <= 4 * MS_PARTS) MS_LAUNCH(4);
  if (a.N <= 8 * MS_PARTS) MS_LAUNCH(8);
  if (a.N <= 16 * MS_PARTS) MS_LAUNCH(16);
  MS_LAUNCH(32)
#undef MS_LAUNCH
#undef MS_LAUNCH_PASS
}
