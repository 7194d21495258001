// A feed-forward of routed experts, computed as ONE gated feed-forward whose inner lanes are the
// experts' lanes side by side (and a shared expert's behind them): every inner lane is scaled by its
// expert's share for the token, which is zero for an expert the token did not choose, so the down
// product over all lanes is the weighted sum of the chosen experts' outputs.
//
//   moe_route   the router's logits (32-bit sums; one more row for the shared expert's gate), then
//               share[t, e] = softmax over the `top` largest logits of token t (ties: the lower
//               index), zero elsewhere; share[t, experts] = sigmoid(the shared expert's gate logit)
//   moe_gate    act[t, c] = f(gate[t, c]) * up[t, c] * share[t, expert of lane c], f the activation
//
// A third way (MOE_SCORE_SOFTMAX): s = the softmax over all router outputs, chosen like the sigmoid's.  For both,
// a group's worth is the sum of its `worth` largest choice scores (1 or 2), and with `renormalize` the chosen
// scores are divided by their sum + 1e-20.  `identity`: the last that many of the outputs that are chosen among
// stand for the token's input itself; the sum of their shares is the row's last column.
//
// moe_route knows a second way to score and choose (`score` = MOE_SCORE_SIGMOID): scores s =
// sigmoid(z); the CHOICE is made on s + correction (a learned number an expert, or none), and only
// among the experts of the `keep` best of `groups` equal groups of neighbouring experts, a group's
// worth being the sum of its two largest choice scores (the others count as minus infinity);
// share[t, e] = s[e] * scale for the chosen, not renormalized.  `shared` = 2: the shared expert's
// share is one (no gate row).  moe_gate knows a clamped activation (MOE_ACT_CLAMPED_SWISH): with
// g = min(gate, limit) and u = clamp(up, -limit, limit), g * sigmoid(alpha g) * (u + 1); the shared
// expert's lanes have a limit of their own.  With `on_input` the share multiplies the expert's INPUT instead
// of its output: the expert's first products are linear in their input, so its inner lanes are
// f(share * gate) * (share * up), and the down product adds the experts up unweighted.
#include "common.cuh"

enum : int { MOE_SCORE_SOFTMAX_OF_CHOSEN = 0, MOE_SCORE_SIGMOID = 1, MOE_SCORE_SOFTMAX = 2 };
enum : int { MOE_SHARED_NONE = 0, MOE_SHARED_GATED = 1, MOE_SHARED_ONE = 2 };
#define MOE_ACT_CLAMPED_SWISH TOKB200_ACT_COUNT

#define MOE_MAX_EXPERTS 1024

// the largest value and, among equals, the lowest index over a warp's lanes (index -1: nothing to offer)
__device__ __forceinline__ void moe_warp_best(float& value, int& index) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float v = __shfl_xor_sync(0xffffffffu, value, o);
    const int i = __shfl_xor_sync(0xffffffffu, index, o);
    if (i >= 0 && (index < 0 || v > value || (v == value && i < index))) {
      value = v;
      index = i;
    }
  }
}

// One warp chooses: the `keep` groups of the largest worth, then the `top` experts of the largest choice score
// inside them (ties: the lower index), and writes the token's row of shares.  z: the scores.  Lane l looks after
// groups and experts l, l + 32, ...
__device__ __forceinline__ void moe_choose(const float* z, const float* choice, float* group_worth, unsigned char* open,
                                           float* out, int experts, int real, int identity, int top, int groups,
                                           int keep, int worth, int renormalize, float scale, int columns, int lane) {
  const int size = experts / groups;
  if (keep < groups) {
    for (int g = lane; g < groups; g += 32) {
      float first = -INFINITY, second = -INFINITY;
      for (int e = g * size; e < (g + 1) * size; ++e) {
        const float c = choice[e];
        if (c > first) { second = first; first = c; } else if (c > second) { second = c; }
      }
      group_worth[g] = worth > 1 && size > 1 ? first + second : first;
      open[g] = 0;
    }
    for (int k = 0; k < keep; ++k) {
      int best = -1;
      float value = -INFINITY;
      for (int g = lane; g < groups; g += 32)
        if (!open[g] && (best < 0 || group_worth[g] > value)) { best = g; value = group_worth[g]; }
      moe_warp_best(value, best);
      if (best >= 0 && best % 32 == lane) open[best] = 1;
    }
    __syncwarp();
  }
  for (int c = lane; c < columns; c += 32) out[c] = 0.f;
  unsigned taken = 0u;                                  // bit i: expert lane + 32 i
  float sum = 0.f;
  for (int k = 0; k < top; ++k) {
    int best = -1;
    float value = -INFINITY;
    for (int e = lane, i = 0; e < experts; e += 32, ++i)
      if (!((taken >> i) & 1u) && (keep == groups || open[e / size]) && (best < 0 || choice[e] > value)) {
        best = e;
        value = choice[e];
      }
    moe_warp_best(value, best);
    if (best < 0) break;
    sum += z[best];
    if (best % 32 == lane) taken |= 1u << (best / 32);
  }
  const float factor = renormalize ? scale / (sum + 1e-20f) : scale;
  float through = 0.f;                                  // the identity experts' shares
  __syncwarp();
  for (int e = lane, i = 0; e < experts; e += 32, ++i)
    if ((taken >> i) & 1u) {
      if (e < real) out[e] = z[e] * factor;
      else through += z[e] * factor;
    }
  if (identity > 0) {
    through = warp_sum(through);
    if (lane == 0) out[columns - 1] = through;
  }
}

// One warp: the softmax over the `top` largest logits alone, zero elsewhere (ties: the lower index).
__device__ __forceinline__ void moe_softmax_of_chosen(const float* z, float* out, int experts, int top, int columns, int lane) {
  unsigned taken = 0u;                                  // bit i: expert lane + 32 i
  float highest = 0.f, sum = 0.f;
  for (int c = lane; c < columns; c += 32) out[c] = 0.f;
  for (int k = 0; k < top; ++k) {
    int best = -1;
    float value = -INFINITY;
    for (int e = lane, i = 0; e < experts; e += 32, ++i)
      if (!((taken >> i) & 1u) && (best < 0 ? z[e] == z[e] : z[e] > value)) {
        best = e;
        value = z[e];
      }
    moe_warp_best(value, best);
    if (best < 0) break;
    if (k == 0) highest = value;
    sum += expf(value - highest);
    if (best % 32 == lane) taken |= 1u << (best / 32);
  }
  __syncwarp();
  for (int e = lane, i = 0; e < experts; e += 32, ++i)
    if ((taken >> i) & 1u) out[e] = expf(z[e] - highest) / sum;
}

__device__ __forceinline__ float4 moe_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 moe_load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}

#define MOE_TOKENS 8       // tokens a block takes where there are many: every router row is then read once for eight

// `experts` counts every router output that is chosen among, the `identity` last ones included.
// h: the feed-forward's input [T, hidden] (float32, or its bfloat16 rounding); w: float32
// [experts + shared, hidden], the router's rows and behind them the shared expert's gate row.
// A block takes TOK tokens: its warps take the logits in turn (32-bit sums, a lane's share of a token's sum
// and the order in which the shares meet do not depend on TOK), then a warp a token chooses.
template <typename TI, int TOK>
__global__ void __launch_bounds__(TOK == 1 ? 1024 : 256, 1)
moe_route_kernel(const TI* __restrict__ h, const float* __restrict__ w, int n_rows, int hidden, int experts, int top,
                 int shared_mode, float* __restrict__ share, int score, const float* __restrict__ correction,
                 int groups, int keep, float scale, int identity, int worth, int renormalize) {
  // a token: logits (then scores) and the shared expert's, choice scores, the groups' worth, the open groups
  extern __shared__ float moe_s[];
  const int shared = shared_mode == MOE_SHARED_GATED ? 1 : 0;      // router rows behind the experts'
  const int real = experts - identity, outputs = experts + shared;
  const int columns = real + (shared_mode != MOE_SHARED_NONE ? 1 : 0) + (identity > 0 ? 1 : 0);
  const int per_token = 2 * experts + 1 + 2 * groups;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int t0 = blockIdx.x * TOK;
  if (TOK == 1) {            // few tokens: the router's rows towards L2 while the predecessor runs
    const size_t bytes = (size_t)outputs * hidden * sizeof(float);
    for (size_t at = (size_t)threadIdx.x * 128; at < bytes; at += (size_t)blockDim.x * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(w) + at));
  }
  pdl_wait();
  pdl_launch();
  const bool wide = hidden % 128 == 0 && ((((uintptr_t)h) | ((uintptr_t)w)) & 15) == 0;
  const TI* rows[TOK];
#pragma unroll
  for (int i = 0; i < TOK; ++i) rows[i] = h + (size_t)(t0 + i < n_rows ? t0 + i : t0) * hidden;
  for (int e = warp; e < outputs; e += warps) {
    const float* we = w + (size_t)e * hidden;
    float acc[TOK];
#pragma unroll
    for (int i = 0; i < TOK; ++i) acc[i] = 0.f;
    if (wide) {
      // four consecutive elements a lane and trip
#pragma unroll (TOK == 1 ? 8 : 2)
      for (int c = lane * 4; c < hidden; c += 128) {
        const float4 wv = moe_load4(we + c);
#pragma unroll
        for (int i = 0; i < TOK; ++i) {
          const float4 hv = moe_load4(rows[i] + c);
          acc[i] = fmaf(hv.x, wv.x, acc[i]);
          acc[i] = fmaf(hv.y, wv.y, acc[i]);
          acc[i] = fmaf(hv.z, wv.z, acc[i]);
          acc[i] = fmaf(hv.w, wv.w, acc[i]);
        }
      }
    } else {
      for (int c = lane; c < hidden; c += 32) {
        const float wv = we[c];
#pragma unroll
        for (int i = 0; i < TOK; ++i) acc[i] = fmaf(to_float(rows[i][c]), wv, acc[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
      const float sum = warp_sum(acc[i]);
      if (lane == 0) moe_s[i * per_token + e] = sum;
    }
  }
  __syncthreads();
  const int t = t0 + warp;
  if (warp >= TOK || t >= n_rows) return;
  float* z = moe_s + warp * per_token;
  float* choice = z + experts + 1;
  float* group_worth = choice + experts;
  unsigned char* open = reinterpret_cast<unsigned char*>(group_worth + groups);
  float* out = share + (size_t)t * columns;
  if (score == MOE_SCORE_SOFTMAX_OF_CHOSEN) {
    moe_softmax_of_chosen(z, out, experts, top, columns, lane);
  } else {
    float highest = 0.f, total = 1.f;
    if (score == MOE_SCORE_SOFTMAX) {
      highest = -INFINITY;
      for (int e = lane; e < experts; e += 32) highest = fmaxf(highest, z[e]);
      highest = warp_max(highest);
      total = 0.f;
      for (int e = lane; e < experts; e += 32) total += expf(z[e] - highest);
      total = warp_sum(total);
    }
    for (int e = lane; e < experts; e += 32) {
      const float s = score == MOE_SCORE_SOFTMAX ? expf(z[e] - highest) / total : 1.0f / (1.0f + expf(-z[e]));
      z[e] = s;
      choice[e] = s + (correction ? correction[e] : 0.f);
    }
    __syncwarp();
    moe_choose(z, choice, group_worth, open, out, experts, real, identity, top, groups, keep, worth, renormalize, scale,
               columns, lane);
  }
  __syncwarp();
  if (lane == 0 && shared_mode == MOE_SHARED_ONE) out[real] = 1.0f;
  if (lane == 0 && shared_mode == MOE_SHARED_GATED) out[real] = 1.0f / (1.0f + expf(-z[experts]));
}

// act(gate) * up of one inner lane: the activations of every gated feed-forward, and the clamped one
__device__ __forceinline__ float moe_glu(int act, float g, float u, float limit, float alpha) {
  if (act == MOE_ACT_CLAMPED_SWISH) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
  }
  return gate_activation(act, g) * u;
}

// gu: [T, 2 I], gates in the first I columns, ups in the last; lanes 0 .. experts * ff belong to the
// routed experts (ff lanes each), the lanes behind to the shared expert.
template <typename T>
__global__ void moe_gate_kernel(const T* __restrict__ gu, const float* __restrict__ share, T* __restrict__ out,
                                int inner, int experts, int ff, int shared, int act, size_t n, float limit,
                                float shared_limit, float alpha, int on_input, int share_ld) {
  pdl_wait();
  pdl_launch();
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride) {
    const size_t t = i / inner;
    const int c = (int)(i % inner);
    const int e = c < experts * ff ? c / ff : experts;
    const float w = share[t * share_ld + e];
    float value = 0.f;
    if (w != 0.f) {
      const float g = to_float(gu[t * 2 * inner + c]), u = to_float(gu[t * 2 * inner + inner + c]);
      const float lim = e < experts ? limit : shared_limit;
      value = on_input ? moe_glu(act, g * w, u * w, lim, alpha) : moe_glu(act, g, u, lim, alpha) * w;
    }
    out[i] = from_float<T>(value);
  }
}

// bfloat16, inner and expert widths in whole 8s: eight consecutive lanes (one expert's) a thread
__global__ void moe_gate_bf16x8_kernel(const __nv_bfloat16* __restrict__ gu, const float* __restrict__ share,
                                       __nv_bfloat16* __restrict__ out, int inner, int experts, int ff, int shared,
                                       int act, size_t n8, float limit, float shared_limit, float alpha,
                                       int on_input, int share_ld) {
  pdl_wait();
  pdl_launch();
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  const int per_row = inner / 8;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n8; i += stride) {
    const size_t t = i / per_row;
    const int c = (int)(i % per_row) * 8;
    const int e = c < experts * ff ? c / ff : experts;
    const float w = share[t * share_ld + e];
    uint4 packed = make_uint4(0u, 0u, 0u, 0u);
    if (w != 0.f) {
      const uint4 graw = *reinterpret_cast<const uint4*>(gu + t * 2 * inner + c);
      const uint4 uraw = *reinterpret_cast<const uint4*>(gu + t * 2 * inner + inner + c);
      const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&graw);
      const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uraw);
      __nv_bfloat162 h[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 g = __bfloat1622float2(g2[k]), u = __bfloat1622float2(u2[k]);
        const float lim = e < experts ? limit : shared_limit;
        h[k] = on_input ? __floats2bfloat162_rn(moe_glu(act, g.x * w, u.x * w, lim, alpha),
                                                moe_glu(act, g.y * w, u.y * w, lim, alpha))
                        : __floats2bfloat162_rn(moe_glu(act, g.x, u.x, lim, alpha) * w,
                                                moe_glu(act, g.y, u.y, lim, alpha) * w);
      }
      packed = *reinterpret_cast<const uint4*>(h);
    }
    *reinterpret_cast<uint4*>(out + i * 8) = packed;
  }
}

TOKB200_API int tokb200_moe_route(const void* h, int h_dtype, const float* w, int hidden, int experts, int top,
                                  int shared, float* share, int n_rows, int score, const float* correction,
                                  int groups, int keep, float scale, int identity, int worth, int renormalize,
                                  cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (identity < 0 || (identity > 0 && score == MOE_SCORE_SOFTMAX_OF_CHOSEN) || worth < 1 || worth > 2 || experts <= 0)
    return TOKB200_BAD_SIZE;
  experts += identity;                 // all that a token chooses among
  if (hidden <= 0 || experts <= 0 || experts > MOE_MAX_EXPERTS || top <= 0 || top > experts ||
      shared < MOE_SHARED_NONE || shared > MOE_SHARED_ONE ||
      score < MOE_SCORE_SOFTMAX_OF_CHOSEN || score > MOE_SCORE_SOFTMAX || groups <= 0 || experts % groups ||
      keep <= 0 || keep > groups || (long long)keep * (experts / groups) < top)
    return TOKB200_BAD_SIZE;
  const int outputs = experts + (shared == MOE_SHARED_GATED ? 1 : 0);
  const size_t per_token = (size_t)(2 * experts + 1 + 2 * groups) * sizeof(float);
  // many tokens of a router that is not large: eight a block; else one a block, a warp an output
  const bool many = n_rows > 148 && MOE_TOKENS * per_token <= 48 * 1024;
  const int warps = outputs < 4 ? 4 : outputs < 32 ? outputs : 32;
  const dim3 grid(many ? (n_rows + MOE_TOKENS - 1) / MOE_TOKENS : n_rows), block(many ? 256 : warps * 32);
  const size_t smem = per_token * (many ? MOE_TOKENS : 1);
#define LAUNCH(TI, TOK)                                                                                           \
  return launch_dependent(moe_route_kernel<TI, TOK>, grid, block, smem, stream, (const TI*)h, w, n_rows, hidden,   \
                          experts, top, shared, share, score, correction, groups, keep, scale, identity, worth,    \
                          renormalize)
  if (h_dtype == TOKB200_F32) {
    if (many) LAUNCH(float, MOE_TOKENS);
    LAUNCH(float, 1);
  }
  if (h_dtype == TOKB200_BF16) {
    if (many) LAUNCH(__nv_bfloat16, MOE_TOKENS);
    LAUNCH(__nv_bfloat16, 1);
  }
#undef LAUNCH
  return TOKB200_BAD_DTYPE;
}

TOKB200_API int tokb200_moe_gate(const void* gu, const float* share, void* out, int dtype, int n_rows, int inner,
                                 int experts, int ff, int shared, int act, float limit, float shared_limit,
                                 float alpha, int on_input, int share_ld, cudaStream_t stream) {
  if (n_rows <= 0) return TOKB200_OK;
  if (inner <= 0 || experts <= 0 || ff <= 0 || share_ld < experts + (shared ? 1 : 0) || (long long)experts * ff > inner || act < 0 || act > MOE_ACT_CLAMPED_SWISH ||
      (!shared && (long long)experts * ff != inner))
    return TOKB200_BAD_SIZE;
  const size_t n = (size_t)n_rows * inner;
  const size_t blocks = (n + 255) / 256;
  const dim3 grid((unsigned)(blocks < 8192 ? blocks : 8192));
  if (dtype == TOKB200_F32)
    return launch_dependent(moe_gate_kernel<float>, grid, dim3(256), 0, stream, (const float*)gu, share, (float*)out,
                            inner, experts, ff, shared, act, n, limit, shared_limit, alpha, on_input, share_ld);
  if (dtype == TOKB200_BF16 && inner % 8 == 0 && ff % 8 == 0 && (((uintptr_t)gu | (uintptr_t)out) & 15) == 0) {
    const size_t n8 = n / 8, blocks8 = (n8 + 255) / 256;
    return launch_dependent(moe_gate_bf16x8_kernel, dim3((unsigned)(blocks8 < 65535 ? blocks8 : 65535)), dim3(256), 0,
                            stream, (const __nv_bfloat16*)gu, share, (__nv_bfloat16*)out, inner, experts, ff, shared,
                            act, n8, limit, shared_limit, alpha, on_input, share_ld);
  }
  if (dtype == TOKB200_BF16)
    return launch_dependent(moe_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)gu,
                            share, (__nv_bfloat16*)out, inner, experts, ff, shared, act, n, limit, shared_limit, alpha,
                            on_input, share_ld);
  return TOKB200_BAD_DTYPE;
}
