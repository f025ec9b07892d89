// Feed-forward layers of which every token uses some of many experts: named by a table over token
// ids, or chosen by a router over the layer's input.
//
//   choose_experts_kernel, route_rows_kernel
//                          a router's choice from its logits (or from the input, logits included, for
//                          a few tokens): sigmoid scores, a correction per expert that only the choice
//                          sees, the best groups of neighbouring experts, the `top` best experts of
//                          those, their scores divided by their sum as weights; or logits with a bias, the
//                          `top` largest, their softmax as weights
//   table_experts_kernel   one block per token: for each of the token's `top` experts act = the
//                          activation of W_up[e] h and sum += weight * W_down[e] act, added to the
//                          float32 residual stream.  (The plain form: any size.)
//   expert_up_rows_kernel, expert_down_rows_kernel
//                          the same as matrix-vector products spread over the grid (small steps
//                          and the float32 path)
//   expert_up_runs_kernel, expert_down_runs_kernel
//                          the same with an expert's rows read once for all its tokens of the step
//   route_pairs_kernel, grouped_gemm_kernel, gather_pairs_kernel
//                          the same as tiled tensor-core products over the pairs ordered by
//                          expert (long bfloat16 steps)
//
// The experts' matrices are stacked: up [experts * rows, width], down [experts * width, ff].  Two
// activations: squared relu (rows = ff), or a gated one (rows = 2 ff, an expert's gate rows before its
// up rows): g = min(g, limit), u = clamp(u, -limit, limit), g sigmoid(alpha (g + cubic g^3)) (u + shift).
// A token id of -1 - r stands for row r of `fed` (the tokens drawn in the step before), as for
// the embedding.  Products are float32 sums of products of the stored operands, in an order that
// depends on the sizes only.
#include "common.cuh"

#include <initializer_list>
#include <math_constants.h>

namespace vx {

// Which experts a token uses and with what weight.  `ids` given: row (token id) of `table` [vocab,
// top]; null: row (token's place in the step), the router's choice.  `weights` [tokens, top], or null:
// 1 / top each.
struct Choice {
  const int* ids;
  const int* fed;
  int num_fed;
  const int* table;
  int vocab, top, experts;
  const float* weights;
};

// The row of the table, or -1.
__device__ __forceinline__ int choice_row(const Choice& c, int t) {
  if (c.ids == nullptr) return t;
  int id = c.ids[t];
  if (id < 0 && c.fed != nullptr && -1 - id < c.num_fed) id = c.fed[-1 - id];
  return id >= 0 && id < c.vocab ? id : -1;
}
__device__ __forceinline__ int choice_expert(const Choice& c, int row, int k) {
  if (row < 0) return -1;
  const int e = c.table[(size_t)row * c.top + k];
  return e >= 0 && e < c.experts ? e : -1;
}
__device__ __forceinline__ float choice_weight(const Choice& c, int t, int k) {
  return c.weights != nullptr ? c.weights[(size_t)t * c.top + k] : 1.0f / (float)c.top;
}

// The gated activation's numbers; `gated` 0: squared relu.
struct ExpertAct {
  int gated;
  float limit, alpha, shift, cubic;
};
__device__ __forceinline__ float expert_glu(const ExpertAct& a, float g, float u) {
  if (a.limit > 0.f) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
  }
  const float bent = fmaf(a.cubic * g, g * g, g);
  return g / (1.0f + expf(-a.alpha * bent)) * (u + a.shift);
}

template <typename T>
__device__ __forceinline__ float dot_row(const T* __restrict__ w, const float* __restrict__ v, int n, int lane);

template <>
__device__ __forceinline__ float dot_row<float>(const float* __restrict__ w, const float* __restrict__ v, int n,
                                                int lane) {
  float acc = 0.f;
  for (int i = lane; i < n; i += 32) acc = fmaf(w[i], v[i], acc);
  return warp_sum(acc);
}

template <>
__device__ __forceinline__ float dot_row<__nv_bfloat16>(const __nv_bfloat16* __restrict__ w,
                                                        const float* __restrict__ v, int n, int lane) {
  float acc = 0.f;
  if ((n & 7) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0 && (reinterpret_cast<uintptr_t>(v) & 15) == 0) {
    // Four 16-byte loads of a lane are under way before the first is used.
    for (int i0 = lane * 8; i0 < n; i0 += 1024) {
      uint4 raw[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256;
        raw[u] = i < n ? __ldg(reinterpret_cast<const uint4*>(w + i)) : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256;
        if (i < n) {
          const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw[u]);
          const float4 v0 = *reinterpret_cast<const float4*>(v + i), v1 = *reinterpret_cast<const float4*>(v + i + 4);
          const float2 f0 = __bfloat1622float2(pairs[0]), f1 = __bfloat1622float2(pairs[1]);
          const float2 f2 = __bfloat1622float2(pairs[2]), f3 = __bfloat1622float2(pairs[3]);
          acc = fmaf(f0.x, v0.x, acc); acc = fmaf(f0.y, v0.y, acc);
          acc = fmaf(f1.x, v0.z, acc); acc = fmaf(f1.y, v0.w, acc);
          acc = fmaf(f2.x, v1.x, acc); acc = fmaf(f2.y, v1.y, acc);
          acc = fmaf(f3.x, v1.z, acc); acc = fmaf(f3.y, v1.w, acc);
        }
      }
    }
  } else {
    for (int i = lane; i < n; i += 32) acc = fmaf(__bfloat162float(w[i]), v[i], acc);
  }
  return warp_sum(acc);
}

// A router's score of a logit: its sigmoid, chosen by score + correction, or (softmax) the logit with the
// correction as a bias, which is then both.
constexpr int ROUTER_SOFTMAX = 1;  // 0: sigmoid
__device__ __forceinline__ void router_score(float z, float correction, int router, float* score, float* choice) {
  const float v = router == ROUTER_SOFTMAX ? z + correction : 1.0f / (1.0f + expf(-z));
  *score = v;
  *choice = router == ROUTER_SOFTMAX ? v : v + correction;
}

// One warp: the choice of a token from its scores.  choice_s [experts] holds score + correction and is
// used up, group_s [groups] is scratch.  A group's strength is the sum of its two best choice scores (of
// its one, if it has one); experts outside the `keep` strongest groups cannot be chosen.  Ties go to the
// lower number.
__device__ __forceinline__ void choose_experts(float* choice_s, const float* score_s, float* group_s, int experts,
                                               int groups, int keep, int top, float scale, int router, int lane,
                                               int* __restrict__ chosen, float* __restrict__ weights) {
  if (groups > 1) {
    const int size = experts / groups;
    for (int g = lane; g < groups; g += 32) {
      float first = -CUDART_INF_F, second = -CUDART_INF_F;
      for (int i = 0; i < size; ++i) {
        const float v = choice_s[g * size + i];
        if (v > first) { second = first; first = v; }
        else if (v > second) second = v;
      }
      group_s[g] = size > 1 ? first + second : first;
    }
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
      const float mine = group_s[g];
      int better = 0;
      for (int i = 0; i < groups; ++i) better += (group_s[i] > mine || (group_s[i] == mine && i < g)) ? 1 : 0;
      if (better >= keep)
        for (int i = 0; i < size; ++i) choice_s[g * size + i] = -CUDART_INF_F;
    }
    __syncwarp();
  }
  float sum = 0.f, largest = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -CUDART_INF_F;
    int at = experts;
    for (int i = lane; i < experts; i += 32) {
      const float v = choice_s[i];
      if (v > best) { best = v; at = i; }
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
      const float other = __shfl_xor_sync(0xffffffffu, best, off);
      const int other_at = __shfl_xor_sync(0xffffffffu, at, off);
      if (other > best || (other == best && other_at < at)) { best = other; at = other_at; }
    }
    if (at >= experts) at = k;  // nothing comparable is left: still a valid expert
    // The softmax over the chosen: against the largest logit, which comes first.
    if (k == 0) largest = score_s[at];
    sum += router == ROUTER_SOFTMAX ? expf(score_s[at] - largest) : score_s[at];
    if (lane == 0) {
      choice_s[at] = -CUDART_INF_F;
      chosen[k] = at;
    }
    __syncwarp();
  }
  for (int k = lane; k < top; k += 32) {
    const float v = score_s[chosen[k]];
    weights[k] = (router == ROUTER_SOFTMAX ? expf(v - largest) / sum : v / (sum + 1e-20f)) * scale;
  }
}

constexpr int CE_WARPS = 4;

__global__ void __launch_bounds__(CE_WARPS * 32)
choose_experts_kernel(const float* __restrict__ logits, long long logit_stride, const float* __restrict__ correction,
                      int experts, int groups, int keep, int top, float scale, int router, int* __restrict__ chosen,
                      float* __restrict__ weights, int num_tokens) {
  extern __shared__ float ce_s[];  // per warp: choice scores [experts], scores [experts], groups [groups]
  allow_dependents();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x * CE_WARPS + warp;
  if (t >= num_tokens) return;
  float* choice_s = ce_s + (size_t)warp * (2 * experts + groups);
  float* score_s = choice_s + experts;
  for (int i = lane; i < experts; i += 32)
    router_score(logits[(size_t)t * logit_stride + i], correction[i], router, score_s + i, choice_s + i);
  __syncwarp();
  choose_experts(choice_s, score_s, score_s + experts, experts, groups, keep, top, scale, router, lane, chosen + (size_t)t * top,
                 weights + (size_t)t * top);
}

// A block per token: the router's logits as warp-wide dot products, then the choice.  With `resid` the input
// is made here, rms_norm(resid) * norm_w rounded to T, and also written to h_out for the experts.
template <typename T>
__global__ void __launch_bounds__(512)
route_rows_kernel(const T* __restrict__ h, long long h_stride, const float* __restrict__ resid,
                  const float* __restrict__ norm_w, float eps, T* __restrict__ h_out, const T* __restrict__ w_router, int width,
                  const float* __restrict__ correction, int experts, int groups, int keep, int top, float scale,
                  int router, int* __restrict__ chosen, float* __restrict__ weights) {
  extern __shared__ __align__(16) float moe_s[];  // [width], choice [experts], scores [experts], groups [groups]
  float* choice_s = moe_s + (width + 3) / 4 * 4;
  float* score_s = choice_s + experts;
  allow_dependents();
  grid_dependency_wait();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  if (resid != nullptr) {
    __shared__ float scratch[32];
    const float* x = resid + (size_t)t * width;
    float ss = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
      const float v = x[i];
      moe_s[i] = v;
      ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
      const T v = from_float<T>(moe_s[i] * inv * norm_w[i]);
      h_out[(size_t)t * width + i] = v;
      moe_s[i] = to_float(v);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) moe_s[i] = to_float(h[(size_t)t * h_stride + i]);
  }
  __syncthreads();
  for (int e = warp; e < experts; e += warps) {
    const float z = dot_row<T>(w_router + (size_t)e * width, moe_s, width, lane);
    if (lane == 0) router_score(z, correction[e], router, score_s + e, choice_s + e);
  }
  __syncthreads();
  if (warp == 0)
    choose_experts(choice_s, score_s, score_s + experts, experts, groups, keep, top, scale, router, lane, chosen + (size_t)t * top,
                   weights + (size_t)t * top);
}

// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void table_experts_kernel(const T* __restrict__ h, long long h_stride, Choice c, ExpertAct a,
                                     const T* __restrict__ w_up, const T* __restrict__ w_down, int width, int ff,
                                     float* __restrict__ resid, const float* __restrict__ out_scale, int* status) {
  extern __shared__ __align__(16) float moe_s[];
  float* h_s = moe_s;           // [width]
  float* act_s = h_s + width;   // [ff]
  float* sum_s = act_s + ff;    // [width]
  allow_dependents();
  grid_dependency_wait();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int row = choice_row(c, t);
  if (row < 0) {
    if (threadIdx.x == 0) atomicOr(status, VX_STATUS_BAD_TOKEN_ID);
    return;
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    h_s[i] = to_float(h[(size_t)t * h_stride + i]);
    sum_s[i] = 0.f;
  }
  const int up_rows = a.gated ? 2 * ff : ff;
  for (int k = 0; k < c.top; ++k) {
    const int e = choice_expert(c, row, k);
    if (e < 0) {
      if (threadIdx.x == 0) atomicOr(status, VX_STATUS_BAD_TOKEN_ID);
      continue;
    }
    __syncthreads();
    const T* up = w_up + (size_t)e * up_rows * width;
    for (int j = warp; j < ff; j += warps) {
      const float v = dot_row<T>(up + (size_t)j * width, h_s, width, lane);
      const float u = a.gated ? dot_row<T>(up + (size_t)(ff + j) * width, h_s, width, lane) : 0.f;
      if (lane == 0) {
        const float r = fmaxf(v, 0.f);
        act_s[j] = a.gated ? expert_glu(a, v, u) : r * r;
      }
    }
    __syncthreads();
    const float weight = choice_weight(c, t, k);
    const T* down = w_down + (size_t)e * width * ff;
    for (int o = warp; o < width; o += warps) {
      const float v = dot_row<T>(down + (size_t)o * ff, act_s, ff, lane);
      if (lane == 0) sum_s[o] += weight * v;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < width; i += blockDim.x)
    resid[(size_t)t * width + i] += out_scale != nullptr ? sum_s[i] * out_scale[i] : sum_s[i];
}


// ---------------------------------------------------------------------------------------------
// Small steps: the two projections of every (token, expert) pair as matrix-vector products
// spread over the grid.  act [tokens, top, ff] float32, times the pair's weight.
template <typename T>
__global__ void expert_up_rows_kernel(const T* __restrict__ h, long long h_stride, Choice c, ExpertAct a,
                                      const T* __restrict__ w_up, int width, int ff, int rows_per_block,
                                      float* __restrict__ act, int* status) {
  extern __shared__ __align__(16) float moe_s[];  // [width]
  allow_dependents();
  grid_dependency_wait();
  const int pair = blockIdx.y, t = pair / c.top, k = pair - t * c.top;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int e = choice_expert(c, choice_row(c, t), k);
  if (e < 0) {
    if (threadIdx.x == 0 && blockIdx.x == 0) atomicOr(status, VX_STATUS_BAD_TOKEN_ID);
    return;
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x) moe_s[i] = to_float(h[(size_t)t * h_stride + i]);
  __syncthreads();
  const float weight = choice_weight(c, t, k);
  const T* up = w_up + (size_t)e * (a.gated ? 2 * ff : ff) * width;
  const int j0 = blockIdx.x * rows_per_block;
  for (int j = j0 + warp; j < min(ff, j0 + rows_per_block); j += warps) {
    const float v = dot_row<T>(up + (size_t)j * width, moe_s, width, lane);
    const float u = a.gated ? dot_row<T>(up + (size_t)(ff + j) * width, moe_s, width, lane) : 0.f;
    if (lane == 0) {
      const float r = fmaxf(v, 0.f);
      act[(size_t)pair * ff + j] = weight * (a.gated ? expert_glu(a, v, u) : r * r);
    }
  }
}

template <typename T>
__global__ void expert_down_rows_kernel(const float* __restrict__ act, Choice c, const T* __restrict__ w_down,
                                        int width, int ff, int rows_per_block, float* __restrict__ resid,
                                        const float* __restrict__ out_scale) {
  extern __shared__ __align__(16) float moe_s[];  // [top][ff]
  allow_dependents();
  grid_dependency_wait();
  const int t = blockIdx.y, top = c.top;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int row = choice_row(c, t);
  if (row < 0) return;
  for (int i = threadIdx.x; i < top * ff; i += blockDim.x) moe_s[i] = act[(size_t)t * top * ff + i];
  __syncthreads();
  const int o0 = blockIdx.x * rows_per_block;
  for (int o = o0 + warp; o < min(width, o0 + rows_per_block); o += warps) {
    float sum = 0.f;
    for (int k = 0; k < top; ++k) {
      const int e = choice_expert(c, row, k);
      if (e < 0) continue;
      sum += dot_row<T>(w_down + ((size_t)e * width + o) * ff, moe_s + (size_t)k * ff, ff, lane);
    }
    if (lane == 0) resid[(size_t)t * width + o] += out_scale != nullptr ? sum * out_scale[o] : sum;
  }
}

// ---------------------------------------------------------------------------------------------
// Small steps whose tokens share experts: the block of a pair goes on only if no earlier pair names the
// same expert, and then works for all pairs that do, RUN_TOKENS at a time, so that an expert's rows come
// from memory once.  The results of different experts for one token meet in the stream by reductions at
// the L2 (an order that is not fixed).
constexpr int RUN_MAX_PAIRS = 64, RUN_TOKENS = 4;

// The pairs of pair `own`'s expert in their order; false: an earlier pair has them, or there is no such expert.
// (A token names an expert at most once, so a step of up to RUN_MAX_PAIRS tokens fits the list.)
__device__ __forceinline__ bool list_run(const Choice& c, int own, int pairs, int* list, int* count, int* expert, int* status) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    const int e = choice_expert(c, choice_row(c, own / c.top), own % c.top);
    int found = 0;
    bool leads = e >= 0;
    if (e < 0 && lane == 0 && blockIdx.x == 0) atomicOr(status, VX_STATUS_BAD_TOKEN_ID);
    for (int base = 0; leads && base < pairs; base += 32) {
      const int q = base + lane;
      const bool same = q < pairs && choice_expert(c, choice_row(c, q / c.top), q % c.top) == e;
      const unsigned mask = __ballot_sync(0xffffffffu, same);
      if (base < own && (mask & (own - base >= 32 ? 0xffffffffu : (1u << (own - base)) - 1u)) != 0) leads = false;
      const int at = found + __popc(mask & ((1u << lane) - 1u));
      if (same && at < RUN_MAX_PAIRS) list[at] = q;
      found += __popc(mask);
    }
    if (lane == 0) {
      *count = leads ? min(found, RUN_MAX_PAIRS) : 0;
      *expert = e;
    }
  }
  __syncthreads();
  return *count > 0;
}

// Eight stored weights as they are loaded, and as floats.
template <typename T>
struct Eight;
template <>
struct Eight<float> {
  float4 a, b;
  static constexpr int BATCH = 2;
  __device__ __forceinline__ void load(const float* p) {
    a = __ldg(reinterpret_cast<const float4*>(p));
    b = __ldg(reinterpret_cast<const float4*>(p + 4));
  }
  __device__ __forceinline__ void clear() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(float (&w)[8]) const {
    w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w; w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
  }
};
template <>
struct Eight<__nv_bfloat16> {
  uint4 raw;
  static constexpr int BATCH = 4;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { raw = __ldg(reinterpret_cast<const uint4*>(p)); }
  __device__ __forceinline__ void clear() { raw = make_uint4(0u, 0u, 0u, 0u); }
  __device__ __forceinline__ void get(float (&w)[8]) const {
    const uint32_t r[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      w[2 * i] = __uint_as_float(r[i] << 16);
      w[2 * i + 1] = __uint_as_float(r[i] & 0xffff0000u);
    }
  }
};

// acc[r][t] = row r (of ROWS, `pitch` apart) times the staged vector of token t.  A staged vector's packs of eight
// lie in two halves of n / 2 floats (elements 0-3 of every pack, then 4-7): neighbouring lanes then read
// neighbouring 16 bytes.  n is a multiple of 8.  BATCH packs of every row are under way before the first is used.
template <typename T, int ROWS>
__device__ __forceinline__ void run_dots(const T* __restrict__ w, size_t pitch, const float* __restrict__ staged, int n,
                                         int tokens, int lane, float (&acc)[ROWS][RUN_TOKENS]) {
#pragma unroll
  for (int r = 0; r < ROWS; ++r)
#pragma unroll
    for (int t = 0; t < RUN_TOKENS; ++t) acc[r][t] = 0.f;
  constexpr int BATCH = Eight<T>::BATCH;
  for (int i0 = lane * 8; i0 - lane * 8 < n; i0 += 256 * BATCH) {
    Eight<T> raw[BATCH][ROWS];
#pragma unroll
    for (int u = 0; u < BATCH; ++u)
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        if (i0 + 256 * u < n) raw[u][r].load(w + r * pitch + i0 + 256 * u);
        else raw[u][r].clear();
      }
#pragma unroll
    for (int u = 0; u < BATCH; ++u) {
      const int i = i0 + 256 * u;
      if (i >= n) break;
      float wv[ROWS][8];
#pragma unroll
      for (int r = 0; r < ROWS; ++r) raw[u][r].get(wv[r]);
#pragma unroll
      for (int t = 0; t < RUN_TOKENS; ++t) {
        if (t >= tokens) break;
        const float4 lo = *reinterpret_cast<const float4*>(staged + (size_t)t * n + i / 2);
        const float4 hi = *reinterpret_cast<const float4*>(staged + (size_t)t * n + n / 2 + i / 2);
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
          float a = acc[r][t];
          a = fmaf(wv[r][0], lo.x, a); a = fmaf(wv[r][1], lo.y, a); a = fmaf(wv[r][2], lo.z, a); a = fmaf(wv[r][3], lo.w, a);
          a = fmaf(wv[r][4], hi.x, a); a = fmaf(wv[r][5], hi.y, a); a = fmaf(wv[r][6], hi.z, a); a = fmaf(wv[r][7], hi.w, a);
          acc[r][t] = a;
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r)
#pragma unroll
    for (int t = 0; t < RUN_TOKENS; ++t)
      if (t < tokens) acc[r][t] = warp_sum(acc[r][t]);
}

__device__ __forceinline__ int staged_at(int i, int n) { return ((i & 4) ? n / 2 : 0) + (i >> 3) * 4 + (i & 3); }

template <typename T>
__global__ void __launch_bounds__(256)
expert_up_runs_kernel(const T* __restrict__ h, long long h_stride, Choice c, ExpertAct a, const T* __restrict__ w_up,
                      int width, int ff, int features_per_block, int pairs, float* __restrict__ act, int* status) {
  extern __shared__ __align__(16) float moe_s[];  // [RUN_TOKENS][width]
  __shared__ int list[RUN_MAX_PAIRS], count, expert;
  allow_dependents();
  grid_dependency_wait();
  if (!list_run(c, blockIdx.y, pairs, list, &count, &expert, status)) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const T* up = w_up + (size_t)expert * (a.gated ? 2 * ff : ff) * width;
  const int j0 = blockIdx.x * features_per_block;
  for (int first = 0; first < count; first += RUN_TOKENS) {
    const int tokens = min(RUN_TOKENS, count - first);
    if (first > 0) __syncthreads();
    for (int idx = threadIdx.x; idx < tokens * width; idx += blockDim.x) {
      const int r = idx / width, i = idx - r * width;
      moe_s[(size_t)r * width + staged_at(i, width)] = to_float(h[(size_t)(list[first + r] / c.top) * h_stride + i]);
    }
    __syncthreads();
    for (int j = j0 + warp; j < min(ff, j0 + features_per_block); j += warps) {
      float acc[2][RUN_TOKENS];
      if (a.gated) {
        run_dots<T, 2>(up + (size_t)j * width, (size_t)ff * width, moe_s, width, tokens, lane, acc);
      } else {
        float one[1][RUN_TOKENS];
        run_dots<T, 1>(up + (size_t)j * width, 0, moe_s, width, tokens, lane, one);
#pragma unroll
        for (int t = 0; t < RUN_TOKENS; ++t) acc[0][t] = one[0][t], acc[1][t] = 0.f;
      }
#pragma unroll
      for (int t = 0; t < RUN_TOKENS; ++t)
        if (lane == t && t < tokens) {
          const int pair = list[first + t];
          const float r = fmaxf(acc[0][t], 0.f);
          act[(size_t)pair * ff + j] = choice_weight(c, pair / c.top, pair % c.top) * (a.gated ? expert_glu(a, acc[0][t], acc[1][t]) : r * r);
        }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
expert_down_runs_kernel(const float* __restrict__ act, Choice c, const T* __restrict__ w_down, int width, int ff,
                        int outputs_per_block, int pairs, float* __restrict__ resid, const float* __restrict__ out_scale,
                        int* status) {
  extern __shared__ __align__(16) float moe_s[];  // [RUN_TOKENS][ff]
  __shared__ int list[RUN_MAX_PAIRS], count, expert;
  allow_dependents();
  grid_dependency_wait();
  if (!list_run(c, blockIdx.y, pairs, list, &count, &expert, status)) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const T* down = w_down + (size_t)expert * width * ff;
  const int o0 = blockIdx.x * outputs_per_block;
  for (int first = 0; first < count; first += RUN_TOKENS) {
    const int tokens = min(RUN_TOKENS, count - first);
    if (first > 0) __syncthreads();
    for (int idx = threadIdx.x; idx < tokens * ff; idx += blockDim.x) {
      const int r = idx / ff, i = idx - r * ff;
      moe_s[(size_t)r * ff + staged_at(i, ff)] = act[(size_t)list[first + r] * ff + i];
    }
    __syncthreads();
    // Two outputs of a warp at a time.
    for (int o = o0 + 2 * warp; o < min(width, o0 + outputs_per_block); o += 2 * warps) {
      float acc[2][RUN_TOKENS];
      const bool both = o + 1 < width;
      run_dots<T, 2>(down + (size_t)o * ff, both ? (size_t)ff : 0, moe_s, ff, tokens, lane, acc);
#pragma unroll
      for (int t = 0; t < RUN_TOKENS; ++t) {
        if (t >= tokens) break;
        const int token = list[first + t] / c.top;
#pragma unroll
        for (int r = 0; r < 2; ++r)
          if (lane == 2 * t + r && (r == 0 || both))
            atomicAdd(resid + (size_t)token * width + o + r, out_scale != nullptr ? acc[r][t] * out_scale[o + r] : acc[r][t]);
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Long steps (bfloat16): the (token, expert) pairs are ordered by expert, every expert's run
// padded to whole tiles of GG_M rows, and the two projections run as tiled tensor-core products
// whose tiles each belong to one expert.
//
//   route_pairs_kernel    one block: counts per expert, the runs' (padded) starts, for every tile
//                         its expert, for every place its token (-1: padding), for every pair
//                         its place
//   grouped_gemm_kernel   out[place, n] = sum_k A[row(place), k] * W[expert(tile)][n, k]; the rows
//                         of A are gathered by token (up) or are the places themselves (down);
//                         the up form squares the positive part, or multiplies the activated gate
//                         with the up half, and writes bfloat16
//   gather_pairs_kernel   resid[t] += scale * (sum over the token's pairs, in their order, by weight)
constexpr int GG_M = 64, GG_N = 128, GG_K = 64, GG_LD = GG_K + 8, GG_STAGES = 2;
constexpr int GG_STAGE_ELEMS = (GG_M + GG_N) * GG_LD;
constexpr size_t GG_SMEM_BYTES = (size_t)GG_STAGES * GG_STAGE_ELEMS * sizeof(__nv_bfloat16);

__device__ __forceinline__ void cp_async_16(void* dst, const void* src, bool valid) {
  const uint32_t addr = (uint32_t)__cvta_generic_to_shared(dst);
  const int bytes = valid ? 16 : 0;  // 0: the sixteen bytes are filled with zeros, nothing is read
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(addr), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(LEFT) : "memory"); }

__global__ void route_pairs_kernel(Choice c, int num_tokens, int capacity, int max_tiles,
                                   int* __restrict__ tile_expert, int* __restrict__ place_token,
                                   int* __restrict__ pair_place, int* status, int* __restrict__ run_ends) {
  const int top = c.top, experts = c.experts;
  extern __shared__ int route_s[];  // counts [experts], starts [experts], cursor [experts]
  int* counts = route_s;
  int* starts = counts + experts;
  int* cursor = starts + experts;
  allow_dependents();
  grid_dependency_wait();
  for (int e = threadIdx.x; e < experts; e += blockDim.x) { counts[e] = 0; cursor[e] = 0; }
  for (int i = threadIdx.x; i < capacity; i += blockDim.x) place_token[i] = -1;
  for (int i = threadIdx.x; i < max_tiles; i += blockDim.x) tile_expert[i] = -1;
  __syncthreads();
  const int pairs = num_tokens * top;
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    const int t = p / top;
    const int e = choice_expert(c, choice_row(c, t), p - t * top);
    if (e < 0) {
      atomicOr(status, VX_STATUS_BAD_TOKEN_ID);
      continue;
    }
    atomicAdd(&counts[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < experts; ++e) {
      starts[e] = at;
      const int tiles = (counts[e] + GG_M - 1) / GG_M;
      for (int i = 0; i < tiles; ++i) tile_expert[at / GG_M + i] = e;
      at += tiles * GG_M;
      if (run_ends != nullptr) run_ends[e] = at;  // where the expert's (padded) run ends
    }
  }
  __syncthreads();
  // Which place of its expert's run a pair gets depends on the timing; its result does not (a
  // product's rows are independent of one another, and a token's pairs are summed in their order).
  for (int e = threadIdx.x; e < experts; e += blockDim.x) cursor[e] = 0;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) pair_place[p] = -1;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    const int t = p / top;
    const int e = choice_expert(c, choice_row(c, t), p - t * top);
    if (e < 0) continue;
    const int place = starts[e] + atomicAdd(&cursor[e], 1);
    place_token[place] = t;
    pair_place[p] = place;
  }
}

// A block of four warps (two by two) makes a tile of GG_M places by GG_N outputs; a warp's share is
// 32 x 64.  Slabs of GG_K inner values of both operands come into shared memory by asynchronous
// 16-byte copies, the next slab while this one is multiplied (two stages).
// GLU (with UP): the block's GG_N rows of W are GG_N / 2 gate rows and as many up rows of the same
// features, in turns of eight (rows n of the gate half, then rows n of the up half), so that a thread holds
// both values of a feature; N counts features.
template <bool UP, bool GLU>
__global__ void __launch_bounds__(128) grouped_gemm_kernel(
    const __nv_bfloat16* __restrict__ a, long long a_stride, const int* __restrict__ place_token,
    const int* __restrict__ tile_expert, const __nv_bfloat16* __restrict__ w, int N, int K,
    __nv_bfloat16* __restrict__ out_lowp, float* __restrict__ out_f32, long long out_stride, ExpertAct act) {
  extern __shared__ __align__(16) __nv_bfloat16 gg_s[];
  __shared__ int row_of[GG_M];
  allow_dependents();
  grid_dependency_wait();
  const int tile = blockIdx.x;
  const int e = tile_expert[tile];
  if (e < 0) return;
  const int n0 = blockIdx.y * (GLU ? GG_N / 2 : GG_N);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int wm = warp >> 1, wn = warp & 1;
  if (tid < GG_M) {
    const int place = tile * GG_M + tid;
    const int token = place_token[place];
    row_of[tid] = token < 0 ? -1 : (UP ? token : place);
  }
  __syncthreads();
  const __nv_bfloat16* wb = w + (size_t)e * (GLU ? 2 * N : N) * K;
  float acc[2][8][4];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[m][j][i] = 0.f;
  // Rows of a slab are eight 16-byte chunks; a thread copies chunk tid % 8 of rows tid / 8 + 16 u.
  const int chunk = (tid & 7) * 8, row0 = tid >> 3;
  auto fetch = [&](int k0, int stage) {
    __nv_bfloat16* a_s = gg_s + stage * GG_STAGE_ELEMS;
    __nv_bfloat16* b_s = a_s + GG_M * GG_LD;
    const bool k_ok = k0 + chunk < K;
#pragma unroll
    for (int u = 0; u < GG_M / 16; ++u) {
      const int r = row0 + 16 * u;
      const int row = row_of[r];
      const bool ok = k_ok && row >= 0;
      cp_async_16(a_s + r * GG_LD + chunk, ok ? a + (size_t)row * a_stride + k0 + chunk : a, ok);
    }
#pragma unroll
    for (int u = 0; u < GG_N / 16; ++u) {
      const int r = row0 + 16 * u;
      const int n = GLU ? n0 + (r >> 4) * 8 + (r & 7) : n0 + r;
      const bool ok = k_ok && n < N;
      const int w_row = GLU && (r & 8) ? N + n : n;
      cp_async_16(b_s + r * GG_LD + chunk, ok ? wb + (size_t)w_row * K + k0 + chunk : wb, ok);
    }
    cp_async_commit();
  };
  const int slabs = (K + GG_K - 1) / GG_K;
  fetch(0, 0);
  for (int slab = 0; slab < slabs; ++slab) {
    const int stage = slab & 1;
    if (slab + 1 < slabs) {
      fetch((slab + 1) * GG_K, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* a_s = gg_s + stage * GG_STAGE_ELEMS;
    const __nv_bfloat16* b_s = a_s + GG_M * GG_LD;
#pragma unroll
    for (int kk = 0; kk < GG_K; kk += 16) {
      uint32_t fa[2][4];
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const __nv_bfloat16* p = a_s + (wm * 32 + m * 16 + (lane & 15)) * GG_LD + kk + (lane >> 4) * 8;
        const uint32_t addr = (uint32_t)__cvta_generic_to_shared(p);
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                     : "=r"(fa[m][0]), "=r"(fa[m][1]), "=r"(fa[m][2]), "=r"(fa[m][3]) : "r"(addr));
      }
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        uint32_t fb[4];
        const __nv_bfloat16* p = b_s + (wn * 64 + j * 8 + (lane & 7) + ((lane >> 4) << 3)) * GG_LD + kk + ((lane >> 3) & 1) * 8;
        const uint32_t addr = (uint32_t)__cvta_generic_to_shared(p);
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                     : "=r"(fb[0]), "=r"(fb[1]), "=r"(fb[2]), "=r"(fb[3]) : "r"(addr));
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                       : "+f"(acc[m][j][0]), "+f"(acc[m][j][1]), "+f"(acc[m][j][2]), "+f"(acc[m][j][3])
                       : "r"(fa[m][0]), "r"(fa[m][1]), "r"(fa[m][2]), "r"(fa[m][3]), "r"(fb[0]), "r"(fb[1]));
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                       : "+f"(acc[m][j + 1][0]), "+f"(acc[m][j + 1][1]), "+f"(acc[m][j + 1][2]), "+f"(acc[m][j + 1][3])
                       : "r"(fa[m][0]), "r"(fa[m][1]), "r"(fa[m][2]), "r"(fa[m][3]), "r"(fb[2]), "r"(fb[3]));
        }
      }
    }
    __syncthreads();  // the stage may be overwritten by the copy after next
  }
  // A thread holds rows g and g + 8 of each of its two sixteens, columns 2 * (lane % 4) + {0, 1} of every n8.
  const int g = lane >> 2, c2 = 2 * (lane & 3);
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = wm * 32 + m * 16 + g + 8 * half;
      if (row_of[r] < 0) continue;
      const size_t place = (size_t)tile * GG_M + r;
      if constexpr (GLU) {
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          const int n = n0 + wn * 32 + j * 4 + c2;
          const float v0 = expert_glu(act, acc[m][j][2 * half], acc[m][j + 1][2 * half]);
          const float v1 = expert_glu(act, acc[m][j][2 * half + 1], acc[m][j + 1][2 * half + 1]);
          if (n + 1 < N) *reinterpret_cast<__nv_bfloat162*>(out_lowp + place * out_stride + n) = __floats2bfloat162_rn(v0, v1);
          else if (n < N) out_lowp[place * out_stride + n] = __float2bfloat16_rn(v0);
        }
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const int n = n0 + wn * 64 + j * 8 + c2;
          float v0 = acc[m][j][2 * half], v1 = acc[m][j][2 * half + 1];
          if (UP) {
            v0 = fmaxf(v0, 0.f); v0 *= v0;
            v1 = fmaxf(v1, 0.f); v1 *= v1;
            if (n + 1 < N) *reinterpret_cast<__nv_bfloat162*>(out_lowp + place * out_stride + n) = __floats2bfloat162_rn(v0, v1);
            else if (n < N) out_lowp[place * out_stride + n] = __float2bfloat16_rn(v0);
          } else {
            if (n + 1 < N) *reinterpret_cast<float2*>(out_f32 + place * out_stride + n) = make_float2(v0, v1);
            else if (n < N) out_f32[place * out_stride + n] = v0;
          }
        }
      }
    }
}

// rows[place, :] = h[token of the place, :], zeros for padding places (16-byte chunks).
__global__ void gather_rows_kernel(const __nv_bfloat16* __restrict__ h, long long h_stride,
                                   const int* __restrict__ place_token, int chunks, long long total,
                                   __nv_bfloat16* __restrict__ rows) {
  allow_dependents();
  grid_dependency_wait();
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (long long)gridDim.x * blockDim.x) {
    const long long place = idx / chunks;
    const int c = (int)(idx - place * chunks) * 8;
    const int token = place_token[place];
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (token >= 0) v = *reinterpret_cast<const uint4*>(h + (size_t)token * h_stride + c);
    *reinterpret_cast<uint4*>(rows + (size_t)place * chunks * 8 + c) = v;
  }
}

template <typename R>
__global__ void gather_pairs_kernel(const R* __restrict__ rows, long long row_stride,
                                    const int* __restrict__ pair_place, int top, int width,
                                    float* __restrict__ resid, const float* __restrict__ weights,
                                    const float* __restrict__ out_scale) {
  allow_dependents();
  grid_dependency_wait();
  const int t = blockIdx.x;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float sum = 0.f;
    for (int k = 0; k < top; ++k) {
      const int place = pair_place[t * top + k];
      const float w = weights != nullptr ? weights[t * top + k] : 1.0f / (float)top;
      if (place >= 0) sum = fmaf(w, to_float(rows[(size_t)place * row_stride + i]), sum);
    }
    resid[(size_t)t * width + i] += out_scale != nullptr ? sum * out_scale[i] : sum;
  }
}

}  // namespace vx

using namespace vx;

// A router's choice: chosen int32 [tokens, top], weights float32 [tokens, top], from the logits float32
// [tokens, logit_stride].
VX_API int vx_choose_experts(const float* logits, long long logit_stride, const float* correction, int experts,
                             int groups, int keep, int top, float scale, int router, int* chosen, float* weights,
                             int num_tokens, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (experts <= 0 || groups <= 0 || experts % groups != 0 || top <= 0 || keep <= 0 || keep > groups ||
      top > experts / groups * keep)
    return (int)cudaErrorInvalidValue;
  const size_t smem = sizeof(float) * CE_WARPS * (2 * (size_t)experts + groups);
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  launch_pdl(choose_experts_kernel, dim3((num_tokens + CE_WARPS - 1) / CE_WARPS), dim3(CE_WARPS * 32), smem, stream, logits,
             logit_stride, correction, experts, groups, keep, top, scale, router, chosen, weights, num_tokens);
  return (int)cudaGetLastError();
}

// The same from the router's input, h or (resid given) the norm of the stream's rows, which is then written to
// h_out [tokens, width]; -1: sizes the kernel does not take.
VX_API int vx_route_rows(const void* h, int dtype, long long h_stride, const float* resid, const float* norm_w, float eps,
                         void* h_out, const void* w_router, int width,
                         const float* correction, int experts, int groups, int keep, int top, float scale, int router,
                         int* chosen, float* weights, int num_tokens, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (experts <= 0 || groups <= 0 || experts % groups != 0 || top <= 0 || keep <= 0 || keep > groups ||
      top > experts / groups * keep)
    return (int)cudaErrorInvalidValue;
  const size_t smem = sizeof(float) * ((size_t)(width + 3) / 4 * 4 + 2 * (size_t)experts + groups);
  if (smem > 48 * 1024) return -1;
  const int threads = experts >= 16 ? 512 : (experts < 4 ? 128 : 32 * experts);
  if (dtype == VX_DTYPE_F32)
    launch_pdl(route_rows_kernel<float>, dim3(num_tokens), dim3(threads), smem, stream, (const float*)h, h_stride, resid,
               norm_w, eps, (float*)h_out, (const float*)w_router, width, correction, experts, groups, keep, top, scale, router,
               chosen, weights);
  else
    launch_pdl(route_rows_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(threads), smem, stream, (const __nv_bfloat16*)h,
               h_stride, resid, norm_w, eps, (__nv_bfloat16*)h_out, (const __nv_bfloat16*)w_router, width, correction, experts, groups, keep, top, scale,
               router, chosen, weights);
  return (int)cudaGetLastError();
}

// `act`: int gated and the gated activation's four numbers; `weights`, `out_scale`: see Choice and
// gather_pairs_kernel (null: 1 / top, 1).  `ids` null: `table` has a row per token of the step.
VX_API int vx_table_experts(const void* h, int dtype, long long h_stride, const int* ids, const int* fed,
                            int num_fed, const int* table, int vocab, int top, int experts, const float* weights,
                            int gated, float limit, float alpha, float shift, float cubic, const void* w_up,
                            const void* w_down, int width, int ff, float* resid, const float* out_scale,
                            int num_tokens, int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const size_t smem = sizeof(float) * ((size_t)2 * width + ff);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  const Choice c = {ids, fed, num_fed, table, vocab, top, experts, weights};
  const ExpertAct a = {gated, limit, alpha, shift, cubic};
  if (dtype == VX_DTYPE_F32) {
    static size_t configured = 48 * 1024;
    if (smem > configured) {
      cudaError_t e = cudaFuncSetAttribute(table_experts_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                           (int)smem);
      if (e != cudaSuccess) return (int)e;
      configured = smem;
    }
    launch_pdl(table_experts_kernel<float>, dim3(num_tokens), dim3(256), smem, stream, (const float*)h, h_stride, c, a,
               (const float*)w_up, (const float*)w_down, width, ff, resid, out_scale, status);
  } else {
    static size_t configured = 48 * 1024;
    if (smem > configured) {
      cudaError_t e = cudaFuncSetAttribute(table_experts_kernel<__nv_bfloat16>,
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
      configured = smem;
    }
    launch_pdl(table_experts_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(256), smem, stream, (const __nv_bfloat16*)h,
               h_stride, c, a, (const __nv_bfloat16*)w_up, (const __nv_bfloat16*)w_down, width, ff, resid, out_scale,
               status);
  }
  return (int)cudaGetLastError();
}

// The two-kernel form for small steps; act_rows: float32 [tokens * top * ff].
VX_API int vx_table_experts_rows(const void* h, int dtype, long long h_stride, const int* ids, const int* fed,
                                 int num_fed, const int* table, int vocab, int top, int experts, const float* weights,
                                 int gated, float limit, float alpha, float shift, float cubic, const void* w_up,
                                 const void* w_down, int width, int ff, float* act_rows, float* resid,
                                 const float* out_scale, int num_tokens, int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const size_t smem_up = sizeof(float) * (size_t)width, smem_down = sizeof(float) * (size_t)top * ff;
  if (smem_up > 48 * 1024 || smem_down > 48 * 1024) return (int)cudaErrorInvalidValue;
  const Choice c = {ids, fed, num_fed, table, vocab, top, experts, weights};
  const ExpertAct a = {gated, limit, alpha, shift, cubic};
  // Eight warps a block: four rows a warp of the first product (two features of a gated one), two of the
  // second (whose rows are `top` dot products each), so that both grids have several blocks for every SM.
  const int rows_up = gated ? 16 : 32, rows_down = 16;
  const dim3 grid_up((ff + rows_up - 1) / rows_up, num_tokens * top);
  const dim3 grid_down((width + rows_down - 1) / rows_down, num_tokens);
  if (dtype == VX_DTYPE_F32) {
    launch_pdl(expert_up_rows_kernel<float>, grid_up, dim3(256), smem_up, stream, (const float*)h, h_stride, c, a,
               (const float*)w_up, width, ff, rows_up, act_rows, status);
    launch_pdl(expert_down_rows_kernel<float>, grid_down, dim3(256), smem_down, stream, (const float*)act_rows, c,
               (const float*)w_down, width, ff, rows_down, resid, out_scale);
  } else {
    launch_pdl(expert_up_rows_kernel<__nv_bfloat16>, grid_up, dim3(256), smem_up, stream, (const __nv_bfloat16*)h,
               h_stride, c, a, (const __nv_bfloat16*)w_up, width, ff, rows_up, act_rows, status);
    launch_pdl(expert_down_rows_kernel<__nv_bfloat16>, grid_down, dim3(256), smem_down, stream, (const float*)act_rows,
               c, (const __nv_bfloat16*)w_down, width, ff, rows_down, resid, out_scale);
  }
  return (int)cudaGetLastError();
}

// The same two launches with an expert's rows read once for all its tokens; -1: sizes it does not take.
VX_API int vx_table_experts_runs(const void* h, int dtype, long long h_stride, const int* ids, const int* fed,
                                 int num_fed, const int* table, int vocab, int top, int experts, const float* weights,
                                 int gated, float limit, float alpha, float shift, float cubic, const void* w_up,
                                 const void* w_down, int width, int ff, float* act_rows, float* resid,
                                 const float* out_scale, int num_tokens, int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const size_t smem_up = sizeof(float) * RUN_TOKENS * (size_t)width, smem_down = sizeof(float) * RUN_TOKENS * (size_t)ff;
  if (num_tokens > RUN_MAX_PAIRS || width % 8 != 0 || ff % 8 != 0 || smem_up > 96 * 1024 || smem_down > 96 * 1024 ||
      ((reinterpret_cast<uintptr_t>(w_up) | reinterpret_cast<uintptr_t>(w_down)) & 15) != 0)
    return -1;
  const Choice c = {ids, fed, num_fed, table, vocab, top, experts, weights};
  const ExpertAct a = {gated, limit, alpha, shift, cubic};
  const int pairs = num_tokens * top, per_up = gated ? 16 : 32, per_down = 32;
  const dim3 grid_up((ff + per_up - 1) / per_up, pairs), grid_down((width + per_down - 1) / per_down, pairs);
#define VX_RUNS(T)                                                                                                   \
  do {                                                                                                               \
    static size_t limit_up = 46 * 1024, limit_down = 46 * 1024;                                                       \
    if (smem_up > limit_up) {                                                                                        \
      cudaFuncSetAttribute(expert_up_runs_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_up);      \
      limit_up = smem_up;                                                                                            \
    }                                                                                                                \
    if (smem_down > limit_down) {                                                                                    \
      cudaFuncSetAttribute(expert_down_runs_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_down);  \
      limit_down = smem_down;                                                                                        \
    }                                                                                                                \
    launch_pdl(expert_up_runs_kernel<T>, grid_up, dim3(256), smem_up, stream, (const T*)h, h_stride, c, a,            \
               (const T*)w_up, width, ff, per_up, pairs, act_rows, status);                                          \
    launch_pdl(expert_down_runs_kernel<T>, grid_down, dim3(256), smem_down, stream, (const float*)act_rows, c,        \
               (const T*)w_down, width, ff, per_down, pairs, resid, out_scale, status);                              \
  } while (0)
  if (dtype == VX_DTYPE_F32) VX_RUNS(float);
  else VX_RUNS(__nv_bfloat16);
#undef VX_RUNS
  return (int)cudaGetLastError();
}

VX_API int vx_grouped_tile_rows() { return GG_M; }

// The grouped tensor-core form for long bfloat16 steps.  capacity: places (a multiple of the
// tile height, at least tokens * top + experts * (tile height - 1)); route: int32 scratch of
// capacity / tile + capacity + tokens * top entries; act: bfloat16 [capacity, act_stride];
// rows: float32 [capacity, width].
VX_API int vx_table_experts_grouped(const void* h, long long h_stride, const int* ids, const int* fed, int num_fed,
                                    const int* table, int vocab, int top, int experts, const float* weights, int gated,
                                    float limit, float alpha, float shift, float cubic, const void* w_up,
                                    const void* w_down, int width, int ff, int* route, int capacity, void* act,
                                    long long act_stride, float* rows, float* resid, const float* out_scale,
                                    int num_tokens, int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (capacity % GG_M != 0 || capacity < num_tokens * top + experts * (GG_M - 1)) return (int)cudaErrorInvalidValue;
  if ((width & 7) != 0 || (ff & 7) != 0 || (h_stride & 7) != 0 || (act_stride & 7) != 0)
    return (int)cudaErrorInvalidValue;
  const int max_tiles = capacity / GG_M;
  int* tile_expert = route;
  int* place_token = route + max_tiles;
  int* pair_place = place_token + capacity;
  const size_t smem = sizeof(int) * 3 * (size_t)experts;
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  const Choice c = {ids, fed, num_fed, table, vocab, top, experts, weights};
  const ExpertAct a = {gated, limit, alpha, shift, cubic};
  launch_pdl(route_pairs_kernel, dim3(1), dim3(1024), smem, stream, c, num_tokens, capacity, max_tiles, tile_expert,
             place_token, pair_place, status, (int*)nullptr);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaSuccess;
    for (auto kernel : {grouped_gemm_kernel<true, false>, grouped_gemm_kernel<true, true>, grouped_gemm_kernel<false, false>})
      if (e == cudaSuccess) e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)GG_SMEM_BYTES);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  auto up = gated ? grouped_gemm_kernel<true, true> : grouped_gemm_kernel<true, false>;
  const int up_tile = gated ? GG_N / 2 : GG_N;
  launch_pdl(up, dim3(max_tiles, (ff + up_tile - 1) / up_tile), dim3(128), GG_SMEM_BYTES, stream,
             (const __nv_bfloat16*)h, h_stride, (const int*)place_token, (const int*)tile_expert,
             (const __nv_bfloat16*)w_up, ff, width, (__nv_bfloat16*)act, (float*)nullptr, act_stride, a);
  launch_pdl(grouped_gemm_kernel<false, false>, dim3(max_tiles, (width + GG_N - 1) / GG_N), dim3(128), GG_SMEM_BYTES,
             stream, (const __nv_bfloat16*)act, act_stride, (const int*)place_token, (const int*)tile_expert,
             (const __nv_bfloat16*)w_down, width, ff, (__nv_bfloat16*)nullptr, rows, (long long)width, a);
  launch_pdl(gather_pairs_kernel<float>, dim3(num_tokens), dim3(256), 0, stream, (const float*)rows, (long long)width,
             (const int*)pair_place, top, width, resid, weights, out_scale);
  return (int)cudaGetLastError();
}

// The same for bfloat16 rows of whole 16-byte chunks: eight values a thread.
__global__ void gather_pairs_vec_kernel(const __nv_bfloat16* __restrict__ rows, long long row_stride,
                                        const int* __restrict__ pair_place, int top, int width,
                                        float* __restrict__ resid, const float* __restrict__ weights,
                                        const float* __restrict__ out_scale) {
  allow_dependents();
  grid_dependency_wait();
  const int t = blockIdx.x;
  for (int i = threadIdx.x * 8; i < width; i += blockDim.x * 8) {
    float sum[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int k = 0; k < top; ++k) {
      const int place = pair_place[t * top + k];
      if (place < 0) continue;
      const float w = weights != nullptr ? weights[t * top + k] : 1.0f / (float)top;
      const uint4 raw = *reinterpret_cast<const uint4*>(rows + (size_t)place * row_stride + i);
      const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 f = __bfloat1622float2(pairs[q]);
        sum[2 * q] = fmaf(w, f.x, sum[2 * q]);
        sum[2 * q + 1] = fmaf(w, f.y, sum[2 * q + 1]);
      }
    }
    float4* out = reinterpret_cast<float4*>(resid + (size_t)t * width + i);
    float4 a = out[0], b = out[1];
    if (out_scale != nullptr) {
#pragma unroll
      for (int q = 0; q < 8; ++q) sum[q] *= out_scale[i + q];
    }
    a.x += sum[0]; a.y += sum[1]; a.z += sum[2]; a.w += sum[3];
    b.x += sum[4]; b.y += sum[5]; b.z += sum[6]; b.w += sum[7];
    out[0] = a;
    out[1] = b;
  }
}

// The routing alone, for a caller that runs the two products as a library's grouped product: the
// places as above, run_ends [experts] (where each expert's padded run ends), and the rows of h
// gathered by place into a_rows [capacity, width] (bfloat16).
VX_API int vx_route_and_gather(const void* h, long long h_stride, const int* ids, const int* fed, int num_fed,
                               const int* table, int vocab, int top, int experts, int width, int* route,
                               int capacity, int* run_ends, void* a_rows, int num_tokens, int* status,
                               cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (capacity % GG_M != 0 || capacity < num_tokens * top + experts * (GG_M - 1)) return (int)cudaErrorInvalidValue;
  if ((width & 7) != 0 || (h_stride & 7) != 0) return (int)cudaErrorInvalidValue;
  const int max_tiles = capacity / GG_M;
  int* tile_expert = route;
  int* place_token = route + max_tiles;
  int* pair_place = place_token + capacity;
  const size_t smem = sizeof(int) * 3 * (size_t)experts;
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  const Choice c = {ids, fed, num_fed, table, vocab, top, experts, nullptr};
  launch_pdl(route_pairs_kernel, dim3(1), dim3(1024), smem, stream, c, num_tokens, capacity, max_tiles, tile_expert,
             place_token, pair_place, status, run_ends);
  const long long total = (long long)capacity * (width / 8);
  long long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  launch_pdl(gather_rows_kernel, dim3((int)blocks), dim3(256), 0, stream, (const __nv_bfloat16*)h, h_stride,
             (const int*)place_token, width / 8, total, (__nv_bfloat16*)a_rows);
  return (int)cudaGetLastError();
}

// resid[t] += out_scale * (sum over the token's pairs, in their order, of weight * rows[place of the pair]);
// rows bfloat16 [capacity, width]; route as written by vx_route_and_gather.
VX_API int vx_gather_pairs(const void* rows, const int* route, int capacity, int top, int width, float* resid,
                           const float* weights, const float* out_scale, int num_tokens, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const int* pair_place = route + capacity / GG_M + capacity;
  if ((width & 7) == 0 && (reinterpret_cast<uintptr_t>(rows) & 15) == 0 && (reinterpret_cast<uintptr_t>(resid) & 15) == 0) {
    const int threads = width / 8 >= 256 ? 256 : (width / 8 + 31) / 32 * 32;
    launch_pdl(gather_pairs_vec_kernel, dim3(num_tokens), dim3(threads), 0, stream, (const __nv_bfloat16*)rows,
               (long long)width, pair_place, top, width, resid, weights, out_scale);
    return (int)cudaGetLastError();
  }
  launch_pdl(gather_pairs_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(256), 0, stream, (const __nv_bfloat16*)rows,
             (long long)width, pair_place, top, width, resid, weights, out_scale);
  return (int)cudaGetLastError();
}
