// Shared by the recurrent mixers' sources: activations in float32, the second half of a low-rank pair for one
// token and the launchers' dtype switch.
#pragma once

#include "common.cuh"

namespace vx {

__device__ __forceinline__ float sq_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float sq_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float sq_silu(float v) { return v * sq_sigmoid(v); }
__device__ __forceinline__ float sq_gelu_tanh(float v) {
  return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
}
__device__ __forceinline__ float sq_act(float v, int kind) {
  if (kind == 1) return sq_silu(v);
  if (kind == 2) return sq_gelu_tanh(v);
  if (kind == 3) { const float r = fmaxf(v, 0.f); return r * r; }
  if (kind == 4) return tanhf(v);
  return v;
}

// Values whose result is rounded to bfloat16 take the special-function unit's exponential.
template <typename T>
__device__ __forceinline__ float silu_for(float v) {
  if constexpr (sizeof(T) == 2) return __fdividef(v, 1.0f + __expf(-v));
  else return sq_silu(v);
}
template <typename T>
__device__ __forceinline__ float act_for(float v, int act) {
  return act == 1 ? silu_for<T>(v) : sq_act(v, act);
}

// 2^v and softplus: a bfloat16 model's logits carry eight bits, so the approximations (relative error about
// 2^-20) are far below what they stand for; a float32 model takes the accurate forms.
template <typename T>
__device__ __forceinline__ float pow2_for(float v) {
  if constexpr (sizeof(T) == 2) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
  } else {
    return exp2f(v);
  }
}
template <typename T>
__device__ __forceinline__ float softplus_for(float v) {
  if constexpr (sizeof(T) == 2) {
    // ln(1 + e) with e = exp(-|v|): its series where 1 + e would drop e's digits.
    const float e = __expf(-fabsf(v));
    const float small = e * (1.0f - e * (0.5f - e * (0.33333333f - 0.25f * e)));
    return fmaxf(v, 0.f) + (e < 0.015625f ? small : __logf(1.0f + e));
  } else {
    return sq_softplus(v);
  }
}

// out[n] = sum over r of w[n][r] * v[r] for n < count, v in shared memory: groups of lanes share a row
// (16-byte packs where `packs` says that every row starts on one and holds whole ones), the loads of
// four rows of a group under way together.
template <typename T, int WARPS>
__device__ __forceinline__ void rank_product(const T* __restrict__ w, const float* __restrict__ v, int rank, int count,
                                             bool packs, float* __restrict__ out) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int PK = 16 / (int)sizeof(T);
  int lanes = 32;
  if (packs)
    while (lanes > 1 && (lanes / 2) * PK >= rank) lanes /= 2;
  const int groups = 32 / lanes, sub = lane & (lanes - 1), mine = warp * groups + lane / lanes;
  const int stride = WARPS * groups;
  for (int n0 = mine; n0 - mine < count; n0 += 4 * stride) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (packs) {
      for (int r = sub * PK; r < rank; r += lanes * PK) {
        uint4 raw[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int n = n0 + u * stride;
          raw[u] = n < count ? *reinterpret_cast<const uint4*>(w + (size_t)n * rank + r) : make_uint4(0u, 0u, 0u, 0u);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const T* e = reinterpret_cast<const T*>(&raw[u]);
#pragma unroll
          for (int q = 0; q < PK; ++q) acc[u] = fmaf(to_float(e[q]), v[r + q], acc[u]);
        }
      }
    } else {
      for (int r = sub; r < rank; r += lanes) {
        const float vr = v[r];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int n = n0 + u * stride;
          if (n < count) acc[u] = fmaf(to_float(w[(size_t)n * rank + r]), vr, acc[u]);
        }
      }
    }
    for (int off = lanes / 2; off > 0; off >>= 1) {
#pragma unroll
      for (int u = 0; u < 4; ++u) acc[u] += __shfl_xor_sync(0xffffffffu, acc[u], off);
    }
    if (sub == 0) {
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (n0 + u * stride < count) out[n0 + u * stride] = acc[u];
    }
  }
}

}  // namespace vx

#define VX_BY_DTYPE(dtype, CALL)                      \
  if ((dtype) == VX_DTYPE_F32) { using T = float; CALL; } \
  else { using T = __nv_bfloat16; CALL; }
