// What the kernels of the gated delta rule share: where a token's decays and step size come from, and how.
#pragma once

#include "common.cuh"

#include <math.h>

// A token's pre-activations as some product stored them.  `z` [rows] x (heads, or heads * dk with a decay per
// key channel), `b` [rows] x heads; rows are `*_stride` elements apart; element types by `*_dtype`.
struct DeltaGates {
  const void* z;
  long long z_stride;
  int z_dtype;
  const void* b;
  long long b_stride;
  int b_dtype;
  const float* a_log;      // [heads]
  const float* dt_bias;    // [heads] or [heads * dk]
};

__device__ __forceinline__ float load_any(const void* p, long long i, int dtype) {
  return dtype == DT_BF16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]) : reinterpret_cast<const float*>(p)[i];
}

// 2^x, with results below float32's normal numbers as zero
__device__ __forceinline__ float exp2_ftz(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// log(1 + e^x) = max(x, 0) + log(1 + t) with t = e^-|x| <= 1, and log(1 + t) = 2 artanh(s) = 2 (s + s^3/3 + s^5/5 + ...)
// with s = t / (2 + t) <= 1/3: six terms leave less than 2e-7 of the result.
__device__ __forceinline__ float delta_softplus(float x) {
  const float t = exp2_ftz(-1.4426950408889634f * fabsf(x));
  const float s = __fdividef(t, 2.0f + t), q = s * s;
  float sum = fmaf(q, 1.0f / 11.0f, 1.0f / 9.0f);
  sum = fmaf(q, sum, 1.0f / 7.0f);
  sum = fmaf(q, sum, 1.0f / 5.0f);
  sum = fmaf(q, sum, 1.0f / 3.0f);
  sum = fmaf(q, sum, 1.0f);
  return fmaxf(x, 0.0f) + 2.0f * s * sum;
}
__device__ __forceinline__ float delta_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float delta_silu(float x) { return x / (1.0f + expf(-x)); }

// log of the decay: -exp(A_log) * softplus(z + dt_bias), `neg_a` = -exp(A_log) of the head, c the column of z
__device__ __forceinline__ float delta_log_decay(const DeltaGates& g, long long row, int c, float neg_a) {
  return neg_a * delta_softplus(load_any(g.z, row * g.z_stride + c, g.z_dtype) + g.dt_bias[c]);
}

__device__ __forceinline__ float delta_beta(const DeltaGates& g, long long row, int head) {
  return delta_sigmoid(load_any(g.b, row * g.b_stride + head, g.b_dtype));
}
