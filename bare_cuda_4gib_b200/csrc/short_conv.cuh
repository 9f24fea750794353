// A short causal convolution over time per channel, four neighbouring channels a thread, over rows that a thread
// walks in order: y_t = sum_j w[:, j] * u_(t - TAPS + 1 + j), zeros before the sequence's start.  Weights and the
// last TAPS inputs stay in registers, so a row's inputs are read once.
#pragma once

#include "common.cuh"

#include <string.h>

// four bfloat16 numbers as they lie in memory, and as floats
__device__ __forceinline__ uint2 conv_load4(const __nv_bfloat16* p) { return *reinterpret_cast<const uint2*>(p); }
__device__ __forceinline__ float4 conv_floats(uint2 raw) {
  return make_float4(__uint_as_float(raw.x << 16), __uint_as_float(raw.x & 0xffff0000u), __uint_as_float(raw.y << 16),
                     __uint_as_float(raw.y & 0xffff0000u));
}
__device__ __forceinline__ uint32_t conv_pack2(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  uint32_t raw;
  memcpy(&raw, &v, 4);
  return raw;
}
__device__ __forceinline__ uint2 conv_pack4(const float (&y)[4]) { return make_uint2(conv_pack2(y[0], y[1]), conv_pack2(y[2], y[3])); }

template <int TAPS>
struct ConvColumns {
  float w[4][TAPS];
  uint2 v[TAPS > 1 ? TAPS - 1 : 1];      // inputs of positions p - TAPS + 1 .. p - 1

  // conv_w [channels][TAPS] float32, 16-byte aligned; c the first of the four channels
  __device__ __forceinline__ void load_weights(const float* conv_w, int c) {
    const float4* src = reinterpret_cast<const float4*>(conv_w + (long long)c * TAPS);      // 4 TAPS numbers, 16-byte aligned
#pragma unroll
    for (int i = 0; i < TAPS; ++i) {
      const float4 f = src[i];
      w[(4 * i) / TAPS][(4 * i) % TAPS] = f.x;
      w[(4 * i + 1) / TAPS][(4 * i + 1) % TAPS] = f.y;
      w[(4 * i + 2) / TAPS][(4 * i + 2) % TAPS] = f.z;
      w[(4 * i + 3) / TAPS][(4 * i + 3) % TAPS] = f.w;
    }
  }

  // The inputs ahead of row t, at position p of a request whose rows start at `q_start`: the step's own rows, the
  // request's ring (`entries` rows of `channels` float32, each a bfloat16 number, entry position % entries) before them.
  __device__ __forceinline__ void history(const __nv_bfloat16* u, long long u_stride, int c, int t, int p, int q_start,
                                          const float* ring_slot, int entries, int channels) {
    const int p0 = p - (t - q_start);
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) {
      const int x = p - (TAPS - 1) + j;
      if (x < 0) {
        v[j] = make_uint2(0u, 0u);
      } else if (x >= p0) {
        v[j] = conv_load4(u + (long long)(t - (p - x)) * u_stride + c);
      } else {
        const float4 f = *reinterpret_cast<const float4*>(ring_slot + (long long)(x % entries) * channels + c);
        v[j] = make_uint2(conv_pack2(f.x, f.y), conv_pack2(f.z, f.w));
      }
    }
  }

  // y of the row whose input is `now`; the window moves on by one.
  __device__ __forceinline__ void step(uint2 now, float (&y)[4]) {
    y[0] = y[1] = y[2] = y[3] = 0.0f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float4 in = conv_floats(j + 1 < TAPS ? v[j] : now);
      y[0] = fmaf(w[0][j], in.x, y[0]);
      y[1] = fmaf(w[1][j], in.y, y[1]);
      y[2] = fmaf(w[2][j], in.z, y[2]);
      y[3] = fmaf(w[3][j], in.w, y[3]);
    }
#pragma unroll
    for (int j = 0; j + 2 < TAPS; ++j) v[j] = v[j + 1];
    if (TAPS > 1) v[TAPS > 1 ? TAPS - 2 : 0] = now;
  }
};
