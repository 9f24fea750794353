// Softmax attention over the paged cache with the pieces that sit between the projection and the
// scores in some designs:
//
//   * a short causal convolution over time on every channel of q, k and v, whose last taps - 1
//     inputs per request are kept in a state slot as a ring indexed by position;
//   * an RMS norm over the whole q projection and over the whole k projection (all heads at once);
//   * a factor on q that grows with the logarithm of the position;
//   * a rotation by position of a head's first entries of q and k, in neighbouring pairs or in halves;
//   * a bias per (distance, head) added to the scaled score, read from a table by distance;
//   * key and value heads of different sizes.
//
// Everything between the projection's stored result and the stored q, k, v is float32; scores,
// softmax and the weighted sum are float32.

#include "common.cuh"
#include "short_conv.cuh"

#include <math.h>

// Keys [kv_heads][page_tokens][k_dim] then values [kv_heads][page_tokens][v_dim] per page and cache.
struct PagedCacheKV {
  void* k;
  void* v;
  const int32_t* block_table;
  long long page_stride;
  int table_stride;
  int page_tokens;
  int kv_heads;
  int k_dim;
  int v_dim;
};

__device__ __forceinline__ int cache_page(const PagedCacheKV& c, int seq, int pos) {
  return c.block_table[(long long)seq * c.table_stride + pos / c.page_tokens];
}

// ------------------------------------ convolution + whole-projection norms + cache write (per row)

// u: the step's projection rows [q | k | v] (C = qd + kd + vd channels).  For row t at position p
// of a request whose portion starts at position p0 (row t0):
//   y[c] = sum_j w[c][j] * U(p - taps + 1 + j)[c],  U(x) = 0 for x < 0, the step's own row for
//   x >= p0, and the ring entry x % (taps - 1) of the request's state otherwise.
// Then q = y_q / rms(y_q) * wq * (1 + coef * ln(floor((p + 1) / every) + 1)), k = y_k / rms(y_k) * wk,
// v = y_v; with `inv_freq` the first `rot_dims` entries of every q and k head are turned pair by pair (entry
// 2i with 2i + 1, or with `halves` i with i + rot_dims / 2) by the angle p * inv_freq[i]; q goes to q_out, k
// and v into the cache.
template <typename T>
__global__ void __launch_bounds__(512) conv_norm_cache_kernel(const T* __restrict__ u, long long u_stride, const float* __restrict__ conv_w,
                                       int taps, const float* __restrict__ ring, const float* __restrict__ q_norm_w,
                                       const float* __restrict__ k_norm_w, T* __restrict__ q_out, PagedCacheKV cache,
                                       const int32_t* __restrict__ positions, const int32_t* __restrict__ row_seq,
                                       const int32_t* __restrict__ seq_slot, const int32_t* __restrict__ seq_q_start,
                                       int qd, int kd, int vd, float eps, float temp_coef, int temp_every,
                                       int write_cache, const float* __restrict__ inv_freq, int rot_dims, int halves) {
  pdl_launch_dependents();
  extern __shared__ float ys[];      // C floats + 32 scratch + rot_dims cosines and sines
  const int C = qd + kd + vd;
  float* scratch = ys + C;
  float* turn = scratch + 32;        // [rot_dims / 2] cosines, then as many sines
  pdl_wait();
  const int t = blockIdx.x;
  const int seq = row_seq[t], p = positions[t];
  const int slot = seq_slot[seq];
  const int p0 = p - (t - seq_q_start[seq]);
  const int hist = taps - 1;
  const float* ring_slot = ring + (long long)slot * (hist > 0 ? hist : 1) * C;
  float sq_q = 0.0f, sq_k = 0.0f;
  // most rows of a prompt's portion have all their taps inside the step's own rows: no case per tap
  const bool inside = p - hist >= p0;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    float y = 0.0f;
    if (inside) {
      const T* col = u + (long long)(t - hist) * u_stride + c;
      const float* w = conv_w + (long long)c * taps;
      for (int j = 0; j < taps; ++j) y += w[j] * to_float(col[(long long)j * u_stride]);
    } else
    for (int j = 0; j < taps; ++j) {
      const int x = p - hist + j;
      if (x < 0) continue;
      float val;
      if (x >= p0) val = to_float(u[(long long)(t - (p - x)) * u_stride + c]);
      else val = ring_slot[(long long)(x % hist) * C + c];
      y += conv_w[(long long)c * taps + j] * val;
    }
    ys[c] = y;
    if (c < qd) sq_q += y * y;
    else if (c < qd + kd) sq_k += y * y;
  }
  const int half = inv_freq ? rot_dims / 2 : 0;
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)p * inv_freq[i], &turn[half + i], &turn[i]);
  const float tq = block_sum(sq_q, scratch);      // (its barriers also make ys and turn whole)
  const float tk = block_sum(sq_k, scratch);
  const float rq = 1.0f / sqrtf(tq / (float)qd + eps) * (1.0f + temp_coef * logf((float)((p + 1) / temp_every + 1)));
  const float rk = 1.0f / sqrtf(tk / (float)kd + eps);
  const int page = cache_page(cache, seq, p);
  const int in_page = p % cache.page_tokens;
  // entry d of a head whose channels start at c0: normed, and turned where the rotation reaches
  auto head_entry = [&](int c0, int d, float r, const float* w) -> float {
    const float v = ys[c0 + d] * r * w[d];
    if (d >= 2 * half) return v;
    const int i = halves ? (d < half ? d : d - half) : d >> 1;
    const bool second = halves ? d >= half : d & 1;
    const int e = halves ? (second ? d - half : d + half) : d ^ 1;
    const float other = ys[c0 + e] * r * w[e];
    return second ? v * turn[i] + other * turn[half + i] : v * turn[i] - other * turn[half + i];
  };
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    if (c < qd) {
      const int d = c % cache.k_dim;
      q_out[(long long)t * qd + c] = from_float<T>(head_entry(c - d, d, rq, q_norm_w + (c - d)));
    } else if (write_cache && page >= 0) {
      if (c < qd + kd) {
        const int e = c - qd, g = e / cache.k_dim, d = e - g * cache.k_dim;
        T* dst = (T*)cache.k + (long long)page * cache.page_stride + ((long long)g * cache.page_tokens + in_page) * cache.k_dim + d;
        *dst = from_float<T>(head_entry(c - d, d, rk, k_norm_w + (e - d)));
      } else {
        const int e = c - qd - kd, g = e / cache.v_dim, d = e - g * cache.v_dim;
        T* dst = (T*)cache.v + (long long)page * cache.page_stride + ((long long)g * cache.page_tokens + in_page) * cache.v_dim + d;
        *dst = from_float<T>(ys[c]);
      }
    }
  }
}

// The same for bfloat16 in pieces of four channels: sizes that are multiples of four, up to four taps, a rotation in
// neighbouring pairs or none.  A block walks `rows_per_block` rows with its channels' weights and last inputs in
// registers, PIECES pieces a thread.  With `write_ring` (steps of one token per request only) it also does what
// conv_ring_write does: the entry it writes is the one the same thread has read as the oldest input.
template <int TAPS, int PIECES>
__global__ void __launch_bounds__(PIECES == 1 ? 768 : 512)
conv_norm_cache_vec_kernel(const __nv_bfloat16* __restrict__ u, long long u_stride, const float* __restrict__ conv_w,
                           float* __restrict__ ring, const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w,
                           __nv_bfloat16* __restrict__ q_out, PagedCacheKV cache, const int32_t* __restrict__ positions,
                           const int32_t* __restrict__ row_seq, const int32_t* __restrict__ seq_slot,
                           const int32_t* __restrict__ seq_q_start, int n_tokens, int rows_per_block, int qd, int kd, int vd,
                           float eps, float temp_coef, int temp_every, int write_cache, int write_ring,
                           const float* __restrict__ inv_freq, int rot_dims) {
  pdl_launch_dependents();
  constexpr int HIST = TAPS - 1, BATCH = PIECES == 1 ? 4 : 2;
  extern __shared__ float turns[];             // [BATCH][rot_dims] cosines, then sines, of a batch of rows
  __shared__ float2 sums[BATCH][32];
  const int C = qd + kd + vd, half = rot_dims / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_warps = blockDim.x >> 5;
  ConvColumns<TAPS> conv[PIECES];
  int at[PIECES];
#pragma unroll
  for (int j = 0; j < PIECES; ++j) {
    at[j] = (threadIdx.x + j * blockDim.x) * 4;
    if (at[j] < C) conv[j].load_weights(conv_w, at[j]);
  }
  pdl_wait();
  const int t0 = blockIdx.x * rows_per_block, rows = min(rows_per_block, n_tokens - t0);
  // where this thread's channels go: 0 q, 1 k, 2 v; its head and the entry in it
  int kind[PIECES], entry[PIECES], in_head[PIECES], head_of[PIECES];
#pragma unroll
  for (int j = 0; j < PIECES; ++j) {
    kind[j] = at[j] < qd ? 0 : (at[j] < qd + kd ? 1 : 2);
    entry[j] = at[j] - (kind[j] == 0 ? 0 : (kind[j] == 1 ? qd : qd + kd));
    const int dim = kind[j] == 2 ? cache.v_dim : cache.k_dim;
    head_of[j] = entry[j] / dim;
    in_head[j] = entry[j] - head_of[j] * dim;
  }
  int seq = -1;
  for (int r0 = 0; r0 < rows; r0 += BATCH) {      // some rows' inputs are asked for together
    uint2 in[PIECES][BATCH];
#pragma unroll
    for (int j = 0; j < PIECES; ++j)
      if (at[j] < C) {
#pragma unroll
        for (int k = 0; k < BATCH; ++k) in[j][k] = conv_load4(u + (long long)(t0 + min(r0 + k, rows - 1)) * u_stride + at[j]);
      }
    const int batch = min(BATCH, rows - r0);
    for (int i = threadIdx.x; i < batch * half; i += blockDim.x) {
      const int k = i / half, x = i - k * half;
      sincosf((float)positions[t0 + r0 + k] * inv_freq[x], &turns[k * rot_dims + half + x], &turns[k * rot_dims + x]);
    }
    float y[BATCH][PIECES][4];
#pragma unroll
    for (int k = 0; k < BATCH; ++k) {
      float2 sq = make_float2(0.0f, 0.0f);
      if (k < batch) {
        const int t = t0 + r0 + k, s = row_seq[t], p = positions[t];
        const bool fresh = s != seq;
        seq = s;
        float* ring_slot = ring + (long long)seq_slot[s] * (HIST > 0 ? HIST : 1) * C;
#pragma unroll
        for (int j = 0; j < PIECES; ++j) {
          if (at[j] >= C) continue;
          if (fresh) conv[j].history(u, u_stride, at[j], t, p, seq_q_start[s], ring_slot, HIST, C);
          conv[j].step(in[j][k], y[k][j]);
          if (HIST > 0 && write_ring)
            *reinterpret_cast<float4*>(ring_slot + (long long)(p % (HIST > 0 ? HIST : 1)) * C + at[j]) = conv_floats(in[j][k]);
          const float e = y[k][j][0] * y[k][j][0] + y[k][j][1] * y[k][j][1] + y[k][j][2] * y[k][j][2] + y[k][j][3] * y[k][j][3];
          if (kind[j] == 0) sq.x += e;
          else if (kind[j] == 1) sq.y += e;
        }
        sq.x = warp_sum(sq.x);
        sq.y = warp_sum(sq.y);
      }
      if (lane == 0) sums[k][warp] = sq;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BATCH; ++k) {
      if (k >= batch) break;
      const int t = t0 + r0 + k, s = row_seq[t], p = positions[t];
      const float* turn = turns + k * rot_dims;
      const float2 sq = lane < n_warps ? sums[k][lane] : make_float2(0.0f, 0.0f);
      float rq = 1.0f / sqrtf(warp_sum(sq.x) / (float)qd + eps);
      const float rk = 1.0f / sqrtf(warp_sum(sq.y) / (float)kd + eps);
      if (temp_coef != 0.0f) rq *= 1.0f + temp_coef * logf((float)((p + 1) / temp_every + 1));
      const int page = cache_page(cache, s, p), in_page = p % cache.page_tokens;
#pragma unroll
      for (int j = 0; j < PIECES; ++j) {
        if (at[j] >= C || (kind[j] != 0 && (!write_cache || page < 0))) continue;
        float v[4] = {y[k][j][0], y[k][j][1], y[k][j][2], y[k][j][3]};
        if (kind[j] != 2) {
          const float4 w = *reinterpret_cast<const float4*>((kind[j] == 0 ? q_norm_w : k_norm_w) + entry[j]);
          const float f = kind[j] == 0 ? rq : rk;
          v[0] *= f * w.x; v[1] *= f * w.y; v[2] *= f * w.z; v[3] *= f * w.w;
#pragma unroll
          for (int x = 0; x < 4; x += 2) {
            const int d = in_head[j] + x;
            if (d < rot_dims) {
              const float c = turn[d / 2], sn = turn[half + d / 2], e0 = v[x], e1 = v[x + 1];
              v[x] = e0 * c - e1 * sn;
              v[x + 1] = e1 * c + e0 * sn;
            }
          }
        }
        __nv_bfloat16* dst =
            kind[j] == 0 ? q_out + (long long)t * qd + entry[j]
                         : (__nv_bfloat16*)(kind[j] == 1 ? cache.k : cache.v) + (long long)page * cache.page_stride +
                               ((long long)head_of[j] * cache.page_tokens + in_page) * (kind[j] == 1 ? cache.k_dim : cache.v_dim) + in_head[j];
        *reinterpret_cast<uint2*>(dst) = conv_pack4(v);
      }
    }
    __syncthreads();      // sums and turns have been read
  }
}

extern "C" int llm_conv_norm_cache(const void* u, int dtype, long long u_stride, const float* conv_w, int taps,
                                   float* ring, const float* q_norm_w, const float* k_norm_w, void* q_out,
                                   void* cache_k, void* cache_v, const int32_t* block_table, long long page_stride,
                                   int table_stride, int page_tokens, int kv_heads, int k_dim, int v_dim,
                                   const int32_t* positions, const int32_t* row_seq, const int32_t* seq_slot,
                                   const int32_t* seq_q_start, int n_tokens, int q_heads, float eps, float temp_coef,
                                   int temp_every, int write_cache, const float* inv_freq, int rot_dims, int halves,
                                   int write_ring, int* ring_written, cudaStream_t stream) {
  *ring_written = 0;
  if (n_tokens <= 0) return 0;
  LLM_HOST_CHECK(taps >= 1 && temp_every >= 1, ERR_BAD_SIZE);
  if (!inv_freq) rot_dims = 0;
  LLM_HOST_CHECK(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= k_dim, ERR_BAD_SIZE);
  const int qd = q_heads * k_dim, kd = kv_heads * k_dim, vd = kv_heads * v_dim;
  const int C = qd + kd + vd;
  const size_t smem = (size_t)(C + 32 + rot_dims) * sizeof(float);
  LLM_HOST_CHECK(smem <= 200 * 1024, ERR_BAD_SIZE);
  const int threads = C >= 2048 ? 512 : (C >= 512 ? 256 : 128);
  PagedCacheKV cache{cache_k, cache_v, block_table, page_stride, table_stride, page_tokens, kv_heads, k_dim, v_dim};
  auto aligned = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) % bytes) == 0; };
  const int pieces = C / 4 <= 768 ? 1 : (C / 4 <= 1024 ? 2 : 3);
  const bool vec = dtype == DT_BF16 && taps <= 4 && !(halves && rot_dims) && k_dim % 4 == 0 && v_dim % 4 == 0 &&
                   C / 4 <= 3 * 512 && u_stride % 4 == 0 && page_stride % 4 == 0 && aligned(u, 8) && aligned(conv_w, 16) && aligned(ring, 16) &&
                   aligned(q_norm_w, 16) && aligned(k_norm_w, 16) && aligned(q_out, 8) && aligned(cache_k, 8) && aligned(cache_v, 8);
  if (vec) {
    *ring_written = write_ring;
    const int wide = ((C / 4 + pieces - 1) / pieces + 31) / 32 * 32, per_block = n_tokens >= 512 ? ((n_tokens + 147) / 148 + 3) / 4 * 4 : (n_tokens >= 256 ? 2 : 1);
    const int blocks = (n_tokens + per_block - 1) / per_block;
#define VEC(TAPS, PIECES)                                                                                              \
  launch_kernel(conv_norm_cache_vec_kernel<TAPS, PIECES>, blocks, wide, (size_t)4 * rot_dims * sizeof(float), stream,  \
                (const __nv_bfloat16*)u, u_stride, conv_w, ring, q_norm_w, k_norm_w, (__nv_bfloat16*)q_out, cache,      \
                positions, row_seq, seq_slot, seq_q_start, n_tokens, per_block, qd, kd, vd, eps, temp_coef, temp_every, \
                write_cache, write_ring, inv_freq, rot_dims)
#define TAPS_OF(PIECES)                                                                                                \
  do {                                                                                                                 \
    if (taps == 1) VEC(1, PIECES); else if (taps == 2) VEC(2, PIECES); else if (taps == 3) VEC(3, PIECES); else VEC(4, PIECES); \
  } while (0)
    if (pieces == 1) TAPS_OF(1); else if (pieces == 2) TAPS_OF(2); else TAPS_OF(3);
#undef TAPS_OF
#undef VEC
    return launch_status();
  }
#define LAUNCH(T)                                                                                                 \
  do {                                                                                                            \
    if (smem > 48 * 1024)                                                                                         \
      cudaFuncSetAttribute(conv_norm_cache_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
    launch_kernel(conv_norm_cache_kernel<T>, n_tokens, threads, smem, stream, (const T*)u, u_stride, conv_w, taps, \
                  ring, q_norm_w, k_norm_w, (T*)q_out, cache, positions, row_seq, seq_slot, seq_q_start, qd, kd, vd, \
                  eps, temp_coef, temp_every, write_cache, inv_freq, rot_dims, halves);                                                        \
  } while (0)
  if (dtype == DT_F32) LAUNCH(float);
  else if (dtype == DT_BF16) LAUNCH(__nv_bfloat16);
  else return ERR_BAD_DTYPE;
#undef LAUNCH
  return launch_status();
}

// The projection rows of each request's last taps - 1 positions go into its ring (entry position %
// (taps - 1)), after the convolution of the step has read the ring.  Grid (request x kept position, slice of channels).
template <typename T>
__global__ void conv_ring_write_kernel(const T* __restrict__ u, long long u_stride, float* __restrict__ ring, int hist,
                                       int C, const int32_t* __restrict__ seq_slot, const int32_t* __restrict__ seq_q_start,
                                       const int32_t* __restrict__ seq_q_len, const int32_t* __restrict__ seq_kv_len) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.x / hist, back = blockIdx.x % hist + 1;      // the request's last position, the last but one, ...
  if (back > seq_q_len[seq]) return;
  const int t = seq_q_start[seq] + seq_q_len[seq] - back, p = seq_kv_len[seq] - back;
  float* dst = ring + ((long long)seq_slot[seq] * hist + (p % hist)) * C;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
    dst[c] = to_float(u[(long long)t * u_stride + c]);
}

extern "C" int llm_conv_ring_write(const void* u, int dtype, long long u_stride, float* ring, int taps, int channels,
                                   const int32_t* seq_slot, const int32_t* seq_q_start, const int32_t* seq_q_len,
                                   const int32_t* seq_kv_len, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0 || taps <= 1) return 0;
  const dim3 grid(n_seqs * (taps - 1), (channels + 1023) / 1024);
  if (dtype == DT_F32)
    launch_kernel(conv_ring_write_kernel<float>, grid, 256, 0, stream, (const float*)u, u_stride, ring, taps - 1, channels,
                  seq_slot, seq_q_start, seq_q_len, seq_kv_len);
  else if (dtype == DT_BF16)
    launch_kernel(conv_ring_write_kernel<__nv_bfloat16>, grid, 256, 0, stream, (const __nv_bfloat16*)u, u_stride, ring,
                  taps - 1, channels, seq_slot, seq_q_start, seq_q_len, seq_kv_len);
  else
    return ERR_BAD_DTYPE;
  return launch_status();
}

// ------------------------------------------------------------- attention with a distance bias

#define BA_WARPS 4

// One warp per (row, query head).  Keys are walked in blocks of 32 absolute positions (block b
// holds positions 32 b .. 32 b + 31), one key per lane: score = (q . k) * scale +
// bias[head][distance] (with `softcap` > 0 the scaled score first becomes softcap * tanh(score / softcap));
// online softmax over blocks, `extras` as AttentionExtras says; the value sum with one output channel group
// per lane.  Each sum's order depends on the sizes and on absolute key positions only.
template <typename T>
__global__ void __launch_bounds__(BA_WARPS * 32)
biased_attention_kernel(const T* __restrict__ q, T* __restrict__ out, long long out_stride, PagedCacheKV cache,
                        const float* __restrict__ bias, int bias_len, const int32_t* __restrict__ positions,
                        const int32_t* __restrict__ row_seq, int q_heads, int n_tokens, float scale, int window,
                        float out_scale, float softcap, AttentionExtras extras) {
  pdl_launch_dependents();
  extern __shared__ float q_sm[];   // [BA_WARPS][k_dim]
  const int dk = cache.k_dim, dv = cache.v_dim;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long item = (long long)blockIdx.x * BA_WARPS + warp;
  pdl_wait();
  if (item >= (long long)n_tokens * q_heads) return;
  const int t = (int)(item / q_heads), h = (int)(item - (long long)t * q_heads);
  const int g = h / (q_heads / cache.kv_heads);
  const int seq = row_seq[t], p = positions[t];
  float* qs = q_sm + warp * dk;
  for (int d = lane; d < dk; d += 32) qs[d] = to_float(q[(long long)t * q_heads * dk + (long long)h * dk + d]);
  __syncwarp();
  const int first = first_visible_key(p, window, extras.chunk);
  const float* bias_h = bias ? bias + (long long)h * bias_len : nullptr;
  float m = -INFINITY, l = 0.0f;
  float acc[8];                      // value channels lane, lane + 32, ... (v_dim <= 256)
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j] = 0.0f;
  for (int b = first / 32; b * 32 <= p; ++b) {
    const int key = b * 32 + lane;
    const bool seen = key >= first && key <= p;
    float s = -INFINITY;
    int page = -1;
    if (seen) page = cache_page(cache, seq, key);
    if (seen && page >= 0) {
      const T* kr = (const T*)cache.k + (long long)page * cache.page_stride +
                    ((long long)g * cache.page_tokens + key % cache.page_tokens) * dk;
      float dot = 0.0f;
      for (int d = 0; d < dk; ++d) dot += qs[d] * to_float(kr[d]);
      s = dot * scale;
      if (softcap > 0.0f) s = softcap * tanhf(s / softcap);
      if (bias_h) s += bias_h[min(p - key, bias_len - 1)];
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float w = (s == -INFINITY) ? 0.0f : expf(s - m_new);
    const float corr = (m == -INFINITY) ? 0.0f : expf(m - m_new);
    l = l * corr + warp_sum(w);
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] *= corr;
    m = m_new;
    const int last = min(31, p - b * 32);
    for (int kk = 0; kk <= last; ++kk) {
      const float wk = __shfl_sync(0xffffffffu, w, kk);
      const int pg = __shfl_sync(0xffffffffu, page, kk);
      if (wk == 0.0f || pg < 0) continue;
      const T* vr = (const T*)cache.v + (long long)pg * cache.page_stride +
                    ((long long)g * cache.page_tokens + (b * 32 + kk) % cache.page_tokens) * dv;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int d = lane + 32 * j;
        if (d < dv) acc[j] += wk * to_float(vr[d]);
      }
    }
  }
  float from_sum = 1.0f;       // what the sums taken against m become against the maximum with the sink
  if (extras.sink) {
    const float s = extras.sink[h], m_new = fmaxf(m, s);
    from_sum = m == -INFINITY ? 0.0f : expf(m - m_new);
    l = l * from_sum + expf(s - m_new);
  }
  const float inv = l > 0.0f ? out_scale * from_sum * head_gate<T>(extras, t, h) / l : 0.0f;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int d = lane + 32 * j;
    if (d < dv) out[(long long)t * out_stride + (long long)h * dv + d] = from_float<T>(acc[j] * inv);
  }
}

extern "C" int llm_biased_attention(const void* q, void* out, int dtype, long long out_stride, void* cache_k,
                                    void* cache_v, const int32_t* block_table, long long page_stride, int table_stride,
                                    int page_tokens, int kv_heads, int k_dim, int v_dim, const float* bias, int bias_len,
                                    const int32_t* positions, const int32_t* row_seq, int q_heads, int n_tokens,
                                    float scale, int window, float out_scale, float softcap, int chunk, const float* sink,
                                    const void* gate, long long gate_stride, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  LLM_HOST_CHECK(v_dim <= 256 && k_dim >= 1 && kv_heads >= 1 && q_heads % kv_heads == 0, ERR_BAD_SIZE);
  LLM_HOST_CHECK(bias == nullptr || bias_len >= 1, ERR_BAD_SIZE);
  const size_t smem = (size_t)BA_WARPS * k_dim * sizeof(float);
  LLM_HOST_CHECK(smem <= 48 * 1024, ERR_BAD_SIZE);
  PagedCacheKV cache{cache_k, cache_v, block_table, page_stride, table_stride, page_tokens, kv_heads, k_dim, v_dim};
  const AttentionExtras extras{chunk, sink, gate, gate_stride};
  const long long items = (long long)n_tokens * q_heads;
  const int blocks = (int)((items + BA_WARPS - 1) / BA_WARPS);
  if (dtype == DT_F32)
    launch_kernel(biased_attention_kernel<float>, blocks, BA_WARPS * 32, smem, stream, (const float*)q, (float*)out,
                  out_stride, cache, bias, bias_len, positions, row_seq, q_heads, n_tokens, scale, window, out_scale, softcap, extras);
  else if (dtype == DT_BF16)
    launch_kernel(biased_attention_kernel<__nv_bfloat16>, blocks, BA_WARPS * 32, smem, stream, (const __nv_bfloat16*)q,
                  (__nv_bfloat16*)out, out_stride, cache, bias, bias_len, positions, row_seq, q_heads, n_tokens, scale,
                  window, out_scale, softcap, extras);
  else
    return ERR_BAD_DTYPE;
  return launch_status();
}
