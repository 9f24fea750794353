// The gated delta rule with a matrix state per (request, head):
//
//   S <- g_t * S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t      (S dk x dv, float32)
//
// g_t is one number per head, or one per key channel (it then acts on the rows of S):
// g = exp(-exp(A_log) * softplus(z + dt_bias)); beta = sigmoid(b).  q, k and v are a projection's rows behind a
// short causal convolution per channel and silu; q and k are then divided by sqrt(sum of squares + unit_eps) per
// head, q also by sqrt(dk).  `heads` value heads share `kv_heads` query/key heads (head h reads h / (heads / kv_heads)).
//
// Kernels: gated_delta_operands (convolution, silu, unit vectors: float32 q, k, v of a step's tokens, or for the
// chunked walk the activations in bfloat16 with the unit vectors' factors beside them),
// gated_delta_scan (the walk over a step's tokens, any sizes, float32), gated_delta_step (steps of one token
// per request: convolution with the ring's update, unit vectors, decays, the state in place, the norm per head
// and the output gate in one kernel).  Long portions of bfloat16 steps take gated_delta_chunked.cu instead of
// the scan.  The convolution's last inputs per request live in a state slot as a ring of `taps` entries indexed
// by position % taps.  Everything after the stored projections is float32.

#include "gated_delta.cuh"
#include "short_conv.cuh"

// ------------------------------------------------------------------------------------------- operands

// One block per token.  u: the projection's rows [q: G dk | k: G dk | v: H dv | ...].  With `compact`: the
// activations rounded to bfloat16, [rows][q | k | v], and in `lengths` [rows][2 G] what makes unit vectors of the
// rounded q and k heads, 1 / sqrt(sum of squares + unit_eps), of q also / sqrt(dk).
template <typename T>
__global__ void __launch_bounds__(256)
gated_delta_operands_kernel(const T* __restrict__ u, long long u_stride, const float* __restrict__ conv_w, int taps,
                            const float* __restrict__ ring, float* __restrict__ qn, float* __restrict__ kn,
                            float* __restrict__ vn, const int32_t* __restrict__ positions,
                            const int32_t* __restrict__ row_seq, const int32_t* __restrict__ seq_slot,
                            const int32_t* __restrict__ seq_q_start, int G, int dk, int vd, float unit_eps, float q_scale,
                            __nv_bfloat16* __restrict__ compact, float* __restrict__ lengths) {
  pdl_launch_dependents();
  extern __shared__ float ys[];      // [2 G dk] q and k after convolution and silu
  const int kd = G * dk, C = 2 * kd + vd;
  pdl_wait();
  const int t = blockIdx.x;
  const int seq = row_seq[t], p = positions[t];
  const int p0 = p - (t - seq_q_start[seq]);
  const int hist = taps - 1;
  const float* ring_slot = ring + (long long)seq_slot[seq] * taps * C;
  const T* row = u + (long long)t * u_stride;
  const bool inside = p - hist >= p0;      // all taps inside the step's own rows
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    float y = 0.0f;
    const float* w = conv_w + (long long)c * taps;
    if (inside) {
      const T* col = row + c - (long long)hist * u_stride;
      for (int j = 0; j < taps; ++j) y += w[j] * to_float(col[(long long)j * u_stride]);
    } else {
      for (int j = 0; j < taps; ++j) {
        const int x = p - hist + j;
        if (x < 0) continue;
        y += w[j] * (x >= p0 ? to_float(u[(long long)(t - (p - x)) * u_stride + c]) : ring_slot[(long long)(x % taps) * C + c]);
      }
    }
    y = delta_silu(y);
    if (compact) {
      const __nv_bfloat16 r = __float2bfloat16_rn(y);
      compact[(long long)t * C + c] = r;
      y = __bfloat162float(r);
    }
    if (c < 2 * kd) ys[c] = y;
    else if (compact) continue;
    else vn[(long long)t * vd + (c - 2 * kd)] = y;
  }
  __syncthreads();
  const int lane = threadIdx.x & 31;
  for (int head = threadIdx.x >> 5; head < 2 * G; head += blockDim.x >> 5) {      // a warp per q or k head
    const float* x = ys + head * dk;
    float sq = 0.0f;
    for (int i = lane; i < dk; i += 32) sq += x[i] * x[i];
    const float s = (head < G ? q_scale : 1.0f) / sqrtf(warp_sum(sq) + unit_eps);
    if (compact) {
      if (lane == 0) lengths[(long long)t * 2 * G + head] = s;
      continue;
    }
    float* dst = (head < G ? qn + (long long)t * kd + head * dk : kn + (long long)t * kd + (head - G) * dk);
    for (int i = lane; i < dk; i += 32) dst[i] = x[i] * s;
  }
}

// The compact form with a thread per four channels that walks OPER_ROWS rows: bfloat16, key heads of 16 to 128
// entries (a power of two, so that a head's lanes sum its squares by shuffles), value sizes that are multiples of four.
#define OPER_ROWS 16
#define OPER_THREADS 128

template <int TAPS>
__global__ void __launch_bounds__(OPER_THREADS)
gated_delta_compact_kernel(const __nv_bfloat16* __restrict__ u, long long u_stride, const float* __restrict__ conv_w,
                           const float* __restrict__ ring, const int32_t* __restrict__ positions,
                           const int32_t* __restrict__ row_seq, const int32_t* __restrict__ seq_slot,
                           const int32_t* __restrict__ seq_q_start, int n_tokens, int G, int dk, int vd, float unit_eps,
                           float q_scale, __nv_bfloat16* __restrict__ compact, float* __restrict__ lengths) {
  pdl_launch_dependents();
  const int kd = G * dk, C = 2 * kd + vd;
  const int c = (blockIdx.y * OPER_THREADS + threadIdx.x) * 4;
  const bool live = c < C;
  const int cc = live ? c : 0;      // (idle lanes follow along on the first channels: the shuffles need every lane)
  ConvColumns<TAPS> conv;
  conv.load_weights(conv_w, cc);
  pdl_wait();
  const int t0 = blockIdx.x * OPER_ROWS, rows = min(OPER_ROWS, n_tokens - t0);
  const int lanes = dk / 4;
  const bool qk = (blockIdx.y * OPER_THREADS + (threadIdx.x & ~31)) * 4 < 2 * kd;      // the warp has a q or k head
  const bool first = live && c < 2 * kd && c % dk == 0;
  int seq = -1;
  for (int i0 = 0; i0 < rows; i0 += 4) {      // four rows' inputs are asked for together
    uint2 in[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) in[k] = conv_load4(u + (long long)(t0 + min(i0 + k, rows - 1)) * u_stride + cc);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (i0 + k >= rows) break;
      const int t = t0 + i0 + k, s = row_seq[t];
      if (s != seq) {
        seq = s;
        conv.history(u, u_stride, cc, t, positions[t], seq_q_start[s], ring + (long long)seq_slot[s] * TAPS * C, TAPS, C);
      }
      float y[4];
      conv.step(in[k], y);
#pragma unroll
      for (int x = 0; x < 4; ++x) y[x] = __fdividef(y[x], 1.0f + __expf(-y[x]));      // silu, to be rounded to bfloat16
      const uint2 raw = conv_pack4(y);
      if (live) *reinterpret_cast<uint2*>(compact + (long long)t * C + c) = raw;
      if (!qk) continue;
      const float4 r = conv_floats(raw);
      float sq = r.x * r.x + r.y * r.y + r.z * r.z + r.w * r.w;
      for (int o = lanes >> 1; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      if (first) lengths[(long long)t * 2 * G + c / dk] = (c < kd ? q_scale : 1.0f) / sqrtf(sq + unit_eps);
    }
  }
}

extern "C" int llm_gated_delta_operands(const void* u, int dtype, long long u_stride, const float* conv_w, int taps,
                                        const float* ring, float* qn, float* kn, float* vn, const int32_t* positions,
                                        const int32_t* row_seq, const int32_t* seq_slot, const int32_t* seq_q_start,
                                        int n_tokens, int kv_heads, int dk, int heads, int dv, float unit_eps, float q_scale,
                                        void* compact, float* lengths, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  LLM_HOST_CHECK(!compact || lengths, ERR_BAD_SIZE);
  LLM_HOST_CHECK(taps >= 1 && kv_heads >= 1 && dk >= 1 && heads >= 1 && dv >= 1, ERR_BAD_SIZE);
  const size_t smem = (size_t)2 * kv_heads * dk * sizeof(float);
  LLM_HOST_CHECK(smem <= 200 * 1024, ERR_BAD_SIZE);
  auto aligned = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) % bytes) == 0; };
  if (compact && dtype == DT_BF16 && taps <= 4 && dk >= 16 && dk <= 128 && (dk & (dk - 1)) == 0 && dv % 4 == 0 &&
      u_stride % 4 == 0 && aligned(u, 8) && aligned(conv_w, 16) && aligned(ring, 16) && aligned(compact, 8)) {
    const int C = 2 * kv_heads * dk + heads * dv;
    const dim3 grid((n_tokens + OPER_ROWS - 1) / OPER_ROWS, (C / 4 + OPER_THREADS - 1) / OPER_THREADS);
#define COMPACT(TAPS)                                                                                                 \
  launch_kernel(gated_delta_compact_kernel<TAPS>, grid, OPER_THREADS, 0, stream, (const __nv_bfloat16*)u, u_stride,    \
                conv_w, ring, positions, row_seq, seq_slot, seq_q_start, n_tokens, kv_heads, dk, heads * dv, unit_eps, \
                q_scale, (__nv_bfloat16*)compact, lengths)
    if (taps == 1) COMPACT(1); else if (taps == 2) COMPACT(2); else if (taps == 3) COMPACT(3); else COMPACT(4);
#undef COMPACT
    return launch_status();
  }
#define LAUNCH(T)                                                                                                       \
  do {                                                                                                                  \
    if (smem > 48 * 1024)                                                                                               \
      cudaFuncSetAttribute(gated_delta_operands_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
    launch_kernel(gated_delta_operands_kernel<T>, n_tokens, 256, smem, stream, (const T*)u, u_stride, conv_w, taps, ring, \
                  qn, kn, vn, positions, row_seq, seq_slot, seq_q_start, kv_heads, dk, heads * dv, unit_eps, q_scale,    \
                  (__nv_bfloat16*)compact, lengths);                                                                    \
  } while (0)
  if (dtype == DT_F32) LAUNCH(float);
  else if (dtype == DT_BF16) LAUNCH(__nv_bfloat16);
  else return ERR_BAD_DTYPE;
#undef LAUNCH
  return launch_status();
}

// ------------------------------------------------------------------------------------------- scan

// Grid (sequence, head, slice of value columns).  A warp's lanes are `ks` row groups times 32 / ks value columns;
// a thread owns rows kr, kr + ks, ... (ROWS of them) of one column.  Tokens come through shared memory SCAN_TOKENS
// at a time; the next ones' loads are not overlapped with the walk (the chunked kernels are the fast form).
#define SCAN_WARPS 4
#define SCAN_THREADS (SCAN_WARPS * 32)
#define SCAN_TOKENS 8

template <int ROWS, bool CHANNEL>
__global__ void __launch_bounds__(SCAN_THREADS)
gated_delta_scan_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ vn,
                        DeltaGates gates, float* __restrict__ state, float* __restrict__ out,
                        const int32_t* __restrict__ seq_slot, const int32_t* __restrict__ seq_q_start,
                        const int32_t* __restrict__ seq_q_len, int heads, int kv_heads, int dk, int dv, int ks) {
  pdl_launch_dependents();
  extern __shared__ float sm[];
  const int span = ROWS * ks;                        // rows the threads cover, at least dk; the rest reads zeros
  const int cols = SCAN_WARPS * (32 / ks);
  float* qs = sm;                                    // [SCAN_TOKENS][span]
  float* kk = qs + SCAN_TOKENS * span;
  float* as = kk + SCAN_TOKENS * span;               // [SCAN_TOKENS][span], or [SCAN_TOKENS]
  float* vs = as + SCAN_TOKENS * (CHANNEL ? span : 1);     // [SCAN_TOKENS][cols]
  float* bs = vs + SCAN_TOKENS * cols;               // [SCAN_TOKENS]
  pdl_wait();
  const int seq = blockIdx.x, h = blockIdx.y, g = h / (heads / kv_heads);
  const int n = seq_q_len[seq];
  if (n <= 0) return;
  const int row0 = seq_q_start[seq];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int kr = lane % ks, my_col = warp * (32 / ks) + lane / ks;
  const int col0 = blockIdx.z * cols, col = col0 + my_col;
  const bool live = col < dv;
  float* S_g = state + (((long long)seq_slot[seq] * heads + h) * dk) * dv;
  const float neg_a = -expf(gates.a_log[h]);
  float S[ROWS];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int i = kr + r * ks;
    S[r] = live && i < dk ? S_g[(long long)i * dv + col] : 0.0f;
  }
  for (int first = 0; first < n; first += SCAN_TOKENS) {
    const int count = min(SCAN_TOKENS, n - first);
    __syncthreads();      // the tokens before these have been walked
    for (int e = threadIdx.x; e < count * span; e += SCAN_THREADS) {
      const int t = e / span, i = e - t * span;
      const long long row = row0 + first + t;
      const bool in = i < dk;
      qs[e] = in ? qn[(row * kv_heads + g) * dk + i] : 0.0f;
      kk[e] = in ? kn[(row * kv_heads + g) * dk + i] : 0.0f;
      if (CHANNEL) as[e] = in ? expf(delta_log_decay(gates, row, h * dk + i, neg_a)) : 0.0f;
    }
    for (int e = threadIdx.x; e < count * cols; e += SCAN_THREADS) {
      const int t = e / cols, c = col0 + e % cols;
      vs[e] = c < dv ? vn[((long long)(row0 + first + t) * heads + h) * dv + c] : 0.0f;
    }
    if (threadIdx.x < count) {
      const long long row = row0 + first + threadIdx.x;
      bs[threadIdx.x] = delta_beta(gates, row, h);
      if (!CHANNEL) as[threadIdx.x] = expf(delta_log_decay(gates, row, h, neg_a));
    }
    __syncthreads();
    for (int t = 0; t < count; ++t) {
      const float* q = qs + t * span + kr;
      const float* k = kk + t * span + kr;
      float dot = 0.0f;
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        S[r] *= CHANNEL ? as[t * span + kr + r * ks] : as[t];
        dot = fmaf(S[r], k[r * ks], dot);
      }
      for (int o = ks >> 1; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
      const float w = bs[t] * (vs[t * cols + my_col] - dot);
      float acc = 0.0f;
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        S[r] = fmaf(k[r * ks], w, S[r]);
        acc = fmaf(S[r], q[r * ks], acc);
      }
      for (int o = ks >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (live && kr == 0) out[((long long)(row0 + first + t) * heads + h) * dv + col] = acc;
    }
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int i = kr + r * ks;
    if (live && i < dk) S_g[(long long)i * dv + col] = S[r];
  }
}

extern "C" int llm_gated_delta_scan(const float* qn, const float* kn, const float* vn, const void* z, long long z_stride,
                                    int z_dtype, const void* b, long long b_stride, int b_dtype, const float* a_log,
                                    const float* dt_bias, int channel, float* state, float* out, const int32_t* seq_slot,
                                    const int32_t* seq_q_start, const int32_t* seq_q_len, int n_seqs, int heads,
                                    int kv_heads, int dk, int dv, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  LLM_HOST_CHECK(heads >= 1 && heads <= 65535 && kv_heads >= 1 && heads % kv_heads == 0 && dk >= 1 && dk <= 1024 && dv >= 1,
                 ERR_BAD_SIZE);
  LLM_HOST_CHECK((z_dtype == DT_F32 || z_dtype == DT_BF16) && (b_dtype == DT_F32 || b_dtype == DT_BF16), ERR_BAD_DTYPE);
  const int rows = dk <= 64 ? 8 : (dk <= 512 ? 16 : 32);
  int ks = 1;
  while (ks * rows < dk) ks <<= 1;          // row groups: a power of two, at most 32
  const int span = rows * ks, cols = SCAN_WARPS * (32 / ks);
  const size_t smem = sizeof(float) * SCAN_TOKENS * (size_t)(2 * span + (channel ? span : 1) + cols + 1);
  const dim3 grid(n_seqs, heads, (dv + cols - 1) / cols);
  LLM_HOST_CHECK(grid.z <= 65535 && smem <= 200 * 1024, ERR_BAD_SIZE);
  const DeltaGates gates{z, z_stride, z_dtype, b, b_stride, b_dtype, a_log, dt_bias};
#define GO(ROWS, CH)                                                                                                  \
  do {                                                                                                                \
    if (smem > 48 * 1024)                                                                                             \
      cudaFuncSetAttribute(gated_delta_scan_kernel<ROWS, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    launch_kernel(gated_delta_scan_kernel<ROWS, CH>, grid, SCAN_THREADS, smem, stream, qn, kn, vn, gates, state, out,  \
                  seq_slot, seq_q_start, seq_q_len, heads, kv_heads, dk, dv, ks);                                     \
  } while (0)
  if (channel) {
    if (rows == 8) GO(8, true); else if (rows == 16) GO(16, true); else GO(32, true);
  } else {
    if (rows == 8) GO(8, false); else if (rows == 16) GO(16, false); else GO(32, false);
  }
#undef GO
  return launch_status();
}

// ---------------------------------------------------------------------------- one token per request

// Grid (sequence, head).  A thread owns rows rg, rg + R, ... (at most NR) of CV neighbouring value columns; W
// column groups make a column block, blocks of columns are walked in turn (one for most sizes).  The state rows of
// the first column block are asked for before anything else.  S^T k and S^T q are added over the R row groups in
// shared memory, in order.  A block of the kv head's first value head keeps the q and k channels' ring.
#define STEP_THREADS 512

struct DeltaStep {
  const void* u;               // [rows] x (q | k | v | ...)
  long long u_stride;
  const float* conv_w;
  int taps;
  float* ring;
  DeltaGates gates;
  float* state;
  const void* gate;            // [rows] x heads * dv: pre-activations of the output gate
  long long gate_stride;
  int gate_dtype, gate_silu;   // silu, or sigmoid
  const float* norm_w;         // [dv]
  void* out;                   // [rows] x heads * dv
  long long out_stride;
  const int32_t* positions;
  const int32_t* seq_slot;
  const int32_t* seq_q_start;
  int heads, kv_heads, dk, dv, write_ring;
  float unit_eps, q_scale, eps;
};

template <typename T, bool CHANNEL, int CV, int NR>
__global__ void __launch_bounds__(STEP_THREADS, NR * CV <= 32 ? 2 : 1) gated_delta_step_kernel(DeltaStep a, int W) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sm[];
  __shared__ float scratch[32];
  const int dk = a.dk, dv = a.dv, R = STEP_THREADS / W, wide = W * CV;
  float* part = sm;                          // [R][W * CV]
  float* xs = part + R * wide;               // [2 dk + dv] q, k, v after convolution and silu
  float* gs = xs + 2 * dk + dv;              // [dk] decays
  float* os = gs + dk;                       // [dv]
  pdl_wait();
  const int seq = blockIdx.x, h = blockIdx.y, share = a.heads / a.kv_heads, kvh = h / share;
  const int t = a.seq_q_start[seq], slot = a.seq_slot[seq], p = a.positions[t];
  const int tid = threadIdx.x, rg = tid / W, cg = tid - rg * W;
  float* S_g = a.state + (((long long)slot * a.heads + h) * dk) * dv;
  float S[NR][CV];
  auto load_state = [&](int c0) {
    const int col = c0 + cg * CV;
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int i = rg + r * R;
      const bool in = rg < R && i < dk && col < dv;
      if constexpr (CV == 4) {
        const float4 v = in ? *reinterpret_cast<const float4*>(S_g + (long long)i * dv + col) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        S[r][0] = v.x; S[r][1] = v.y; S[r][2] = v.z; S[r][3] = v.w;
      } else {
        S[r][0] = in ? S_g[(long long)i * dv + col] : 0.0f;
      }
    }
  };
  load_state(0);

  // ---- convolution, silu, the ring; decays
  const int kd = a.kv_heads * dk, C = 2 * kd + a.heads * dv, hist = a.taps - 1;
  const T* row = reinterpret_cast<const T*>(a.u) + (long long)t * a.u_stride;
  float* ring_slot = a.ring + (long long)slot * a.taps * C;
  const bool owner = kvh * share == h;
  for (int i = tid; i < 2 * dk + dv; i += STEP_THREADS) {
    const int c = i < dk ? kvh * dk + i : (i < 2 * dk ? kd + kvh * dk + (i - dk) : 2 * kd + h * dv + (i - 2 * dk));
    const float now = to_float(row[c]);
    const float* w = a.conv_w + (long long)c * a.taps;
    float y = 0.0f;
    for (int j = 0; j < hist; ++j) {
      const int x = p - hist + j;
      if (x >= 0) y += w[j] * ring_slot[(long long)(x % a.taps) * C + c];
    }
    y += w[hist] * now;
    if (a.write_ring && hist > 0 && (i >= 2 * dk || owner)) ring_slot[(long long)(p % a.taps) * C + c] = now;
    xs[i] = delta_silu(y);
  }
  const float neg_a = -expf(a.gates.a_log[h]);
  if (CHANNEL) {
    for (int i = tid; i < dk; i += STEP_THREADS) gs[i] = expf(delta_log_decay(a.gates, t, h * dk + i, neg_a));
  } else if (tid == 0) {
    gs[0] = expf(delta_log_decay(a.gates, t, h, neg_a));
  }
  __syncthreads();
  if (tid < 64) {      // warp 0: the length of q, warp 1: of k
    const float* x = xs + (tid >> 5) * dk;
    float sq = 0.0f;
    for (int i = tid & 31; i < dk; i += 32) sq += x[i] * x[i];
    sq = warp_sum(sq);
    if ((tid & 31) == 0) scratch[tid >> 5] = (tid == 0 ? a.q_scale : 1.0f) / sqrtf(sq + a.unit_eps);
  }
  __syncthreads();
  const float q_len = scratch[0], k_len = scratch[1], beta = delta_beta(a.gates, t, h);
  const float* qs = xs;
  const float* ks = xs + dk;
  const float* vs = xs + 2 * dk;

  for (int c0 = 0; c0 < dv; c0 += wide) {
    if (c0 > 0) load_state(c0);
    const int col = c0 + cg * CV;
    float acc[CV];
#pragma unroll
    for (int e = 0; e < CV; ++e) acc[e] = 0.0f;
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int i = rg + r * R;
      if (rg < R && i < dk) {
        const float g = CHANNEL ? gs[i] : gs[0], k = ks[i];
#pragma unroll
        for (int e = 0; e < CV; ++e) {
          S[r][e] *= g;
          acc[e] = fmaf(S[r][e], k, acc[e]);
        }
      }
    }
    if (rg < R) {
#pragma unroll
      for (int e = 0; e < CV; ++e) part[rg * wide + cg * CV + e] = acc[e];
    }
    __syncthreads();
    float w[CV];
#pragma unroll
    for (int e = 0; e < CV; ++e) {
      float sum = 0.0f;
      for (int k = 0; k < R; ++k) sum += part[k * wide + cg * CV + e];
      w[e] = col + e < dv ? beta * (vs[col + e] - sum * k_len) * k_len : 0.0f;      // u_t times the key's 1 / length
      acc[e] = 0.0f;
    }
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int i = rg + r * R;
      if (rg < R && i < dk) {
        const float k = ks[i], q = qs[i];
#pragma unroll
        for (int e = 0; e < CV; ++e) {
          S[r][e] = fmaf(k, w[e], S[r][e]);
          acc[e] = fmaf(S[r][e], q, acc[e]);
        }
        if (col < dv) {
          if constexpr (CV == 4)
            *reinterpret_cast<float4*>(S_g + (long long)i * dv + col) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
          else
            S_g[(long long)i * dv + col] = S[r][0];
        }
      }
    }
    __syncthreads();      // every thread has read the sums of S^T k
    if (rg < R) {
#pragma unroll
      for (int e = 0; e < CV; ++e) part[rg * wide + cg * CV + e] = acc[e];
    }
    __syncthreads();
    for (int i = tid; i < wide; i += STEP_THREADS) {
      float sum = 0.0f;
      for (int k = 0; k < R; ++k) sum += part[k * wide + i];
      if (c0 + i < dv) os[c0 + i] = sum * q_len;
    }
    __syncthreads();
  }
  // ---- the head's norm, weight and gate
  float sq = 0.0f;
  for (int i = tid; i < dv; i += STEP_THREADS) sq += os[i] * os[i];
  const float s = 1.0f / sqrtf(block_sum(sq, scratch) / (float)dv + a.eps);
  T* dst = reinterpret_cast<T*>(a.out) + (long long)t * a.out_stride + h * dv;
  for (int i = tid; i < dv; i += STEP_THREADS) {
    const float z = load_any(a.gate, (long long)t * a.gate_stride + h * dv + i, a.gate_dtype);
    dst[i] = from_float<T>(os[i] * s * a.norm_w[i] * (a.gate_silu ? delta_silu(z) : delta_sigmoid(z)));
  }
}

// Column groups of a column block: as many as the value size has, so that a thread holds at most 16 rows.
static int step_width(int dk, int dv, int cv) {
  int w = (dv + cv - 1) / cv;
  if (w > STEP_THREADS) w = STEP_THREADS;
  while (w > 0 && (dk + STEP_THREADS / w - 1) / (STEP_THREADS / w) > 16) --w;
  return w;
}

extern "C" long long llm_gated_delta_step_shared_bytes(int dk, int dv) {
  const int cv = dv % 4 == 0 ? 4 : 1, w = step_width(dk, dv, cv);
  if (w < 1) return -1;
  return 4LL * ((STEP_THREADS / w) * w * cv + 3 * dk + 2 * dv);
}

extern "C" int llm_gated_delta_step(const void* u, int dtype, long long u_stride, const float* conv_w, int taps, float* ring,
                                    const void* z, long long z_stride, int z_dtype, const void* b, long long b_stride,
                                    int b_dtype, const float* a_log, const float* dt_bias, int channel, float* state,
                                    const void* gate, long long gate_stride, int gate_dtype, int gate_silu,
                                    const float* norm_w, void* out, long long out_stride, const int32_t* positions,
                                    const int32_t* seq_slot, const int32_t* seq_q_start, int n_seqs, int heads, int kv_heads,
                                    int dk, int dv, int write_ring, float unit_eps, float q_scale, float eps,
                                    cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  const long long smem = llm_gated_delta_step_shared_bytes(dk, dv);
  LLM_HOST_CHECK(smem > 0 && smem <= 200 * 1024 && taps >= 1 && heads <= 65535 && kv_heads >= 1 && heads % kv_heads == 0,
                 ERR_BAD_SIZE);
  LLM_HOST_CHECK((z_dtype == DT_F32 || z_dtype == DT_BF16) && (b_dtype == DT_F32 || b_dtype == DT_BF16) &&
                     (gate_dtype == DT_F32 || gate_dtype == DT_BF16), ERR_BAD_DTYPE);
  const int cv = dv % 4 == 0 ? 4 : 1, w = step_width(dk, dv, cv);
  LLM_HOST_CHECK(cv == 1 || ((uintptr_t)state % 16) == 0, ERR_BAD_ALIGN);
  const int rows = (dk + STEP_THREADS / w - 1) / (STEP_THREADS / w);
  DeltaStep a{u, u_stride, conv_w, taps, ring, DeltaGates{z, z_stride, z_dtype, b, b_stride, b_dtype, a_log, dt_bias}, state,
              gate, gate_stride, gate_dtype, gate_silu, norm_w, out, out_stride, positions, seq_slot, seq_q_start, heads,
              kv_heads, dk, dv, write_ring, unit_eps, q_scale, eps};
  const dim3 grid(n_seqs, heads);
#define GO(T, CH, CV, NR)                                                                                                \
  do {                                                                                                                   \
    if (smem > 48 * 1024)                                                                                                \
      cudaFuncSetAttribute(gated_delta_step_kernel<T, CH, CV, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    launch_kernel(gated_delta_step_kernel<T, CH, CV, NR>, grid, STEP_THREADS, (size_t)smem, stream, a, w);               \
  } while (0)
#define ROWS(T, CH, CV) do { if (rows <= 4) GO(T, CH, CV, 4); else if (rows <= 8) GO(T, CH, CV, 8); else GO(T, CH, CV, 16); } while (0)
#define FORM(T) do { if (channel) { if (cv == 4) ROWS(T, true, 4); else ROWS(T, true, 1); } \
                     else { if (cv == 4) ROWS(T, false, 4); else ROWS(T, false, 1); } } while (0)
  LLM_HOST_CHECK(rows <= 16, ERR_BAD_SIZE);
  if (dtype == DT_F32) FORM(float);
  else if (dtype == DT_BF16) FORM(__nv_bfloat16);
  else return ERR_BAD_DTYPE;
#undef FORM
#undef ROWS
#undef GO
  return launch_status();
}
