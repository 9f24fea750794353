// The gated delta rule of a step's portions in chunks of 64 tokens, on the tensor cores (mma.sync m16n8k16,
// bfloat16 operands, float32 sums), for bfloat16 steps.  Per head, with c_t the sum over the chunk's tokens up to
// t of the decays' logarithms (a vector over the key channels, or one number for all of them) and S the state at
// the chunk's start, the recurrence S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q written out is
//
//   L_tj = beta_t sum_i k_t[i] k_j[i] exp(c_t[i] - c_j[i])  (j < t),     T = (1 + L)^-1 diag(beta)
//   P_tj =        sum_i q_t[i] k_j[i] exp(c_t[i] - c_j[i])  (j <= t)
//   U  = T V - (T K') S              (K'_t = k_t exp(c_t): row t of U is u_t)
//   O  = Q' S + P U                  (Q'_t = q_t exp(c_t))
//   S <- diag(exp(c_last)) S + K''^T U    (K''_j = k_j exp(c_last - c_j))
//
// gated_delta_prepare, a block per (chunk, head), makes everything that does not depend on S: T V, T K', Q', K'',
// P and exp(c_last).  gated_delta_walk, a block per (request, head, PC value columns), walks a request's chunks
// in order with its columns of S in registers: the state's columns are independent, so blocks never wait on one
// another.  Decays are differences of logarithms that are never positive, so no factor overflows: a block of 16 x
// 16 pairs of tokens takes its factors against the last token ahead of its rows, exp(c_t - r) exp(r - c_j); inside a
// block on the diagonal the second one can grow, and where it would leave float32's range the pairs are formed
// one by one.  Every product's operands are two bfloat16 numbers each, a rounded one and what rounding left, of
// whose four products the three large ones are taken: 16 significant bits.  L's inverse, the decays and the state
// are float32.
//
// Built per key size with -DGD_DK (a multiple of 16 up to 128).

#include "gated_delta.cuh"

#ifndef GD_DK
#define GD_DK 128
#endif

namespace {

constexpr int DK = GD_DK;
static_assert(DK % 16 == 0 && DK >= 16 && DK <= 128, "GD_DK must be a multiple of 16 up to 128");
constexpr int L = 64;                  // tokens of a chunk
constexpr int LDF = DK + 4;            // float rows in shared memory
constexpr int LDT = L + 4;
constexpr int PREP_THREADS = 512;
constexpr float SAFE_RANGE = 80.0f;    // exp(80) times a chunk's sums stays inside float32

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {      // `valid` false fills zeros
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(bytes) : "memory");
}

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}

__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// two neighbouring numbers as a rounded pair and the pair of what rounding left
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

struct Tiles {              // what the prepare kernel leaves for the walk; `hl` bytes apart: rounded parts, then the rests
  __nv_bfloat16* w;         // [rows][heads * DK]  T K'
  __nv_bfloat16* q;         // Q'
  __nv_bfloat16* k;         // K''
  __nv_bfloat16* p;         // [rows][heads * L]
  float* u;                 // [rows][heads * dv]  T V
  float* end;               // [chunks][heads * DK]  exp(c_last)
  long long hl, p_hl;       // elements from a rounded part to its rest
};

// The number of a request's `chunk`-th chunk in the step: every chunk of the step has its own.
__device__ __forceinline__ long long chunk_id(int q_start, int seq, int chunk) { return (long long)(q_start / L) + seq + chunk; }

// ------------------------------------------------------------------------------------------- prepare

template <bool CHANNEL>
struct PrepShared {
  static constexpr int C_FLOATS = CHANNEL ? L * LDF : L;
  static constexpr size_t BYTES = sizeof(float) * (size_t)(2 * L * LDF + C_FLOATS + L * LDT + L);
};

template <bool CHANNEL>
__global__ void __launch_bounds__(PREP_THREADS)
gated_delta_prepare_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ vn,
                           DeltaGates gates, Tiles o, const int32_t* __restrict__ seq_q_start,
                           const int32_t* __restrict__ seq_q_len, int H, int G, int dv) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sm[];
  float* ks = sm;                                        // [L][LDF] k, later K'
  float* qs = ks + L * LDF;                              // [L][LDF]
  float* cs = qs + L * LDF;                              // [L][LDF] sums of logarithms, or [L]
  float* Lm = cs + PrepShared<CHANNEL>::C_FLOATS;        // [L][LDT] L, later (1 + L)^-1
  float* betas = Lm + L * LDT;                           // [L]
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int q_len = seq_q_len[seq];
  if (chunk * L >= q_len) return;
  const int count = min(L, q_len - chunk * L), q_start = seq_q_start[seq];
  const long long row0 = q_start + (long long)chunk * L;
  const int g = h / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3;
  const float neg_a = -expf(gates.a_log[h]);

  for (int e = tid; e < L * (DK / 4); e += PREP_THREADS) {
    const int t = e / (DK / 4), c = (e % (DK / 4)) * 4;
    const bool in = t < count;
    const long long src = (row0 + t) * ((long long)G * DK) + g * DK + c;
    *reinterpret_cast<float4*>(ks + t * LDF + c) = in ? *reinterpret_cast<const float4*>(kn + src) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    *reinterpret_cast<float4*>(qs + t * LDF + c) = in ? *reinterpret_cast<const float4*>(qn + src) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  if (CHANNEL) {
    for (int e = tid; e < L * DK; e += PREP_THREADS) {
      const int t = e / DK, i = e % DK;
      cs[t * LDF + i] = t < count ? delta_log_decay(gates, row0 + t, h * DK + i, neg_a) : 0.0f;
    }
  } else if (tid < L) {
    cs[tid] = tid < count ? delta_log_decay(gates, row0 + tid, h, neg_a) : 0.0f;
  }
  if (tid < L) betas[tid] = tid < count ? delta_beta(gates, row0 + tid, h) : 0.0f;
  __syncthreads();
  // ---- running sums over the chunk
  if (CHANNEL) {      // a thread per (channel, 16 tokens); then what the groups of 16 before have summed to
    const int i = tid % DK, s = tid / DK;
    float run = 0.0f;
    if (s < 4) {
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        run += cs[(s * 16 + t) * LDF + i];
        cs[(s * 16 + t) * LDF + i] = run;
      }
    }
    __syncthreads();
    float before = 0.0f;
    if (s < 4)
      for (int j = 0; j < s; ++j) before += cs[(j * 16 + 15) * LDF + i];
    __syncthreads();
    if (s > 0 && s < 4) {
#pragma unroll
      for (int t = 0; t < 16; ++t) cs[(s * 16 + t) * LDF + i] += before;
    }
  } else if (warp == 0) {      // a lane takes two neighbours
    const float v0 = cs[2 * lane], v1 = cs[2 * lane + 1];
    float run = v0 + v1;
#pragma unroll
    for (int s = 1; s < 32; s <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, run, s);
      if (lane >= s) run += up;
    }
    cs[2 * lane] = run - v1;
    cs[2 * lane + 1] = run;
  }
  __syncthreads();

  // ---- L and P, a warp per block of 16 x 16 pairs on or below the diagonal
  __nv_bfloat16* p_row = o.p + h * L;
  const long long p_stride = (long long)H * L;
  if (warp < 10) {
    const int a = warp < 1 ? 0 : (warp < 3 ? 1 : (warp < 6 ? 2 : 3)), b = warp - a * (a + 1) / 2;
    const int t0 = 16 * a + gq;
    bool one_by_one = false;
    if (CHANNEL && a == b) {
      float range = 0.0f;
      for (int i = lane; i < DK; i += 32) range = fmaxf(range, (a ? cs[(16 * a - 1) * LDF + i] : 0.0f) - cs[(16 * a + 15) * LDF + i]);
      one_by_one = warp_max(range) > SAFE_RANGE;
    }
    float kk[2][4] = {}, qk[2][4] = {};
    if (!one_by_one) {
#pragma unroll 2
      for (int s = 0; s < DK / 16; ++s) {
        uint32_t kh[4], kl[4], qh[4], ql[4];
#pragma unroll
        for (int f = 0; f < 4; ++f) {      // rows gq, gq + 8 of columns 2 tq, then of columns 2 tq + 8
          const int t = t0 + (f & 1) * 8, c = s * 16 + tq * 2 + (f >> 1) * 8;
          float2 k2 = *reinterpret_cast<const float2*>(ks + t * LDF + c), q2 = *reinterpret_cast<const float2*>(qs + t * LDF + c);
          if (CHANNEL) {
            const float2 ct = *reinterpret_cast<const float2*>(cs + t * LDF + c);
            const float2 r = a ? *reinterpret_cast<const float2*>(cs + (16 * a - 1) * LDF + c) : make_float2(0.0f, 0.0f);
            const float e0 = expf(ct.x - r.x), e1 = expf(ct.y - r.y);
            k2.x *= e0; k2.y *= e1;
            q2.x *= e0; q2.y *= e1;
          }
          split2(k2.x, k2.y, kh[f], kl[f]);
          split2(q2.x, q2.y, qh[f], ql[f]);
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int f = 0; f < 2; ++f) {
            const int j = 16 * b + nt * 8 + gq, c = s * 16 + tq * 2 + f * 8;
            float2 k2 = *reinterpret_cast<const float2*>(ks + j * LDF + c);
            if (CHANNEL) {
              const float2 cj = *reinterpret_cast<const float2*>(cs + j * LDF + c);
              const float2 r = a ? *reinterpret_cast<const float2*>(cs + (16 * a - 1) * LDF + c) : make_float2(0.0f, 0.0f);
              k2.x *= expf(r.x - cj.x);
              k2.y *= expf(r.y - cj.y);
            }
            split2(k2.x, k2.y, bh[f], bl[f]);
          }
          mma_bf16(kk[nt], kh, bh[0], bh[1]);
          mma_bf16(kk[nt], kh, bl[0], bl[1]);
          mma_bf16(kk[nt], kl, bh[0], bh[1]);
          mma_bf16(qk[nt], qh, bh[0], bh[1]);
          mma_bf16(qk[nt], qh, bl[0], bl[1]);
          mma_bf16(qk[nt], ql, bh[0], bh[1]);
        }
      }
    } else {
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = t0 + (e >> 1) * 8, j = 16 * b + nt * 8 + tq * 2 + (e & 1);
          if (j > t) continue;
          float x = 0.0f, y = 0.0f;
          for (int i = 0; i < DK; ++i) {
            const float f = ks[j * LDF + i] * expf(cs[t * LDF + i] - cs[j * LDF + i]);
            x = fmaf(ks[t * LDF + i], f, x);
            y = fmaf(qs[t * LDF + i], f, y);
          }
          kk[nt][e] = x;
          qk[nt][e] = y;
        }
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = t0 + r * 8, j = 16 * b + nt * 8 + tq * 2;
        float pv[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float f = CHANNEL ? 1.0f : (j + e <= t ? expf(cs[t] - cs[j + e]) : 0.0f);
          pv[e] = j + e <= t ? qk[nt][r * 2 + e] * f : 0.0f;
          Lm[t * LDT + j + e] = j + e < t ? betas[t] * kk[nt][r * 2 + e] * f : 0.0f;
        }
        if (t < count) {
          uint32_t hi, lo;
          split2(pv[0], pv[1], hi, lo);
          __nv_bfloat16* dst = p_row + (row0 + t) * p_stride + j;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + o.p_hl) = lo;
        }
      }
  }
  __syncthreads();

  // ---- Q', K'' and (in place of k) K'; the decay over the chunk
  for (int e = tid; e < L * (DK / 4); e += PREP_THREADS) {
    const int t = e / (DK / 4), c = (e % (DK / 4)) * 4;
    float kd[4], qd[4], kend[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const float ct = CHANNEL ? cs[t * LDF + c + x] : cs[t], last = CHANNEL ? cs[(L - 1) * LDF + c + x] : cs[L - 1];
      const float k = ks[t * LDF + c + x], f = expf(ct);
      kd[x] = k * f;
      qd[x] = qs[t * LDF + c + x] * f;
      kend[x] = k * expf(last - ct);
    }
    *reinterpret_cast<float4*>(ks + t * LDF + c) = make_float4(kd[0], kd[1], kd[2], kd[3]);
    if (t < count) {
      const long long at = (row0 + t) * ((long long)H * DK) + h * DK + c;
      uint2 hi, lo;
      split2(qd[0], qd[1], hi.x, lo.x);
      split2(qd[2], qd[3], hi.y, lo.y);
      *reinterpret_cast<uint2*>(o.q + at) = hi;
      *reinterpret_cast<uint2*>(o.q + o.hl + at) = lo;
      split2(kend[0], kend[1], hi.x, lo.x);
      split2(kend[2], kend[3], hi.y, lo.y);
      *reinterpret_cast<uint2*>(o.k + at) = hi;
      *reinterpret_cast<uint2*>(o.k + o.hl + at) = lo;
    }
  }
  if (tid < DK)
    o.end[chunk_id(q_start, seq, chunk) * ((long long)H * DK) + h * DK + tid] = expf(CHANNEL ? cs[(L - 1) * LDF + tid] : cs[L - 1]);

  // ---- (1 + L)^-1 in place: the blocks on the diagonal by substitution, a lane per column ...
  if (warp < 4 && lane < 16) {
    float x[16];
    const float* l = Lm + (16 * warp) * LDT + 16 * warp;
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float v = t == lane ? 1.0f : 0.0f;
#pragma unroll
      for (int s = 0; s < t; ++s) v = fmaf(-l[t * LDT + s], x[s], v);
      x[t] = v;
    }
    __syncwarp(0xffffu);
#pragma unroll
    for (int t = 0; t < 16; ++t) Lm[(16 * warp + t) * LDT + 16 * warp + lane] = x[t];
  }
  __syncthreads();
  // ... then row of blocks by row of blocks: T_ab = -T_aa sum_c L_ac T_cb
  for (int a = 1; a < 4; ++a) {
    float x[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int e = tid + y * PREP_THREADS;
      x[y] = 0.0f;
      if (e < a * 256) {
        const int t = (e >> 4) & 15, j = (e >> 8) * 16 + (e & 15);
        for (int s = (j >> 4) * 16; s < 16 * a; ++s) x[y] = fmaf(Lm[(16 * a + t) * LDT + s], Lm[s * LDT + j], x[y]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int e = tid + y * PREP_THREADS;
      if (e < a * 256) Lm[(16 * a + ((e >> 4) & 15)) * LDT + (e >> 8) * 16 + (e & 15)] = x[y];
    }
    __syncthreads();
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int e = tid + y * PREP_THREADS;
      x[y] = 0.0f;
      if (e < a * 256) {
        const int t = (e >> 4) & 15, j = (e >> 8) * 16 + (e & 15);
#pragma unroll
        for (int s = 0; s < 16; ++s) x[y] = fmaf(-Lm[(16 * a + t) * LDT + 16 * a + s], Lm[(16 * a + s) * LDT + j], x[y]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int e = tid + y * PREP_THREADS;
      if (e < a * 256) Lm[(16 * a + ((e >> 4) & 15)) * LDT + (e >> 8) * 16 + (e & 15)] = x[y];
    }
    __syncthreads();
  }

  // ---- T K' and T V with T = (1 + L)^-1 diag(beta), a warp per 16 rows and 16 columns
  const int tasks = 4 * (DK + dv) / 16;
  for (int task = warp; task < tasks; task += PREP_THREADS / 32) {
    const int m = 3 - (task & 3), n0 = (task >> 2) * 16;
    const bool is_w = n0 < DK;
    float acc[2][4] = {};
    for (int kk = 0; kk <= m; ++kk) {
      uint32_t th[4], tl[4];
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int t = 16 * m + gq + (f & 1) * 8, j = kk * 16 + tq * 2 + (f >> 1) * 8;
        split2(Lm[t * LDT + j] * betas[j], Lm[t * LDT + j + 1] * betas[j + 1], th[f], tl[f]);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int f = 0; f < 2; ++f) {
          const int j = kk * 16 + tq * 2 + f * 8;
          float v0, v1;
          if (is_w) {
            const int c = n0 + nt * 8 + gq;
            v0 = ks[j * LDF + c];
            v1 = ks[(j + 1) * LDF + c];
          } else {
            const long long src = (row0 + j) * ((long long)H * dv) + (long long)h * dv + (n0 - DK) + nt * 8 + gq;
            v0 = j < count ? vn[src] : 0.0f;
            v1 = j + 1 < count ? vn[src + (long long)H * dv] : 0.0f;
          }
          split2(v0, v1, bh[f], bl[f]);
        }
        mma_bf16(acc[nt], th, bh[0], bh[1]);
        mma_bf16(acc[nt], th, bl[0], bl[1]);
        mma_bf16(acc[nt], tl, bh[0], bh[1]);
      }
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = 16 * m + gq + r * 8;
        if (t >= count) continue;
        if (is_w) {
          __nv_bfloat16* dst = o.w + (row0 + t) * ((long long)H * DK) + h * DK + n0 + nt * 8 + tq * 2;
          uint32_t hi, lo;
          split2(acc[nt][r * 2], acc[nt][r * 2 + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + o.hl) = lo;
        } else {
          *reinterpret_cast<float2*>(o.u + (row0 + t) * ((long long)H * dv) + (long long)h * dv + (n0 - DK) + nt * 8 + tq * 2) =
              make_float2(acc[nt][r * 2], acc[nt][r * 2 + 1]);
        }
      }
  }
}

// ------------------------------------------------------------------------------------------- walk

constexpr int WARPS = 4, THREADS = WARPS * 32;
constexpr int LDN = DK + 8, LDP = L + 8;          // padded bfloat16 rows (conflict-free ldmatrix)
constexpr int MT_N = DK / 16;                     // row tiles of the state
constexpr int MTW = (MT_N + WARPS - 1) / WARPS;   // of which a warp owns at most this many

template <int PC>
struct WalkShared {
  static constexpr int LDC = PC + 8;
  static constexpr size_t BYTES = 2 * (size_t)(6 * L * LDN + 2 * L * LDP + 2 * DK * LDC + 2 * L * LDC) + 4 * DK;
};

template <int PC>
__global__ void __launch_bounds__(THREADS)
gated_delta_walk_kernel(Tiles in, float* __restrict__ state, float* __restrict__ out, const int32_t* __restrict__ seq_slot,
                        const int32_t* __restrict__ seq_q_start, const int32_t* __restrict__ seq_q_len, int H, int dv) {
  pdl_launch_dependents();
  constexpr int LDC = WalkShared<PC>::LDC, NT = PC / 8;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* Ws = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [2][L][LDN]: rounded, rest (and so on below)
  __nv_bfloat16* Qs = Ws + 2 * L * LDN;
  __nv_bfloat16* Ks = Qs + 2 * L * LDN;
  __nv_bfloat16* Ps = Ks + 2 * L * LDN;                                // [2][L][LDP]
  __nv_bfloat16* Ss = Ps + 2 * L * LDP;                                // [2][DK][LDC]
  __nv_bfloat16* Us = Ss + 2 * DK * LDC;                               // [2][L][LDC]
  float* ends = reinterpret_cast<float*>(Us + 2 * L * LDC);            // [DK]
  pdl_wait();
  const int col0 = blockIdx.x * PC, h = blockIdx.y, seq = blockIdx.z;
  const int q_len = seq_q_len[seq];
  if (q_len <= 0) return;
  const int q_start = seq_q_start[seq];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3, mid = lane >> 3;
  float* S_g = state + (((long long)seq_slot[seq] * H + h) * DK) * dv + col0;
  const int n_chunks = (q_len + L - 1) / L;

  constexpr int CN = DK / 8;
  auto load_wq = [&](int ch) {
    if (ch < n_chunks) {
      const int count = min(L, q_len - ch * L);
      const long long row0 = q_start + (long long)ch * L;
      for (int i = threadIdx.x; i < L * CN; i += THREADS) {
        const int r = i / CN, c = (i % CN) * 8;
        const bool valid = r < count;
        const long long src = valid ? (row0 + r) * ((long long)H * DK) + h * DK + c : 0;
        cp_async16(Ws + r * LDN + c, in.w + src, valid);
        cp_async16(Ws + (L + r) * LDN + c, in.w + in.hl + src, valid);
        cp_async16(Qs + r * LDN + c, in.q + src, valid);
        cp_async16(Qs + (L + r) * LDN + c, in.q + in.hl + src, valid);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_pk = [&](int ch) {
    if (ch < n_chunks) {
      const int count = min(L, q_len - ch * L);
      const long long row0 = q_start + (long long)ch * L;
      for (int i = threadIdx.x; i < L * CN; i += THREADS) {
        const int r = i / CN, c = (i % CN) * 8;
        const bool valid = r < count;
        const long long src = valid ? (row0 + r) * ((long long)H * DK) + h * DK + c : 0;
        cp_async16(Ks + r * LDN + c, in.k + src, valid);
        cp_async16(Ks + (L + r) * LDN + c, in.k + in.hl + src, valid);
      }
      for (int i = threadIdx.x; i < L * (L / 8); i += THREADS) {
        const int r = i / (L / 8), c = (i % (L / 8)) * 8;
        const bool valid = r < count;
        const long long src = valid ? (row0 + r) * ((long long)H * L) + h * L + c : 0;
        cp_async16(Ps + r * LDP + c, in.p + src, valid);
        cp_async16(Ps + (L + r) * LDP + c, in.p + in.p_hl + src, valid);
      }
      const float* end = in.end + chunk_id(q_start, seq, ch) * ((long long)H * DK) + h * DK;
      for (int i = threadIdx.x; i < DK / 4; i += THREADS) cp_async16(ends + i * 4, end + i * 4, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float u0[NT][4];      // T V of this warp's rows, asked for one chunk ahead
  auto load_u = [&](int ch) {
    const int count = ch < n_chunks ? min(L, q_len - ch * L) : 0;
    const int t = warp * 16 + gq;
    const float* src = in.u + (q_start + (long long)ch * L + t) * ((long long)H * dv) + (long long)h * dv + col0 + tq * 2;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float2 v = t + r * 8 < count ? *reinterpret_cast<const float2*>(src + (long long)r * 8 * H * dv + nt * 8) : make_float2(0.0f, 0.0f);
        u0[nt][r * 2] = v.x;
        u0[nt][r * 2 + 1] = v.y;
      }
  };
  load_wq(0);
  load_pk(0);
  load_u(0);

  float sreg[MTW][NT][4];      // the state's tiles this warp owns, float32, for the whole walk
  auto keep_state = [&]() {    // ... and as the products' operand in shared memory
#pragma unroll
    for (int i = 0; i < MTW; ++i) {
      const int mt = warp + i * WARPS;
      if (mt >= MT_N) break;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          split2(sreg[i][nt][r * 2], sreg[i][nt][r * 2 + 1], hi, lo);
          const int at = (mt * 16 + gq + r * 8) * LDC + nt * 8 + tq * 2;
          *reinterpret_cast<uint32_t*>(Ss + at) = hi;
          *reinterpret_cast<uint32_t*>(Ss + DK * LDC + at) = lo;
        }
    }
  };
#pragma unroll
  for (int i = 0; i < MTW; ++i) {
    const int mt = warp + i * WARPS;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float2 v = mt < MT_N ? *reinterpret_cast<const float2*>(S_g + (long long)(mt * 16 + gq + r * 8) * dv + nt * 8 + tq * 2)
                                   : make_float2(0.0f, 0.0f);
        sreg[i][nt][r * 2] = v.x;
        sreg[i][nt][r * 2 + 1] = v.y;
      }
  }
  keep_state();
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();

  for (int ch = 0; ch < n_chunks; ++ch) {
    const int count = min(L, q_len - ch * L);
    const long long row0 = q_start + (long long)ch * L;
    // ---- U = T V - W S and O = Q' S, this warp's 16 tokens
    float ws[NT][4] = {}, acc[NT][4] = {};
#pragma unroll
    for (int s = 0; s < DK / 16; ++s) {
      uint32_t wh[4], wl[4], qh[4], ql[4];
      const int at = (warp * 16 + (lane & 15)) * LDN + s * 16 + (lane >> 4) * 8;
      ldmatrix_x4(wh, Ws + at);
      ldmatrix_x4(wl, Ws + L * LDN + at);
      ldmatrix_x4(qh, Qs + at);
      ldmatrix_x4(ql, Qs + L * LDN + at);
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        uint32_t sh[4], sl[4];
        const int sat = (s * 16 + (mid & 1) * 8 + (lane & 7)) * LDC + (nt + (mid >> 1)) * 8;
        ldmatrix_x4_trans(sh, Ss + sat);
        ldmatrix_x4_trans(sl, Ss + DK * LDC + sat);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          mma_bf16(ws[nt + x], wh, sh[x * 2], sh[x * 2 + 1]);
          mma_bf16(acc[nt + x], qh, sh[x * 2], sh[x * 2 + 1]);
          mma_bf16(ws[nt + x], wl, sh[x * 2], sh[x * 2 + 1]);
          mma_bf16(acc[nt + x], ql, sh[x * 2], sh[x * 2 + 1]);
          mma_bf16(ws[nt + x], wh, sl[x * 2], sl[x * 2 + 1]);
          mma_bf16(acc[nt + x], qh, sl[x * 2], sl[x * 2 + 1]);
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        uint32_t hi, lo;
        split2(u0[nt][r * 2] - ws[nt][r * 2], u0[nt][r * 2 + 1] - ws[nt][r * 2 + 1], hi, lo);
        const int at = (warp * 16 + gq + r * 8) * LDC + nt * 8 + tq * 2;
        *reinterpret_cast<uint32_t*>(Us + at) = hi;
        *reinterpret_cast<uint32_t*>(Us + L * LDC + at) = lo;
      }
    asm volatile("cp.async.wait_group 0;" ::: "memory");      // this chunk's P and K''
    __syncthreads();      // U is whole; every warp has read the old state, W and Q'
    load_wq(ch + 1);
    load_u(ch + 1);
#pragma unroll
    for (int i = 0; i < MTW; ++i) {
      const int mt = warp + i * WARPS;
      if (mt >= MT_N) break;
      const float e0 = ends[mt * 16 + gq], e1 = ends[mt * 16 + gq + 8];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        sreg[i][nt][0] *= e0; sreg[i][nt][1] *= e0;
        sreg[i][nt][2] *= e1; sreg[i][nt][3] *= e1;
      }
    }
    // ---- O += P U and S <- diag(exp(c_last)) S + K''^T U
#pragma unroll
    for (int kk = 0; kk < L / 16; ++kk) {
      uint32_t uh[NT / 2][4], ul[NT / 2][4];
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        const int at = (kk * 16 + (mid & 1) * 8 + (lane & 7)) * LDC + (nt + (mid >> 1)) * 8;
        ldmatrix_x4_trans(uh[nt / 2], Us + at);
        ldmatrix_x4_trans(ul[nt / 2], Us + L * LDC + at);
      }
      if (kk <= warp) {
        uint32_t ph[4], pl[4];
        const int at = (warp * 16 + (lane & 15)) * LDP + kk * 16 + (lane >> 4) * 8;
        ldmatrix_x4(ph, Ps + at);
        ldmatrix_x4(pl, Ps + L * LDP + at);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int f = nt / 2, x = (nt & 1) * 2;
          mma_bf16(acc[nt], ph, uh[f][x], uh[f][x + 1]);
          mma_bf16(acc[nt], pl, uh[f][x], uh[f][x + 1]);
          mma_bf16(acc[nt], ph, ul[f][x], ul[f][x + 1]);
        }
      }
#pragma unroll
      for (int i = 0; i < MTW; ++i) {
        const int mt = warp + i * WARPS;
        if (mt >= MT_N) break;
        uint32_t kh[4], kl[4];      // K''^T as the row operand: the stored [token][channel] tile, transposed on the way in
        const int at = (kk * 16 + (mid >> 1) * 8 + (lane & 7)) * LDN + mt * 16 + (mid & 1) * 8;
        ldmatrix_x4_trans(kh, Ks + at);
        ldmatrix_x4_trans(kl, Ks + L * LDN + at);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int f = nt / 2, x = (nt & 1) * 2;
          mma_bf16(sreg[i][nt], kh, uh[f][x], uh[f][x + 1]);
          mma_bf16(sreg[i][nt], kl, uh[f][x], uh[f][x + 1]);
          mma_bf16(sreg[i][nt], kh, ul[f][x], ul[f][x + 1]);
        }
      }
    }
    {
      const int t = warp * 16 + gq;
      float* dst = out + (row0 + t) * ((long long)H * dv) + (long long)h * dv + col0 + tq * 2;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          if (t + r * 8 < count)
            *reinterpret_cast<float2*>(dst + (long long)r * 8 * H * dv + nt * 8) = make_float2(acc[nt][r * 2], acc[nt][r * 2 + 1]);
    }
    keep_state();
    asm volatile("cp.async.wait_group 0;" ::: "memory");      // the next chunk's W and Q'
    __syncthreads();      // the new state is whole; every warp has read P, K'' and U
    load_pk(ch + 1);
  }
#pragma unroll
  for (int i = 0; i < MTW; ++i) {
    const int mt = warp + i * WARPS;
    if (mt >= MT_N) break;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<float2*>(S_g + (long long)(mt * 16 + gq + r * 8) * dv + nt * 8 + tq * 2) =
            make_float2(sreg[i][nt][r * 2], sreg[i][nt][r * 2 + 1]);
  }
}

}  // namespace

extern "C" int llm_gated_delta_prepare(const float* qn, const float* kn, const float* vn, const void* z, long long z_stride,
                                       int z_dtype, const void* b, long long b_stride, int b_dtype, const float* a_log,
                                       const float* dt_bias, int channel, void* w, void* q, void* k, long long hl, void* p,
                                       long long p_hl, float* u, float* end, const int32_t* seq_q_start,
                                       const int32_t* seq_q_len, int n_seqs, int max_q_len, int heads, int kv_heads, int dk,
                                       int dv, cudaStream_t stream) {
  if (n_seqs <= 0 || max_q_len <= 0) return 0;
  LLM_HOST_CHECK(dk == DK && dv >= 16 && dv % 16 == 0 && kv_heads >= 1 && heads % kv_heads == 0, ERR_BAD_SIZE);
  LLM_HOST_CHECK(heads <= 65535 && n_seqs <= 65535 && hl % 8 == 0 && p_hl % 8 == 0, ERR_BAD_SIZE);
  LLM_HOST_CHECK((z_dtype == DT_F32 || z_dtype == DT_BF16) && (b_dtype == DT_F32 || b_dtype == DT_BF16), ERR_BAD_DTYPE);
  LLM_HOST_CHECK((((uintptr_t)qn | (uintptr_t)kn | (uintptr_t)w | (uintptr_t)q | (uintptr_t)k | (uintptr_t)p | (uintptr_t)u |
                   (uintptr_t)end) & 15) == 0, ERR_BAD_ALIGN);
  const DeltaGates gates{z, z_stride, z_dtype, b, b_stride, b_dtype, a_log, dt_bias};
  const Tiles o{(__nv_bfloat16*)w, (__nv_bfloat16*)q, (__nv_bfloat16*)k, (__nv_bfloat16*)p, u, end, hl, p_hl};
  const dim3 grid((max_q_len + L - 1) / L, heads, n_seqs);
#define GO(CH)                                                                                                          \
  do {                                                                                                                  \
    constexpr size_t smem = PrepShared<CH>::BYTES;                                                                      \
    static bool configured = false;                                                                                     \
    if (!configured) {                                                                                                  \
      if (cudaFuncSetAttribute(gated_delta_prepare_kernel<CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != \
          cudaSuccess)                                                                                                  \
        return launch_status();                                                                                         \
      configured = true;                                                                                                \
    }                                                                                                                   \
    launch_kernel(gated_delta_prepare_kernel<CH>, grid, PREP_THREADS, smem, stream, qn, kn, vn, gates, o, seq_q_start,  \
                  seq_q_len, heads, kv_heads, dv);                                                                      \
  } while (0)
  if (channel) GO(true); else GO(false);
#undef GO
  return launch_status();
}

extern "C" int llm_gated_delta_walk(const void* w, const void* q, const void* k, long long hl, const void* p, long long p_hl,
                                    const float* u, const float* end, float* state, float* out, const int32_t* seq_slot,
                                    const int32_t* seq_q_start, const int32_t* seq_q_len, int n_seqs, int heads, int dk,
                                    int dv, int columns, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  LLM_HOST_CHECK(dk == DK && (columns == 16 || columns == 32) && dv % columns == 0, ERR_BAD_SIZE);
  LLM_HOST_CHECK(heads <= 65535 && n_seqs <= 65535 && hl % 8 == 0 && p_hl % 8 == 0, ERR_BAD_SIZE);
  LLM_HOST_CHECK((((uintptr_t)w | (uintptr_t)q | (uintptr_t)k | (uintptr_t)p | (uintptr_t)u | (uintptr_t)end | (uintptr_t)state |
                   (uintptr_t)out) & 15) == 0, ERR_BAD_ALIGN);
  const Tiles in{(__nv_bfloat16*)w, (__nv_bfloat16*)q, (__nv_bfloat16*)k, (__nv_bfloat16*)p, (float*)u, (float*)end, hl, p_hl};
  const dim3 grid(dv / columns, heads, n_seqs);
#define GO(PC)                                                                                                          \
  do {                                                                                                                  \
    constexpr size_t smem = WalkShared<PC>::BYTES;                                                                      \
    static bool configured = false;                                                                                     \
    if (!configured) {                                                                                                  \
      if (cudaFuncSetAttribute(gated_delta_walk_kernel<PC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) !=  \
          cudaSuccess)                                                                                                  \
        return launch_status();                                                                                         \
      configured = true;                                                                                                \
    }                                                                                                                   \
    launch_kernel(gated_delta_walk_kernel<PC>, grid, THREADS, smem, stream, in, state, out, seq_slot, seq_q_start,      \
                  seq_q_len, heads, dv);                                                                                \
  } while (0)
  if (columns == 16) GO(16); else GO(32);
#undef GO
  return launch_status();
}
