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
// one by one.  (One decay for all channels is a factor of the pair, behind an exact product of bfloat16 rows.)
// q, k and v arrive as bfloat16 activations, q and k with the float32 factors that make unit vectors of them.
// Every other operand of a product is two bfloat16 numbers, a rounded one and what rounding left, of whose four
// products the three large ones are taken: 16 significant bits.  Sums, decays and the state are float32.
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

constexpr int PREP_THREADS = 256;
constexpr int LDN = DK + 8;            // padded bfloat16 rows (conflict-free ldmatrix)
constexpr int LDF = DK + 4;            // float rows
constexpr int LDL = L + 4;             // float rows of L
constexpr int LDP = L + 8;             // bfloat16 rows of T and P
constexpr int LDD = 24;                // bfloat16 rows of a block on T's diagonal
constexpr float LOG2E = 1.4426950408889634f;
constexpr float SAFE_RANGE = 100.0f;   // 2^100 times a sum over the key channels stays inside float32

template <bool CHANNEL>
struct PrepShared {      // in bytes
  static constexpr size_t TILE = (size_t)L * LDN * 2;                    // k or q; later one part of K'
  static constexpr size_t SUMS = CHANNEL ? (size_t)L * LDF * 4 : L * 4 + TILE;      // sums of logarithms; later (or behind them) values
  static constexpr size_t BYTES = 2 * TILE + SUMS + (size_t)L * LDL * 4 + 2 * (size_t)L * LDP * 2 + 2 * 4 * 16 * LDD * 2 + 3 * L * 4;
};

// Blocks of three products of two-part operands.
__device__ __forceinline__ void mma_split(float (&c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0,
                                          uint32_t bh1, uint32_t bl0, uint32_t bl1) {
  mma_bf16(c, ah, bh0, bh1);
  mma_bf16(c, al, bh0, bh1);
  mma_bf16(c, ah, bl0, bl1);
}

__device__ __forceinline__ float2 pair_of(const __nv_bfloat16* p) {
  const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(p);
  return make_float2(__low2float(v), __high2float(v));
}

template <bool CHANNEL>
__global__ void __launch_bounds__(PREP_THREADS, 2)
gated_delta_prepare_kernel(const __nv_bfloat16* __restrict__ qkv, const float* __restrict__ lengths, DeltaGates gates, Tiles o,
                           const int32_t* __restrict__ seq_q_start, const int32_t* __restrict__ seq_q_len, int H, int G, int dv) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t smem_raw[];
  using Sh = PrepShared<CHANNEL>;
  __nv_bfloat16* kt = reinterpret_cast<__nv_bfloat16*>(smem_raw);                  // [L][LDN] k; later K' rounded
  __nv_bfloat16* qt = kt + L * LDN;                                                // [L][LDN] q; later what rounding K' left
  float* cs = reinterpret_cast<float*>(smem_raw + 2 * Sh::TILE);                   // [L][LDF] or [L], in units of log 2
  __nv_bfloat16* vt = reinterpret_cast<__nv_bfloat16*>(cs + (CHANNEL ? 0 : L));    // [L][LDN] a piece of the values
  float* Lm = reinterpret_cast<float*>(smem_raw + 2 * Sh::TILE + Sh::SUMS);        // [L][LDL]
  __nv_bfloat16* T = reinterpret_cast<__nv_bfloat16*>(Lm + L * LDL);               // [2][L][LDP] T: rounded, rest
  __nv_bfloat16* D = T + 2 * L * LDP;                                              // [2][4][16][LDD] (1 + L)^-1's diagonal blocks
  float* betas = reinterpret_cast<float*>(D + 2 * 4 * 16 * LDD);                   // [L]
  float* k_len = betas + L;                                                        // [L] factors that make unit vectors
  float* q_len_ = k_len + L;                                                       // [L]
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int q_len = seq_q_len[seq];
  if (chunk * L >= q_len) return;
  const int count = min(L, q_len - chunk * L), q_start = seq_q_start[seq];
  const long long row0 = q_start + (long long)chunk * L;
  const int g = h / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3, mid = lane >> 3;
  const long long C = 2LL * G * DK + (long long)H * dv;      // columns of qkv
  const float neg_a = -LOG2E * expf(gates.a_log[h]);

  for (int e = tid; e < L * (DK / 8); e += PREP_THREADS) {
    const int t = e / (DK / 8), c = (e % (DK / 8)) * 8;
    const bool in = t < count;
    const __nv_bfloat16* src = qkv + (in ? (row0 + t) * C + g * DK + c : 0);
    cp_async16(qt + t * LDN + c, src, in);
    cp_async16(kt + t * LDN + c, src + (in ? G * DK : 0), in);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (CHANNEL) {      // a channel per thread, eight tokens' numbers asked for together
    constexpr int STEP = PREP_THREADS / DK;
    const int i = tid % DK, first = tid / DK;
    if (first < STEP) {
      const float bias = gates.dt_bias[h * DK + i];
      for (int t0 = first; t0 < L; t0 += 8 * STEP) {
        float z[8];
#pragma unroll
        for (int k = 0; k < 8; ++k)
          z[k] = load_any(gates.z, (row0 + min(t0 + k * STEP, count - 1)) * gates.z_stride + h * DK + i, gates.z_dtype);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const int t = t0 + k * STEP;
          if (t < L) cs[t * LDF + i] = t < count ? neg_a * delta_softplus(z[k] + bias) : 0.0f;
        }
      }
    }
  } else if (tid < L) {
    cs[tid] = tid < count ? delta_log_decay(gates, row0 + tid, h, neg_a) : 0.0f;
  }
  if (tid < L) {
    const bool in = tid < count;
    betas[tid] = in ? delta_beta(gates, row0 + tid, h) : 0.0f;
    q_len_[tid] = in ? lengths[(row0 + tid) * 2 * G + g] : 0.0f;
    k_len[tid] = in ? lengths[(row0 + tid) * 2 * G + G + g] : 0.0f;
  }
  __syncthreads();
  // ---- running sums over the chunk
  if (CHANNEL) {      // a thread per (channel, 16 or 32 tokens); then what the groups before have summed to
    constexpr int PARTS = 4 * DK <= PREP_THREADS ? 4 : 2, LEN = L / PARTS;
    const int i = tid % DK, s = tid / DK;
    float run = 0.0f;
    if (s < PARTS) {
#pragma unroll 16
      for (int t = 0; t < LEN; ++t) {
        run += cs[(s * LEN + t) * LDF + i];
        cs[(s * LEN + t) * LDF + i] = run;
      }
    }
    __syncthreads();
    float before = 0.0f;
    if (s < PARTS)
      for (int j = 0; j < s; ++j) before += cs[(j * LEN + LEN - 1) * LDF + i];
    __syncthreads();
    if (s > 0 && s < PARTS) {
#pragma unroll 16
      for (int t = 0; t < LEN; ++t) cs[(s * LEN + t) * LDF + i] += before;
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
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();

  // ---- L and P, a warp per block of 16 x 16 pairs on or below the diagonal
  __nv_bfloat16* p_row = o.p + h * L;
  const long long p_stride = (long long)H * L;
  for (int task = warp; task < 10; task += PREP_THREADS / 32) {
    const int a = task < 1 ? 0 : (task < 3 ? 1 : (task < 6 ? 2 : 3)), b = task - a * (a + 1) / 2;
    const int t0 = 16 * a + gq;
    const float* ref = cs + (16 * a - 1) * LDF;      // (CHANNEL, a > 0)
    bool one_by_one = false;
    if (CHANNEL && a == b) {
      float range = 0.0f;
      for (int i = lane; i < DK; i += 32) range = fmaxf(range, (a ? ref[i] : 0.0f) - cs[(16 * a + 15) * LDF + i]);
      one_by_one = warp_max(range) > SAFE_RANGE;
    }
    float kk[2][4] = {}, qk[2][4] = {};
    if (!CHANNEL) {
#pragma unroll
      for (int s = 0; s < DK / 16; ++s) {
        uint32_t ka[4], qa[4], kb[4];
        const int at = (16 * a + (lane & 15)) * LDN + s * 16 + (lane >> 4) * 8;
        ldmatrix_x4(ka, kt + at);
        ldmatrix_x4(qa, qt + at);
        ldmatrix_x4(kb, kt + (16 * b + (mid >> 1) * 8 + (lane & 7)) * LDN + s * 16 + (mid & 1) * 8);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_bf16(kk[nt], ka, kb[nt * 2], kb[nt * 2 + 1]);
          mma_bf16(qk[nt], qa, kb[nt * 2], kb[nt * 2 + 1]);
        }
      }
    } else if (!one_by_one) {
#pragma unroll 2
      for (int s = 0; s < DK / 16; ++s) {
        uint32_t kh[4], kl[4], qh[4], ql[4];
        float2 r[2];
#pragma unroll
        for (int f = 0; f < 2; ++f)
          r[f] = a ? *reinterpret_cast<const float2*>(ref + s * 16 + tq * 2 + f * 8) : make_float2(0.0f, 0.0f);
#pragma unroll
        for (int f = 0; f < 4; ++f) {      // rows gq, gq + 8 of columns 2 tq, then of columns 2 tq + 8
          const int t = t0 + (f & 1) * 8, c = s * 16 + tq * 2 + (f >> 1) * 8;
          const float2 k2 = pair_of(kt + t * LDN + c), q2 = pair_of(qt + t * LDN + c);
          const float2 ct = *reinterpret_cast<const float2*>(cs + t * LDF + c);
          const float e0 = exp2_ftz(ct.x - r[f >> 1].x), e1 = exp2_ftz(ct.y - r[f >> 1].y);
          split2(k2.x * e0, k2.y * e1, kh[f], kl[f]);
          split2(q2.x * e0, q2.y * e1, qh[f], ql[f]);
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int f = 0; f < 2; ++f) {
            const int j = 16 * b + nt * 8 + gq, c = s * 16 + tq * 2 + f * 8;
            const float2 k2 = pair_of(kt + j * LDN + c), cj = *reinterpret_cast<const float2*>(cs + j * LDF + c);
            split2(k2.x * exp2_ftz(r[f].x - cj.x), k2.y * exp2_ftz(r[f].y - cj.y), bh[f], bl[f]);
          }
          mma_split(kk[nt], kh, kl, bh[0], bh[1], bl[0], bl[1]);
          mma_split(qk[nt], qh, ql, bh[0], bh[1], bl[0], bl[1]);
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
            const float f = __bfloat162float(kt[j * LDN + i]) * exp2_ftz(cs[t * LDF + i] - cs[j * LDF + i]);
            x = fmaf(__bfloat162float(kt[t * LDN + i]), f, x);
            y = fmaf(__bfloat162float(qt[t * LDN + i]), f, y);
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
          const float f = j + e <= t ? (CHANNEL ? 1.0f : exp2_ftz(cs[t] - cs[j + e])) * k_len[j + e] : 0.0f;
          pv[e] = j + e <= t ? qk[nt][r * 2 + e] * q_len_[t] * f : 0.0f;
          Lm[t * LDL + j + e] = j + e < t ? betas[t] * k_len[t] * kk[nt][r * 2 + e] * f : 0.0f;
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

  // ---- Q', K'' and (in place of k and q) K'; the decay over the chunk
  for (int e = tid; e < L * (DK / 8); e += PREP_THREADS) {
    const int t = e / (DK / 8), c = (e % (DK / 8)) * 8;
    const uint4 k8 = *reinterpret_cast<const uint4*>(kt + t * LDN + c), q8 = *reinterpret_cast<const uint4*>(qt + t * LDN + c);
    const __nv_bfloat16 *kp = reinterpret_cast<const __nv_bfloat16*>(&k8), *qp = reinterpret_cast<const __nv_bfloat16*>(&q8);
    const float kn = k_len[t], qn = q_len_[t];
    uint32_t hd[4], ld[4], hq[4], lq[4], he[4], le[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const float2 k2 = pair_of(kp + 2 * x), q2 = pair_of(qp + 2 * x);
      float f[2], last[2];
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const float ct = CHANNEL ? cs[t * LDF + c + 2 * x + y] : cs[t];
        f[y] = exp2_ftz(ct);
        last[y] = exp2_ftz((CHANNEL ? cs[(L - 1) * LDF + c + 2 * x + y] : cs[L - 1]) - ct);
      }
      split2(k2.x * kn * f[0], k2.y * kn * f[1], hd[x], ld[x]);
      split2(q2.x * qn * f[0], q2.y * qn * f[1], hq[x], lq[x]);
      split2(k2.x * kn * last[0], k2.y * kn * last[1], he[x], le[x]);
    }
    *reinterpret_cast<uint4*>(kt + t * LDN + c) = make_uint4(hd[0], hd[1], hd[2], hd[3]);
    *reinterpret_cast<uint4*>(qt + t * LDN + c) = make_uint4(ld[0], ld[1], ld[2], ld[3]);
    if (t < count) {
      const long long at = (row0 + t) * ((long long)H * DK) + h * DK + c;
      *reinterpret_cast<uint4*>(o.q + at) = make_uint4(hq[0], hq[1], hq[2], hq[3]);
      *reinterpret_cast<uint4*>(o.q + o.hl + at) = make_uint4(lq[0], lq[1], lq[2], lq[3]);
      *reinterpret_cast<uint4*>(o.k + at) = make_uint4(he[0], he[1], he[2], he[3]);
      *reinterpret_cast<uint4*>(o.k + o.hl + at) = make_uint4(le[0], le[1], le[2], le[3]);
    }
  }
  if (tid < DK)
    o.end[chunk_id(q_start, seq, chunk) * ((long long)H * DK) + h * DK + tid] = exp2_ftz(CHANNEL ? cs[(L - 1) * LDF + tid] : cs[L - 1]);
  // ---- (1 + L)^-1, the blocks on the diagonal by substitution, a lane per column ...
  if (warp >= PREP_THREADS / 32 - 4 && lane < 16) {
    const int a = warp - (PREP_THREADS / 32 - 4);
    float x[16];
    const float* l = Lm + (16 * a) * LDL + 16 * a;
    const float beta = betas[16 * a + lane];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float v = t == lane ? 1.0f : 0.0f;
#pragma unroll
      for (int s = 0; s < t; ++s) v = fmaf(-l[t * LDL + s], x[s], v);
      x[t] = v;
    }
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const __nv_bfloat16 xh = __float2bfloat16_rn(x[t]), yh = __float2bfloat16_rn(x[t] * beta);
      D[(a * 16 + t) * LDD + lane] = xh;
      D[(64 + a * 16 + t) * LDD + lane] = __float2bfloat16_rn(x[t] - __bfloat162float(xh));
      T[(16 * a + t) * LDP + 16 * a + lane] = yh;
      T[(L + 16 * a + t) * LDP + 16 * a + lane] = __float2bfloat16_rn(x[t] * beta - __bfloat162float(yh));
    }
  }
  __syncthreads();
  // the values of the first piece, into the place of the sums
  auto load_values = [&](int v0) {
    const int w8 = min(DK, dv - v0) / 8;
    for (int e = tid; e < L * w8; e += PREP_THREADS) {
      const int t = e / w8, c = (e % w8) * 8;
      const bool in = t < count;
      cp_async16(vt + t * LDN + c, qkv + (in ? (row0 + t) * C + 2LL * G * DK + (long long)h * dv + v0 + c : 0), in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_values(0);
  // ... then T = (1 + L)^-1 diag(beta) row of blocks by row of blocks, T_ab = -(1 + L)^-1_aa sum_c L_ac T_cb, a warp per
  // block.  The sum is formed transposed: its accumulators then are the second product's operand as they lie.
  for (int a = 1; a < 4; ++a) {
    if (warp < a) {
      const int b = warp;
      float xt[2][4] = {};      // [half of the rows t][...]: rows are the columns j of the block
      for (int c = b; c < a; ++c) {
        uint32_t th[4], tl[4];
        const int at = (16 * c + (mid >> 1) * 8 + (lane & 7)) * LDP + 16 * b + (mid & 1) * 8;
        ldmatrix_x4_trans(th, T + at);
        ldmatrix_x4_trans(tl, T + L * LDP + at);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int f = 0; f < 2; ++f) {
            const float2 l2 = *reinterpret_cast<const float2*>(Lm + (16 * a + nt * 8 + gq) * LDL + 16 * c + tq * 2 + f * 8);
            split2(l2.x, l2.y, bh[f], bl[f]);
          }
          mma_split(xt[nt], th, tl, bh[0], bh[1], bl[0], bl[1]);
        }
      }
      uint32_t dh[4], dl[4];
      const int at = (a * 16 + (lane & 15)) * LDD + (lane >> 4) * 8;
      ldmatrix_x4(dh, D + at);
      ldmatrix_x4(dl, D + 64 * LDD + at);
#pragma unroll
      for (int nj = 0; nj < 2; ++nj) {
        uint32_t bh[2], bl[2];
        split2(xt[0][nj * 2], xt[0][nj * 2 + 1], bh[0], bl[0]);
        split2(xt[1][nj * 2], xt[1][nj * 2 + 1], bh[1], bl[1]);
        float y[4] = {};
        mma_split(y, dh, dl, bh[0], bh[1], bl[0], bl[1]);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          split2(-y[r * 2], -y[r * 2 + 1], hi, lo);
          const int dst = (16 * a + gq + r * 8) * LDP + 16 * b + nj * 8 + tq * 2;
          *reinterpret_cast<uint32_t*>(T + dst) = hi;
          *reinterpret_cast<uint32_t*>(T + L * LDP + dst) = lo;
        }
      }
    }
    __syncthreads();
  }

  // ---- T K' and T V: a warp has rows of blocks m0 and 3 - m0 (five blocks of T together) and every fourth 16 columns
  const int m0 = warp & 1;
  uint32_t th[2][4][4], tl[2][4][4];
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    const int m = y ? 3 - m0 : m0;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk)
      if (kk <= m) {
        const int at = (16 * m + (lane & 15)) * LDP + kk * 16 + (lane >> 4) * 8;
        ldmatrix_x4(th[y][kk], T + at);
        ldmatrix_x4(tl[y][kk], T + L * LDP + at);
      }
  }
  for (int n0 = (warp >> 1) * 16; n0 < DK; n0 += 64) {
    float acc[2][2][4] = {};
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t bh[4], bl[4];
      const int at = (kk * 16 + (mid & 1) * 8 + (lane & 7)) * LDN + n0 + (mid >> 1) * 8;
      ldmatrix_x4_trans(bh, kt + at);
      ldmatrix_x4_trans(bl, qt + at);
#pragma unroll
      for (int y = 0; y < 2; ++y)
        if (kk <= (y ? 3 - m0 : m0)) {
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
            mma_split(acc[y][nt], th[y][kk], tl[y][kk], bh[nt * 2], bh[nt * 2 + 1], bl[nt * 2], bl[nt * 2 + 1]);
        }
    }
#pragma unroll
    for (int y = 0; y < 2; ++y)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = 16 * (y ? 3 - m0 : m0) + gq + r * 8;
        if (t >= count) continue;
        __nv_bfloat16* dst = o.w + (row0 + t) * ((long long)H * DK) + h * DK + n0 + tq * 2;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          uint32_t hi, lo;
          split2(acc[y][nt][r * 2], acc[y][nt][r * 2 + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(dst + nt * 8) = hi;
          *reinterpret_cast<uint32_t*>(dst + o.hl + nt * 8) = lo;
        }
      }
  }
  for (int v0 = 0; v0 < dv; v0 += DK) {
    if (v0 > 0) {
      __syncthreads();      // the piece before this one has been read
      load_values(v0);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int width = min(DK, dv - v0);
    for (int n0 = (warp >> 1) * 16; n0 < width; n0 += 64) {
      float acc[2][2][4] = {};
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t vf[4];
        ldmatrix_x4_trans(vf, vt + (kk * 16 + (mid & 1) * 8 + (lane & 7)) * LDN + n0 + (mid >> 1) * 8);
#pragma unroll
        for (int y = 0; y < 2; ++y)
          if (kk <= (y ? 3 - m0 : m0)) {
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
              mma_bf16(acc[y][nt], th[y][kk], vf[nt * 2], vf[nt * 2 + 1]);
              mma_bf16(acc[y][nt], tl[y][kk], vf[nt * 2], vf[nt * 2 + 1]);
            }
          }
      }
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = 16 * (y ? 3 - m0 : m0) + gq + r * 8;
          if (t >= count) continue;
          float* dst = o.u + (row0 + t) * ((long long)H * dv) + (long long)h * dv + v0 + n0 + tq * 2;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
            *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(acc[y][nt][r * 2], acc[y][nt][r * 2 + 1]);
        }
    }
  }
}

// ------------------------------------------------------------------------------------------- walk

constexpr int WARPS = 4;                          // warps that share the 64 tokens (and the state's row tiles)
constexpr int MT_N = DK / 16;                     // row tiles of the state
constexpr int MTW = (MT_N + WARPS - 1) / WARPS;   // of which a warp owns at most this many

template <int PC>
struct WalkShared {      // two chunks' W, K'' and decays; one's Q' and P; the state and U as operands
  static constexpr int LDC = PC + 8;
  static constexpr size_t BYTES = 2 * (size_t)(10 * L * LDN + 2 * L * LDP + 2 * DK * LDC + 2 * L * LDC) + 2 * 4 * DK;
};

// A block's warps, WARPS of them in each of two roles and every one with all PC columns: the first half makes U and carries
// the state, the second half makes the outputs.  A chunk's W and K'' arrive by cp.async while the chunk before it is
// worked on, Q' and P (which the state does not wait for) as soon as their one place is free; T V is read straight into
// the registers that need it, one chunk ahead.
template <int PC>
__global__ void __launch_bounds__(WARPS * 64)
gated_delta_walk_kernel(Tiles in, float* __restrict__ state, float* __restrict__ out, const int32_t* __restrict__ seq_slot,
                        const int32_t* __restrict__ seq_q_start, const int32_t* __restrict__ seq_q_len, int H, int dv) {
  pdl_launch_dependents();
  constexpr int LDC = WalkShared<PC>::LDC, NT = PC / 8, THREADS = WARPS * 64, KS = DK / 16;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* W0 = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [2 chunks][2][L][LDN]: rounded, rest (and so on below)
  __nv_bfloat16* K0 = W0 + 4 * L * LDN;                                // [2 chunks][2][L][LDN]
  __nv_bfloat16* Qs = K0 + 4 * L * LDN;                                // [2][L][LDN]
  __nv_bfloat16* Ps = Qs + 2 * L * LDN;                                // [2][L][LDP]
  __nv_bfloat16* Ss = Ps + 2 * L * LDP;                                // [2][DK][LDC]
  __nv_bfloat16* Us = Ss + 2 * DK * LDC;                               // [2][L][LDC]
  float* ends0 = reinterpret_cast<float*>(Us + 2 * L * LDC);           // [2 chunks][DK]
  pdl_wait();
  const int h = blockIdx.y, seq = blockIdx.z;
  const int q_len = seq_q_len[seq];
  if (q_len <= 0) return;
  const int q_start = seq_q_start[seq];
  const int warp = (threadIdx.x >> 5) % WARPS, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3, mid = lane >> 3;
  const bool carries = threadIdx.x < THREADS / 2;
  const int col0 = blockIdx.x * PC;
  float* S_g = state + (((long long)seq_slot[seq] * H + h) * DK) * dv + col0;
  const int n_chunks = (q_len + L - 1) / L;

  // rows of one chunk's tile of `in` (both parts), zero behind the request's last token
  auto load_tile = [&](__nv_bfloat16* dst, const __nv_bfloat16* from, int ch) {
    constexpr int CN = DK / 8;
    const int count = min(L, q_len - ch * L);
    const long long row0 = q_start + (long long)ch * L;
    for (int i = threadIdx.x; i < L * CN; i += THREADS) {
      const int r = i / CN, c = (i % CN) * 8;
      const bool valid = r < count;
      const long long src = valid ? (row0 + r) * ((long long)H * DK) + h * DK + c : 0;
      cp_async16(dst + r * LDN + c, from + src, valid);
      cp_async16(dst + (L + r) * LDN + c, from + in.hl + src, valid);
    }
  };
  auto load_wk = [&](int ch) {
    if (ch < n_chunks) {
      const int st = ch & 1;
      load_tile(W0 + st * 2 * L * LDN, in.w, ch);
      load_tile(K0 + st * 2 * L * LDN, in.k, ch);
      const float* end = in.end + chunk_id(q_start, seq, ch) * ((long long)H * DK) + h * DK;
      for (int i = threadIdx.x; i < DK / 4; i += THREADS) cp_async16(ends0 + st * DK + i * 4, end + i * 4, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_q = [&](int ch) {
    if (ch < n_chunks) load_tile(Qs, in.q, ch);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_p = [&](int ch) {
    const int count = min(L, q_len - ch * L);
    const long long row0 = q_start + (long long)ch * L;
    for (int i = threadIdx.x; i < L * (L / 8); i += THREADS) {
      const int r = i / (L / 8), c = (i % (L / 8)) * 8;
      const bool valid = r < count;
      const long long src = valid ? (row0 + r) * ((long long)H * L) + h * L + c : 0;
      cp_async16(Ps + r * LDP + c, in.p + src, valid);
      cp_async16(Ps + (L + r) * LDP + c, in.p + in.p_hl + src, valid);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float u0[NT][4];      // (carries) T V of this warp's rows
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
  load_wk(0);
  load_q(0);

  float sreg[MTW][NT][4];      // (carries) the state's tiles this warp owns, float32, for the whole walk
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
  if (carries) {
    load_u(0);
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
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();

  for (int ch = 0; ch < n_chunks; ++ch) {
    const int count = min(L, q_len - ch * L), st = ch & 1;
    const long long row0 = q_start + (long long)ch * L;
    const __nv_bfloat16 *Ws = W0 + st * 2 * L * LDN, *Ks = K0 + st * 2 * L * LDN;
    const float* ends = ends0 + st * DK;
    load_p(ch);
    load_wk(ch + 1);      // into the other set, which every warp left at the last chunk's end
    // ---- W S (for U = T V - W S) or Q' S (the outputs' first part), this warp's 16 tokens
    float acc[NT][4] = {};
    const __nv_bfloat16* As = carries ? Ws : Qs;
#pragma unroll
    for (int s = 0; s < KS; ++s) {
      uint32_t ah[4], al[4];
      const int at = (warp * 16 + (lane & 15)) * LDN + s * 16 + (lane >> 4) * 8;
      ldmatrix_x4(ah, As + at);
      ldmatrix_x4(al, As + L * LDN + at);
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        uint32_t sh[4], sl[4];
        const int sat = (s * 16 + (mid & 1) * 8 + (lane & 7)) * LDC + (nt + (mid >> 1)) * 8;
        ldmatrix_x4_trans(sh, Ss + sat);
        ldmatrix_x4_trans(sl, Ss + DK * LDC + sat);
#pragma unroll
        for (int x = 0; x < 2; ++x) mma_split(acc[nt + x], ah, al, sh[x * 2], sh[x * 2 + 1], sl[x * 2], sl[x * 2 + 1]);
      }
    }
    if (carries) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          split2(u0[nt][r * 2] - acc[nt][r * 2], u0[nt][r * 2 + 1] - acc[nt][r * 2 + 1], hi, lo);
          const int at = (warp * 16 + gq + r * 8) * LDC + nt * 8 + tq * 2;
          *reinterpret_cast<uint32_t*>(Us + at) = hi;
          *reinterpret_cast<uint32_t*>(Us + L * LDC + at) = lo;
        }
      load_u(ch + 1);
    }
    asm volatile("cp.async.wait_group 1;" ::: "memory");      // this chunk's P
    __syncthreads();      // U is whole; every warp has read the old state and Q'
    load_q(ch + 1);
    // ---- S <- diag(exp(c_last)) S + K''^T U, or the outputs' second part, P U
    if (carries) {
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
    }
#pragma unroll
    for (int kk = 0; kk < L / 16; ++kk) {
      if (!carries && kk > warp) break;
      uint32_t uh[NT / 2][4], ul[NT / 2][4];
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        const int uat = (kk * 16 + (mid & 1) * 8 + (lane & 7)) * LDC + (nt + (mid >> 1)) * 8;
        ldmatrix_x4_trans(uh[nt / 2], Us + uat);
        ldmatrix_x4_trans(ul[nt / 2], Us + L * LDC + uat);
      }
      if (carries) {
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
            const uint32_t *h2 = uh[nt / 2] + (nt & 1) * 2, *l2 = ul[nt / 2] + (nt & 1) * 2;
            mma_split(sreg[i][nt], kh, kl, h2[0], h2[1], l2[0], l2[1]);
          }
        }
      } else {
        uint32_t ph[4], pl[4];
        const int at = (warp * 16 + (lane & 15)) * LDP + kk * 16 + (lane >> 4) * 8;
        ldmatrix_x4(ph, Ps + at);
        ldmatrix_x4(pl, Ps + L * LDP + at);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const uint32_t *h2 = uh[nt / 2] + (nt & 1) * 2, *l2 = ul[nt / 2] + (nt & 1) * 2;
          mma_split(acc[nt], ph, pl, h2[0], h2[1], l2[0], l2[1]);
        }
      }
    }
    if (carries) {
      keep_state();
    } else {
      const int t = warp * 16 + gq;
      float* dst = out + (row0 + t) * ((long long)H * dv) + (long long)h * dv + col0 + tq * 2;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          if (t + r * 8 < count)
            *reinterpret_cast<float2*>(dst + (long long)r * 8 * H * dv + nt * 8) = make_float2(acc[nt][r * 2], acc[nt][r * 2 + 1]);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");      // the next chunk's W, K'' and Q'
    __syncthreads();      // the new state is whole; every warp has read this chunk's tiles and U
  }
  if (!carries) return;
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

extern "C" int llm_gated_delta_prepare(const void* qkv, const float* lengths, const void* z, long long z_stride,
                                       int z_dtype, const void* b, long long b_stride, int b_dtype, const float* a_log,
                                       const float* dt_bias, int channel, void* w, void* q, void* k, long long hl, void* p,
                                       long long p_hl, float* u, float* end, const int32_t* seq_q_start,
                                       const int32_t* seq_q_len, int n_seqs, int max_q_len, int heads, int kv_heads, int dk,
                                       int dv, cudaStream_t stream) {
  if (n_seqs <= 0 || max_q_len <= 0) return 0;
  LLM_HOST_CHECK(dk == DK && dv >= 16 && dv % 16 == 0 && kv_heads >= 1 && heads % kv_heads == 0, ERR_BAD_SIZE);
  LLM_HOST_CHECK(heads <= 65535 && n_seqs <= 65535 && hl % 8 == 0 && p_hl % 8 == 0, ERR_BAD_SIZE);
  LLM_HOST_CHECK((z_dtype == DT_F32 || z_dtype == DT_BF16) && (b_dtype == DT_F32 || b_dtype == DT_BF16), ERR_BAD_DTYPE);
  LLM_HOST_CHECK((((uintptr_t)qkv | (uintptr_t)w | (uintptr_t)q | (uintptr_t)k | (uintptr_t)p | (uintptr_t)u |
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
    launch_kernel(gated_delta_prepare_kernel<CH>, grid, PREP_THREADS, smem, stream, (const __nv_bfloat16*)qkv, lengths,  \
                  gates, o, seq_q_start, seq_q_len, heads, kv_heads, dv);                                               \
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
    launch_kernel(gated_delta_walk_kernel<PC>, grid, WARPS * 64, smem, stream, in, state, out, seq_slot, seq_q_start,      \
                  seq_q_len, heads, dv);                                                                                \
  } while (0)
  if (columns == 16) GO(16); else GO(32);
#undef GO
  return launch_status();
}
