// A gated delta rule: per head a d x dv matrix state S that decays, is corrected along the current key and read along the
// current query.  Everything behind the mixer's products is 32-bit; T is the activation type of the products' results.
//
// The mixer's input product leaves, per token, [q (G*d) | k (G*d) | v (H*dv)] from column x_off on (row stride ld) and one
// logit per head for beta (column b_off); the decay's pre-activation is one value per head, or one per (head, key channel),
// in rows of its own (`dec`, stride dec_ld).  Head h reads q and k of group h / (H/G).  Then
//
//     q, k, v   a short causal convolution per channel (shortconv.cuh), then silu
//     q, k      divided by sqrt(sum of squares + 1e-6) per head; q also times d^(-1/2)
//     beta      sigmoid(logit) ;   log g = -exp(A_log_h) * softplus(dec + dt_bias)      (per head or per key channel)
//     S <- g S ;  u = beta (v - S^T k) ;  S <- S + k u^T ;  o = S^T q
//     out       o / sqrt(mean over the head's dv of o^2 + eps) * norm_w * act(gate)     (act: silu or sigmoid; gate [H*dv])
//
// The state lives transposed, [slots, H, dv, dp] with dp = d rounded up to a multiple of four (the rows beyond d stay zero),
// so that a value column's key vector is one piece of memory: the lanes of a warp hold RPL neighbouring rows each of a few
// columns, and the sums over the key channels are warp sums.  Decays are applied as S + S * (g - 1) with g - 1 = expm1(log g):
// a decay close to one keeps its distance from one.
//
// A step of many tokens goes by groups of eight tokens.  With G_i the sum of the log decays of a group's tokens 0..i,
//
//     u_i = beta_i (v_i - (k_i e^{G_i})^T S0) - sum_{j<i} beta_i A_ij u_j ,    A_ij = sum_c k_i k_j e^{G_i - G_j}
//     o_i = (q_i e^{G_i})^T S0 + sum_{j<=i} P_ij u_j ,                         P_ij = sum_c q_i k_j e^{G_i - G_j}
//     S8  = e^{G_7} S0 + sum_j (k_j e^{G_7 - G_j}) u_j^T
//
// so the sixteen products with S0 of a group do not wait for one another and their warp sums are formed together; every
// exponent is a sum of log decays, hence never positive.
//
//   delta_prep    one block per (tile of a sequence's tokens, head): a warp a group; leaves a record per (group, head), vectors
//                 of dr = 32, 64, 128 or 256 floats (the key size rounded up, zeros behind it):
//                 [beta_i k_i e^{G_i}: 8 dr | q_i e^{G_i}: 8 dr | k_j e^{G_7-G_j}: 8 dr | expm1(G_7): dr | beta 8 |
//                 beta_i A_ij: 28 | P: 8 x 8].  Further blocks convolve v into [n, H, dvp] floats.
//   delta_walk    one block per (slice of value columns, head, sequence), the columns dealt to its warps: groups in order from
//                 the slot's state, records and v brought to shared memory ahead by cp.async; the sums of a warp and
//                 group are formed by one butterfly that leaves every lane one or two of them.  Leaves o [n, H*dv] and the
//                 slot's state.
//   delta_norm    one warp per (token, head): the norm over dv, the weight and the gate.  Further blocks store the convolution's
//                 last inputs in the ring (this launch runs behind the one that reads it).
//   delta_decode  one token per sequence: one block per (head, sequence) does all of it, the ring's new row included.
// Sequences with slot -1 (padding) are skipped (their output rows are zeros).  No block waits on another block; the only waits
// are cp.async.wait_group and __syncthreads.
#include "shortconv.cuh"
#include <math.h>

namespace {
constexpr float UNIT_EPS = 1e-6f;     // inside the root of the unit vectors' length: fixed by the rule
constexpr int GRP = 8;                // tokens of a group
constexpr int PAIRS = GRP * (GRP - 1) / 2;
constexpr int VECS = 3 * GRP + 1;     // vectors of a record
constexpr int SCAL = GRP + PAIRS + GRP * GRP;   // numbers behind them
constexpr int PREP_THREADS = 128;
constexpr int V_SPLIT = 4;            // blocks a tile's groups are dealt to while v is convolved
constexpr int WALK_WARPS = 4;
constexpr int WALK_STAGES = 4;        // records of the walk in shared memory at once
constexpr long long FEW_COLUMNS = 8 * 148;
constexpr int V_PAD = 16;             // rows of the convolved v are padded to whole blocks of columns
constexpr int DEC_COLS = 8;           // value columns a warp of the decode kernel holds at once
constexpr int DEC_THREADS = 512;
constexpr unsigned FULL = 0xffffffffu;

constexpr float LOG2E = 1.4426950408889634f, LN2 = 0.6931471805599453f;

// two to the power x, one instruction (2 ulp)
__device__ __forceinline__ float exp2_(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float sigmoidf_(float v) { return __fdividef(1.f, 1.f + exp2_(-LOG2E * v)); }
__device__ __forceinline__ float siluf_(float v) { return v * sigmoidf_(v); }
__device__ __forceinline__ float softplusf_(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
template <typename T> __device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<unsigned*>(&a);
  raw.y = *reinterpret_cast<unsigned*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}

__device__ __forceinline__ int seq_of(const int* __restrict__ cu_q, int n_seqs, int t) {
  int lo = 0, hi = n_seqs - 1;        // largest b with cu_q[b] <= t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// the first group's record of sequence b whose first packed token is t0: sequences take disjoint ranges in order
__device__ __forceinline__ size_t group_base(int t0, int b) { return (size_t)(((long long)t0 + (long long)(GRP - 1) * b) / GRP); }

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N)); }

// RPL neighbouring floats; rows behind dp read as zeros (dp is a multiple of four, RPL a divisor or a multiple of it)
template <int RPL>
__device__ __forceinline__ void load_rows(float (&v)[RPL], const float* p, int row0, int dp) {
  if constexpr (RPL >= 4) {
#pragma unroll
    for (int e = 0; e < RPL; e += 4) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (row0 + e < dp) x = *reinterpret_cast<const float4*>(p + row0 + e);
      v[e] = x.x; v[e + 1] = x.y; v[e + 2] = x.z; v[e + 3] = x.w;
    }
  } else if constexpr (RPL == 2) {
    float2 x = make_float2(0.f, 0.f);
    if (row0 < dp) x = *reinterpret_cast<const float2*>(p + row0);
    v[0] = x.x; v[1] = x.y;
  } else {
    v[0] = row0 < dp ? p[row0] : 0.f;
  }
}
template <int RPL>
__device__ __forceinline__ void store_rows(const float (&v)[RPL], float* p, int row0, int dp) {
  if constexpr (RPL >= 4) {
#pragma unroll
    for (int e = 0; e < RPL; e += 4)
      if (row0 + e < dp) *reinterpret_cast<float4*>(p + row0 + e) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
  } else if constexpr (RPL == 2) {
    if (row0 < dp) *reinterpret_cast<float2*>(p + row0) = make_float2(v[0], v[1]);
  } else {
    if (row0 < dp) p[row0] = v[0];
  }
}

// x[i] summed over the L lanes of a group, i < N (powers of two): lane l of the group is left with the sums of index
// l * N / L .. in x[0 .. N / L - 1] (N >= L), or with the sum of index l / (L / N) in x[0]
template <int N, int L>
__device__ __forceinline__ void butterfly(float (&x)[N], int l) {
  int n = N;
#pragma unroll
  for (int off = L / 2; off > 0; off >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = (l & off) != 0;
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        if (i < n) {
          const float send = up ? x[i] : x[i + n], keep = up ? x[i + n] : x[i];
          x[i] = keep + __shfl_xor_sync(FULL, send, off);
        }
      }
    } else {
      x[0] += __shfl_xor_sync(FULL, x[0], off);
    }
  }
}

template <typename T, bool CHAN>
__global__ void __launch_bounds__(PREP_THREADS, 3) delta_prep_kernel(
    const T* __restrict__ proj, int ld, int x_off, int b_off, const T* __restrict__ dec, int dec_ld, const float* __restrict__ conv_w,
    int taps, const T* __restrict__ ring, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
    const int* __restrict__ tile_tok0, const int* __restrict__ tile_rows, const int* __restrict__ cu_q, int n_seqs,
    const int* __restrict__ tok_slot, const int* __restrict__ tok_pos, int H, int G, int d, int dv, int dr, int dvp,
    float* __restrict__ rec, float* __restrict__ vbuf) {
  extern __shared__ float own[];      // per warp: q, k and log decays of a group, [3][GRP][dr]; every lane reads what it wrote
  const int tile = blockIdx.x;
  const int tok0 = tile_tok0[tile], rows = tile_rows[tile];
  const int slot = tok_slot[tok0];
  if (slot < 0 || rows <= 0) return;
  const int b = seq_of(cu_q, n_seqs, tok0);
  const int t0 = cu_q[b], n = cu_q[b + 1] - t0, p0 = tok_pos[t0], i_tile = tok0 - t0;
  const T* x = proj + x_off;
  const int CH = 2 * G * d + H * dv;
  const int ng = (rows + GRP - 1) / GRP;

  if ((int)blockIdx.y >= H) {      // v: a thread a column of [H, dvp]
    const int part = (int)blockIdx.y - H;
    const int col = (part / V_SPLIT) * PREP_THREADS + threadIdx.x;
    if (col >= H * dvp) return;
    const int h = col / dvp, c = col % dvp;
    for (int gi = part % V_SPLIT; gi < ng; gi += V_SPLIT) {
      const int i0 = i_tile + gi * GRP;
      float acc[GRP];
#pragma unroll
      for (int k = 0; k < GRP; ++k) acc[k] = 0.f;
      if (c < dv) conv_run<T, GRP>(acc, conv_w, x, ld, ring, taps, CH, slot, t0, p0, i0, n, 2 * G * d + h * dv + c);
#pragma unroll
      for (int k = 0; k < GRP; ++k)
        if (i0 + k < n) vbuf[(size_t)(t0 + i0 + k) * H * dvp + col] = c < dv ? siluf_(acc[k]) : 0.f;
    }
    return;
  }

  const int h = blockIdx.y, g = h / (H / G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float rate = -LOG2E * expf(a_log[h]);      // log decays in powers of two
  const size_t RS = (size_t)VECS * dr + SCAL;
  float* qs = own + (size_t)warp * 3 * GRP * dr;
  float *ks = qs + GRP * dr, *ls = ks + GRP * dr;
  for (int gi = warp; gi < ng; gi += PREP_THREADS / 32) {
    const int i0 = i_tile + gi * GRP, m = min(GRP, n - i0);
    // lane i < GRP: beta of token i, and its log decay where there is one per head
    float beta = 0.f, head_lg = 0.f;
    if (lane < m) {
      beta = sigmoidf_(to_f32<T>(proj[(size_t)(t0 + i0 + lane) * ld + b_off + h]));
      if (!CHAN) head_lg = rate * softplusf_(to_f32<T>(dec[(size_t)(t0 + i0 + lane) * dec_ld + h]) + dt_bias[h]);
    }
    float ss[2 * GRP];        // sums of squares: q of each token, then k
#pragma unroll
    for (int i = 0; i < 2 * GRP; ++i) ss[i] = 0.f;
    for (int c = lane; c < dr; c += 32) {
      float aq[GRP], ak[GRP], z[GRP];
#pragma unroll
      for (int i = 0; i < GRP; ++i) aq[i] = ak[i] = z[i] = 0.f;
      if (c < d) {
        if (CHAN) {
#pragma unroll
          for (int i = 0; i < GRP; ++i)
            if (i < m) z[i] = to_f32<T>(dec[(size_t)(t0 + i0 + i) * dec_ld + h * d + c]);
        }
        conv_run<T, GRP>(aq, conv_w, x, ld, ring, taps, CH, slot, t0, p0, i0, n, g * d + c);
        conv_run<T, GRP>(ak, conv_w, x, ld, ring, taps, CH, slot, t0, p0, i0, n, (G + g) * d + c);
      }
      const float bias = CHAN && c < d ? dt_bias[h * d + c] : 0.f;
#pragma unroll
      for (int i = 0; i < GRP; ++i) {
        const bool on = c < d && i < m;
        const float qv = on ? siluf_(aq[i]) : 0.f, kv = on ? siluf_(ak[i]) : 0.f;
        ss[i] = fmaf(qv, qv, ss[i]);
        ss[GRP + i] = fmaf(kv, kv, ss[GRP + i]);
        qs[i * dr + c] = qv;
        ks[i * dr + c] = kv;
        if (CHAN) ls[i * dr + c] = on ? rate * softplusf_(z[i] + bias) : 0.f;
      }
    }
    butterfly<2 * GRP, 32>(ss, lane);      // lane l: sum l / 2
    const float len = (lane < 16 ? 1.f / sqrtf((float)d) : 1.f) / sqrtf(ss[0] + UNIT_EPS);
    float rq[GRP], rk[GRP], be[GRP], hl[GRP];
#pragma unroll
    for (int i = 0; i < GRP; ++i) {
      rq[i] = __shfl_sync(FULL, len, 2 * i);
      rk[i] = __shfl_sync(FULL, len, 16 + 2 * i);
      be[i] = __shfl_sync(FULL, beta, i);
      hl[i] = CHAN ? 0.f : __shfl_sync(FULL, head_lg, i);
    }
    float sums[64];           // A_ij (i(i-1)/2 + j), then P_ij (i(i+1)/2 + j)
#pragma unroll
    for (int i = 0; i < 64; ++i) sums[i] = 0.f;
    float* rc = rec + ((group_base(t0, b) + (size_t)(i0 / GRP)) * H + h) * RS;
    for (int c = lane; c < dr; c += 32) {
      float q[GRP], k[GRP], l[GRP];
#pragma unroll
      for (int i = 0; i < GRP; ++i) {
        q[i] = qs[i * dr + c] * rq[i];
        k[i] = ks[i * dr + c] * rk[i];
        l[i] = CHAN ? ls[i * dr + c] : hl[i];
      }
      float cum = 0.f;
#pragma unroll
      for (int i = 0; i < GRP; ++i) {
        cum += l[i];
        const float e = exp2_(cum);
        rc[i * dr + c] = be[i] * k[i] * e;
        rc[(GRP + i) * dr + c] = q[i] * e;
      }
      rc[3 * GRP * dr + c] = c < d ? expm1f(LN2 * cum) : 0.f;
#pragma unroll
      for (int i = 0; i < GRP; ++i) {
        float* P = sums + PAIRS + i * (i + 1) / 2;
        P[i] = fmaf(q[i], k[i], P[i]);
        float s = 0.f;          // from token j to token i: the log decays in between
#pragma unroll
        for (int j = i - 1; j >= 0; --j) {
          s += l[j + 1];
          const float t = k[j] * exp2_(s);
          sums[i * (i - 1) / 2 + j] = fmaf(k[i], t, sums[i * (i - 1) / 2 + j]);
          P[j] = fmaf(q[i], t, P[j]);
          if (i == GRP - 1) rc[(2 * GRP + j) * dr + c] = t;
        }
      }
      rc[(3 * GRP - 1) * dr + c] = k[GRP - 1];
    }
    butterfly<64, 32>(sums, lane);         // lane l: sums 2 l and 2 l + 1
    float* sc = rc + (size_t)VECS * dr;
    if (lane < GRP) sc[lane] = beta;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int idx = 2 * lane + e, p = idx < PAIRS ? idx : idx - PAIRS;
      int i = 0;
      while ((idx < PAIRS ? i * (i + 1) : (i + 1) * (i + 2)) / 2 <= p) ++i;      // the row of the triangle
      const int j = p - (idx < PAIRS ? i * (i - 1) : i * (i + 1)) / 2;
      const float bi = __shfl_sync(FULL, beta, i);
      if (idx < PAIRS) {
        sc[GRP + idx] = bi * sums[e];
        sc[GRP + PAIRS + j * GRP + i] = 0.f;            // P above its diagonal
      } else {
        sc[GRP + PAIRS + i * GRP + j] = sums[e];
      }
    }
  }
}

// two neighbouring rows at once: fused multiply-adds on register pairs (each half rounds like the single one)
typedef unsigned long long pair_t;
__device__ __forceinline__ pair_t fma2(pair_t a, pair_t b, pair_t c) {
  pair_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ pair_t mul2(pair_t a, pair_t b) {
  pair_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ pair_t pack2(float lo, float hi) {
  pair_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float sum2(pair_t a) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(a));
  return lo + hi;
}

// L lanes share CPG value columns; lane l of them holds the rows 4 (l + L m) .. + 3 for m < RPL / 4 (vectors of 16 bytes,
// neighbouring lanes side by side).  Records hold vectors of L * RPL floats, so no lane needs a bound.
template <int L, int RPL, int CPG>
__global__ void __launch_bounds__(WALK_WARPS * 32) delta_walk_kernel(
    const float* __restrict__ rec, const float* __restrict__ vbuf, const int* __restrict__ cu_q, const int* __restrict__ seq_slot,
    int H, int dv, int dp, int dvp, float* __restrict__ state, float* __restrict__ o) {
  constexpr int DR = L * RPL, RS = VECS * DR + SCAL;
  constexpr int COLS = WALK_WARPS * (32 / L) * CPG;         // value columns of the block
  constexpr int NV = GRP * COLS / 4;                        // 16-byte pieces of a group's v
  constexpr int STAGE = RS + GRP * COLS;
  constexpr int NST = WALK_STAGES;
  constexpr int VALS = 2 * GRP * CPG, NPL = VALS / L;       // sums L lanes form, sums a lane is left with
  constexpr int THREADS = WALK_WARPS * 32;
  static_assert(VALS >= L && NV <= THREADS, "every lane is left with a sum; a thread a piece of v");
  extern __shared__ __align__(16) float stage_mem[];
  __shared__ __align__(16) float ksum[WALK_WARPS][32 / L][GRP * CPG];
  const int b = blockIdx.z, h = blockIdx.y;
  const int slot = seq_slot[b];
  const int t0 = cu_q[b], n = cu_q[b + 1] - t0;
  if (slot < 0 || n <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gl = lane % L;
  const int blk0 = blockIdx.x * COLS, lcol = (warp * (32 / L) + lane / L) * CPG, col0 = blk0 + lcol;
  const int ng = (n + GRP - 1) / GRP;
  const float* rc0 = rec + (group_base(t0, b) * H + h) * (size_t)RS;
  const size_t rstep = (size_t)H * RS;
  const float* v0 = vbuf + (size_t)t0 * H * dvp + (size_t)h * dvp + blk0;
  const size_t vstep = (size_t)H * dvp;

  auto issue = [&](int j) {      // record and v rows of group j -> its stage
    if (j < ng) {
      float* sm = stage_mem + (j % NST) * STAGE;
      const float* src = rc0 + (size_t)j * rstep;
#pragma unroll
      for (int k = 0; k < (RS / 4 + THREADS - 1) / THREADS; ++k) {
        const int i = (tid + k * THREADS) * 4;
        if (i < RS) cp_async16(sm + i, src + i);
      }
      if (tid < NV) {
        const int r = tid / (COLS / 4), c = (tid % (COLS / 4)) * 4;
        const int t = min(j * GRP + r, n - 1);      // a group's missing tokens have beta = 0: any finite row will do
        cp_async16(sm + RS + r * COLS + c, v0 + (size_t)t * vstep + c);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int j = 0; j < NST - 1; ++j) issue(j);

  pair_t S[CPG][RPL / 2];
  float* sp = state + (((size_t)slot * H + h) * dv + col0) * dp;
#pragma unroll
  for (int c = 0; c < CPG; ++c)
#pragma unroll
    for (int m = 0; m < RPL / 4; ++m) {
      const int row = 4 * (gl + L * m);
      ulonglong2 x = make_ulonglong2(0ull, 0ull);
      if (col0 + c < dv && row < dp) x = *reinterpret_cast<const ulonglong2*>(sp + (size_t)c * dp + row);
      S[c][2 * m] = x.x;
      S[c][2 * m + 1] = x.y;
    }
  // the sums this lane is left with: index -> (token, or GRP + token for the query; column)
  const int tok0 = gl * NPL / CPG;
  float* op = o + (size_t)t0 * H * dv + (size_t)h * dv + col0;

  for (int j = 0; j < ng; ++j) {
    cp_async_wait<NST - 2>();
    __syncthreads();               // group j is in shared memory; everyone is done with group j - 1
    issue(j + NST - 1);
    const float* sm = stage_mem + (j % NST) * STAGE;
    const float* vec = sm + 4 * gl;
    auto rows = [&](pair_t (&r)[RPL / 2], int i) {
#pragma unroll
      for (int m = 0; m < RPL / 4; ++m) {
        const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(vec + i * DR + 4 * L * m);
        r[2 * m] = t.x;
        r[2 * m + 1] = t.y;
      }
    };
    float x[VALS];
#pragma unroll
    for (int i = 0; i < 2 * GRP; ++i) {
      pair_t kt[RPL / 2];
      rows(kt, i);
#pragma unroll
      for (int c = 0; c < CPG; ++c) {
        pair_t a = mul2(kt[0], S[c][0]);
#pragma unroll
        for (int r = 1; r < RPL / 2; ++r) a = fma2(kt[r], S[c][r], a);
        x[i * CPG + c] = sum2(a);
      }
    }
    // what the update will read is on its way while the sums are formed
    pair_t gm[RPL / 2], kb[GRP][RPL / 2];
    rows(gm, 3 * GRP);
#pragma unroll
    for (int i = 0; i < GRP; ++i) rows(kb[i], 2 * GRP + i);
    butterfly<VALS, L>(x, gl);
    if (tok0 < GRP) {
#pragma unroll
      for (int e = 0; e < NPL; ++e) ksum[warp][lane / L][gl * NPL + e] = x[e];
    }
    __syncwarp();
    const float* sc = sm + VECS * DR;
    const float* ksm = ksum[warp][lane / L];
    float u[GRP][CPG];
#pragma unroll
    for (int i = 0; i < GRP; ++i) {
#pragma unroll
      for (int c = 0; c < CPG; ++c) u[i][c] = fmaf(sc[i], sm[RS + i * COLS + lcol + c], -ksm[i * CPG + c]);
#pragma unroll
      for (int jj = 0; jj < i; ++jj) {
        const float a = sc[GRP + i * (i - 1) / 2 + jj];
#pragma unroll
        for (int c = 0; c < CPG; ++c) u[i][c] = fmaf(-a, u[jj][c], u[i][c]);
      }
    }
#pragma unroll
    for (int c = 0; c < CPG; ++c)
#pragma unroll
      for (int r = 0; r < RPL / 2; ++r) S[c][r] = fma2(S[c][r], gm[r], S[c][r]);
#pragma unroll
    for (int i = 0; i < GRP; ++i) {
#pragma unroll
      for (int c = 0; c < CPG; ++c) {
        const pair_t uu = pack2(u[i][c], u[i][c]);
#pragma unroll
        for (int r = 0; r < RPL / 2; ++r) S[c][r] = fma2(kb[i][r], uu, S[c][r]);
      }
    }
    // the lanes that hold queries' sums finish their outputs
#pragma unroll
    for (int e = 0; e < NPL; ++e) {
      const int idx = gl * NPL + e, i = (idx / CPG) % GRP, oc = idx % CPG;
      const float* pr = sc + GRP + PAIRS + i * GRP;
      float val = x[e];
#pragma unroll
      for (int jj = 0; jj < GRP; ++jj) {
        float uc = u[jj][0];
#pragma unroll
        for (int cc = 1; cc < CPG; ++cc) uc = oc == cc ? u[jj][cc] : uc;
        val = fmaf(pr[jj], uc, val);
      }
      const int t = j * GRP + i;
      if (idx >= GRP * CPG && t < n && col0 + oc < dv) op[(size_t)t * H * dv + oc] = val;
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int c = 0; c < CPG; ++c)
#pragma unroll
    for (int m = 0; m < RPL / 4; ++m) {
      const int row = 4 * (gl + L * m);
      if (col0 + c < dv && row < dp) *reinterpret_cast<ulonglong2*>(sp + (size_t)c * dp + row) = make_ulonglong2(S[c][2 * m], S[c][2 * m + 1]);
    }
}

constexpr int NORM_WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(NORM_WARPS * 32) delta_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, int gate_ld,
                                                                    const float* __restrict__ w, float eps, int sigmoid_gate,
                                                                    const int* __restrict__ tok_slot, T* __restrict__ out, int n, int H,
                                                                    int dv, int norm_blocks, const T* __restrict__ x, int ld,
                                                                    const int* __restrict__ cu_q, const int* __restrict__ seq_slot,
                                                                    const int* __restrict__ tok_pos, T* __restrict__ ring, int taps, int CH) {
  if ((int)blockIdx.x >= norm_blocks) {      // the ring: a thread a (sequence, channel)
    const int cb = (CH + NORM_WARPS * 32 - 1) / (NORM_WARPS * 32), i = (int)blockIdx.x - norm_blocks;
    const int b = i / cb, c = (i % cb) * NORM_WARPS * 32 + threadIdx.x, slot = seq_slot[b];
    const int t1 = cu_q[b + 1], nb = t1 - cu_q[b];
    if (slot < 0 || nb <= 0 || c >= CH) return;
    const int last = tok_pos[t1 - 1];
    for (int k = 0; k < taps - 1 && k < nb; ++k)
      ring[((size_t)slot * taps + (last - k) % taps) * CH + c] = x[(size_t)(t1 - 1 - k) * ld + c];
    return;
  }
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * NORM_WARPS + (threadIdx.x >> 5);
  if (item >= (long long)n * H) return;
  const int t = (int)(item / H), h = (int)(item % H);
  T* dst = out + (size_t)t * H * dv + (size_t)h * dv;
  if (tok_slot[t] < 0) {
    for (int c = lane; c < dv; c += 32) dst[c] = from_f32<T>(0.f);
    return;
  }
  const float* src = o + (size_t)t * H * dv + (size_t)h * dv;
  const T* gt = gate + (size_t)t * gate_ld + (size_t)h * dv;
  float ss = 0.f;
  // heads of up to 256 values in steps of four, rows on their vectors' boundaries: a lane keeps its values in registers
  if (dv % 4 == 0 && dv <= 256 && gate_ld % 4 == 0 && reinterpret_cast<uintptr_t>(gate) % (4 * sizeof(T)) == 0) {
    float4 v[2], z[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int c = 4 * (lane + 32 * k);
      v[k] = z[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < dv) { v[k] = *reinterpret_cast<const float4*>(src + c); z[k] = load4<T>(gt + c); }
    }
#pragma unroll
    for (int k = 0; k < 2; ++k) ss = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, fmaf(v[k].z, v[k].z, fmaf(v[k].w, v[k].w, ss))));
    const float rinv = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int c = 4 * (lane + 32 * k);
      if (c < dv) {
        const float4 ww = *reinterpret_cast<const float4*>(w + c);
        auto act = [&](float x) { return sigmoid_gate ? sigmoidf_(x) : siluf_(x); };
        store4<T>(dst + c, make_float4(v[k].x * rinv * ww.x * act(z[k].x), v[k].y * rinv * ww.y * act(z[k].y),
                                       v[k].z * rinv * ww.z * act(z[k].z), v[k].w * rinv * ww.w * act(z[k].w)));
      }
    }
    return;
  }
  for (int c = lane; c < dv; c += 32) { const float v = src[c]; ss = fmaf(v, v, ss); }
  const float rinv = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
  for (int c = lane; c < dv; c += 32) {
    const float z = to_f32<T>(gt[c]);
    dst[c] = from_f32<T>(src[c] * rinv * w[c] * (sigmoid_gate ? sigmoidf_(z) : siluf_(z)));
  }
}

template <typename T, int RPL, bool CHAN>
__global__ void __launch_bounds__(DEC_THREADS) delta_decode_kernel(
    const T* __restrict__ proj, int ld, int x_off, int b_off, const T* __restrict__ dec, int dec_ld, const T* __restrict__ gate,
    int gate_ld, const float* __restrict__ conv_w, int taps, T* __restrict__ ring, const float* __restrict__ a_log,
    const float* __restrict__ dt_bias, const float* __restrict__ norm_w, float eps, int sigmoid_gate, const int* __restrict__ tok_slot,
    const int* __restrict__ tok_pos, int H, int G, int d, int dv, int dp, float* __restrict__ state, T* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float scratch[33];
  const int h = blockIdx.x, t = blockIdx.y;
  const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31, nwarp = nthr >> 5;
  const int slot = tok_slot[t];
  if (slot < 0) {
    for (int c = tid; c < dv; c += nthr) out[(size_t)t * H * dv + (size_t)h * dv + c] = from_f32<T>(0.f);
    return;
  }
  const int row0 = lane * RPL;
  float* sp = state + ((size_t)slot * H + h) * dv * dp;
  float S[DEC_COLS][RPL];
  // the first columns' state is requested before anything else
#pragma unroll
  for (int c = 0; c < DEC_COLS; ++c) {
    const int col = warp * DEC_COLS + c;
    if (col < dv) load_rows<RPL>(S[c], sp + (size_t)col * dp, row0, dp);
    else
#pragma unroll
      for (int r = 0; r < RPL; ++r) S[c][r] = 0.f;
  }
  float *qs = sm, *ks = qs + dp, *gm = ks + dp, *vs = gm + dp, *os = vs + dv;
  const int pos = tok_pos[t], g = h / (H / G), CH = 2 * G * d + H * dv;
  const bool first = h % (H / G) == 0;                       // one head of a group stores the group's q and k in the ring
  const T* x = proj + x_off;
  T* ring_row = ring + ((size_t)slot * taps + pos % taps) * CH;
  const ConvRows<T> conv(conv_w, x, ld, ring, taps, CH, slot, t, pos, 0);
  float aq = 0.f, ak = 0.f, aqk = 0.f;
  for (int c = tid; c < dp; c += nthr) {
    float q = 0.f, k = 0.f, gmc = 0.f;
    if (c < d) {
      const int cq = g * d + c, ck = (G + g) * d + c;
      q = siluf_(conv(cq));
      k = siluf_(conv(ck));
      if (first && taps > 1) { ring_row[cq] = x[(size_t)t * ld + cq]; ring_row[ck] = x[(size_t)t * ld + ck]; }
      const int gi = CHAN ? h * d + c : h;
      gmc = expm1f(-expf(a_log[h]) * softplusf_(to_f32<T>(dec[(size_t)t * dec_ld + gi]) + dt_bias[gi]));
    }
    qs[c] = q; ks[c] = k; gm[c] = gmc;
    aq = fmaf(q, q, aq); ak = fmaf(k, k, ak); aqk = fmaf(q, k, aqk);
  }
  for (int c = tid; c < dv; c += nthr) {
    const int cv = 2 * G * d + h * dv + c;
    vs[c] = siluf_(conv(cv));
    if (taps > 1) ring_row[cv] = x[(size_t)t * ld + cv];
  }
  const float rq = 1.f / (sqrtf((float)d) * sqrtf(block_sum(aq, scratch) + UNIT_EPS));
  const float rk = 1.f / sqrtf(block_sum(ak, scratch) + UNIT_EPS);
  const float qk = block_sum(aqk, scratch) * rq * rk;        // (the barriers inside also publish q, k, v and the decays)
  const float beta = sigmoidf_(to_f32<T>(proj[(size_t)t * ld + b_off + h]));
  float kr[RPL], qr[RPL], gr[RPL];
  load_rows<RPL>(kr, ks, row0, dp);
  load_rows<RPL>(qr, qs, row0, dp);
  load_rows<RPL>(gr, gm, row0, dp);
#pragma unroll
  for (int r = 0; r < RPL; ++r) { kr[r] *= rk; qr[r] *= rq; }

  for (int base = warp * DEC_COLS; base < dv; base += nwarp * DEC_COLS) {
    if (base != warp * DEC_COLS) {
#pragma unroll
      for (int c = 0; c < DEC_COLS; ++c) {
        if (base + c < dv) load_rows<RPL>(S[c], sp + (size_t)(base + c) * dp, row0, dp);
        else
#pragma unroll
          for (int r = 0; r < RPL; ++r) S[c][r] = 0.f;
      }
    }
    float xs[2 * DEC_COLS];
#pragma unroll
    for (int c = 0; c < DEC_COLS; ++c) {
      float a = 0.f, q = 0.f;
#pragma unroll
      for (int r = 0; r < RPL; ++r) {
        S[c][r] = fmaf(S[c][r], gr[r], S[c][r]);
        a = fmaf(kr[r], S[c][r], a);
        q = fmaf(qr[r], S[c][r], q);
      }
      xs[c] = a;
      xs[DEC_COLS + c] = q;
    }
    butterfly<2 * DEC_COLS, 32>(xs, lane);
    const float mine = xs[0];                                // lane l: sum l / 2 (key sums of the eight columns, then query sums)
    const int id = lane >> 1, c_own = id & (DEC_COLS - 1), col = base + c_own;
    const float uval = col < dv ? beta * (vs[col] - mine) : 0.f;
    const float u_own = __shfl_sync(FULL, uval, 2 * c_own);
    if (id >= DEC_COLS && !(lane & 1) && col < dv) os[col] = fmaf(qk, u_own, mine);
#pragma unroll
    for (int c = 0; c < DEC_COLS; ++c) {
      const float u = __shfl_sync(FULL, uval, 2 * c);
#pragma unroll
      for (int r = 0; r < RPL; ++r) S[c][r] = fmaf(kr[r], u, S[c][r]);
      if (base + c < dv) store_rows<RPL>(S[c], sp + (size_t)(base + c) * dp, row0, dp);
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < dv; c += nthr) ss = fmaf(os[c], os[c], ss);
  const float rinv = 1.f / sqrtf(block_sum(ss, scratch) / (float)dv + eps);
  for (int c = tid; c < dv; c += nthr) {
    const float z = to_f32<T>(gate[(size_t)t * gate_ld + (size_t)h * dv + c]);
    out[(size_t)t * H * dv + (size_t)h * dv + c] = from_f32<T>(os[c] * rinv * norm_w[c] * (sigmoid_gate ? sigmoidf_(z) : siluf_(z)));
  }
}

template <typename T, bool CHAN>
int prep_launch(const void* proj, int ld, int x_off, int b_off, const void* dec, int dec_ld, const float* conv_w, int taps,
                const void* ring, const float* a_log, const float* dt_bias, const int* tile_tok0, const int* tile_rows, int n_tiles,
                const int* cu_q, int n_seqs, const int* tok_slot, const int* tok_pos, int H, int G, int d, int dv, int dr, int dvp,
                float* rec, float* vbuf, cudaStream_t st) {
  const long long vb = ((long long)H * dvp + PREP_THREADS - 1) / PREP_THREADS * V_SPLIT;
  if (H + vb > 65535) return DRYFT_ERR_UNSUPPORTED;
  const size_t smem = sizeof(float) * (PREP_THREADS / 32) * 3 * GRP * (size_t)dr;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(delta_prep_kernel<T, CHAN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  dim3 grid(n_tiles, (unsigned)(H + vb));
  delta_prep_kernel<T, CHAN><<<grid, PREP_THREADS, smem, st>>>(
      (const T*)proj, ld, x_off, b_off, (const T*)dec, dec_ld, conv_w, taps, (const T*)ring, a_log, dt_bias, tile_tok0, tile_rows, cu_q,
      n_seqs, tok_slot, tok_pos, H, G, d, dv, dr, dvp, rec, vbuf);
  return launch_status();
}

template <int L, int RPL, int CPG>
int walk_launch(const float* rec, const float* vbuf, const int* cu_q, const int* seq_slot, int n_seqs, int H, int dv, int dp, int dvp,
                float* state, float* o, cudaStream_t st) {
  constexpr int COLS = WALK_WARPS * (32 / L) * CPG;
  static_assert(V_PAD % COLS == 0, "a block's columns lie within a padded row of v");
  const size_t smem = sizeof(float) * WALK_STAGES * (size_t)(VECS * L * RPL + SCAL + GRP * COLS);
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(delta_walk_kernel<L, RPL, CPG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  dim3 grid((dv + COLS - 1) / COLS, H, n_seqs);
  delta_walk_kernel<L, RPL, CPG><<<grid, WALK_WARPS * 32, smem, st>>>(rec, vbuf, cu_q, seq_slot, H, dv, dp, dvp, state, o);
  return launch_status();
}

template <typename T, int RPL, bool CHAN>
int decode_launch(const void* proj, int ld, int x_off, int b_off, const void* dec, int dec_ld, const void* gate, int gate_ld,
                  const float* conv_w, int taps, void* ring, const float* a_log, const float* dt_bias, const float* norm_w, float eps,
                  int sigmoid_gate, const int* tok_slot, const int* tok_pos, int n, int H, int G, int d, int dv, int dp, float* state,
                  void* out, cudaStream_t st) {
  const size_t smem = sizeof(float) * ((size_t)3 * dp + 2 * dv);
  if (smem > 48 * 1024) return DRYFT_ERR_UNSUPPORTED;
  int warps = (dv + DEC_COLS - 1) / DEC_COLS;
  warps = warps < 4 ? 4 : (warps > DEC_THREADS / 32 ? DEC_THREADS / 32 : warps);
  dim3 grid(H, n);
  delta_decode_kernel<T, RPL, CHAN><<<grid, warps * 32, smem, st>>>(
      (const T*)proj, ld, x_off, b_off, (const T*)dec, dec_ld, (const T*)gate, gate_ld, conv_w, taps, (T*)ring, a_log, dt_bias, norm_w, eps,
      sigmoid_gate, tok_slot, tok_pos, H, G, d, dv, dp, state, (T*)out);
  return launch_status();
}

bool sizes_ok(int H, int G, int d, int dv, int taps) {
  return H >= 1 && G >= 1 && H % G == 0 && H <= 32768 && d >= 1 && d <= 256 && dv >= 1 && dv <= 4096 && taps >= 1 && taps <= DRYFT_CONV_MAX_TAPS;
}
int rows_per_lane(int d) { return d <= 32 ? 1 : d <= 64 ? 2 : d <= 128 ? 4 : 8; }
}  // namespace

DRYFT_API int dryft_delta_prep(int is_bf16, int per_channel, const void* proj, int ld, int x_off, int b_off, const void* dec, int dec_ld,
                               const float* conv_w, int taps, const void* ring, const float* a_log, const float* dt_bias,
                               const int* tile_tok0, const int* tile_rows, int n_tiles, int tile_size, const int* cu_q, int n_seqs,
                               const int* tok_slot, const int* tok_pos, int H, int G, int d, int dv, float* rec, float* vbuf,
                               cudaStream_t st) {
  if (n_tiles <= 0) return 0;
  if (!sizes_ok(H, G, d, dv, taps) || tile_size % GRP || (taps > 1 && ring == nullptr)) return DRYFT_ERR_UNSUPPORTED;
  const int dr = 32 * rows_per_lane(d), dvp = (dv + V_PAD - 1) / V_PAD * V_PAD;
#define DRYFT_PREP(T, CH)                                                                                                        \
  return prep_launch<T, CH>(proj, ld, x_off, b_off, dec, dec_ld, conv_w, taps, ring, a_log, dt_bias, tile_tok0, tile_rows, n_tiles, \
                            cu_q, n_seqs, tok_slot, tok_pos, H, G, d, dv, dr, dvp, rec, vbuf, st)
  if (is_bf16) {
    if (per_channel) DRYFT_PREP(__nv_bfloat16, true);
    DRYFT_PREP(__nv_bfloat16, false);
  }
  if (per_channel) DRYFT_PREP(float, true);
  DRYFT_PREP(float, false);
#undef DRYFT_PREP
}

DRYFT_API int dryft_delta_walk(const float* rec, const float* vbuf, const int* cu_q, const int* seq_slot, int n_seqs, int H, int d, int dv,
                               float* state, float* o, cudaStream_t st) {
  if (n_seqs <= 0) return 0;
  if (!sizes_ok(H, 1, d, dv, 1) || n_seqs > 65535) return DRYFT_ERR_UNSUPPORTED;
  const int dp = (d + 3) / 4 * 4, dvp = (dv + V_PAD - 1) / V_PAD * V_PAD;
#define DRYFT_WALK(L, R, C) return walk_launch<L, R, C>(rec, vbuf, cu_q, seq_slot, n_seqs, H, dv, dp, dvp, state, o, st)
  switch (rows_per_lane(d)) {      // L * RPL = 32 * rows_per_lane: the length of a record's vectors
    case 1: DRYFT_WALK(8, 4, 1);
    case 2: DRYFT_WALK(16, 4, 2);
    case 4:      // few columns for the device (at most eight an SM): two a warp instead of four
      if ((long long)n_seqs * H * dv <= FEW_COLUMNS) DRYFT_WALK(32, 4, 2);
      DRYFT_WALK(16, 8, 2);
    default: DRYFT_WALK(32, 8, 4);
  }
#undef DRYFT_WALK
}

DRYFT_API int dryft_delta_norm(int is_bf16, const float* o, const void* gate, int gate_ld, const float* w, float eps, int sigmoid_gate,
                               const int* tok_slot, void* out, int n, int H, int G, int d, int dv, const void* proj, int ld, int x_off,
                               const int* cu_q, const int* seq_slot, int n_seqs, const int* tok_pos, void* ring, int taps, cudaStream_t st) {
  if (n <= 0) return 0;
  if (!sizes_ok(H, G, d, dv, taps)) return DRYFT_ERR_UNSUPPORTED;
  const int CH = 2 * G * d + H * dv;
  const long long nblk = ((long long)n * H + NORM_WARPS - 1) / NORM_WARPS;
  const long long rblk = taps > 1 ? (long long)n_seqs * ((CH + NORM_WARPS * 32 - 1) / (NORM_WARPS * 32)) : 0;
  if (nblk + rblk > 0x7fffffffLL) return DRYFT_ERR_UNSUPPORTED;
  typedef __nv_bfloat16 bf;
  const unsigned grid = (unsigned)(nblk + rblk);
  if (is_bf16)
    delta_norm_kernel<bf><<<grid, NORM_WARPS * 32, 0, st>>>(o, (const bf*)gate, gate_ld, w, eps, sigmoid_gate, tok_slot, (bf*)out, n, H, dv,
                                                            (int)nblk, (const bf*)proj + x_off, ld, cu_q, seq_slot, tok_pos, (bf*)ring, taps, CH);
  else
    delta_norm_kernel<float><<<grid, NORM_WARPS * 32, 0, st>>>(o, (const float*)gate, gate_ld, w, eps, sigmoid_gate, tok_slot, (float*)out, n, H,
                                                               dv, (int)nblk, (const float*)proj + x_off, ld, cu_q, seq_slot, tok_pos,
                                                               (float*)ring, taps, CH);
  return launch_status();
}

DRYFT_API int dryft_delta_decode(int is_bf16, int per_channel, const void* proj, int ld, int x_off, int b_off, const void* dec, int dec_ld,
                                 const void* gate, int gate_ld, const float* conv_w, int taps, void* ring, const float* a_log,
                                 const float* dt_bias, const float* norm_w, float eps, int sigmoid_gate, const int* tok_slot,
                                 const int* tok_pos, int n, int H, int G, int d, int dv, float* state, void* out, cudaStream_t st) {
  if (n <= 0) return 0;
  if (!sizes_ok(H, G, d, dv, taps) || n > 65535 || (taps > 1 && ring == nullptr)) return DRYFT_ERR_UNSUPPORTED;
  const int dp = (d + 3) / 4 * 4;
#define DRYFT_DEC(T, R, CH)                                                                                                          \
  return decode_launch<T, R, CH>(proj, ld, x_off, b_off, dec, dec_ld, gate, gate_ld, conv_w, taps, ring, a_log, dt_bias, norm_w, eps, \
                                 sigmoid_gate, tok_slot, tok_pos, n, H, G, d, dv, dp, state, out, st)
#define DRYFT_DEC_R(T, CH)                  \
  switch (rows_per_lane(d)) {               \
    case 1: DRYFT_DEC(T, 1, CH);            \
    case 2: DRYFT_DEC(T, 2, CH);            \
    case 4: DRYFT_DEC(T, 4, CH);            \
    default: DRYFT_DEC(T, 8, CH);           \
  }
  if (is_bf16) {
    if (per_channel) { DRYFT_DEC_R(__nv_bfloat16, true) } else { DRYFT_DEC_R(__nv_bfloat16, false) }
  } else {
    if (per_channel) { DRYFT_DEC_R(float, true) } else { DRYFT_DEC_R(float, false) }
  }
#undef DRYFT_DEC_R
#undef DRYFT_DEC
}
