// Time mixing with a decay per head and key channel: the projections read mixtures of a token's input and the one before it,
// and the state per head is a matrix [d, dv] that takes in an outer product per token.
//
//   wkv_mix     m_j[t] = T( h[t] + (h[t-1] - h[t]) * mu_j )  for the five projections j = r, k, v, g, w: out [5, n, width].
//               The token before the first one of a step is per-sequence state (`last` [slots, width], zero when a sequence
//               starts); the launch that follows the products leaves the step's last inputs there.
//   wkv_tanh    T( tanh(low) ): the low-rank input of the decay's second product (steps of many tokens)
//   wkv_walk    per head, with w = exp(-exp(z + w0)) per key channel (z: the decay's second product) and the bonus u:
//                   o_t = S^T r_t + (sum_c r_c u_c k_c) v_t ;   S <- diag(w_t) S + k_t v_t^T
//               MODE 0: a block per (sequence, head, slice of value columns), tokens in order from the slot's state, which is
//               left advanced.  A step of many tokens is cut into chunks of `cht` tokens that run side by side: MODE 1, every
//               chunk from a ZERO state, leaving its own state and the product of its decays per key channel; wkv_prefix, per
//               sequence, start(k+1) = decays_k * start(k) + own(k), which turns the chunks' own states into their start states
//               and leaves the final state in the slot; MODE 2, every chunk again from its start state, writing o.
//               Where a block holds all of a head's value columns it also norms and gates a tile's read-outs before they leave it:
//                   out = T( o / sqrt(mean(o^2) + eps) * norm_w * silu(g) )      (the mean over a head's values)
//               and leaves the step's last inputs in `last`; else
//   wkv_norm    does both behind the walk
//   wkv_decode  one token per sequence: tanh, the decay's second product, decay, bonus, read-out, state update, norm, gate and
//               `last` in ONE launch behind the products; a block per (sequence, head)
//
// T is the activation type.  Everything from the products' results to the gated output is 32-bit.  A chunk's decays multiply to
// exp(-sum exp(z + w0)): no exponent is positive, nothing is divided, so decays of any strength are served.  The state is
// [slots, H, d, dv], 32-bit, zero when a sequence starts.  Sequences with slot -1 (padding) are skipped.
// No block waits on another block.
#include "common.cuh"
#include <math.h>

namespace {
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
__device__ __forceinline__ void unpack2(pair_t a, float* lo, float* hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(*lo), "=f"(*hi) : "l"(a)); }

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }

// V consecutive elements as floats (V 8 or 4: one or two vector loads; 1: a scalar)
template <typename T, int V> __device__ __forceinline__ void load_piece(const T* p, float* f) {
  if constexpr (V * sizeof(T) >= 16) {
#pragma unroll
    for (int i = 0; i < V; i += 16 / (int)sizeof(T)) {
      const uint4 raw = *reinterpret_cast<const uint4*>(p + i);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int j = 0; j < 16 / (int)sizeof(T); ++j) f[i + j] = to_f32<T>(e[j]);
    }
  } else if constexpr (V * sizeof(T) == 8) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = to_f32<T>(e[j]);
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = to_f32<T>(p[j]);
  }
}
template <typename T, int V> __device__ __forceinline__ void store_piece(T* p, const float* f) {
  if constexpr (V == 1) {
    p[0] = from_f32<T>(f[0]);
  } else {
    __align__(16) T e[V];
#pragma unroll
    for (int j = 0; j < V; ++j) e[j] = from_f32<T>(f[j]);
#pragma unroll
    for (int i = 0; i < V; i += 16 / (int)sizeof(T)) {
      if constexpr (V * sizeof(T) == 8) *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(e);
      else *reinterpret_cast<uint4*>(p + i) = *reinterpret_cast<const uint4*>(e + i);
    }
  }
}

constexpr int MIX_THREADS = 256;

template <typename T, int V>
__global__ void __launch_bounds__(MIX_THREADS) wkv_mix_kernel(const T* __restrict__ h, const T* __restrict__ last, const float* __restrict__ mu,
                                                            const int* __restrict__ tok_slot, T* __restrict__ out, int n, int width) {
  const int t = blockIdx.x;
  const int c = ((int)blockIdx.y * MIX_THREADS + (int)threadIdx.x) * V;
  if (c >= width) return;
  const int slot = tok_slot[t];
  const bool same = t > 0 && slot >= 0 && tok_slot[t - 1] == slot;      // the row before belongs to the same sequence
  float x[V], p[V];
  load_piece<T, V>(h + (size_t)t * width + c, x);
  if (same) load_piece<T, V>(h + (size_t)(t - 1) * width + c, p);
  else if (slot >= 0) load_piece<T, V>(last + (size_t)slot * width + c, p);
  else {
#pragma unroll
    for (int j = 0; j < V; ++j) p[j] = 0.f;
  }
#pragma unroll
  for (int i = 0; i < 5; ++i) {
    float m[V], o[V];
    load_piece<float, V>(mu + (size_t)i * width + c, m);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = fmaf(p[j] - x[j], m[j], x[j]);
    store_piece<T, V>(out + ((size_t)i * n + t) * width + c, o);
  }
}

template <typename T> __global__ void wkv_tanh_kernel(const float* __restrict__ low, T* __restrict__ out, size_t count) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < count) out[i] = from_f32<T>(tanhf(low[i]));
}

// chunk `ci` of the step (chunks counted through the sequences in order) -> its sequence and its index within it
__device__ __forceinline__ bool chunk_of(const int* __restrict__ cu_q, int n_seqs, int cht, int ci, int* b_out, int* c_out) {
  int base = 0;
  for (int b = 0; b < n_seqs; ++b) {
    const int nc = (cu_q[b + 1] - cu_q[b] + cht - 1) / cht;
    if (ci < base + nc) { *b_out = b; *c_out = ci - base; return true; }
    base += nc;
  }
  return false;
}

// N bytes (8 or 16) from global to shared memory behind the threads' backs
template <int N> __device__ __forceinline__ void cp_async(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  if constexpr (N == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem));
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(s), "l"(gmem));
}

constexpr int ROWS = 16;     // key channels a thread's piece of the state has (four groups of four, RS * 4 apart)
constexpr int COLS = 4;      // value columns a thread's piece of the state has

// RS: threads that share a group of value columns (RS * 16 >= d); blockDim = RS * CG, CG groups of four columns.
// V: elements a vector load of the operands takes (4, or 1 where sizes are no multiple of four).  TT: tokens staged at once.
struct Finish { const void* g; const float* norm_w; float eps; const void* h; int width; void *last, *out; };   // out null: the read-outs leave as they are

template <typename T, int RS, int MODE, int V, int TT>
__global__ void __launch_bounds__(256, 2) wkv_walk_kernel(
    const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v, int ld, const float* __restrict__ z,
    const float* __restrict__ w0, const float* __restrict__ u, const int* __restrict__ cu_q, const int* __restrict__ seq_slot, int n_seqs,
    int cht, int H, int d, int dv, float* __restrict__ state, float* __restrict__ cstate, float* __restrict__ cdecay, float* __restrict__ o,
    Finish fin) {
  constexpr int DP = RS * ROWS;
  constexpr int LG = DP / 4 < 32 ? DP / 4 : 32, PER = DP / 4 / LG;      // lanes that share a token's key channels, vectors of four a lane takes
  extern __shared__ __align__(16) float sm[];
  const int CG = blockDim.x / RS, CW = CG * COLS;
  float* rs_ = sm;                          // [TT][DP]
  float* ks_ = rs_ + TT * DP;               // [TT][DP]
  float* ws_ = ks_ + TT * DP;               // [TT][DP]
  float* vs_ = ws_ + TT * DP;               // [TT][CW]
  float* bs_ = vs_ + TT * CW;               // [TT]
  float* us_ = bs_ + TT;                    // [DP]
  float* w0s = us_ + DP;                    // [DP]
  float* os_ = w0s + DP;                    // MODE 0 and 2: [TT][CW] read-outs of a tile
  float* ds_ = w0s + DP;                    // MODE 1: [token groups][DP] sums of exp(z + w0)
  // V = 4: the next tile's operands as they lie in memory, on their way while this tile is walked
  float* zn = w0s + DP + (MODE == 1 ? (int)blockDim.x / LG * DP : TT * CW);      // [TT][DP]
  T* kn = reinterpret_cast<T*>(zn + TT * DP);                                    // [TT][DP]
  T* rn = kn + TT * DP;                                                          // [TT][DP]
  T* vn = rn + TT * DP;                                                          // [TT][CW]
  T* gn = vn + TT * CW;                                                          // [2][TT][CW] this tile's and the next one's gates
  int b, ci = 0;
  if (MODE == 0) b = blockIdx.x;
  else if (!chunk_of(cu_q, n_seqs, cht, blockIdx.x, &b, &ci)) return;
  const int slot = seq_slot[b];
  if (slot < 0) return;
  const int hd = blockIdx.y, col0 = (int)blockIdx.z * CW;
  const int t_begin = cu_q[b] + ci * cht, t_end = MODE == 0 ? cu_q[b + 1] : min(cu_q[b + 1], t_begin + cht);
  const int tid = threadIdx.x, rs = tid % RS, cg = tid / RS;
  const int c0 = col0 + cg * COLS;          // this thread's value columns

  // the state's piece: rows 4 * (rs + RS * q) + i, columns c0 + j; pairs of neighbouring rows
  pair_t S[COLS][ROWS / 2];
  const size_t per = (size_t)d * dv;
  float* start = MODE == 0 ? state + ((size_t)slot * H + hd) * per : cstate + ((size_t)blockIdx.x * H + hd) * per;
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int i = 0; i < 4; i += 2) {
      const int row = 4 * (rs + RS * q) + i;
      float a[2][COLS];
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int j = 0; j < COLS; ++j)
          a[e][j] = (MODE != 1 && row + e < d && c0 + j < dv) ? start[(size_t)(row + e) * dv + c0 + j] : 0.f;
#pragma unroll
      for (int j = 0; j < COLS; ++j) S[j][q * 2 + i / 2] = pack2(a[0][j], a[1][j]);
    }
  for (int c = tid; c < DP; c += blockDim.x) {
    us_[c] = c < d ? u[hd * d + c] : 0.f;
    w0s[c] = c < d ? w0[hd * d + c] : 0.f;
  }

  // staging: LG lanes take a token's key channels
  const int groups = blockDim.x / LG, grp = tid / LG, gl = tid % LG;
  constexpr int LGV = LG, VPER = PER;                                  // the same for a token's value columns (d = dv there)
  float esum[PER][4];
#pragma unroll
  for (int p = 0; p < PER; ++p)
#pragma unroll
    for (int e = 0; e < 4; ++e) esum[p][e] = 0.f;
  const size_t hoff = (size_t)hd * d, voff = (size_t)hd * dv;
  constexpr int CB = 4 * (int)sizeof(T);     // bytes of four operands
  auto request = [&](int t0) {
    const int cnt = min(TT, t_end - t0), dq = d / 4;
    for (int i = tid; i < cnt * dq; i += blockDim.x) {
      const int tt = i / dq, c = (i - tt * dq) * 4;
      const size_t at = (size_t)(t0 + tt) * ld + hoff + c;
      cp_async<16>(zn + tt * DP + c, z + (size_t)(t0 + tt) * (size_t)(H * d) + hoff + c);
      cp_async<CB>(kn + tt * DP + c, k + at);
      if (MODE != 1) cp_async<CB>(rn + tt * DP + c, r + at);
    }
    const int vq = min(CW, dv - col0) / 4;
    for (int i = tid; i < cnt * vq; i += blockDim.x) {
      const int tt = i / vq, c = (i - tt * vq) * 4;
      cp_async<CB>(vn + tt * CW + c, v + (size_t)(t0 + tt) * ld + voff + col0 + c);
      if (MODE != 1 && fin.out != nullptr) cp_async<CB>(gn + (((t0 - t_begin) / TT & 1) * TT + tt) * CW + c, static_cast<const T*>(fin.g) + (size_t)(t0 + tt) * H * dv + voff + c);
    }
    asm volatile("cp.async.commit_group;");
  };
  if (V == 4 && t_begin < t_end) request(t_begin);
  for (int t0 = t_begin; t0 < t_end; t0 += TT) {
    const int cnt = min(TT, t_end - t0);
    if (V == 4) asm volatile("cp.async.wait_group 0;");
    __syncthreads();          // this tile's operands are there, and the tile before has been walked and left
    for (int tt = grp; tt < TT; tt += groups) {       // every lane of a group takes the same turns
      if (tt >= cnt) break;
      const size_t at = (size_t)(t0 + tt);
      float bonus = 0.f;
#pragma unroll
      for (int p = 0; p < PER; ++p) {
        const int c = 4 * (gl + LG * p);
        float rr[4] = {0.f, 0.f, 0.f, 0.f}, kk[4] = {0.f, 0.f, 0.f, 0.f}, zz[4] = {0.f, 0.f, 0.f, 0.f}, ww[4];
        if (V == 4) {
          if (c < d) {
            if (MODE != 1) load_piece<T, 4>(rn + tt * DP + c, rr);
            load_piece<T, 4>(kn + tt * DP + c, kk);
            load_piece<float, 4>(zn + tt * DP + c, zz);
          }
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (c + e < d) {
              if (MODE != 1) rr[e] = to_f32<T>(r[at * ld + hoff + c + e]);
              kk[e] = to_f32<T>(k[at * ld + hoff + c + e]);
              zz[e] = z[at * (size_t)(H * d) + hoff + c + e];
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = expf(zz[e] + w0s[c + e]);
          ww[e] = expf(-x);
          if (MODE == 1) esum[p][e] += x;
          bonus = fmaf(rr[e] * kk[e], us_[c + e], bonus);
        }
        if (MODE != 1) *reinterpret_cast<float4*>(rs_ + tt * DP + c) = make_float4(rr[0], rr[1], rr[2], rr[3]);
        *reinterpret_cast<float4*>(ks_ + tt * DP + c) = make_float4(kk[0], kk[1], kk[2], kk[3]);
        *reinterpret_cast<float4*>(ws_ + tt * DP + c) = make_float4(ww[0], ww[1], ww[2], ww[3]);
      }
      if (MODE != 1) {
        const unsigned mask = LG == 32 ? 0xffffffffu : ((1u << LG) - 1u) << ((tid & 31) / LG * LG);
#pragma unroll
        for (int s = LG / 2; s > 0; s >>= 1) bonus += __shfl_xor_sync(mask, bonus, s);
        if (gl == 0) bs_[tt] = bonus;
      }
    }
    if (V == 4) {
      for (int i = tid; i < cnt * CG; i += blockDim.x) {
        const int tt = i / CG, c = (i % CG) * 4;
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (col0 + c < dv) load_piece<T, 4>(vn + tt * CW + c, f);
        *reinterpret_cast<float4*>(vs_ + tt * CW + c) = make_float4(f[0], f[1], f[2], f[3]);
      }
    } else {
      for (int i = tid; i < cnt * CW; i += blockDim.x) {
        const int tt = i / CW, c = i % CW;
        vs_[tt * CW + c] = col0 + c < dv ? to_f32<T>(v[(size_t)(t0 + tt) * ld + voff + col0 + c]) : 0.f;
      }
    }
    __syncthreads();
    if (V == 4 && t0 + TT < t_end) request(t0 + TT);
    for (int tt = 0; tt < cnt; ++tt) {
      const float4 v4 = *reinterpret_cast<const float4*>(vs_ + tt * CW + cg * COLS);
      const pair_t vv[COLS] = {pack2(v4.x, v4.x), pack2(v4.y, v4.y), pack2(v4.z, v4.z), pack2(v4.w, v4.w)};
      pair_t acc[COLS];
#pragma unroll
      for (int j = 0; j < COLS; ++j) acc[j] = 0ull;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int row = 4 * (rs + RS * q);
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(ks_ + tt * DP + row);
        const ulonglong2 w2 = *reinterpret_cast<const ulonglong2*>(ws_ + tt * DP + row);
        ulonglong2 r2 = make_ulonglong2(0ull, 0ull);
        if (MODE != 1) r2 = *reinterpret_cast<const ulonglong2*>(rs_ + tt * DP + row);
#pragma unroll
        for (int j = 0; j < COLS; ++j) {
          if (MODE != 1) {
            acc[j] = fma2(r2.x, S[j][q * 2], acc[j]);
            acc[j] = fma2(r2.y, S[j][q * 2 + 1], acc[j]);
          }
          S[j][q * 2] = fma2(w2.x, S[j][q * 2], mul2(k2.x, vv[j]));
          S[j][q * 2 + 1] = fma2(w2.y, S[j][q * 2 + 1], mul2(k2.y, vv[j]));
        }
      }
      if (MODE != 1) {
        float a[COLS];
#pragma unroll
        for (int j = 0; j < COLS; ++j) { float lo, hi; unpack2(acc[j], &lo, &hi); a[j] = lo + hi; }
        // the RS threads of a column group add their rows; the first two exchanges also split the columns among them
        int c = 0, left = COLS;
        if (RS >= 2) {
          const bool up = rs & 1;
          const float s0 = up ? a[0] : a[2], s1 = up ? a[1] : a[3];
          const float k0 = up ? a[2] : a[0], k1 = up ? a[3] : a[1];
          a[0] = k0 + __shfl_xor_sync(0xffffffffu, s0, 1);
          a[1] = k1 + __shfl_xor_sync(0xffffffffu, s1, 1);
          c += up ? 2 : 0;
          left = 2;
        }
        if (RS >= 4) {
          const bool up = rs & 2;
          const float s0 = up ? a[0] : a[1], k0 = up ? a[1] : a[0];
          a[0] = k0 + __shfl_xor_sync(0xffffffffu, s0, 2);
          c += up ? 1 : 0;
          left = 1;
        }
        if (RS >= 8) a[0] += __shfl_xor_sync(0xffffffffu, a[0], 4);
        if (RS >= 16) a[0] += __shfl_xor_sync(0xffffffffu, a[0], 8);
        if (RS < 8 || rs < 4) {
          const float bonus = bs_[tt];
#pragma unroll
          for (int j = 0; j < COLS; ++j)
            if (j < left) {
              const int cc = cg * COLS + c + j;
              const float y = fmaf(bonus, vs_[tt * CW + cc], a[j]);
              if (fin.out != nullptr) os_[tt * CW + cc] = y;
              else if (col0 + cc < dv) o[(size_t)(t0 + tt) * H * dv + voff + col0 + cc] = y;
            }
        }
      }
    }
    __syncthreads();
    if (MODE != 1 && fin.out != nullptr) {
      // a tile's read-outs: LGV lanes a token, four value columns each (columns beyond dv hold zeros)
      const T* gate = static_cast<const T*>(fin.g);
      T* out = static_cast<T*>(fin.out);
      const int vgrp = tid / LGV, vl = tid % LGV, vgroups = blockDim.x / LGV;
      for (int tt = vgrp; tt < cnt; tt += vgroups) {
        const size_t at = (size_t)(t0 + tt) * H * dv + voff;
        float y[VPER][4], gg[VPER][4];
        float ss = 0.f;
#pragma unroll
        for (int p = 0; p < VPER; ++p) {
          const int c = 4 * (vl + LGV * p);
#pragma unroll
          for (int e = 0; e < 4; ++e) { y[p][e] = 0.f; gg[p][e] = 0.f; }
          if (c < CW) {
            const float4 y4 = *reinterpret_cast<const float4*>(os_ + tt * CW + c);
            y[p][0] = y4.x; y[p][1] = y4.y; y[p][2] = y4.z; y[p][3] = y4.w;
          }
          if (V == 4) {
            if (c < dv) load_piece<T, 4>(gn + (((t0 - t_begin) / TT & 1) * TT + tt) * CW + c, gg[p]);
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (c + e < dv) gg[p][e] = to_f32<T>(gate[at + c + e]);
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) ss = fmaf(y[p][e], y[p][e], ss);
        }
        const unsigned mask = LGV == 32 ? 0xffffffffu : ((1u << LGV) - 1u) << ((tid & 31) / LGV * LGV);
#pragma unroll
        for (int s = LGV / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(mask, ss, s);
        const float rinv = 1.f / sqrtf(ss / (float)dv + fin.eps);
#pragma unroll
        for (int p = 0; p < VPER; ++p) {
          const int c = 4 * (vl + LGV * p);
          float f[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) f[e] = c + e < dv ? y[p][e] * rinv * fin.norm_w[voff + c + e] * silu(gg[p][e]) : 0.f;
          if (V == 4) {
            if (c < dv) store_piece<T, 4>(out + at + c, f);
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (c + e < dv) out[at + c + e] = from_f32<T>(f[e]);
          }
        }
      }
    }
  }
  if (MODE != 1 && fin.out != nullptr && t_end == cu_q[b + 1]) {      // the sequence's last token of this step: a slice a head
    const T* h = static_cast<const T*>(fin.h) + (size_t)(t_end - 1) * fin.width;
    T* last = static_cast<T*>(fin.last) + (size_t)slot * fin.width;
    for (int c = hd * blockDim.x + tid; c < fin.width; c += H * blockDim.x) last[c] = h[c];
  }
  // MODE 0: the slot's new state; MODE 1: the chunk's own state
#pragma unroll
  for (int q = 0; q < (MODE == 2 ? 0 : 4); ++q)
#pragma unroll
    for (int i = 0; i < 4; i += 2) {
      const int row = 4 * (rs + RS * q) + i;
#pragma unroll
      for (int j = 0; j < COLS; ++j) {
        float lo, hi;
        unpack2(S[j][q * 2 + i / 2], &lo, &hi);
        if (c0 + j < dv) {
          if (row < d) start[(size_t)row * dv + c0 + j] = lo;
          if (row + 1 < d) start[(size_t)(row + 1) * dv + c0 + j] = hi;
        }
      }
    }
  if constexpr (MODE == 1) {
    if (blockIdx.z != 0) return;           // the chunk's decays: exp of minus the sum over its tokens
#pragma unroll
    for (int p = 0; p < PER; ++p)
#pragma unroll
      for (int e = 0; e < 4; ++e) ds_[grp * DP + 4 * (gl + LG * p) + e] = esum[p][e];
    __syncthreads();
    for (int c = tid; c < d; c += blockDim.x) {
      float s = 0.f;
      for (int g = 0; g < groups; ++g) s += ds_[g * DP + c];
      cdecay[((size_t)blockIdx.x * H + hd) * d + c] = expf(-s);
    }
  }
}

__global__ void __launch_bounds__(256) wkv_prefix_kernel(const int* __restrict__ cu_q, const int* __restrict__ seq_slot, int cht, int H, int d,
                                                       int dv, float* __restrict__ state, float* __restrict__ cstate,
                                                       const float* __restrict__ cdecay) {
  const int b = blockIdx.x;
  const size_t per = (size_t)H * d * dv, e = (size_t)blockIdx.y * 256 + threadIdx.x;
  const int slot = seq_slot[b];
  if (slot < 0 || e >= per) return;
  int first = 0;
  for (int bb = 0; bb < b; ++bb) first += (cu_q[bb + 1] - cu_q[bb] + cht - 1) / cht;
  const int nc = (cu_q[b + 1] - cu_q[b] + cht - 1) / cht;
  const size_t row = e / dv;               // (head, key channel)
  float S = state[(size_t)slot * per + e];
  constexpr int AHEAD = 8;                 // chunks whose states and decays are requested before the first is used
  for (int k0 = 0; k0 < nc; k0 += AHEAD) {
    float own[AHEAD], dec[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      own[i] = k0 + i < nc ? cstate[(size_t)(first + k0 + i) * per + e] : 0.f;
      dec[i] = k0 + i < nc ? cdecay[(size_t)(first + k0 + i) * H * d + row] : 1.f;
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (k0 + i < nc) cstate[(size_t)(first + k0 + i) * per + e] = S;
      S = fmaf(dec[i], S, own[i]);         // behind the last chunk: 1 * S + 0
    }
  }
  state[(size_t)slot * per + e] = S;
}

constexpr int NORM_WARPS = 8;
template <typename T>
__global__ void __launch_bounds__(NORM_WARPS * 32) wkv_norm_kernel(const float* __restrict__ o, const T* __restrict__ g, int ld,
                                                                const float* __restrict__ norm_w, float eps, const T* __restrict__ h, int width,
                                                                T* __restrict__ last, const int* __restrict__ tok_slot, int n, int H, int dv,
                                                                T* __restrict__ out) {
  const int t = blockIdx.x, slot = tok_slot[t];
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int hd = warp; hd < H; hd += NORM_WARPS) {
    const float* row = o + (size_t)t * H * dv + (size_t)hd * dv;
    const T* gr = g + (size_t)t * ld + (size_t)hd * dv;
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) { const float x = row[c]; ss = fmaf(x, x, ss); }
    const float rinv = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
    for (int c = lane; c < dv; c += 32)
      out[(size_t)t * H * dv + (size_t)hd * dv + c] = from_f32<T>(row[c] * rinv * norm_w[hd * dv + c] * silu(to_f32<T>(gr[c])));
  }
  if (t + 1 == n || tok_slot[t + 1] != slot)      // the sequence's last token of this step
    for (int c = threadIdx.x; c < width; c += NORM_WARPS * 32) last[(size_t)slot * width + c] = h[(size_t)t * width + c];
}

constexpr int DEC_THREADS = 256, DEC_LANES = 8;     // lanes that share a key channel's decay

template <typename T>
__global__ void __launch_bounds__(DEC_THREADS) wkv_decode_kernel(
    const float* __restrict__ r, const float* __restrict__ k, const float* __restrict__ v, const float* __restrict__ g, int ld,
    const float* __restrict__ low, int low_ld, int R, const T* __restrict__ w2, const float* __restrict__ w0, const float* __restrict__ u,
    const float* __restrict__ norm_w, float eps, const T* __restrict__ h, int width, T* __restrict__ last, const int* __restrict__ tok_slot, int H,
    int d, int dv, float* __restrict__ state, T* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];      // r, k, w [d each], v [dv], tanh(low) [R], partial read-outs [row groups][dv]
  __shared__ float scratch[33];
  const int t = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x;
  const int slot = tok_slot[t];
  if (slot < 0) return;
  float* rsm = sm;
  float* ksm = rsm + d;
  float* wsm = ksm + d;
  float* vsm = wsm + d;
  float* tl = vsm + dv;
  float* red = tl + R;
  // a thread owns one value column and every RG-th row of it
  const int CT = min(dv, DEC_THREADS), RG = DEC_THREADS / CT;
  const int col = tid % CT, rg = tid / CT;
  float* S = state + ((size_t)slot * H + hd) * (size_t)d * dv;
  constexpr int AHEAD = 16;
  float pre[AHEAD];                                // the first rows are requested before anything else
  const bool mine = rg < RG;
#pragma unroll
  for (int i = 0; i < AHEAD; ++i) {
    const int row = rg + RG * i;
    pre[i] = mine && row < d ? S[(size_t)row * dv + col] : 0.f;
  }
  for (int c = tid; c < d; c += DEC_THREADS) {
    rsm[c] = r[(size_t)t * ld + (size_t)hd * d + c];
    ksm[c] = k[(size_t)t * ld + (size_t)hd * d + c];
  }
  for (int c = tid; c < dv; c += DEC_THREADS) vsm[c] = v[(size_t)t * ld + (size_t)hd * dv + c];
  for (int c = tid; c < R; c += DEC_THREADS) tl[c] = tanhf(low[(size_t)t * low_ld + c]);
  for (int c = hd * DEC_THREADS + tid; c < width; c += H * DEC_THREADS) last[(size_t)slot * width + c] = h[(size_t)t * width + c];
  __syncthreads();
  // decays: eight lanes a key channel
  const int ln = tid % DEC_LANES;
  constexpr int VN = 16 / (int)sizeof(T);
  for (int c0 = 0; c0 < d; c0 += DEC_THREADS / DEC_LANES) {
    const int c = c0 + tid / DEC_LANES;
    float a = 0.f;
    if (c < d) {
      const T* wr = w2 + ((size_t)hd * d + c) * R;
      if (R % VN == 0) {
        for (int j = ln * VN; j < R; j += DEC_LANES * VN) {
          float f[VN];
          load_piece<T, VN>(wr + j, f);
#pragma unroll
          for (int e = 0; e < VN; ++e) a = fmaf(f[e], tl[j + e], a);
        }
      } else {
        for (int j = ln; j < R; j += DEC_LANES) a = fmaf(to_f32<T>(wr[j]), tl[j], a);
      }
    }
#pragma unroll
    for (int s = DEC_LANES / 2; s > 0; s >>= 1) a += __shfl_xor_sync(0xffffffffu, a, s);
    if (c < d && ln == 0) wsm[c] = expf(-expf(a + w0[(size_t)hd * d + c]));
  }
  float bp = 0.f;
  for (int c = tid; c < d; c += DEC_THREADS) bp = fmaf(rsm[c] * ksm[c], u[(size_t)hd * d + c], bp);
  const float bonus = block_sum(bp, scratch);       // its barriers also make the decays visible
  float ss = 0.f;
  for (int cb = 0; cb < dv; cb += CT) {             // one pass where a head's values fit the block's threads
    const int cc = cb + col;
    float acc = 0.f;
    if (mine && cc < dv) {
      const float vv = vsm[cc];
      for (int i0 = 0; rg + RG * i0 < d; i0 += AHEAD) {
        float cur[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
          const int row = rg + RG * (i0 + i);
          cur[i] = (i0 == 0 && cb == 0) ? pre[i] : (row < d ? S[(size_t)row * dv + cc] : 0.f);
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
          const int row = rg + RG * (i0 + i);
          if (row < d) {
            acc = fmaf(rsm[row], cur[i], acc);
            S[(size_t)row * dv + cc] = fmaf(wsm[row], cur[i], ksm[row] * vv);
          }
        }
      }
      red[(size_t)rg * dv + cc] = acc;
    }
  }
  __syncthreads();
  for (int c = tid; c < dv; c += DEC_THREADS) {
    float a = 0.f;
    for (int i = 0; i < RG; ++i) a += red[(size_t)i * dv + c];
    a = fmaf(bonus, vsm[c], a);
    vsm[c] = a;                                     // the thread's own entry
    ss = fmaf(a, a, ss);
  }
  const float rinv = 1.f / sqrtf(block_sum(ss, scratch) / (float)dv + eps);
  for (int c = tid; c < dv; c += DEC_THREADS)
    out[(size_t)t * H * dv + (size_t)hd * dv + c] =
        from_f32<T>(vsm[c] * rinv * norm_w[(size_t)hd * dv + c] * silu(g[(size_t)t * ld + (size_t)hd * dv + c]));
}

struct Walk {
  const void *r, *k, *v; int ld; const float *z, *w0, *u; const int *cu_q, *seq_slot; int n_seqs, cht, H, d, dv; float *state, *cstate, *cdecay, *o;
  Finish fin;
};

template <typename T, int RS, int MODE, int V>
int walk_mode(const Walk& a, int blocks_x, cudaStream_t st) {
  constexpr int TT = 8, DP = RS * ROWS, LG = DP / 4 < 32 ? DP / 4 : 32;
  int cg = (a.dv + COLS - 1) / COLS;
  const int least = (32 + RS - 1) / RS, most = 256 / RS;
  cg = cg > most ? most : cg;
  const int unit = least;                      // whole warps
  cg = (cg + unit - 1) / unit * unit;
  if (cg > most) cg = most;
  const int slices = (a.dv + cg * COLS - 1) / (cg * COLS), threads = RS * cg;
  const size_t smem = sizeof(float) * ((size_t)TT * (3 * DP + cg * COLS + 1) + 2 * DP + (MODE == 1 ? (size_t)(threads / LG) * DP : (size_t)TT * cg * COLS)) +
                      (V == 4 ? TT * (sizeof(float) * DP + sizeof(T) * (2 * DP + 3 * (size_t)cg * COLS)) : 0);
  if (smem > 200 * 1024) return DRYFT_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(wkv_walk_kernel<T, RS, MODE, V, TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  dim3 grid(blocks_x, a.H, slices);
  wkv_walk_kernel<T, RS, MODE, V, TT><<<grid, threads, smem, st>>>((const T*)a.r, (const T*)a.k, (const T*)a.v, a.ld, a.z, a.w0, a.u, a.cu_q, a.seq_slot,
                                                                 a.n_seqs, a.cht, a.H, a.d, a.dv, a.state, a.cstate, a.cdecay, a.o, a.fin);
  return launch_status();
}

template <typename T, int RS, int V>
int walk_all(const Walk& a, int n_chunks, cudaStream_t st) {
  if (n_chunks <= 0) return walk_mode<T, RS, 0, V>(a, a.n_seqs, st);
  int e = walk_mode<T, RS, 1, V>(a, n_chunks, st);
  if (e) return e;
  const size_t per = (size_t)a.H * a.d * a.dv;
  wkv_prefix_kernel<<<dim3(a.n_seqs, (unsigned)((per + 255) / 256)), 256, 0, st>>>(a.cu_q, a.seq_slot, a.cht, a.H, a.d, a.dv, a.state, a.cstate,
                                                                                 a.cdecay);
  e = launch_status();
  if (e) return e;
  return walk_mode<T, RS, 2, V>(a, n_chunks, st);
}

template <typename T>
int walk_sizes(const Walk& a, int n_chunks, cudaStream_t st) {
  const bool vec = a.d % 4 == 0 && a.dv % 4 == 0 && a.ld % 4 == 0 &&
                   (((uintptr_t)a.r | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.z | (uintptr_t)a.fin.g | (uintptr_t)a.fin.out) & 15) == 0;
#define DRYFT_WALK(RS) return vec ? walk_all<T, RS, 4>(a, n_chunks, st) : walk_all<T, RS, 1>(a, n_chunks, st)
  if (a.d <= 16) { DRYFT_WALK(1); }
  if (a.d <= 32) { DRYFT_WALK(2); }
  if (a.d <= 64) { DRYFT_WALK(4); }
  if (a.d <= 128) { DRYFT_WALK(8); }
  if (a.d <= 256) { DRYFT_WALK(16); }
#undef DRYFT_WALK
  return DRYFT_ERR_UNSUPPORTED;
}

template <typename T>
int mix_launch(const void* h, const void* last, const float* mu, const int* tok_slot, void* out, int n, int width, cudaStream_t st) {
  const bool vec = width % 8 == 0 && (((uintptr_t)h | (uintptr_t)last | (uintptr_t)mu | (uintptr_t)out) & 15) == 0;
  const int per = MIX_THREADS * (vec ? 8 : 1);
  dim3 grid(n, (width + per - 1) / per);
  if (vec) wkv_mix_kernel<T, 8><<<grid, MIX_THREADS, 0, st>>>((const T*)h, (const T*)last, mu, tok_slot, (T*)out, n, width);
  else wkv_mix_kernel<T, 1><<<grid, MIX_THREADS, 0, st>>>((const T*)h, (const T*)last, mu, tok_slot, (T*)out, n, width);
  return launch_status();
}
}  // namespace

DRYFT_API int dryft_wkv_mix(int is_bf16, const void* h, const void* last, const float* mu, const int* tok_slot, void* out, int n, int width,
                            cudaStream_t st) {
  if (n <= 0) return 0;
  if (width < 1) return DRYFT_ERR_UNSUPPORTED;
  return is_bf16 ? mix_launch<__nv_bfloat16>(h, last, mu, tok_slot, out, n, width, st) : mix_launch<float>(h, last, mu, tok_slot, out, n, width, st);
}

DRYFT_API int dryft_wkv_tanh(int is_bf16, const float* low, void* out, long long count, cudaStream_t st) {
  if (count <= 0) return 0;
  const unsigned blocks = (unsigned)((count + 255) / 256);
  if (is_bf16) wkv_tanh_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>(low, (__nv_bfloat16*)out, (size_t)count);
  else wkv_tanh_kernel<float><<<blocks, 256, 0, st>>>(low, (float*)out, (size_t)count);
  return launch_status();
}

// head sizes up to this run the norm and the gate inside the walk (a block holds all of a head's value columns)
DRYFT_API int dryft_wkv_fused_dim() { return 128; }

// `out` given (d = dv up to dryft_wkv_fused_dim): norm, gate and the step's last inputs inside; else the read-outs go to o.
// n_chunks = 0: the tokens of each sequence in order (one launch); else the chunked form (three launches) with scratch
// cstate [n_chunks, H, d, dv] and cdecay [n_chunks, H, d], n_chunks at least the number of chunks of `cht` tokens in the step.
DRYFT_API int dryft_wkv_walk(int is_bf16, const void* r, const void* k, const void* v, int ld, const float* z, const float* w0, const float* u,
                             const int* cu_q, const int* seq_slot, int n_seqs, int cht, int n_chunks, int H, int d, int dv, float* state,
                             float* cstate, float* cdecay, float* o, const void* g, const float* norm_w, float eps, const void* h, int width,
                             void* last, void* out, cudaStream_t st) {
  if (n_seqs <= 0) return 0;
  if (out == nullptr && o == nullptr) return DRYFT_ERR_UNSUPPORTED;
  if (out != nullptr && (d != dv || d > dryft_wkv_fused_dim() || ld != H * dv || !g || !norm_w || !h || !last || width < 1)) return DRYFT_ERR_UNSUPPORTED;
  if (H < 1 || H > 65535 || d < 1 || d > 256 || dv < 1 || (n_chunks > 0 && (cht <= 0 || !cstate || !cdecay))) return DRYFT_ERR_UNSUPPORTED;
  Walk a{r, k, v, ld, z, w0, u, cu_q, seq_slot, n_seqs, cht, H, d, dv, state, cstate, cdecay, o, {g, norm_w, eps, h, width, last, out}};
  return is_bf16 ? walk_sizes<__nv_bfloat16>(a, n_chunks, st) : walk_sizes<float>(a, n_chunks, st);
}

DRYFT_API int dryft_wkv_norm(int is_bf16, const float* o, const void* g, int ld, const float* norm_w, float eps, const void* h, int width,
                             void* last, const int* tok_slot, int n, int H, int dv, void* out, cudaStream_t st) {
  if (n <= 0) return 0;
  if (H < 1 || dv < 1 || width < 1) return DRYFT_ERR_UNSUPPORTED;
  typedef __nv_bfloat16 bf;
  if (is_bf16)
    wkv_norm_kernel<bf><<<n, NORM_WARPS * 32, 0, st>>>(o, (const bf*)g, ld, norm_w, eps, (const bf*)h, width, (bf*)last, tok_slot, n, H, dv, (bf*)out);
  else
    wkv_norm_kernel<float><<<n, NORM_WARPS * 32, 0, st>>>(o, (const float*)g, ld, norm_w, eps, (const float*)h, width, (float*)last, tok_slot, n, H,
                                                        dv, (float*)out);
  return launch_status();
}

DRYFT_API int dryft_wkv_decode(int is_bf16, const float* r, const float* k, const float* v, const float* g, int ld, const float* low, int low_ld,
                               int R, const void* w2, const float* w0, const float* u, const float* norm_w, float eps, const void* h, int width,
                               void* last, const int* tok_slot, int n, int H, int d, int dv, float* state, void* out, cudaStream_t st) {
  if (n <= 0) return 0;
  if (H < 1 || H > 65535 || d < 1 || dv < 1 || R < 1 || width < 1) return DRYFT_ERR_UNSUPPORTED;
  const int ct = dv < DEC_THREADS ? dv : DEC_THREADS;
  const size_t smem = sizeof(float) * ((size_t)3 * d + dv + R + (size_t)(DEC_THREADS / ct) * dv);
  if (smem > 48 * 1024) return DRYFT_ERR_UNSUPPORTED;
  dim3 grid(n, H);
  typedef __nv_bfloat16 bf;
  if (is_bf16)
    wkv_decode_kernel<bf><<<grid, DEC_THREADS, smem, st>>>(r, k, v, g, ld, low, low_ld, R, (const bf*)w2, w0, u, norm_w, eps, (const bf*)h, width,
                                                         (bf*)last, tok_slot, H, d, dv, state, (bf*)out);
  else
    wkv_decode_kernel<float><<<grid, DEC_THREADS, smem, st>>>(r, k, v, g, ld, low, low_ld, R, (const float*)w2, w0, u, norm_w, eps,
                                                            (const float*)h, width, (float*)last, tok_slot, H, d, dv, state, (float*)out);
  return launch_status();
}
