// A short causal convolution over time per channel, whose memory is a ring: the projected value of the token at position p
// of a sequence lies in row p % taps of  ring [slots, taps, CH]  (CH channels, activation type T).  A token at position p
// needs the values of p - 1 .. p - taps + 1, none of which shares a row with p: a decode step may therefore store its own
// value in the launch that reads the others, whoever reads them.  A step of many tokens stores its last taps - 1 values in a
// launch behind the one that reads (conv_ring_store).  Values before a sequence's start are zeros (never read).
//
//     y_t[c] = sum_j w[c, j] * u_(t - taps + 1 + j)[c]          (w [CH, taps]: the last column is the current token's)
#pragma once
#include "common.cuh"

#define DRYFT_CONV_MAX_TAPS 16

// The input of channel c at step index i of its sequence (i < 0: before this step; n: the step's tokens of the sequence), for a
// sequence whose first token of the step is packed row t0 at position p0.  x points at channel 0 of packed row 0, row stride ld.
// The address is chosen without a branch, so that a run's loads are all on their way at once; what does not exist (before the
// sequence's start, behind its end) reads the step's first row and counts as zero.
template <typename T>
__device__ __forceinline__ float conv_input(const T* __restrict__ x, int ld, const T* __restrict__ ring, int taps, int CH,
                                            int slot, int t0, int p0, int i, int n, int c) {
  const int p = p0 + i;
  const bool here = i >= 0 && i < n, before = i < 0 && p >= 0;
  const T* src = x + (size_t)(here ? t0 + i : t0) * ld + c;
  if (before) src = ring + ((size_t)slot * taps + (taps == 4 ? p & 3 : p % taps)) * CH + c;
  const float u = to_f32<T>(*src);
  return here || before ? u : 0.f;
}

// acc[k] = the convolution's result at step indices i0 + k, k < N, of channel c
template <typename T, int N>
__device__ __forceinline__ void conv_run(float (&acc)[N], const float* __restrict__ w, const T* __restrict__ x, int ld,
                                         const T* __restrict__ ring, int taps, int CH, int slot, int t0, int p0, int i0, int n, int c) {
  const float* wc = w + (size_t)c * taps;
  if (taps == 4) {      // the usual case, unrolled
    const float4 ww = *reinterpret_cast<const float4*>(wc);
    float u[N + 3];
    if (i0 >= 3 && i0 + N <= n) {      // all inputs belong to this step
      const T* src = x + (size_t)(t0 + i0 - 3) * ld + c;
#pragma unroll
      for (int s = 0; s < N + 3; ++s) u[s] = to_f32<T>(src[(size_t)s * ld]);
    } else {
#pragma unroll
      for (int s = 0; s < N + 3; ++s) u[s] = conv_input<T>(x, ld, ring, 4, CH, slot, t0, p0, i0 - 3 + s, n, c);
    }
#pragma unroll
    for (int k = 0; k < N; ++k) acc[k] = fmaf(ww.w, u[k + 3], fmaf(ww.z, u[k + 2], fmaf(ww.y, u[k + 1], ww.x * u[k])));
    return;
  }
#pragma unroll
  for (int k = 0; k < N; ++k) acc[k] = 0.f;
#pragma unroll 1
  for (int j = 0; j < taps; ++j) {
    const float wj = wc[j];
#pragma unroll
    for (int k = 0; k < N; ++k) acc[k] = fmaf(wj, conv_input<T>(x, ld, ring, taps, CH, slot, t0, p0, i0 + k - (taps - 1) + j, n, c), acc[k]);
  }
}

// The rows that the convolution of ONE token (packed row t at position p) reads, worked out once for all its channels: `back`
// of the rows before t belong to its sequence and this step, older ones lie in the ring, and a row before the sequence's
// start counts as zeros (its weight is dropped; the pointer then names the token's own row).
template <typename T> struct ConvRows {
  const T* src[4];
  float on[4];
  const float* w;
  const T* x;
  const T* ring_slot;
  int ld, taps, CH, t, p, back;

  __device__ __forceinline__ ConvRows(const float* __restrict__ w_, const T* __restrict__ x_, int ld_, const T* __restrict__ ring, int taps_,
                                      int CH_, int slot, int t_, int p_, int back_)
      : w(w_), x(x_), ring_slot(ring + (size_t)slot * taps_ * CH_), ld(ld_), taps(taps_), CH(CH_), t(t_), p(p_), back(back_) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = 3 - j;
      const bool seen = d <= back || p >= d;
      on[j] = seen ? 1.f : 0.f;
      src[j] = d <= back || !seen || taps != 4 ? x + (size_t)(t - (seen && d <= back ? d : 0)) * ld : ring_slot + (size_t)((p - d) & 3) * CH;
    }
  }
  __device__ __forceinline__ float operator()(int c) const {
    const float* wc = w + (size_t)c * taps;
    if (taps == 4) {
      const float4 ww = *reinterpret_cast<const float4*>(wc);
      const float u0 = to_f32<T>(src[0][c]), u1 = to_f32<T>(src[1][c]), u2 = to_f32<T>(src[2][c]), u3 = to_f32<T>(src[3][c]);
      return fmaf(ww.w, u3, fmaf(ww.z * on[2], u2, fmaf(ww.y * on[1], u1, ww.x * on[0] * u0)));
    }
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int d = taps - 1 - j;
      float u = 0.f;
      if (d <= back) u = to_f32<T>(x[(size_t)(t - d) * ld + c]);
      else if (p >= d) u = to_f32<T>(ring_slot[(size_t)((p - d) % taps) * CH + c]);
      acc = fmaf(wc[j], u, acc);
    }
    return acc;
  }
};
