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

// The input of channel c at step index i of its sequence (i < 0: before this step), for a sequence whose first token of the
// step is packed row t0 at position p0.  x points at channel 0 of packed row 0, row stride ld.
template <typename T>
__device__ __forceinline__ float conv_input(const T* __restrict__ x, int ld, const T* __restrict__ ring, int taps, int CH,
                                            int slot, int t0, int p0, int i, int c) {
  if (i >= 0) return to_f32<T>(x[(size_t)(t0 + i) * ld + c]);
  const int p = p0 + i;
  return p >= 0 ? to_f32<T>(ring[((size_t)slot * taps + p % taps) * CH + c]) : 0.f;
}

// acc[k] = the convolution's result at step indices i0 + k, k = 0..3, of channel c; tokens from index n on do not exist
template <typename T>
__device__ __forceinline__ void conv4(float (&acc)[4], const float* __restrict__ w, const T* __restrict__ x, int ld,
                                      const T* __restrict__ ring, int taps, int CH, int slot, int t0, int p0, int i0, int n, int c) {
#pragma unroll
  for (int k = 0; k < 4; ++k) acc[k] = 0.f;
  const float* wc = w + (size_t)c * taps;
  if (taps == 4) {      // the usual case, unrolled: seven inputs, four weights
    const float w0 = wc[0], w1 = wc[1], w2 = wc[2], w3 = wc[3];
    float u[7];
#pragma unroll
    for (int s = 0; s < 7; ++s) {
      const int i = i0 - 3 + s;
      u[s] = i < n ? conv_input<T>(x, ld, ring, taps, CH, slot, t0, p0, i, c) : 0.f;
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) acc[k] = fmaf(w3, u[k + 3], fmaf(w2, u[k + 2], fmaf(w1, u[k + 1], w0 * u[k])));
    return;
  }
  for (int s = 0; s < taps + 3; ++s) {
    const int i = i0 - (taps - 1) + s;
    if (i >= n) break;
    const float u = conv_input<T>(x, ld, ring, taps, CH, slot, t0, p0, i, c);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int j = s - k;
      if (j >= 0 && j < taps) acc[k] = fmaf(wc[j], u, acc[k]);
    }
  }
}

// the convolution's result of ONE token (packed row t at position p), of channel c: `back` of the rows before it belong to
// its sequence and this step
template <typename T>
__device__ __forceinline__ float conv1(const float* __restrict__ w, const T* __restrict__ x, int ld, const T* __restrict__ ring,
                                       int taps, int CH, int slot, int t, int p, int back, int c) {
  const float* wc = w + (size_t)c * taps;
  float acc = 0.f;
  for (int j = 0; j < taps; ++j) {
    const int d = taps - 1 - j;
    float u = 0.f;
    if (d <= back) u = to_f32<T>(x[(size_t)(t - d) * ld + c]);
    else if (p - d >= 0) u = to_f32<T>(ring[((size_t)slot * taps + (p - d) % taps) * CH + c]);
    acc = fmaf(wc[j], u, acc);
  }
  return acc;
}
