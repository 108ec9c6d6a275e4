// Sliding-window attention with pooled blocks and a sink, over the paged cache.  Compiled for one key size D
// (DRYFT_QK_DIM), one value size DV (DRYFT_V_DIM) and REP query heads per key/value head (DRYFT_GROUP).
//
// The query at position i of its sequence sees the tokens j with 0 <= i - j < size and, beside them, ONE key and value
// for every block of P positions that lies wholly before the window (block b = positions bP .. bP + P - 1, seen when
// bP + P - 1 <= i - size): the mean of the block's P cached keys and the mean of its P cached values, kept in pages of
// their own, one row per block.  Tokens and blocks share one softmax, whose denominator also holds exp(sink_h), a
// number per head without key or value.  `keep` > 0: the first `keep` tokens of the sequence stay visible whatever the window
// (each key once; their cached rows are those of their true positions).  Scores, weights and sums are 32-bit; q, k, v and the pooled rows have the
// activation type T.
//
//   pool_attn_prep    per token: q, k (+ bias) rotated over their first `rot` dims (dims i and i + rot/2 turn together by
//                     the angle pos * inv_freq[i], evaluated in 32-bit), THEN divided by their root mean square over D
//                     (no weight; skipped when eps < 0); v (+ bias); k and v written into the cache at the token's position.  A warp a vector, or several of
//                     one token in a step of many tokens.
//                     `v_eps` >= 0: each value head is divided by its root mean square too, and cached so.  `qt_every` > 0: the
//                     query of position p is multiplied by 1 + qt_coef * ln((p + 1) / qt_every + 1), whole quotient.
//                     With convolution weights (shortconv.cuh) q, k and v first pass a short causal convolution per channel
//                     of [q | k | v], and a decode step stores its own projected values in the convolution's ring.
//   pool_attn_prep_run  the same behind a convolution for steps of many tokens: a block a run of eight tokens, a warp a vector of
//                     all of them.
//   pool_attn_prep_tok  the same per token for projections that are normed as a whole: q (all H * D values at once) and k (all
//                     G * D) are divided by their root mean square and multiplied by a weight per entry BEFORE the rotation,
//                     and the rotation pairs either dims i and i + rot/2 or (interleaved) dims 2i and 2i + 1.  One block a
//                     token: the two sums of squares first, then a warp a vector.
//   pool_attn_blocks  every token that completes a block (pos % P == P - 1) averages the block's P cached keys and
//                     values into the pooled pages.  One block per (token, kv head); all others return at once.
//   pool_attn_rows    one block per (token, kv head, split): the REP query heads of the kv head over the visible pooled
//                     rows and tokens (one list of keys; a lane a key for the scores, a lane a value column for the
//                     weighted sum), online softmax per warp, warps combined in shared memory; with one split the sink
//                     joins there and the output is written, else partial (max, sum, weighted sum) go to memory and
//   pool_attn_combine joins the splits and the sink.  With `gate` logits every output value is multiplied by the sigmoid of its own.
// Tokens with slot -1 (padding) are skipped.  No block waits on another block.
#include "shortconv.cuh"
#include <math.h>

#ifndef DRYFT_QK_DIM
#error "compile with -DDRYFT_QK_DIM, -DDRYFT_V_DIM and -DDRYFT_GROUP"
#endif

namespace {
constexpr int D = DRYFT_QK_DIM, DV = DRYFT_V_DIM, REP = DRYFT_GROUP;
constexpr int DR = (D + 31) / 32, DVR = (DV + 31) / 32;
constexpr int ROWS_WARPS = 4;
constexpr int BLOCKS_THREADS = (D + DV + 31) / 32 * 32 < 1024 ? (D + DV + 31) / 32 * 32 : 1024;   // a thread a column of a key or a value
constexpr int PREP_WARPS = 4;
constexpr int PREP_TOK_WARPS = 8;    // pool_attn_prep_tok: a block a token, its vectors dealt to the warps

// sin and cos of  pos * (f_hi + f_lo): the product is formed in 32-bit, and what its rounding drops (recovered exactly with
// one fused multiply-add) plus the low half of the frequency are applied as a first-order turn.  f_lo = 0 gives the plain
// 32-bit angle to within that correction.
__device__ __forceinline__ void sincos_split(float pos, float f_hi, float f_lo, float* sn, float* cs) {
  const float a = pos * f_hi;
  const float e = fmaf(pos, f_hi, -a) + pos * f_lo;
  float s, c;
  sincosf(a, &s, &c);
  *sn = fmaf(e, c, s);
  *cs = fmaf(-e, s, c);
}

template <typename T>
__global__ void __launch_bounds__(PREP_WARPS * 32) pool_attn_prep_kernel(
    const T* __restrict__ proj, int ld, const float* __restrict__ qb, const float* __restrict__ kb, const float* __restrict__ vb,
    const float* __restrict__ inv_freq, const float* __restrict__ inv_freq_lo, int rot, const int* __restrict__ tok_slot,
    const int* __restrict__ tok_pos, T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages, const int* __restrict__ page_table, int max_pages,
    int page_size, int n_tokens, int H, int G, float eps, int write_kv, const float* __restrict__ conv_w, int taps, T* __restrict__ ring,
    int store_ring, int per_warp, float v_eps, float qt_coef, int qt_every) {
  __shared__ float sm[PREP_WARPS][D > DV ? D : DV];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per_tok = H + (write_kv ? 2 * G : 0), parts = (per_tok + per_warp - 1) / per_warp;
  const long long item = (long long)blockIdx.x * PREP_WARPS + warp;
  if (item >= (long long)n_tokens * parts) return;
  const int t = (int)(item / parts), vec0 = (int)(item % parts) * per_warp, vec1 = min(per_tok, vec0 + per_warp);
  const int slot = tok_slot[t];
  if (slot < 0) return;
  const int pos = tok_pos[t];
  const T* row = proj + (size_t)t * ld;
  const int CH = H * D + G * (D + DV);
  int back = 0;              // rows before this one that belong to its sequence and this step, as far as the convolution looks
  if (conv_w != nullptr)
    while (back < taps - 1 && t - back - 1 >= 0 && tok_slot[t - back - 1] == slot) ++back;
  // channel c of [q | k | v]: the projected value, or the convolution over it
  const ConvRows<T> conv(conv_w, proj, ld, ring, conv_w != nullptr ? taps : 4, CH, slot, t, pos, back);
  T* ring_row = store_ring ? ring + ((size_t)slot * taps + pos % taps) * CH : nullptr;
  auto input = [&](int c) {
    if (conv_w == nullptr) return to_f32<T>(row[c]);
    if (store_ring) ring_row[c] = row[c];
    return conv(c);
  };
  // the token's angles, once for all its vectors: entry c turns with its partner half a rotation away
  const int half = rot / 2;
  float sn[DR], cs[DR];
#pragma unroll
  for (int r = 0; r < DR; ++r) {
    const int c = lane + 32 * r;
    sn[r] = 0.f;
    cs[r] = 1.f;
    if (vec0 < H + G && c < rot) {
      const int i = c < half ? c : c - half;
      sincos_split((float)pos, inv_freq[i], inv_freq_lo != nullptr ? inv_freq_lo[i] : 0.f, &sn[r], &cs[r]);
      if (c < half) sn[r] = -sn[r];
    }
  }
  float* s = sm[warp];
  for (int vec = vec0; vec < vec1; ++vec) {
    size_t cache_row = 0;
    if (vec >= H) {
      const int g = (vec - H) % G;
      const int page = page_table[(size_t)slot * max_pages + pos / page_size];
      cache_row = ((size_t)page * G + g) * page_size + pos % page_size;
    }
    if (vec >= H + G) {     // a value vector: bias, cache
      const int g = vec - H - G, src = H * D + G * D + g * DV;
      if (v_eps >= 0.f) {   // divided by its root mean square
        float vv[DVR];
        float ss = 0.f;
#pragma unroll
        for (int r = 0; r < DVR; ++r) {
          const int c = lane + 32 * r;
          vv[r] = c < DV ? input(src + c) + (vb != nullptr ? vb[g * DV + c] : 0.f) : 0.f;
          ss = fmaf(vv[r], vv[r], ss);
        }
        const float vinv = 1.f / sqrtf(warp_sum(ss) / (float)DV + v_eps);
#pragma unroll
        for (int r = 0; r < DVR; ++r) {
          const int c = lane + 32 * r;
          if (c < DV) v_pages[cache_row * DV + c] = from_f32<T>(vv[r] * vinv);
        }
        continue;
      }
      for (int c = lane; c < DV; c += 32)
        v_pages[cache_row * DV + c] = from_f32<T>(input(src + c) + (vb != nullptr ? vb[g * DV + c] : 0.f));
      continue;
    }
    const bool is_q = vec < H;
    const int hd = is_q ? vec : vec - H;
    const int src = is_q ? hd * D : H * D + hd * D;
    const float* bias = is_q ? qb : kb;
    __syncwarp();           // the vector before this one has been read
    for (int c = lane; c < D; c += 32) s[c] = input(src + c) + (bias != nullptr ? bias[hd * D + c] : 0.f);
    __syncwarp();
    float o[DR];
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < DR; ++r) {
      const int c = lane + 32 * r;
      float v = 0.f;
      if (c < D) v = c < rot ? s[c] * cs[r] + s[c < half ? c + half : c - half] * sn[r] : s[c];
      o[r] = v;
      ss = fmaf(v, v, ss);
    }
    float rinv = 1.f;                                                      // eps < 0: no unit norm
    if (eps >= 0.f) rinv = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);
    if (is_q && qt_every > 0) rinv *= fmaf(qt_coef, logf((float)((pos + 1) / qt_every + 1)), 1.f);
    T* dst = is_q ? q_out + ((size_t)t * H + hd) * D : k_pages + cache_row * D;
#pragma unroll
    for (int r = 0; r < DR; ++r) {
      const int c = lane + 32 * r;
      if (c < D) dst[c] = from_f32<T>(o[r] * rinv);
    }
  }
}

// The same behind a convolution, for steps of many tokens: a block takes RUN consecutive tokens of one sequence (part
// blockIdx.y of tile blockIdx.x), a warp a vector of all of them, so that the weights are read once and a row's value serves
// every token that it reaches.  The tokens' angles are formed once per block.
constexpr int RUN = 8, RUN_WARPS = 8;

template <typename T>
__global__ void __launch_bounds__(RUN_WARPS * 32) pool_attn_prep_run_kernel(
    const T* __restrict__ proj, int ld, const float* __restrict__ inv_freq, const float* __restrict__ inv_freq_lo, int rot,
    const int* __restrict__ tile_tok0, const int* __restrict__ tile_rows, const int* __restrict__ cu_q, int n_seqs,
    const int* __restrict__ tok_slot, const int* __restrict__ tok_pos, T* __restrict__ q_out, T* __restrict__ k_pages,
    T* __restrict__ v_pages, const int* __restrict__ page_table, int max_pages, int page_size, int H, int G, float eps,
    const float* __restrict__ conv_w, int taps, const T* __restrict__ ring) {
  extern __shared__ float mem[];                  // [RUN_WARPS][RUN][D] convolved vectors, then [RUN][rot / 2][2] sines and cosines
  const int tok0 = tile_tok0[blockIdx.x] + (int)blockIdx.y * RUN, rows = min(RUN, tile_rows[blockIdx.x] - (int)blockIdx.y * RUN);
  if (rows <= 0) return;
  const int slot = tok_slot[tok0];
  if (slot < 0) return;
  int lo = 0, hi = n_seqs - 1;                    // the sequence: the largest b with cu_q[b] <= tok0
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= tok0) lo = mid; else hi = mid - 1;
  }
  const int t0 = cu_q[lo], n = cu_q[lo + 1] - t0, p0 = tok_pos[t0], i0 = tok0 - t0, pos0 = p0 + i0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = rot / 2;
  const int CH = H * D + G * (D + DV);
  float* s = mem + (size_t)warp * RUN * D;
  float* ang = mem + (size_t)RUN_WARPS * RUN * D;
  for (int i = threadIdx.x; i < RUN * half; i += RUN_WARPS * 32) {
    const int k = i / half, f = i % half;
    float sn, cs;
    sincos_split((float)(pos0 + k), inv_freq[f], inv_freq_lo != nullptr ? inv_freq_lo[f] : 0.f, &sn, &cs);
    ang[2 * i] = sn;
    ang[2 * i + 1] = cs;
  }
  __syncthreads();
  const int* pages = page_table + (size_t)slot * max_pages;
  for (int vec = warp; vec < H + 2 * G; vec += RUN_WARPS) {
    const int g = vec < H ? 0 : (vec - H) % G;
    if (vec >= H + G) {      // a value vector
      for (int c = lane; c < DV; c += 32) {
        float acc[RUN];
        conv_run<T, RUN>(acc, conv_w, proj, ld, ring, taps, CH, slot, t0, p0, i0, n, H * D + G * D + g * DV + c);
#pragma unroll
        for (int k = 0; k < RUN; ++k) {
          const int p = pos0 + k;
          if (k < rows) v_pages[(((size_t)pages[p / page_size] * G + g) * page_size + p % page_size) * DV + c] = from_f32<T>(acc[k]);
        }
      }
      continue;
    }
    const bool is_q = vec < H;
    const int src = is_q ? vec * D : H * D + g * D;
    __syncwarp();            // the vector before this one has been read
#pragma unroll 2
    for (int r = 0; r < DR; ++r) {
      const int c = lane + 32 * r;
      if (c < D) {
        float acc[RUN];
        conv_run<T, RUN>(acc, conv_w, proj, ld, ring, taps, CH, slot, t0, p0, i0, n, src + c);
#pragma unroll
        for (int k = 0; k < RUN; ++k) s[k * D + c] = acc[k];
      }
    }
    __syncwarp();
#pragma unroll 1
    for (int k = 0; k < rows; ++k) {
      float o[DR];
      float ss = 0.f;
#pragma unroll
      for (int r = 0; r < DR; ++r) {
        const int c = lane + 32 * r;
        float v = 0.f;
        if (c < D) {
          v = s[k * D + c];
          if (c < rot) {
            const float* a = ang + 2 * (k * half + (c < half ? c : c - half));
            v = c < half ? v * a[1] - s[k * D + c + half] * a[0] : v * a[1] + s[k * D + c - half] * a[0];
          }
        }
        o[r] = v;
        ss = fmaf(v, v, ss);
      }
      float rinv = 1.f;
      if (eps >= 0.f) rinv = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);     // eps < 0: no unit norm
      const int p = pos0 + k;
      T* dst = is_q ? q_out + ((size_t)(tok0 + k) * H + vec) * D
                    : k_pages + (((size_t)pages[p / page_size] * G + g) * page_size + p % page_size) * D;
#pragma unroll
      for (int r = 0; r < DR; ++r) {
        const int c = lane + 32 * r;
        if (c < D) dst[c] = from_f32<T>(o[r] * rinv);
      }
    }
  }
}

template <typename T>
int prep_run_launch(const void* proj, int ld, const float* inv_freq, const float* inv_freq_lo, int rot, const int* tile_tok0,
                    const int* tile_rows, int n_tiles, int tile_size, const int* cu_q, int n_seqs, const int* tok_slot, const int* tok_pos,
                    void* q_out, void* k_pages, void* v_pages, const int* page_table, int max_pages, int page_size, int H, int G, float eps,
                    const float* conv_w, int taps, const void* ring, cudaStream_t st) {
  const size_t smem = sizeof(float) * ((size_t)RUN_WARPS * RUN * D + (size_t)RUN * rot);
  if (smem > 200 * 1024) return DRYFT_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(pool_attn_prep_run_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  dim3 grid(n_tiles, (tile_size + RUN - 1) / RUN);
  pool_attn_prep_run_kernel<T><<<grid, RUN_WARPS * 32, smem, st>>>((const T*)proj, ld, inv_freq, inv_freq_lo, rot, tile_tok0, tile_rows, cu_q, n_seqs,
                                                                  tok_slot, tok_pos, (T*)q_out, (T*)k_pages, (T*)v_pages, page_table, max_pages,
                                                                  page_size, H, G, eps, conv_w, taps, (const T*)ring);
  return launch_status();
}

// One block per token.  q_w [H * D] / k_w [G * D]: the weights of a norm over the whole projection (nullptr: no such norm).
template <typename T>
__global__ void __launch_bounds__(PREP_TOK_WARPS * 32) pool_attn_prep_tok_kernel(
    const T* __restrict__ proj, int ld, const float* __restrict__ q_w, const float* __restrict__ k_w, float norm_eps,
    const float* __restrict__ inv_freq, const float* __restrict__ inv_freq_lo, int rot, int interleaved, const int* __restrict__ tok_slot,
    const int* __restrict__ tok_pos, T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages,
    const int* __restrict__ page_table, int max_pages, int page_size, int H, int G, float eps, int write_kv) {
  __shared__ float sm[PREP_TOK_WARPS][D];
  __shared__ float scratch[33];
  const int t = blockIdx.x;
  const int slot = tok_slot[t];
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = tok_pos[t];
  const T* row = proj + (size_t)t * ld;
  float rq = 1.f, rk = 1.f;
  if (q_w != nullptr) {
    float a = 0.f;
    for (int c = threadIdx.x; c < H * D; c += PREP_TOK_WARPS * 32) { const float v = to_f32<T>(row[c]); a = fmaf(v, v, a); }
    rq = 1.f / sqrtf(block_sum(a, scratch) / (float)(H * D) + norm_eps);
  }
  if (k_w != nullptr && write_kv) {
    float a = 0.f;
    for (int c = threadIdx.x; c < G * D; c += PREP_TOK_WARPS * 32) { const float v = to_f32<T>(row[(size_t)H * D + c]); a = fmaf(v, v, a); }
    rk = 1.f / sqrtf(block_sum(a, scratch) / (float)(G * D) + norm_eps);
  }
  size_t cache_row0 = 0;
  if (write_kv) cache_row0 = (size_t)page_table[(size_t)slot * max_pages + pos / page_size];
  const int per_tok = H + (write_kv ? 2 * G : 0);
  const int half = rot / 2;
  const float fpos = (float)pos;
  float* s = sm[warp];
  for (int vec = warp; vec < per_tok; vec += PREP_TOK_WARPS) {
    if (vec >= H + G) {     // a value vector: into the cache as it is
      const int g = vec - H - G;
      const size_t cr = (cache_row0 * G + g) * page_size + pos % page_size;
      const T* src = row + (size_t)H * D + (size_t)G * D + (size_t)g * DV;
      for (int c = lane; c < DV; c += 32) v_pages[cr * DV + c] = src[c];
      continue;
    }
    const bool is_q = vec < H;
    const int hd = is_q ? vec : vec - H;
    const T* src = row + (is_q ? (size_t)hd * D : (size_t)H * D + (size_t)hd * D);
    const float* w = is_q ? q_w : k_w;
    const float r = is_q ? rq : rk;
    __syncwarp();
    for (int c = lane; c < D; c += 32) s[c] = w != nullptr ? to_f32<T>(src[c]) * r * w[hd * D + c] : to_f32<T>(src[c]);
    __syncwarp();
    float o[DR];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < DR; ++k) {
      const int c = lane + 32 * k;
      float v = 0.f;
      if (c < D) {
        if (c < rot) {
          // the entry this one turns with, the pair's frequency, and which of the two it is
          const int i = interleaved ? (c >> 1) : (c < half ? c : c - half);
          const bool first = interleaved ? !(c & 1) : c < half;
          const int other = interleaved ? (c ^ 1) : (first ? c + half : c - half);
          float sn, cs;
          sincos_split(fpos, inv_freq[i], inv_freq_lo != nullptr ? inv_freq_lo[i] : 0.f, &sn, &cs);
          v = first ? s[c] * cs - s[other] * sn : s[c] * cs + s[other] * sn;
        } else {
          v = s[c];
        }
      }
      o[k] = v;
      ss = fmaf(v, v, ss);
    }
    float rinv = 1.f;
    if (eps >= 0.f) rinv = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);    // eps < 0: no unit norm
    T* dst = is_q ? q_out + ((size_t)t * H + hd) * D : k_pages + ((cache_row0 * G + hd) * page_size + pos % page_size) * D;
#pragma unroll
    for (int k = 0; k < DR; ++k) {
      const int c = lane + 32 * k;
      if (c < D) dst[c] = from_f32<T>(o[k] * rinv);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(BLOCKS_THREADS) pool_attn_blocks_kernel(
    const T* __restrict__ k_pages, const T* __restrict__ v_pages, const int* __restrict__ page_table, int max_pages, int page_size,
    T* __restrict__ pk_pages, T* __restrict__ pv_pages, const int* __restrict__ pool_table, int pool_max_pages,
    const int* __restrict__ tok_slot, const int* __restrict__ tok_pos, int G, int P) {
  const int t = blockIdx.x, g = blockIdx.y;
  const int slot = tok_slot[t];
  if (slot < 0) return;
  const int pos = tok_pos[t];
  if (pos % P != P - 1) return;
  const int b = pos / P, p0 = pos - (P - 1);
  const int ppage = pool_table[(size_t)slot * pool_max_pages + b / page_size];
  const size_t prow = ((size_t)ppage * G + g) * page_size + b % page_size;
  const float inv = 1.f / (float)P;
  for (int c = threadIdx.x; c < D + DV; c += blockDim.x) {
    float acc = 0.f;
#pragma unroll 8
    for (int j = 0; j < P; ++j) {   // rows in order: the sum does not depend on how the loads are scheduled
      const int pj = p0 + j;
      const int page = page_table[(size_t)slot * max_pages + pj / page_size];
      const size_t r = ((size_t)page * G + g) * page_size + pj % page_size;
      acc += c < D ? to_f32<T>(k_pages[r * D + c]) : to_f32<T>(v_pages[r * DV + (c - D)]);
    }
    if (c < D) pk_pages[prow * D + c] = from_f32<T>(acc * inv);
    else pv_pages[prow * DV + (c - D)] = from_f32<T>(acc * inv);
  }
}

template <typename T> __device__ __forceinline__ void dot_row(const T* __restrict__ kr, const float (*qs)[D], float* dots) {
  constexpr int V = 16 / sizeof(T);
  if (D % V == 0) {
#pragma unroll 2
    for (int c = 0; c < D; c += V) {
      const uint4 kv = *reinterpret_cast<const uint4*>(kr + c);
      const T* ke = reinterpret_cast<const T*>(&kv);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float kf = to_f32<T>(ke[e]);
#pragma unroll
        for (int h = 0; h < REP; ++h) dots[h] = fmaf(kf, qs[h][c + e], dots[h]);
      }
    }
  } else {
    for (int c = 0; c < D; ++c) {
      const float kf = to_f32<T>(kr[c]);
#pragma unroll
      for (int h = 0; h < REP; ++h) dots[h] = fmaf(kf, qs[h][c], dots[h]);
    }
  }
}

// the factor of output value c of a token's head: the sigmoid of its logit in [n, H * DV] (no gate: one)
template <typename T> __device__ __forceinline__ float gate_at(const T* __restrict__ gate, int gate_ld, int t, int head, int c) {
  return gate == nullptr ? 1.f : 1.f / (1.f + expf(-to_f32<T>(gate[(size_t)t * gate_ld + (size_t)head * DV + c])));
}

// How a score is changed before the softmax: squashed to cap * tanh(s / cap) (cap > 0), then r1_h * ln(1 + r2_h * distance) taken off
// (r1 given; distances in tokens, so not together with pooled rows).  32-bit path: CUDA's tanhf and log1pf; bfloat16 path: the
// same functions from one exponential and one logarithm, absolute errors below 1e-6 of the cap or of r1.
struct ScoreMods { float cap; const float* r1; const float* r2; };
template <typename T> __device__ __forceinline__ float mod_score(float s, float cap, float r1, float r2, float dist) {
  if (sizeof(T) == 4) {
    if (cap > 0.f) s = cap * tanhf(s / cap);
    return s - r1 * log1pf(r2 * dist);
  }
  if (cap > 0.f) s = cap - __fdividef(2.f * cap, 1.f + __expf(2.f * s / cap));      // cap * (1 - 2 / (1 + e^(2 s / cap)))
  return s - r1 * __logf(fmaf(r2, dist, 1.f));
}

template <typename T, bool MODS>
__global__ void __launch_bounds__(ROWS_WARPS * 32) pool_attn_rows_kernel(
    const T* __restrict__ q, const T* __restrict__ k_pages, const T* __restrict__ v_pages, const int* __restrict__ page_table,
    int max_pages, int page_size, const T* __restrict__ pk_pages, const T* __restrict__ pv_pages, const int* __restrict__ pool_table,
    int pool_max_pages, const float* __restrict__ sink, const int* __restrict__ tok_slot, const int* __restrict__ tok_pos,
    T* __restrict__ out, float* __restrict__ part_o, float* __restrict__ part_ml, int G, int n_splits, float scale, int size, int P, int keep, const T* __restrict__ gate,
    int gate_ld, ScoreMods mods) {
  __shared__ float qs[REP][D];
  __shared__ float wo[ROWS_WARPS][REP][DV];
  __shared__ float wml[ROWS_WARPS][REP][2];
  const int t = blockIdx.x, g = blockIdx.y, sp = blockIdx.z;
  const int slot = tok_slot[t];
  if (slot < 0) return;
  const int H = G * REP;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int i = tok_pos[t];
  const int lo = max(0, i - size + 1);
  const int nb = (P > 0 && i - size + 1 >= P) ? (i - size + 1) / P : 0;
  const int nk = min(keep, lo);                   // kept tokens that the window has passed
  const int nkeys = nb + nk + (i - lo + 1);
  int chunk = (nkeys + n_splits - 1) / n_splits;
  chunk = (chunk + 31) / 32 * 32;
  const int u0 = sp * chunk, u1 = min(nkeys, u0 + chunk);
  for (int c = threadIdx.x; c < REP * D; c += blockDim.x) qs[c / D][c % D] = to_f32<T>(q[((size_t)t * H + (size_t)g * REP) * D + c]);
  __syncthreads();

  float m[REP], l[REP], o[REP][DVR];
  float mr1[MODS ? REP : 1], mr2[MODS ? REP : 1];
#pragma unroll
  for (int h = 0; h < REP; ++h) {
    if (MODS) {
      mr1[h] = mods.r1 != nullptr ? mods.r1[g * REP + h] : 0.f;
      mr2[h] = mods.r1 != nullptr ? mods.r2[g * REP + h] : 0.f;
    }
    m[h] = -INFINITY;
    l[h] = 0.f;
#pragma unroll
    for (int r = 0; r < DVR; ++r) o[h][r] = 0.f;
  }
  for (int tile = u0 + warp * 32; tile < u1; tile += ROWS_WARPS * 32) {
    const int u = tile + lane;
    const bool valid = u < u1;
    const T* kr = k_pages;
    const T* vr = v_pages;
    float dist = 0.f;
    if (valid) {
      if (u < nb) {
        const int page = pool_table[(size_t)slot * pool_max_pages + u / page_size];
        const size_t r = ((size_t)page * G + g) * page_size + u % page_size;
        kr = pk_pages + r * D;
        vr = pv_pages + r * DV;
      } else {
        const int j = u - nb < nk ? u - nb : lo + (u - nb - nk);
        dist = (float)(i - j);
        const int page = page_table[(size_t)slot * max_pages + j / page_size];
        const size_t r = ((size_t)page * G + g) * page_size + j % page_size;
        kr = k_pages + r * D;
        vr = v_pages + r * DV;
      }
    }
    float dots[REP];
#pragma unroll
    for (int h = 0; h < REP; ++h) dots[h] = 0.f;
    if (valid) dot_row<T>(kr, qs, dots);
    float pr[REP];
#pragma unroll
    for (int h = 0; h < REP; ++h) {
      float sc = valid ? dots[h] * scale : -INFINITY;
      if (MODS && valid) sc = mod_score<T>(sc, mods.cap, mr1[h], mr2[h], dist);
      const float mn = fmaxf(m[h], warp_max(sc));          // finite: the tile holds at least one key
      const float corr = expf(m[h] - mn);                  // exp(-inf) = 0 for the first tile
      const float pv = valid ? expf(sc - mn) : 0.f;
      l[h] = fmaf(l[h], corr, warp_sum(pv));
      m[h] = mn;
      pr[h] = pv;
#pragma unroll
      for (int r = 0; r < DVR; ++r) o[h][r] *= corr;
    }
    const int cnt = min(32, u1 - tile);
    const unsigned long long vaddr = reinterpret_cast<unsigned long long>(vr);
    for (int jj = 0; jj < cnt; ++jj) {
      const T* vj = reinterpret_cast<const T*>(__shfl_sync(0xffffffffu, vaddr, jj));
      float vv[DVR];
#pragma unroll
      for (int r = 0; r < DVR; ++r) {
        const int c = lane + 32 * r;
        vv[r] = c < DV ? to_f32<T>(vj[c]) : 0.f;
      }
#pragma unroll
      for (int h = 0; h < REP; ++h) {
        const float pj = __shfl_sync(0xffffffffu, pr[h], jj);
#pragma unroll
        for (int r = 0; r < DVR; ++r) o[h][r] = fmaf(pj, vv[r], o[h][r]);
      }
    }
  }
  // the warps' partial results meet in shared memory
#pragma unroll
  for (int h = 0; h < REP; ++h) {
    if (lane == 0) { wml[warp][h][0] = m[h]; wml[warp][h][1] = l[h]; }
#pragma unroll
    for (int r = 0; r < DVR; ++r) {
      const int c = lane + 32 * r;
      if (c < DV) wo[warp][h][c] = o[h][r];
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < REP * DV; e += blockDim.x) {
    const int h = e / DV, c = e % DV;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < ROWS_WARPS; ++w) M = fmaxf(M, wml[w][h][0]);
    float L = 0.f, O = 0.f;
#pragma unroll
    for (int w = 0; w < ROWS_WARPS; ++w) {
      const float mw = wml[w][h][0];
      const float f = mw == -INFINITY ? 0.f : expf(mw - M);
      L = fmaf(wml[w][h][1], f, L);
      O = fmaf(wo[w][h][c], f, O);
    }
    const int head = g * REP + h;
    if (n_splits == 1) {
      const float sk = sink != nullptr ? sink[head] : -INFINITY;
      const float Mx = fmaxf(M, sk);
      const float f = M == -INFINITY ? 0.f : expf(M - Mx);
      const float den = L * f + (sk == -INFINITY ? 0.f : expf(sk - Mx));
      out[((size_t)t * H + head) * DV + c] = from_f32<T>(den > 0.f ? O * f / den * gate_at<T>(gate, gate_ld, t, head, c) : 0.f);
    } else {
      const size_t pi = ((size_t)t * H + head) * n_splits + sp;
      part_o[pi * DV + c] = O;
      if (c == 0) { part_ml[pi * 2] = M; part_ml[pi * 2 + 1] = L; }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) pool_attn_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                                const float* __restrict__ sink, const int* __restrict__ tok_slot,
                                                                T* __restrict__ out, int H, int n_splits, const T* __restrict__ gate, int gate_ld) {
  const int t = blockIdx.x, head = blockIdx.y;
  if (tok_slot[t] < 0) return;
  const size_t base = ((size_t)t * H + head) * n_splits;
  const float sk = sink != nullptr ? sink[head] : -INFINITY;
  float Mx = sk;
  for (int s = 0; s < n_splits; ++s) Mx = fmaxf(Mx, part_ml[(base + s) * 2]);
  float den = sk == -INFINITY ? 0.f : expf(sk - Mx);
  for (int s = 0; s < n_splits; ++s) {
    const float ms = part_ml[(base + s) * 2];
    if (ms != -INFINITY) den = fmaf(part_ml[(base + s) * 2 + 1], expf(ms - Mx), den);
  }
  for (int c = threadIdx.x; c < DV; c += blockDim.x) {
    float O = 0.f;
    for (int s = 0; s < n_splits; ++s) {
      const float ms = part_ml[(base + s) * 2];
      if (ms != -INFINITY) O = fmaf(part_o[(base + s) * DV + c], expf(ms - Mx), O);
    }
    out[((size_t)t * H + head) * DV + c] = from_f32<T>(den > 0.f ? O / den * gate_at<T>(gate, gate_ld, t, head, c) : 0.f);
  }
}

template <typename T>
int prep_launch(const void* proj, int ld, const float* qb, const float* kb, const float* vb, const float* inv_freq,
                const float* inv_freq_lo, int rot, const int* tok_slot, const int* tok_pos, void* q_out, void* k_pages, void* v_pages, const int* page_table,
                int max_pages, int page_size, int n, int H, int G, float eps, int write_kv, const float* conv_w, int taps, void* ring,
                int store_ring, float v_eps, float qt_coef, int qt_every, cudaStream_t st) {
  // many tokens: a warp takes several vectors of one token, which share its angles and the rows its convolution reads
  const int per_tok = H + (write_kv ? 2 * G : 0), per_warp = n >= 512 ? 8 : n >= 128 ? 4 : 1;
  const long long items = (long long)n * ((per_tok + per_warp - 1) / per_warp);
  const long long blocks = (items + PREP_WARPS - 1) / PREP_WARPS;
  if (blocks > 0x7fffffffLL) return DRYFT_ERR_UNSUPPORTED;
  pool_attn_prep_kernel<T><<<(unsigned)blocks, PREP_WARPS * 32, 0, st>>>(
      (const T*)proj, ld, qb, kb, vb, inv_freq, inv_freq_lo, rot, tok_slot, tok_pos, (T*)q_out, (T*)k_pages, (T*)v_pages, page_table, max_pages,
      page_size, n, H, G, eps, write_kv, conv_w, taps, (T*)ring, store_ring, per_warp, v_eps, qt_coef, qt_every);
  return launch_status();
}

template <typename T>
int rows_launch(const void* q, const void* k_pages, const void* v_pages, const int* page_table, int max_pages, int page_size,
                const void* pk, const void* pv, const int* pool_table, int pool_max_pages, const float* sink, const int* tok_slot,
                const int* tok_pos, void* out, float* part_o, float* part_ml, int n, int G, int n_splits, float scale, int size, int P,
                int keep, const void* gate, int gate_ld, ScoreMods mods, cudaStream_t st) {
  dim3 grid(n, G, n_splits);
  auto kernel = mods.cap > 0.f || mods.r1 != nullptr ? pool_attn_rows_kernel<T, true> : pool_attn_rows_kernel<T, false>;
  kernel<<<grid, ROWS_WARPS * 32, 0, st>>>((const T*)q, (const T*)k_pages, (const T*)v_pages, page_table, max_pages, page_size, (const T*)pk,
                                           (const T*)pv, pool_table, pool_max_pages, sink, tok_slot, tok_pos, (T*)out, part_o, part_ml, G,
                                           n_splits, scale, size, P, keep, (const T*)gate, gate_ld, mods);
  int rc = launch_status();
  if (rc || n_splits == 1) return rc;
  dim3 cgrid(n, G * REP);
  pool_attn_combine_kernel<T><<<cgrid, 128, 0, st>>>(part_o, part_ml, sink, tok_slot, (T*)out, G * REP, n_splits, (const T*)gate, gate_ld);
  return launch_status();
}
}  // namespace

DRYFT_API int dryft_pool_attn_qk_dim() { return D; }
DRYFT_API int dryft_pool_attn_v_dim() { return DV; }
DRYFT_API int dryft_pool_attn_group() { return REP; }

DRYFT_API int dryft_pool_attn_prep(int is_bf16, const void* proj, int ld, const float* qb, const float* kb, const float* vb,
                                   const float* inv_freq, const float* inv_freq_lo, int rot, const int* tok_slot, const int* tok_pos,
                                   void* q_out, void* k_pages, void* v_pages, const int* page_table, int max_pages, int page_size, int n, int H, int G, float eps,
                                   int write_kv, const float* conv_w, int taps, void* ring, int store_ring, float v_eps, float qt_coef,
                                   int qt_every, cudaStream_t st) {
  if (n <= 0) return 0;
  if (H != G * REP || rot < 0 || rot % 2 || rot > D || (rot > 0 && inv_freq == nullptr) || (write_kv && page_size < 1))
    return DRYFT_ERR_UNSUPPORTED;
  if (conv_w != nullptr && (taps < 1 || taps > DRYFT_CONV_MAX_TAPS || !write_kv || ((taps > 1 || store_ring) && ring == nullptr)))
    return DRYFT_ERR_UNSUPPORTED;
  return is_bf16 ? prep_launch<__nv_bfloat16>(proj, ld, qb, kb, vb, inv_freq, inv_freq_lo, rot, tok_slot, tok_pos, q_out, k_pages, v_pages, page_table,
                                              max_pages, page_size, n, H, G, eps, write_kv, conv_w, taps, ring, store_ring, v_eps, qt_coef, qt_every, st)
                 : prep_launch<float>(proj, ld, qb, kb, vb, inv_freq, inv_freq_lo, rot, tok_slot, tok_pos, q_out, k_pages, v_pages, page_table,
                                      max_pages, page_size, n, H, G, eps, write_kv, conv_w, taps, ring, store_ring, v_eps, qt_coef, qt_every, st);
}

DRYFT_API int dryft_pool_attn_prep_run(int is_bf16, const void* proj, int ld, const float* inv_freq, const float* inv_freq_lo, int rot,
                                       const int* tile_tok0, const int* tile_rows, int n_tiles, int tile_size, const int* cu_q, int n_seqs,
                                       const int* tok_slot, const int* tok_pos, void* q_out, void* k_pages, void* v_pages,
                                       const int* page_table, int max_pages, int page_size, int H, int G, float eps, const float* conv_w,
                                       int taps, const void* ring, cudaStream_t st) {
  if (n_tiles <= 0) return 0;
  if (H != G * REP || rot < 0 || rot % 2 || rot > D || (rot > 0 && inv_freq == nullptr) || page_size < 1 || tile_size < 1 || taps < 1 ||
      taps > DRYFT_CONV_MAX_TAPS || (taps > 1 && ring == nullptr))
    return DRYFT_ERR_UNSUPPORTED;
  return is_bf16 ? prep_run_launch<__nv_bfloat16>(proj, ld, inv_freq, inv_freq_lo, rot, tile_tok0, tile_rows, n_tiles, tile_size, cu_q, n_seqs,
                                                  tok_slot, tok_pos, q_out, k_pages, v_pages, page_table, max_pages, page_size, H, G, eps, conv_w,
                                                  taps, ring, st)
                 : prep_run_launch<float>(proj, ld, inv_freq, inv_freq_lo, rot, tile_tok0, tile_rows, n_tiles, tile_size, cu_q, n_seqs, tok_slot,
                                          tok_pos, q_out, k_pages, v_pages, page_table, max_pages, page_size, H, G, eps, conv_w, taps, ring, st);
}

DRYFT_API int dryft_pool_attn_prep_tok(int is_bf16, const void* proj, int ld, const float* q_w, const float* k_w, float norm_eps,
                                       const float* inv_freq, const float* inv_freq_lo, int rot, int interleaved, const int* tok_slot,
                                       const int* tok_pos, void* q_out, void* k_pages, void* v_pages, const int* page_table, int max_pages,
                                       int page_size, int n, int H, int G, float eps, int write_kv, cudaStream_t st) {
  if (n <= 0) return 0;
  if (H != G * REP || rot < 0 || rot % 2 || rot > D || (rot > 0 && inv_freq == nullptr) || (write_kv && page_size < 1))
    return DRYFT_ERR_UNSUPPORTED;
  typedef __nv_bfloat16 bf;
  if (is_bf16)
    pool_attn_prep_tok_kernel<bf><<<n, PREP_TOK_WARPS * 32, 0, st>>>((const bf*)proj, ld, q_w, k_w, norm_eps, inv_freq, inv_freq_lo, rot, interleaved,
                                                                 tok_slot, tok_pos, (bf*)q_out, (bf*)k_pages, (bf*)v_pages, page_table, max_pages,
                                                                 page_size, H, G, eps, write_kv);
  else
    pool_attn_prep_tok_kernel<float><<<n, PREP_TOK_WARPS * 32, 0, st>>>((const float*)proj, ld, q_w, k_w, norm_eps, inv_freq, inv_freq_lo, rot,
                                                                    interleaved, tok_slot, tok_pos, (float*)q_out, (float*)k_pages,
                                                                    (float*)v_pages, page_table, max_pages, page_size, H, G, eps, write_kv);
  return launch_status();
}

DRYFT_API int dryft_pool_attn_blocks(int is_bf16, const void* k_pages, const void* v_pages, const int* page_table, int max_pages,
                                     int page_size, void* pk, void* pv, const int* pool_table, int pool_max_pages, const int* tok_slot,
                                     const int* tok_pos, int n, int G, int P, cudaStream_t st) {
  if (n <= 0 || P <= 0) return 0;
  if (G < 1 || G > 65535 || page_size < 1) return DRYFT_ERR_UNSUPPORTED;
  dim3 grid(n, G);
  if (is_bf16)
    pool_attn_blocks_kernel<__nv_bfloat16><<<grid, BLOCKS_THREADS, 0, st>>>((const __nv_bfloat16*)k_pages, (const __nv_bfloat16*)v_pages, page_table,
                                                                 max_pages, page_size, (__nv_bfloat16*)pk, (__nv_bfloat16*)pv, pool_table,
                                                                 pool_max_pages, tok_slot, tok_pos, G, P);
  else
    pool_attn_blocks_kernel<float><<<grid, BLOCKS_THREADS, 0, st>>>((const float*)k_pages, (const float*)v_pages, page_table, max_pages, page_size,
                                                         (float*)pk, (float*)pv, pool_table, pool_max_pages, tok_slot, tok_pos, G, P);
  return launch_status();
}

DRYFT_API int dryft_pool_attn_rows(int is_bf16, const void* q, const void* k_pages, const void* v_pages, const int* page_table,
                                   int max_pages, int page_size, const void* pk, const void* pv, const int* pool_table,
                                   int pool_max_pages, const float* sink, const int* tok_slot, const int* tok_pos, void* out,
                                   float* part_o, float* part_ml, int n, int G, int n_splits, float scale, int size, int P, int keep,
                                   const void* gate, int gate_ld, float softcap, const float* r1, const float* r2, cudaStream_t st) {
  if (n <= 0) return 0;
  if (!(softcap >= 0.f) || (r1 != nullptr) != (r2 != nullptr) || ((softcap > 0.f || r1 != nullptr) && P > 0)) return DRYFT_ERR_UNSUPPORTED;
  const ScoreMods mods{softcap, r1, r2};
  if (G < 1 || G > 65535 || n_splits < 1 || n_splits > 65535 || size < 1 || keep < 0 || page_size < 1 || (P > 0 && pk == nullptr) ||
      (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)))
    return DRYFT_ERR_UNSUPPORTED;
  return is_bf16 ? rows_launch<__nv_bfloat16>(q, k_pages, v_pages, page_table, max_pages, page_size, pk, pv, pool_table, pool_max_pages,
                                              sink, tok_slot, tok_pos, out, part_o, part_ml, n, G, n_splits, scale, size, P, keep, gate, gate_ld, mods, st)
                 : rows_launch<float>(q, k_pages, v_pages, page_table, max_pages, page_size, pk, pv, pool_table, pool_max_pages, sink,
                                      tok_slot, tok_pos, out, part_o, part_ml, n, G, n_splits, scale, size, P, keep, gate, gate_ld, mods, st);
}
