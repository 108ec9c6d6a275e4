// The memory of a short convolution after a step of many tokens (shortconv.cuh): the projected values of each sequence's last
// min(tokens of the step, taps - 1) tokens go to row (position % taps) of its slot's ring.  A thread a (sequence, channel).
// Sequences with slot -1 (padding) are skipped.  No block waits on another block.
#include "shortconv.cuh"

namespace {
constexpr int THREADS = 128;

template <typename T>
__global__ void __launch_bounds__(THREADS) conv_ring_store_kernel(const T* __restrict__ x, int ld, const int* __restrict__ cu_q,
                                                                 const int* __restrict__ seq_slot, const int* __restrict__ tok_pos,
                                                                 T* __restrict__ ring, int taps, int CH) {
  const int b = blockIdx.x;
  const int slot = seq_slot[b];
  const int t1 = cu_q[b + 1], n = t1 - cu_q[b];
  if (slot < 0 || n <= 0) return;
  const int c = blockIdx.y * THREADS + threadIdx.x;
  if (c >= CH) return;
  const int last = tok_pos[t1 - 1];
  for (int k = 0; k < taps - 1 && k < n; ++k)
    ring[((size_t)slot * taps + (last - k) % taps) * CH + c] = x[(size_t)(t1 - 1 - k) * ld + c];
}
}  // namespace

DRYFT_API int dryft_conv_ring_store(int is_bf16, const void* x, int ld, const int* cu_q, const int* seq_slot, const int* tok_pos,
                                    void* ring, int taps, int CH, int n_seqs, cudaStream_t st) {
  if (n_seqs <= 0) return 0;
  if (taps < 2 || taps > DRYFT_CONV_MAX_TAPS || CH < 1 || (CH + THREADS - 1) / THREADS > 65535) return DRYFT_ERR_UNSUPPORTED;
  dim3 grid(n_seqs, (CH + THREADS - 1) / THREADS);
  typedef __nv_bfloat16 bf;
  if (is_bf16)
    conv_ring_store_kernel<bf><<<grid, THREADS, 0, st>>>((const bf*)x, ld, cu_q, seq_slot, tok_pos, (bf*)ring, taps, CH);
  else
    conv_ring_store_kernel<float><<<grid, THREADS, 0, st>>>((const float*)x, ld, cu_q, seq_slot, tok_pos, (float*)ring, taps, CH);
  return launch_status();
}
