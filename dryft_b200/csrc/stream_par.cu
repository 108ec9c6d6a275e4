// Kernels around a 32-bit residual stream whose layers add several results at once (a mixer and a feed-forward that read
// the same normed input, two mixers side by side), and around a stretch of layers that is entered through a product over
// the stream joined with an earlier copy of it.  T is the activation type; every sum and norm is 32-bit.
//
//   stream_sum    x32[n] += s0 * y0[n] + s1 * y1[n] + s2 * y2[n] + sr * sum_k yr[n * top + k] + vec        (every term optional)
//                 and, when a norm weight is given, h[n] = T( x32[n] / sqrt(mean(x32[n]^2) + eps) * w ): the sum of a layer
//                 and the norm of the next in one launch.  `src` (optional, 32-bit) replaces x32 as the sum's start
//                 (x32[n] = src[n] + ...).
//   stream_sum_ln the same sum of up to three terms, then up to two LAYER norms of the new row in the same launch:
//                 h_i[n] = T( (x32[n] - mean) / sqrt(mean((x32[n] - mean)^2) + eps) * w_i + b_i ); the row stays in shared memory
//                 (4 * width bytes), the mean is formed before the deviations are squared.  `rows` (optional): output row r
//                 reads stream row rows[r] (no terms then: nothing is written to the stream).
//   stream_norm_join  y = s0 * y0[n] + s1 * y1[n] + s2 * y2[n] + sum_k wts[n, k] * yr[n * top + k] ;  x32[n] += y / sqrt(mean(y^2) + eps) * factor :
//                 the norm on a sublayer's OUTPUT; and, when a norm weight is given, h[n] = T( norm of the new row ), the norm in
//                 front of the sublayer that comes next, in the same launch.  The row stays in registers (widths up to 4,096 in steps of four, everything
//                 a thread needs requested before the first sum) or in shared memory (4 * width bytes).
//   pack_pair     out[n] = T([a32[n] | b32[n]]): two 32-bit rows side by side as one operand row of a product
//   softcap       z <- cap * tanh(z / cap) over 32-bit logits, in place
//
// One block per row; widths are runtime arguments of any size.  Rows whose slot is -1 (padding) are computed like any
// other: they read and write only their own row.  No block waits on another.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(THREADS) stream_sum_kernel(
    float* __restrict__ x32, const float* __restrict__ src, const T* __restrict__ y0, float s0, const T* __restrict__ y1, float s1,
    const T* __restrict__ y2, float s2, const T* __restrict__ yr, int top, float sr, const float* __restrict__ vec,
    const float* __restrict__ norm_w, float eps, T* __restrict__ h, int width) {
  __shared__ float scratch[33];
  const size_t n = blockIdx.x;
  float* x = x32 + n * width;
  const float* xs = src != nullptr ? src + n * width : x;
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += THREADS) {
    float v = xs[c];
    float add = 0.f;
    if (y0 != nullptr) add = fmaf(s0, to_f32<T>(y0[n * width + c]), add);
    if (y1 != nullptr) add = fmaf(s1, to_f32<T>(y1[n * width + c]), add);
    if (y2 != nullptr) add = fmaf(s2, to_f32<T>(y2[n * width + c]), add);
    if (yr != nullptr) {
      float r = 0.f;
      for (int k = 0; k < top; ++k) r += to_f32<T>(yr[(n * top + k) * width + c]);   // in the order of the choices
      add = fmaf(sr, r, add);
    }
    if (vec != nullptr) add += vec[c];
    v += add;
    x[c] = v;
    ss = fmaf(v, v, ss);
  }
  if (norm_w == nullptr) return;
  ss = block_sum(ss, scratch);
  const float rinv = 1.f / sqrtf(ss / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += THREADS) h[n * width + c] = from_f32<T>(x[c] * rinv * norm_w[c]);   // the thread's own writes
}

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

// VEC 4 (widths that are a multiple of four) or 1
template <typename T, int VEC>
__global__ void __launch_bounds__(THREADS) stream_sum_ln_kernel(
    float* __restrict__ x32, const int* __restrict__ rows, const T* __restrict__ y0, float s0, const T* __restrict__ y1, float s1,
    const T* __restrict__ y2, float s2, const float* __restrict__ w0, const float* __restrict__ b0, T* __restrict__ h0,
    const float* __restrict__ w1, const float* __restrict__ b1, T* __restrict__ h1, float eps, int width) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  const size_t n = blockIdx.x;
  float* x = x32 + (rows != nullptr ? (size_t)rows[n] : n) * width;
  const bool adds = y0 != nullptr || y1 != nullptr || y2 != nullptr;
  float sum = 0.f;
  if (VEC == 4) {
    for (int c = threadIdx.x * 4; c < width; c += THREADS * 4) {
      float4 v = *reinterpret_cast<const float4*>(x + c);
      auto term = [&](const T* y, float s) {
        const float4 t = load4<T>(y + n * width + c);
        v.x = fmaf(s, t.x, v.x); v.y = fmaf(s, t.y, v.y); v.z = fmaf(s, t.z, v.z); v.w = fmaf(s, t.w, v.w);
      };
      if (y0 != nullptr) term(y0, s0);
      if (y1 != nullptr) term(y1, s1);
      if (y2 != nullptr) term(y2, s2);
      if (adds) *reinterpret_cast<float4*>(x + c) = v;
      *reinterpret_cast<float4*>(row + c) = v;
      sum += (v.x + v.y) + (v.z + v.w);
    }
  } else {
    for (int c = threadIdx.x; c < width; c += THREADS) {
      float v = x[c];
      if (y0 != nullptr) v = fmaf(s0, to_f32<T>(y0[n * width + c]), v);
      if (y1 != nullptr) v = fmaf(s1, to_f32<T>(y1[n * width + c]), v);
      if (y2 != nullptr) v = fmaf(s2, to_f32<T>(y2[n * width + c]), v);
      if (adds) x[c] = v;
      row[c] = v;
      sum += v;
    }
  }
  if (h0 == nullptr && h1 == nullptr) return;
  const float mean = block_sum(sum, scratch) / (float)width;
  float ss = 0.f;      // every thread reads the entries it wrote itself
  if (VEC == 4) {
    for (int c = threadIdx.x * 4; c < width; c += THREADS * 4) {
      const float4 v = *reinterpret_cast<const float4*>(row + c);
      const float a = v.x - mean, b = v.y - mean, d = v.z - mean, e = v.w - mean;
      ss = fmaf(a, a, fmaf(b, b, fmaf(d, d, fmaf(e, e, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < width; c += THREADS) { const float d = row[c] - mean; ss = fmaf(d, d, ss); }
  }
  const float rinv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  if (VEC == 4) {
    for (int c = threadIdx.x * 4; c < width; c += THREADS * 4) {
      float4 v = *reinterpret_cast<const float4*>(row + c);
      v.x = (v.x - mean) * rinv; v.y = (v.y - mean) * rinv; v.z = (v.z - mean) * rinv; v.w = (v.w - mean) * rinv;
      auto out = [&](const float* w, const float* b, T* h) {
        const float4 ww = *reinterpret_cast<const float4*>(w + c), bb = *reinterpret_cast<const float4*>(b + c);
        store4<T>(h + n * width + c, make_float4(fmaf(v.x, ww.x, bb.x), fmaf(v.y, ww.y, bb.y), fmaf(v.z, ww.z, bb.z), fmaf(v.w, ww.w, bb.w)));
      };
      if (h0 != nullptr) out(w0, b0, h0);
      if (h1 != nullptr) out(w1, b1, h1);
    }
  } else {
    for (int c = threadIdx.x; c < width; c += THREADS) {
      const float v = (row[c] - mean) * rinv;
      if (h0 != nullptr) h0[n * width + c] = from_f32<T>(fmaf(v, w0[c], b0[c]));
      if (h1 != nullptr) h1[n * width + c] = from_f32<T>(fmaf(v, w1[c], b1[c]));
    }
  }
}

template <typename T, int VEC>
int sum_ln_launch(float* x32, const int* rows, const void* y0, float s0, const void* y1, float s1, const void* y2, float s2, const float* w0,
                  const float* b0, void* h0, const float* w1, const float* b1, void* h1, float eps, int n, int width, cudaStream_t st) {
  const size_t smem = sizeof(float) * (size_t)width;
  if (smem > 200 * 1024) return DRYFT_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(stream_sum_ln_kernel<T, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  stream_sum_ln_kernel<T, VEC><<<n, THREADS, smem, st>>>(x32, rows, (const T*)y0, s0, (const T*)y1, s1, (const T*)y2, s2, w0, b0, (T*)h0, w1, b1,
                                                        (T*)h1, eps, width);
  return launch_status();
}

template <typename T, int VEC>
__global__ void __launch_bounds__(THREADS) stream_norm_join_kernel(
    float* __restrict__ x32, const T* __restrict__ y0, float s0, const T* __restrict__ y1, float s1, const T* __restrict__ y2, float s2,
    const T* __restrict__ yr, const float* __restrict__ wts, int top, const float* __restrict__ factor, float eps,
    const float* __restrict__ norm_w, float norm_eps, T* __restrict__ h, int width) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  const size_t n = blockIdx.x;
  float* x = x32 + n * width;
  const float* wt = wts + n * top;
  float ss = 0.f;
  // a thread reads and writes the same entries of the row in every pass
  if (VEC == 4) {
    for (int c = threadIdx.x * 4; c < width; c += THREADS * 4) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      auto term = [&](const T* y, float s) {
        const float4 t = load4<T>(y + c);
        v.x = fmaf(s, t.x, v.x); v.y = fmaf(s, t.y, v.y); v.z = fmaf(s, t.z, v.z); v.w = fmaf(s, t.w, v.w);
      };
      if (y0 != nullptr) term(y0 + n * width, s0);
      if (y1 != nullptr) term(y1 + n * width, s1);
      if (y2 != nullptr) term(y2 + n * width, s2);
      if (yr != nullptr) {
#pragma unroll 4
        for (int k = 0; k < top; ++k) term(yr + (n * top + k) * width, wt[k]);      // in the order of the choices
      }
      *reinterpret_cast<float4*>(row + c) = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < width; c += THREADS) {
      float v = 0.f;
      if (y0 != nullptr) v = fmaf(s0, to_f32<T>(y0[n * width + c]), v);
      if (y1 != nullptr) v = fmaf(s1, to_f32<T>(y1[n * width + c]), v);
      if (y2 != nullptr) v = fmaf(s2, to_f32<T>(y2[n * width + c]), v);
      if (yr != nullptr)
        for (int k = 0; k < top; ++k) v = fmaf(wt[k], to_f32<T>(yr[(n * top + k) * width + c]), v);
      row[c] = v;
      ss = fmaf(v, v, ss);
    }
  }
  float rinv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  ss = 0.f;
  if (VEC == 4) {
    for (int c = threadIdx.x * 4; c < width; c += THREADS * 4) {
      const float4 y = *reinterpret_cast<const float4*>(row + c), f = *reinterpret_cast<const float4*>(factor + c);
      float4 v = *reinterpret_cast<const float4*>(x + c);
      v.x = fmaf(y.x * rinv, f.x, v.x); v.y = fmaf(y.y * rinv, f.y, v.y); v.z = fmaf(y.z * rinv, f.z, v.z); v.w = fmaf(y.w * rinv, f.w, v.w);
      *reinterpret_cast<float4*>(x + c) = v;
      *reinterpret_cast<float4*>(row + c) = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < width; c += THREADS) {
      const float v = fmaf(row[c] * rinv, factor[c], x[c]);
      x[c] = v;
      row[c] = v;
      ss = fmaf(v, v, ss);
    }
  }
  if (norm_w == nullptr) return;
  rinv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + norm_eps);
  if (VEC == 4) {
    for (int c = threadIdx.x * 4; c < width; c += THREADS * 4) {
      const float4 v = *reinterpret_cast<const float4*>(row + c), w = *reinterpret_cast<const float4*>(norm_w + c);
      store4<T>(h + n * width + c, make_float4(v.x * rinv * w.x, v.y * rinv * w.y, v.z * rinv * w.z, v.w * rinv * w.w));
    }
  } else {
    for (int c = threadIdx.x; c < width; c += THREADS) h[n * width + c] = from_f32<T>(row[c] * rinv * norm_w[c]);
  }
}

// The same for widths up to 1024 * NV in steps of four: a thread owns NV vectors of four and asks for its part of the results, the
// stream and both factors at once, so that the launch is one trip to memory and two block-wide sums long.
template <typename T, int NV>
__global__ void __launch_bounds__(THREADS) stream_norm_join_regs_kernel(
    float* __restrict__ x32, const T* __restrict__ y0, float s0, const T* __restrict__ y1, float s1, const T* __restrict__ y2, float s2,
    const T* __restrict__ yr, const float* __restrict__ wts, int top, const float* __restrict__ factor, float eps,
    const float* __restrict__ norm_w, float norm_eps, T* __restrict__ h, int width) {
  __shared__ float scratch[33];
  const size_t n = blockIdx.x;
  float* x = x32 + n * width;
  float4 y[NV], xv[NV], f[NV], w[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * THREADS + (int)threadIdx.x) * 4;
    y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < width) {
      xv[i] = *reinterpret_cast<const float4*>(x + c);
      f[i] = *reinterpret_cast<const float4*>(factor + c);
      if (norm_w != nullptr) w[i] = *reinterpret_cast<const float4*>(norm_w + c);
      auto term = [&](const T* p, float s) {
        const float4 t = load4<T>(p + c);
        y[i].x = fmaf(s, t.x, y[i].x); y[i].y = fmaf(s, t.y, y[i].y); y[i].z = fmaf(s, t.z, y[i].z); y[i].w = fmaf(s, t.w, y[i].w);
      };
      if (y0 != nullptr) term(y0 + n * width, s0);
      if (y1 != nullptr) term(y1 + n * width, s1);
      if (y2 != nullptr) term(y2 + n * width, s2);
      if (yr != nullptr) {
#pragma unroll 4
        for (int k = 0; k < top; ++k) term(yr + (n * top + k) * width, wts[n * top + k]);      // in the order of the choices
      }
    }
    ss = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, ss))));
  }
  float rinv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * THREADS + (int)threadIdx.x) * 4;
    if (c < width) {
      float4 v = xv[i];
      v.x = fmaf(y[i].x * rinv, f[i].x, v.x); v.y = fmaf(y[i].y * rinv, f[i].y, v.y);
      v.z = fmaf(y[i].z * rinv, f[i].z, v.z); v.w = fmaf(y[i].w * rinv, f[i].w, v.w);
      *reinterpret_cast<float4*>(x + c) = v;
      y[i] = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  }
  if (norm_w == nullptr) return;
  rinv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + norm_eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * THREADS + (int)threadIdx.x) * 4;
    if (c < width) store4<T>(h + n * width + c, make_float4(y[i].x * rinv * w[i].x, y[i].y * rinv * w[i].y, y[i].z * rinv * w[i].z, y[i].w * rinv * w[i].w));
  }
}

template <typename T, int VEC>
int norm_join_launch(float* x32, const void* y0, float s0, const void* y1, float s1, const void* y2, float s2, const void* yr, const float* wts,
                     int top, const float* factor, float eps, const float* norm_w, float norm_eps, void* h, int n, int width, cudaStream_t st) {
  if (VEC == 4 && width <= 4096) {
    auto kernel = width <= 1024 ? stream_norm_join_regs_kernel<T, 1> : width <= 2048 ? stream_norm_join_regs_kernel<T, 2> : stream_norm_join_regs_kernel<T, 4>;
    kernel<<<n, THREADS, 0, st>>>(x32, (const T*)y0, s0, (const T*)y1, s1, (const T*)y2, s2, (const T*)yr, wts, top, factor, eps, norm_w, norm_eps, (T*)h,
                                  width);
    return launch_status();
  }
  const size_t smem = sizeof(float) * (size_t)width;
  if (smem > 200 * 1024) return DRYFT_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(stream_norm_join_kernel<T, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  stream_norm_join_kernel<T, VEC><<<n, THREADS, smem, st>>>(x32, (const T*)y0, s0, (const T*)y1, s1, (const T*)y2, s2, (const T*)yr, wts, top, factor,
                                                          eps, norm_w, norm_eps, (T*)h, width);
  return launch_status();
}

template <typename T>
__global__ void __launch_bounds__(THREADS) pack_pair_kernel(const float* __restrict__ a, const float* __restrict__ b,
                                                           T* __restrict__ out, int width) {
  const size_t n = blockIdx.x;
  for (int c = threadIdx.x; c < 2 * width; c += THREADS)
    out[n * 2 * width + c] = from_f32<T>(c < width ? a[n * width + c] : b[n * width + (c - width)]);
}

__global__ void softcap_kernel(float* __restrict__ z, size_t count, float cap) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < count) z[i] = cap * tanhf(z[i] / cap);
}
}  // namespace

DRYFT_API int dryft_stream_sum(int is_bf16, float* x32, const float* src, const void* y0, float s0, const void* y1, float s1,
                               const void* y2, float s2, const void* yr, int top, float sr, const float* vec, const float* norm_w,
                               float eps, void* h, int n, int width, cudaStream_t st) {
  if (n <= 0) return 0;
  if (width <= 0 || (yr != nullptr && top < 1) || (norm_w != nullptr && h == nullptr)) return DRYFT_ERR_UNSUPPORTED;
  typedef __nv_bfloat16 bf;
  if (is_bf16)
    stream_sum_kernel<bf><<<n, THREADS, 0, st>>>(x32, src, (const bf*)y0, s0, (const bf*)y1, s1, (const bf*)y2, s2, (const bf*)yr, top, sr,
                                                 vec, norm_w, eps, (bf*)h, width);
  else
    stream_sum_kernel<float><<<n, THREADS, 0, st>>>(x32, src, (const float*)y0, s0, (const float*)y1, s1, (const float*)y2, s2,
                                                    (const float*)yr, top, sr, vec, norm_w, eps, (float*)h, width);
  return launch_status();
}

DRYFT_API int dryft_stream_sum_ln(int is_bf16, float* x32, const int* rows, const void* y0, float s0, const void* y1, float s1, const void* y2,
                                  float s2, const float* w0, const float* b0, void* h0, const float* w1, const float* b1, void* h1, float eps,
                                  int n, int width, cudaStream_t st) {
  if (n <= 0) return 0;
  if (width <= 0 || (rows != nullptr && (y0 != nullptr || y1 != nullptr || y2 != nullptr)) || (h0 != nullptr && (w0 == nullptr || b0 == nullptr)) ||
      (h1 != nullptr && (w1 == nullptr || b1 == nullptr)))
    return DRYFT_ERR_UNSUPPORTED;
  const bool vec = width % 4 == 0;
  if (is_bf16)
    return vec ? sum_ln_launch<__nv_bfloat16, 4>(x32, rows, y0, s0, y1, s1, y2, s2, w0, b0, h0, w1, b1, h1, eps, n, width, st)
               : sum_ln_launch<__nv_bfloat16, 1>(x32, rows, y0, s0, y1, s1, y2, s2, w0, b0, h0, w1, b1, h1, eps, n, width, st);
  return vec ? sum_ln_launch<float, 4>(x32, rows, y0, s0, y1, s1, y2, s2, w0, b0, h0, w1, b1, h1, eps, n, width, st)
             : sum_ln_launch<float, 1>(x32, rows, y0, s0, y1, s1, y2, s2, w0, b0, h0, w1, b1, h1, eps, n, width, st);
}

DRYFT_API int dryft_stream_norm_join(int is_bf16, float* x32, const void* y0, float s0, const void* y1, float s1, const void* y2, float s2,
                                     const void* yr, const float* wts, int top, const float* factor, float eps, const float* norm_w,
                                     float norm_eps, void* h, int n, int width, cudaStream_t st) {
  if (n <= 0) return 0;
  if (width <= 0 || factor == nullptr || (yr != nullptr && (top < 1 || wts == nullptr)) || (norm_w != nullptr && h == nullptr)) return DRYFT_ERR_UNSUPPORTED;
  typedef __nv_bfloat16 bf;
  const bool vec = width % 4 == 0;
  if (is_bf16)
    return vec ? norm_join_launch<bf, 4>(x32, y0, s0, y1, s1, y2, s2, yr, wts, top, factor, eps, norm_w, norm_eps, h, n, width, st)
               : norm_join_launch<bf, 1>(x32, y0, s0, y1, s1, y2, s2, yr, wts, top, factor, eps, norm_w, norm_eps, h, n, width, st);
  return vec ? norm_join_launch<float, 4>(x32, y0, s0, y1, s1, y2, s2, yr, wts, top, factor, eps, norm_w, norm_eps, h, n, width, st)
             : norm_join_launch<float, 1>(x32, y0, s0, y1, s1, y2, s2, yr, wts, top, factor, eps, norm_w, norm_eps, h, n, width, st);
}

DRYFT_API int dryft_pack_pair(int is_bf16, const float* a, const float* b, void* out, int n, int width, cudaStream_t st) {
  if (n <= 0) return 0;
  if (width <= 0) return DRYFT_ERR_UNSUPPORTED;
  if (is_bf16) pack_pair_kernel<__nv_bfloat16><<<n, THREADS, 0, st>>>(a, b, (__nv_bfloat16*)out, width);
  else pack_pair_kernel<float><<<n, THREADS, 0, st>>>(a, b, (float*)out, width);
  return launch_status();
}

DRYFT_API int dryft_softcap(float* z, long long count, float cap, cudaStream_t st) {
  if (count <= 0) return 0;
  if (!(cap > 0.f)) return DRYFT_ERR_UNSUPPORTED;
  softcap_kernel<<<(unsigned)((count + 255) / 256), 256, 0, st>>>(z, (size_t)count, cap);
  return launch_status();
}
