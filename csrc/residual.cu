// Rows of an fp32 residual stream: embedding (scaled, with an optional hashed second table), the update
// x += mult * norm(y) * w fused with the low-precision copy the next product reads, the update x += y + weighted
// expert rows fused with the norm that the next layer starts with, norms of fp32 rows, and gated activations in any
// precision. All statistics are fp32; the layer norm's variance is the mean of the squared
// deviations from the mean (two passes over the row, which stays in registers when it is aligned).
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&v)[8]) {
  if constexpr (sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
  } else {
    const bf16x8 a = ld_bf16x8(p);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(a.u[j]);
      v[2 * j] = f.x, v[2 * j + 1] = f.y;
    }
  }
}
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&v)[8]) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  } else {
    bf16x8 o;
#pragma unroll
    for (int j = 0; j < 4; ++j) o.u[j] = pack_bf16x2(v[2 * j], v[2 * j + 1]);
    st_bf16x8(p, o);
  }
}

// ---- embedding -------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) embed_rows_kernel(const T* __restrict__ table, const int* __restrict__ ids,
                                                         float scale, const T* __restrict__ hash,
                                                         const int* __restrict__ prev, int64_t mul_prev, int64_t mul_cur,
                                                         int64_t buckets, float* __restrict__ out, int W,
                                                         int64_t rows, int* status) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int64_t id = ids[t];
  if (id < 0 || id >= rows) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, PXL_DEV_BAD_ROW_ID);
    for (int i = threadIdx.x; i < W; i += blockDim.x) out[static_cast<int64_t>(t) * W + i] = 0.f;
    return;
  }
  const T* src = table + id * W;
  const T* h = nullptr;
  if (hash) {
    const int64_t p = prev[t];
    int64_t row = buckets;
    if (p >= 0) {
      row = (p * mul_prev + id * mul_cur) % buckets;
      if (row < 0) row += buckets;
    }
    h = hash + row * W;
  }
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    float v = to_f(src[i]) * scale;
    if (h) v += to_f(h[i]);
    out[static_cast<int64_t>(t) * W + i] = v;
  }
}

__global__ void __launch_bounds__(256) to_low_kernel(const float* __restrict__ x, bf16* __restrict__ out, int64_t n) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) * 4;
  if (i + 3 < n) {
    const float4 v = *reinterpret_cast<const float4*>(x + i);
    uint2 o;
    o.x = pack_bf16x2(v.x, v.y);
    o.y = pack_bf16x2(v.z, v.w);
    *reinterpret_cast<uint2*>(out + i) = o;
  } else {
    for (int64_t j = i; j < n; ++j) out[j] = __float2bfloat16(x[j]);
  }
}

// ---- norms -----------------------------------------------------------------------------------------------
// kUpdate: src = y (type TI), x updated in place, low = TO copy of x (null when TO is fp32).
// else:    src = x (type TI, row index optional), low = norm(x) * w.
struct NormArgs {
  float* x;
  const void* src;
  const float* w;
  void* low;
  const int* rows;  // row gather (plain norm only)
  int64_t num_rows;
  int W;
  float eps, mult;
  int* status;
};

template <typename TI, typename TO, bool kUpdate, bool kLayer, int NV>
__global__ void __launch_bounds__(256) norm_vec_kernel(const NormArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  int64_t r = t;
  if (!kUpdate && a.rows) {
    r = a.rows[t];
    if (r < 0 || r >= a.num_rows) {
      if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_ROW_ID);
      r = 0;
    }
  }
  const TI* src = static_cast<const TI*>(a.src) + r * a.W;
  float v[NV][8];
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < a.W) {
      load8(src + c, v[i]);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) sum += v[i][j];
  }
  float mean = 0.f;
  if (kLayer) mean = block_reduce_sum(sum, red) / a.W;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < a.W) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        v[i][j] -= mean;
        sq = fmaf(v[i][j], v[i][j], sq);
      }
    }
  }
  sq = block_reduce_sum(sq, red);
  const float inv = a.mult / sqrtf(sq / a.W + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c >= a.W) continue;
    float w[8], o[8];
    load8(a.w + c, w);
    if constexpr (kUpdate) {
      float* x = a.x + t * a.W + c;
      load8(x, o);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = fmaf(v[i][j] * inv, w[j], o[j]);
      store8(x, o);
      if constexpr (sizeof(TO) == 2) store8(static_cast<TO*>(a.low) + t * a.W + c, o);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = v[i][j] * inv * w[j];
      store8(static_cast<TO*>(a.low) + t * a.W + c, o);
    }
  }
}

// any width: three passes over the row in global memory (L1 keeps it)
template <typename TI, typename TO, bool kUpdate, bool kLayer>
__global__ void __launch_bounds__(256) norm_any_kernel(const NormArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  int64_t r = t;
  if (!kUpdate && a.rows) {
    r = a.rows[t];
    if (r < 0 || r >= a.num_rows) {
      if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_ROW_ID);
      r = 0;
    }
  }
  const TI* src = static_cast<const TI*>(a.src) + r * a.W;
  float mean = 0.f;
  if (kLayer) {
    float sum = 0.f;
    for (int c = threadIdx.x; c < a.W; c += blockDim.x) sum += to_f(src[c]);
    mean = block_reduce_sum(sum, red) / a.W;
  }
  float sq = 0.f;
  for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
    const float d = to_f(src[c]) - mean;
    sq = fmaf(d, d, sq);
  }
  sq = block_reduce_sum(sq, red);
  const float inv = a.mult / sqrtf(sq / a.W + a.eps);
  for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
    const float n = (to_f(src[c]) - mean) * inv;
    TO* low = static_cast<TO*>(a.low) + t * a.W + c;
    if constexpr (kUpdate) {
      float* x = a.x + t * a.W + c;
      const float o = fmaf(n, a.w[c], *x);
      *x = o;
      if constexpr (sizeof(TO) == 2) put(low, o);
    } else {
      put(low, n * a.w[c]);
    }
  }
}

template <typename TI, typename TO, bool kUpdate, bool kLayer>
int launch_norm(const NormArgs& a, int T, bool vec, cudaStream_t stream) {
  if (vec && a.W % 8 == 0 && a.W <= 256 * 8 * 8) {
    const int nvec = a.W / 8;
    const int threads = nvec >= 256 ? 256 : ceil_div(nvec, 32) * 32;
    const int per = ceil_div(nvec, threads);
    const dim3 g(T), b(threads);
    if (per <= 1) pxl_host::launch(norm_vec_kernel<TI, TO, kUpdate, kLayer, 1>, g, b, 0, stream, a);
    else if (per <= 2) pxl_host::launch(norm_vec_kernel<TI, TO, kUpdate, kLayer, 2>, g, b, 0, stream, a);
    else if (per <= 4) pxl_host::launch(norm_vec_kernel<TI, TO, kUpdate, kLayer, 4>, g, b, 0, stream, a);
    else pxl_host::launch(norm_vec_kernel<TI, TO, kUpdate, kLayer, 8>, g, b, 0, stream, a);
  } else {
    pxl_host::launch(norm_any_kernel<TI, TO, kUpdate, kLayer>, dim3(T), dim3(256), 0, stream, a);
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
template <typename TI, typename TO, bool kUpdate>
int launch_norm(const NormArgs& a, int T, int kind, bool vec, cudaStream_t stream) {
  return kind == PXL_NORM_LAYER ? launch_norm<TI, TO, kUpdate, true>(a, T, vec, stream)
                                : launch_norm<TI, TO, kUpdate, false>(a, T, vec, stream);
}
inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// RMS norm of (gathered) fp32 rows whose equal parts have statistics of their own; a warp per part
template <typename TO, int VEC>
__global__ void __launch_bounds__(256) group_norm_kernel(const NormArgs a, int groups) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  int64_t r = a.rows ? a.rows[t] : t;
  if (a.rows && (r < 0 || r >= a.num_rows)) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_ROW_ID);
    r = 0;
  }
  const float* x = static_cast<const float*>(a.src) + r * a.W;
  const int lane = threadIdx.x & 31, n = a.W / groups;
  for (int g = threadIdx.x >> 5; g < groups; g += blockDim.x >> 5) {
    float sq = 0.f;
    for (int c = lane * VEC; c < n; c += 32 * VEC) {
      float v[8];
      if constexpr (VEC == 8) load8(x + g * n + c, v);
      else v[0] = x[g * n + c];
#pragma unroll
      for (int j = 0; j < VEC; ++j) sq = fmaf(v[j], v[j], sq);
    }
    const float inv = 1.f / sqrtf(warp_reduce_sum(sq) / n + a.eps);
    for (int c = lane * VEC; c < n; c += 32 * VEC) {
      const int at = g * n + c;
      TO* low = static_cast<TO*>(a.low) + t * a.W + at;
      if constexpr (VEC == 8) {
        float v[8], w[8];
        load8(x + at, v);
        load8(a.w + at, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= inv * w[j];
        store8(low, v);
      } else {
        put(low, x[at] * inv * a.w[at]);
      }
    }
  }
}

template <typename TO>
int launch_group_norm(const NormArgs& a, int T, int groups, bool vec, cudaStream_t stream) {
  const dim3 block(32 * (groups < 8 ? groups : 8));
  if (vec && a.W / groups % 8 == 0) pxl_host::launch(group_norm_kernel<TO, 8>, dim3(T), block, 0, stream, a, groups);
  else pxl_host::launch(group_norm_kernel<TO, 1>, dim3(T), block, 0, stream, a, groups);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

// ---- x += y + sum of chosen experts' rows; low = RMSnorm(x) * w ------------------------------------------
// kNormed: two updates, each RMS-normed over the row: x += mult * (y / rms(y) * yw + y2 / rms(y2) * y2w) instead of y.
// The norm of low has statistics per row, or per each of `groups` equal parts of it.
struct AddArgs {
  float* x;
  const void* y;         // [T, ldy], or null
  int64_t ldy;
  const void* rows;      // [P, ldr] expert outputs, or null
  int64_t ldr, num_rows;
  const int* pos_of;     // [T, k]: row of the pair in `rows`; negative: the identity expert, whose output is h[t]
  const float* weights;  // [T, k]
  int k;
  const void* h;         // [T, W]
  const float* w;        // norm weight, or null (no norm)
  void* low;
  int W;
  float eps;
  int* status;
  const float* yw;       // kNormed: norm weights of y and y2
  const void* y2;        // [T, ldy]
  const float* y2w;
  float mult;
  int groups;
};

template <typename T>
__device__ __forceinline__ const T* expert_row(const AddArgs& a, int64_t t, int j) {
  const int64_t r = a.pos_of[t * a.k + j];
  if (r < 0) return static_cast<const T*>(a.h) + t * a.W;
  if (r >= a.num_rows) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_ROW_ID);
    return static_cast<const T*>(a.h) + t * a.W;
  }
  return static_cast<const T*>(a.rows) + r * a.ldr;
}

// NV vectors of 8 elements per thread
template <typename T, int NV, bool kNormed>
__global__ void __launch_bounds__(256) residual_add_vec_kernel(const AddArgs a) {
  __shared__ float red[32];
  extern __shared__ float parts[];  // groups > 1: sums of the row's vectors, then the parts' factors
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  float v[NV][8], f[8];
  if constexpr (kNormed) {
    float s1 = 0.f, s2 = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 8;
      if (c < a.W) {
        load8(static_cast<const T*>(a.y) + t * a.ldy + c, v[i]);
        load8(static_cast<const T*>(a.y2) + t * a.ldy + c, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) s1 = fmaf(v[i][j], v[i][j], s1), s2 = fmaf(f[j], f[j], s2);
      }
    }
    const float i1 = a.mult / sqrtf(block_reduce_sum(s1, red) / a.W + a.eps);
    const float i2 = a.mult / sqrtf(block_reduce_sum(s2, red) / a.W + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 8;
      if (c < a.W) {
        float w[8];
        load8(a.yw + c, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] *= i1 * w[j];
        load8(a.y2w + c, w);
        load8(static_cast<const T*>(a.y2) + t * a.ldy + c, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] = fmaf(i2 * w[j], f[j], v[i][j]);
        load8(a.x + t * a.W + c, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] += f[j];
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 8;
      if (c < a.W) {
        load8(a.x + t * a.W + c, v[i]);
        if (a.y) {
          load8(static_cast<const T*>(a.y) + t * a.ldy + c, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) v[i][j] += f[j];
        }
      }
    }
  }
  if (a.rows) {
    for (int e = 0; e < a.k; ++e) {
      const T* r = expert_row<T>(a, t, e);
      const float g = a.weights[t * a.k + e];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * blockDim.x + threadIdx.x) * 8;
        if (c < a.W) {
          load8(r + c, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) v[i][j] = fmaf(g, f[j], v[i][j]);
        }
      }
    }
  }
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < a.W) {
      store8(a.x + t * a.W + c, v[i]);
      float one = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) one = fmaf(v[i][j], v[i][j], one);
      if (a.groups > 1) parts[c / 8] = one;
      sq += one;
    }
  }
  if (!a.w) return;
  float inv = 1.f;
  float* factor = parts + a.W / 8;
  const int n8 = a.W / 8 / a.groups;
  if (a.groups > 1) {
    __syncthreads();
    for (int g = threadIdx.x >> 5; g < a.groups; g += blockDim.x >> 5) {
      float sum = 0.f;
      for (int i = threadIdx.x & 31; i < n8; i += 32) sum += parts[g * n8 + i];
      sum = warp_reduce_sum(sum);
      if ((threadIdx.x & 31) == 0) factor[g] = 1.f / sqrtf(sum / (n8 * 8) + a.eps);
    }
    __syncthreads();
  } else {
    inv = 1.f / sqrtf(block_reduce_sum(sq, red) / a.W + a.eps);
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < a.W) {
      load8(a.w + c, f);
      if (a.groups > 1) inv = factor[c / 8 / n8];
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= v[i][j] * inv;
      store8(static_cast<T*>(a.low) + t * a.W + c, f);
    }
  }
}

// any width
template <typename T>
__global__ void __launch_bounds__(256) residual_add_any_kernel(const AddArgs a) {
  __shared__ float red[32];
  extern __shared__ float factor[];  // [groups]
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  float* x = a.x + t * a.W;
  const T* y = a.y ? static_cast<const T*>(a.y) + t * a.ldy : nullptr;
  const T* y2 = a.y2 ? static_cast<const T*>(a.y2) + t * a.ldy : nullptr;
  float i1 = 1.f, i2 = 0.f;
  if (y2) {
    float s1 = 0.f, s2 = 0.f;
    for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
      s1 = fmaf(to_f(y[c]), to_f(y[c]), s1);
      s2 = fmaf(to_f(y2[c]), to_f(y2[c]), s2);
    }
    i1 = a.mult / sqrtf(block_reduce_sum(s1, red) / a.W + a.eps);
    i2 = a.mult / sqrtf(block_reduce_sum(s2, red) / a.W + a.eps);
  }
  for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
    float v = x[c];
    if (y2) v += fmaf(i1 * a.yw[c], to_f(y[c]), i2 * a.y2w[c] * to_f(y2[c]));
    else if (y) v += to_f(y[c]);
    if (a.rows)
      for (int e = 0; e < a.k; ++e) v = fmaf(a.weights[t * a.k + e], to_f(expert_row<T>(a, t, e)[c]), v);
    x[c] = v;
  }
  if (!a.w) return;
  __syncthreads();
  const int n = a.W / a.groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int g = warp; g < a.groups; g += blockDim.x >> 5) {
    float sq = 0.f;
    for (int c = lane; c < n; c += 32) sq = fmaf(x[g * n + c], x[g * n + c], sq);
    sq = warp_reduce_sum(sq);
    if (lane == 0) factor[g] = 1.f / sqrtf(sq / n + a.eps);
  }
  __syncthreads();
  for (int c = threadIdx.x; c < a.W; c += blockDim.x) put(static_cast<T*>(a.low) + t * a.W + c, x[c] * factor[c / n] * a.w[c]);
}

template <typename T, bool kNormed>
int launch_add(const AddArgs& a, int rows, bool vec, cudaStream_t stream) {
  if (vec && a.W % 8 == 0 && a.W <= 256 * 8 * 8 && (a.groups == 1 || a.W / a.groups % 8 == 0)) {
    const int nvec = a.W / 8, threads = nvec >= 256 ? 256 : ceil_div(nvec, 32) * 32, per = ceil_div(nvec, threads);
    const dim3 g(rows), b(threads);
    const size_t smem = a.groups > 1 ? sizeof(float) * (nvec + a.groups) : 0;
    if (per <= 1) pxl_host::launch(residual_add_vec_kernel<T, 1, kNormed>, g, b, smem, stream, a);
    else if (per <= 2) pxl_host::launch(residual_add_vec_kernel<T, 2, kNormed>, g, b, smem, stream, a);
    else if (per <= 4) pxl_host::launch(residual_add_vec_kernel<T, 4, kNormed>, g, b, smem, stream, a);
    else pxl_host::launch(residual_add_vec_kernel<T, 8, kNormed>, g, b, smem, stream, a);
  } else {
    pxl_host::launch(residual_add_any_kernel<T>, dim3(rows), dim3(256), sizeof(float) * a.groups, stream, a);
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
template <typename T>
int launch_add(const AddArgs& a, int rows, bool vec, cudaStream_t stream) {
  return a.y2 ? launch_add<T, true>(a, rows, vec, stream) : launch_add<T, false>(a, rows, vec, stream);
}

// ---- gated activation of gate / up columns interleaved in groups of 64 --------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) glu_act_kernel(const T* __restrict__ x, const float* __restrict__ row_gate, int64_t ldg,
                                                      T* __restrict__ out, int64_t ldo, int I, int64_t n, int mode, float limit) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= n) return;
  const int64_t t = i / I, c = i % I, col = c / 64 * 128 + c % 64;
  float g = to_f(x[t * 2 * I + col]), u = to_f(x[t * 2 * I + col + 64]);
  if (mode == 1) g = fminf(g, limit), u = fminf(fmaxf(u, -limit), limit) + 1.f;
  // gelu, tanh form: z (1 + tanh(s)) / 2 = z / (1 + exp(-2 s))
  const float s = mode == 2 ? 1.5957691216057308f * (g + 0.044715f * g * g * g) : mode == 1 ? 1.702f * g : g;
  float y = g / (1.f + expf(-s)) * u;
  if (row_gate) y /= 1.f + expf(-row_gate[t * ldg]);
  put(out + t * ldo + c, y);
}

// ---- clipped GLU and friends in fp32 -------------------------------------------------------------------------
__global__ void __launch_bounds__(256) act_mul_f32_kernel(const float* __restrict__ x, float* __restrict__ out, int I,
                                                          int64_t n, int mode, float limit) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= n) return;
  const int64_t t = i / I, c = i % I;
  float g = x[t * 2 * I + c], u = x[t * 2 * I + I + c];
  float y;
  if (mode == 1) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    y = g / (1.f + expf(-1.702f * g)) * (u + 1.f);
  } else if (mode == 0) {
    y = g / (1.f + expf(-g)) * u;
  } else {
    y = 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
  }
  out[i] = y;
}
}  // namespace

PXL_EXPORT int pxl_embed_rows(const void* table, const int* ids, float scale, const void* hash, const int* prev,
                              int64_t mul_prev, int64_t mul_cur, int64_t buckets, float* out, int T, int W,
                              int64_t num_rows, int is_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (W <= 0 || (hash && (prev == nullptr || buckets <= 0))) return PXL_ERR_INVALID_ARG;
  if (is_f32)
    pxl_host::launch(embed_rows_kernel<float>, dim3(T), dim3(128), 0, stream, static_cast<const float*>(table), ids, scale,
                     static_cast<const float*>(hash), prev, mul_prev, mul_cur, buckets, out, W, num_rows, status);
  else
    pxl_host::launch(embed_rows_kernel<pxl::bf16>, dim3(T), dim3(128), 0, stream, static_cast<const pxl::bf16*>(table), ids,
                     scale, static_cast<const pxl::bf16*>(hash), prev, mul_prev, mul_cur, buckets, out, W, num_rows, status);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

PXL_EXPORT int pxl_f32_to_bf16(const float* x, void* out, int64_t n, cudaStream_t stream) {
  if (n <= 0) return PXL_OK;
  if (!aligned16(x) || !aligned16(out)) return PXL_ERR_INVALID_ARG;
  pxl_host::launch(to_low_kernel, dim3(static_cast<unsigned>((n + 1023) / 1024)), dim3(256), 0, stream, x,
                   static_cast<pxl::bf16*>(out), n);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

PXL_EXPORT int pxl_residual_norm(float* x, const void* y, const float* w, void* low, int T, int W, float eps, float mult,
                                 int kind, int y_f32, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (W <= 0 || (!y_f32 && low == nullptr)) return PXL_ERR_INVALID_ARG;
  NormArgs a{x, y, w, low, nullptr, T, W, eps, mult, nullptr};
  const bool vec = aligned16(x) && aligned16(y) && aligned16(w) && aligned16(low);
  return y_f32 ? launch_norm<float, float, true>(a, T, kind, vec, stream)
               : launch_norm<pxl::bf16, pxl::bf16, true>(a, T, kind, vec, stream);
}

PXL_EXPORT int pxl_row_norm(const float* x, const float* w, const int* rows, int64_t num_rows, void* out, int T, int W,
                            float eps, int kind, int groups, int out_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (W <= 0 || groups < 1 || W % groups || (groups > 1 && kind != PXL_NORM_RMS)) return PXL_ERR_INVALID_ARG;
  NormArgs a{nullptr, x, w, out, rows, num_rows, W, eps, 1.f, status};
  const bool vec = aligned16(x) && aligned16(w) && aligned16(out);
  if (groups > 1)
    return out_f32 ? launch_group_norm<float>(a, T, groups, vec, stream) : launch_group_norm<pxl::bf16>(a, T, groups, vec, stream);
  return out_f32 ? launch_norm<float, float, false>(a, T, kind, vec, stream)
                 : launch_norm<float, pxl::bf16, false>(a, T, kind, vec, stream);
}

PXL_EXPORT int pxl_act_mul_f32(const float* x, float* out, int T, int I, int mode, float limit, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (I <= 0) return PXL_ERR_INVALID_ARG;
  const int64_t n = static_cast<int64_t>(T) * I;
  pxl_host::launch(act_mul_f32_kernel, dim3(static_cast<unsigned>((n + 255) / 256)), dim3(256), 0, stream, x, out, I, n,
                   mode, limit);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

PXL_EXPORT int pxl_residual_add(float* x, const void* y, int64_t ldy, const void* rows, int64_t ldr, int64_t num_rows,
                                const int* pos_of, const float* weights, int k, const void* h, const float* w, void* low,
                                int T, int W, float eps, const float* yw, const void* y2, const float* y2w, float mult, int groups,
                                int y_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (W <= 0 || (w && !low) || (rows && (!pos_of || !weights || !h || k <= 0)) || (y2 && (!y || !yw || !y2w)) || groups < 1 ||
      groups > 8192 || W % groups)
    return PXL_ERR_INVALID_ARG;
  const AddArgs a{x, y, ldy, rows, ldr, num_rows, pos_of, weights, k, h, w, low, W, eps, status, yw, y2, y2w, mult, groups};
  const bool vec = aligned16(x) && aligned16(y2) && aligned16(yw) && aligned16(y2w) && aligned16(y) && aligned16(rows) && aligned16(h) && aligned16(w) && aligned16(low) &&
                   ldy % 8 == 0 && ldr % 8 == 0;
  return y_f32 ? launch_add<float>(a, T, vec, stream) : launch_add<pxl::bf16>(a, T, vec, stream);
}

PXL_EXPORT int pxl_glu_act(const void* x, const float* row_gate, int64_t ldg, void* out, int64_t ldo, int T, int I, int mode,
                           float limit, int is_f32, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (I <= 0 || I % 64 || mode < 0 || mode > 2) return PXL_ERR_INVALID_ARG;
  const int64_t n = static_cast<int64_t>(T) * I;
  const dim3 grid(static_cast<unsigned>((n + 255) / 256));
  if (is_f32)
    pxl_host::launch(glu_act_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(x), row_gate, ldg,
                     static_cast<float*>(out), ldo, I, n, mode, limit);
  else
    pxl_host::launch(glu_act_kernel<pxl::bf16>, grid, dim3(256), 0, stream, static_cast<const pxl::bf16*>(x), row_gate, ldg,
                     static_cast<pxl::bf16*>(out), ldo, I, n, mode, limit);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
