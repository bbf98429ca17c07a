// The fp32 residual between two products, for layers with tanh norms (tanh(alpha x) w + b: no statistics):
//
//  * pxl_residual_step: x += norm(y + sum of expert rows), norm a tanh norm or RMS norm; x += table[ids]; x += step; and
//    the next product's operand, a tanh norm or a copy of the new x - one pass over the row for all of it.
//  * pxl_tanh_norm: tanh norm of (gathered) rows.
//  * pxl_act_rows: activation (square of relu, GELU) of a product's rows, times rows of a table picked by token id.
//
// This file is compiled without fast math: the divisions are the accurate ones.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

// VEC consecutive elements (VEC == 8: 16-byte aligned)
template <int VEC, typename T>
__device__ __forceinline__ void load_v(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 1) {
    v[0] = to_f(*p);
  } else if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(p + i);
      v[i] = a.x, v[i + 1] = a.y, v[i + 2] = a.z, v[i + 3] = a.w;
    }
  } else {
    const bf16x8 a = ld_bf16x8(p);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(a.u[j]);
      v[2 * j] = f.x, v[2 * j + 1] = f.y;
    }
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void store_v(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 1) {
    put(p, v[0]);
  } else if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4)
      *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
    bf16x8 o;
#pragma unroll
    for (int j = 0; j < 4; ++j) o.u[j] = pack_bf16x2(v[2 * j], v[2 * j + 1]);
    st_bf16x8(p, o);
  }
}

// tanh to a few 1e-7: its Taylor series (to x^9) near zero, 1 - 2 / (e^(2|x|) + 1) elsewhere, without a branch
__device__ __forceinline__ float tanh_of(float x) {
  const float t = fabsf(x), s = x * x;
  const float series = x * fmaf(s, fmaf(s, fmaf(s, fmaf(s, 62.f / 2835.f, -17.f / 315.f), 2.f / 15.f), -1.f / 3.f), 1.f);
  const float far = 1.f - __fdividef(2.f, __expf(2.f * fminf(t, 15.f)) + 1.f);
  return t < 0.3f ? series : copysignf(far, x);
}

struct StepArgs {
  float* x;
  const void* y;         // [T, ldy] or null
  int64_t ldy;
  const void* rows;      // [P, ldr] expert outputs or null
  int64_t ldr, num_rows;
  const int* pos_of;     // [T, k]
  const float* weights;  // [T, k], null: 1
  int k;
  int post;              // 0 none, 1 tanh norm, 2 RMS norm
  const float *post_w, *post_b;
  float post_alpha, eps;
  const void* table;     // [num_ids, W] or null
  const int* ids;
  int64_t num_ids;
  const float* step;     // [W] or null
  int pre;               // 0 none, 1 tanh norm, 2 copy
  const float *pre_w, *pre_b;
  float pre_alpha;
  void* low;
  int W;
  int* status;
};

// row index, or -1 (status set) outside [0, n)
__device__ __forceinline__ int64_t checked(int64_t r, int64_t n, int* status) {
  if (r >= 0 && r < n) return r;
  if (threadIdx.x == 0 && status) atomicCAS(status, 0, PXL_DEV_BAD_ROW_ID);
  return -1;
}

template <int VEC>
__device__ __forceinline__ void tanh_row(float (&v)[VEC], const float* w, const float* b, float alpha, int c) {
  float wv[VEC], bv[VEC];
  load_v<VEC>(w + c, wv);
  load_v<VEC>(b + c, bv);
#pragma unroll
  for (int j = 0; j < VEC; ++j) v[j] = fmaf(tanh_of(alpha * v[j]), wv[j], bv[j]);
}

// one CTA per row; NV vectors of VEC columns per thread (NV == 0: any width, columns in a loop, no RMS norm statistics
// kept in registers)
template <typename T, int VEC>
__device__ __forceinline__ void load_update(const StepArgs& a, int64_t t, int c, float (&v)[VEC]) {
  if (a.y) {
    load_v<VEC>(static_cast<const T*>(a.y) + t * a.ldy + c, v);
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = 0.f;
  }
  if (a.rows) {
    for (int e = 0; e < a.k; ++e) {
      const int64_t r = checked(a.pos_of[t * a.k + e], a.num_rows, a.status);
      if (r < 0) continue;
      const float g = a.weights ? a.weights[t * a.k + e] : 1.f;
      float f[VEC];
      load_v<VEC>(static_cast<const T*>(a.rows) + r * a.ldr + c, f);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = fmaf(g, f[j], v[j]);
    }
  }
}

template <typename T, int VEC>
__device__ __forceinline__ void finish(const StepArgs& a, int64_t t, int64_t id, int c, float inv, float (&v)[VEC]) {
  float x[VEC], f[VEC];
  load_v<VEC>(a.x + t * a.W + c, x);
  if (a.post == 1) {
    tanh_row<VEC>(v, a.post_w, a.post_b, a.post_alpha, c);
  } else if (a.post == 2) {
    load_v<VEC>(a.post_w + c, f);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= inv * f[j];
  }
  if (a.post) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) x[j] += v[j];
  }
  if (id >= 0) {
    load_v<VEC>(static_cast<const T*>(a.table) + id * a.W + c, f);
#pragma unroll
    for (int j = 0; j < VEC; ++j) x[j] += f[j];
  }
  if (a.step) {
    load_v<VEC>(a.step + c, f);
#pragma unroll
    for (int j = 0; j < VEC; ++j) x[j] += f[j];
  }
  if (a.post || id >= 0 || a.step) store_v<VEC>(a.x + t * a.W + c, x);
  if (a.pre == 1) tanh_row<VEC>(x, a.pre_w, a.pre_b, a.pre_alpha, c);
  if (a.pre) store_v<VEC>(static_cast<T*>(a.low) + t * a.W + c, x);
}

template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(256) residual_step_kernel(const StepArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const int64_t id = a.table ? checked(a.ids[t], a.num_ids, a.status) : -1;
  float v[NV][VEC];
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * VEC;
    if (c < a.W && a.post) {
      load_update<T, VEC>(a, t, c, v[i]);
#pragma unroll
      for (int j = 0; j < VEC; ++j) sq = fmaf(v[i][j], v[i][j], sq);
    }
  }
  const float inv = a.post == 2 ? 1.f / sqrtf(block_reduce_sum(sq, red) / a.W + a.eps) : 1.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * VEC;
    if (c < a.W) finish<T, VEC>(a, t, id, c, inv, v[i]);
  }
}

// any width: the row's update is formed twice
template <typename T>
__global__ void __launch_bounds__(256) residual_step_any_kernel(const StepArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const int64_t id = a.table ? checked(a.ids[t], a.num_ids, a.status) : -1;
  float v[1], inv = 1.f;
  if (a.post == 2) {
    float sq = 0.f;
    for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
      load_update<T, 1>(a, t, c, v);
      sq = fmaf(v[0], v[0], sq);
    }
    inv = 1.f / sqrtf(block_reduce_sum(sq, red) / a.W + a.eps);
  }
  for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
    if (a.post) load_update<T, 1>(a, t, c, v);
    finish<T, 1>(a, t, id, c, inv, v);
  }
}

template <typename T>
int launch_step(const StepArgs& a, int rows, bool vec, cudaStream_t stream) {
  const dim3 g(rows);
  const int nvec = a.W / 8;
  if (vec && a.W % 8 == 0 && nvec <= 256 * 4) {
    // a few long rows: one vector per thread keeps more loads in flight
    const int threads = nvec >= 256 ? 256 : ceil_div(nvec, 32) * 32, per = ceil_div(nvec, threads);
    if (per <= 1) pxl_host::launch(residual_step_kernel<T, 8, 1>, g, dim3(threads), 0, stream, a);
    else if (per <= 2) pxl_host::launch(residual_step_kernel<T, 8, 2>, g, dim3(threads), 0, stream, a);
    else pxl_host::launch(residual_step_kernel<T, 8, 4>, g, dim3(threads), 0, stream, a);
  } else {
    pxl_host::launch(residual_step_any_kernel<T>, g, dim3(256), 0, stream, a);
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) tanh_norm_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                        const float* __restrict__ b, float alpha, const int* __restrict__ rows,
                                                        int64_t num_rows, T* __restrict__ out, int W, int* status) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  int64_t r = rows ? checked(rows[t], num_rows, status) : t;
  if (r < 0) r = 0;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC];
    load_v<VEC>(x + r * W + c, v);
    tanh_row<VEC>(v, w, b, alpha, c);
    store_v<VEC>(out + t * W + c, v);
  }
}

// ---- activation of a product's rows -----------------------------------------------------------------------
template <typename TI, typename TO, int VEC>
__global__ void __launch_bounds__(256) act_rows_kernel(const TI* __restrict__ x, int64_t ldx, int act, const TO* __restrict__ table,
                                                       int64_t ldt, int col, const int* __restrict__ ids, int64_t num_ids,
                                                       TO* __restrict__ out, int64_t ldo, int N, int64_t n, int* status) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) * VEC;
  if (i >= n) return;
  const int64_t t = i / N;
  const int c = static_cast<int>(i % N);
  float v[VEC];
  load_v<VEC>(x + t * ldx + c, v);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    if (act == 3) {
      const float r = fmaxf(v[j], 0.f);
      v[j] = r * r;
    } else {
      const float z = v[j];
      v[j] = 0.5f * z * (1.f + tanh_of(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    }
  }
  if (table) {
    int64_t id = ids[t];
    if (id < 0 || id >= num_ids) {
      if (status) atomicCAS(status, 0, PXL_DEV_BAD_ROW_ID);
      id = 0;
    }
    float e[VEC];
    load_v<VEC>(table + id * ldt + col + c, e);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= e[j];
  }
  store_v<VEC>(out + t * ldo + c, v);
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename TI, typename TO>
int launch_act(const void* x, int64_t ldx, int act, const void* table, int64_t ldt, int col, const int* ids, int64_t num_ids,
               void* out, int64_t ldo, int T, int N, int* status, cudaStream_t stream) {
  const bool vec = !((N | ldx | ldo | ldt | col) & 7) && aligned16(x) && aligned16(table) && aligned16(out);
  const int64_t n = static_cast<int64_t>(T) * N, work = vec ? n / 8 : n;
  const dim3 grid(static_cast<unsigned>((work + 255) / 256));
  const TI* xp = static_cast<const TI*>(x);
  const TO* tp = static_cast<const TO*>(table);
  TO* op = static_cast<TO*>(out);
  if (vec)
    pxl_host::launch(act_rows_kernel<TI, TO, 8>, grid, dim3(256), 0, stream, xp, ldx, act, tp, ldt, col, ids, num_ids, op, ldo, N,
                     n, status);
  else
    pxl_host::launch(act_rows_kernel<TI, TO, 1>, grid, dim3(256), 0, stream, xp, ldx, act, tp, ldt, col, ids, num_ids, op, ldo, N,
                     n, status);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
}  // namespace

PXL_EXPORT int pxl_residual_step(float* x, const void* y, int64_t ldy, const void* rows, int64_t ldr, int64_t num_rows,
                                 const int* pos_of, const float* weights, int k, int post, const float* post_w,
                                 const float* post_b, float post_alpha, float eps, const void* table, const int* ids,
                                 int64_t num_ids, const float* step, int pre, const float* pre_w, const float* pre_b,
                                 float pre_alpha, void* low, int T, int W, int is_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (W <= 0 || (post && !y && !rows) || (post && !post_w) || (post == 1 && !post_b) || (pre && !low) ||
      (pre == 1 && (!pre_w || !pre_b)) || (rows && (!pos_of || k <= 0)) || (table && !ids))
    return PXL_ERR_INVALID_ARG;
  const StepArgs a{x, y, ldy, rows, ldr, num_rows, pos_of, weights, k, post, post_w, post_b, post_alpha, eps, table, ids,
                   num_ids, step, pre, pre_w, pre_b, pre_alpha, low, W, status};
  const bool vec = aligned16(x) && aligned16(y) && aligned16(rows) && aligned16(post_w) && aligned16(post_b) &&
                   aligned16(table) && aligned16(step) && aligned16(pre_w) && aligned16(pre_b) && aligned16(low) &&
                   !((ldy | ldr) & 7);
  return is_f32 ? launch_step<float>(a, T, vec, stream) : launch_step<pxl::bf16>(a, T, vec, stream);
}

PXL_EXPORT int pxl_tanh_norm(const float* x, const float* w, const float* b, float alpha, const int* rows, int64_t num_rows,
                             void* out, int T, int W, int out_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (W <= 0) return PXL_ERR_INVALID_ARG;
  const bool vec = W % 8 == 0 && aligned16(x) && aligned16(w) && aligned16(b) && aligned16(out);
  const dim3 g(T), t(256);
  float* of = static_cast<float*>(out);
  pxl::bf16* ob = static_cast<pxl::bf16*>(out);
  if (out_f32) {
    if (vec) pxl_host::launch(tanh_norm_kernel<float, 8>, g, t, 0, stream, x, w, b, alpha, rows, num_rows, of, W, status);
    else pxl_host::launch(tanh_norm_kernel<float, 1>, g, t, 0, stream, x, w, b, alpha, rows, num_rows, of, W, status);
  } else {
    if (vec) pxl_host::launch(tanh_norm_kernel<pxl::bf16, 8>, g, t, 0, stream, x, w, b, alpha, rows, num_rows, ob, W, status);
    else pxl_host::launch(tanh_norm_kernel<pxl::bf16, 1>, g, t, 0, stream, x, w, b, alpha, rows, num_rows, ob, W, status);
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

PXL_EXPORT int pxl_act_rows(const void* x, int64_t ldx, int x_f32, int act, const void* table, int64_t ldt, int col,
                            const int* ids, int64_t num_ids, void* out, int64_t ldo, int out_f32, int T, int N, int* status,
                            cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (N <= 0 || (act != 2 && act != 3) || (table && !ids) || (out_f32 && !x_f32)) return PXL_ERR_INVALID_ARG;
  if (out_f32) return launch_act<float, float>(x, ldx, act, table, ldt, col, ids, num_ids, out, ldo, T, N, status, stream);
  if (x_f32) return launch_act<float, pxl::bf16>(x, ldx, act, table, ldt, col, ids, num_ids, out, ldo, T, N, status, stream);
  return launch_act<pxl::bf16, pxl::bf16>(x, ldx, act, table, ldt, col, ids, num_ids, out, ldo, T, N, status, stream);
}
