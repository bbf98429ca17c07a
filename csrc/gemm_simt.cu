// Matrix products on the FMA pipes for what the tensor-core GEMM does not take: fp32 operands (true 32-bit,
// no TF32) and bf16 shapes or strides that break the TMA alignment rules.
//
//   C[m, h, n] = sum_k A[m, h * a_head + k] * W[h * N + n, k]      (h < heads; heads == 1: a plain linear)
//
// with an optional bf16 / fp32 bias per row of W, residual, or sigmoid gate. Sums are formed in fp32 in K
// order, so a row's result does not depend on the rows beside it.
//
// The grouped form multiplies every 128-row tile of an expert-sorted list with its expert's matrix (the same device
// lists as the tensor-core GEMM's); its rows of A may be gathered.
//
// One CTA of 256 threads computes a 64 x 64 tile, K in steps of 16 through shared memory; every thread owns
// 4 x 4 outputs. Rows of few (decode) launch 16-row tiles so that more SMs take part.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

constexpr int kBN = 64, kBK = 16;

struct SimtArgs {
  const void* A;
  const void* W;
  void* C;
  const void* bias;
  const void* residual;
  const void* gate;
  int64_t lda, ldw, ldc, ldg, a_head, c_head;
  int M, N, K;
  // grouped form: lists of 128-row tiles, optional row of A for every row of C
  const int* mt_expert;
  const int* mt_row0;
  const int* mt_row_end;
  const int* num_mt;
  const int* a_rows;
};

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

template <typename T, typename TO, int kBM, bool kGrouped>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const SimtArgs a) {
  constexpr int kRM = kBM / 16;  // output rows per thread
  __shared__ float As[kBK][kBM + 4];
  __shared__ float Ws[kBK][kBN + 4];
  int h = blockIdx.z, m0 = blockIdx.y * kBM, M = a.M;
  const int n0 = blockIdx.x * kBN;
  pdl_wait();
  pdl_launch_dependents();
  if constexpr (kGrouped) {
    const int mt = blockIdx.y / (128 / kBM);
    if (mt >= *a.num_mt) return;
    h = a.mt_expert[mt];
    m0 = a.mt_row0[mt] + blockIdx.y % (128 / kBM) * kBM;
    M = a.mt_row_end[mt];
    if (m0 >= M) return;
  }
  const T* A = static_cast<const T*>(a.A) + (kGrouped ? 0 : h * a.a_head);
  const T* W = static_cast<const T*>(a.W) + static_cast<int64_t>(h) * a.N * a.ldw;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[kRM][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += kBK) {
    for (int i = threadIdx.x; i < kBM * kBK; i += 256) {
      const int r = i / kBK, k = i % kBK;
      const bool in = m0 + r < M && k0 + k < a.K;
      const int64_t ar = kGrouped && a.a_rows && in ? a.a_rows[m0 + r] : m0 + r;
      As[k][r] = in ? to_f(A[ar * a.lda + k0 + k]) : 0.f;
    }
    for (int i = threadIdx.x; i < kBN * kBK; i += 256) {
      const int r = i / kBK, k = i % kBK;
      Ws[k][r] = (n0 + r < a.N && k0 + k < a.K) ? to_f(W[(n0 + r) * a.ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kBK; ++k) {
      float x[kRM], w[4];
#pragma unroll
      for (int i = 0; i < kRM; ++i) x[i] = As[k][ty * kRM + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) w[j] = Ws[k][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < kRM; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < kRM; ++i) {
    const int m = m0 + ty * kRM + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= a.N) continue;
      float v = acc[i][j];
      const int64_t wrow = static_cast<int64_t>(h) * a.N + n;
      const int64_t off = m * a.ldc + (kGrouped ? 0 : h * a.c_head) + n;
      if (a.bias) v += to_f(static_cast<const T*>(a.bias)[wrow]);
      if (a.residual) v += to_f(static_cast<const TO*>(a.residual)[off]);
      if (a.gate) v *= 1.f / (1.f + expf(-to_f(static_cast<const T*>(a.gate)[m * a.ldg + wrow])));
      put(static_cast<TO*>(a.C) + off, v);
    }
  }
}

template <typename T, typename TO>
int launch(const SimtArgs& a, int heads, cudaStream_t stream) {
  if (a.M <= 64) {
    const dim3 grid(ceil_div(a.N, kBN), ceil_div(a.M, 16), heads);
    pxl_host::launch(gemm_simt_kernel<T, TO, 16, false>, grid, dim3(256), 0, stream, a);
  } else {
    const dim3 grid(ceil_div(a.N, kBN), ceil_div(a.M, 64), heads);
    pxl_host::launch(gemm_simt_kernel<T, TO, 64, false>, grid, dim3(256), 0, stream, a);
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
}  // namespace

PXL_EXPORT int pxl_gemm_simt(const void* A, const void* W, void* C, const void* bias, const void* residual,
                             const void* gate, int M, int N, int K, int64_t lda, int64_t ldw, int64_t ldc, int64_t ldg,
                             int heads, int64_t a_head, int64_t c_head, int in_f32, int out_f32, cudaStream_t stream) {
  if (M <= 0) return PXL_OK;
  if (N <= 0 || K <= 0 || heads <= 0 || heads > 65535) return PXL_ERR_INVALID_ARG;
  if (in_f32 && !out_f32) return PXL_ERR_INVALID_ARG;
  SimtArgs a{A, W, C, bias, residual, gate, lda, ldw, ldc, ldg, a_head, c_head, M, N, K, nullptr, nullptr, nullptr, nullptr,
             nullptr};
  if (in_f32) return launch<float, float>(a, heads, stream);
  return out_f32 ? launch<pxl::bf16, float>(a, heads, stream) : launch<pxl::bf16, pxl::bf16>(a, heads, stream);
}

PXL_EXPORT int pxl_gemm_simt_grouped(const void* A, const void* W, void* C, const int* a_rows, int N, int K, int64_t lda,
                                     int64_t ldw, int64_t ldc, const int* mt_expert, const int* mt_row0,
                                     const int* mt_row_end, const int* num_mt, int max_m_tiles, int is_f32,
                                     cudaStream_t stream) {
  if (max_m_tiles <= 0) return PXL_OK;
  if (N <= 0 || K <= 0 || max_m_tiles > 32767) return PXL_ERR_INVALID_ARG;
  SimtArgs a{A, W, C, nullptr, nullptr, nullptr, lda, ldw, ldc, 0, 0, 0, 0, N, K, mt_expert, mt_row0, mt_row_end, num_mt, a_rows};
  const dim3 grid(pxl::ceil_div(N, kBN), max_m_tiles * 2);
  if (is_f32) pxl_host::launch(gemm_simt_kernel<float, float, 64, true>, grid, dim3(256), 0, stream, a);
  else pxl_host::launch(gemm_simt_kernel<pxl::bf16, pxl::bf16, 64, true>, grid, dim3(256), 0, stream, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
