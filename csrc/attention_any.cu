// Paged attention with grouped heads on the FMA pipes, bf16 or fp32, any head size: what the tensor-core kernels
// (attention.cu, attention_prefill_tc.cu) do not take - fp32 models, head sizes other than 64 and 128, many query
// heads per key head. Causal, optional sliding window (which may keep a sequence's first keys), optional sink per head (exp(sink) in the softmax
// denominator, no key, no value, not scaled), optional soft cap of the scores, or sigmoid weights. Cache layout as in attention.cu: K, V = [blocks, Hkv, page, D].
//
// One CTA per (query token, up to four query heads of one key head); keys stream through shared memory in small
// tiles with an online softmax, all in fp32.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

constexpr int kTile = 32;  // keys per tile
constexpr int kHG = 4;     // query heads per CTA
constexpr int kThreads = 128;

struct AnyArgs {
  const void* q;
  int64_t q_stride;
  const void* k;
  const void* v;
  const int* block_tables;
  const int* cu_q;  // null: token i is the only query of sequence i
  const int* ctx_lens;
  void* out;
  int64_t out_stride;
  const float* sinks;
  int Hq, Hkv, D, page, max_blocks, window, keep;
  int64_t num_blocks;
  float scale;
  float softcap;          // scores: softcap * tanh(score / softcap) (0: none)
  const float* sig_bias;  // [Hq]: weights sigmoid(score + bias), not normalised (null: softmax)
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) attn_any_kernel(const AnyArgs a) {
  extern __shared__ float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int group = a.Hq / a.Hkv, per_kv = ceil_div(group, kHG);
  const int b = blockIdx.z, kvh = blockIdx.y / per_kv, h0 = kvh * group + blockIdx.y % per_kv * kHG;
  const int left = (kvh + 1) * group - h0, nh = left < kHG ? left : kHG;
  const int t0 = a.cu_q ? a.cu_q[b] : b;
  const int len = a.cu_q ? a.cu_q[b + 1] - t0 : 1;
  const int ti = blockIdx.x, D = a.D;
  if (ti >= len) return;
  const int64_t t = t0 + ti;
  const int pos = a.ctx_lens[b] - len + ti;
  const int lo = (a.window > 0 && pos - a.window + 1 > 0) ? pos - a.window + 1 : 0;
  // the visible keys are [0, keep) and [lo, pos], walked as one run
  const int keep = a.keep < lo ? a.keep : lo, total = keep + pos + 1 - lo;
  float* q = sm;                    // [kHG][D]
  float* acc = q + kHG * D;         // [kHG][D]
  float* ks = acc + kHG * D;        // [kTile][D]
  float* vs = ks + kTile * D;       // [kTile][D]
  float* s = vs + kTile * D;        // [kHG][kTile]
  float* st = s + kHG * kTile;      // running max, sum, rescale: [3][kHG]
  const T* qg = static_cast<const T*>(a.q) + t * a.q_stride + static_cast<int64_t>(h0) * D;
  for (int i = threadIdx.x; i < nh * D; i += kThreads) {
    q[i] = to_f(qg[i]);
    acc[i] = 0.f;
  }
  if (threadIdx.x < kHG) {
    st[threadIdx.x] = -INFINITY;
    st[kHG + threadIdx.x] = 0.f;
  }
  const int* bt = a.block_tables + static_cast<int64_t>(b) * a.max_blocks;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int k0 = 0; k0 < total; k0 += kTile) {
    const int n = total - k0 < kTile ? total - k0 : kTile;
    __syncthreads();
    for (int i = threadIdx.x; i < n * D; i += kThreads) {
      const int at = k0 + i / D, kp = at < keep ? at : at - keep + lo, pg = kp / a.page;
      int64_t blk = pg < a.max_blocks ? bt[pg] : -1;
      if (blk < 0 || blk >= a.num_blocks) {
        if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_BLOCK_PREFILL);
        blk = 0;
      }
      const int64_t off = ((blk * a.Hkv + kvh) * a.page + kp % a.page) * D + i % D;
      ks[i] = to_f(static_cast<const T*>(a.k)[off]);
      vs[i] = to_f(static_cast<const T*>(a.v)[off]);
    }
    __syncthreads();
    for (int p = warp; p < nh * n; p += kThreads / 32) {
      const int h = p / n, k = p % n;
      float d = 0.f;
      for (int i = lane; i < D; i += 32) d = fmaf(q[h * D + i], ks[k * D + i], d);
      d = warp_reduce_sum(d);
      if (lane == 0) {
        float x = d * a.scale;
        if (a.softcap > 0.f) x = a.softcap * tanhf(x / a.softcap);
        s[h * kTile + k] = a.sig_bias ? 1.f / (1.f + expf(-(x + a.sig_bias[h0 + h]))) : x;
      }
    }
    __syncthreads();
    if (threadIdx.x < nh && a.sig_bias) {
      st[2 * kHG + threadIdx.x] = 1.f;
    } else if (threadIdx.x < nh) {
      const int h = threadIdx.x;
      float m = st[h];
      for (int k = 0; k < n; ++k) m = fmaxf(m, s[h * kTile + k]);
      const float al = expf(st[h] - m);  // 0 on the first tile
      float l = st[kHG + h] * al;
      for (int k = 0; k < n; ++k) {
        const float p = expf(s[h * kTile + k] - m);
        s[h * kTile + k] = p;
        l += p;
      }
      st[h] = m;
      st[kHG + h] = l;
      st[2 * kHG + h] = al;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nh * D; i += kThreads) {
      const int h = i / D, c = i % D;
      float o = acc[i] * st[2 * kHG + h];
      for (int k = 0; k < n; ++k) o = fmaf(s[h * kTile + k], vs[k * D + c], o);
      acc[i] = o;
    }
  }
  __syncthreads();
  T* out = static_cast<T*>(a.out) + t * a.out_stride + static_cast<int64_t>(h0) * D;
  for (int i = threadIdx.x; i < nh * D; i += kThreads) {
    const int h = i / D;
    float m = st[h], l = st[kHG + h], f = 1.f;
    if (a.sig_bias) {
      l = 1.f;
    } else if (a.sinks) {
      const float sink = a.sinks[h0 + h], mm = fmaxf(m, sink);
      f = expf(m - mm);
      l = l * f + expf(sink - mm);
    }
    put(out + i, l > 0.f ? acc[i] * f / l : 0.f);
  }
}

template <typename T>
int launch_any(const AnyArgs& a, int B, int max_q, cudaStream_t stream) {
  const size_t smem = sizeof(float) * (2 * kHG * a.D + 2 * kTile * a.D + kHG * kTile + 3 * kHG);
  if (smem > 227 * 1024) return PXL_ERR_TOO_LARGE;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(attn_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem)) != cudaSuccess)
    return PXL_ERR_CUDA;
  const dim3 grid(max_q, a.Hkv * ceil_div(a.Hq / a.Hkv, kHG), B);
  pxl_host::launch(attn_any_kernel<T>, grid, dim3(kThreads), smem, stream, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
}  // namespace

PXL_EXPORT int pxl_attn_any(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, const int* block_tables,
                            const int* cu_q, const int* ctx_lens, void* out, int64_t out_stride, const float* sinks, int B,
                            int max_q, int Hq, int Hkv, int D, int page, int max_blocks, int64_t num_blocks, float scale,
                            int window, int keep_first, float softcap, const float* sig_bias, int is_f32, int* status,
                            cudaStream_t stream) {
  if (B <= 0 || max_q <= 0) return PXL_OK;
  if (Hkv <= 0 || Hq % Hkv || D <= 0 || page <= 0 || B > 65535) return PXL_ERR_INVALID_ARG;
  AnyArgs a{q, q_stride, k_cache, v_cache, block_tables, cu_q, ctx_lens, out, out_stride, sinks, Hq, Hkv, D, page, max_blocks,
            window, keep_first, num_blocks, scale, softcap, sig_bias, status};
  return is_f32 ? launch_any<float>(a, B, max_q, stream) : launch_any<pxl::bf16>(a, B, max_q, stream);
}
