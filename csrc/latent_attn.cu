// Latent attention over a paged cache of rows [latent | rotated key] of any widths, in absorbed form:
// scores = scale * (q_lat . latent + q_rot . key), values = latents. Causal, with an optional sliding window
// and an optional learned sink per head (exp(sink) in the softmax denominator, no key, no value, not scaled).
//
//  * pxl_latent_prep: one launch per layer and step turns the packed projection into cache rows (RMS norm of
//    the latent, interleaved rotation of the key part) and the rotated query parts. Where queries go through a normed
//    latent of their own, pxl_latent_rows makes the cache rows and that latent, and pxl_latent_queries the rotated parts.
//  * pxl_latent_attn: FMA-pipe kernel for fp32 models and for bf16 sizes that the tensor-core kernel
//    (latent_attn_tc.cu) does not take. One CTA per (query token, group of heads); keys stream through shared
//    memory in small tiles with an online softmax.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

struct PrepArgs {
  const void* proj;  // [T, ld]: latent | key part at kv_off
  int64_t ld;
  int kv_off;
  const void* q;     // [T, ldq]: query heads from column 0 (null: none)
  int64_t ldq;
  int heads, q_width, q_rot_off, L, R, rot;
  int cq_off, cq_rank;  // query latent in proj (cq_rank 0: none), normed into c_q [T, cq_rank]
  const float* cq_norm;
  void* c_q;
  const float* norm_w;
  const float* cos_sin;  // [max_pos, rot]: cos | sin halves
  const int* positions;
  const int64_t* slots;
  void* cache;    // [num_slots, L + R] (null: no cache rows)
  void* q_cat;    // [T, heads, L + R]: columns L.. written here
  int64_t num_slots;
  int max_pos;
  float eps;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const PrepArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const T* row = static_cast<const T*>(a.proj) + t * a.ld;
  const int half = a.rot / 2;
  int pos = a.positions[t];
  if (pos < 0 || pos >= a.max_pos) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_POSITION);
    pos = 0;
  }
  const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
  int64_t slot = a.cache ? a.slots[t] : -1;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_SLOT);
    slot = -1;
  }
  const int row_w = a.L + a.R;
  if (a.cq_rank > 0) {  // query latent
    const T* c = row + a.cq_off;
    float sq = 0.f;
    for (int i = threadIdx.x; i < a.cq_rank; i += blockDim.x) {
      const float v = to_f(c[i]);
      sq = fmaf(v, v, sq);
    }
    const float inv = 1.f / sqrtf(block_reduce_sum(sq, red) / a.cq_rank + a.eps);
    T* dst = static_cast<T*>(a.c_q) + t * a.cq_rank;
    for (int i = threadIdx.x; i < a.cq_rank; i += blockDim.x) put(dst + i, to_f(c[i]) * inv * a.cq_norm[i]);
  }
  // cache row
  const T* c = row + a.kv_off;
  float inv = 0.f;
  if (a.cache) {
    float sq = 0.f;
    for (int i = threadIdx.x; i < a.L; i += blockDim.x) {
      const float v = to_f(c[i]);
      sq = fmaf(v, v, sq);
    }
    inv = 1.f / sqrtf(block_reduce_sum(sq, red) / a.L + a.eps);
  }
  if (slot >= 0) {
    T* dst = static_cast<T*>(a.cache) + slot * row_w;
    for (int i = threadIdx.x; i < a.L; i += blockDim.x) put(dst + i, to_f(c[i]) * inv * a.norm_w[i]);
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      const float u = to_f(c[a.L + 2 * i]), v = to_f(c[a.L + 2 * i + 1]);
      put(dst + a.L + 2 * i, u * cs[i] - v * cs[half + i]);
      put(dst + a.L + 2 * i + 1, v * cs[i] + u * cs[half + i]);
    }
    for (int i = a.rot + threadIdx.x; i < a.R; i += blockDim.x) dst[a.L + i] = c[a.L + i];
  }
  // rotated query parts
  if (a.q == nullptr) return;
  const T* q_row = static_cast<const T*>(a.q) + t * a.ldq;
  T* q_out = static_cast<T*>(a.q_cat) + t * a.heads * row_w + a.L;
  const int rest = a.R - a.rot, per = half + rest;
  for (int i = threadIdx.x; i < a.heads * per; i += blockDim.x) {
    const int h = i / per, j = i % per;
    const T* q = q_row + static_cast<int64_t>(h) * a.q_width + a.q_rot_off;
    T* o = q_out + static_cast<int64_t>(h) * row_w;
    if (j < half) {
      const float u = to_f(q[2 * j]), v = to_f(q[2 * j + 1]);
      put(o + 2 * j, u * cs[j] - v * cs[half + j]);
      put(o + 2 * j + 1, v * cs[j] + u * cs[half + j]);
    } else {
      o[a.rot + j - half] = q[a.rot + j - half];
    }
  }
}

// ---- FMA-pipe attention -----------------------------------------------------------------------------------
constexpr int kTile = 16;     // keys per tile
constexpr int kHG = 4;        // heads per CTA
constexpr int kThreads = 128;

struct AttnArgs {
  const void* q;       // [T, H, L + R]
  const void* cache;   // [blocks, page, L + R]
  const int* block_tables;
  const int* cu_q;     // null: token i is the only query of sequence i
  const int* ctx_lens;
  void* out;           // [T, H, L]
  const float* sinks;
  int H, L, R, page, max_blocks, window;
  int64_t num_blocks;
  float scale;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) latent_attn_simt_kernel(const AttnArgs a) {
  extern __shared__ float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, h0 = blockIdx.y * kHG;
  const int t0 = a.cu_q ? a.cu_q[b] : b;
  const int len = a.cu_q ? a.cu_q[b + 1] - t0 : 1;
  const int ti = blockIdx.x;
  if (ti >= len) return;
  const int64_t t = t0 + ti;
  const int pos = a.ctx_lens[b] - len + ti;
  const int lo = (a.window > 0 && pos - a.window + 1 > 0) ? pos - a.window + 1 : 0;
  const int D = a.L + a.R;
  float* q = sm;                       // [kHG][D]
  float* acc = q + kHG * D;            // [kHG][L]
  float* kv = acc + kHG * a.L;         // [kTile][D]
  float* s = kv + kTile * D;           // [kHG][kTile]
  float* st = s + kHG * kTile;         // running max, sum, rescale: [3][kHG]
  const int nh = a.H - h0 < kHG ? a.H - h0 : kHG;
  const T* qg = static_cast<const T*>(a.q) + (t * a.H + h0) * D;
  for (int i = threadIdx.x; i < nh * D; i += kThreads) q[i] = to_f(qg[i]);
  for (int i = threadIdx.x; i < kHG * a.L; i += kThreads) acc[i] = 0.f;
  if (threadIdx.x < kHG) {
    st[threadIdx.x] = -INFINITY;
    st[kHG + threadIdx.x] = 0.f;
  }
  const int* bt = a.block_tables + static_cast<int64_t>(b) * a.max_blocks;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int k0 = lo; k0 <= pos; k0 += kTile) {
    const int n = pos + 1 - k0 < kTile ? pos + 1 - k0 : kTile;
    __syncthreads();
    for (int i = threadIdx.x; i < n * D; i += kThreads) {
      const int kp = k0 + i / D;
      const int pg = kp / a.page;
      int64_t blk = pg < a.max_blocks ? bt[pg] : -1;
      if (blk < 0 || blk >= a.num_blocks) {
        if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_BLOCK_PREFILL);
        blk = 0;
      }
      kv[i] = to_f(static_cast<const T*>(a.cache)[(blk * a.page + kp % a.page) * D + i % D]);
    }
    __syncthreads();
    for (int p = warp; p < nh * n; p += kThreads / 32) {
      const int h = p / n, k = p % n;
      float d = 0.f;
      for (int i = lane; i < D; i += 32) d = fmaf(q[h * D + i], kv[k * D + i], d);
      d = warp_reduce_sum(d);
      if (lane == 0) s[h * kTile + k] = d * a.scale;
    }
    __syncthreads();
    if (threadIdx.x < nh) {
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
    for (int i = threadIdx.x; i < nh * a.L; i += kThreads) {
      const int h = i / a.L, c = i % a.L;
      float o = acc[i] * st[2 * kHG + h];
      for (int k = 0; k < n; ++k) o = fmaf(s[h * kTile + k], kv[k * D + c], o);
      acc[i] = o;
    }
  }
  __syncthreads();
  T* out = static_cast<T*>(a.out) + (t * a.H + h0) * a.L;
  for (int i = threadIdx.x; i < nh * a.L; i += kThreads) {
    const int h = i / a.L;
    float m = st[h], l = st[kHG + h], f = 1.f;
    if (a.sinks) {
      const float sink = a.sinks[h0 + h];
      const float mm = fmaxf(m, sink);
      f = expf(m - mm);
      l = l * f + expf(sink - mm);
    }
    put(out + i, l > 0.f ? acc[i] * f / l : 0.f);
  }
}

template <typename T>
int launch_simt(const AttnArgs& a, int B, int max_q, cudaStream_t stream) {
  const int D = a.L + a.R;
  const size_t smem = sizeof(float) * (kHG * D + kHG * a.L + kTile * D + kHG * kTile + 3 * kHG);
  if (smem > 227 * 1024) return PXL_ERR_TOO_LARGE;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(latent_attn_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem)) != cudaSuccess)
    return PXL_ERR_CUDA;
  const dim3 grid(max_q, ceil_div(a.H, kHG), B);
  pxl_host::launch(latent_attn_simt_kernel<T>, grid, dim3(kThreads), smem, stream, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

int launch_prep(const PrepArgs& a, int T, int is_f32, cudaStream_t stream) {
  if (is_f32) pxl_host::launch(latent_prep_kernel<float>, dim3(T), dim3(256), 0, stream, a);
  else pxl_host::launch(latent_prep_kernel<pxl::bf16>, dim3(T), dim3(256), 0, stream, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
}  // namespace

PXL_EXPORT int pxl_latent_prep(const void* proj, int64_t ld, int kv_off, int heads, int q_width, int q_rot_off,
                               const float* norm_w, const float* cos_sin, const int* positions, int max_pos,
                               const int64_t* slots, void* cache, int64_t num_slots, void* q_cat, int T, int L, int R,
                               int rot, float eps, int is_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (heads <= 0 || L <= 0 || R < 0 || rot < 0 || rot > R || (rot % 2) || q_rot_off + R > q_width) return PXL_ERR_INVALID_ARG;
  const PrepArgs a{proj, ld, kv_off, proj, ld, heads, q_width, q_rot_off, L, R, rot, 0, 0, nullptr, nullptr, norm_w, cos_sin,
                   positions, slots, cache, q_cat, num_slots, max_pos, eps, status};
  return launch_prep(a, T, is_f32, stream);
}

PXL_EXPORT int pxl_latent_rows(const void* proj, int64_t ld, int q_off, int q_rank, const float* q_norm, void* c_q, int kv_off,
                               const float* norm_w, const float* cos_sin, const int* positions, int max_pos,
                               const int64_t* slots, void* cache, int64_t num_slots, int T, int L, int R, int rot, float eps,
                               int is_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (q_rank <= 0 || L <= 0 || R < 0 || rot < 0 || rot > R || (rot % 2) || !cache) return PXL_ERR_INVALID_ARG;
  const PrepArgs a{proj, ld, kv_off, nullptr, 0, 0, 0, 0, L, R, rot, q_off, q_rank, q_norm, c_q, norm_w, cos_sin, positions, slots,
                   cache, nullptr, num_slots, max_pos, eps, status};
  return launch_prep(a, T, is_f32, stream);
}

PXL_EXPORT int pxl_latent_queries(const void* q, int64_t ldq, int heads, int q_width, int q_rot_off, const float* cos_sin,
                                  const int* positions, int max_pos, void* q_cat, int T, int L, int R, int rot, int is_f32,
                                  int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (heads <= 0 || L <= 0 || R < 0 || rot < 0 || rot > R || (rot % 2) || q_rot_off + R > q_width) return PXL_ERR_INVALID_ARG;
  const PrepArgs a{q, ldq, 0, q, ldq, heads, q_width, q_rot_off, L, R, rot, 0, 0, nullptr, nullptr, nullptr, cos_sin, positions,
                   nullptr, nullptr, q_cat, 0, max_pos, 0.f, status};
  return launch_prep(a, T, is_f32, stream);
}

PXL_EXPORT int pxl_latent_attn(const void* q, const void* cache, const int* block_tables, const int* cu_q,
                               const int* ctx_lens, void* out, const float* sinks, int B, int max_q, int H, int L, int R,
                               int page, int max_blocks, int64_t num_blocks, float scale, int window, int is_f32,
                               int* status, cudaStream_t stream) {
  if (B <= 0 || max_q <= 0) return PXL_OK;
  if (H <= 0 || L <= 0 || R < 0 || page <= 0 || B > 65535) return PXL_ERR_INVALID_ARG;
  AttnArgs a{q, cache, block_tables, cu_q, ctx_lens, out, sinks, H, L, R, page, max_blocks, window, num_blocks, scale, status};
  return is_f32 ? launch_simt<float>(a, B, max_q, stream) : launch_simt<pxl::bf16>(a, B, max_q, stream);
}
