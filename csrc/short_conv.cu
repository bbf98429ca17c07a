// Short causal convolution per channel with SiLU, in front of a recurrence: y_t = silu(b + sum_j w[j] u[t - taps + 1 + j]),
// zeros before the sequence, any number of taps, bf16 or fp32 rows, fp32 arithmetic. The last taps - 1 inputs of a request
// live in its state slot. Prompt slices: a thread walks a run of tokens of 8 channels with weights and inputs in registers;
// other sizes and decoded tokens: a thread per token and vector, which for a decoded token also advances the slot. The slot of
// a prompt slice is rewritten by a launch of its own, because the slice's first tokens read what its last ones replace.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

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
    for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
    bf16x8 o;
#pragma unroll
    for (int j = 0; j < 4; ++j) o.u[j] = pack_bf16x2(v[2 * j], v[2 * j + 1]);
    st_bf16x8(p, o);
  }
}

struct ConvArgs {
  const void* x;  // [T, ldx], C channels
  int64_t ldx;
  int C, taps;
  const void* w;     // [taps, C]
  const void* bias;  // [C] or null
  void* state;       // [slots, taps - 1, C], oldest first
  int num_slots;
  const int* positions;
  const int* seq_cu;
  const int* seq_slots;
  int prefill_seqs, prefill_tokens, T;
  void* out;  // [T, C]
  int* status;
};

__device__ __forceinline__ float silu(float v) { return v / (1.f + expf(-v)); }

// last prompt slice that starts at or before token t
__device__ __forceinline__ int slice_of(const ConvArgs& a, int t) {
  int lo = 0, hi = a.prefill_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (a.seq_cu[mid] <= t) lo = mid;
    else hi = mid - 1;
  }
  return lo;
}

// state rows of a sequence, or null (status set) for a slot outside the pool
template <typename T>
__device__ __forceinline__ T* state_of(const ConvArgs& a, int seq) {
  const int slot = a.seq_slots[seq];
  if (slot >= 0 && slot < a.num_slots) return static_cast<T*>(a.state) + static_cast<int64_t>(slot) * (a.taps - 1) * a.C;
  if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_INDEX);
  return nullptr;
}

template <typename T, int VEC>
__global__ void __launch_bounds__(128) conv_token_kernel(const ConvArgs a, int begin) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC, t = begin + blockIdx.y;
  if (c >= a.C) return;
  const bool decoded = t >= a.prefill_tokens;
  const int seq = decoded ? a.prefill_seqs + t - a.prefill_tokens : slice_of(a, t);
  const int li = t - a.seq_cu[seq], back = a.taps - 1, pos = a.positions[t];
  T* state = nullptr;
  if (back > 0 && li < back) {
    state = state_of<T>(a, seq);
    if (!state) return;
    state += c;
  }
  const T* cur = static_cast<const T*>(a.x) + static_cast<int64_t>(t) * a.ldx + c;
  const T* w = static_cast<const T*>(a.w) + c;
  float u[VEC], y[VEC], h[VEC], wv[VEC];
  if (a.bias) {
    load_v<VEC>(static_cast<const T*>(a.bias) + c, y);
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) y[j] = 0.f;
  }
  load_v<VEC>(cur, u);
  load_v<VEC>(w + static_cast<int64_t>(back) * a.C, wv);
#pragma unroll
  for (int j = 0; j < VEC; ++j) y[j] = fmaf(wv[j], u[j], y[j]);
  for (int b = back; b >= 1; --b) {
    if (pos - b < 0) continue;
    if (b <= li) load_v<VEC>(cur - static_cast<int64_t>(b) * a.ldx, h);
    else load_v<VEC>(state + static_cast<int64_t>(back + li - b) * a.C, h);
    load_v<VEC>(w + static_cast<int64_t>(back - b) * a.C, wv);
#pragma unroll
    for (int j = 0; j < VEC; ++j) y[j] = fmaf(wv[j], h[j], y[j]);
  }
  if (decoded && back > 0) {  // this thread is the only reader and writer of these channels
    for (int m = 0; m + 1 < back; ++m) {
      load_v<VEC>(state + static_cast<int64_t>(m + 1) * a.C, h);
      store_v<VEC>(state + static_cast<int64_t>(m) * a.C, h);
    }
    store_v<VEC>(state + static_cast<int64_t>(back - 1) * a.C, u);
  }
#pragma unroll
  for (int j = 0; j < VEC; ++j) y[j] = silu(y[j]);
  store_v<VEC>(static_cast<T*>(a.out) + static_cast<int64_t>(t) * a.C + c, y);
}

template <int TAPS>
__global__ void __launch_bounds__(128) conv_run_kernel(const ConvArgs a, int run) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= a.C) return;
  constexpr int kBack = TAPS - 1;
  const int first = blockIdx.y * run, last = first + run < a.prefill_tokens ? first + run : a.prefill_tokens;
  int seq = slice_of(a, first);
  const bf16x8 zero8 = {{0u, 0u, 0u, 0u}};
  const bf16* w = static_cast<const bf16*>(a.w) + c;
  const bf16* cur = static_cast<const bf16*>(a.x) + static_cast<int64_t>(first) * a.ldx + c;
  bf16x8 wt[TAPS], hist[kBack > 0 ? kBack : 1];
  float b0[8] = {};
#pragma unroll
  for (int j = 0; j < TAPS; ++j) wt[j] = ld_bf16x8(w + static_cast<int64_t>(j) * a.C);
  if (a.bias) load_v<8>(static_cast<const bf16*>(a.bias) + c, b0);
  constexpr int kAhead = 4;  // tokens whose inputs are on their way
  bf16x8 ahead[kAhead];
#pragma unroll
  for (int i = 0; i < kAhead; ++i) ahead[i] = first + i < last ? ld_bf16x8(cur + static_cast<int64_t>(i) * a.ldx) : zero8;
  int start = a.seq_cu[seq], end = a.seq_cu[seq + 1];
  for (int t4 = first; t4 < last; t4 += kAhead) {
#pragma unroll
    for (int i4 = 0; i4 < kAhead; ++i4, cur += a.ldx) {
      const int t = t4 + i4;
      if (t >= last) break;
      while (end <= t) ++seq, start = end, end = a.seq_cu[seq + 1];
      const int li = t - start;
      if (kBack > 0 && (t == first || li == 0)) {  // the inputs before this run, or of this sequence's earlier steps
        const int pos = a.positions[t];
        const bf16* state = li < kBack ? state_of<bf16>(a, seq) : nullptr;
#pragma unroll
        for (int j = 0; j < kBack; ++j) {
          const int b = kBack - j;
          hist[j] = zero8;
          if (pos - b < 0) continue;
          if (b <= li) hist[j] = ld_bf16x8(cur - static_cast<int64_t>(b) * a.ldx);
          else if (state) hist[j] = ld_bf16x8(state + static_cast<int64_t>(li + j) * a.C + c);
        }
      }
      const bf16x8 here = ahead[i4];
      if (t + kAhead < last) ahead[i4] = ld_bf16x8(cur + kAhead * a.ldx);
      float y[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = b0[e];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const bf16x8& x = j < kBack ? hist[j < kBack ? j : 0] : here;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 xf = unpack_bf16x2(x.u[e]), wf = unpack_bf16x2(wt[j].u[e]);
          y[2 * e] = fmaf(wf.x, xf.x, y[2 * e]);
          y[2 * e + 1] = fmaf(wf.y, xf.y, y[2 * e + 1]);
        }
      }
#pragma unroll
      for (int j = 0; j + 1 < kBack; ++j) hist[j] = hist[j + 1];
      if constexpr (kBack > 0) hist[kBack - 1] = here;
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = silu(y[e]);
      store_v<8>(static_cast<bf16*>(a.out) + static_cast<int64_t>(t) * a.C + c, y);
    }
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) conv_state_kernel(const ConvArgs a) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 256 + threadIdx.x) * VEC, seq = blockIdx.y, back = a.taps - 1;
  const int t0 = a.seq_cu[seq], n = a.seq_cu[seq + 1] - t0;
  if (c >= a.C || n <= 0) return;
  T* state = state_of<T>(a, seq);
  if (!state) return;
  state += c;
  for (int m = 0; m < back; ++m) {
    const int li = n - back + m;  // entry m holds the input at this place of the slice, or an older one
    float h[VEC];
    if (li >= 0) load_v<VEC>(static_cast<const T*>(a.x) + static_cast<int64_t>(t0 + li) * a.ldx + c, h);
    else load_v<VEC>(state + static_cast<int64_t>(m + n) * a.C, h);
    store_v<VEC>(state + static_cast<int64_t>(m) * a.C, h);
  }
}

// the prompt slices of an aligned bf16 step; false: a number of taps this kernel does not take
bool launch_run(const ConvArgs& a, cudaStream_t stream) {
  const int blocks = ceil_div(a.C, 1024);
  // enough threads for every SM, runs long enough that a run's first loads do not count
  int run = ceil_div(a.prefill_tokens * blocks, 8 * pxl_host::num_sms());
  run = run < 4 ? 4 : run > 64 ? 64 : run;
  const dim3 grid(blocks, ceil_div(a.prefill_tokens, run));
  switch (a.taps) {
    case 1: pxl_host::launch(conv_run_kernel<1>, grid, dim3(128), 0, stream, a, run); return true;
    case 2: pxl_host::launch(conv_run_kernel<2>, grid, dim3(128), 0, stream, a, run); return true;
    case 3: pxl_host::launch(conv_run_kernel<3>, grid, dim3(128), 0, stream, a, run); return true;
    case 4: pxl_host::launch(conv_run_kernel<4>, grid, dim3(128), 0, stream, a, run); return true;
    default: return false;
  }
}

template <typename T, int VEC>
int run_conv(const ConvArgs& a, cudaStream_t stream) {
  int begin = 0;
  if constexpr (VEC == 8 && sizeof(T) == 2) {
    if (a.prefill_tokens > 0 && launch_run(a, stream)) begin = a.prefill_tokens;
  }
  for (; begin < a.T; begin += 65535) {
    const int n = a.T - begin < 65535 ? a.T - begin : 65535;
    pxl_host::launch(conv_token_kernel<T, VEC>, dim3(ceil_div(a.C, 128 * VEC), n), dim3(128), 0, stream, a, begin);
  }
  if (a.taps > 1 && a.prefill_seqs > 0)
    pxl_host::launch(conv_state_kernel<T, VEC>, dim3(ceil_div(a.C, 256 * VEC), a.prefill_seqs), dim3(256), 0, stream, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
}  // namespace

PXL_EXPORT int pxl_short_conv(const void* x, int64_t ldx, int C, int taps, const void* w, const void* bias, void* state,
                              int num_slots, const int* positions, const int* seq_cu, const int* seq_slots, int prefill_seqs,
                              int prefill_tokens, int T, void* out, int is_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (C <= 0 || taps < 1 || (taps > 1 && !state) || prefill_seqs > 65535) return PXL_ERR_INVALID_ARG;
  const ConvArgs a{x, ldx, C, taps, w, bias, state, num_slots, positions, seq_cu, seq_slots, prefill_seqs, prefill_tokens, T, out,
                   status};
  const bool vec = !((C | static_cast<int>(ldx)) & 7) && aligned16(x) && aligned16(w) && aligned16(bias) && aligned16(state) &&
                   aligned16(out);
  if (is_f32) return vec ? run_conv<float, 8>(a, stream) : run_conv<float, 1>(a, stream);
  return vec ? run_conv<pxl::bf16, 8>(a, stream) : run_conv<pxl::bf16, 1>(a, stream);
}
