// Around softmax attention with grouped heads, rows of any size in bf16 or fp32:
//
//  * pxl_conv_qkv_prep: one launch per layer and step turns the packed projection q | k | v into queries and
//    cache rows: short causal convolution per channel (y_t = sum_j w[j] u[t - taps + 1 + j], zeros before the
//    sequence), RMS norm over the whole q row and the whole k row, half-split rotation, and the scatter of k and
//    v into their pages. Heads are padded with zeros to `cols` columns. v is neither normed nor rotated. Without
//    convolution and norms a kernel of its own does the rest, in which no thread waits for another.
//  * pxl_conv_state_update: the last taps - 1 projected rows of every prompt slice become the state of its slot
//    (a launch of its own: the first tokens of the slice read the state that its last tokens replace; a decoded
//    token reads and replaces it in pxl_conv_qkv_prep itself).
//  * pxl_head_qkv_prep: the same hand-over for heads that are normed one by one without weights: half-split rotation (or
//    none), every head of q and k over its root mean square, factors of the queries per head and per position, values mixed
//    with those of another layer, scatter. A few lanes per head, no barrier.
//  * pxl_gated_norm_rows: concatenated heads times silu(gate), then RMS norm over equal parts of the row.
//  * pxl_gated_rows: concatenated heads, optionally RMS-normed together or one by one, times sigmoid(gate) and a factor,
//    into the columns of the output product's operand.
//
// All arithmetic is fp32.
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

struct PrepArgs {
  const void* proj;  // [T, ld]
  int64_t ld;
  int q_off, k_off, v_off;      // first column of each part (k and v absent: G == 0)
  int H, G, dk, dv, cols, rot, taps;
  const void* conv_w;           // [taps, C] over channels q | k | v, or null
  void* conv_state;             // [slots, taps - 1, C]: previous projected values, oldest first
  int num_state_slots;
  const float* q_norm;
  const float* k_norm;
  const float* cos_sin;         // [max_pos, rot]: cos | sin halves
  const int* positions;
  int max_pos;
  const int* seq_cu;            // [seqs + 1] token ranges: prompt slices first, then one token per decoded sequence
  const int* seq_slots;
  int prefill_seqs, prefill_tokens, T;
  const int64_t* slots;         // cache row of every token
  int64_t num_slots;
  int page;
  void* k_cache;                // [blocks, G, page, cols]
  void* v_cache;
  void* q_out;                  // [T, H, cols]
  float eps;
  int* status;
};

// inv * row, rotated; VEC elements of one head from d0, all in one part of the head (rot / 2 is a multiple of VEC)
template <int VEC>
__device__ __forceinline__ void rotated(const float* row, float inv, const float* cs, int dk, int rot, int d0, float (&o)[VEC]) {
  const int half = rot / 2;
  if (d0 >= dk) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    return;
  }
  load_v<VEC>(row + d0, o);
#pragma unroll
  for (int j = 0; j < VEC; ++j) o[j] *= inv;
  if (d0 >= rot) return;
  const bool lower = d0 < half;
  const int f = lower ? d0 : d0 - half;  // pair
  float c[VEC], sn[VEC], other[VEC];
  load_v<VEC>(cs + f, c);
  load_v<VEC>(cs + half + f, sn);
  load_v<VEC>(row + (lower ? d0 + half : f), other);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const float x = other[j] * inv;
    o[j] = lower ? o[j] * c[j] - x * sn[j] : o[j] * c[j] + x * sn[j];
  }
}

// both sums over the block; red holds 64 floats
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  a = warp_reduce_sum(a);
  b = warp_reduce_sum(b);
  if (lane == 0) red[warp] = a, red[32 + warp] = b;
  __syncthreads();
  return make_float2(warp_reduce_sum(lane < nwarps ? red[lane] : 0.f), warp_reduce_sum(lane < nwarps ? red[32 + lane] : 0.f));
}

template <typename T, int VEC>
__global__ void __launch_bounds__(512) conv_qkv_prep_kernel(const PrepArgs a, int begin, int tokens_per_cta) {
  extern __shared__ __align__(16) float row[];  // convolved q | k of one token, times the norm weights
  __shared__ float red[64];
  pdl_wait();
  pdl_launch_dependents();
  const int Cq = a.H * a.dk, Ck = a.G * a.dk, Cv = a.G * a.dv, C = Cq + Ck + Cv;
  const int back = a.conv_w ? a.taps - 1 : 0;
  const T* w = static_cast<const T*>(a.conv_w);
  const int first = begin + blockIdx.x * tokens_per_cta;
  int seq = 0;
  if (first < a.prefill_tokens) {  // last slice that starts at or before the token
    int lo = 0, hi = a.prefill_seqs - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) / 2;
      if (a.seq_cu[mid] <= first) lo = mid;
      else hi = mid - 1;
    }
    seq = lo;
  }
  for (int t = first; t < a.T && t < first + tokens_per_cta; ++t) {
    const bool decoded = t >= a.prefill_tokens;
    if (decoded) seq = a.prefill_seqs + t - a.prefill_tokens;
    else
      while (a.seq_cu[seq + 1] <= t) ++seq;
    const int li = t - a.seq_cu[seq];
    int pos = a.positions[t];
    const T* cur = static_cast<const T*>(a.proj) + static_cast<int64_t>(t) * a.ld;
    T* state = nullptr;
    if (back) {
      const int slot = a.seq_slots[seq];
      if (slot >= 0 && slot < a.num_state_slots) state = static_cast<T*>(a.conv_state) + static_cast<int64_t>(slot) * back * C;
      else if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_INDEX);
    }
    int64_t cslot = a.G ? a.slots[t] : -1;
    if (cslot >= a.num_slots) {
      if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_SLOT);
      cslot = -1;
    }
    const int in_page = cslot >= 0 ? static_cast<int>(static_cast<uint32_t>(cslot) % static_cast<uint32_t>(a.page)) : 0;
    const int64_t blk = cslot >= 0 ? static_cast<uint32_t>(cslot) / static_cast<uint32_t>(a.page) : 0;
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
      const int col = c < Cq ? a.q_off + c : c < Cq + Ck ? a.k_off + c - Cq : a.v_off + c - Cq - Ck;
      float u[VEC], y[VEC];
      load_v<VEC>(cur + col, u);
      if (w) {
        float wv[VEC];
        load_v<VEC>(w + static_cast<int64_t>(back) * C + c, wv);
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] = wv[j] * u[j];
        for (int b = back; b >= 1; --b) {
          if (pos - b < 0) continue;
          float h[VEC];
          if (b <= li) {
            load_v<VEC>(cur - static_cast<int64_t>(b) * a.ld + col, h);
          } else {
            if (!state) continue;
            load_v<VEC>(state + static_cast<int64_t>(back + li - b) * C + c, h);
          }
          load_v<VEC>(w + static_cast<int64_t>(back - b) * C + c, wv);
#pragma unroll
          for (int j = 0; j < VEC; ++j) y[j] = fmaf(wv[j], h[j], y[j]);
        }
        if (decoded && state) {  // this thread is the only reader and writer of these channels
          for (int m = 0; m + 1 < back; ++m) {
            float h[VEC];
            load_v<VEC>(state + static_cast<int64_t>(m + 1) * C + c, h);
            store_v<VEC>(state + static_cast<int64_t>(m) * C + c, h);
          }
          store_v<VEC>(state + static_cast<int64_t>(back - 1) * C + c, u);
        }
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] = u[j];
      }
      if (c < Cq + Ck) {
        float nw[VEC], sum = 0.f;
        load_v<VEC>(c < Cq ? a.q_norm + c : a.k_norm + c - Cq, nw);
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          sum = fmaf(y[j], y[j], sum);
          y[j] *= nw[j];
        }
        (c < Cq ? sq : sk) += sum;
        store_v<VEC>(row + c, y);
      } else if (cslot >= 0) {
        const int vc = c - Cq - Ck, g = vc / a.dv;
        store_v<VEC>(static_cast<T*>(a.v_cache) + ((blk * a.G + g) * a.page + in_page) * a.cols + vc % a.dv, y);
      }
    }
    const float2 sums = block_sum2(sq, sk, red);  // (its barrier also publishes the row)
    if (pos < 0 || pos >= a.max_pos) {
      if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_POSITION);
      pos = 0;
    }
    const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
    const float inv_q = 1.f / sqrtf(sums.x / Cq + a.eps), inv_k = a.G ? 1.f / sqrtf(sums.y / Ck + a.eps) : 0.f;
    const int per = a.cols / VEC;
    for (int i = threadIdx.x; i < (a.H + a.G) * per; i += blockDim.x) {
      const int h = i / per, d0 = i % per * VEC;
      float o[VEC];
      if (h < a.H) {
        rotated<VEC>(row + h * a.dk, inv_q, cs, a.dk, a.rot, d0, o);
        store_v<VEC>(static_cast<T*>(a.q_out) + (static_cast<int64_t>(t) * a.H + h) * a.cols + d0, o);
      } else if (cslot >= 0) {
        const int g = h - a.H;
        rotated<VEC>(row + Cq + g * a.dk, inv_k, cs, a.dk, a.rot, d0, o);
        store_v<VEC>(static_cast<T*>(a.k_cache) + ((blk * a.G + g) * a.page + in_page) * a.cols + d0, o);
        if (d0 + VEC > a.dv) {  // zero columns behind the value
          T* v = static_cast<T*>(a.v_cache) + ((blk * a.G + g) * a.page + in_page) * a.cols;
          for (int d = d0 > a.dv ? d0 : a.dv; d < d0 + VEC; ++d) put(v + d, 0.f);
        }
      }
    }
    __syncthreads();  // the next token overwrites the row
  }
}

// Prompt slices in bf16: a thread keeps its NV vectors of 8 channels for a run of tokens - weights, norm weights and
// the last TAPS - 1 inputs stay in registers, one load per token and vector - and the next token's input is on its way
// while this one is normed, rotated and stored.
constexpr int run_threads(int nv) { return nv == 1 ? 768 : nv == 2 ? 512 : 448; }  // what the registers allow
template <int TAPS, int NV>
__global__ void __launch_bounds__(run_threads(NV)) conv_qkv_prep_run_kernel(const PrepArgs a, int run) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[64];
  pdl_wait();
  pdl_launch_dependents();
  const int Cq = a.H * a.dk, Ck = a.G * a.dk, C = Cq + Ck + a.G * a.dv;
  constexpr int kBack = TAPS - 1;
  const bf16* w = static_cast<const bf16*>(a.conv_w);
  const int first = blockIdx.x * run, last = first + run < a.prefill_tokens ? first + run : a.prefill_tokens;
  int seq = 0;
  {
    int lo = 0, hi = a.prefill_seqs - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) / 2;
      if (a.seq_cu[mid] <= first) lo = mid;
      else hi = mid - 1;
    }
    seq = lo;
  }
  const bf16x8 zero8 = {{0u, 0u, 0u, 0u}};
  int col[NV], ch[NV], v_off[NV];  // column of proj, channel, place in a token's value rows (values only)
  bf16x8 wt[NV][TAPS], hist[NV][kBack > 0 ? kBack : 1], next[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    ch[i] = c;
    col[i] = c < Cq ? a.q_off + c : c < Cq + Ck ? a.k_off + c - Cq : a.v_off + c - Cq - Ck;
    const int vc = c - Cq - Ck;
    v_off[i] = vc >= 0 && c < C ? vc / a.dv * a.page * a.cols + vc % a.dv : 0;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wt[i][j] = c < C ? ld_bf16x8(w + static_cast<int64_t>(j) * C + c) : zero8;
    next[i] = c < C ? ld_bf16x8(static_cast<const bf16*>(a.proj) + static_cast<int64_t>(first) * a.ld + col[i]) : zero8;
  }
  float* cs = row + Cq + Ck;  // cosines | sines of the token: fetched while it is convolved
  const int per = a.cols / 8, outs = (a.H + a.G) * per;
  for (int t = first; t < last; ++t) {
    while (a.seq_cu[seq + 1] <= t) ++seq;
    const int li = t - a.seq_cu[seq];
    const int pos = a.positions[t];
    const int table_row = pos < 0 || pos >= a.max_pos ? 0 : pos;
    float4 angle;
    if (threadIdx.x * 4 < a.rot)
      angle = *reinterpret_cast<const float4*>(a.cos_sin + static_cast<int64_t>(table_row) * a.rot + threadIdx.x * 4);
    const bf16* cur = static_cast<const bf16*>(a.proj) + static_cast<int64_t>(t) * a.ld;
    if (kBack > 0 && (t == first || li == 0)) {  // the inputs before this run, or of this sequence's earlier steps
      const int slot = a.seq_slots[seq];
      const bool ok = slot >= 0 && slot < a.num_state_slots;
      if (!ok && threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_INDEX);
      const bf16* state = static_cast<const bf16*>(a.conv_state) + static_cast<int64_t>(ok ? slot : 0) * kBack * C;
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int j = 0; j < kBack; ++j) {
          const int b = kBack - j;
          hist[i][j] = zero8;
          if (ch[i] >= C || pos - b < 0) continue;
          if (b <= li) hist[i][j] = ld_bf16x8(cur - static_cast<int64_t>(b) * a.ld + col[i]);
          else if (ok) hist[i][j] = ld_bf16x8(state + static_cast<int64_t>(li + j) * C + ch[i]);
        }
    }
    int64_t cslot = a.G ? a.slots[t] : -1;
    if (cslot >= a.num_slots) {
      if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_SLOT);
      cslot = -1;
    }
    const uint32_t us = cslot >= 0 ? static_cast<uint32_t>(cslot) : 0u, page = static_cast<uint32_t>(a.page);
    // first element of (block, head 0, place in the page); heads are page * cols apart
    const int64_t kv0 = (static_cast<int64_t>(us / page) * a.G * a.page + us % page) * a.cols;
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (ch[i] >= C) continue;
      float y[8] = {};
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const bf16x8& x = j < kBack ? hist[i][j < kBack ? j : 0] : next[i];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 xf = unpack_bf16x2(x.u[e]), wf = unpack_bf16x2(wt[i][j].u[e]);
          y[2 * e] = fmaf(wf.x, xf.x, y[2 * e]);
          y[2 * e + 1] = fmaf(wf.y, xf.y, y[2 * e + 1]);
        }
      }
#pragma unroll
      for (int j = 0; j + 1 < kBack; ++j) hist[i][j] = hist[i][j + 1];
      if constexpr (kBack > 0) hist[i][kBack - 1] = next[i];
      if (t + 1 < last) next[i] = ld_bf16x8(cur + a.ld + col[i]);
      if (ch[i] < Cq + Ck) {
        float nw[8], sum = 0.f;
        load_v<8>(ch[i] < Cq ? a.q_norm + ch[i] : a.k_norm + ch[i] - Cq, nw);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          sum = fmaf(y[e], y[e], sum);
          y[e] *= nw[e];
        }
        (ch[i] < Cq ? sq : sk) += sum;
        store_v<8>(row + ch[i], y);
      } else if (cslot >= 0) {
        store_v<8>(static_cast<bf16*>(a.v_cache) + kv0 + v_off[i], y);
      }
    }
    if (threadIdx.x * 4 < a.rot) *reinterpret_cast<float4*>(cs + threadIdx.x * 4) = angle;
    if (pos != table_row && threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_POSITION);
    const float2 sums = block_sum2(sq, sk, red);
    const float inv_q = 1.f / sqrtf(sums.x / Cq + a.eps), inv_k = a.G ? 1.f / sqrtf(sums.y / Ck + a.eps) : 0.f;
    for (int i = threadIdx.x; i < outs; i += blockDim.x) {
      const int h = i / per, d0 = (i - h * per) * 8;
      float o[8];
      if (h < a.H) {
        rotated<8>(row + h * a.dk, inv_q, cs, a.dk, a.rot, d0, o);
        store_v<8>(static_cast<bf16*>(a.q_out) + (static_cast<int64_t>(t) * a.H + h) * a.cols + d0, o);
      } else if (cslot >= 0) {
        const int g = h - a.H;
        const int64_t at = kv0 + static_cast<int64_t>(g) * a.page * a.cols + d0;
        rotated<8>(row + Cq + g * a.dk, inv_k, cs, a.dk, a.rot, d0, o);
        store_v<8>(static_cast<bf16*>(a.k_cache) + at, o);
        if (d0 >= a.dv) st_bf16x8(static_cast<bf16*>(a.v_cache) + at, zero8);  // zero columns behind the value
      }
    }
    __syncthreads();  // the next token overwrites the row
  }
}

// Neither convolution nor norms: every vector of an output head is made by one thread from the projection.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) rotate_qkv_kernel(const PrepArgs a, int64_t n) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= n) return;
  const int per = a.cols / VEC, heads = a.H + 2 * a.G;
  const int d0 = static_cast<int>(i % per) * VEC, h = static_cast<int>(i / per % heads);
  const int64_t t = i / per / heads;
  int pos = a.positions[t];
  if (pos < 0 || pos >= a.max_pos) {
    if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_POSITION);
    pos = 0;
  }
  const T* row = static_cast<const T*>(a.proj) + t * a.ld;
  const bool value = h >= a.H + a.G;
  const T* src = h < a.H ? row + a.q_off + h * a.dk : value ? row + a.v_off + (h - a.H - a.G) * a.dv : row + a.k_off + (h - a.H) * a.dk;
  const int width = value ? a.dv : a.dk, half = a.rot / 2;
  float o[VEC];
  if (d0 >= width) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
  } else {
    load_v<VEC>(src + d0, o);
    if (!value && d0 < a.rot) {
      const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
      const bool lower = d0 < half;
      const int f = lower ? d0 : d0 - half;
      float c[VEC], sn[VEC], x[VEC];
      load_v<VEC>(cs + f, c);
      load_v<VEC>(cs + half + f, sn);
      load_v<VEC>(src + (lower ? d0 + half : f), x);
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = lower ? o[j] * c[j] - x[j] * sn[j] : o[j] * c[j] + x[j] * sn[j];
    }
  }
  if (h < a.H) {
    store_v<VEC>(static_cast<T*>(a.q_out) + (t * a.H + h) * a.cols + d0, o);
    return;
  }
  const int64_t slot = a.slots[t];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_SLOT);
    return;
  }
  const uint32_t us = static_cast<uint32_t>(slot), page = static_cast<uint32_t>(a.page);
  const int g = value ? h - a.H - a.G : h - a.H;
  T* pages = static_cast<T*>(value ? a.v_cache : a.k_cache);
  store_v<VEC>(pages + ((static_cast<int64_t>(us / page) * a.G + g) * a.page + us % page) * a.cols + d0, o);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) conv_state_update_kernel(const PrepArgs a) {
  pdl_wait();
  pdl_launch_dependents();
  const int Cq = a.H * a.dk, Ck = a.G * a.dk, C = Cq + Ck + a.G * a.dv, back = a.taps - 1;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC, seq = blockIdx.y;
  if (c >= C) return;
  const int t0 = a.seq_cu[seq], n = a.seq_cu[seq + 1] - t0, slot = a.seq_slots[seq];
  if (n <= 0) return;
  if (slot < 0 || slot >= a.num_state_slots) {
    if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_INDEX);
    return;
  }
  const int col = c < Cq ? a.q_off + c : c < Cq + Ck ? a.k_off + c - Cq : a.v_off + c - Cq - Ck;
  T* state = static_cast<T*>(a.conv_state) + static_cast<int64_t>(slot) * back * C + c;
  for (int m = 0; m < back; ++m) {
    const int li = n - back + m;  // entry m holds the value at this place of the slice, or an older one
    float h[VEC];
    if (li >= 0) load_v<VEC>(static_cast<const T*>(a.proj) + static_cast<int64_t>(t0 + li) * a.ld + col, h);
    else load_v<VEC>(state + static_cast<int64_t>(m + n) * C, h);
    store_v<VEC>(state + static_cast<int64_t>(m) * C, h);
  }
}

struct HeadPrepArgs {
  const void* proj;  // [T, ld]
  int64_t ld;
  int q_off, k_off, v_off, H, G, dk, dv, cols, rot;
  float eps;
  const float* cos_sin;     // [max_pos, rot], or null
  const float* pos_scale;   // [max_pos], or null
  const float* head_scale;  // [H], or null
  const int* positions;
  int max_pos;
  const void* v_first;      // [T, ldf], or null
  int64_t ldf;
  float v_mix;
  const int64_t* slots;
  int64_t num_slots;
  int page;
  void* k_cache;  // [blocks, G, page, cols]
  void* v_cache;
  void* q_out;    // [T, H, cols]
  int* status;
};

// LANES neighbouring threads make one head of one token (query heads, key heads, value heads)
template <typename T, int VEC, int LANES>
__global__ void __launch_bounds__(256) head_prep_kernel(const HeadPrepArgs a, int64_t items) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x % LANES;
  int64_t i = static_cast<int64_t>(blockIdx.x) * (256 / LANES) + threadIdx.x / LANES;
  const bool live = i < items;
  if (!live) i = items - 1;  // (takes part in the shuffles)
  const int heads = a.H + 2 * a.G, h = static_cast<int>(i % heads);
  const int64_t t = i / heads;
  const bool query = h < a.H, value = h >= a.H + a.G;
  const int g = value ? h - a.H - a.G : h - a.H;
  const T* row = static_cast<const T*>(a.proj) + t * a.ld;
  const T* src = query ? row + a.q_off + h * a.dk : value ? row + a.v_off + g * a.dv : row + a.k_off + g * a.dk;
  const int width = value ? a.dv : a.dk, half = a.rot / 2;
  float factor = 1.f;
  int pos = a.positions[t];
  if (!value) {
    float sq = 0.f;
    for (int d0 = lane * VEC; d0 < width; d0 += LANES * VEC) {
      float v[VEC];
      load_v<VEC>(src + d0, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) sq = fmaf(v[j], v[j], sq);
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    factor = 1.f / sqrtf(sq / width + a.eps);  // (a rotation leaves the norm alone)
    if ((a.cos_sin || a.pos_scale) && (pos < 0 || pos >= a.max_pos)) {
      if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_POSITION);
      pos = 0;
    }
    if (query && a.head_scale) factor *= a.head_scale[h];
    if (query && a.pos_scale) factor *= a.pos_scale[pos];
  }
  T* dst = nullptr;
  if (query) {
    dst = static_cast<T*>(a.q_out) + (t * a.H + h) * a.cols;
  } else {
    const int64_t slot = a.slots[t];
    if (slot >= a.num_slots) {
      if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_SLOT);
    } else if (slot >= 0) {
      const uint32_t us = static_cast<uint32_t>(slot), page = static_cast<uint32_t>(a.page);
      dst = static_cast<T*>(value ? a.v_cache : a.k_cache) +
            ((static_cast<int64_t>(us / page) * a.G + g) * a.page + us % page) * a.cols;
    }
  }
  if (!live || dst == nullptr) return;
  const T* first = value && a.v_first ? static_cast<const T*>(a.v_first) + t * a.ldf + g * a.dv : nullptr;
  const float* cs = a.cos_sin ? a.cos_sin + static_cast<int64_t>(pos) * a.rot : nullptr;
  for (int d0 = lane * VEC; d0 < a.cols; d0 += LANES * VEC) {
    float o[VEC];
    if (d0 >= width) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    } else {
      load_v<VEC>(src + d0, o);
      if (first) {
        float f[VEC];
        load_v<VEC>(first + d0, f);
#pragma unroll
        for (int j = 0; j < VEC; ++j) o[j] = fmaf(a.v_mix, f[j], (1.f - a.v_mix) * o[j]);
      } else if (!value) {
        if (d0 < a.rot) {
          const bool lower = d0 < half;
          const int f = lower ? d0 : d0 - half;
          float c[VEC], sn[VEC], x[VEC];
          load_v<VEC>(cs + f, c);
          load_v<VEC>(cs + half + f, sn);
          load_v<VEC>(src + (lower ? d0 + half : f), x);
#pragma unroll
          for (int j = 0; j < VEC; ++j) o[j] = lower ? o[j] * c[j] - x[j] * sn[j] : o[j] * c[j] + x[j] * sn[j];
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) o[j] *= factor;
      }
    }
    store_v<VEC>(dst + d0, o);
  }
}

// x [T, n] (the heads of a token) times silu(gate), RMS norm over `groups` equal parts, times w
struct GatedNormArgs {
  const void* x;
  const void* gate;  // [T, ldg]
  int64_t ldg;
  const float* w;
  int n, groups;
  float eps;
  void* out;  // [T, ldo], out_cols columns: n, then zeros
  int64_t ldo;
  int out_cols;
};

template <typename T, int VEC>
__device__ __forceinline__ void gated_vector(const T* x, const T* g, float (&v)[VEC]) {
  float z[VEC];
  load_v<VEC>(x, v);
  load_v<VEC>(g, z);
#pragma unroll
  for (int j = 0; j < VEC; ++j) v[j] *= z[j] / (1.f + expf(-z[j]));
}

// eight warps: several per part, or several parts one after the other for a warp
template <typename T, int VEC>
__global__ void __launch_bounds__(256) gated_norm_rows_kernel(const GatedNormArgs a) {
  __shared__ float sums[8];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const T* x = static_cast<const T*>(a.x) + t * a.n;
  const T* gate = static_cast<const T*>(a.gate) + t * a.ldg;
  T* out = static_cast<T*>(a.out) + t * a.ldo;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int share = a.groups >= 8 ? 1 : a.groups >= 4 ? 2 : a.groups >= 2 ? 4 : 8;  // warps per part
  const int per = a.n / a.groups, sub = warp % share;
  for (int g0 = 0; g0 < a.groups; g0 += 8 / share) {
    const int g = g0 + warp / share;
    const bool mine = g < a.groups;
    float sq = 0.f;
    for (int c = (sub * 32 + lane) * VEC; mine && c < per; c += share * 32 * VEC) {
      float v[VEC];
      gated_vector<T, VEC>(x + g * per + c, gate + g * per + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) sq = fmaf(v[j], v[j], sq);
    }
    sq = warp_reduce_sum(sq);
    if (lane == 0) sums[warp] = sq;
    __syncthreads();
    float sum = 0.f;
    for (int i = 0; i < share; ++i) sum += sums[warp / share * share + i];
    __syncthreads();
    const float inv = 1.f / sqrtf(sum / per + a.eps);
    for (int c = (sub * 32 + lane) * VEC; mine && c < per; c += share * 32 * VEC) {
      float v[VEC], w[VEC];
      gated_vector<T, VEC>(x + g * per + c, gate + g * per + c, v);
      load_v<VEC>(a.w + g * per + c, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= inv * w[j];
      store_v<VEC>(out + g * per + c, v);
    }
  }
  for (int c = a.n + threadIdx.x; c < a.out_cols; c += blockDim.x) put(out + c, 0.f);
}

struct GateArgs {
  const void* x;        // [T, heads, x_cols]
  int heads, x_cols, dv;
  const void* gate;     // [T, ldg], heads * dv columns
  int64_t ldg;
  const float* norm_w;  // [heads * dv] or null
  float eps, scale;
  int per_head;         // the norm's statistics are those of one head
  void* out;            // [T, ldo], out_cols columns: heads * dv, then zeros
  int64_t ldo;
  int out_cols;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(256) gated_rows_kernel(const GateArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const int N = a.heads * a.dv;
  const T* x = static_cast<const T*>(a.x) + t * a.heads * a.x_cols;
  const T* g = static_cast<const T*>(a.gate) + t * a.ldg;
  T* out = static_cast<T*>(a.out) + t * a.ldo;
  float inv = 1.f;
  extern __shared__ float head_inv[];  // per_head: [heads]
  if (a.norm_w && a.per_head) {
    const int lane = threadIdx.x & 31;
    for (int h = threadIdx.x >> 5; h < a.heads; h += blockDim.x >> 5) {  // one warp per head
      float sq = 0.f;
      for (int c = lane * VEC; c < a.dv; c += 32 * VEC) {
        float v[VEC];
        load_v<VEC>(x + static_cast<int64_t>(h) * a.x_cols + c, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) sq = fmaf(v[j], v[j], sq);
      }
      sq = warp_reduce_sum(sq);
      if (lane == 0) head_inv[h] = 1.f / sqrtf(sq / a.dv + a.eps);
    }
    __syncthreads();
  } else if (a.norm_w) {
    float sq = 0.f;
    for (int c = threadIdx.x * VEC; c < N; c += blockDim.x * VEC) {
      float v[VEC];
      load_v<VEC>(x + c / a.dv * a.x_cols + c % a.dv, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) sq = fmaf(v[j], v[j], sq);
    }
    inv = 1.f / sqrtf(block_reduce_sum(sq, red) / N + a.eps);
  }
  for (int c = threadIdx.x * VEC; c < N; c += blockDim.x * VEC) {
    float v[VEC], gv[VEC];
    load_v<VEC>(x + c / a.dv * a.x_cols + c % a.dv, v);
    load_v<VEC>(g + c, gv);
    if (a.norm_w) {
      float w[VEC];
      load_v<VEC>(a.norm_w + c, w);
      const float f = a.per_head ? head_inv[c / a.dv] : inv;
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= f * w[j];
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= a.scale / (1.f + expf(-gv[j]));
    store_v<VEC>(out + c, v);
  }
  for (int c = N + threadIdx.x; c < a.out_cols; c += blockDim.x) put(out + c, 0.f);
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename K>
bool opt_in_smem(K kern, size_t smem) {
  return smem <= 48 * 1024 ||
         cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) == cudaSuccess;
}

template <int TAPS, int NV>
bool launch_run(const PrepArgs& a, int threads, size_t smem, cudaStream_t stream) {
  if (!opt_in_smem(conv_qkv_prep_run_kernel<TAPS, NV>, smem)) return false;
  int run = ceil_div(a.prefill_tokens, pxl_host::num_sms());
  if (run < 4) run = 4;
  if (run > 64) run = 64;
  pxl_host::launch(conv_qkv_prep_run_kernel<TAPS, NV>, dim3(ceil_div(a.prefill_tokens, run)), dim3(threads), smem, stream, a, run);
  return true;
}

// the prompt slices of an aligned bf16 step; false: sizes this kernel does not take
bool launch_run(const PrepArgs& a, size_t smem, cudaStream_t stream) {
  const int vecs = (a.H * a.dk + a.G * (a.dk + a.dv)) / 8;
  int nv = 1;
  while (nv <= 3 && vecs > nv * run_threads(nv)) ++nv;
  if (!a.conv_w || nv > 3) return false;
  const int threads = ceil_div(ceil_div(vecs, nv), 32) * 32;
  if (a.rot > 4 * threads) return false;
  smem += sizeof(float) * a.rot;
#define PXL_RUN(N)                                                          \
  case N:                                                                   \
    return nv == 1   ? launch_run<N, 1>(a, threads, smem, stream)           \
           : nv == 2 ? launch_run<N, 2>(a, threads, smem, stream)           \
                     : launch_run<N, 3>(a, threads, smem, stream)
  switch (a.taps) {
    PXL_RUN(1);
    PXL_RUN(2);
    PXL_RUN(3);
    PXL_RUN(4);
    default: return false;
  }
#undef PXL_RUN
}

template <typename T, int VEC>
int launch_prep(const PrepArgs& a, bool update, cudaStream_t stream) {
  if (!a.conv_w && !a.q_norm) {
    const int64_t n = static_cast<int64_t>(a.T) * (a.H + 2 * a.G) * (a.cols / VEC);
    pxl_host::launch(rotate_qkv_kernel<T, VEC>, dim3(static_cast<unsigned>((n + 255) / 256)), dim3(256), 0, stream, a, n);
  } else if (update) {
    const int C = a.H * a.dk + a.G * (a.dk + a.dv);
    pxl_host::launch(conv_state_update_kernel<T, VEC>, dim3(ceil_div(C, 256 * VEC), a.prefill_seqs), dim3(256), 0, stream, a);
  } else {
    const size_t smem = sizeof(float) * (a.H + a.G) * a.dk;
    if (smem > 220 * 1024) return PXL_ERR_TOO_LARGE;
    if (!opt_in_smem(conv_qkv_prep_kernel<T, VEC>, smem)) return PXL_ERR_CUDA;
    int begin = 0;
    if constexpr (VEC == 8 && sizeof(T) == 2) {
      if (a.prefill_tokens > 0 && launch_run(a, smem, stream)) begin = a.prefill_tokens;
    }
    if (begin < a.T) {
      // long prompts: neighbours share taps through L1; few tokens: more threads for each
      const int sms = pxl_host::num_sms(), per = a.T - begin >= 16 * sms ? 4 : 1, threads = a.T - begin <= 2 * sms ? 512 : 256;
      pxl_host::launch(conv_qkv_prep_kernel<T, VEC>, dim3(ceil_div(a.T - begin, per)), dim3(threads), smem, stream, a, begin, per);
    }
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

template <typename T>
int dispatch_prep(const PrepArgs& a, bool update, cudaStream_t stream) {
  const bool vec = !((a.q_off | a.k_off | a.v_off | a.dk | a.dv | a.cols | (a.rot / 2) | static_cast<int>(a.ld)) & 7) &&
                   aligned16(a.proj) && aligned16(a.conv_w) && aligned16(a.conv_state) && aligned16(a.k_cache) &&
                   aligned16(a.v_cache) && aligned16(a.q_out) && aligned16(a.q_norm) && aligned16(a.k_norm) &&
                   aligned16(a.cos_sin);
  return vec ? launch_prep<T, 8>(a, update, stream) : launch_prep<T, 1>(a, update, stream);
}

template <typename T, int VEC>
int launch_head_prep(const HeadPrepArgs& a, int T_, cudaStream_t stream) {
  const int64_t items = static_cast<int64_t>(T_) * (a.H + 2 * a.G);
  const int vecs = a.cols / VEC;
  auto grid = [&](int lanes) { return dim3(static_cast<unsigned>((items + 256 / lanes - 1) / (256 / lanes))); };
  if (vecs <= 8) pxl_host::launch(head_prep_kernel<T, VEC, 8>, grid(8), dim3(256), 0, stream, a, items);
  else if (vecs <= 16) pxl_host::launch(head_prep_kernel<T, VEC, 16>, grid(16), dim3(256), 0, stream, a, items);
  else pxl_host::launch(head_prep_kernel<T, VEC, 32>, grid(32), dim3(256), 0, stream, a, items);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

inline bool bad_prep(const PrepArgs& a) {
  return a.H <= 0 || a.G < 0 || a.dk <= 0 || (a.G && a.dv <= 0) || a.cols < a.dk || (a.G && a.cols < a.dv) || a.rot < 0 ||
         a.rot > a.dk || (a.rot & 1) || a.taps < 1 || a.page <= 0 || a.num_slots >= (1ll << 31) || (a.q_norm == nullptr && a.conv_w) ||
         (a.G && (a.q_norm == nullptr) != (a.k_norm == nullptr)) || (a.taps > 1 && a.conv_w && a.conv_state == nullptr);
}
}  // namespace

PXL_EXPORT int pxl_conv_qkv_prep(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int G, int dk, int dv,
                                 int cols, int rot, int taps, const void* conv_w, void* conv_state, int num_state_slots,
                                 const float* q_norm, const float* k_norm, const float* cos_sin, const int* positions,
                                 int max_pos, const int* seq_cu, const int* seq_slots, int prefill_seqs, int prefill_tokens,
                                 int T, const int64_t* slots, int64_t num_slots, int page, void* k_cache, void* v_cache,
                                 void* q_out, float eps, int is_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  PrepArgs a{proj, ld, q_off, k_off, v_off, H, G, dk, dv, cols, rot, taps, conv_w, conv_state, num_state_slots, q_norm, k_norm,
             cos_sin, positions, max_pos, seq_cu, seq_slots, prefill_seqs, prefill_tokens, T, slots, num_slots, page, k_cache,
             v_cache, q_out, eps, status};
  if (bad_prep(a)) return PXL_ERR_INVALID_ARG;
  int code = is_f32 ? dispatch_prep<float>(a, false, stream) : dispatch_prep<pxl::bf16>(a, false, stream);
  if (code == PXL_OK && conv_w && taps > 1 && prefill_seqs > 0)
    code = is_f32 ? dispatch_prep<float>(a, true, stream) : dispatch_prep<pxl::bf16>(a, true, stream);
  return code;
}

PXL_EXPORT int pxl_gated_rows(const void* x, int heads, int x_cols, int dv, const void* gate, int64_t ldg,
                              const float* norm_w, float eps, int per_head, float scale, void* out, int64_t ldo, int out_cols,
                              int T, int is_f32, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  const size_t smem = norm_w && per_head ? sizeof(float) * heads : 0;
  if (smem > 40 * 1024) return PXL_ERR_TOO_LARGE;
  if (heads <= 0 || dv <= 0 || x_cols < dv || out_cols < heads * dv) return PXL_ERR_INVALID_ARG;
  const GateArgs a{x, heads, x_cols, dv, gate, ldg, norm_w, eps, scale, per_head, out, ldo, out_cols};
  const bool vec = !((x_cols | dv | static_cast<int>(ldg) | static_cast<int>(ldo)) & 7) && aligned16(x) && aligned16(gate) &&
                   aligned16(out) && aligned16(norm_w);
  if (is_f32) {
    if (vec) pxl_host::launch(gated_rows_kernel<float, 8>, dim3(T), dim3(256), smem, stream, a);
    else pxl_host::launch(gated_rows_kernel<float, 1>, dim3(T), dim3(256), smem, stream, a);
  } else {
    if (vec) pxl_host::launch(gated_rows_kernel<pxl::bf16, 8>, dim3(T), dim3(256), smem, stream, a);
    else pxl_host::launch(gated_rows_kernel<pxl::bf16, 1>, dim3(T), dim3(256), smem, stream, a);
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

PXL_EXPORT int pxl_head_qkv_prep(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int G, int dk, int dv,
                                 int cols, int rot, float eps, const float* cos_sin, const float* pos_scale,
                                 const float* head_scale, const int* positions, int max_pos, const void* v_first, int64_t ldf,
                                 float v_mix, const int64_t* slots, int64_t num_slots, int page, void* k_cache, void* v_cache,
                                 void* q_out, int T, int is_f32, int* status, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (H <= 0 || G <= 0 || dk <= 0 || dv <= 0 || cols < dk || cols < dv || rot < 0 || rot > dk || (rot & 1) || page <= 0 ||
      num_slots >= (1ll << 31) || (rot && !cos_sin))
    return PXL_ERR_INVALID_ARG;
  const HeadPrepArgs a{proj, ld, q_off, k_off, v_off, H, G, dk, dv, cols, rot, eps, rot ? cos_sin : nullptr, pos_scale, head_scale,
                       positions, max_pos, v_first, ldf, v_mix, slots, num_slots, page, k_cache, v_cache, q_out, status};
  const bool vec = !((q_off | k_off | v_off | dk | dv | cols | (rot / 2) | static_cast<int>(ld) | static_cast<int>(ldf)) & 7) &&
                   aligned16(proj) && aligned16(v_first) && aligned16(k_cache) && aligned16(v_cache) && aligned16(q_out) &&
                   aligned16(cos_sin);
  if (is_f32) return vec ? launch_head_prep<float, 8>(a, T, stream) : launch_head_prep<float, 1>(a, T, stream);
  return vec ? launch_head_prep<pxl::bf16, 8>(a, T, stream) : launch_head_prep<pxl::bf16, 1>(a, T, stream);
}

PXL_EXPORT int pxl_gated_norm_rows(const void* x, int n, const void* gate, int64_t ldg, const float* w, int groups, float eps,
                                   void* out, int64_t ldo, int out_cols, int T, int is_f32, cudaStream_t stream) {
  if (T <= 0) return PXL_OK;
  if (n <= 0 || groups <= 0 || n % groups || out_cols < n) return PXL_ERR_INVALID_ARG;
  const GatedNormArgs a{x, gate, ldg, w, n, groups, eps, out, ldo, out_cols};
  const bool vec = !((n | (n / groups) | static_cast<int>(ldg) | static_cast<int>(ldo)) & 7) && aligned16(x) && aligned16(gate) &&
                   aligned16(out) && aligned16(w);
  if (is_f32) {
    if (vec) pxl_host::launch(gated_norm_rows_kernel<float, 8>, dim3(T), dim3(256), 0, stream, a);
    else pxl_host::launch(gated_norm_rows_kernel<float, 1>, dim3(T), dim3(256), 0, stream, a);
  } else {
    if (vec) pxl_host::launch(gated_norm_rows_kernel<pxl::bf16, 8>, dim3(T), dim3(256), 0, stream, a);
    else pxl_host::launch(gated_norm_rows_kernel<pxl::bf16, 1>, dim3(T), dim3(256), 0, stream, a);
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
