// Linear attention over a matrix state whose decay and input weight are gates of the token, in two forms.
//
// Matrix memory (mLSTM), per head, in fp32,
//
//   i = cap tanh((gi + bi) / cap)   f = log sigmoid(cap tanh((gf + bf) / cap))   (logarithms)
//   m' = max(f + m, i)              S' = e^(f + m - m') S + e^(i - m') k v^T     n' = e^(f + m - m') n + e^(i - m') k
//   o  = S'^T q / (max(|n' . q|, e^-m') + 1e-6),                                 q scaled by dk^-1/2
//
// State space (Mamba-2, kSpace), with q = C and k = B shared by the heads of a group,
//
//   d = softplus(dt + bias)   S' = e^(-a d) S + d k v^T   o = S'^T q + D v,      a = e^A_log
//
// whose state slot is S [dk, dv] alone. In the chunked kernel it is the case m_0 = 0, M_t = -F_t with F_t = -a times the sum
// of d, a_j = ln d_j - F_j, without a normaliser.
//
// State slots of the matrix memory [slots, H, words] fp32: S [dk, dv], then for every slice of 32 columns of v a copy of n
// [dk], then the slices' copies of m (all equal). A CTA owns whole slices with their copies, so the CTAs of a head never
// wait for one another and none reads what another one writes. A sequence whose first token of this step sits at position 0
// starts from zero (m too). Two kernels share the state:
//
//  * recurrent: one CTA per (head, 32 or 128 columns of v, sequence) keeps its part of S in registers and walks the
//    sequence's tokens. Decoding (one pass over the state per token, memory bound), fp32, odd sizes.
//  * chunked (bf16 prompts): 64 tokens at a time on the tensor cores. With F_t = sum of f over the chunk up to t,
//    a_j = i_j - F_j and M_t = max(m_0, a_0 .. a_t), m_t is F_t + M_t and F drops out of every weight:
//        S'_t^T q = e^(m_0 - M_t) S_0^T q + sum_(j<=t) e^(a_j - M_t) (q . k_j) v_j
//        S_end    = e^(m_0 - M_n) S_0 + sum_j k_j (e^(a_j - M_n) v_j)^T
//    and the same with v = 1 for n: one more column of v, of S and of the products. Every weight is at most 1. The state
//    is accumulated in fp32 registers; operands that are not bf16 to begin with (weighted scores, weighted values, the
//    state) enter the products as a sum of two bf16 numbers, so their rounding is 2^-17, not 2^-9. One warp prepares the
//    next chunk's gates while the others compute.
//
// This file is compiled without fast math: what enters the recurrence uses the accurate functions.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

constexpr int kSlice = 32;  // columns of v that share a copy of n and m
constexpr float kLog2E = 1.4426950408889634f;
constexpr float kTiny = 1e-6f;

struct MemoryArgs {
  const void* proj;  // [T, ld]
  int64_t ld;
  int q_off, k_off, v_off, H, dk, dv;
  const float* gates;  // [T, ldg]: H input gates, H forget gates
  int64_t ldg;
  const float* bias;  // [2 H]
  float cap, scale;
  float* state;  // [slots, H, words]
  int64_t words;
  int num_slots;
  const int* seq_cu;
  const int* seq_slots;
  const int* positions;
  void* out;  // [T, ldo]: heads side by side
  int64_t ldo;
  int* status;
  int rep = 1;                  // heads that share q and k
  const float* A_log = nullptr;  // kSpace: [H]
  const float* D = nullptr;      // kSpace: [H]
};

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// state of (sequence, head), or null for a slot outside the pool (the status word is set)
__device__ __forceinline__ float* state_of(const MemoryArgs& a, int seq, int h) {
  const int slot = a.seq_slots[seq];
  if (slot < 0 || slot >= a.num_slots) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_INDEX);
    return nullptr;
  }
  return a.state + (static_cast<int64_t>(slot) * a.H + h) * a.words;
}

// ---- recurrent ---------------------------------------------------------------------------------------------
// 256 threads = 256 / CL row lanes x CL column lanes of VW columns (CL < 32: narrow states, kSpace only); R rows of S per
// thread in registers (R == 0: the state stays in global memory, any dk).
template <typename T, int VW, int R, bool kSpace, int CL = 32>
__global__ void __launch_bounds__(256) memory_recurrent_kernel(const MemoryArgs a, int seq0) {
  extern __shared__ float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.x, seq = seq0 + blockIdx.z;
  static_assert(CL == 32 || kSpace, "the normaliser is summed warp by warp");
  constexpr int RL = 256 / CL;
  const int cl = threadIdx.x % CL, rl = threadIdx.x / CL;
  const int c0 = (blockIdx.y * CL + cl) * VW;
  const int t0 = a.seq_cu[seq], t1 = a.seq_cu[seq + 1];
  if (t1 <= t0) return;
  float* Sg = state_of(a, seq, h);
  if (Sg == nullptr) return;
  const bool fresh = a.positions[t0] == 0, live = c0 < a.dv;
  float* qs = sm;              // [dk]
  float* ks = qs + a.dk;       // [dk], times the input weight
  float* ns = ks + a.dk;       // [dk], every entry kept by one thread
  float* dens = ns + a.dk;     // [8] partial n . q
  float* red = dens + 8;       // [RL][CL * VW]
  const int slices = ceil_div(a.dv, kSlice), slice0 = blockIdx.y * VW, own = min(VW, slices - slice0);
  float* ng = Sg + static_cast<int64_t>(a.dk) * a.dv + static_cast<int64_t>(slice0) * a.dk;
  float* mg = Sg + static_cast<int64_t>(a.dk) * a.dv + static_cast<int64_t>(slices) * a.dk + slice0;
  float m = fresh || kSpace ? 0.f : *mg;
  const bool owns_n = !kSpace && threadIdx.x < a.dk;  // (stored below, so that the loads of S do not wait for it)
  const float n_first = owns_n && !fresh ? ng[threadIdx.x] : 0.f;
  constexpr int RR = R > 0 ? R : 1;
  float S[RR][VW];
  auto load_row = [&](int r, float (&s)[VW]) {
    if constexpr (VW == 4) {
      const float4 v = *reinterpret_cast<const float4*>(Sg + static_cast<int64_t>(r) * a.dv + c0);
      s[0] = v.x, s[1] = v.y, s[2] = v.z, s[3] = v.w;
    } else {
      s[0] = Sg[static_cast<int64_t>(r) * a.dv + c0];
    }
  };
  auto store_row = [&](int r, const float (&s)[VW]) {
    if constexpr (VW == 4) *reinterpret_cast<float4*>(Sg + static_cast<int64_t>(r) * a.dv + c0) = make_float4(s[0], s[1], s[2], s[3]);
    else Sg[static_cast<int64_t>(r) * a.dv + c0] = s[0];
  };
  if constexpr (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rl + RL * i;
      if (!fresh && live && r < a.dk) {
        load_row(r, S[i]);
      } else {
#pragma unroll
        for (int c = 0; c < VW; ++c) S[i][c] = 0.f;
      }
    }
  } else if (fresh && live) {
    const float zero[VW] = {};
    for (int r = rl; r < a.dk; r += RL) store_row(r, zero);
  }
  if (owns_n) ns[threadIdx.x] = n_first;
  if constexpr (!kSpace)
    for (int i = threadIdx.x + 256; i < a.dk; i += 256) ns[i] = fresh ? 0.f : ng[i];
  const int hq = h / a.rep;
  float rate = 0.f, skip = 0.f;
  if constexpr (kSpace) rate = expf(a.A_log[h]), skip = a.D[h];
  for (int t = t0; t < t1; ++t) {
    const T* row = static_cast<const T*>(a.proj) + static_cast<int64_t>(t) * a.ld;
    const float* g = a.gates + static_cast<int64_t>(t) * a.ldg;
    float keep, take;
    if constexpr (kSpace) {
      take = softplus(g[h] + a.bias[h]);
      keep = expf(-rate * take);
    } else {
      const float li = soft_cap(g[h] + a.bias[h], a.cap);
      const float lf = log_sigmoid(soft_cap(g[a.H + h] + a.bias[a.H + h], a.cap));
      const float top = fmaxf(lf + m, li);
      keep = expf(lf + m - top), take = expf(li - top);
      m = top;
    }
    float dot = 0.f;
    for (int i = threadIdx.x; i < a.dk; i += 256) {
      const float q = to_f(row[a.q_off + hq * a.dk + i]) * a.scale, k = to_f(row[a.k_off + hq * a.dk + i]) * take;
      qs[i] = q, ks[i] = k;
      if constexpr (!kSpace) {
        const float n = fmaf(keep, ns[i], k);
        ns[i] = n;
        dot = fmaf(n, q, dot);
      }
    }
    if constexpr (!kSpace) {
      dot = warp_reduce_sum(dot);
      if (cl == 0) dens[rl] = dot;
    }
    float v[VW], o[VW];
#pragma unroll
    for (int c = 0; c < VW; ++c) {
      v[c] = live ? to_f(row[a.v_off + h * a.dv + c0 + c]) : 0.f;
      o[c] = 0.f;
    }
    __syncthreads();
    float den = 0.f;
    if constexpr (!kSpace) {
#pragma unroll
      for (int w = 0; w < 8; ++w) den += dens[w];
    }
    if constexpr (R > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = rl + RL * i;
        if (r < a.dk) {
          const float k = ks[r], q = qs[r];
#pragma unroll
          for (int c = 0; c < VW; ++c) {
            S[i][c] = fmaf(k, v[c], keep * S[i][c]);
            o[c] = fmaf(q, S[i][c], o[c]);
          }
        }
      }
    } else if (live) {
      for (int r = rl; r < a.dk; r += RL) {
        float s[VW];
        load_row(r, s);
        const float k = ks[r], q = qs[r];
#pragma unroll
        for (int c = 0; c < VW; ++c) {
          s[c] = fmaf(k, v[c], keep * s[c]);
          o[c] = fmaf(q, s[c], o[c]);
        }
        store_row(r, s);
      }
    }
#pragma unroll
    for (int c = 0; c < VW; ++c) red[(rl * VW + c) * CL + cl] = o[c];
    __syncthreads();
    const float inv = kSpace ? 1.f : 1.f / (fmaxf(fabsf(den), expf(-m)) + kTiny);
    for (int i = threadIdx.x; i < CL * VW; i += 256) {  // column i of this CTA's slices
      const int col = blockIdx.y * CL * VW + i;
      if (col < a.dv) {
        float sum = 0.f;
#pragma unroll
        for (int r = 0; r < RL; ++r) sum += red[(r * VW + i % VW) * CL + i / VW];
        if constexpr (kSpace) sum = fmaf(skip, to_f(row[a.v_off + h * a.dv + col]), sum);
        put(static_cast<T*>(a.out) + static_cast<int64_t>(t) * a.ldo + h * a.dv + col, sum * inv);
      }
    }
  }
  if constexpr (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rl + RL * i;
      if (live && r < a.dk) store_row(r, S[i]);
    }
  }
  if constexpr (!kSpace) {
    for (int i = threadIdx.x; i < a.dk; i += 256)
      for (int s = 0; s < own; ++s) ng[static_cast<int64_t>(s) * a.dk + i] = ns[i];
    if (threadIdx.x < own) mg[threadIdx.x] = m;  // (every thread has read m before the first barrier)
  }
}

template <bool kSpace, typename T, int VW, int CL>
int launch_recurrent(const MemoryArgs& a, int seq0, int n, cudaStream_t stream) {
  constexpr int RL = 256 / CL;
  const dim3 grid(a.H, ceil_div(a.dv, CL * VW), n);
  const size_t smem = sizeof(float) * (3 * a.dk + 8 + 256 * VW);
  if (smem > 48 * 1024 || n > 65535) return PXL_ERR_TOO_LARGE;
  if (a.dk <= 4 * RL) pxl_host::launch(memory_recurrent_kernel<T, VW, 4, kSpace, CL>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 8 * RL) pxl_host::launch(memory_recurrent_kernel<T, VW, 8, kSpace, CL>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 16 * RL) pxl_host::launch(memory_recurrent_kernel<T, VW, 16, kSpace, CL>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 32 * RL) pxl_host::launch(memory_recurrent_kernel<T, VW, 32, kSpace, CL>, grid, dim3(256), smem, stream, a, seq0);
  else pxl_host::launch(memory_recurrent_kernel<T, VW, 0, kSpace, CL>, grid, dim3(256), smem, stream, a, seq0);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
template <bool kSpace, typename T, int VW>
int launch_recurrent(const MemoryArgs& a, int seq0, int n, cudaStream_t stream) {
  if constexpr (kSpace) {
    if (a.dv <= 8 * VW) return launch_recurrent<kSpace, T, VW, 8>(a, seq0, n, stream);
    if (a.dv <= 16 * VW) return launch_recurrent<kSpace, T, VW, 16>(a, seq0, n, stream);
  }
  return launch_recurrent<kSpace, T, VW, 32>(a, seq0, n, stream);
}
template <bool kSpace, typename T>
int launch_recurrent(const MemoryArgs& a, int seq0, int n, cudaStream_t stream) {
  const bool vec = !((a.dv | static_cast<int>(a.words)) & 3) && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0;
  return vec ? launch_recurrent<kSpace, T, 4>(a, seq0, n, stream) : launch_recurrent<kSpace, T, 1>(a, seq0, n, stream);
}

// ---- chunked -----------------------------------------------------------------------------------------------
constexpr int kChunk = 64;
constexpr int kWarps = 8, kGateWarp = 7;

__device__ __forceinline__ float fast_exp2(float x) {  // 2^x, -inf -> 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 f = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - f.x, b - f.y);
}
__device__ __forceinline__ void mma2(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  const uint32_t b[2] = {b0, b1};
  mma_m16n8k16_bf16(d, a, b);
}

struct ChunkGates {
  float a[kChunk];     // a_j log2(e); -inf past the end
  float M[kChunk];     // M_t log2(e)
  float from0[kChunk]; // e^(m_0 - M_t)
  float into[kChunk];  // e^(a_j - M_n)
  float floor[kChunk]; // e^-m_t
  float all;           // e^(m_0 - M_n)
  float pad[3];        // (16-byte multiples: the arrays are read in pairs)
};

template <int DK>
struct ChunkSmem {
  static constexpr int kQ = DK + 8, kV = kSlice + 8, kP = kChunk + 8;  // row pitches: 16-byte steps fall into distinct banks
  bf16 q[kChunk][kQ], k[kChunk][kQ];
  bf16 v[kChunk][kV], vd_hi[kChunk][kV], vd_lo[kChunk][kV];
  bf16 p_hi[kChunk][kP], p_lo[kChunk][kP];
  bf16 s_hi[DK][kV], s_lo[DK][kV];  // column kSlice: n; zeros behind it
  ChunkGates g[2];
};

// grid (slices of v, heads, sequences). Per chunk: stage q, k, v | scores and S_0^T q | P v, new state.
template <int DK, bool kSpace>
__global__ void __launch_bounds__(kWarps * 32) memory_chunk_kernel(const MemoryArgs a) {
  extern __shared__ __align__(16) uint8_t raw[];
  using Sm = ChunkSmem<DK>;
  Sm& s = *reinterpret_cast<Sm*>(raw);
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kSlice;
  const int t0 = a.seq_cu[seq], n_all = a.seq_cu[seq + 1] - t0;
  if (n_all <= 0) return;
  float* Sg = state_of(a, seq, h);
  if (Sg == nullptr) return;
  float* ng = Sg + static_cast<int64_t>(a.dk) * a.dv + static_cast<int64_t>(blockIdx.x) * a.dk;
  float* mg = Sg + static_cast<int64_t>(a.dk) * a.dv + static_cast<int64_t>(ceil_div(a.dv, kSlice)) * a.dk + blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, hq = h / a.rep;
  const int mi = lane >> 3, r8 = lane & 7;
  const bool fresh = a.positions[t0] == 0;

  // this warp's 16 x 16 tiles of the state and, for some, the 16 rows of n beside them, in the layout of the accumulators
  // (n is column 0 of an 8-column tile)
  constexpr int kTilesK = DK / 16, kTiles = kTilesK * 2, NT = (kTiles + kWarps - 1) / kWarps, NN = (kTilesK + kWarps - 1) / kWarps;
  float S[NT][2][4], N[NN][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int tile = warp + i * kWarps, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = m0 + (lane >> 2) + (e >> 1) * 8, c = v0 + n0 + j * 8 + (lane & 3) * 2 + (e & 1);
        S[i][j][e] = (!fresh && tile < kTiles && r < a.dk && c < a.dv) ? Sg[static_cast<int64_t>(r) * a.dv + c] : 0.f;
      }
    if (!kSpace && i < NN) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = m0 + (lane >> 2) + (e >> 1) * 8;
        N[i][e] = (!fresh && tile < kTilesK && r < a.dk && (lane & 3) == 0 && (e & 1) == 0) ? ng[r] : 0.f;
      }
    }
  }
  auto publish_state = [&]() {
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int tile = warp + i * kWarps, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
      if (tile >= kTiles) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = m0 + (lane >> 2) + e * 8, c = n0 + j * 8 + (lane & 3) * 2;
          uint32_t hi, lo;
          split2(S[i][j][2 * e], S[i][j][2 * e + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(&s.s_hi[r][c]) = hi;
          *reinterpret_cast<uint32_t*>(&s.s_lo[r][c]) = lo;
        }
      if (!kSpace && i < NN && tile < kTilesK) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = m0 + (lane >> 2) + e * 8, c = kSlice + (lane & 3) * 2;
          uint32_t hi, lo;
          split2(N[i < NN ? i : 0][2 * e], N[i < NN ? i : 0][2 * e + 1], hi, lo);  // (zeros in columns 1 to 7)
          *reinterpret_cast<uint32_t*>(&s.s_hi[r][c]) = hi;
          *reinterpret_cast<uint32_t*>(&s.s_lo[r][c]) = lo;
        }
      }
    }
  };
  publish_state();

  // gates of a chunk, by one warp: two neighbouring tokens per lane, prefix sums and maxima across the lanes
  float m = fresh || kSpace ? 0.f : *mg;   // running maximum (natural units) after the chunks prepared so far; used by the gate warp
  float raw_i[2], raw_f[2];      // gates of the chunk that is prepared next
  float rate = 0.f, skip = 0.f;
  if constexpr (kSpace) rate = expf(a.A_log[h]), skip = a.D[h];
  auto fetch_gates = [&](int c0) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = c0 + lane * 2 + u;
      const float* g = a.gates + static_cast<int64_t>(t0 + t) * a.ldg;
      raw_i[u] = t < n_all ? g[h] : 0.f;
      if constexpr (!kSpace) raw_f[u] = t < n_all ? g[a.H + h] : 0.f;
    }
  };
  auto prepare_gates = [&](int c0, ChunkGates& g) {
    float F[2], A[2], M[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const bool in = c0 + lane * 2 + u < n_all;
      if constexpr (kSpace) {
        const float d = softplus(raw_i[u] + a.bias[h]);
        F[u] = in ? -rate * d : 0.f;
        A[u] = in ? logf(d) : -INFINITY;
      } else {
        F[u] = in ? log_sigmoid(soft_cap(raw_f[u] + a.bias[a.H + h], a.cap)) : 0.f;
        A[u] = in ? soft_cap(raw_i[u] + a.bias[h], a.cap) : -INFINITY;
      }
    }
    F[1] += F[0];
    float sum = F[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += x;
    }
    float before = __shfl_up_sync(0xffffffffu, sum, 1);
    if (lane == 0) before = 0.f;
    F[0] += before, F[1] += before;
    A[0] -= F[0], A[1] -= F[1];
    float top = fmaxf(A[0], A[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, top, o);
      if (lane >= o) top = fmaxf(top, x);
    }
    float prev = __shfl_up_sync(0xffffffffu, top, 1);
    if (lane == 0) prev = -INFINITY;
    M[0] = kSpace ? -F[0] : fmaxf(fmaxf(m, prev), A[0]);
    M[1] = kSpace ? -F[1] : fmaxf(M[0], A[1]);
    const float last_M = __shfl_sync(0xffffffffu, M[1], 31), last_F = __shfl_sync(0xffffffffu, F[1], 31);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int j = lane * 2 + u;
      g.a[j] = A[u] * kLog2E;
      g.M[j] = M[u] * kLog2E;
      g.from0[j] = expf(m - M[u]);
      g.into[j] = expf(A[u] - last_M);
      g.floor[j] = expf(-(F[u] + M[u]));
    }
    if (lane == 0) g.all = expf(m - last_M);
    m = kSpace ? 0.f : last_F + last_M;
  };

  // rows of the next chunk travel through registers while this one is computed
  constexpr int kVecQ = kChunk * DK / 8 / (kWarps * 32), kVecV = kChunk * kSlice / 8 / (kWarps * 32);
  bf16x8 rq[kVecQ], rk[kVecQ], rv[kVecV];
  const bf16* base = static_cast<const bf16*>(a.proj) + static_cast<int64_t>(t0) * a.ld;
  const bf16x8 zero8 = {{0u, 0u, 0u, 0u}};
  auto fetch = [&](int c0) {
#pragma unroll
    for (int i = 0; i < kVecQ; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (DK / 8), d = x % (DK / 8) * 8;
      const bool in = c0 + r < n_all && d < a.dk;
      const bf16* p = base + static_cast<int64_t>(c0 + r) * a.ld + hq * a.dk + d;
      rq[i] = in ? ld_bf16x8(p + a.q_off) : zero8;
      rk[i] = in ? ld_bf16x8(p + a.k_off) : zero8;
    }
#pragma unroll
    for (int i = 0; i < kVecV; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (kSlice / 8), d = v0 + x % (kSlice / 8) * 8;
      const bool in = c0 + r < n_all && d < a.dv;
      rv[i] = in ? ld_bf16x8(base + static_cast<int64_t>(c0 + r) * a.ld + a.v_off + h * a.dv + d) : zero8;
    }
  };
  fetch(0);
  if (warp == kGateWarp) {
    fetch_gates(0);
    prepare_gates(0, s.g[0]);
    fetch_gates(kChunk);
  }
  __syncthreads();

  const int rg = warp & 3, ch = warp >> 2;  // 16 query rows; half of the columns of the scores and of v
  const uint32_t ones = lane < 4 ? 0x3f803f80u : 0u;  // B operand whose column 0 is all ones
  int buf = 0;
  for (int c0 = 0; c0 < n_all; c0 += kChunk, buf ^= 1) {
    const int n = n_all - c0 < kChunk ? n_all - c0 : kChunk;
    const ChunkGates& g = s.g[buf];
    // ---- rows into shared memory
#pragma unroll
    for (int i = 0; i < kVecQ; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (DK / 8), d = x % (DK / 8) * 8;
      st_bf16x8(&s.q[r][d], rq[i]);
      st_bf16x8(&s.k[r][d], rk[i]);
    }
#pragma unroll
    for (int i = 0; i < kVecV; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (kSlice / 8), d = x % (kSlice / 8) * 8;
      st_bf16x8(&s.v[r][d], rv[i]);
      const float w = g.into[r];
      bf16x8 hi, lo;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 u = unpack_bf16x2(rv[i].u[j]);
        split2(u.x * w, u.y * w, hi.u[j], lo.u[j]);
      }
      st_bf16x8(&s.vd_hi[r][d], hi);
      st_bf16x8(&s.vd_lo[r][d], lo);
    }
    __syncthreads();
    const bool more = c0 + kChunk < n_all;
    if (more) fetch(c0 + kChunk);

    // ---- scores of 16 rows x 32 columns; S_0^T q for 16 rows x 16 columns, n_0 . q beside them
    const int r_lo = rg * 16 + (lane >> 2);
    float o[3][4] = {};
    {
      float p[4][4] = {};
      const bool needed = ch * 32 <= rg * 16 + 15;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t qa[4], b[4];
        ldmatrix_x4(qa, smem_u32(&s.q[rg * 16 + (mi & 1) * 8 + r8][kk * 16 + (mi >> 1) * 8]));
        if (needed) {
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            ldmatrix_x4(b, smem_u32(&s.k[ch * 32 + u * 16 + (mi >> 1) * 8 + r8][kk * 16 + (mi & 1) * 8]));
            mma2(p[2 * u], qa, b[0], b[1]);
            mma2(p[2 * u + 1], qa, b[2], b[3]);
          }
        }
        ldmatrix_x4_trans(b, smem_u32(&s.s_hi[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
        mma2(o[0], qa, b[0], b[1]);
        mma2(o[1], qa, b[2], b[3]);
        ldmatrix_x4_trans(b, smem_u32(&s.s_lo[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
        mma2(o[0], qa, b[0], b[1]);
        mma2(o[1], qa, b[2], b[3]);
        if constexpr (!kSpace) {
          const bf16* nrow = mi < 2 ? &s.s_hi[kk * 16 + (mi & 1) * 8 + r8][kSlice] : &s.s_lo[kk * 16 + (mi & 1) * 8 + r8][kSlice];
          ldmatrix_x4_trans(b, smem_u32(nrow));
          mma2(o[2], qa, b[0], b[1]);
          mma2(o[2], qa, b[2], b[3]);
        }
      }
      if (needed) {
        const float M[2] = {g.M[r_lo], g.M[r_lo + 8]};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int c = ch * 32 + j * 8 + (lane & 3) * 2;
          const float2 ac = *reinterpret_cast<const float2*>(&g.a[c]);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int r = r_lo + e * 8;
            const float x = c <= r ? p[j][2 * e] * a.scale * fast_exp2(ac.x - M[e]) : 0.f;
            const float y = c + 1 <= r ? p[j][2 * e + 1] * a.scale * fast_exp2(ac.y - M[e]) : 0.f;
            uint32_t hi, lo;
            split2(x, y, hi, lo);
            *reinterpret_cast<uint32_t*>(&s.p_hi[r][c]) = hi;
            *reinterpret_cast<uint32_t*>(&s.p_lo[r][c]) = lo;
          }
        }
      }
    }
    if (more && warp == kGateWarp) {
      prepare_gates(c0 + kChunk, s.g[buf ^ 1]);
      fetch_gates(c0 + 2 * kChunk);
    }
    __syncthreads();

    // ---- o += P v (keys up to this row group), and the state at the chunk's end
    {
      const float w[2] = {g.from0[r_lo] * a.scale, g.from0[r_lo + 8] * a.scale};
#pragma unroll
      for (int j = 0; j < 3; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] *= w[e >> 1];
    }
    for (int kk = 0; kk <= rg; ++kk) {
      uint32_t pa[4], b[4];
      ldmatrix_x4_trans(b, smem_u32(&s.v[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
      ldmatrix_x4(pa, smem_u32(&s.p_hi[rg * 16 + (mi & 1) * 8 + r8][kk * 16 + (mi >> 1) * 8]));
      mma2(o[0], pa, b[0], b[1]);
      mma2(o[1], pa, b[2], b[3]);
      if constexpr (!kSpace) mma2(o[2], pa, ones, ones);
      ldmatrix_x4(pa, smem_u32(&s.p_lo[rg * 16 + (mi & 1) * 8 + r8][kk * 16 + (mi >> 1) * 8]));
      mma2(o[0], pa, b[0], b[1]);
      mma2(o[1], pa, b[2], b[3]);
      if constexpr (!kSpace) mma2(o[2], pa, ones, ones);
    }
    float inv[2] = {1.f, 1.f};
#pragma unroll
    for (int e = 0; e < 2 && !kSpace; ++e) {
      const float den = __shfl_sync(0xffffffffu, o[2][2 * e], lane & ~3);
      inv[e] = 1.f / (fmaxf(fabsf(den), g.floor[r_lo + e * 8]) + kTiny);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = r_lo + e * 8, c = v0 + ch * 16 + j * 8 + (lane & 3) * 2;
        if constexpr (kSpace) {
          const float2 v = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(&s.v[r][c - v0]));
          o[j][2 * e] = fmaf(skip, v.x, o[j][2 * e]);
          o[j][2 * e + 1] = fmaf(skip, v.y, o[j][2 * e + 1]);
        }
        if (r < n && c < a.dv)
          *reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.out) + static_cast<int64_t>(t0 + c0 + r) * a.ldo + h * a.dv + c) =
              pack_bf16x2(o[j][2 * e] * inv[e], o[j][2 * e + 1] * inv[e]);
      }
    const float keep = g.all;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int tile = warp + i * kWarps, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
      if (tile >= kTiles) continue;
      const bool with_n = !kSpace && i < NN && tile < kTilesK;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][j][e] *= keep;
      if (with_n) {
#pragma unroll
        for (int e = 0; e < 4; ++e) N[i < NN ? i : 0][e] *= keep;
      }
#pragma unroll
      for (int kk = 0; kk < kChunk / 16; ++kk) {
        uint32_t ka[4], b[4];
        ldmatrix_x4_trans(ka, smem_u32(&s.k[kk * 16 + (mi >> 1) * 8 + r8][m0 + (mi & 1) * 8]));
        ldmatrix_x4_trans(b, smem_u32(&s.vd_hi[kk * 16 + (mi & 1) * 8 + r8][n0 + (mi >> 1) * 8]));
        mma2(S[i][0], ka, b[0], b[1]);
        mma2(S[i][1], ka, b[2], b[3]);
        ldmatrix_x4_trans(b, smem_u32(&s.vd_lo[kk * 16 + (mi & 1) * 8 + r8][n0 + (mi >> 1) * 8]));
        mma2(S[i][0], ka, b[0], b[1]);
        mma2(S[i][1], ka, b[2], b[3]);
        if (with_n) {
          uint32_t hi[2] = {0u, 0u}, lo[2] = {0u, 0u};
          if (lane < 4) {
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              const float2 w = *reinterpret_cast<const float2*>(&g.into[kk * 16 + u * 8 + lane * 2]);
              split2(w.x, w.y, hi[u], lo[u]);
            }
          }
          mma2(N[i < NN ? i : 0], ka, hi[0], hi[1]);
          mma2(N[i < NN ? i : 0], ka, lo[0], lo[1]);
        }
      }
    }
    publish_state();  // every read of the old state happened before the last barrier
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int tile = warp + i * kWarps, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = m0 + (lane >> 2) + (e >> 1) * 8, c = v0 + n0 + j * 8 + (lane & 3) * 2 + (e & 1);
        if (tile < kTiles && r < a.dk && c < a.dv) Sg[static_cast<int64_t>(r) * a.dv + c] = S[i][j][e];
      }
    if (!kSpace && i < NN && tile < kTilesK && (lane & 3) == 0) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = m0 + (lane >> 2) + e * 8;
        if (r < a.dk) ng[r] = N[i < NN ? i : 0][2 * e];
      }
    }
  }
  if (!kSpace && warp == kGateWarp && lane == 0) *mg = m;
}

template <bool kSpace, int DK>
int launch_chunk(const MemoryArgs& a, int n, cudaStream_t stream) {
  constexpr int smem = sizeof(ChunkSmem<DK>);
  static bool done[64] = {false};
  const int dev = pxl_host::current_device_slot();
  if (!done[dev]) {
    if (cudaFuncSetAttribute(memory_chunk_kernel<DK, kSpace>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return PXL_ERR_CUDA;
    done[dev] = true;
  }
  if (n > 65535) return PXL_ERR_TOO_LARGE;
  pxl_host::launch(memory_chunk_kernel<DK, kSpace>, dim3(ceil_div(a.dv, kSlice), a.H, n), dim3(kWarps * 32), smem, stream, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

inline bool chunkable(const MemoryArgs& a) {
  return a.dk <= 256 && !((a.q_off | a.k_off | a.v_off | a.dk | a.dv | static_cast<int>(a.ld) | static_cast<int>(a.ldo)) & 7) &&
         ((reinterpret_cast<uintptr_t>(a.proj) | reinterpret_cast<uintptr_t>(a.out)) & 15) == 0;
}

template <bool kSpace>
int run(const MemoryArgs& a, int prefill_seqs, int decode_seqs, int is_f32, cudaStream_t stream) {
  int code = PXL_OK;
  if (prefill_seqs > 0) {
    if (is_f32) code = launch_recurrent<kSpace, float>(a, 0, prefill_seqs, stream);
    else if (!chunkable(a)) code = launch_recurrent<kSpace, bf16>(a, 0, prefill_seqs, stream);
    else if (a.dk <= 32) code = launch_chunk<kSpace, 32>(a, prefill_seqs, stream);
    else if (a.dk <= 64) code = launch_chunk<kSpace, 64>(a, prefill_seqs, stream);
    else if (a.dk <= 96) code = launch_chunk<kSpace, 96>(a, prefill_seqs, stream);
    else if (a.dk <= 128) code = launch_chunk<kSpace, 128>(a, prefill_seqs, stream);
    else code = launch_chunk<kSpace, 256>(a, prefill_seqs, stream);
  }
  if (code == PXL_OK && decode_seqs > 0)
    code = is_f32 ? launch_recurrent<kSpace, float>(a, prefill_seqs, decode_seqs, stream)
                  : launch_recurrent<kSpace, bf16>(a, prefill_seqs, decode_seqs, stream);
  return code;
}
}  // namespace

PXL_EXPORT int pxl_matrix_memory(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int dk, int dv,
                                 const float* gates, int64_t ldg, const float* bias, float cap, float* state, int64_t words,
                                 int num_slots, const int* seq_cu, const int* seq_slots, const int* positions, void* out,
                                 int64_t ldo, int prefill_seqs, int decode_seqs, int is_f32, int* status, cudaStream_t stream) {
  if (H <= 0 || dk <= 0 || dv <= 0 || !(cap > 0.f)) return PXL_ERR_INVALID_ARG;
  if (words < static_cast<int64_t>(dk) * dv + static_cast<int64_t>(pxl::ceil_div(dv, kSlice)) * (dk + 1)) return PXL_ERR_INVALID_ARG;
  const MemoryArgs a{proj, ld, q_off, k_off, v_off, H, dk, dv, gates, ldg, bias, cap, 1.f / sqrtf(static_cast<float>(dk)), state,
                     words, num_slots, seq_cu, seq_slots, positions, out, ldo, status};
  return run<false>(a, prefill_seqs, decode_seqs, is_f32, stream);
}

PXL_EXPORT int pxl_state_space(const void* x, int64_t ld, int x_off, int b_off, int c_off, int H, int groups, int n, int dv,
                               const float* dt, int64_t ldt, const float* dt_bias, const float* A_log, const float* D, float* state,
                               int num_slots, const int* seq_cu, const int* seq_slots, const int* positions, void* out, int64_t ldo,
                               int prefill_seqs, int decode_seqs, int is_f32, int* status, cudaStream_t stream) {
  if (H <= 0 || groups <= 0 || H % groups || n <= 0 || dv <= 0) return PXL_ERR_INVALID_ARG;
  const MemoryArgs a{x, ld, c_off, b_off, x_off, H, n, dv, dt, ldt, dt_bias, 1.f, 1.f, state, static_cast<int64_t>(n) * dv,
                     num_slots, seq_cu, seq_slots, positions, out, ldo, status, H / groups, A_log, D};
  return run<true>(a, prefill_seqs, decode_seqs, is_f32, stream);
}
