// Gated delta rule with a decay per head and key channel. Per head, in fp32, with unit vectors q (times dk^-1/2) and k,
//
//   g = exp(-e^A_log softplus(decay + dt_bias))   b = sigmoid(beta)
//   S <- g S (rows)   u = b (v - S^T k)   S <- S + k u^T   o = S^T q
//
// q and k are shared by the heads of a group. State slots [slots, H, dk, dv] fp32; a sequence whose first token of this step
// sits at position 0 starts from zero. Two forms share the state:
//
//  * recurrent: one CTA per (head, 32 or 128 columns of v, sequence) keeps its part of S in registers and walks the tokens;
//    S^T k and S^T q come out of one pass (o = S'^T q + (k . q) u with the decayed S'), one exchange between the warps per
//    token. Decoding (one pass over the state, memory bound), fp32, odd sizes.
//  * chunked (bf16 prompts), two kernels over chunks of 64 tokens. With G_t the sum of log g over the chunk up to t,
//        A_tj = b_t sum_c k_t k_j e^(G_t - G_j)  (j < t)      P_tj = sum_c q_t k_j e^(G_t - G_j)  (j <= t)
//        U = (1 + A)^-1 (b v)    W = (1 + A)^-1 (b k e^G)     u = U - W S_0
//        o = (q e^G) S_0 + P u                                S_end = e^(G_n) S_0 + (k e^(G_n - G))^T u
//    The first kernel makes U, W, P, q e^G and k e^(G_n - G) of every chunk in parallel; the second walks the chunks of a
//    (sequence, head, 32 columns of v) with S in registers. No exponent is ever positive: inside blocks of 8 tokens
//    A and P are summed with the exact differences G_t - G_j; between blocks the factors are split at a border between them
//    (e^(G_t - G_border) on the row, e^(G_border - G_j) on the column) and multiplied on the tensor cores. The triangular
//    system is solved column by column in fp32. Products take operands as sums of two bf16 numbers (rounding 2^-17).
//
// This file is compiled without fast math: what enters the recurrence uses the accurate functions.
#include <type_traits>

#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

constexpr float kUnitEps = 1e-6f;
constexpr float kLog2E = 1.4426950408889634f;

struct DeltaArgs {
  const void* x;  // [T, ld]: q | k | v columns, behind the convolution
  int64_t ld;
  int q_off, k_off, v_off, H, rep, dk, dv;
  const float* decay;  // [T, ldd], H x dk logits
  int64_t ldd;
  const float* dt_bias;  // [H x dk]
  const float* A_log;    // [H]
  const float* beta;     // [T, ldb], H logits
  int64_t ldb;
  float scale;  // dk^-1/2
  float* state;
  int num_slots;
  const int* seq_cu;
  const int* seq_slots;
  const int* positions;
  void* out;  // [T, ldo]: heads side by side
  int64_t ldo;
  int* status;
};

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// state of (sequence, head), or null for a slot outside the pool (the status word is set)
__device__ __forceinline__ float* state_of(const DeltaArgs& a, int seq, int h) {
  const int slot = a.seq_slots[seq];
  if (slot < 0 || slot >= a.num_slots) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_INDEX);
    return nullptr;
  }
  return a.state + (static_cast<int64_t>(slot) * a.H + h) * a.dk * a.dv;
}

// ---- recurrent ---------------------------------------------------------------------------------------------
// 256 threads = 256 / CL row lanes x CL column lanes of VW columns; R rows of S per thread in registers (R == 0: the
// state stays in global memory, any dk).
template <typename T, int VW, int R, int CL>
__global__ void __launch_bounds__(256) delta_recurrent_kernel(const DeltaArgs a, int seq0) {
  extern __shared__ float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.x, seq = seq0 + blockIdx.z, hq = h / a.rep;
  constexpr int RL = 256 / CL;
  const int cl = threadIdx.x % CL, rl = threadIdx.x / CL;
  const int c0 = (blockIdx.y * CL + cl) * VW;
  const int t0 = a.seq_cu[seq], t1 = a.seq_cu[seq + 1];
  if (t1 <= t0) return;
  float* Sg = state_of(a, seq, h);
  if (Sg == nullptr) return;
  const bool fresh = a.positions[t0] == 0, live = c0 < a.dv;
  float* red = sm + 6 * a.dk;  // [2][RL][VW][CL], behind two sets of q, k, g
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
  const float rate = expf(a.A_log[h]);
  for (int t = t0; t < t1; ++t) {
    float* qs = sm + (t & 1) * 3 * a.dk;  // two sets: a slow warp may still read the last token's
    float* ks = qs + a.dk;
    float* gs = ks + a.dk;
    const T* row = static_cast<const T*>(a.x) + static_cast<int64_t>(t) * a.ld;
    const float* dec = a.decay + static_cast<int64_t>(t) * a.ldd + h * a.dk;
    for (int i = threadIdx.x; i < a.dk; i += 256) {
      qs[i] = to_f(row[a.q_off + hq * a.dk + i]);
      ks[i] = to_f(row[a.k_off + hq * a.dk + i]);
      gs[i] = expf(-rate * softplus(dec[i] + a.dt_bias[h * a.dk + i]));
    }
    float v[VW], sk[VW], sq[VW];
#pragma unroll
    for (int c = 0; c < VW; ++c) {
      v[c] = live ? to_f(row[a.v_off + h * a.dv + c0 + c]) : 0.f;
      sk[c] = sq[c] = 0.f;
    }
    const float b = sigmoid(a.beta[static_cast<int64_t>(t) * a.ldb + h]);
    __syncthreads();
    float qq = 0.f, kk = 0.f, qk = 0.f;  // every warp for itself
    for (int i = threadIdx.x & 31; i < a.dk; i += 32) {
      qq = fmaf(qs[i], qs[i], qq);
      kk = fmaf(ks[i], ks[i], kk);
      qk = fmaf(qs[i], ks[i], qk);
    }
    const float iq = a.scale / sqrtf(warp_reduce_sum(qq) + kUnitEps), ik = 1.f / sqrtf(warp_reduce_sum(kk) + kUnitEps);
    qk = warp_reduce_sum(qk) * iq * ik;
    if constexpr (R > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = rl + RL * i;
        if (r < a.dk) {
          const float k = ks[r], q = qs[r], g = gs[r];
#pragma unroll
          for (int c = 0; c < VW; ++c) {
            S[i][c] *= g;
            sk[c] = fmaf(k, S[i][c], sk[c]);
            sq[c] = fmaf(q, S[i][c], sq[c]);
          }
        }
      }
    } else if (live) {
      for (int r = rl; r < a.dk; r += RL) {
        float s[VW];
        load_row(r, s);
#pragma unroll
        for (int c = 0; c < VW; ++c) {
          s[c] *= gs[r];
          sk[c] = fmaf(ks[r], s[c], sk[c]);
          sq[c] = fmaf(qs[r], s[c], sq[c]);
        }
      }
    }
#pragma unroll
    for (int c = 0; c < VW; ++c) {
      red[(rl * VW + c) * CL + cl] = sk[c];
      red[((RL + rl) * VW + c) * CL + cl] = sq[c];
    }
    __syncthreads();
    float u[VW], o[VW];
#pragma unroll
    for (int c = 0; c < VW; ++c) {
      float s1 = 0.f, s2 = 0.f;
#pragma unroll
      for (int w = 0; w < RL; ++w) {
        s1 += red[(w * VW + c) * CL + cl];
        s2 += red[((RL + w) * VW + c) * CL + cl];
      }
      u[c] = b * (v[c] - s1 * ik);
      o[c] = fmaf(qk, u[c], s2 * iq);
      u[c] *= ik;  // (the unit vector's factor, for the update with the raw k)
    }
    if constexpr (R > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = rl + RL * i;
        if (r < a.dk) {
          const float k = ks[r];
#pragma unroll
          for (int c = 0; c < VW; ++c) S[i][c] = fmaf(k, u[c], S[i][c]);
        }
      }
    } else if (live) {
      for (int r = rl; r < a.dk; r += RL) {
        float s[VW];
        load_row(r, s);
#pragma unroll
        for (int c = 0; c < VW; ++c) s[c] = fmaf(ks[r], u[c], gs[r] * s[c]);
        store_row(r, s);
      }
    }
    if (rl == 0 && live) {
      T* out = static_cast<T*>(a.out) + static_cast<int64_t>(t) * a.ldo + h * a.dv + c0;
#pragma unroll
      for (int c = 0; c < VW; ++c) put(out + c, o[c]);
    }
  }
  if constexpr (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rl + RL * i;
      if (live && r < a.dk) store_row(r, S[i]);
    }
  }
}

template <typename T, int VW, int CL>
int launch_recurrent(const DeltaArgs& a, int seq0, int n, cudaStream_t stream) {
  constexpr int RL = 256 / CL;
  const dim3 grid(a.H, ceil_div(a.dv, CL * VW), n);
  const size_t smem = sizeof(float) * (6 * a.dk + 2 * 256 * VW);
  if (smem > 48 * 1024 || n > 65535) return PXL_ERR_TOO_LARGE;
  if (a.dk <= 4 * RL) pxl_host::launch(delta_recurrent_kernel<T, VW, 4, CL>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 8 * RL) pxl_host::launch(delta_recurrent_kernel<T, VW, 8, CL>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 16 * RL) pxl_host::launch(delta_recurrent_kernel<T, VW, 16, CL>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 32 * RL) pxl_host::launch(delta_recurrent_kernel<T, VW, 32, CL>, grid, dim3(256), smem, stream, a, seq0);
  else pxl_host::launch(delta_recurrent_kernel<T, VW, 0, CL>, grid, dim3(256), smem, stream, a, seq0);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
template <typename T, int VW>
int launch_recurrent(const DeltaArgs& a, int seq0, int n, cudaStream_t stream) {
  return a.dv <= 16 * VW ? launch_recurrent<T, VW, 16>(a, seq0, n, stream) : launch_recurrent<T, VW, 32>(a, seq0, n, stream);
}
template <typename T>
int launch_recurrent(const DeltaArgs& a, int seq0, int n, cudaStream_t stream) {
  const bool vec = !(a.dv & 3) && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0;
  return vec ? launch_recurrent<T, 4>(a, seq0, n, stream) : launch_recurrent<T, 1>(a, seq0, n, stream);
}

// ---- chunked -----------------------------------------------------------------------------------------------
constexpr int kChunk = 64, kBlock = 16;
constexpr int kSlice = 32;  // columns of v per CTA of the walk

__device__ __forceinline__ float ex2(float x) {  // 2^x
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 f = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - f.x, b - f.y);
}
// one number as its two bf16 parts: high part in the low half of the word
__device__ __forceinline__ uint32_t split1(float a) {
  const bf16 hi = __float2bfloat16(a);
  return pack_bf16x2(__bfloat162float(hi), a - __bfloat162float(hi));
}
// two such words -> (high, high) and (low, low)
__device__ __forceinline__ void join2(uint2 w, uint32_t& hi, uint32_t& lo) {
  hi = __byte_perm(w.x, w.y, 0x5410);
  lo = __byte_perm(w.x, w.y, 0x7632);
}
__device__ __forceinline__ void mma3(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1,
                                     uint32_t bl0, uint32_t bl1) {
  const uint32_t bh[2] = {bh0, bh1}, bl[2] = {bl0, bl1};
  mma_m16n8k16_bf16(d, ah, bh);
  mma_m16n8k16_bf16(d, ah, bl);
  mma_m16n8k16_bf16(d, al, bh);
}

// log2(e) * softplus(z) to a few 1e-6 of itself: log2(1 + e^-|z|) by its series where that is small
__device__ __forceinline__ float softplus_log2(float z) {
  const float w = z * kLog2E, e = ex2(-fabsf(w));
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(1.f + e));
  const float series = e * kLog2E * fmaf(e, fmaf(e, fmaf(e, fmaf(e, 0.2f, -0.25f), 1.f / 3.f), -0.5f), 1.f);
  return fmaxf(w, 0.f) + (e < 0.0625f ? series : y);
}

// two fp32 numbers in a register pair
__device__ __forceinline__ uint64_t pair(float a, float b) {
  uint64_t v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(a), "f"(b));
  return v;
}
__device__ __forceinline__ float2 unpair(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}

// What the first kernel hands to the second, per (chunk, head), in 32-bit words
template <int DK>
struct Record {
  static constexpr int W = 0;                       // [64][DK] split words
  static constexpr int Q = W + kChunk * DK;         // [64][DK]: q e^G
  static constexpr int K = Q + kChunk * DK;         // [DK][64]: k e^(G_n - G), transposed
  static constexpr int P = K + kChunk * DK;         // [64][64], blocks up to the diagonal
  static constexpr int G = P + kChunk * kChunk;     // [DK] fp32: e^(G_n)
  static constexpr int U = G + DK;                  // [slices][64][32] fp32
  __host__ __device__ static int64_t words(int slices) { return U + static_cast<int64_t>(slices) * kChunk * kSlice; }
};

// chunk number `id` of the prompt slices: sequence and number within it; false past the last one. Warp-collective.
__device__ __forceinline__ bool find_chunk(const int* seq_cu, int seqs, int id, int& seq, int& index) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int s0 = 0; s0 < seqs; s0 += 32) {
    const int s = s0 + lane, n = s < seqs ? (seq_cu[s + 1] - seq_cu[s] + kChunk - 1) / kChunk : 0;
    int sum = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int y = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += y;
    }
    const unsigned past = __ballot_sync(0xffffffffu, base + sum > id);
    if (past) {
      const int l = __ffs(past) - 1;
      seq = s0 + l;
      index = id - base - __shfl_sync(0xffffffffu, sum - n, l);
      return true;
    }
    base += __shfl_sync(0xffffffffu, sum, 31);
  }
  return false;
}
// chunks of the sequences before `seq`. Warp-collective.
__device__ __forceinline__ int chunks_before(const int* seq_cu, int seq) {
  int n = 0;
  for (int s = threadIdx.x & 31; s < seq; s += 32) n += (seq_cu[s + 1] - seq_cu[s] + kChunk - 1) / kChunk;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
  return n;
}

template <int DK>
struct MakeSmem {
  static constexpr int kQ = DK + 8, kL = DK + 8, kA = kChunk + 4;
  bf16 q[kChunk][kQ], k[kChunk][kQ];
  float L[kChunk][kL];            // log2 g summed from the start of the token's block
  float E[kChunk / kBlock][DK];   // the block's whole sum
  float at[kChunk][kA];           // A transposed: [j][t]
  float p[kChunk][kA];
  float iq[kChunk], ik[kChunk], b[kChunk];
  int next;                       // next piece of work on A and P
};

constexpr int kMakeThreads = 256;

template <int DK>
__global__ void __launch_bounds__(kMakeThreads, 2) delta_make_kernel(const DeltaArgs a, int seqs, int chunk0, int slices,
                                                                    uint32_t* __restrict__ work) {
  extern __shared__ __align__(16) uint8_t raw[];
  using Sm = MakeSmem<DK>;
  using Rec = Record<DK>;
  Sm& s = *reinterpret_cast<Sm*>(raw);
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.y, hq = h / a.rep, tid = threadIdx.x, lane = tid & 31;
  int seq, index;
  if (!find_chunk(a.seq_cu, seqs, chunk0 + blockIdx.x, seq, index)) return;
  const int t0 = a.seq_cu[seq] + index * kChunk, left = a.seq_cu[seq + 1] - t0, n = left < kChunk ? left : kChunk;
  uint32_t* rec = work + (static_cast<int64_t>(blockIdx.x) * a.H + h) * Rec::words(slices);
  const bf16* x = static_cast<const bf16*>(a.x) + static_cast<int64_t>(t0) * a.ld;
  if (tid == 0) s.next = 0;
  // logits of the decays (a channel and 16 tokens at a time) are on their way first, and v into L2
  constexpr int kBlocks = kChunk / kBlock, kStride = kMakeThreads / DK, kMine = kBlocks > kStride ? kBlocks / kStride : 1;
  const int chan = tid % DK, blk0 = tid / DK;
  const bool has = chan < a.dk;
  float z[kMine][kBlock];
  {
    const float* dec = a.decay + static_cast<int64_t>(t0) * a.ldd + h * a.dk + chan;
#pragma unroll
    for (int m = 0; m < kMine; ++m)
#pragma unroll
      for (int i = 0; i < kBlock; ++i) {
        const int t = (blk0 + m * kStride) * kBlock + i;
        z[m][i] = t < n && has ? dec[static_cast<int64_t>(t) * a.ldd] : 0.f;
      }
    const int lines = ceil_div(a.dv, 64);
    for (int i = tid; i < n * lines; i += kMakeThreads)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(x + static_cast<int64_t>(i / lines) * a.ld + a.v_off + h * a.dv + i % lines * 64));
  }

  // ---- q and k with the factors that make them unit vectors; the rate of every token's update
  {
    const int r = tid >> 2, part = tid & 3;
    float qq = 0.f, kk = 0.f;
    const bf16x8 zero8 = {{0u, 0u, 0u, 0u}};
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) {
      const int d = (i * 4 + part) * 8;
      const bool in = r < n && d < a.dk;
      const bf16* row = x + static_cast<int64_t>(r) * a.ld + hq * a.dk + d;
      const bf16x8 q = in ? ld_bf16x8(row + a.q_off) : zero8, k = in ? ld_bf16x8(row + a.k_off) : zero8;
      st_bf16x8(&s.q[r][d], q);
      st_bf16x8(&s.k[r][d], k);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 qf = unpack_bf16x2(q.u[j]), kf = unpack_bf16x2(k.u[j]);
        qq += qf.x * qf.x + qf.y * qf.y;
        kk += kf.x * kf.x + kf.y * kf.y;
      }
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, o);
      kk += __shfl_xor_sync(0xffffffffu, kk, o);
    }
    if (part == 0) {
      s.iq[r] = a.scale / sqrtf(qq + kUnitEps);
      s.ik[r] = 1.f / sqrtf(kk + kUnitEps);
      s.b[r] = r < n ? sigmoid(a.beta[static_cast<int64_t>(t0 + r) * a.ldb + h]) : 0.f;
    }
  }
  // ---- decays: sums of log2 g inside every block of 16 tokens
  {
    const float rate = expf(a.A_log[h]), bias = has ? a.dt_bias[h * a.dk + chan] : 0.f;
#pragma unroll
    for (int m = 0; m < kMine; ++m) {
      const int blk = blk0 + m * kStride;
      if (blk >= kBlocks) break;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kBlock; ++i) {
        const int t = blk * kBlock + i;
        if (t < n && has) sum -= rate * softplus_log2(z[m][i] + bias);
        s.L[t][chan] = sum;
      }
      s.E[blk][chan] = sum;
    }
  }
  __syncthreads();

  // ---- A and P: 6 pairs of different blocks and the lower left quarters of 4 diagonal blocks (tensor cores), 64 rows of
  // the 8 x 8 blocks on the diagonal
  const int g8 = lane >> 2, t2 = (lane & 3) * 2;
  for (;;) {
    int job = 0;
    if (lane == 0) job = atomicAdd(&s.next, 1);
    job = __shfl_sync(0xffffffffu, job, 0);
    if (job >= 10 + kChunk) break;
    if (job < 6) {
      const int ra = job < 1 ? 1 : job < 3 ? 2 : 3, cb = job - (ra * (ra - 1)) / 2;  // (1,0) (2,0) (2,1) (3,0) (3,1) (3,2)
      const int r0 = ra * kBlock, j0 = cb * kBlock;
      float da[2][4] = {}, dp[2][4] = {};
#pragma unroll 1
      for (int kk = 0; kk < DK; kk += 16) {
        uint32_t kh[4], kl[4], qh[4], ql[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {  // rows g8 and g8 + 8, columns t2 and t2 + 8
          const int r = r0 + g8 + (i & 1) * 8, c = kk + t2 + (i >> 1) * 8;
          const float2 L = *reinterpret_cast<const float2*>(&s.L[r][c]);
          const float e0 = ex2(L.x), e1 = ex2(L.y);
          const float2 k = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(&s.k[r][c]));
          const float2 q = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(&s.q[r][c]));
          split2(k.x * e0, k.y * e1, kh[i], kl[i]);
          split2(q.x * e0, q.y * e1, qh[i], ql[i]);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          uint32_t bh[2], bl[2];
          const int j = j0 + u * 8 + g8;
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int c = kk + t2 + i * 8;
            const float2 L = *reinterpret_cast<const float2*>(&s.L[j][c]);
            float2 rest = *reinterpret_cast<const float2*>(&s.E[cb][c]);
            rest.x -= L.x, rest.y -= L.y;
            for (int m = cb + 1; m < ra; ++m) {
              const float2 E = *reinterpret_cast<const float2*>(&s.E[m][c]);
              rest.x += E.x, rest.y += E.y;
            }
            const float2 k = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(&s.k[j][c]));
            split2(k.x * ex2(rest.x), k.y * ex2(rest.y), bh[i], bl[i]);
          }
          mma3(da[u], kh, kl, bh[0], bh[1], bl[0], bl[1]);
          mma3(dp[u], qh, ql, bh[0], bh[1], bl[0], bl[1]);
        }
      }
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = r0 + g8 + (e >> 1) * 8, j = j0 + u * 8 + t2 + (e & 1);
          s.at[j][t] = da[u][e] * s.b[t] * s.ik[t] * s.ik[j];
          s.p[t][j] = dp[u][e] * s.iq[t] * s.ik[j];
        }
    } else if (job < 10) {  // rows of k above rows of q: A and P in one product
      const int j0 = (job - 6) * kBlock, t = j0 + 8 + g8, j = j0 + g8;
      float d[4] = {};
#pragma unroll 1
      for (int kk = 0; kk < DK; kk += 16) {
        uint32_t ah[4], al[4], bh[2], bl[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int c = kk + t2 + i * 8;
          const float2 mid = *reinterpret_cast<const float2*>(&s.L[j0 + 7][c]);
          const float2 Lt = *reinterpret_cast<const float2*>(&s.L[t][c]), Lj = *reinterpret_cast<const float2*>(&s.L[j][c]);
          const float e0 = ex2(Lt.x - mid.x), e1 = ex2(Lt.y - mid.y);
          const float2 k = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(&s.k[t][c]));
          const float2 q = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(&s.q[t][c]));
          const float2 kj = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(&s.k[j][c]));
          split2(k.x * e0, k.y * e1, ah[2 * i], al[2 * i]);
          split2(q.x * e0, q.y * e1, ah[2 * i + 1], al[2 * i + 1]);
          split2(kj.x * ex2(mid.x - Lj.x), kj.y * ex2(mid.y - Lj.y), bh[i], bl[i]);
        }
        mma3(d, ah, al, bh[0], bh[1], bl[0], bl[1]);
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = j0 + t2 + e;
        s.at[col][t] = d[e] * s.b[t] * s.ik[t] * s.ik[col];
        s.p[t][col] = d[2 + e] * s.iq[t] * s.ik[col];
      }
    } else {
      const int t = job - 10, j0 = t & ~7, last = t - j0;
      constexpr int V = DK / 32;
      float kt[V], qt[V], Lt[V], acc[16];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const int c = v * 32 + lane;
        kt[v] = __bfloat162float(s.k[t][c]), qt[v] = __bfloat162float(s.q[t][c]), Lt[v] = s.L[t][c];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        acc[j] = acc[8 + j] = 0.f;
        if (j <= last) {
#pragma unroll
          for (int v = 0; v < V; ++v) {
            const int c = v * 32 + lane;
            const float w = __bfloat162float(s.k[j0 + j][c]) * ex2(Lt[v] - s.L[j0 + j][c]);
            acc[j] = fmaf(kt[v], w, acc[j]);
            acc[8 + j] = fmaf(qt[v], w, acc[8 + j]);
          }
        }
      }
      // sums over the lanes; lanes 2 i and 2 i + 1 end with number i
#pragma unroll
      for (int o = 16; o > 1; o >>= 1) {
#pragma unroll
        for (int i = 0; i < o / 2; ++i) {
          const bool up = lane & o;
          const float give = up ? acc[i] : acc[i + o / 2], keep = up ? acc[i + o / 2] : acc[i];
          acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
      }
      const float sum = acc[0] + __shfl_xor_sync(0xffffffffu, acc[0], 1);
      const int i = lane >> 1, j = j0 + (i & 7);
      if ((lane & 1) == 0) {
        if (i < 8) s.at[j][t] = i < last ? sum * s.b[t] * s.ik[t] * s.ik[j] : 0.f;
        else s.p[t][j] = sum * s.iq[t] * s.ik[j];
      }
    }
  }
  __syncthreads();

  // ---- sums of the blocks before, for the whole chunk's exponents
  auto before = [&](int blk, int c) {
    float sum = 0.f;
    for (int m = 0; m < blk; ++m) sum += s.E[m][c];
    return sum;
  };
  // ---- (1 + A) X = [b k e^G | b v], a column per thread
  for (int col = tid; col < DK + slices * kSlice; col += kMakeThreads) {
    const bool key = col < DK;
    const int c = key ? col : col - DK;
    uint64_t y[kChunk / 2];  // two tokens each
    if (key) {
      float base = 0.f;
#pragma unroll
      for (int t = 0; t < kChunk; t += 2) {
        if (t % kBlock == 0 && t > 0) base += s.E[t / kBlock - 1][c];
        y[t / 2] = pair(s.b[t] * s.ik[t] * __bfloat162float(s.k[t][c]) * ex2(base + s.L[t][c]),
                        s.b[t + 1] * s.ik[t + 1] * __bfloat162float(s.k[t + 1][c]) * ex2(base + s.L[t + 1][c]));
      }
    } else {
      const bf16* v = x + a.v_off + h * a.dv + c;
      auto value = [&](int t) { return t < n && c < a.dv ? s.b[t] * __bfloat162float(v[static_cast<int64_t>(t) * a.ld]) : 0.f; };
#pragma unroll
      for (int t = 0; t < kChunk; t += 2) y[t / 2] = pair(value(t), value(t + 1));
    }
#pragma unroll
    for (int j = 0; j + 1 < kChunk; ++j) {
      const float2 yj = unpair(y[j / 2]);
      const float xj = j & 1 ? yj.y : yj.x;
      const uint64_t xx = pair(-xj, -xj);
#pragma unroll
      for (int t4 = (j + 1) / 4 * 4; t4 < kChunk; t4 += 4) {
        const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(&s.at[j][t4]);
        if (t4 > j) y[t4 / 2] = fma2(w.x, xx, y[t4 / 2]);
        else if (t4 == j) y[t4 / 2] = pair(yj.x, fmaf(-unpair(w.x).y, xj, yj.y));
        if (t4 + 2 > j) y[t4 / 2 + 1] = fma2(w.y, xx, y[t4 / 2 + 1]);
        else if (t4 + 2 == j) y[t4 / 2 + 1] = pair(yj.x, fmaf(-unpair(w.y).y, xj, yj.y));
      }
    }
    if (key) {
#pragma unroll
      for (int t = 0; t < kChunk; t += 2) {
        const float2 f = unpair(y[t / 2]);
        rec[Rec::W + t * DK + c] = split1(f.x);
        rec[Rec::W + (t + 1) * DK + c] = split1(f.y);
      }
    } else {
      float* U = reinterpret_cast<float*>(rec) + Rec::U + static_cast<int64_t>(c / kSlice) * kChunk * kSlice + c % kSlice;
#pragma unroll
      for (int t = 0; t < kChunk; t += 2) {
        const float2 f = unpair(y[t / 2]);
        U[t * kSlice] = f.x;
        U[(t + 1) * kSlice] = f.y;
      }
    }
  }
  // ---- q e^G, k e^(G_n - G), e^(G_n): a channel and a part of the tokens per thread
  {
    constexpr int kShare = kMakeThreads / DK, kTokens = kChunk / kShare;
    const int c = tid % DK, first = tid / DK * kTokens;
    const float whole = before(kChunk / kBlock, c);
    float base = before(first / kBlock, c);
    uint32_t kd[4];
#pragma unroll 4
    for (int i = 0; i < kTokens; ++i) {
      const int t = first + i;
      if (i > 0 && t % kBlock == 0) base += s.E[t / kBlock - 1][c];
      const float G = base + s.L[t][c];
      rec[Rec::Q + t * DK + c] = split1(__bfloat162float(s.q[t][c]) * s.iq[t] * ex2(G));
      kd[i & 3] = split1(__bfloat162float(s.k[t][c]) * s.ik[t] * ex2(whole - G));
      if ((i & 3) == 3) *reinterpret_cast<uint4*>(&rec[Rec::K + c * kChunk + t - 3]) = make_uint4(kd[0], kd[1], kd[2], kd[3]);
    }
    if (tid < DK) reinterpret_cast<float*>(rec)[Rec::G + c] = ex2(whole);
  }
  for (int i = tid; i < kChunk * kChunk; i += kMakeThreads) {
    const int t = i / kChunk, j = i % kChunk;
    if (j / kBlock <= t / kBlock) rec[Rec::P + i] = t < n && j <= t ? split1(s.p[t][j]) : 0u;
  }
}

template <int DK>
struct WalkSmem {
  static constexpr int kW = DK + 8, kT = kChunk + 8, kV = kSlice + 8;  // row pitches without bank conflicts
  uint32_t w[kChunk][kW], q[kChunk][kW];
  uint32_t k[DK][kT], p[kChunk][kT];
  float u0[kChunk][kV];
  float g[DK];
  bf16 s_hi[DK][kV], s_lo[DK][kV];
  bf16 u_hi[kChunk][kV], u_lo[kChunk][kV];
};

// Warps 0 to 7 make u and keep the state, warps 8 to 15 make the outputs.
constexpr int kHalf = 8, kWalkWarps = 2 * kHalf;

__device__ __forceinline__ void copy16(void* dst, const void* src) { cp_async_16(smem_u32(dst), src, true); }

// grid (slices of v, heads, sequences): the chunks [chunk0, chunk0 + chunks) of one sequence, in order
template <int DK>
__global__ void __launch_bounds__(kWalkWarps * 32, 1) delta_walk_kernel(const DeltaArgs a, int chunk0, int chunks, int slices,
                                                                    const uint32_t* __restrict__ work) {
  extern __shared__ __align__(16) uint8_t raw[];
  using Sm = WalkSmem<DK>;
  using Rec = Record<DK>;
  Sm& s = *reinterpret_cast<Sm*>(raw);
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kSlice;
  const int t0 = a.seq_cu[seq], n_all = a.seq_cu[seq + 1] - t0;
  const int mine = (n_all + kChunk - 1) / kChunk, base = chunks_before(a.seq_cu, seq);
  // chunks of this sequence in the range: [first, last)
  const int first = chunk0 > base ? chunk0 - base : 0, last = chunk0 + chunks - base < mine ? chunk0 + chunks - base : mine;
  if (first >= last) return;
  float* Sg = state_of(a, seq, h);
  if (Sg == nullptr) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, r8 = lane & 7, g8 = lane >> 2, t2 = (lane & 3) * 2;
  const bool fresh = first == 0 && a.positions[t0] == 0;

  auto record = [&](int i) { return work + (static_cast<int64_t>(base + i - chunk0) * a.H + h) * Rec::words(slices); };
  auto load_front = [&](int i) {  // W, q e^G, U
    const uint32_t* r = record(i);
    for (int x = tid * 4; x < kChunk * DK; x += kWalkWarps * 128) {
      copy16(&s.w[x / DK][x % DK], r + Rec::W + x);
      copy16(&s.q[x / DK][x % DK], r + Rec::Q + x);
    }
    for (int x = tid * 4; x < kChunk * kSlice; x += kWalkWarps * 128)
      copy16(&s.u0[x / kSlice][x % kSlice], r + Rec::U + static_cast<int64_t>(blockIdx.x) * kChunk * kSlice + x);
    cp_async_commit();
  };
  auto load_back = [&](int i) {  // k e^(G_n - G), P, e^(G_n)
    const uint32_t* r = record(i);
    for (int x = tid * 4; x < kChunk * DK; x += kWalkWarps * 128) copy16(&s.k[x / kChunk][x % kChunk], r + Rec::K + x);
    for (int x = tid * 4; x < kChunk * kChunk; x += kWalkWarps * 128) copy16(&s.p[x / kChunk][x % kChunk], r + Rec::P + x);
    if (tid < DK / 4) copy16(&s.g[tid * 4], r + Rec::G + tid * 4);
    cp_async_commit();
  };
  load_front(first);
  load_back(first);

  // 16 x 16 tiles of the state, in the layout of the accumulators (first half of the warps)
  constexpr int kTilesK = DK / 16, kTiles = kTilesK * 2, NT = (kTiles + kHalf - 1) / kHalf;
  const bool keeper = warp < kHalf;
  const int w8 = warp % kHalf, rg = w8 & 3, ch = w8 >> 2;  // 16 tokens; half of the slice's columns
  float S[NT][2][4];
  auto each = [&](auto f) {  // f(element, row, column)
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int tile = w8 + i * kHalf, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (tile < kTiles) f(S[i][j][e], m0 + g8 + (e >> 1) * 8, n0 + j * 8 + t2 + (e & 1));
    }
  };
  auto publish = [&]() {
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int tile = w8 + i * kHalf, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
      if (tile >= kTiles) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          uint32_t hi, lo;
          split2(S[i][j][2 * e], S[i][j][2 * e + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(&s.s_hi[m0 + g8 + e * 8][n0 + j * 8 + t2]) = hi;
          *reinterpret_cast<uint32_t*>(&s.s_lo[m0 + g8 + e * 8][n0 + j * 8 + t2]) = lo;
        }
    }
  };
  if (keeper) {
    each([&](float& v, int r, int c) {
      v = !fresh && r < a.dk && v0 + c < a.dv ? Sg[static_cast<int64_t>(r) * a.dv + v0 + c] : 0.f;
    });
    publish();
  }

  for (int i = first; i < last; ++i) {
    const int c0 = i * kChunk, n = n_all - c0 < kChunk ? n_all - c0 : kChunk;
    cp_async_wait<1>();  // front part (the back part may still be on its way)
    __syncthreads();
    // ---- W S and (q e^G) S: 16 tokens x 16 columns, the three products of the split operands side by side
    float o[2][4] = {}, o1[2][4] = {}, o2[2][4] = {};
    const auto& rows = keeper ? s.w : s.q;
#pragma unroll
    for (int kk = 0; kk < kTilesK; ++kk) {
      uint32_t ah[4], al[4], sh[4], sl[4];
#pragma unroll
      for (int x = 0; x < 4; ++x)
        join2(*reinterpret_cast<const uint2*>(&rows[rg * 16 + g8 + (x & 1) * 8][kk * 16 + t2 + (x >> 1) * 8]), ah[x], al[x]);
      ldmatrix_x4_trans(sh, smem_u32(&s.s_hi[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
      ldmatrix_x4_trans(sl, smem_u32(&s.s_lo[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const uint32_t bh[2] = {sh[2 * j], sh[2 * j + 1]}, bl[2] = {sl[2 * j], sl[2 * j + 1]};
        mma_m16n8k16_bf16(o[j], ah, bh);
        mma_m16n8k16_bf16(o1[j], ah, bl);
        mma_m16n8k16_bf16(o2[j], al, bh);
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[j][e] += o1[j][e] + o2[j][e];
    if (keeper) {  // u = U - W S
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = rg * 16 + g8 + e * 8, c = ch * 16 + j * 8 + t2;
          const float2 u0 = *reinterpret_cast<const float2*>(&s.u0[r][c]);
          uint32_t hi, lo;
          split2(u0.x - o[j][2 * e], u0.y - o[j][2 * e + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(&s.u_hi[r][c]) = hi;
          *reinterpret_cast<uint32_t*>(&s.u_lo[r][c]) = lo;
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    if (i + 1 < last) load_front(i + 1);

    if (!keeper) {
      // ---- o += P u (blocks up to this one)
      for (int kk = 0; kk <= rg; ++kk) {
        uint32_t ph[4], pl[4], bh[4], bl[4];
#pragma unroll
        for (int x = 0; x < 4; ++x)
          join2(*reinterpret_cast<const uint2*>(&s.p[rg * 16 + g8 + (x & 1) * 8][kk * 16 + t2 + (x >> 1) * 8]), ph[x], pl[x]);
        ldmatrix_x4_trans(bh, smem_u32(&s.u_hi[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
        ldmatrix_x4_trans(bl, smem_u32(&s.u_lo[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
#pragma unroll
        for (int j = 0; j < 2; ++j) mma3(o[j], ph, pl, bh[2 * j], bh[2 * j + 1], bl[2 * j], bl[2 * j + 1]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = rg * 16 + g8 + e * 8, c = v0 + ch * 16 + j * 8 + t2;
          if (r < n && c < a.dv)
            *reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.out) + static_cast<int64_t>(t0 + c0 + r) * a.ldo + h * a.dv + c) =
                pack_bf16x2(o[j][2 * e], o[j][2 * e + 1]);
        }
    } else {
      // ---- S = e^(G_n) S + (k e^(G_n - G))^T u
      each([&](float& v, int r, int) { v *= s.g[r]; });
#pragma unroll
      for (int kk = 0; kk < kChunk / 16; ++kk) {
#pragma unroll
        for (int x = 0; x < NT; ++x) {
          const int tile = w8 + x * kHalf, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
          if (tile >= kTiles) continue;
          uint32_t kh[4], kl[4], bh[4], bl[4];
#pragma unroll
          for (int y = 0; y < 4; ++y)
            join2(*reinterpret_cast<const uint2*>(&s.k[m0 + g8 + (y & 1) * 8][kk * 16 + t2 + (y >> 1) * 8]), kh[y], kl[y]);
          ldmatrix_x4_trans(bh, smem_u32(&s.u_hi[kk * 16 + (mi & 1) * 8 + r8][n0 + (mi >> 1) * 8]));
          ldmatrix_x4_trans(bl, smem_u32(&s.u_lo[kk * 16 + (mi & 1) * 8 + r8][n0 + (mi >> 1) * 8]));
#pragma unroll
          for (int j = 0; j < 2; ++j) mma3(S[x][j], kh, kl, bh[2 * j], bh[2 * j + 1], bl[2 * j], bl[2 * j + 1]);
        }
      }
      publish();  // every read of the old state happened before the last barrier
    }
    __syncthreads();
    if (i + 1 < last) load_back(i + 1);
  }
  if (keeper)
    each([&](float& v, int r, int c) {
      if (r < a.dk && v0 + c < a.dv) Sg[static_cast<int64_t>(r) * a.dv + v0 + c] = v;
    });
}

template <typename K>
bool opt_in(K kern, int smem) {
  return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) == cudaSuccess;
}

template <typename F>
auto with_dim(int dk, F f) {
  return dk <= 32 ? f(std::integral_constant<int, 32>{}) : dk <= 64 ? f(std::integral_constant<int, 64>{})
                                                                    : f(std::integral_constant<int, 128>{});
}

// The chunks are worked off in runs whose records fit the workspace.
template <int DK>
int launch_chunked(const DeltaArgs& a, int seqs, int tokens, uint32_t* work, int64_t work_words, cudaStream_t stream) {
  static bool done[64] = {false};
  const int dev = pxl_host::current_device_slot();
  constexpr int make_smem = sizeof(MakeSmem<DK>), walk_smem = sizeof(WalkSmem<DK>);
  if (!done[dev]) {
    if (!opt_in(delta_make_kernel<DK>, make_smem) || !opt_in(delta_walk_kernel<DK>, walk_smem)) return PXL_ERR_CUDA;
    done[dev] = true;
  }
  const int slices = ceil_div(a.dv, kSlice), bound = tokens / kChunk + seqs;  // at most this many chunks
  const int64_t fit = work_words / (Record<DK>::words(slices) * a.H);
  if (fit < 1 || seqs > 65535 || a.H > 65535) return PXL_ERR_TOO_LARGE;
  const int run = fit < bound ? static_cast<int>(fit) : bound;
  for (int c0 = 0; c0 < bound; c0 += run) {
    const int n = bound - c0 < run ? bound - c0 : run;
    pxl_host::launch(delta_make_kernel<DK>, dim3(n, a.H), dim3(kMakeThreads), make_smem, stream, a, seqs, c0, slices, work);
    pxl_host::launch(delta_walk_kernel<DK>, dim3(slices, a.H, seqs), dim3(kWalkWarps * 32), walk_smem, stream, a, c0, n, slices,
                     static_cast<const uint32_t*>(work));
  }
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

inline bool chunkable(const DeltaArgs& a) {
  return a.dk <= 128 && !((a.q_off | a.k_off | a.v_off | a.dk | a.dv | static_cast<int>(a.ld) | static_cast<int>(a.ldo)) & 7) &&
         ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.out)) & 15) == 0;
}
}  // namespace

PXL_EXPORT int64_t pxl_delta_rule_workspace(int H, int dk, int dv, int prefill_seqs, int prefill_tokens) {
  if (dk > 128 || prefill_seqs <= 0) return 0;
  const int slices = pxl::ceil_div(dv, kSlice);
  const int64_t words = with_dim(dk, [&](auto d) { return Record<decltype(d)::value>::words(slices); });
  const int64_t all = 4 * words * H * (prefill_tokens / kChunk + prefill_seqs), one = 4 * words * H, cap = 256ll << 20;
  return all < cap ? all : one > cap ? one : cap / one * one;
}

PXL_EXPORT int pxl_delta_rule(const void* x, int64_t ld, int q_off, int k_off, int v_off, int H, int Hk, int dk, int dv,
                              const float* decay, int64_t ldd, const float* dt_bias, const float* A_log, const float* beta,
                              int64_t ldb, float* state, int num_slots, const int* seq_cu, const int* seq_slots,
                              const int* positions, void* out, int64_t ldo, int prefill_seqs, int prefill_tokens, int decode_seqs,
                              void* work, int64_t work_bytes, int is_f32, int* status, cudaStream_t stream) {
  if (H <= 0 || Hk <= 0 || H % Hk || dk <= 0 || dv <= 0) return PXL_ERR_INVALID_ARG;
  const DeltaArgs a{x, ld, q_off, k_off, v_off, H, H / Hk, dk, dv, decay, ldd, dt_bias, A_log, beta, ldb,
                    1.f / sqrtf(static_cast<float>(dk)), state, num_slots, seq_cu, seq_slots, positions, out, ldo, status};
  int code = PXL_OK;
  if (prefill_seqs > 0) {
    if (is_f32) code = launch_recurrent<float>(a, 0, prefill_seqs, stream);
    else if (!chunkable(a) || work == nullptr) code = launch_recurrent<pxl::bf16>(a, 0, prefill_seqs, stream);
    else
      code = with_dim(dk, [&](auto d) {
        return launch_chunked<decltype(d)::value>(a, prefill_seqs, prefill_tokens, static_cast<uint32_t*>(work), work_bytes / 4, stream);
      });
  }
  if (code == PXL_OK && decode_seqs > 0)
    code = is_f32 ? launch_recurrent<float>(a, prefill_seqs, decode_seqs, stream)
                  : launch_recurrent<pxl::bf16>(a, prefill_seqs, decode_seqs, stream);
  return code;
}
