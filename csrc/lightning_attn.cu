// Lightning attention: linear attention with a fixed decay per head and a state matrix per request,
//
//   q = silu(.), k = silu(.), v = silu(.) of the packed projection's columns
//   S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
//
// State slots [slots, H, dk, dv] fp32; a sequence whose first token of this step sits at position 0 starts from
// zero. Two kernels share the state:
//
//  * recurrent: one CTA per (head, 32 or 128 columns of v, sequence) keeps its part of S in registers and walks the
//    sequence's tokens. Decoding (one pass over the state per token, memory bound), fp32, odd sizes.
//  * chunked (bf16 prompts): 64 tokens at a time on the tensor cores. With local places i, j of a chunk,
//        o_i = decay^(i+1) S_0^T q_i + sum_(j<=i) decay^(i-j) (q_i . k_j) v_j
//        S   = decay^n S_0 + sum_j k_j (decay^(n-1-j) v_j)^T
//    The state is accumulated in fp32 registers. Operands that are not bf16 to begin with (decayed scores, decayed
//    values, the state) enter the products as a sum of two bf16 numbers, so their rounding is 2^-17, not 2^-9.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float silu(float v) { return v / (1.f + expf(-v)); }
// activation in the precision of the model
__device__ __forceinline__ float act(float v) { return silu(v); }
__device__ __forceinline__ float act(bf16 v) { return __bfloat162float(__float2bfloat16(silu(__bfloat162float(v)))); }

constexpr int kChunk = 64;

struct LightningArgs {
  const void* proj;  // [T, ld]
  int64_t ld;
  int q_off, k_off, v_off, H, dk, dv;
  const float* pow;  // [H, kChunk + 1]: decay^n
  float* state;      // [slots, H, dk, dv]
  int num_slots;
  const int* seq_cu;
  const int* seq_slots;
  const int* positions;
  void* out;  // [T, ldo]: heads side by side
  int64_t ldo;
  int* status;
};

// state of (sequence, head), or null for a slot outside the pool (the status word is set)
__device__ __forceinline__ float* state_of(const LightningArgs& a, int seq, int h) {
  const int slot = a.seq_slots[seq];
  if (slot < 0 || slot >= a.num_slots) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_INDEX);
    return nullptr;
  }
  return a.state + (static_cast<int64_t>(slot) * a.H + h) * a.dk * a.dv;
}

// ---- recurrent ---------------------------------------------------------------------------------------------
// 256 threads = 8 row lanes x 32 column lanes of VW columns; R rows of S per thread in registers (R == 0: the state
// stays in global memory, any dk).
template <typename T, int VW, int R>
__global__ void __launch_bounds__(256) lightning_recurrent_kernel(const LightningArgs a, int seq0) {
  extern __shared__ float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.x, seq = seq0 + blockIdx.z;
  const int cl = threadIdx.x & 31, rl = threadIdx.x >> 5;
  const int c0 = (blockIdx.y * 32 + cl) * VW;
  const int t0 = a.seq_cu[seq], t1 = a.seq_cu[seq + 1];
  if (t1 <= t0) return;
  float* Sg = state_of(a, seq, h);
  if (Sg == nullptr) return;
  const bool fresh = a.positions[t0] == 0, live = c0 < a.dv;
  float* qs = sm;
  float* ks = qs + a.dk;
  float* red = ks + a.dk;  // [8][32 * VW]
  const float decay = a.pow[h * (kChunk + 1) + 1];
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
      const int r = rl + 8 * i;
      if (!fresh && live && r < a.dk) {
        load_row(r, S[i]);
      } else {
#pragma unroll
        for (int c = 0; c < VW; ++c) S[i][c] = 0.f;
      }
    }
  } else if (fresh && live) {
    const float zero[VW] = {};
    for (int r = rl; r < a.dk; r += 8) store_row(r, zero);
  }
  for (int t = t0; t < t1; ++t) {
    const T* row = static_cast<const T*>(a.proj) + static_cast<int64_t>(t) * a.ld;
    for (int i = threadIdx.x; i < a.dk; i += 256) {
      qs[i] = act(row[a.q_off + h * a.dk + i]);
      ks[i] = act(row[a.k_off + h * a.dk + i]);
    }
    float v[VW], o[VW];
#pragma unroll
    for (int c = 0; c < VW; ++c) {
      v[c] = live ? act(row[a.v_off + h * a.dv + c0 + c]) : 0.f;
      o[c] = 0.f;
    }
    __syncthreads();
    if constexpr (R > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = rl + 8 * i;
        if (r < a.dk) {
          const float k = ks[r], q = qs[r];
#pragma unroll
          for (int c = 0; c < VW; ++c) {
            S[i][c] = fmaf(k, v[c], decay * S[i][c]);
            o[c] = fmaf(q, S[i][c], o[c]);
          }
        }
      }
    } else if (live) {
      for (int r = rl; r < a.dk; r += 8) {
        float s[VW];
        load_row(r, s);
        const float k = ks[r], q = qs[r];
#pragma unroll
        for (int c = 0; c < VW; ++c) {
          s[c] = fmaf(k, v[c], decay * s[c]);
          o[c] = fmaf(q, s[c], o[c]);
        }
        store_row(r, s);
      }
    }
#pragma unroll
    for (int c = 0; c < VW; ++c) red[(rl * VW + c) * 32 + cl] = o[c];
    __syncthreads();
    for (int i = threadIdx.x; i < 32 * VW; i += 256) {  // column i of this CTA's slice
      const int col = blockIdx.y * 32 * VW + i;
      if (col < a.dv) {
        float sum = 0.f;
#pragma unroll
        for (int r = 0; r < 8; ++r) sum += red[(r * VW + i % VW) * 32 + i / VW];
        put(static_cast<T*>(a.out) + static_cast<int64_t>(t) * a.ldo + h * a.dv + col, sum);
      }
    }
  }
  if constexpr (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rl + 8 * i;
      if (live && r < a.dk) store_row(r, S[i]);
    }
  }
}

template <typename T, int VW>
int launch_recurrent(const LightningArgs& a, int seq0, int n, cudaStream_t stream) {
  const dim3 grid(a.H, ceil_div(a.dv, 32 * VW), n);
  const size_t smem = sizeof(float) * (2 * a.dk + 8 * 32 * VW);
  if (smem > 48 * 1024 || n > 65535) return PXL_ERR_TOO_LARGE;
  if (a.dk <= 32) pxl_host::launch(lightning_recurrent_kernel<T, VW, 4>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 64) pxl_host::launch(lightning_recurrent_kernel<T, VW, 8>, grid, dim3(256), smem, stream, a, seq0);
  else if (a.dk <= 128) pxl_host::launch(lightning_recurrent_kernel<T, VW, 16>, grid, dim3(256), smem, stream, a, seq0);
  else pxl_host::launch(lightning_recurrent_kernel<T, VW, 0>, grid, dim3(256), smem, stream, a, seq0);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
template <typename T>
int launch_recurrent(const LightningArgs& a, int seq0, int n, cudaStream_t stream) {
  const bool vec = a.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0;
  return vec ? launch_recurrent<T, 4>(a, seq0, n, stream) : launch_recurrent<T, 1>(a, seq0, n, stream);
}

// ---- chunked -----------------------------------------------------------------------------------------------
constexpr int kVS = 32;  // columns of v (and of the state) per CTA
constexpr int kWarps = 8;

__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 f = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - f.x, b - f.y);
}
__device__ __forceinline__ void mma2(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  const uint32_t b[2] = {b0, b1};
  mma_m16n8k16_bf16(d, a, b);
}

template <int DK>
struct ChunkSmem {
  static constexpr int kQ = DK + 8, kV = kVS + 8, kP = kChunk + 8;  // row pitches: 16-byte steps fall into distinct banks
  bf16 q[kChunk][kQ], k[kChunk][kQ];
  bf16 v[kChunk][kV], vd_hi[kChunk][kV], vd_lo[kChunk][kV];
  bf16 p_hi[kChunk][kP], p_lo[kChunk][kP];
  bf16 s_hi[DK][kV], s_lo[DK][kV];
  float pow[kChunk + 1];
};

// grid (slices of v, heads, sequences). Per chunk: stage q, k, v | scores and S_0^T q | P v, new state.
template <int DK>
__global__ void __launch_bounds__(kWarps * 32) lightning_chunk_kernel(const LightningArgs a) {
  extern __shared__ __align__(16) uint8_t raw[];
  using Sm = ChunkSmem<DK>;
  Sm& s = *reinterpret_cast<Sm*>(raw);
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kVS;
  const int t0 = a.seq_cu[seq], n_all = a.seq_cu[seq + 1] - t0;
  if (n_all <= 0) return;
  float* Sg = state_of(a, seq, h);
  if (Sg == nullptr) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int mi = lane >> 3, r8 = lane & 7;
  for (int i = tid; i <= kChunk; i += kWarps * 32) s.pow[i] = a.pow[h * (kChunk + 1) + i];

  // this warp's 16 x 16 tiles of the state, in the layout of the accumulators
  constexpr int kTilesK = DK / 16, kTiles = kTilesK * 2, NT = (kTiles + kWarps - 1) / kWarps;
  float S[NT][2][4];
  const bool fresh = a.positions[t0] == 0;
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
    }
  };
  publish_state();

  // rows of the next chunk travel through registers while this one is computed
  constexpr int kVecQ = kChunk * DK / 8 / (kWarps * 32), kVecV = kChunk * kVS / 8 / (kWarps * 32);
  bf16x8 rq[kVecQ], rk[kVecQ], rv[kVecV];
  const bf16* base = static_cast<const bf16*>(a.proj) + static_cast<int64_t>(t0) * a.ld;
  const bf16x8 zero8 = {{0u, 0u, 0u, 0u}};
  auto fetch = [&](int c0) {
#pragma unroll
    for (int i = 0; i < kVecQ; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (DK / 8), d = x % (DK / 8) * 8;
      const bool in = c0 + r < n_all && d < a.dk;
      const bf16* p = base + static_cast<int64_t>(c0 + r) * a.ld + h * a.dk + d;
      rq[i] = in ? ld_bf16x8(p + a.q_off) : zero8;
      rk[i] = in ? ld_bf16x8(p + a.k_off) : zero8;
    }
#pragma unroll
    for (int i = 0; i < kVecV; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (kVS / 8), d = v0 + x % (kVS / 8) * 8;
      const bool in = c0 + r < n_all && d < a.dv;
      rv[i] = in ? ld_bf16x8(base + static_cast<int64_t>(c0 + r) * a.ld + a.v_off + h * a.dv + d) : zero8;
    }
  };
  auto act8 = [](const bf16x8& x, float (&f)[8]) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 u = unpack_bf16x2(x.u[j]);
      f[2 * j] = silu(u.x), f[2 * j + 1] = silu(u.y);
    }
  };
  auto pack8 = [](const float (&f)[8]) {
    bf16x8 o;
#pragma unroll
    for (int j = 0; j < 4; ++j) o.u[j] = pack_bf16x2(f[2 * j], f[2 * j + 1]);
    return o;
  };
  fetch(0);
  __syncthreads();

  const int rg = warp & 3, ch = warp >> 2;  // 16 query rows; half of the columns of the scores and of v
  for (int c0 = 0; c0 < n_all; c0 += kChunk) {
    const int n = n_all - c0 < kChunk ? n_all - c0 : kChunk;
    // ---- activations into shared memory
#pragma unroll
    for (int i = 0; i < kVecQ; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (DK / 8), d = x % (DK / 8) * 8;
      float f[8];
      act8(rq[i], f);
      st_bf16x8(&s.q[r][d], pack8(f));
      act8(rk[i], f);
      st_bf16x8(&s.k[r][d], pack8(f));
    }
#pragma unroll
    for (int i = 0; i < kVecV; ++i) {
      const int x = i * kWarps * 32 + tid, r = x / (kVS / 8), d = x % (kVS / 8) * 8;
      float f[8];
      act8(rv[i], f);
      const bf16x8 v = pack8(f);
      st_bf16x8(&s.v[r][d], v);
      const float w = r < n ? s.pow[n - 1 - r] : 0.f;
      bf16x8 hi, lo;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 u = unpack_bf16x2(v.u[j]);
        split2(u.x * w, u.y * w, hi.u[j], lo.u[j]);
      }
      st_bf16x8(&s.vd_hi[r][d], hi);
      st_bf16x8(&s.vd_lo[r][d], lo);
    }
    __syncthreads();
    if (c0 + kChunk < n_all) fetch(c0 + kChunk);

    // ---- scores of 16 rows x 32 columns, and S_0^T q for 16 rows x 16 columns
    float o[2][4] = {};
    {
      float p[4][4] = {};
      const bool needed = ch * 32 <= rg * 16 + 15;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t qa[4], b[4];
        ldmatrix_x4(qa, smem_u32(&s.q[rg * 16 + (mi & 1) * 8 + r8][kk * 16 + (mi >> 1) * 8]));
        if (needed) {
#pragma unroll
          for (int g = 0; g < 2; ++g) {
            ldmatrix_x4(b, smem_u32(&s.k[ch * 32 + g * 16 + (mi >> 1) * 8 + r8][kk * 16 + (mi & 1) * 8]));
            mma2(p[2 * g], qa, b[0], b[1]);
            mma2(p[2 * g + 1], qa, b[2], b[3]);
          }
        }
        ldmatrix_x4_trans(b, smem_u32(&s.s_hi[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
        mma2(o[0], qa, b[0], b[1]);
        mma2(o[1], qa, b[2], b[3]);
        ldmatrix_x4_trans(b, smem_u32(&s.s_lo[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
        mma2(o[0], qa, b[0], b[1]);
        mma2(o[1], qa, b[2], b[3]);
      }
      if (needed) {
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int r = rg * 16 + (lane >> 2) + e * 8, c = ch * 32 + j * 8 + (lane & 3) * 2;
            const float x = c <= r ? p[j][2 * e] * s.pow[r - c] : 0.f;
            const float y = c + 1 <= r ? p[j][2 * e + 1] * s.pow[r - c - 1] : 0.f;
            uint32_t hi, lo;
            split2(x, y, hi, lo);
            *reinterpret_cast<uint32_t*>(&s.p_hi[r][c]) = hi;
            *reinterpret_cast<uint32_t*>(&s.p_lo[r][c]) = lo;
          }
      }
    }
    __syncthreads();

    // ---- o += P v (keys up to this row group), and the state at the chunk's end
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[j][e] *= s.pow[rg * 16 + (lane >> 2) + (e >> 1) * 8 + 1];
    for (int kk = 0; kk <= rg; ++kk) {
      uint32_t pa[4], b[4];
      ldmatrix_x4_trans(b, smem_u32(&s.v[kk * 16 + (mi & 1) * 8 + r8][ch * 16 + (mi >> 1) * 8]));
      ldmatrix_x4(pa, smem_u32(&s.p_hi[rg * 16 + (mi & 1) * 8 + r8][kk * 16 + (mi >> 1) * 8]));
      mma2(o[0], pa, b[0], b[1]);
      mma2(o[1], pa, b[2], b[3]);
      ldmatrix_x4(pa, smem_u32(&s.p_lo[rg * 16 + (mi & 1) * 8 + r8][kk * 16 + (mi >> 1) * 8]));
      mma2(o[0], pa, b[0], b[1]);
      mma2(o[1], pa, b[2], b[3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = rg * 16 + (lane >> 2) + e * 8, c = v0 + ch * 16 + j * 8 + (lane & 3) * 2;
        if (r < n && c < a.dv)
          *reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.out) + static_cast<int64_t>(t0 + c0 + r) * a.ldo + h * a.dv + c) =
              pack_bf16x2(o[j][2 * e], o[j][2 * e + 1]);
      }
    const float dn = s.pow[n];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int tile = warp + i * kWarps, m0 = tile % kTilesK * 16, n0 = tile / kTilesK * 16;
      if (tile >= kTiles) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][j][e] *= dn;
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
  }
}

template <int DK>
int launch_chunk(const LightningArgs& a, int n, cudaStream_t stream) {
  constexpr int smem = sizeof(ChunkSmem<DK>);
  static bool done[64] = {false};
  const int dev = pxl_host::current_device_slot();
  if (!done[dev]) {
    if (cudaFuncSetAttribute(lightning_chunk_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return PXL_ERR_CUDA;
    done[dev] = true;
  }
  if (n > 65535) return PXL_ERR_TOO_LARGE;
  pxl_host::launch(lightning_chunk_kernel<DK>, dim3(ceil_div(a.dv, kVS), a.H, n), dim3(kWarps * 32), smem, stream, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}

inline bool chunkable(const LightningArgs& a) {
  return a.dk <= 256 && !((a.q_off | a.k_off | a.v_off | a.dk | a.dv | static_cast<int>(a.ld) | static_cast<int>(a.ldo)) & 7) &&
         ((reinterpret_cast<uintptr_t>(a.proj) | reinterpret_cast<uintptr_t>(a.out)) & 15) == 0;
}
}  // namespace

PXL_EXPORT int pxl_lightning_attn(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int dk, int dv,
                                  const float* decay_pow, int pow_len, float* state, int num_slots, const int* seq_cu,
                                  const int* seq_slots, const int* positions, void* out, int64_t ldo, int prefill_seqs,
                                  int decode_seqs, int is_f32, int* status, cudaStream_t stream) {
  if (H <= 0 || dk <= 0 || dv <= 0 || pow_len != kChunk + 1) return PXL_ERR_INVALID_ARG;
  const LightningArgs a{proj, ld, q_off, k_off, v_off, H, dk, dv, decay_pow, state, num_slots, seq_cu, seq_slots, positions,
                        out, ldo, status};
  int code = PXL_OK;
  if (prefill_seqs > 0) {
    if (is_f32) code = launch_recurrent<float>(a, 0, prefill_seqs, stream);
    else if (!chunkable(a)) code = launch_recurrent<pxl::bf16>(a, 0, prefill_seqs, stream);
    else if (dk <= 32) code = launch_chunk<32>(a, prefill_seqs, stream);
    else if (dk <= 64) code = launch_chunk<64>(a, prefill_seqs, stream);
    else if (dk <= 96) code = launch_chunk<96>(a, prefill_seqs, stream);
    else if (dk <= 128) code = launch_chunk<128>(a, prefill_seqs, stream);
    else code = launch_chunk<256>(a, prefill_seqs, stream);
  }
  if (code == PXL_OK && decode_seqs > 0)
    code = is_f32 ? launch_recurrent<float>(a, prefill_seqs, decode_seqs, stream)
                  : launch_recurrent<pxl::bf16>(a, prefill_seqs, decode_seqs, stream);
  return code;
}
