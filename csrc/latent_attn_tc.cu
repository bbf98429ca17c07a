// Latent attention on the 5th-generation tensor cores, prompts and decoding alike (bf16; see latent_attn.cu for
// the op). One kernel serves every size with L + R <= 576.
//
// A query row is a (token, head) pair: q [T, H, L + R] is a matrix of T * H rows that all read the same cached
// rows, so a CTA takes 128 consecutive rows of one sequence - 128 / H tokens (one token and a block of 128 heads
// when H > 128) - and walks the keys that its first and last token may see in tiles of 64.
//
//   warp 4    : TMA producer. The query tile once (chunks of 64 columns, 128-byte swizzle), then tiles of cache
//               rows (page boxes), chunk by chunk. A cache row is key AND value and is loaded once: the chunks this
//               CTA accumulates as values go to whole-tile V buffers, all others - needed for the scores only - to a
//               ring of chunk slots that are free again as soon as the scores have read them.
//   warp 5    : MMA issuer. S = Q K^T over L + R (both operands K-major) into one of two TMEM score buffers, chunk
//               by chunk as the loads land, so the scores of tile i + 1 are computed while the softmax warps work
//               on tile i; then O += P V, P from tensor memory, V taken MN-major from the V buffer, all of its
//               columns by one instruction per 16 keys (narrow instructions cost almost as much as wide ones).
//   warps 0-3 : softmax, one row per thread (its TMEM lane): mask (causal, window), running reference maximum
//               that only moves when a row grew by more than 2^8 (then the TMEM rows of O are rescaled), P
//               back to tensor memory as bf16 (two buffers), row sums in fp32; at the end the sink and the
//               division.
//
// O takes 64 TMEM columns per 64 latent columns and scores need room beside it, so a CTA accumulates at most 256
// latent columns; wider latents run as several CTAs per query tile that repeat the scores (L = 512: two). The host
// sizes the ring and the number of V buffers to what the query tile leaves of shared memory.
// Every wait is bounded; on expiry the kernel records a status code, all roles unwind, TMEM is freed.
#include "common.cuh"
#include "pxl_api.h"

namespace {
using namespace pxl;

constexpr int kRows = 128;
constexpr int kQChunk = kRows * 128;   // bytes of 64 columns of a full query tile
constexpr int kMaxV = 4;               // 64-column latent chunks a CTA accumulates
constexpr int NK = 64;                 // keys per tile
constexpr int kKvChunk = NK * 128;     // bytes of 64 columns of a key tile
constexpr int kMaxSlots = 16, kMaxVBufs = 3;
constexpr int kProducerWarp = 4, kMmaWarp = 5;
constexpr int kThreads = 192;
constexpr int kBarBytes = 512;
constexpr int kMaxSmem = 227 * 1024;
constexpr float kLog2eF = 1.4426950408889634f;

struct TcArgs {
  const int* block_tables;
  const int* cu_q;      // null: token i is the only query of sequence i
  const int* ctx_lens;
  bf16* out;            // [T, H, L]
  const float* sinks;
  int H, L, D, page, max_blocks, window, vsplit, head_blocks;
  int k_slots, v_bufs;  // ring slots for score-only chunks, buffers for value chunks
  int q_rows;           // rows of the query tile kept in shared memory (decoding: the heads of one token)
  int64_t num_blocks;
  float scale_log2;
  int* status;
};

// B stored as 64-column chunks of [key rows, 64]: MN-major, 8-row groups 1024 B apart, chunks kKvChunk apart
__device__ __forceinline__ uint64_t desc_mn_sw128(uint32_t addr) {
  return (umma_desc_k_sw128(addr) & ~(0x3fffull << 16)) | (static_cast<uint64_t>(kKvChunk >> 4) << 16);
}
__device__ __forceinline__ bool mbar_test(uint32_t bar, uint32_t parity) {  // never suspends, unlike mbar_try_wait
  uint32_t ok;
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t"
      "}\n"
      : "=r"(ok)
      : "r"(bar), "r"(parity)
      : "memory");
  return ok != 0;
}
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// The MMA and producer warps run their loops with all lanes, so that addresses and descriptors stay in uniform registers (a loop in one
// lane moves them there before every instruction and issues at half the rate); `leader` is non-zero in the lane
// that issues.
__device__ __forceinline__ uint32_t elect_leader() {
  uint32_t r;
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "elect.sync _|p, 0xffffffff;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t"
      "}\n"
      : "=r"(r));
  return r;
}
// D[tmem] (+)= A[smem desc] * B[smem desc]
__device__ __forceinline__ void mma_ss(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate,
                                       uint32_t leader) {
  asm volatile(
      "{\n\t"
      ".reg .pred p, q;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(leader)
      : "memory");
}
// D[tmem] (+)= A[tmem] * B[smem desc]; A holds two bf16 per 32-bit column, one row per lane
__device__ __forceinline__ void mma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate,
                                       uint32_t leader) {
  asm volatile(
      "{\n\t"
      ".reg .pred p, q;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(leader)
      : "memory");
}
__device__ __forceinline__ void tma_box(uint32_t smem_dst, const CUtensorMap* tmap, uint32_t bar, int x, int y,
                                        uint32_t leader) {
  asm volatile(
      "{\n\t"
      ".reg .pred q;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "@q cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];\n\t"
      "}\n"
      :
      : "r"(smem_dst), "l"(reinterpret_cast<uint64_t>(tmap)), "r"(bar), "r"(x), "r"(y), "r"(leader)
      : "memory");
}
__device__ __forceinline__ void commit(uint32_t bar, uint32_t leader) {
  asm volatile(
      "{\n\t"
      ".reg .pred q;\n\t"
      "setp.ne.b32 q, %1, 0;\n\t"
      "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t"
      "}\n"
      :
      : "r"(bar), "r"(leader)
      : "memory");
}
__device__ __forceinline__ void tmem_st_32x32b_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      :
      : "r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
        "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}

__global__ void __launch_bounds__(kThreads, 1)
latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv,
                      const TcArgs a) {
  constexpr uint32_t kIdescS = umma_idesc(kRows, NK, 1, 1);
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int nck = ceil_div(a.D, 64);
  // The MMA always reads 128 rows. With fewer in shared memory the rest are whatever follows (other chunks, the
  // key ring): those rows' scores are masked and their outputs never stored.
  const uint32_t q_chunk = a.q_rows * 128;
  const uint32_t sm_q = smem_u32(smem);
  // latent chunks of this CTA
  const int vs = blockIdx.x % a.vsplit, tile = blockIdx.x / a.vsplit;
  const int ncv = ceil_div(a.L, 64), per = ceil_div(ncv, a.vsplit);
  const int v0 = vs * per;
  const int nv = ncv - v0 < per ? ncv - v0 : per;
  const int nkc = nck - nv;                                   // chunks that only the scores read
  auto k_chunk = [&](int j) { return j < v0 ? j : j + nv; };  // their column chunks
  const uint32_t sm_v = sm_q + nck * q_chunk;
  const uint32_t sm_k = sm_v + a.v_bufs * per * kKvChunk;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + nck * q_chunk + (a.v_bufs * per + a.k_slots) * kKvChunk);
  // q_full | v_full, v_empty [kMaxVBufs] | k_full, k_empty [kMaxSlots] | s_full, p_ready, o_full [2]
  const uint32_t q_full = smem_u32(bars), v_full = q_full + 8, v_empty = v_full + 8 * kMaxVBufs,
                 k_full = v_empty + 8 * kMaxVBufs, k_empty = k_full + 8 * kMaxSlots, s_full = k_empty + 8 * kMaxSlots,
                 p_ready = s_full + 16, o_full = p_ready + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 1 + 2 * kMaxVBufs + 2 * kMaxSlots + 6);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  pdl_wait();
  pdl_launch_dependents();

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const int b = blockIdx.z, hb = blockIdx.y;
  const int t0 = a.cu_q ? a.cu_q[b] : b;
  const int len = a.cu_q ? a.cu_q[b + 1] - t0 : 1;
  const int ctx = a.ctx_lens[b];
  const int h0 = hb * kRows;
  const int heads = a.H - h0 < kRows ? a.H - h0 : kRows;  // heads per token of this tile
  const int tpt = a.H <= kRows ? kRows / a.H : 1;         // tokens per tile
  const int tok0 = tile * tpt;
  if (tok0 >= len) return;  // uniform for the CTA, before any barrier or allocation
  const int ntok = len - tok0 < tpt ? len - tok0 : tpt;
  const int rows = ntok * heads;
  const int64_t row0 = static_cast<int64_t>(t0 + tok0) * a.H + h0;  // row of q / out
  const int pos0 = ctx - len + tok0;
  const int hi = pos0 + ntok;  // keys [lo, hi) are visible to some row
  const int lo = (a.window > 0 && pos0 - a.window + 1 > 0) ? pos0 - a.window + 1 : 0;
  const int t_begin = lo / NK;
  const int n_tiles = __shfl_sync(0xffffffffu, ceil_div(hi, NK) - t_begin, 0);

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    mbar_init(q_full, 1);
    for (int s = 0; s < a.v_bufs; ++s) {
      mbar_init(v_full + 8 * s, 1);
      mbar_init(v_empty + 8 * s, 1);
    }
    for (int s = 0; s < a.k_slots; ++s) {
      mbar_init(k_full + 8 * s, 1);
      mbar_init(k_empty + 8 * s, 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(s_full + 8 * s, 1);
      mbar_init(p_ready + 8 * s, 4);  // one arrival per softmax warp
      mbar_init(o_full + 8 * s, 1);
    }
    mbar_fence_init();
    fence_proxy_async_smem();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_kv);
  }
  const uint32_t tmem_cols = 64 * per + 3 * NK <= 256 ? 256 : 512;  // O | two score | two probability buffers
  if (warp == kMmaWarp) {
    tmem_alloc(smem_u32(tmem_slot), tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tm_o = *tmem_slot;             // O: 64 columns per latent chunk
  const uint32_t tm_s = tm_o + 64 * per;        // two score buffers of NK columns
  const uint32_t tm_p = tm_s + 2 * NK;          // two probability buffers of NK / 2 columns

  if (warp == kProducerWarp) {
    // ------------------------------------------------------------------ TMA producer
    // Lane p looks up the block of piece p of the tile; one lane issues all boxes.
    const uint32_t leader = elect_leader();
    if (leader) mbar_arrive_expect_tx(q_full, nck * q_chunk);
    __syncwarp();
    for (int c = 0; c < nck; ++c) tma_box(sm_q + c * q_chunk, &tm_q, q_full, c * 64, static_cast<int>(row0), leader);
    const int* bt = a.block_tables + static_cast<int64_t>(b) * a.max_blocks;
    const int box = a.page < NK ? a.page : NK;
    const int pieces = NK / box;
    bool ok = true;
    // wait for the buffer behind `bar_empty` to be free again (its `use`-th use), announce `bytes`
    auto acquire = [&](uint32_t bar_empty, uint32_t bar_full, int use, uint32_t bytes) {
      bool free = true;
      if (use > 0)
        free = __all_sync(0xffffffffu, mbar_wait_bounded(bar_empty, (use - 1) & 1, abort_flag, a.status, PXL_DEV_TIMEOUT_EMPTY));
      if (free && leader) mbar_arrive_expect_tx(bar_full, bytes);
      __syncwarp();
      return free;
    };
    auto tile_row = [&](int it) {  // cache row of this lane's piece of tile `it`
      int row = 0;
      if (lane < pieces && it < n_tiles) {
        int key = (t_begin + it) * NK + lane * box;
        if (key >= ctx) key = (ctx - 1) / box * box;  // beyond the context: re-read its last piece (masked)
        const int bi = key / a.page;
        int64_t blk = bi < a.max_blocks ? bt[bi] : -1;
        if (blk < 0 || blk >= a.num_blocks) {
          if (a.status) atomicCAS(a.status, 0, PXL_DEV_BAD_BLOCK_PREFILL);
          blk = 0;
        }
        row = static_cast<int>(blk * a.page + key % a.page);
      }
      return row;
    };
    int slot = 0, slot_use = 0, vb = 0, vb_use = 0;
    int row = tile_row(0);
    for (int it = 0; ok && it < n_tiles; ++it) {
      const int next_row = tile_row(it + 1);  // its table reads are in flight while this tile is issued
      for (int j = 0; ok && j < nkc; ++j) {
        ok = acquire(k_empty + 8 * slot, k_full + 8 * slot, slot_use, kKvChunk);
        if (ok)
          for (int p = 0; p < pieces; ++p)
            tma_box(sm_k + slot * kKvChunk + p * box * 128, &tm_kv, k_full + 8 * slot, k_chunk(j) * 64,
                    __shfl_sync(0xffffffffu, row, p), leader);
        if (++slot == a.k_slots) {
          slot = 0;
          ++slot_use;
        }
      }
      if (!ok) break;
      ok = acquire(v_empty + 8 * vb, v_full + 8 * vb, vb_use, nv * kKvChunk);
      if (ok)
        for (int p = 0; p < pieces; ++p) {
          const int r = __shfl_sync(0xffffffffu, row, p);
          for (int c = 0; c < nv; ++c)
            tma_box(sm_v + (vb * per + c) * kKvChunk + p * box * 128, &tm_kv, v_full + 8 * vb, (v0 + c) * 64, r, leader);
        }
      if (++vb == a.v_bufs) {
        vb = 0;
        ++vb_use;
      }
      row = next_row;
    }
  } else if (warp == kMmaWarp) {
    // ------------------------------------------------------------------ MMA issuer
    {
      const uint32_t leader = elect_leader();
      const uint32_t idesc_pv = umma_idesc(kRows, 64 * nv, 1, 1) | (1u << 16);  // B (V) is MN-major
      const uint64_t dq0 = umma_desc_k_sw128(sm_q);
      // descriptors advance by 16-byte units: 2 per k-step inside a chunk (columns past D are zeros on both sides)
      auto ready = [](uint32_t bar, uint32_t parity) { return __all_sync(0xffffffffu, mbar_test(bar, parity)) != 0; };
      auto s_chunk = [&](int it, int col_chunk, uint32_t rows_addr, bool first) {  // S[it % 2] (+)= Q[:, chunk] K[:, chunk]^T
        const uint64_t dq = dq0 + static_cast<uint64_t>(col_chunk) * (q_chunk >> 4), dk = umma_desc_k_sw128(rows_addr);
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)
          mma_ss(tm_s + (it & 1) * NK, dq + 2 * ks, dk + 2 * ks, kIdescS, first && ks == 0 ? 0u : 1u, leader);
      };
      // Whichever is ready goes next: the product of a tile whose probabilities are written, or the next chunk of the
      // scores (at most one tile ahead of the products: two score buffers). A load in flight never holds back a
      // product, which is what frees the buffers for the loads after it.
      bool ok = __all_sync(0xffffffffu, mbar_wait_bounded(q_full, 0, abort_flag, a.status, PXL_DEV_TIMEOUT_FULL));
      int next_s = 0, next_pv = 0;   // tiles whose scores / products come next
      int j = 0, slot = 0, slot_phase = 0;  // score-only chunk of tile next_s and its ring slot
      int s_vb = 0, s_vb_phase = 0, pv_vb = 0;
      uint64_t since = 0;
      uint32_t spins = 0;
      while (ok && next_pv < n_tiles) {
        bool moved = false;
        if (next_s < n_tiles && next_s <= next_pv + 1) {
          while (j < nkc && ready(k_full + 8 * slot, slot_phase)) {
            tc_fence_after_sync();
            s_chunk(next_s, k_chunk(j), sm_k + slot * kKvChunk, j == 0);
            commit(k_empty + 8 * slot, leader);  // free again once these have read it
            ++j;
            if (++slot == a.k_slots) {
              slot = 0;
              slot_phase ^= 1;
            }
            moved = true;
          }
          if (j == nkc && ready(v_full + 8 * s_vb, s_vb_phase)) {
            tc_fence_after_sync();
            const uint32_t v = sm_v + s_vb * per * kKvChunk;
            for (int c = 0; c < nv; ++c) s_chunk(next_s, v0 + c, v + c * kKvChunk, nkc == 0 && c == 0);
            commit(s_full + 8 * (next_s & 1), leader);
            ++next_s;
            j = 0;
            if (++s_vb == a.v_bufs) {
              s_vb = 0;
              s_vb_phase ^= 1;
            }
            moved = true;
          }
        }
        if (next_pv < next_s && ready(p_ready + 8 * (next_pv & 1), (next_pv >> 1) & 1)) {  // O += P V
          tc_fence_after_sync();
          const uint64_t dv = desc_mn_sw128(sm_v + pv_vb * per * kKvChunk);
          const uint32_t p = tm_p + (next_pv & 1) * (NK / 2);
#pragma unroll
          for (int ks = 0; ks < NK / 16; ++ks)
            mma_ts(tm_o, p + ks * 8, dv + 128 * ks, idesc_pv, (next_pv > 0 || ks > 0) ? 1u : 0u, leader);
          commit(o_full + 8 * (next_pv & 1), leader);
          commit(v_empty + 8 * pv_vb, leader);
          ++next_pv;
          if (++pv_vb == a.v_bufs) pv_vb = 0;
          moved = true;
        }
        if (moved) {
          spins = 0;
          since = 0;
        } else if ((++spins & 0x3ffu) == 0) {
          const uint64_t now = global_timer_ns();
          if (since == 0) since = now;
          const bool late = now - since > kWaitLimitNs;
          if (late && leader) {
            *abort_flag = 1;
            if (a.status) atomicCAS(a.status, 0, PXL_DEV_TIMEOUT_TMEM_EMPTY);
          }
          ok = __all_sync(0xffffffffu, !late && !*abort_flag);
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax warps
    const int r = warp * 32 + lane;  // query row = TMEM lane
    const int pos = pos0 + r / heads, head = h0 + r % heads;
    const bool row_valid = r < rows;
    const int key_lo = (a.window > 0 && pos - a.window + 1 > 0) ? pos - a.window + 1 : 0;
    const int key_hi = row_valid ? pos + 1 : 0;
    const uint32_t lane_sel = static_cast<uint32_t>(warp * 32) << 16;
    float m_run = -INFINITY, l_run = 0.f;
    int failed = 0;
    for (int it = 0; it < n_tiles; ++it) {
      const int par = it & 1;
      failed = mbar_wait_bounded(s_full + 8 * par, (it >> 1) & 1, abort_flag, a.status, PXL_DEV_TIMEOUT_TMEM_FULL) ? 0 : 1;
      failed = __any_sync(0xffffffffu, failed);  // warp-uniform: the TMEM accesses below are warp-wide
      if (failed) break;
      tc_fence_after_sync();
      uint32_t sc[NK];
#pragma unroll
      for (int c = 0; c < NK; c += 32)
        tmem_ld_32x32b_x32(tm_s + par * NK + c + lane_sel, *reinterpret_cast<uint32_t(*)[32]>(&sc[c]));
      tmem_ld_wait();
      const int key0 = (t_begin + it) * NK;
      const int ma = key_lo - key0, me = key_hi - key0;  // this row sees columns [ma, me)
      if (!__all_sync(0xffffffffu, ma <= 0 && me >= NK)) {
#pragma unroll
        for (int j = 0; j < NK; ++j)
          if (j < ma || j >= me) sc[j] = 0xff800000u;  // -inf
      }
      float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < NK; j += 4) {
#pragma unroll
        for (int k = 0; k < 4; ++k) m4[k] = fmaxf(m4[k], __uint_as_float(sc[j + k]));
      }
      const float m_new = fmaxf(m_run, fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * a.scale_log2);  // scale > 0
      if (it == 0) {
        m_run = m_new;
      } else if (__any_sync(0xffffffffu, m_new > m_run + 8.f)) {
        // O accumulates relative to m_run: move the reference and rescale, once O of the tile before is complete
        failed = mbar_wait_bounded(o_full + 8 * (par ^ 1), ((it - 1) >> 1) & 1, abort_flag, a.status,
                                   PXL_DEV_TIMEOUT_TMEM_FULL) ? 0 : 1;
        failed = __any_sync(0xffffffffu, failed);
        if (failed) break;
        const float corr = fast_exp2(m_run - (m_new == -INFINITY ? 0.f : m_new));
        m_run = m_new;
        l_run *= corr;
        tc_fence_after_sync();
        for (int c = 0; c < nv * 64; c += 32) {
          uint32_t v[32];
          tmem_ld_32x32b_x32(tm_o + lane_sel + c, v);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(__uint_as_float(v[j]) * corr);
          tmem_st_32x32b_x32(tm_o + lane_sel + c, v);
        }
        tmem_st_wait();
      }
      const float m_use = (m_run == -INFINITY) ? 0.f : m_run;
      // the P buffer was last read by the product of tile it - 2
      if (it >= 2) {
        failed = mbar_wait_bounded(o_full + 8 * par, ((it - 2) >> 1) & 1, abort_flag, a.status, PXL_DEV_TIMEOUT_TMEM_FULL) ? 0 : 1;
        failed = __any_sync(0xffffffffu, failed);
        if (failed) break;
        tc_fence_after_sync();
      }
      float sum2[2] = {0.f, 0.f};
      uint32_t pk[NK / 2];
#pragma unroll
      for (int j = 0; j < NK; j += 2) {
        const float p0 = fast_exp2(fmaf(__uint_as_float(sc[j]), a.scale_log2, -m_use));
        const float p1 = fast_exp2(fmaf(__uint_as_float(sc[j + 1]), a.scale_log2, -m_use));
        sum2[0] += p0;
        sum2[1] += p1;
        pk[j >> 1] = pack_bf16x2(p0, p1);
      }
      l_run += sum2[0] + sum2[1];
#pragma unroll
      for (int c = 0; c < NK / 2; c += 16)
        tmem_st_32x32b_x16(tm_p + par * (NK / 2) + c + lane_sel, *reinterpret_cast<uint32_t(*)[16]>(&pk[c]));
      tmem_st_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready + 8 * par);
    }
    if (!failed)
      failed = mbar_wait_bounded(o_full + 8 * ((n_tiles - 1) & 1), ((n_tiles - 1) >> 1) & 1, abort_flag, a.status,
                                 PXL_DEV_TIMEOUT_TMEM_FULL) ? 0 : 1;
    failed = __any_sync(0xffffffffu, failed);
    if (!failed) {
      float denom = l_run, f = 1.f;
      if (a.sinks && row_valid) {
        const float sink = a.sinks[head] * kLog2eF;
        const float M = fmaxf(m_run, sink);
        f = exp2f(m_run - M);
        denom = denom * f + exp2f(sink - M);
      }
      const float inv = denom > 0.f ? f / denom : 0.f;
      bf16* dst = a.out + (row0 + r) * a.L + v0 * 64;
      const int ncol = a.L - v0 * 64 < nv * 64 ? a.L - v0 * 64 : nv * 64;
      tc_fence_after_sync();
      for (int c = 0; c < nv * 64; c += 32) {
        uint32_t v[32];
        tmem_ld_32x32b_x32(tm_o + lane_sel + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int c8 = 0; c8 < 32; c8 += 8) {
          bf16x8 ov;
#pragma unroll
          for (int j = 0; j < 4; ++j)
            ov.u[j] = pack_bf16x2(__uint_as_float(v[c8 + 2 * j]) * inv, __uint_as_float(v[c8 + 2 * j + 1]) * inv);
          if (row_valid && c + c8 < ncol) st_bf16x8(dst + c + c8, ov);
        }
      }
      tc_fence_before_sync();
    }
  }

  // ---------------------------------------------------------------------- teardown
  __syncwarp();
  if (*abort_flag) __nanosleep(200000);  // loads that are still in flight must land before smem is released
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == kMmaWarp) tmem_dealloc(tm_o, tmem_cols);
}

struct TilePlan {
  int k_slots, v_bufs, smem;
};

// Ring slots and V buffers beside a query tile of q_rows rows; false when the sizes do not fit.
bool plan_tiles(int L, int D, int q_rows, int page, TilePlan* p) {
  if (page % 8 != 0 || (page % NK != 0 && NK % page != 0)) return false;
  const int nck = ceil_div(D, 64), ncv = ceil_div(L, 64);
  const int vsplit = ceil_div(ncv, kMaxV), per = ceil_div(ncv, vsplit);
  const int nkc = nck - (ncv - (vsplit - 1) * per);  // score-only chunks of the CTA that has most of them
  const int q_bytes = nck * q_rows * 128;
  const int slots = (kMaxSmem - 1024 - kBarBytes - q_bytes) / kKvChunk;
  p->k_slots = 0;
  for (int vb = kMaxVBufs; vb >= 1; --vb) {
    const int ks = slots - vb * per;
    if (ks >= (vb > 1 ? nkc + 1 : (nkc > 0 ? 1 : 0))) {
      p->v_bufs = vb;
      p->k_slots = ks < kMaxSlots ? ks : kMaxSlots;
      if (p->k_slots < 1) p->k_slots = 1;
      const int tiles = q_bytes + (vb * per + p->k_slots) * kKvChunk;
      const int reach = (nck - 1) * q_rows * 128 + kQChunk;  // what the MMA reads of the query tile
      p->smem = 1024 + (tiles > reach ? tiles : reach) + kBarBytes;
      return p->smem <= kMaxSmem;
    }
  }
  return false;
}
}  // namespace

PXL_EXPORT int pxl_latent_attn_tc_supported(int L, int R, int page, float scale) {
  TilePlan plan;
  return L > 0 && R >= 0 && L % 8 == 0 && R % 8 == 0 && page > 0 && page % 8 == 0 && scale > 0.f &&
         plan_tiles(L, L + R, kRows, page, &plan);
}

PXL_EXPORT int pxl_latent_attn_tc(const void* q, const void* cache, const int* block_tables, const int* cu_q,
                                  const int* ctx_lens, void* out, const float* sinks, int B, int max_q, int total_q, int H,
                                  int L, int R, int page, int max_blocks, int64_t num_blocks, float scale, int window,
                                  int* status, cudaStream_t stream) {
  if (B <= 0 || max_q <= 0 || total_q <= 0) return PXL_OK;
  if (H <= 0 || B > 65535 || !pxl_latent_attn_tc_supported(L, R, page, scale)) return PXL_ERR_INVALID_ARG;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15)
    return PXL_ERR_INVALID_ARG;
  if (num_blocks * page >= (1ll << 31) || static_cast<int64_t>(total_q) * H >= (1ll << 31)) return PXL_ERR_TOO_LARGE;
  TcArgs a{};
  TilePlan plan;
  // short queries (decoding) leave most of the tile's rows empty: keep only the others, and more keys in flight
  const int rows = max_q * (H < kRows ? H : kRows);
  a.q_rows = rows >= kRows ? kRows : pxl::ceil_div(rows, 8) * 8;
  if (!plan_tiles(L, L + R, a.q_rows, page, &plan)) return PXL_ERR_INVALID_ARG;
  a.k_slots = plan.k_slots;
  a.v_bufs = plan.v_bufs;
  a.block_tables = block_tables;
  a.cu_q = cu_q;
  a.ctx_lens = ctx_lens;
  a.out = static_cast<pxl::bf16*>(out);
  a.sinks = sinks;
  a.H = H, a.L = L, a.D = L + R, a.page = page, a.max_blocks = max_blocks, a.window = window, a.num_blocks = num_blocks;
  a.vsplit = pxl::ceil_div(pxl::ceil_div(L, 64), kMaxV);
  a.head_blocks = pxl::ceil_div(H, kRows);
  a.scale_log2 = scale * kLog2eF;
  a.status = status;
  CUtensorMap tq, tkv;
  if (!pxl_host::make_tmap_2d(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, q, static_cast<uint64_t>(total_q) * H, a.D, a.D,
                              a.q_rows, 64) ||
      !pxl_host::make_tmap_2d(&tkv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, cache, static_cast<uint64_t>(num_blocks) * page, a.D,
                              a.D, page < NK ? page : NK, 64))
    return PXL_ERR_TENSORMAP;
  const int tpt = H <= kRows ? kRows / H : 1;
  const dim3 grid(pxl::ceil_div(max_q, tpt) * a.vsplit, a.head_blocks, B);
  static bool configured[64] = {false};
  const int dev = pxl_host::current_device_slot();
  if (!configured[dev]) {
    if (cudaFuncSetAttribute(latent_attn_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem) != cudaSuccess)
      return PXL_ERR_CUDA;
    configured[dev] = true;
  }
  pxl_host::launch(latent_attn_tc_kernel, grid, dim3(kThreads), plan.smem, stream, tq, tkv, a);
  return cudaGetLastError() == cudaSuccess ? PXL_OK : PXL_ERR_CUDA;
}
