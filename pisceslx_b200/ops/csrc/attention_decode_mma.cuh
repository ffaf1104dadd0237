// Paged-KV decode attention on the tensor cores (heads of up to 128 numbers, up to 16 query heads per CTA).
//
// A decode step has G = hq / hk real query rows per KV head, far below the 128-row UMMA tile, but the op is bound by
// the K/V bytes, not by FLOPs: padding the query-head dimension to N = 16 costs tensor-core time that stays well
// under the time the bytes take to arrive, and it removes the 2 * G * D fp32 FMAs per key that bound the CUDA-core
// kernels.  Keys are the M dimension:
//
//   S^T[128 keys, 16 heads]   = K_tile[128 keys, dim] * Qpad[16, dim]^T          (SS, K-major operands)
//   O^T[128 dims, 16 heads]  += V_tile^T[vdim, 128 keys] * P[16 heads, 128 keys]^T   (SS, A MN-major = V as stored)
//
// dim and vdim are any multiples of 8 up to 64 NB (slabs of 64 columns; the copies zero-fill a slab past the size).  With
// one slab the second 64 rows of the V operand are whatever lies behind the slab (the stage's K tile): those lanes of O^T
// are never read.
//
// grid = (kv heads x chunks of G query heads, sequences, splits), 224 threads; three K/V stages, one CTA per SM with
// two slabs and two with one:
//   warps 0..3  softmax: thread t owns key t of the tile (TMEM lane t of S^T) and output dimension t (lane t of O^T);
//               the reference maximum per head is kept identically by every thread, the running sum per thread
//   warp 4      one lane issues S^T, up to two tiles ahead of the softmax (two TMEM buffers)
//   warp 5      one lane issues the P V product (two P buffers), which also frees the tile's stage
//   warp 6      one lane issues the TMA copies of the K/V ring (a tile is two cache blocks of 64 tokens, 128B swizzle)
// The issuing is spread over three warps because a tile is short: neither a copy that has not landed nor the descriptor
// arithmetic of one product may hold up the other.  Hand-offs are mbarriers, one per buffer, so that no barrier can run
// two phases ahead of a waiter.  The softmax warps meet at ONE named barrier per tile, which asks whether any score
// exceeds its reference maximum by 2^8; maxima are exchanged and O^T is rescaled only then.
// Output: with one split the normalised heads (with an optional sink in the denominator and an optional sigmoid gate),
// otherwise an unnormalised partial (max, sum, out) per query head and split, merged by another kernel.
#pragma once
#include "per_device.h"
#include "sm100.cuh"
#include "tensormap.h"

namespace yv {

struct PagedDecodeMmaParams {
  CUtensorMap tma_k;               // 3-D (dim, kv head, token slot), box (64, 1, 64), 128B swizzle
  CUtensorMap tma_v;               // 3-D (vdim, kv head, token slot)
  const __nv_bfloat16* q;          // row b at q + b * q_ld, head h at h * dim
  int64_t q_ld;
  __nv_bfloat16* o;                // row b at o + b * o_ld, head h at h * vdim (one split)
  int64_t o_ld;
  const __nv_bfloat16* sink;       // [hq] logits, null = none
  const __nv_bfloat16* gate;       // logits, row b at gate + b * gate_ld, head h at h * gate_step (1 or vdim numbers)
  int64_t gate_ld;
  int gate_step;
  float* partial_o;                // [B, hq, splits, vdim]
  float* partial_ml;               // [B, hq, splits, 2]
  const int* block_table;          // [B, max_blocks_per_seq]
  const int* seq_lens;             // [B]
  int hq, group, chunks;           // query heads, query heads per kv head, CTAs per kv head
  int dim, vdim, max_blocks_per_seq, splits, num_blocks;
  float scale_log2;
  uint32_t* status;
};

constexpr int kDmStages = 3;
constexpr int kDmTileKeys = 128;
constexpr int kDmBlock = 64;                                // tokens per cache block
constexpr int kDmThreads = 224;
constexpr int kDmSlab = kDmTileKeys * 128;                  // [128 keys][64 columns] bf16
constexpr int kDmPBytes = 2 * 16 * 128;                     // one P buffer [16 heads][128 keys] as two 64-key slabs
constexpr float kDmLog2e = 1.4426950408889634f;

template <int NB>
struct DecodeMmaSmem {
  static constexpr int kTile = NB * kDmSlab;                // K (or V) tile
  static constexpr int kStage = 2 * kTile;                  // V, then K
  static constexpr int kQ = NB * 16 * 128;                  // Qpad [16][64 NB] in slabs of 64 columns
  static constexpr int kTotal = kDmStages * kStage + kQ + 2 * kDmPBytes + 1024;
};

// byte offset of element (row, col) in a K-major 128B-swizzled slab of 64 columns (rows of 128 bytes)
__device__ __forceinline__ uint32_t sw128_off(int row, int col) {
  return static_cast<uint32_t>(row * 128 + ((((col >> 3) ^ (row & 7)) << 4) | ((col & 7) << 1)));
}

// Barrier over the 128 softmax threads with an OR reduction of `v`.  The instruction is warp-aligned: lanes that left a
// bounded wait at different times are brought together first.
__device__ __forceinline__ bool softmax_barrier_or(bool v) {
  uint32_t any;
  __syncwarp();
  asm volatile(
      "{\n"
      ".reg .pred pin, pout;\n"
      "setp.ne.u32 pin, %1, 0;\n"
      "bar.red.or.pred pout, 1, 128, pin;\n"
      "selp.u32 %0, 1, 0, pout;\n"
      "}\n"
      : "=r"(any)
      : "r"(static_cast<uint32_t>(v))
      : "memory");
  return any != 0u;
}

__device__ __forceinline__ float dm_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int G, int NB>
__global__ void __launch_bounds__(kDmThreads, NB == 1 && G < 16 ? 2 : 1) paged_decode_mma_kernel(const __grid_constant__ PagedDecodeMmaParams p) {
  using S = DecodeMmaSmem<NB>;
  constexpr uint32_t kIdescQK = make_idesc_bf16(128, 16, false, false);
  constexpr uint32_t kIdescPV = make_idesc_bf16(128, 16, true, false);
  constexpr int kTableCap = 512;
  extern __shared__ uint8_t dsm_raw[];
  uint8_t* dsm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(dsm_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = dsm + kDmStages * S::kStage;
  uint8_t* sP = sQ + S::kQ;
  __shared__ uint64_t full_bar[kDmStages], empty_bar[kDmStages];
  __shared__ uint64_t s_bar[2], pv_bar[2], p_bar[2];
  __shared__ uint32_t tmem_slot;
  __shared__ float s_red[4][G];
  __shared__ int s_table[kTableCap];

  const int kvh = blockIdx.x / p.chunks, chunk = blockIdx.x % p.chunks, b = blockIdx.y, split = blockIdx.z;
  const int h0 = kvh * p.group + chunk * G;                               // first query head of this CTA
  const int heads = min(G, p.group - chunk * G);
  const int tid = threadIdx.x, lane = tid & 31;
  const int warp = __shfl_sync(0xFFFFFFFFu, tid >> 5, 0);                 // known to be uniform
  int seq_len = p.seq_lens[b];
  if (seq_len < 0 || seq_len > static_cast<int64_t>(p.max_blocks_per_seq) * kDmBlock) {   // reported and cut to the row
    if (tid == 0 && p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
    seq_len = seq_len < 0 ? 0 : p.max_blocks_per_seq * kDmBlock;
  }
  const int n_blocks = (seq_len + kDmBlock - 1) / kDmBlock;
  const int blocks_per_split = (n_blocks + p.splits - 1) / p.splits;
  const int blk0 = split * blocks_per_split;
  const int blk1 = min(n_blocks, blk0 + blocks_per_split);
  const int n_tiles = blk1 > blk0 ? (blk1 - blk0 + 1) / 2 : 0;
  // The block-table entries of this split are staged in shared memory once: the per-tile look-ups would otherwise be
  // dependent global loads on the tile chain.
  const int* gtable = p.block_table + static_cast<int64_t>(b) * p.max_blocks_per_seq;
  const bool staged = (blk1 - blk0) <= kTableCap;
  if (staged)
    for (int i = tid; i < blk1 - blk0; i += kDmThreads) s_table[i] = gtable[blk0 + i];
  const int* table = staged ? (s_table - blk0) : gtable;          // indexed by absolute block number either way

  if (tid == 0) {
    tma_prefetch_desc(&p.tma_k);
    tma_prefetch_desc(&p.tma_v);
    for (int s = 0; s < kDmStages; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&s_bar[i], 1); mbar_init(&pv_bar[i], 1); mbar_init(&p_bar[i], 128); }
    fence_barrier_init();
  }
  if (warp == 0) {
    tmem_alloc(&tmem_slot, 64);
    tmem_relinquish();
  }
  // Qpad: heads and columns that do not exist are zero.  P: rows >= G stay zero for the whole kernel.
  for (int i = tid; i < NB * 16 * 8; i += kDmThreads) {
    const int v = i & 7, g = (i >> 3) & 15, c = i >> 7, col = c * 64 + v * 8;
    uint4 val = make_uint4(0, 0, 0, 0);
    if (g < heads && col < p.dim)
      val = *reinterpret_cast<const uint4*>(p.q + b * p.q_ld + static_cast<int64_t>(h0 + g) * p.dim + col);
    *reinterpret_cast<uint4*>(sQ + c * 2048 + g * 128 + ((v ^ (g & 7)) << 4)) = val;
  }
  for (int i = tid; i < 2 * kDmPBytes / 16; i += kDmThreads) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = tmem_slot;
  const uint32_t tS = tmem_base, tO = tmem_base + 32u;      // S^T buffers at columns 0 and 16, O^T at 32

  // tile j = cache blocks blk0 + 2j (and + 1 when it exists); an out-of-range table entry is reported and its
  // half of the tile is treated as empty
  auto block_ok = [&](int blk) { const int ph = table[blk]; return ph >= 0 && ph < p.num_blocks; };

  // descriptors differ in their address field only (the low word): base + byte offset / 16
  const uint32_t hi_desc = static_cast<uint32_t>(make_smem_desc(0, 16, 1024) >> 32);
  const uint32_t lo_k = static_cast<uint32_t>(make_smem_desc(0, 16, 1024)), lo_mn = static_cast<uint32_t>(make_smem_desc(0, kDmSlab, 1024));
  auto desc = [&](uint32_t lo) { return (static_cast<uint64_t>(hi_desc) << 32) | lo; };
  const uint32_t stage0 = smem_u32(dsm) >> 4;

  if (warp == 6) {
    // ------------------------------------ TMA producer ---------------------------------------
    if (elect_one()) {
      const int slabs_k = (p.dim + 63) / 64, slabs_v = (p.vdim + 63) / 64;
      int s = 0;
      for (int j = 0; j < n_tiles; ++j) {
        if (j >= kDmStages && !mbar_wait(&empty_bar[s], (j / kDmStages - 1) & 1u, p.status)) break;
        uint8_t* sv = dsm + static_cast<size_t>(s) * S::kStage;
        uint8_t* sk = sv + S::kTile;
        int slot[2];
        uint32_t halves = 0;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int blk = blk0 + 2 * j + h;
          slot[h] = -1;
          if (blk < blk1) {
            if (block_ok(blk)) { slot[h] = table[blk] * kDmBlock; ++halves; }
            else if (p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
          }
        }
        if (halves == 0) {
          mbar_arrive(&full_bar[s]);
        } else {
          mbar_expect_tx(&full_bar[s], halves * static_cast<uint32_t>(slabs_k + slabs_v) * (kDmSlab / 2));
#pragma unroll
          for (int c = 0; c < NB; ++c)
#pragma unroll
            for (int h = 0; h < 2; ++h)
              if (slot[h] >= 0 && c < slabs_k) tma_load_3d(sk + c * kDmSlab + h * (kDmSlab / 2), &p.tma_k, &full_bar[s], c * 64, kvh, slot[h]);
#pragma unroll
          for (int c = 0; c < NB; ++c)
#pragma unroll
            for (int h = 0; h < 2; ++h)
              if (slot[h] >= 0 && c < slabs_v) tma_load_3d(sv + c * kDmSlab + h * (kDmSlab / 2), &p.tma_v, &full_bar[s], c * 64, kvh, slot[h]);
        }
        if (++s == kDmStages) s = 0;
      }
    }
  } else if (warp == 4) {
    // ------------------------------------ S^T issuer -----------------------------------------
    if (elect_one()) {
      const int steps = (p.dim + 15) / 16;
      const uint32_t dQ = lo_k + (smem_u32(sQ) >> 4);
      int s = 0;
      for (int j = 0; j < n_tiles; ++j) {
        // the buffer was last read for tile j - 2, whose weights have been reported
        if (j >= 2 && !mbar_wait(&p_bar[j & 1], ((j - 2) >> 1) & 1u, p.status)) break;
        if (!mbar_wait(&full_bar[s], (j / kDmStages) & 1u, p.status)) break;
        tc_fence_after_sync();
        const uint32_t dK = lo_k + stage0 + static_cast<uint32_t>((s * S::kStage + S::kTile) >> 4);
        const uint32_t dS = tS + static_cast<uint32_t>((j & 1) * 16);
#pragma unroll
        for (int kk = 0; kk < NB * 4; ++kk)
          if (kk < steps)
            tc_mma_f16_ss(dS, desc(dK + ((kk / 4) * kDmSlab + (kk % 4) * 32) / 16), desc(dQ + ((kk / 4) * 2048 + (kk % 4) * 32) / 16),
                          kIdescQK, kk != 0 ? 1u : 0u);
        tc_commit(&s_bar[j & 1]);
        if (++s == kDmStages) s = 0;
      }
    }
  } else if (warp == 5) {
    // ------------------------------------ P V issuer -----------------------------------------
    if (elect_one()) {
      const uint32_t dP0 = lo_k + (smem_u32(sP) >> 4);
      int s = 0;
      for (int j = 0; j < n_tiles; ++j) {
        if (!mbar_wait(&full_bar[s], (j / kDmStages) & 1u, p.status)) break;
        if (!mbar_wait(&p_bar[j & 1], (j >> 1) & 1u, p.status)) break;   // P(j), the V fix-ups, all reads of S^T(j)
        tc_fence_after_sync();
        const uint32_t dV = lo_mn + stage0 + static_cast<uint32_t>((s * S::kStage) >> 4);
        const uint32_t dP = dP0 + static_cast<uint32_t>((j & 1) * (kDmPBytes >> 4));
#pragma unroll
        for (int kk = 0; kk < kDmTileKeys / 16; ++kk)
          tc_mma_f16_ss(tO, desc(dV + kk * (2048 / 16)), desc(dP + ((kk / 4) * 2048 + (kk % 4) * 32) / 16), kIdescPV,
                        (j | kk) != 0 ? 1u : 0u);
        tc_commit(&pv_bar[j & 1]);
        tc_commit(&empty_bar[s]);
        if (++s == kDmStages) s = 0;
      }
    }
  } else {
    // ------------------------------------ softmax --------------------------------------------
    const uint32_t lane_off = static_cast<uint32_t>(warp * 32) << 16;
    float m_run[G], l_run[G];
#pragma unroll
    for (int g = 0; g < G; ++g) { m_run[g] = -1.0e29f; l_run[g] = 0.f; }
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      uint8_t* sv = dsm + static_cast<size_t>(j % kDmStages) * S::kStage;
      // keys of this tile that exist: whole blocks except the last one of the sequence
      int n_keys = 0;
      for (int h = 0; h < 2; ++h) {
        const int blk = blk0 + 2 * j + h;
        if (blk < blk1) n_keys = h * 64 + (block_ok(blk) ? min(64, seq_len - blk * 64) : 0);
      }
      const bool first_half_ok = block_ok(blk0 + 2 * j);
      const bool exists = tid < n_keys && (tid >= 64 || first_half_ok);
      ok = ok && mbar_wait(&s_bar[j & 1], (j >> 1) & 1u, p.status);
      ok = __all_sync(0xFFFFFFFFu, ok);              // the aligned tcgen05 instructions below need warp-uniform flow
      // scores of my key for the G heads (log2 domain); keys that do not exist are masked
      float sc[G];
      bool high = false;
      if (ok) {
        tc_fence_after_sync();
        uint32_t r[16];
        tmem_ld16(tS + static_cast<uint32_t>((j & 1) * 16) + lane_off, r);
        tc_wait_ld();
#pragma unroll
        for (int g = 0; g < G; ++g) {
          sc[g] = exists ? __uint_as_float(r[g]) * p.scale_log2 : -1.0e30f;
          high |= sc[g] > m_run[g] + 8.f;
        }
      } else {
#pragma unroll
        for (int g = 0; g < G; ++g) sc[g] = -1.0e30f;
      }
      tc_fence_before_sync();
      // lazy: the reference maximum moves only when a score exceeds it by more than 2^8, so most tiles leave the
      // accumulator alone (p <= 256 stays exact enough in bf16; the final division uses the same reference)
      const bool moves = softmax_barrier_or(high || !ok);
      float alpha[G];
      if (moves) {
#pragma unroll
        for (int g = 0; g < G; ++g) {
          float v = sc[g];
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xFFFFFFFFu, v, o));
          if (lane == 0) s_red[warp][g] = v;
        }
        ok = !softmax_barrier_or(!ok);               // the per-warp maxima are visible; every thread agrees on `ok`
        if (!ok) break;
#pragma unroll
        for (int g = 0; g < G; ++g) {
          const float mt = fmaxf(fmaxf(s_red[0][g], s_red[1][g]), fmaxf(s_red[2][g], s_red[3][g]));
          const float mn = (mt > m_run[g] + 8.f) ? mt : m_run[g];
          alpha[g] = dm_exp2(m_run[g] - mn);
          m_run[g] = mn;
          l_run[g] *= alpha[g];
        }
        if (j > 0) {                                 // the previous product must be complete before O is rescaled
          ok = mbar_wait(&pv_bar[(j - 1) & 1], ((j - 1) >> 1) & 1u, p.status);
          ok = __all_sync(0xFFFFFFFFu, ok);
          if (ok) {
            tc_fence_after_sync();
            uint32_t o[16];
            tmem_ld16(tO + lane_off, o);
            tc_wait_ld();
#pragma unroll
            for (int g = 0; g < G; ++g) o[g] = __float_as_uint(__uint_as_float(o[g]) * alpha[g]);
            tmem_st16(tO + lane_off, o);
            tc_wait_st();
          }
        }
      }
      float pj[G];
#pragma unroll
      for (int g = 0; g < G; ++g) pj[g] = dm_exp2(sc[g] - m_run[g]);      // masked keys: exp2(-1e30 - m) = 0
      if (j >= 2) {                                  // this P buffer was read by the product of tile j - 2
        ok = ok && mbar_wait(&pv_bar[j & 1], ((j - 2) >> 1) & 1u, p.status);
        ok = __all_sync(0xFFFFFFFFu, ok);
      }
      if (ok) {
        uint8_t* sp = sP + (j & 1) * kDmPBytes;
#pragma unroll
        for (int g = 0; g < G; ++g) {
          const __nv_bfloat16 pb = __float2bfloat16(pj[g]);
          *reinterpret_cast<__nv_bfloat16*>(sp + (tid >> 6) * 2048 + sw128_off(g, tid & 63)) = pb;
          l_run[g] += __bfloat162float(pb);          // the sum uses the rounded value that the tensor core multiplies
        }
        // rows of V that this tile did not fill: key t's row in every slab (0 * NaN would be NaN)
        if (!exists) {
          for (int c = 0; c < NB; ++c)
            for (int i = 0; i < 8; ++i) reinterpret_cast<uint4*>(sv + c * kDmSlab + tid * 128)[i] = make_uint4(0, 0, 0, 0);
        }
      }
      // After a wait that ran out P is not reported as ready; the warp keeps walking the loop (without waiting) so
      // that every warp meets the named barrier the same number of times, and all leave together through its OR.
      if (ok) {
        fence_proxy_async_smem();
        tc_fence_before_sync();
        mbar_arrive(&p_bar[j & 1]);
      }
    }
    if (ok && n_tiles > 0) ok = mbar_wait(&pv_bar[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1u, p.status);
    ok = __all_sync(0xFFFFFFFFu, ok);
#pragma unroll
    for (int g = 0; g < G; ++g) {
      float v = l_run[g];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
      l_run[g] = v;
    }
    softmax_barrier_or(false);                        // earlier readers of s_red are done
    if (lane == 0) {
#pragma unroll
      for (int g = 0; g < G; ++g) s_red[warp][g] = l_run[g];
    }
    ok = !softmax_barrier_or(!ok);
    // A wait that ran out (status bit set) leaves an empty partial (or zeros): what an earlier launch left is never read.
    uint32_t o[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) o[i] = 0u;
    if (ok && n_tiles > 0) {
      tc_fence_after_sync();
      tmem_ld16(tO + lane_off, o);
      tc_wait_ld();
    }
#pragma unroll
    for (int g = 0; g < G; ++g) {
      if (g >= heads) break;
      const int h = h0 + g;
      float l = ok ? s_red[0][g] + s_red[1][g] + s_red[2][g] + s_red[3][g] : 0.f;
      if (p.splits > 1) {
        const int64_t base = (static_cast<int64_t>(b) * p.hq + h) * p.splits + split;
        if (tid < p.vdim) p.partial_o[base * p.vdim + tid] = __uint_as_float(o[g]);
        if (tid == 0) {
          p.partial_ml[base * 2] = ok ? m_run[g] : -1.0e29f;
          p.partial_ml[base * 2 + 1] = l;
        }
      } else if (tid < p.vdim) {
        if (p.sink != nullptr) l += exp2f(__bfloat162float(p.sink[h]) * kDmLog2e - m_run[g]);
        float f = l > 0.f ? 1.f / l : 0.f;
        if (p.gate != nullptr) {
          const float z = __bfloat162float(p.gate[b * p.gate_ld + static_cast<int64_t>(h) * p.gate_step + (p.gate_step > 1 ? tid : 0)]);
          f *= 1.f / (1.f + expf(-z));
        }
        p.o[b * p.o_ld + static_cast<int64_t>(h) * p.vdim + tid] = __float2bfloat16(__uint_as_float(o[g]) * f);
      }
    }
    if (!ok) {
      // let copies that may still be in flight land before shared memory and TMEM are released
      const uint64_t t0 = globaltimer_ns();
      while (globaltimer_ns() - t0 < 200000ull) { __nanosleep(1000); }
    }
  }
  __syncwarp();
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, 64);
  }
}

template <int G, int NB>
int paged_decode_mma_run(const PagedDecodeMmaParams& p, dim3 grid, cudaStream_t stream) {
  static PerDeviceInt configured;
  if (!configured.cur()) {
    const cudaError_t e = cudaFuncSetAttribute(paged_decode_mma_kernel<G, NB>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               DecodeMmaSmem<NB>::kTotal);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.cur() = 1;
  }
  paged_decode_mma_kernel<G, NB><<<grid, kDmThreads, DecodeMmaSmem<NB>::kTotal, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// (size, kv head, slot) map of cache pages [slots, kv_heads, size]; copies of 64 columns of one block
inline int paged_decode_map(CUtensorMap* m, const void* pages, int size, int kv_heads, int64_t slots) {
  return make_tmap_3d(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, pages, static_cast<uint64_t>(size),
                      static_cast<uint64_t>(kv_heads), static_cast<uint64_t>(slots), static_cast<uint64_t>(size) * 2,
                      static_cast<uint64_t>(kv_heads) * size * 2, 64, 1, kDmBlock);
}

}  // namespace yv
