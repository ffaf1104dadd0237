// Decode in the latent space on the tensor cores: every head of a sequence attends over the same cached rows
// [latent | rotated key part], which are keys with all their columns and values with the latent ones.
//
// A tile is one cache page of 64 tokens, stored in shared memory as slabs of 64 columns (128-byte swizzle) and used
// twice from there:
//   S[128 heads, 64 keys]   = Q[heads, row] * C[64 keys, row]^T            (SS, both K-major; NH rows of Q are real)
//   O^T[128 dims, NH heads] += C^T[dims, 64 keys] * P[NH heads, 64 keys]^T  (SS, A MN-major), one product per 128 dims
// The M dimension of the first product reads past the NH real rows of Q into whatever follows in shared memory; those
// lanes of S are never read.
//
// grid = (head groups of NH, sequences, key ranges), 288 threads.  A warp reads the 32 TMEM lanes of its index modulo
// four, so two warps share the scores of the same heads, half a page each:
//   scoring     warps with (index % 4) < NH / 32: thread = (head, half of the page); both threads of a head keep the
//               same reference maximum, which moves only when a score exceeds it by 2^8 (one flag per page, agreed at
//               the barrier; the exchange of maxima and the rescaling of O^T are a rare path)
//   rescaling   warps 0..3 (lane = latent dimension), also the final output
//   warps 6, 8  one lane each issues the first and the second product.  The products are short, so issuing them is a
//               part of the page's time that is worth sharing; scores run up to two pages ahead
//   warp 7      one lane issues the TMA copies
// The page slabs travel through a ring counted in slabs, so that a part of the page after next is already in flight
// when two whole pages do not leave room for a third.  A page takes an even number of ring slots: the pair of slabs
// behind one 128-row product is always contiguous.
// Output: normalised bf16 when there is one key range, otherwise (max, sum, fp32 sums) per range, merged below.
#pragma once
#include "latent_ops.h"
#include "per_device.h"
#include "sm100.cuh"
#include "tensormap.h"

namespace yv {

struct LatentDecodeParams {
  CUtensorMap tma_c;               // 2-D (row, token slot), box (64, 64), 128B swizzle
  const __nv_bfloat16* q;          // [heads, rows_pad, row]
  __nv_bfloat16* out;              // [heads, rows_pad, kv_rank]
  const int* block_table;
  const int* seq_lens;
  float* partial_o;
  float* partial_ml;
  int64_t rows_pad;
  int heads, kv_rank, row, max_blocks, num_blocks, window, splits;
  int slabs, slots, ring, chunks;  // slabs and ring slots per page, ring size in slabs, 128-dim chunks of the latent
  uint32_t tmem_cols;
  float scale_log2;
  uint32_t* status;
};

constexpr int kLdThreads = 288;
constexpr int kLdKeys = 64;
constexpr int kLdSlab = kLdKeys * 128;
constexpr int kLdBars = 4;                                  // pages whose arrival can be tracked at a time
constexpr int kLdSmemMax = 227 * 1024;
constexpr int kLdTableCap = 512;                            // block-table entries of a key range staged in shared memory
constexpr int kLdStatic = 4096;                             // bound on the kernel's static shared memory

// Barrier over the scoring and rescaling threads (COUNT of them) with an OR of `v`.  The instruction is warp-aligned:
// lanes that left a bounded wait at different times are brought together first.
template <int COUNT>
__device__ __forceinline__ bool ld_barrier_or(bool v) {
  uint32_t r;
  __syncwarp();
  asm volatile(
      "{\n"
      ".reg .pred pin, pout;\n"
      "setp.ne.u32 pin, %1, 0;\n"
      "bar.red.or.pred pout, 1, %2, pin;\n"
      "selp.u32 %0, 1, 0, pout;\n"
      "}\n"
      : "=r"(r)
      : "r"(static_cast<uint32_t>(v)), "n"(COUNT)
      : "memory");
  return r != 0u;
}

__device__ __forceinline__ float ld_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int NH>
__global__ void __launch_bounds__(kLdThreads, 2) latent_decode_kernel(const __grid_constant__ LatentDecodeParams p) {
  constexpr uint32_t kIdescQK = make_idesc_bf16(128, kLdKeys, false, false);
  constexpr uint32_t kIdescPV = make_idesc_bf16(128, NH, true, false);
  constexpr int kScoreCols = NH > 32 ? 2 : 1;               // warps per half page that hold heads
  constexpr int kTeam = 32 * (kScoreCols + 4);              // scoring and rescaling threads
  constexpr int kQSlab = NH * 128;                          // bytes of one 64-column slab of Q (and of one P buffer)
  extern __shared__ uint8_t ld_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ld_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = sm;                                         // [slabs][NH][128 B]
  uint8_t* sP = sQ + p.slabs * kQSlab;                      // [2][NH][128 B]
  uint8_t* ring = sP + 2 * kQSlab;                          // [ring][64 keys][128 B]
  __shared__ uint64_t full_bar[kLdBars], empty_bar[kLdBars], s_bar[2], pv_bar[2], p_bar[2];
  __shared__ uint32_t tmem_slot;
  __shared__ float s_alpha[2][NH], s_max[2][NH], s_sum[2][NH];
  __shared__ int s_table[kLdTableCap];

  const int tid = threadIdx.x, lane = tid & 31;
  const int warp = __shfl_sync(0xFFFFFFFFu, tid >> 5, 0);      // known to be uniform: the issue loops run on it
  const int h0 = blockIdx.x * NH, b = blockIdx.y, split = blockIdx.z;
  int n = p.seq_lens[b];
  {
    const int64_t cap = static_cast<int64_t>(p.max_blocks) * kLdKeys;
    if (n < 0 || n > cap) {
      if (tid == 0 && p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
      n = n < 0 ? 0 : static_cast<int>(cap);
    }
  }
  const int first = (p.window > 0 && n > p.window) ? n - p.window : 0;
  const int page_lo = first / kLdKeys, page_hi = (n + kLdKeys - 1) / kLdKeys;
  const int per = (page_hi - page_lo + p.splits - 1) / p.splits;
  const int pg0 = page_lo + split * per;
  const int pg1 = min(page_hi, pg0 + per);
  const int n_tiles = pg1 > pg0 ? pg1 - pg0 : 0;
  const int* gtable = p.block_table + static_cast<int64_t>(b) * p.max_blocks + pg0;
  const int* table = n_tiles <= kLdTableCap ? s_table : gtable;       // pages of this key range
  if (n_tiles <= kLdTableCap)
    for (int i = tid; i < n_tiles; i += kLdThreads) s_table[i] = gtable[i];

  if (tid == 0) {
    tma_prefetch_desc(&p.tma_c);
    for (int i = 0; i < kLdBars; ++i) { mbar_init(&full_bar[i], 1); mbar_init(&empty_bar[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&s_bar[i], 1); mbar_init(&pv_bar[i], 1); mbar_init(&p_bar[i], kTeam); }
    fence_barrier_init();
  }
  if (warp == 0) {
    tmem_alloc(&tmem_slot, p.tmem_cols);
    tmem_relinquish();
  }
  // Q as K-major swizzled slabs; heads and columns that do not exist are zero.  P rows are written every tile.
  for (int i = tid; i < p.slabs * NH * 8; i += kLdThreads) {
    const int v = i & 7, r = (i >> 3) % NH, c = (i >> 3) / NH;
    const int col = c * 64 + v * 8;
    uint4 val = make_uint4(0, 0, 0, 0);
    if (h0 + r < p.heads && col < p.row)
      val = *reinterpret_cast<const uint4*>(p.q + (static_cast<int64_t>(h0 + r) * p.rows_pad + b) * p.row + col);
    *reinterpret_cast<uint4*>(sQ + c * kQSlab + r * 128 + ((v ^ (r & 7)) << 4)) = val;
  }
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = tmem_slot;
  const uint32_t tO = tmem_base + 128u;                     // S buffers at columns 0 and 64

  if (warp == 7) {
    // ------------------------------------ TMA producer ---------------------------------------
    if (elect_one()) {
      bool ok = true;
      int slot = 0;                                         // ring slot of the next slab
      int room = p.ring;                                    // free ring slots
      int freed = 0;                                        // pages known to have been consumed
      for (int j = 0; j < n_tiles && ok; ++j) {
        // the barrier of page j was last used by page j - kLdBars
        while (ok && freed + kLdBars <= j) {
          ok = mbar_wait(&empty_bar[freed % kLdBars], (freed / kLdBars) & 1u, p.status);
          ++freed;
          room += p.slots;
        }
        if (!ok) break;
        uint64_t* full = &full_bar[j % kLdBars];
        mbar_expect_tx(full, static_cast<uint32_t>(p.slabs) * kLdSlab);
        int page = table[j];
        if (page < 0 || page >= p.num_blocks) {             // reported; its keys are masked by the softmax warps
          if (p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
          page = 0;
        }
        for (int c = 0; c < p.slots && ok; ++c) {
          while (ok && room == 0) {
            ok = mbar_wait(&empty_bar[freed % kLdBars], (freed / kLdBars) & 1u, p.status);
            ++freed;
            room += p.slots;
          }
          if (!ok) break;
          if (c < p.slabs) tma_load_2d(ring + static_cast<size_t>(slot) * kLdSlab, &p.tma_c, full, c * 64, page * kLdKeys);
          --room;
          if (++slot == p.ring) slot = 0;
        }
      }
    }
  } else if (warp == 6 || warp == 8) {
    // ------------------------------------ MMA issuers ----------------------------------------
    // descriptors differ in their address field only (the low word): base + byte offset / 16
    const uint32_t hiK = static_cast<uint32_t>(make_smem_desc(0, 16, 1024) >> 32), loK = static_cast<uint32_t>(make_smem_desc(0, 16, 1024));
    const uint32_t hiC = static_cast<uint32_t>(make_smem_desc(0, kLdSlab, 1024) >> 32);
    const uint32_t loC = static_cast<uint32_t>(make_smem_desc(0, kLdSlab, 1024));
    auto desc = [](uint32_t hi, uint32_t lo) { return (static_cast<uint64_t>(hi) << 32) | lo; };
    const uint32_t aRing = smem_u32(ring) >> 4;
    if (warp == 6) {
      if (elect_one()) {
        const uint32_t dQ = loK + (smem_u32(sQ) >> 4), dR = loK + aRing;
        int start = 0;                                      // ring slot of the page
        for (int j = 0; j < n_tiles; ++j) {
          // S buffer j & 1 was read for page j - 2: its weights have been reported
          if (j >= 2 && !mbar_wait(&p_bar[j & 1], ((j - 2) >> 1) & 1u, p.status)) break;
          if (!mbar_wait(&full_bar[j % kLdBars], (j / kLdBars) & 1u, p.status)) break;
          tc_fence_after_sync();
          const uint32_t dS = tmem_base + static_cast<uint32_t>((j & 1) * 64);
          int slot = start;
          for (int c = 0; c < p.slabs; ++c) {               // columns past the row are zero in both operands
            const uint32_t a = dQ + static_cast<uint32_t>(c * (kQSlab >> 4)), k = dR + static_cast<uint32_t>(slot * (kLdSlab >> 4));
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              tc_mma_f16_ss(dS, desc(hiK, a + kk * 2), desc(hiK, k + kk * 2), kIdescQK, (c | kk) != 0 ? 1u : 0u);
            if (++slot == p.ring) slot = 0;
          }
          start += p.slots;
          if (start >= p.ring) start -= p.ring;
          tc_commit(&s_bar[j & 1]);
        }
      }
    } else if (elect_one()) {
      const uint32_t dC = loC + aRing, dP = loK + (smem_u32(sP) >> 4);
      int start = 0;
      for (int j = 0; j < n_tiles; ++j) {
        // one barrier per P buffer: the softmax warps may finish page j + 1 before this thread looks at page j
        if (!mbar_wait(&p_bar[j & 1], (j >> 1) & 1u, p.status)) break;
        tc_fence_after_sync();
        const uint32_t bP = dP + static_cast<uint32_t>((j & 1) * (kQSlab >> 4));
        int slot = start;
        for (int m = 0; m < p.chunks; ++m) {
          const uint32_t aC = dC + static_cast<uint32_t>(slot * (kLdSlab >> 4));
#pragma unroll
          for (int kk = 0; kk < kLdKeys / 16; ++kk)
            tc_mma_f16_ss(tO + static_cast<uint32_t>(m * NH), desc(hiC, aC + kk * (2048 >> 4)), desc(hiK, bP + kk * 2),
                          kIdescPV, (j | kk) != 0 ? 1u : 0u);
          slot += 2;
          if (slot >= p.ring) slot -= p.ring;
        }
        start += p.slots;
        if (start >= p.ring) start -= p.ring;
        tc_commit(&pv_bar[j & 1]);
        tc_commit(&empty_bar[j % kLdBars]);
      }
    }
    __syncwarp();
  } else if ((warp & 3) < kScoreCols || warp < 4) {
    // ------------------------------------ softmax, rescaling, output -------------------------
    const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const bool scoring = (warp & 3) < kScoreCols;           // warp-uniform: the lanes of this warp hold heads
    const int half = warp >> 2;                             // keys half * 32 .. + 31 of every page
    const int hr = (warp & 3) * 32 + lane;                  // head row = TMEM lane of S
    const bool head = scoring && hr < NH;
    float m_used = -1.0e29f, l_sum = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      uint32_t s[32];
      float mx = -1.0e30f;
      if (scoring) {
        ok = ok && mbar_wait(&s_bar[j & 1], (j >> 1) & 1u, p.status);
        ok = __all_sync(0xFFFFFFFFu, ok);
        if (ok) {
          tc_fence_after_sync();
          tmem_ld32(tmem_base + lane_off + static_cast<uint32_t>((j & 1) * 64 + half * 32), s);
          tc_wait_ld();
          const int page = table[j];
          const bool page_ok = page >= 0 && page < p.num_blocks;
          const int k0 = (pg0 + j) * kLdKeys + half * 32;
          if (k0 < first || k0 + 32 > n || !page_ok) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (k0 + i < first || k0 + i >= n || !page_ok) s[i] = 0xFF800000u;
          }
          float t[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) t[i] = fmaxf(__uint_as_float(s[2 * i]), __uint_as_float(s[2 * i + 1]));
#pragma unroll
          for (int w = 8; w > 0; w >>= 1)
#pragma unroll
            for (int i = 0; i < w; ++i) t[i] = fmaxf(t[i], t[i + w]);
          mx = fmaxf(t[0], -1.0e30f);
          mx = mx > -0.5e30f ? mx * p.scale_log2 : -1.0e30f;
          tc_fence_before_sync();
        }
      }
      if (ld_barrier_or<kTeam>((head && mx > m_used + 8.f) || !ok)) {
        ok = !ld_barrier_or<kTeam>(!ok);                    // everyone agrees
        if (!ok) break;
        if (head) s_max[half][hr] = mx;
        // O^T holds sums relative to the old maxima: the previous product must be complete before it is scaled
        if (j > 0) {
          ok = mbar_wait(&pv_bar[(j - 1) & 1], ((j - 1) >> 1) & 1u, p.status);
          ok = __all_sync(0xFFFFFFFFu, ok);
        }
        ok = !ld_barrier_or<kTeam>(!ok);
        if (!ok) break;
        if (head) {
          const float all = fmaxf(s_max[0][hr], s_max[1][hr]);
          float alpha = 1.f;
          if (all > m_used + 8.f) {
            alpha = ld_exp2(m_used - all);
            m_used = all;
            l_sum *= alpha;
          }
          if (half == 0) s_alpha[j & 1][hr] = alpha;
        }
        ld_barrier_or<kTeam>(false);
        if (warp < 4 && j > 0) {
          tc_fence_after_sync();
          for (int m = 0; m < p.chunks; ++m) {
#pragma unroll
            for (int g = 0; g < NH; g += 16) {
              uint32_t o[16];
              __syncwarp();
              tmem_ld16(tO + lane_off + static_cast<uint32_t>(m * NH + g), o);
              tc_wait_ld();
#pragma unroll
              for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_alpha[j & 1][g + i]);
              tmem_st16(tO + lane_off + static_cast<uint32_t>(m * NH + g), o);
            }
          }
          tc_wait_st();
          tc_fence_before_sync();
        }
      }
      if (scoring) {
        // P buffer j & 1 was read by the product of page j - 2
        if (j >= 2) {
          ok = mbar_wait(&pv_bar[j & 1], ((j - 2) >> 1) & 1u, p.status);
          ok = __all_sync(0xFFFFFFFFu, ok);                 // a failure is agreed on at the next barrier
        }
        uint32_t pk[16];
        float ls[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float e0 = ld_exp2(fmaf(__uint_as_float(s[2 * i]), p.scale_log2, -m_used));
          const float e1 = ld_exp2(fmaf(__uint_as_float(s[2 * i + 1]), p.scale_log2, -m_used));
          pk[i] = pack_bf16(e0, e1);
          ls[i & 3] += __uint_as_float(pk[i] << 16) + __uint_as_float(pk[i] & 0xFFFF0000u);   // the weights as multiplied
        }
        l_sum += (ls[0] + ls[1]) + (ls[2] + ls[3]);
        if (head && ok) {
          uint8_t* row = sP + (j & 1) * kQSlab + hr * 128;
#pragma unroll
          for (int c = 0; c < 4; ++c)
            *reinterpret_cast<uint4*>(row + (((4 * half + c) ^ (hr & 7)) << 4)) =
                make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
        }
        __syncwarp();
        fence_proxy_async_smem();
      }
      if (ok) mbar_arrive(&p_bar[j & 1]);
    }
    if (ok && n_tiles > 0) ok = mbar_wait(&pv_bar[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1u, p.status);
    ok = __all_sync(0xFFFFFFFFu, ok);
    if (head) s_sum[half][hr] = l_sum;
    ok = !ld_barrier_or<kTeam>(!ok);
    // after a wait that ran out (status set) the outputs are still written, as zeros
    if (head && half == 0 && h0 + hr < p.heads && p.splits > 1) {
      const int64_t base = (static_cast<int64_t>(b) * p.heads + h0 + hr) * p.splits + split;
      p.partial_ml[base * 2] = ok ? m_used : -1.0e29f;
      p.partial_ml[base * 2 + 1] = ok ? s_sum[0][hr] + s_sum[1][hr] : 0.f;
    }
    if (warp < 4) {
      tc_fence_after_sync();
      for (int m = 0; m < p.chunks; ++m) {
        const int dim = m * 128 + tid;
#pragma unroll
        for (int g = 0; g < NH; g += 16) {
          uint32_t o[16];
          __syncwarp();
          if (ok && n_tiles > 0) {
            tmem_ld16(tO + lane_off + static_cast<uint32_t>(m * NH + g), o);
            tc_wait_ld();
          } else {
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = 0u;
          }
          if (dim < p.kv_rank) {
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              const int h = h0 + g + i;
              if (h < p.heads) {
                const float v = __uint_as_float(o[i]);
                if (p.splits > 1) {
                  p.partial_o[((static_cast<int64_t>(b) * p.heads + h) * p.splits + split) * p.kv_rank + dim] = v;
                } else {
                  const float l = s_sum[0][g + i] + s_sum[1][g + i];
                  p.out[(static_cast<int64_t>(h) * p.rows_pad + b) * p.kv_rank + dim] = __float2bfloat16(l > 0.f ? v / l : 0.f);
                }
              }
            }
          }
        }
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
    tmem_dealloc(tmem_base, p.tmem_cols);
  }
}

// One block per (head, sequence).
__global__ void __launch_bounds__(128) latent_decode_merge_kernel(const float* __restrict__ po, const float* __restrict__ pml,
                                                                  __nv_bfloat16* __restrict__ out, int64_t rows_pad,
                                                                  int heads, int kv_rank, int splits) {
  const int h = blockIdx.x, b = blockIdx.y;
  const int64_t base = (static_cast<int64_t>(b) * heads + h) * splits;
  float m = -1.0e29f;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, pml[(base + s) * 2]);
  float l = 0.f;
  for (int s = 0; s < splits; ++s) l += pml[(base + s) * 2 + 1] * exp2f(pml[(base + s) * 2] - m);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int d = threadIdx.x; d < kv_rank; d += 128) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) v += po[(base + s) * kv_rank + d] * exp2f(pml[(base + s) * 2] - m);
    out[(static_cast<int64_t>(h) * rows_pad + b) * kv_rank + d] = __float2bfloat16(v * inv);
  }
}

struct LatentDecodePlan {
  int nh = 0, slabs = 0, slots = 0, ring = 0, chunks = 0, smem = 0;
  uint32_t tmem_cols = 0;
};

// Heads per CTA, ring size and tensor-memory columns; nh == 0 when the sizes do not fit.
inline LatentDecodePlan latent_decode_plan(int heads, int kv_rank, int row) {
  LatentDecodePlan pl;
  pl.slabs = (row + 63) / 64;
  pl.chunks = (kv_rank + 127) / 128;
  const int need = pl.slabs > 2 * pl.chunks ? pl.slabs : 2 * pl.chunks;
  pl.slots = (need + 1) / 2 * 2;
  for (int nh = heads > 32 ? 64 : (heads > 16 ? 32 : 16); nh >= 16; nh /= 2) {
    const int cols = 128 + pl.chunks * nh;
    if (cols > 512) continue;
    const int fixed = 1024 + (pl.slabs + 2) * nh * 128;
    int ring = (kLdSmemMax - fixed - kLdStatic) / kLdSlab / 2 * 2;
    if (ring < 2 * pl.slots) continue;
    const int small = 3 * pl.slots;                                 // three pages, if that lets two CTAs share an SM
    if (ring > small && 2 * (fixed + small * kLdSlab + kLdStatic) <= kLdSmemMax && cols <= 256) ring = small;
    if (ring > kLdBars * pl.slots) ring = kLdBars * pl.slots;
    pl.nh = nh;
    pl.ring = ring;
    pl.smem = fixed + ring * kLdSlab;
    pl.tmem_cols = 32;
    while (pl.tmem_cols < static_cast<uint32_t>(cols)) pl.tmem_cols *= 2;
    return pl;
  }
  return pl;
}

inline bool latent_decode_on_tensor_cores(const LatentDecodeArgs& a) {
  const int row = a.kv_rank + a.rot_dim;
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
  return a.dtype == 0 && a.block == kLdKeys && (row & 7) == 0 && a.kv_rank > 0 && a.scale > 0.f && al16(a.q) &&
         al16(a.cache) && static_cast<int64_t>(a.num_blocks) * a.block < (1ll << 31) && a.splits <= 65535 &&
         latent_decode_plan(a.heads, a.kv_rank, row).nh != 0;
}

template <int NH>
int latent_decode_run(const LatentDecodeParams& p, dim3 grid, int smem, cudaStream_t stream) {
  static PerDeviceInt configured;
  if (configured.cur() < smem) {
    const cudaError_t e =
        cudaFuncSetAttribute(latent_decode_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.cur() = smem;
  }
  latent_decode_kernel<NH><<<grid, kLdThreads, smem, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

inline int launch_latent_decode_mma(const LatentDecodeArgs& a, cudaStream_t stream) {
  const int row = a.kv_rank + a.rot_dim;
  const LatentDecodePlan pl = latent_decode_plan(a.heads, a.kv_rank, row);
  if (pl.nh == 0) return -60;
  if (a.splits > 1 && (a.partial_o == nullptr || a.partial_ml == nullptr)) return -61;
  LatentDecodeParams p;
  const int64_t slots = static_cast<int64_t>(a.num_blocks) * a.block;
  int r = make_tmap_2d(&p.tma_c, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.cache, static_cast<uint64_t>(row),
                       static_cast<uint64_t>(slots), static_cast<uint64_t>(row), 64, kLdKeys);
  if (r != 0) return -70 + r;
  p.q = static_cast<const __nv_bfloat16*>(a.q); p.out = static_cast<__nv_bfloat16*>(a.out);
  p.block_table = a.block_table; p.seq_lens = a.seq_lens;
  p.partial_o = a.partial_o; p.partial_ml = a.partial_ml;
  p.rows_pad = a.rows_pad;
  p.heads = a.heads; p.kv_rank = a.kv_rank; p.row = row; p.max_blocks = a.max_blocks_per_seq; p.num_blocks = a.num_blocks;
  p.window = a.window; p.splits = a.splits;
  p.slabs = pl.slabs; p.slots = pl.slots; p.ring = pl.ring; p.chunks = pl.chunks; p.tmem_cols = pl.tmem_cols;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.status = a.status;
  dim3 grid(static_cast<unsigned>((a.heads + pl.nh - 1) / pl.nh), static_cast<unsigned>(a.batch),
            static_cast<unsigned>(a.splits));
  switch (pl.nh) {
    case 16: r = latent_decode_run<16>(p, grid, pl.smem, stream); break;
    case 32: r = latent_decode_run<32>(p, grid, pl.smem, stream); break;
    default: r = latent_decode_run<64>(p, grid, pl.smem, stream); break;
  }
  if (r != 0 || a.splits == 1) return r;
  latent_decode_merge_kernel<<<dim3(static_cast<unsigned>(a.heads), static_cast<unsigned>(a.batch)), 128, 0, stream>>>(
      a.partial_o, a.partial_ml, p.out, a.rows_pad, a.heads, a.kv_rank, a.splits);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace yv
