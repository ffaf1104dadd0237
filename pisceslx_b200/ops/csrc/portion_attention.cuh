// Prompt attention of layered models on the tensor cores: causal, optionally with a sliding window, packed sequences whose
// keys may start before their queries (a portion that continues from the cache), query / key and value heads of sizes of
// their own.  Options, each without cost when it is not there:
//   key/value heads shared by groups of query heads; a further key part shared by all heads (SHARED);
//   keys and values in cache pages (a block table per sequence) or in packed rows;
//   a sink per head (a logit that only counts in the denominator); a sigmoid gate on the output, per head or per number
//
// One CTA per (head, 128-query block, sequence), 192 threads, in the roles of attention_fwd.cuh:
//   warp 0      TMA producer: Q once, then K_j / V_j tiles of 128 keys through rings, 64 rows to a copy (a page is a
//               multiple of 64).  A K tile is the head's own part (NBN slabs of 64 columns), then the shared part
//               (one slab); columns past a part's width are zero-filled by the copy, so any multiple of 8 up to the slab
//               width is a valid size
//   warp 1      MMA issuer: S_j = Q K_j^T (SS) into a TMEM buffer, O += P_j V_j (TS)
//   warps 2..5  softmax: thread r owns query row r; scores, maxima, exponentials and sums are fp32.  Value rows past the
//               end of a sequence are cleared: what a page holds there must not meet a zero weight as 0 * NaN
// Key tiles start at the first one that any row of the block can see.
// The fp32 exponentials of a tile take as long as its two products, so the products of one block have to run under the
// softmax of another.  Without a shared part two CTAs fit an SM and cover each other: one score buffer, and one stage of
// keys and values where two do not fit.  With it, one CTA per SM issues S_{j+1} ahead into a second score buffer.
// TMEM columns: kScores buffers of 128 for S / P, then 64 NBV for O.
#pragma once
#include "per_device.h"
#include "sm100.cuh"
#include "tensormap.h"

namespace yv {

struct PortionAttnParams {
  CUtensorMap tma_qn;   // 3-D (dim, head, token), box (64, 1, 128)
  CUtensorMap tma_qr;   // 3-D (shared part, head, token); SHARED
  CUtensorMap tma_k;    // 3-D (dim, key/value head, row), box (64, 1, 64)
  CUtensorMap tma_kr;   // 2-D (shared part, row), box (64, 64); SHARED
  CUtensorMap tma_v;    // 3-D (vdim, key/value head, row), box (64, 1, 64)
  __nv_bfloat16* o;
  int64_t o_ld;
  const __nv_bfloat16* gate;     // logits [token, gate_ld]: gate_step numbers per head (1, or vdim), null = none
  int64_t gate_ld;
  int gate_step;
  const __nv_bfloat16* sink;     // [heads], null = none
  const int* cu_q;
  const int* cu_k;               // packed rows: offsets of the sequences' keys
  const int* table;              // pages: [sequences, table_width] block numbers, null = packed rows
  const int* lens;               // pages: keys of every sequence
  int table_width, block, num_blocks;
  int dim, rot_dim, vdim, window, group;
  float scale_log2;
  uint32_t* status;
};

constexpr int kLpThreads = 192;
constexpr int kLpBlock = 128;
constexpr uint32_t kLpSlab = kLpBlock * 128;         // 128 rows x 64 columns
constexpr float kLpMask = -1.0e30f;
constexpr float kLpLog2e = 1.4426950408889634f;
constexpr float kLpRescale = 8.0f;                   // log2 units

template <int NBN, int NBV, bool SHARED>
struct PortionAttnSmem {
  static constexpr int kQK = (NBN + (SHARED ? 1 : 0)) * static_cast<int>(kLpSlab);
  static constexpr int kV = NBV * static_cast<int>(kLpSlab);
  static constexpr int kCtas = SHARED ? 1 : 2;                       // per SM
  static constexpr int kScores = SHARED ? 2 : 1;                     // score buffers
  static constexpr int kStages = SHARED || NBN + NBV == 2 ? 2 : 1;   // tiles of K and V
  static constexpr uint32_t kTmemCols = SHARED ? 512 : 256;
  static constexpr int kTotal = kQK + kStages * (kQK + kV) + 256 + 1024;
};

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float lp_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

template <int NBN, int NBV, bool SHARED>
__global__ void __launch_bounds__(kLpThreads, PortionAttnSmem<NBN, NBV, SHARED>::kCtas)
portion_attn_kernel(const __grid_constant__ PortionAttnParams p) {
  using S = PortionAttnSmem<NBN, NBV, SHARED>;
  constexpr int D = NBV * 64;
  constexpr uint32_t kIdescQK = make_idesc_bf16(128, 128, false, false);
  constexpr uint32_t kIdescPV = make_idesc_bf16(128, D, false, true);
  constexpr int kStages = S::kStages, kScores = S::kScores;
  constexpr uint32_t kTmemCols = S::kTmemCols;
  constexpr uint32_t kOCol = kScores * 128;

  extern __shared__ uint8_t lp_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lp_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + S::kQK;
  uint8_t* sV = sK + kStages * S::kQK;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + kStages * S::kV);
  uint64_t* q_full = bars;                 // [1]
  uint64_t* k_full = bars + 1;             // [2]
  uint64_t* k_empty = bars + 3;            // [2]
  uint64_t* v_full = bars + 5;             // [2]
  uint64_t* v_empty = bars + 7;            // [2]
  uint64_t* s_full = bars + 9;             // [2]
  uint64_t* p_full = bars + 11;            // [2]
  uint64_t* o_done = bars + 13;            // [1]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 14);

  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.x;
  const int q_begin = p.cu_q[b], q_len = p.cu_q[b + 1] - q_begin;
  const bool paged = p.table != nullptr;
  const int k_begin = paged ? 0 : p.cu_k[b];
  int k_len = paged ? p.lens[b] : p.cu_k[b + 1] - k_begin;
  if (paged && (k_len < 0 || static_cast<int64_t>(k_len) > static_cast<int64_t>(p.table_width) * p.block)) {
    if (threadIdx.x == 0 && p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
    k_len = 0;
  }
  const int n_qblk = (q_len + kLpBlock - 1) / kLpBlock;
  const int q_blk = n_qblk - 1 - static_cast<int>(blockIdx.y);       // all heads' late (longer) blocks first
  if (q_blk < 0) return;
  const int q0 = q_blk * kLpBlock;
  const int shift = k_len - q_len;                                   // key index of query i is i + shift
  const int last_key = min(q0 + kLpBlock - 1 + shift, k_len - 1);
  const int first_key = p.window > 0 ? max(q0 + shift - p.window + 1, 0) : 0;
  const int j0 = first_key / kLpBlock;
  const int n_kv = last_key < first_key ? 0 : last_key / kLpBlock + 1 - j0;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&p.tma_qn);
    tma_prefetch_desc(&p.tma_k);
    if constexpr (SHARED) {
      tma_prefetch_desc(&p.tma_qr);
      tma_prefetch_desc(&p.tma_kr);
    }
    tma_prefetch_desc(&p.tma_v);
    mbar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1);
      mbar_init(&p_full[s], 128);
    }
    mbar_init(o_done, 1);
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------ producer ------------------------------------------
    if (elect_one() && n_kv > 0) {
      mbar_expect_tx(q_full, S::kQK);
#pragma unroll
      for (int c = 0; c < NBN; ++c) tma_load_3d(sQ + c * kLpSlab, &p.tma_qn, q_full, c * 64, h, q_begin + q0);
      if constexpr (SHARED) tma_load_3d(sQ + NBN * kLpSlab, &p.tma_qr, q_full, 0, h, q_begin + q0);
      const int kvh = h / p.group;
      // row of the K / V maps where the 64 keys from `key` on start; past the last page, or at a table entry outside the
      // pool (reported), some valid row: its scores are masked and its values cleared or never used
      auto source = [&](int key) {
        if (!paged) return k_begin + key;
        const int bi = min(key, k_len - 1) / p.block;
        int page = p.table[static_cast<int64_t>(b) * p.table_width + bi];
        if (page < 0 || page >= p.num_blocks) {
          if (p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
          page = 0;
        }
        return page * p.block + (key - bi * p.block < p.block ? key - bi * p.block : 0);
      };
      constexpr uint32_t kHalf = kLpSlab / 2;
      bool ok = true;
      for (int j = 0; j < n_kv && ok; ++j) {
        const int s = j % kStages;
        const uint32_t ph = (j / kStages) & 1u;
        const int row[2] = {source((j0 + j) * kLpBlock), source((j0 + j) * kLpBlock + 64)};
        ok = mbar_wait(&k_empty[s], ph ^ 1u, p.status);
        if (!ok) break;
        mbar_expect_tx(&k_full[s], S::kQK);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint8_t* dst = sK + s * S::kQK + half * kHalf;
#pragma unroll
          for (int c = 0; c < NBN; ++c) tma_load_3d(dst + c * kLpSlab, &p.tma_k, &k_full[s], c * 64, kvh, row[half]);
          if constexpr (SHARED) tma_load_2d(dst + NBN * kLpSlab, &p.tma_kr, &k_full[s], 0, row[half]);
        }
        ok = mbar_wait(&v_empty[s], ph ^ 1u, p.status);
        if (!ok) break;
        mbar_expect_tx(&v_full[s], S::kV);
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int c = 0; c < NBV; ++c)
            tma_load_3d(sV + s * S::kV + half * kHalf + c * kLpSlab, &p.tma_v, &v_full[s], c * 64, kvh, row[half]);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------ MMA issuer ----------------------------------------
    if (elect_one() && n_kv > 0) {
      bool ok = mbar_wait(q_full, 0, p.status);
      const uint32_t aQ = smem_u32(sQ);
      const int steps_n = (p.dim + 15) / 16, steps_r = SHARED ? (p.rot_dim + 15) / 16 : 0;
      auto issue_qk = [&](int j) -> bool {
        const int s = j % kStages;
        if (!mbar_wait(&k_full[s], (j / kStages) & 1u, p.status)) return false;
        // a single score buffer still holds the weights of tile j - 1
        if (kScores == 1 && j > 0 && !mbar_wait(o_done, (j - 1) & 1u, p.status)) return false;
        tc_fence_after_sync();
        const uint32_t aK = smem_u32(sK + s * S::kQK);
        const uint32_t tS = tmem_base + static_cast<uint32_t>((j % kScores) * 128);
#pragma unroll
        for (int kk = 0; kk < NBN * 4; ++kk) {
          const uint32_t off = (kk / 4) * kLpSlab + (kk % 4) * 32;
          if (kk < steps_n)
            tc_mma_f16_ss(tS, make_smem_desc(aQ + off, 16, 1024), make_smem_desc(aK + off, 16, 1024), kIdescQK,
                          kk != 0 ? 1u : 0u);
        }
        if constexpr (SHARED) {
          for (int kk = 0; kk < steps_r; ++kk) {
            const uint32_t off = NBN * kLpSlab + kk * 32;
            tc_mma_f16_ss(tS, make_smem_desc(aQ + off, 16, 1024), make_smem_desc(aK + off, 16, 1024), kIdescQK, 1u);
          }
        }
        tc_commit(&k_empty[s]);
        tc_commit(&s_full[j % kScores]);
        return true;
      };
      if (ok) ok = issue_qk(0);
      for (int j = 0; j < n_kv && ok; ++j) {
        if (kScores == 2 ? j + 1 < n_kv : j > 0) {
          ok = issue_qk(kScores == 2 ? j + 1 : j);
          if (!ok) break;
        }
        const int s = j % kStages;
        ok = mbar_wait(&p_full[j % kScores], (j / kScores) & 1u, p.status);
        if (!ok) break;
        ok = mbar_wait(&v_full[s], (j / kStages) & 1u, p.status);
        if (!ok) break;
        tc_fence_after_sync();
        const uint32_t aV = smem_u32(sV + s * S::kV);
        const uint32_t tP = tmem_base + static_cast<uint32_t>((j % kScores) * 128);
        const uint32_t tO = tmem_base + kOCol;
#pragma unroll
        for (int kk = 0; kk < kLpBlock / 16; ++kk) {
          tc_mma_f16_ts(tO, tP + kk * 8, make_smem_desc(aV + kk * 2048, kLpSlab, 1024), kIdescPV,
                        (j | kk) != 0 ? 1u : 0u);
        }
        tc_commit(&v_empty[s]);
        tc_commit(o_done);
      }
    }
  } else {
    // ------------------------------------ softmax / epilogue --------------------------------
    const int quarter = warp & 3;
    const int row = quarter * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
    const int q_pos = q0 + row;
    const int hi = min(q_pos + shift, k_len - 1);                                    // last visible key
    const int lo = p.window > 0 ? q_pos + shift - p.window + 1 : 0;                  // first visible key
    float m_used = -1.0e29f;
    float l_sum = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv && ok; ++j) {
      ok = mbar_wait(&s_full[j % kScores], (j / kScores) & 1u, p.status);
      ok = __all_sync(0xFFFFFFFFu, ok);                  // the aligned tcgen05 instructions need a converged warp
      if (!ok) break;
      tc_fence_after_sync();
      const uint32_t tS = tmem_base + lane_off + static_cast<uint32_t>((j % kScores) * 128);
      uint32_t sreg[128];
      {
        uint32_t(&c0)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sreg[0]);
        uint32_t(&c1)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sreg[32]);
        uint32_t(&c2)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sreg[64]);
        uint32_t(&c3)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sreg[96]);
        tmem_ld32(tS, c0);
        tmem_ld32(tS + 32, c1);
        tmem_ld32(tS + 64, c2);
        tmem_ld32(tS + 96, c3);
        tc_wait_ld();
      }
      const int kbase = (j0 + j) * kLpBlock;
      if (kbase < lo || kbase + kLpBlock - 1 > hi) {
#pragma unroll
        for (int i = 0; i < 128; ++i)
          if (kbase + i > hi || kbase + i < lo) sreg[i] = 0xFF800000u;               // -inf
      }
      float mx4[4] = {kLpMask, kLpMask, kLpMask, kLpMask};
#pragma unroll
      for (int i = 0; i < 128; i += 2)
        mx4[(i >> 1) & 3] = fmaxf(mx4[(i >> 1) & 3], fmaxf(__uint_as_float(sreg[i]), __uint_as_float(sreg[i + 1])));
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      mx = (mx > 0.5f * kLpMask) ? mx * p.scale_log2 : kLpMask;
      float alpha = 1.f;
      bool rescale = false;
      if (mx > m_used + kLpRescale) {                    // lazy: the reference maximum moves in large steps only
        alpha = fast_exp2(m_used - mx);
        m_used = mx;
        rescale = (j > 0);
      }
      if (__any_sync(0xFFFFFFFFu, rescale)) {
        ok = mbar_wait(o_done, (j - 1) & 1u, p.status);
        ok = __all_sync(0xFFFFFFFFu, ok);
        if (!ok) break;
        tc_fence_after_sync();
        const uint32_t tO = tmem_base + lane_off + kOCol;
#pragma unroll
        for (int c = 0; c < D / 16; ++c) {
          uint32_t ov[16];
          tmem_ld16(tO + c * 16, ov);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 16; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * alpha);
          tmem_st16(tO + c * 16, ov);
        }
      }
      // P overwrites the scores, half a tile at a time
      float2 rs2[4] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
      const float2 sc2 = make_float2(p.scale_log2, p.scale_log2);
      const float2 nm2 = make_float2(-m_used, -m_used);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t pk[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const int e = 64 * half + 2 * i;
          const float2 x = __ffma2_rn(make_float2(__uint_as_float(sreg[e]), __uint_as_float(sreg[e + 1])), sc2, nm2);
          const uint32_t bits = pack_bf16(fast_exp2(x.x), fast_exp2(x.y));
          pk[i] = bits;
          // the sum takes the rounded weights that the tensor core multiplies
          rs2[i & 3] = __fadd2_rn(rs2[i & 3], make_float2(__uint_as_float(bits << 16), __uint_as_float(bits & 0xFFFF0000u)));
        }
        tmem_st32(tS + 32 * half, pk);
      }
      const float2 rsum = __fadd2_rn(__fadd2_rn(rs2[0], rs2[1]), __fadd2_rn(rs2[2], rs2[3]));
      l_sum = l_sum * alpha + (rsum.x + rsum.y);
      tc_wait_st();
      if (kbase + kLpBlock > k_len) {                    // the sequence ends in this tile: clear the rows behind it
        ok = mbar_wait(&v_full[j % kStages], (j / kStages) & 1u, p.status);
        ok = __all_sync(0xFFFFFFFFu, ok);
        if (!ok) break;
        if (kbase + row >= k_len) {
#pragma unroll
          for (int c = 0; c < NBV; ++c) {
            uint4* vr = reinterpret_cast<uint4*>(sV + (j % kStages) * S::kV + c * kLpSlab + row * 128);
#pragma unroll
            for (int i = 0; i < 8; ++i) vr[i] = make_uint4(0, 0, 0, 0);
          }
        }
        fence_proxy_async_smem();
      }
      tc_fence_before_sync();
      mbar_arrive(&p_full[j % kScores]);
    }
    if (ok && n_kv > 0) {
      ok = mbar_wait(o_done, (n_kv - 1) & 1u, p.status);
      ok = __all_sync(0xFFFFFFFFu, ok);
    }
    if (ok) {
      tc_fence_after_sync();
      const bool valid = q_pos < q_len;
      if (p.sink != nullptr) l_sum += fast_exp2(__bfloat162float(p.sink[h]) * kLpLog2e - m_used);
      float f = (l_sum > 0.f) ? 1.f / l_sum : 0.f;
      const __nv_bfloat16* grow = nullptr;               // a gate per number
      if (valid && p.gate != nullptr) {
        const __nv_bfloat16* g = p.gate + static_cast<int64_t>(q_begin + q_pos) * p.gate_ld + static_cast<int64_t>(h) * p.gate_step;
        if (p.gate_step == 1) f *= lp_sigmoid(__bfloat162float(*g));
        else grow = g;
      }
      __nv_bfloat16* orow = p.o + static_cast<int64_t>(q_begin + q_pos) * p.o_ld + static_cast<int64_t>(h) * p.vdim;
      const uint32_t tO = tmem_base + lane_off + kOCol;
#pragma unroll
      for (int c = 0; c < D / 32; ++c) {
        uint32_t ov[32];
        if (n_kv > 0) {
          tmem_ld32(tO + c * 32, ov);
          tc_wait_ld();
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) ov[i] = 0u;
        }
        if (valid) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (c * 32 + i * 8 < p.vdim) {
              float e[8];
#pragma unroll
              for (int k = 0; k < 8; ++k) e[k] = __uint_as_float(ov[8 * i + k]) * f;
              if (grow != nullptr) {
                const uint4 z = *reinterpret_cast<const uint4*>(grow + c * 32 + i * 8);
                const uint32_t zz[4] = {z.x, z.y, z.z, z.w};
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                  e[2 * k] *= lp_sigmoid(__uint_as_float(zz[k] << 16));
                  e[2 * k + 1] *= lp_sigmoid(__uint_as_float(zz[k] & 0xFFFF0000u));
                }
              }
              uint4 v;
              v.x = pack_bf16(e[0], e[1]);
              v.y = pack_bf16(e[2], e[3]);
              v.z = pack_bf16(e[4], e[5]);
              v.w = pack_bf16(e[6], e[7]);
              *reinterpret_cast<uint4*>(orow + c * 32 + i * 8) = v;
            }
          }
        }
      }
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (p.status != nullptr && *reinterpret_cast<volatile uint32_t*>(p.status) != 0u) {
    // a wait may have run out with copies still in flight: let them land before the memory is released
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) { __nanosleep(1000); }
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

template <int NBN, int NBV, bool SHARED>
int portion_attn_run(const PortionAttnParams& p, dim3 grid, cudaStream_t stream) {
  using S = PortionAttnSmem<NBN, NBV, SHARED>;
  static PerDeviceInt configured;
  if (!configured.cur()) {
    const cudaError_t e = cudaFuncSetAttribute(portion_attn_kernel<NBN, NBV, SHARED>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, S::kTotal);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.cur() = 1;
  }
  portion_attn_kernel<NBN, NBV, SHARED><<<grid, kLpThreads, S::kTotal, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <bool SHARED>
int portion_attn_dispatch(const PortionAttnParams& p, int max_q, int heads, int batch, cudaStream_t stream) {
  if ((max_q + kLpBlock - 1) / kLpBlock > 65535) return -3;
  dim3 grid(static_cast<unsigned>(heads), static_cast<unsigned>((max_q + kLpBlock - 1) / kLpBlock),
            static_cast<unsigned>(batch));
  if (p.dim <= 64)
    return p.vdim <= 64 ? portion_attn_run<1, 1, SHARED>(p, grid, stream) : portion_attn_run<1, 2, SHARED>(p, grid, stream);
  return p.vdim <= 64 ? portion_attn_run<2, 1, SHARED>(p, grid, stream) : portion_attn_run<2, 2, SHARED>(p, grid, stream);
}

// (size, head, row) map of heads `head_elems` apart in rows of `ld` elements; copies of 64 columns of `rows` rows
inline int portion_head_map(CUtensorMap* m, const void* base, int size, int64_t heads, int64_t head_elems, int64_t tokens,
                            int64_t ld, uint32_t rows) {
  return make_tmap_3d(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, base, static_cast<uint64_t>(size),
                      static_cast<uint64_t>(heads), static_cast<uint64_t>(tokens), static_cast<uint64_t>(head_elems) * 2,
                      static_cast<uint64_t>(ld) * 2, 64, 1, rows);
}

}  // namespace yv
