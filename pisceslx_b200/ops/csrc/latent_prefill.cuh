// Prompt attention of latent layers: the portion kernel over reconstructed keys and values in packed rows, with the rotated
// key part shared by the heads.
#pragma once
#include "latent_ops.h"
#include "portion_attention.cuh"

namespace yv {

// The tensor-core kernel takes bf16, parts of up to 128 + 64 columns and values of up to 128, all sizes and pitches
// multiples of 8 elements, and a positive scale (the row maximum is taken before scaling).
inline bool latent_attn_on_tensor_cores(const LatentAttnArgs& a) {
  auto mul8 = [](int64_t v) { return (v & 7) == 0; };
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
  return a.dtype == 0 && a.scale > 0.f && a.dim > 0 && a.dim <= 128 && a.rot_dim > 0 && a.rot_dim <= 64 && a.vdim > 0 &&
         a.vdim <= 128 && mul8(a.dim) && mul8(a.rot_dim) && mul8(a.vdim) && mul8(a.q_ld) && mul8(a.k_ld) &&
         mul8(a.v_ld) && mul8(a.kr_ld) && mul8(a.o_ld) && al16(a.q) && al16(a.k) && al16(a.v) && al16(a.kr) && al16(a.o);
}

inline int launch_latent_prefill_mma(const LatentAttnArgs& a, cudaStream_t stream) {
  PortionAttnParams p = {};
  const int hd = a.dim + a.rot_dim;
  int r = portion_head_map(&p.tma_qn, a.q, a.dim, a.heads, hd, a.Tq, a.q_ld, kLpBlock);
  if (r != 0) return -10 + r;
  r = portion_head_map(&p.tma_qr, static_cast<const __nv_bfloat16*>(a.q) + a.dim, a.rot_dim, a.heads, hd, a.Tq, a.q_ld, kLpBlock);
  if (r != 0) return -20 + r;
  r = portion_head_map(&p.tma_k, a.k, a.dim, a.heads, a.dim, a.Tk, a.k_ld, 64);
  if (r != 0) return -30 + r;
  r = portion_head_map(&p.tma_v, a.v, a.vdim, a.heads, a.vdim, a.Tk, a.v_ld, 64);
  if (r != 0) return -40 + r;
  r = make_tmap_2d(&p.tma_kr, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.kr, static_cast<uint64_t>(a.rot_dim),
                   static_cast<uint64_t>(a.Tk), static_cast<uint64_t>(a.kr_ld), 64, 64);
  if (r != 0) return -50 + r;
  p.o = static_cast<__nv_bfloat16*>(a.o); p.o_ld = a.o_ld;
  p.gate = static_cast<const __nv_bfloat16*>(a.gate); p.gate_ld = a.gate_ld; p.gate_step = 1;
  p.cu_q = a.cu_q; p.cu_k = a.cu_k;
  p.dim = a.dim; p.rot_dim = a.rot_dim; p.vdim = a.vdim; p.window = a.window; p.group = 1;
  p.scale_log2 = a.scale * kLpLog2e;
  p.status = a.status;
  return portion_attn_dispatch<true>(p, a.max_q, a.heads, a.batch, stream);
}

}  // namespace yv
