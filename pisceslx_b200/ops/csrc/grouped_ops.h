// Launcher declarations for grouped-query attention of layered models over pages of keys and values (grouped.cu).
// `dtype` is 0 for bf16 and 1 for fp32: activations, weights and pages of one call share it; angles, head norms, the
// query temperature, scores and softmax are fp32 in both.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace yv {

// Finishes the projections of T tokens: biases, unit norm of every query and key head, rotation of its first rot_dims
// numbers, the query temperature 1 + coef ln(floor((position + 1) / every) + 1).  Queries stay in place, keys and values
// go to row slot_map[t] (-1: nowhere; null map: row t) of pages [num_slots, kv_heads, size].
struct GroupedPrepArgs {
  void* q = nullptr; int64_t q_ld = 0;             // [T, heads, dim]
  const void* k = nullptr; int64_t k_ld = 0;       // [T, kv_heads, dim]
  const void* v = nullptr; int64_t v_ld = 0;       // [T, kv_heads, vdim]
  const void* bq = nullptr; const void* bk = nullptr; const void* bv = nullptr;   // optional, like one token's row
  void* k_pages = nullptr; void* v_pages = nullptr;
  const int* slot_map = nullptr;
  int64_t num_slots = 0;
  const int* positions = nullptr;                  // [T]
  const float* cos_t = nullptr; const float* sin_t = nullptr;   // [max_pos, rot_dims / 2]
  int max_pos = 0;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, rot_dims = 0;
  int unit = 0;                                    // 1: divide query and key heads by their root mean square
  float temp_coef = 0.f;
  int temp_every = 0;                              // 0: no temperature
  int64_t T = 0;
  float eps = 0.f;
  int dtype = 0;
  uint32_t* status = nullptr;
};
int launch_grouped_prep(const GroupedPrepArgs& a, cudaStream_t stream);

// Causal attention over pages [num_blocks, block, kv_heads, size]; the last query of a sequence sits at its last key.
struct GroupedAttnArgs {
  const void* q = nullptr; int64_t q_ld = 0;       // [Tq, heads, dim]
  const void* k = nullptr; const void* v = nullptr;
  const int* table = nullptr;                      // [batch, table_width] block numbers; null: key i of sequence b is
  int table_width = 0;                             // slot cu_q[b] + i, and there are as many keys as queries
  const int* lens = nullptr;                       // [batch] keys of every sequence (with a table)
  const int* cu_q = nullptr;                       // [batch + 1]; null: one query per sequence (a decode step)
  int batch = 0, max_q = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0, block = 0, num_blocks = 0;
  int64_t Tq = 0;
  float scale = 1.f;
  const void* sink = nullptr;                      // [heads] logits that only count in the denominator
  const void* gate = nullptr; int64_t gate_ld = 0; // logits of a sigmoid on the output, gate_step (1 or vdim) per head
  int gate_step = 1;
  void* o = nullptr; int64_t o_ld = 0;             // [Tq, heads, vdim]
  float* partial_o = nullptr;                      // decode with splits > 1: [batch, heads, splits, vdim]
  float* partial_ml = nullptr;                     // [batch, heads, splits, 2]
  int splits = 1;
  int dtype = 0;
  int simt = 0;                                    // 1: the CUDA-core kernel whatever the sizes
  uint32_t* status = nullptr;
};
int launch_grouped_attn(const GroupedAttnArgs& a, cudaStream_t stream);
int launch_grouped_decode(const GroupedAttnArgs& a, cudaStream_t stream);

}  // namespace yv
