// Launcher declarations for latent (low-rank key/value) attention (latent.cu).  `dtype` is 0 for bf16 and 1 for fp32:
// activations, weights and cache rows of one call share it; the angles, the scores and every norm are fp32 in both.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace yv {

// ------------------------------------------------------------------------------------------------
// latent.cu
// ------------------------------------------------------------------------------------------------
struct LatentPrepArgs {
  const void* in = nullptr;        // [T, ld]: columns [query latent | key/value latent | rotary key | ...]
  int64_t ld = 0;
  int q_rank = 0, kv_rank = 0, rot_dim = 0;
  const void* w_q = nullptr; const void* w_kv = nullptr;   // norm weights
  const float* cos_t = nullptr; const float* sin_t = nullptr;   // [max_pos, rot_dim / 2]
  const int* positions = nullptr;
  int max_pos = 0;
  void* cq = nullptr;              // [T, cq_ld] normed query latent
  int64_t cq_ld = 0;
  void* rows = nullptr;            // optional [T, kv_rank + rot_dim]: normed latent | rotated key part
  void* cache = nullptr;           // optional [num_slots, kv_rank + rot_dim], the same row at slot_map[t]
  const int* slot_map = nullptr;   // -1 = do not store
  int64_t num_slots = 0;
  int64_t T = 0;
  float eps = 0.f;
  int dtype = 0;
  uint32_t* status = nullptr;
};
int launch_latent_prep(const LatentPrepArgs& a, cudaStream_t stream);

// q [T, heads * (dim + rot_dim)]: the rotary part is rotated into rope_out + h * rope_hs + t * rope_ts, the plain part
// copied to nope_out + h * nope_hs + t * nope_ts unless nope_out is null.  rope_out may address q itself.
struct LatentQueryArgs {
  const void* q = nullptr; int64_t ld = 0;
  int heads = 0, dim = 0, rot_dim = 0;
  const float* cos_t = nullptr; const float* sin_t = nullptr; const int* positions = nullptr; int max_pos = 0;
  void* nope_out = nullptr; int64_t nope_hs = 0, nope_ts = 0;
  void* rope_out = nullptr; int64_t rope_hs = 0, rope_ts = 0;
  int64_t T = 0;
  int dtype = 0;
  uint32_t* status = nullptr;
};
int launch_latent_query(const LatentQueryArgs& a, cudaStream_t stream);

// out[i] = cache[slots[i]]
int launch_latent_gather(const void* cache, int64_t num_slots, const int* slots, void* out, int64_t n, int row,
                         int dtype, uint32_t* status, cudaStream_t stream);

// Prompt attention over reconstructed keys and values.  Sequence b has queries cu_q[b]..cu_q[b+1] and keys
// cu_k[b]..cu_k[b+1]; the last query sits at the last key.  A query sees itself and the window - 1 keys before it
// (window <= 0: everything before it).
struct LatentAttnArgs {
  const void* q = nullptr; int64_t q_ld = 0;       // [Tq, heads, dim + rot_dim], rotated
  const void* k = nullptr; int64_t k_ld = 0;       // [Tk, heads, dim]
  const void* v = nullptr; int64_t v_ld = 0;       // [Tk, heads, vdim]
  const void* kr = nullptr; int64_t kr_ld = 0;     // [Tk, rot_dim], rotated, shared by the heads
  const void* gate = nullptr; int64_t gate_ld = 0; // optional logits [Tq, heads]: outputs scaled by their sigmoid
  void* o = nullptr; int64_t o_ld = 0;             // [Tq, heads, vdim]
  const int* cu_q = nullptr; const int* cu_k = nullptr;
  int batch = 0, max_q = 0, heads = 0, dim = 0, rot_dim = 0, vdim = 0, window = 0;
  int64_t Tq = 0, Tk = 0;
  float scale = 1.f;
  int dtype = 0;
  int simt = 0;                                    // 1: the CUDA-core kernel whatever the sizes
  uint32_t* status = nullptr;
};
int launch_latent_attn(const LatentAttnArgs& a, cudaStream_t stream);
inline bool latent_attn_on_tensor_cores(const LatentAttnArgs& a);

// One query token per batch row in the latent space.  q [heads, rows_pad, kv_rank + rot_dim] = [W_uk^T q | q rotated];
// the weighted sum of the latents goes to out [heads, rows_pad, kv_rank].
struct LatentDecodeArgs {
  const void* q = nullptr; const void* cache = nullptr;
  const int* block_table = nullptr; const int* seq_lens = nullptr;
  void* out = nullptr;
  float* partial_o = nullptr;      // [B, heads, splits, kv_rank] scratch when splits > 1
  float* partial_ml = nullptr;     // [B, heads, splits, 2]
  int batch = 0, heads = 0, kv_rank = 0, rot_dim = 0, block = 64, max_blocks_per_seq = 0, num_blocks = 0, window = 0;
  int64_t rows_pad = 0;
  int splits = 1;
  float scale = 1.f;
  int dtype = 0;
  int simt = 0;
  uint32_t* status = nullptr;
};
int launch_latent_decode(const LatentDecodeArgs& a, cudaStream_t stream);
inline bool latent_decode_on_tensor_cores(const LatentDecodeArgs& a);

// out[t, h * vdim + j] = v[h, t, j] * sigmoid(gate[t, h])   (gate null: a plain transpose)
int launch_head_gate(const void* v, int64_t v_hs, int64_t v_ts, const void* gate, int64_t gate_ld, void* out,
                     int64_t T, int heads, int vdim, int dtype, cudaStream_t stream);

}  // namespace yv
