// Launcher declarations for the fp32 residual stream of layered models, their activations and the exact products
// (stream.cu).  `dtype` is 0 for bf16 and 1 for fp32: activations and weights of one call share it; the stream and every
// norm are fp32 in both.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace yv {

struct StreamNormArgs {
  float* x = nullptr;              // fp32 stream [rows, cols]; read unless `start`, written when y is given
  const void* y = nullptr;         // branch output [.., cols] (dtype, or fp32 with y_fp32), null = nothing to add
  const int64_t* y_rows = nullptr; // optional gather: row t of the branch is y[y_rows[t]]
  int64_t y_num_rows = 0;          // rows of y when gathered
  const void* w_y = nullptr;       // weight of the norm on the branch
  const void* w_h = nullptr;       // weight of the norm in front of the next branch; null = h is the plain stream
  void* h = nullptr;               // dtype [rows, cols], null = not wanted
  int64_t rows = 0;
  int cols = 0;
  int start = 0;                   // 1: the stream starts here, x = rms(y) * w_y
  int y_fp32 = 0;
  float eps = 0.f;
  int dtype = 0;
  uint32_t* status = nullptr;
};
// x (+)= rms(y) * w_y;  h = rms(x) * w_h (or x).  rms(v) = v / sqrt(mean(v^2) + eps)
int launch_stream_norm(const StreamNormArgs& a, cudaStream_t stream);
struct StreamAddArgs {
  float* x = nullptr;              // fp32 stream [rows, cols]; read unless `start`, written when anything is added
  const float* parts = nullptr;    // [num_parts][.., cols]: row t of part s is parts[s * part_stride + t * cols]
  int num_parts = 0;
  int64_t part_stride = 0;
  const void* table = nullptr;     // dtype [table_num_rows, cols]; row t adds table_scale * table[table_rows[t]]
  const int64_t* table_rows = nullptr;
  int64_t table_num_rows = 0;
  float table_scale = 1.f;
  const void* vec = nullptr;       // dtype [cols], added to every row
  const void* w[2] = {nullptr, nullptr};   // norm weights, dtype [cols]
  void* h[2] = {nullptr, nullptr}; // dtype [rows, cols]: rms(x) * (offset + w); null = not wanted
  float offset = 0.f;
  int64_t rows = 0;
  int cols = 0;
  int start = 0;
  float eps = 0.f;
  int dtype = 0;
  uint32_t* status = nullptr;
};
int launch_stream_add(const StreamAddArgs& a, cudaStream_t stream);
// out[t, j] = silu(in[t, j]) * in[t, F + j],  j < F; row pitches in elements
int launch_gated_silu(const void* in, int64_t in_ld, void* out, int64_t out_ld, int64_t rows, int F, int dtype,
                      cudaStream_t stream);
// out = gelu(in) with the error function; n elements
int launch_gelu(const void* in, void* out, int64_t n, int dtype, cudaStream_t stream);
// out[t, j] = gelu_tanh(a[t, j]) * table[token[t], offset + j],  j < dim
int launch_token_gate(const void* a, int64_t a_stride, const void* table, int64_t table_stride, int64_t vocab,
                      int64_t offset, const int64_t* token, void* out, int64_t rows, int dim, int dtype,
                      uint32_t* status, cudaStream_t stream);
// C[g][m][n] = sum_k A[g][m][k] * B[g][n][k] on the CUDA cores with fp32 accumulation: the exact 32-bit product, and
// the product for operands a tensor map cannot describe.  Strides in elements.
struct LinearSimtArgs {
  const void* a = nullptr; const void* b = nullptr; void* c = nullptr;
  int64_t M = 0, N = 0, K = 0, groups = 1;
  int64_t lda = 0, ldb = 0, ldc = 0, a_group = 0, b_group = 0, c_group = 0;
  int dtype = 0, out_fp32 = 0;
};
int launch_linear_simt(const LinearSimtArgs& a, cudaStream_t stream);

}  // namespace yv
