// The fp32 residual stream around normed branches: the branch norm, the residual add and the norm in front of the
// next branch in one pass over a row, or a plain join (parts of a product, a table row, a vector) in front of one or two
// norms; the exact GELU, the gated SiLU and the per-layer token gate; and a CUDA-core product that keeps 32 bits (and
// takes operands of any size and pitch).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "stream_ops.h"
#include "sm100.cuh"

namespace yv {

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ void load4(const float* p, float (&f)[4]) {
  const float4 t = *reinterpret_cast<const float4*>(p);
  f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 t = *reinterpret_cast<const uint2*>(p);
  f[0] = __uint_as_float(t.x << 16); f[1] = __uint_as_float(t.x & 0xFFFF0000u);
  f[2] = __uint_as_float(t.y << 16); f[3] = __uint_as_float(t.y & 0xFFFF0000u);
}
__device__ __forceinline__ void store4(float* p, const float (&f)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&f)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]));
}

constexpr int kStreamThreads = 256;

// Sum over the block; every thread gets it.  `red` holds one float per warp.
__device__ __forceinline__ float block_sum_all(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  __syncthreads();                                   // earlier readers of `red` are done
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kStreamThreads / 32; ++i) t += red[i];
  return t;
}

// Branch row of output row `row`; -1 when the gather index is outside the table (reported, row treated as zeros).
__device__ __forceinline__ int64_t branch_row(const StreamNormArgs& p, int64_t row) {
  if (p.y_rows == nullptr) return row;
  const int64_t r = p.y_rows[row];
  if (r < 0 || r >= p.y_num_rows) {
    if (threadIdx.x == 0 && p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
    return -1;
  }
  return r;
}

// One block per row, the row in registers: VPT groups of four columns per thread.
template <typename T, typename TY, int VPT>
__global__ void __launch_bounds__(kStreamThreads) stream_norm_kernel(const StreamNormArgs p) {
  __shared__ float red[kStreamThreads / 32];
  const int64_t row = blockIdx.x;
  const int nvec = p.cols >> 2;
  float* xr = p.x + row * p.cols;
  float v[VPT][4];
  if (p.y != nullptr) {
    const int64_t yr = branch_row(p, row);
    const TY* y = static_cast<const TY*>(p.y) + (yr < 0 ? 0 : yr) * p.cols;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * kStreamThreads;
      v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
      if (c < nvec && yr >= 0) load4(y + c * 4, v[i]);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += v[i][j] * v[i][j];
    }
    const float r = 1.f / sqrtf(block_sum_all(ss, red) / static_cast<float>(p.cols) + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * kStreamThreads;
      if (c < nvec) {
        float w[4], x[4] = {0.f, 0.f, 0.f, 0.f};
        load4(static_cast<const T*>(p.w_y) + c * 4, w);
        if (!p.start) load4(xr + c * 4, x);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[i][j] = x[j] + v[i][j] * r * w[j];
        store4(xr + c * 4, v[i]);
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * kStreamThreads;
      v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
      if (c < nvec) load4(xr + c * 4, v[i]);
    }
  }
  if (p.h == nullptr) return;
  float r = 1.f;
  if (p.w_h != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += v[i][j] * v[i][j];
    r = 1.f / sqrtf(block_sum_all(ss, red) / static_cast<float>(p.cols) + p.eps);
  }
  T* h = static_cast<T*>(p.h) + row * p.cols;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * kStreamThreads;
    if (c < nvec) {
      float w[4] = {1.f, 1.f, 1.f, 1.f}, o[4];
      if (p.w_h != nullptr) load4(static_cast<const T*>(p.w_h) + c * 4, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = v[i][j] * r * w[j];
      store4(h + c * 4, o);
    }
  }
}

// Any row length: scalar accesses, the row is read again for the second norm.
template <typename T, typename TY>
__global__ void __launch_bounds__(kStreamThreads) stream_norm_any_kernel(const StreamNormArgs p) {
  __shared__ float red[kStreamThreads / 32];
  const int64_t row = blockIdx.x;
  float* xr = p.x + row * p.cols;
  float hs = 0.f;
  if (p.y != nullptr) {
    const int64_t yr = branch_row(p, row);
    const TY* y = static_cast<const TY*>(p.y) + (yr < 0 ? 0 : yr) * p.cols;
    float ss = 0.f;
    for (int c = threadIdx.x; c < p.cols; c += kStreamThreads) {
      const float v = yr < 0 ? 0.f : to_f(y[c]);
      ss += v * v;
    }
    const float r = 1.f / sqrtf(block_sum_all(ss, red) / static_cast<float>(p.cols) + p.eps);
    for (int c = threadIdx.x; c < p.cols; c += kStreamThreads) {
      const float v = yr < 0 ? 0.f : to_f(y[c]);
      const float n = (p.start ? 0.f : xr[c]) + v * r * to_f(static_cast<const T*>(p.w_y)[c]);
      xr[c] = n;
      hs += n * n;
    }
  } else {
    for (int c = threadIdx.x; c < p.cols; c += kStreamThreads) hs += xr[c] * xr[c];
  }
  if (p.h == nullptr) return;
  float r = 1.f;
  if (p.w_h != nullptr) r = 1.f / sqrtf(block_sum_all(hs, red) / static_cast<float>(p.cols) + p.eps);
  T* h = static_cast<T*>(p.h) + row * p.cols;
  for (int c = threadIdx.x; c < p.cols; c += kStreamThreads)
    h[c] = from_f<T>(xr[c] * r * (p.w_h != nullptr ? to_f(static_cast<const T*>(p.w_h)[c]) : 1.f));
}

template <typename T, typename TY>
int stream_norm_dispatch(const StreamNormArgs& a, cudaStream_t stream) {
  const unsigned grid = static_cast<unsigned>(a.rows);
  auto aligned = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) % bytes) == 0; };
  const bool vec = (a.cols % 4) == 0 && a.cols <= 8 * 4 * kStreamThreads && aligned(a.x, 16) &&
                   aligned(a.y, 4 * sizeof(TY)) && aligned(a.w_y, 4 * sizeof(T)) && aligned(a.w_h, 4 * sizeof(T)) &&
                   aligned(a.h, 4 * sizeof(T));
  if (!vec) stream_norm_any_kernel<T, TY><<<grid, kStreamThreads, 0, stream>>>(a);
  else if (a.cols <= 4 * kStreamThreads) stream_norm_kernel<T, TY, 1><<<grid, kStreamThreads, 0, stream>>>(a);
  else if (a.cols <= 2 * 4 * kStreamThreads) stream_norm_kernel<T, TY, 2><<<grid, kStreamThreads, 0, stream>>>(a);
  else if (a.cols <= 4 * 4 * kStreamThreads) stream_norm_kernel<T, TY, 4><<<grid, kStreamThreads, 0, stream>>>(a);
  else stream_norm_kernel<T, TY, 8><<<grid, kStreamThreads, 0, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// One block per row: the joined row in registers (VPT groups of four columns per thread), then up to two norms of it.
template <typename T, int VPT>
__global__ void __launch_bounds__(kStreamThreads) stream_add_kernel(const StreamAddArgs p) {
  __shared__ float red[kStreamThreads / 32];
  const int64_t row = blockIdx.x;
  const int nvec = p.cols >> 2;
  float* xr = p.x + row * p.cols;
  float v[VPT][4];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * kStreamThreads;
    v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
    if (!p.start && c < nvec) load4(xr + c * 4, v[i]);
  }
#pragma unroll 4
  for (int s = 0; s < p.num_parts; ++s) {
    const float* y = p.parts + s * p.part_stride + row * p.cols;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * kStreamThreads;
      float f[4] = {0.f, 0.f, 0.f, 0.f};
      if (c < nvec) load4(y + c * 4, f);
#pragma unroll
      for (int j = 0; j < 4; ++j) v[i][j] += f[j];
    }
  }
  const T* extra[2] = {nullptr, static_cast<const T*>(p.vec)};
  if (p.table != nullptr) {
    const int64_t id = p.table_rows[row];
    if (id >= 0 && id < p.table_num_rows) extra[0] = static_cast<const T*>(p.table) + id * p.cols;
    else if (threadIdx.x == 0 && p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    if (extra[e] == nullptr) continue;
    const float scale = e == 0 ? p.table_scale : 1.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * kStreamThreads;
      float f[4] = {0.f, 0.f, 0.f, 0.f};
      if (c < nvec) load4(extra[e] + c * 4, f);
#pragma unroll
      for (int j = 0; j < 4; ++j) v[i][j] += f[j] * scale;
    }
  }
  if (p.start || p.num_parts > 0 || p.table != nullptr || p.vec != nullptr) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * kStreamThreads;
      if (c < nvec) store4(xr + c * 4, v[i]);
    }
  }
  if (p.h[0] == nullptr) return;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) ss += v[i][j] * v[i][j];
  const float r = 1.f / sqrtf(block_sum_all(ss, red) / static_cast<float>(p.cols) + p.eps);
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    if (p.h[n] == nullptr) continue;
    T* h = static_cast<T*>(p.h[n]) + row * p.cols;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * kStreamThreads;
      if (c < nvec) {
        float w[4], o[4];
        load4(static_cast<const T*>(p.w[n]) + c * 4, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] = v[i][j] * r * (p.offset + w[j]);
        store4(h + c * 4, o);
      }
    }
  }
}

// Any row length: scalar accesses, the row is read again for the norms.
template <typename T>
__global__ void __launch_bounds__(kStreamThreads) stream_add_any_kernel(const StreamAddArgs p) {
  __shared__ float red[kStreamThreads / 32];
  const int64_t row = blockIdx.x;
  float* xr = p.x + row * p.cols;
  const T* tab = nullptr;
  if (p.table != nullptr) {
    const int64_t id = p.table_rows[row];
    if (id >= 0 && id < p.table_num_rows) tab = static_cast<const T*>(p.table) + id * p.cols;
    else if (threadIdx.x == 0 && p.status != nullptr) atomicOr(p.status, kStatusIndexOutOfRange);
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.cols; c += kStreamThreads) {
    float n = p.start ? 0.f : xr[c];
    for (int s = 0; s < p.num_parts; ++s) n += p.parts[s * p.part_stride + row * p.cols + c];
    if (tab != nullptr) n += to_f(tab[c]) * p.table_scale;
    if (p.vec != nullptr) n += to_f(static_cast<const T*>(p.vec)[c]);
    xr[c] = n;
    ss += n * n;
  }
  if (p.h[0] == nullptr) return;
  const float r = 1.f / sqrtf(block_sum_all(ss, red) / static_cast<float>(p.cols) + p.eps);
  for (int n = 0; n < 2; ++n) {
    if (p.h[n] == nullptr) continue;
    T* h = static_cast<T*>(p.h[n]) + row * p.cols;
    for (int c = threadIdx.x; c < p.cols; c += kStreamThreads)
      h[c] = from_f<T>(xr[c] * r * (p.offset + to_f(static_cast<const T*>(p.w[n])[c])));
  }
}

template <typename T>
int stream_add_dispatch(const StreamAddArgs& a, cudaStream_t stream) {
  const unsigned grid = static_cast<unsigned>(a.rows);
  auto aligned = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) % bytes) == 0; };
  bool vec = (a.cols % 4) == 0 && a.cols <= 8 * 4 * kStreamThreads && aligned(a.x, 16) && aligned(a.parts, 16) &&
             (a.part_stride % 4) == 0;
  for (const void* q : {a.table, a.vec, a.w[0], a.w[1], static_cast<const void*>(a.h[0]), static_cast<const void*>(a.h[1])})
    vec = vec && aligned(q, 4 * sizeof(T));
  if (!vec) stream_add_any_kernel<T><<<grid, kStreamThreads, 0, stream>>>(a);
  else if (a.cols <= 4 * kStreamThreads) stream_add_kernel<T, 1><<<grid, kStreamThreads, 0, stream>>>(a);
  else if (a.cols <= 2 * 4 * kStreamThreads) stream_add_kernel<T, 2><<<grid, kStreamThreads, 0, stream>>>(a);
  else if (a.cols <= 4 * 4 * kStreamThreads) stream_add_kernel<T, 4><<<grid, kStreamThreads, 0, stream>>>(a);
  else stream_add_kernel<T, 8><<<grid, kStreamThreads, 0, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// out[t, j] = silu(in[t, j]) * in[t, F + j], N elements (8 or 1) per thread
template <typename T, int N>
__global__ void __launch_bounds__(256) gated_silu_kernel(const T* __restrict__ in, int64_t in_ld, T* __restrict__ out,
                                                         int64_t out_ld, int F) {
  const int64_t t = blockIdx.x;
  const int j = (blockIdx.y * 256 + threadIdx.x) * N;
  if (j >= F) return;
  const T* g = in + t * in_ld + j;
  T* o = out + t * out_ld + j;
  auto act = [](float z, float u) { return z / (1.f + expf(-z)) * u; };
  if constexpr (N == 8) {
    float a[2][4], b[2][4];
#pragma unroll
    for (int q = 0; q < 2; ++q) { load4(g + q * 4, a[q]); load4(g + F + q * 4, b[q]); }
#pragma unroll
    for (int q = 0; q < 2; ++q) {
#pragma unroll
      for (int k = 0; k < 4; ++k) a[q][k] = act(a[q][k], b[q][k]);
      store4(o + q * 4, a[q]);
    }
  } else {
    o[0] = from_f<T>(act(to_f(g[0]), to_f(g[F])));
  }
}

template <typename T>
int gated_silu_dispatch(const void* in, int64_t in_ld, void* out, int64_t out_ld, int64_t rows, int F, cudaStream_t stream) {
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) % (4 * sizeof(T))) == 0; };
  const bool vec = (F % 8) == 0 && (in_ld % 4) == 0 && (out_ld % 4) == 0 && al(in) && al(out);
  const int blocks = ((vec ? F / 8 : F) + 255) / 256;
  if (rows > 0x7FFFFFFFll || blocks > 65535) return -1;
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>(blocks));
  if (vec) gated_silu_kernel<T, 8><<<grid, 256, 0, stream>>>(static_cast<const T*>(in), in_ld, static_cast<T*>(out), out_ld, F);
  else gated_silu_kernel<T, 1><<<grid, 256, 0, stream>>>(static_cast<const T*>(in), in_ld, static_cast<T*>(out), out_ld, F);
  return static_cast<int>(cudaGetLastError());
}

__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.f + erff(z * 0.7071067811865476f)); }
__device__ __forceinline__ float gelu_tanh(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename T>
__global__ void __launch_bounds__(256) gelu_kernel(const T* __restrict__ in, T* __restrict__ out, int64_t n) {
  // four groups of four per thread, all loads before the arithmetic
  const int64_t i0 = static_cast<int64_t>(blockIdx.x) * 4096 + threadIdx.x * 4;
  float f[4][4];
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    const int64_t i = i0 + u * 1024;
    if (i + 4 <= n) load4(in + i, f[u]);
  }
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    const int64_t i = i0 + u * 1024;
    if (i + 4 <= n) {
#pragma unroll
      for (int j = 0; j < 4; ++j) f[u][j] = gelu_erf(f[u][j]);
      store4(out + i, f[u]);
    } else {
      for (int64_t j = i; j < n; ++j) out[j] = from_f<T>(gelu_erf(to_f(in[j])));
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) token_gate_kernel(const T* __restrict__ a, int64_t a_stride, const T* __restrict__ table,
                                                         int64_t table_stride, int64_t vocab, int64_t offset,
                                                         const int64_t* __restrict__ token, T* __restrict__ out,
                                                         int64_t rows, int dim, uint32_t* status) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= rows * dim) return;
  const int64_t t = i / dim;
  const int j = static_cast<int>(i - t * dim);
  const int64_t id = token[t];
  if (id < 0 || id >= vocab) {
    if (status != nullptr && j == 0) atomicOr(status, kStatusIndexOutOfRange);
    out[i] = from_f<T>(0.f);
    return;
  }
  out[i] = from_f<T>(gelu_tanh(to_f(a[t * a_stride + j])) * to_f(table[id * table_stride + offset + j]));
}

// 64 x 64 output tile, 256 threads of 4 x 4 outputs, 16 columns of K at a time.
template <typename T, typename TC>
__global__ void __launch_bounds__(256) linear_simt_kernel(const LinearSimtArgs p) {
  __shared__ float sa[16][68], sb[16][68];
  const int64_t g = blockIdx.z;
  const int64_t m0 = static_cast<int64_t>(blockIdx.y) * 64, n0 = static_cast<int64_t>(blockIdx.x) * 64;
  const T* A = static_cast<const T*>(p.a) + g * p.a_group;
  const T* B = static_cast<const T*>(p.b) + g * p.b_group;
  TC* C = static_cast<TC*>(p.c) + g * p.c_group;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int64_t k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = threadIdx.x + i * 256, r = e >> 4, c = e & 15;
      const bool kin = k0 + c < p.K;
      sa[c][r] = (kin && m0 + r < p.M) ? to_f(A[(m0 + r) * p.lda + k0 + c]) : 0.f;
      sb[c][r] = (kin && n0 + r < p.N) ? to_f(B[(n0 + r) * p.ldb + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float av[4], bv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { av[i] = sa[k][ty * 4 + i]; bv[i] = sb[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int64_t m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < p.M && n < p.N) C[m * p.ldc + n] = from_f<TC>(acc[i][j]);
    }
}

}  // namespace

int launch_stream_norm(const StreamNormArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  if (a.x == nullptr || a.cols <= 0 || (a.y != nullptr && a.w_y == nullptr) || (a.start && a.y == nullptr)) return -1;
  if (a.rows > 0x7FFFFFFFll) return -2;
  if (a.dtype == 1) return stream_norm_dispatch<float, float>(a, stream);
  return a.y_fp32 ? stream_norm_dispatch<__nv_bfloat16, float>(a, stream)
                  : stream_norm_dispatch<__nv_bfloat16, __nv_bfloat16>(a, stream);
}

int launch_stream_add(const StreamAddArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  if (a.x == nullptr || a.cols <= 0 || (a.num_parts > 0 && a.parts == nullptr) || (a.table != nullptr && a.table_rows == nullptr)) return -1;
  if (a.rows > 0x7FFFFFFFll || (a.h[0] == nullptr && a.h[1] != nullptr)) return -2;
  for (int n = 0; n < 2; ++n)
    if (a.h[n] != nullptr && a.w[n] == nullptr) return -3;
  return a.dtype == 1 ? stream_add_dispatch<float>(a, stream) : stream_add_dispatch<__nv_bfloat16>(a, stream);
}

int launch_gated_silu(const void* in, int64_t in_ld, void* out, int64_t out_ld, int64_t rows, int F, int dtype,
                      cudaStream_t stream) {
  if (rows <= 0 || F <= 0) return 0;
  return dtype == 1 ? gated_silu_dispatch<float>(in, in_ld, out, out_ld, rows, F, stream)
                    : gated_silu_dispatch<__nv_bfloat16>(in, in_ld, out, out_ld, rows, F, stream);
}

int launch_gelu(const void* in, void* out, int64_t n, int dtype, cudaStream_t stream) {
  if (n <= 0) return 0;
  if ((reinterpret_cast<uintptr_t>(in) & 15u) != 0 || (reinterpret_cast<uintptr_t>(out) & 15u) != 0) return -1;
  const unsigned grid = static_cast<unsigned>((n + 4095) / 4096);
  if (dtype == 1) gelu_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const float*>(in), static_cast<float*>(out), n);
  else gelu_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(static_cast<const __nv_bfloat16*>(in),
                                                            static_cast<__nv_bfloat16*>(out), n);
  return static_cast<int>(cudaGetLastError());
}

int launch_token_gate(const void* a, int64_t a_stride, const void* table, int64_t table_stride, int64_t vocab,
                      int64_t offset, const int64_t* token, void* out, int64_t rows, int dim, int dtype,
                      uint32_t* status, cudaStream_t stream) {
  if (rows <= 0 || dim <= 0) return 0;
  const unsigned grid = static_cast<unsigned>((rows * dim + 255) / 256);
  if (dtype == 1)
    token_gate_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const float*>(a), a_stride,
                                                       static_cast<const float*>(table), table_stride, vocab, offset,
                                                       token, static_cast<float*>(out), rows, dim, status);
  else
    token_gate_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(
        static_cast<const __nv_bfloat16*>(a), a_stride, static_cast<const __nv_bfloat16*>(table), table_stride, vocab,
        offset, token, static_cast<__nv_bfloat16*>(out), rows, dim, status);
  return static_cast<int>(cudaGetLastError());
}

int launch_linear_simt(const LinearSimtArgs& a, cudaStream_t stream) {
  if (a.M <= 0 || a.N <= 0 || a.groups <= 0) return 0;
  if (a.K <= 0 || a.groups > 65535 || (a.M + 63) / 64 > 65535) return -1;
  dim3 grid(static_cast<unsigned>((a.N + 63) / 64), static_cast<unsigned>((a.M + 63) / 64),
            static_cast<unsigned>(a.groups));
  if (a.dtype == 1) linear_simt_kernel<float, float><<<grid, 256, 0, stream>>>(a);
  else if (a.out_fp32) linear_simt_kernel<__nv_bfloat16, float><<<grid, 256, 0, stream>>>(a);
  else linear_simt_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, 256, 0, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace yv
