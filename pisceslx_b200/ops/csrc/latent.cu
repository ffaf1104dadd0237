// Latent attention: keys and values of all heads are linear maps of one low-rank latent per token, next to one rotated
// key part shared by the heads, and [latent | rotated key part] is all that the paged cache stores.
//   prep     norms of the two latents, rotation of the shared key part, cache append: one pass over the projection
//   query    rotation of the queries' rotary part (and the split into the latent-space query of a decode step)
//   prompts  attention over keys and values reconstructed for the visible part of the context
//   decode   attention over the latents themselves: the key map is folded into the query and the value map is
//            applied to the weighted sum, so a step reads kv_rank + rot_dim numbers per visible token for all heads
// Prompts and decode have a tensor-core kernel (latent_prefill.cuh, latent_decode.cuh) for bf16 and a CUDA-core kernel
// here for fp32 and for sizes the tensor-core kernels do not take.
#include "latent_ops.h"
#include "latent_decode.cuh"
#include "latent_prefill.cuh"
#include "per_device.h"
#include "sm100.cuh"
#include "tensormap.h"

namespace yv {

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xFFFFFFFFu, v, o));
  return v;
}

__device__ __forceinline__ void report(uint32_t* status, uint32_t bit) {
  if (status != nullptr) atomicOr(status, bit);
}

// Row of the angle tables for a position; a position outside them is reported and clamped.
__device__ __forceinline__ int table_row(const int* positions, int64_t t, int max_pos, uint32_t* status) {
  int pos = positions[t];
  if (pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0) report(status, kStatusIndexOutOfRange);
    pos = pos < 0 ? 0 : max_pos - 1;
  }
  return pos;
}

// Four consecutive elements (8 bytes of bf16, 16 of fp32).
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
constexpr int kPrepThreads = 128;
constexpr int kPrepVecs = 4;           // groups of four per thread and latent kept in registers

// One block per token, both latents in registers (ranks up to 2048, all sizes and pitches multiples of 8).
template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_vec_kernel(const LatentPrepArgs p) {
  __shared__ float red[2][kPrepThreads / 32];
  const int64_t t = blockIdx.x;
  const T* in = static_cast<const T*>(p.in) + t * p.ld;
  const T* kv = in + p.q_rank;
  const int nq = p.q_rank >> 2, nk = p.kv_rank >> 2;
  float q[kPrepVecs][4], k[kPrepVecs][4];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < kPrepVecs; ++i) {
    const int c = threadIdx.x + i * kPrepThreads;
#pragma unroll
    for (int j = 0; j < 4; ++j) q[i][j] = k[i][j] = 0.f;
    if (c < nq) load4(in + c * 4, q[i]);
    if (c < nk) load4(kv + c * 4, k[i]);
  }
#pragma unroll
  for (int i = 0; i < kPrepVecs; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) { sq += q[i][j] * q[i][j]; sk += k[i][j] * k[i][j]; }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < kPrepThreads / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float rq = 1.f / sqrtf(sq / static_cast<float>(p.q_rank) + p.eps);
  const float rk = 1.f / sqrtf(sk / static_cast<float>(p.kv_rank) + p.eps);
  const int row = p.kv_rank + p.rot_dim;
  T* out_rows = p.rows != nullptr ? static_cast<T*>(p.rows) + t * row : nullptr;
  T* out_cache = nullptr;
  if (p.cache != nullptr) {
    const int64_t slot = p.slot_map[t];
    if (slot >= p.num_slots) { if (threadIdx.x == 0) report(p.status, kStatusIndexOutOfRange); }
    else if (slot >= 0) out_cache = static_cast<T*>(p.cache) + slot * row;
  }
  auto put = [&](int i, const float (&f)[4]) {
    if (out_rows != nullptr) store4(out_rows + i, f);
    if (out_cache != nullptr) store4(out_cache + i, f);
  };
  T* cq = static_cast<T*>(p.cq) + t * p.cq_ld;
#pragma unroll
  for (int i = 0; i < kPrepVecs; ++i) {
    const int c = threadIdx.x + i * kPrepThreads;
    float w[4];
    if (c < nq) {
      load4(static_cast<const T*>(p.w_q) + c * 4, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) q[i][j] *= rq * w[j];
      store4(cq + c * 4, q[i]);
    }
    if (c < nk) {
      load4(static_cast<const T*>(p.w_kv) + c * 4, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) k[i][j] *= rk * w[j];
      put(c * 4, k[i]);
    }
  }
  const int half = p.rot_dim >> 1;
  const int64_t pos = table_row(p.positions, t, p.max_pos, p.status);
  for (int i = threadIdx.x * 4; i < half; i += kPrepThreads * 4) {
    float c[4], s[4], u[4], v[4], a[4], b[4];
    load4(p.cos_t + pos * half + i, c);
    load4(p.sin_t + pos * half + i, s);
    load4(kv + p.kv_rank + i, u);
    load4(kv + p.kv_rank + half + i, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) { a[j] = u[j] * c[j] - v[j] * s[j]; b[j] = v[j] * c[j] + u[j] * s[j]; }
    put(p.kv_rank + i, a);
    put(p.kv_rank + half + i, b);
  }
}

// One block per token, any sizes.
template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(const LatentPrepArgs p) {
  __shared__ float red[2][kPrepThreads / 32];
  const int64_t t = blockIdx.x;
  const T* in = static_cast<const T*>(p.in) + t * p.ld;
  const T* kv = in + p.q_rank;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < p.q_rank; i += kPrepThreads) { const float v = to_f(in[i]); sq += v * v; }
  for (int i = threadIdx.x; i < p.kv_rank; i += kPrepThreads) { const float v = to_f(kv[i]); sk += v * v; }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < kPrepThreads / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float rq = 1.f / sqrtf(sq / static_cast<float>(p.q_rank) + p.eps);
  const float rk = 1.f / sqrtf(sk / static_cast<float>(p.kv_rank) + p.eps);

  const int row = p.kv_rank + p.rot_dim;
  T* out_rows = p.rows != nullptr ? static_cast<T*>(p.rows) + t * row : nullptr;
  T* out_cache = nullptr;
  if (p.cache != nullptr) {
    const int64_t slot = p.slot_map[t];
    if (slot >= p.num_slots) { if (threadIdx.x == 0) report(p.status, kStatusIndexOutOfRange); }
    else if (slot >= 0) out_cache = static_cast<T*>(p.cache) + slot * row;
  }
  auto put = [&](int i, T v) {
    if (out_rows != nullptr) out_rows[i] = v;
    if (out_cache != nullptr) out_cache[i] = v;
  };
  T* cq = static_cast<T*>(p.cq) + t * p.cq_ld;
  for (int i = threadIdx.x; i < p.q_rank; i += kPrepThreads)
    cq[i] = from_f<T>(to_f(in[i]) * rq * to_f(static_cast<const T*>(p.w_q)[i]));
  for (int i = threadIdx.x; i < p.kv_rank; i += kPrepThreads)
    put(i, from_f<T>(to_f(kv[i]) * rk * to_f(static_cast<const T*>(p.w_kv)[i])));
  const int half = p.rot_dim >> 1;
  const int64_t pos = table_row(p.positions, t, p.max_pos, p.status);
  for (int i = threadIdx.x; i < half; i += kPrepThreads) {
    const float c = p.cos_t[pos * half + i], s = p.sin_t[pos * half + i];
    const float u = to_f(kv[p.kv_rank + i]), v = to_f(kv[p.kv_rank + half + i]);
    put(p.kv_rank + i, from_f<T>(u * c - v * s));
    put(p.kv_rank + half + i, from_f<T>(v * c + u * s));
  }
}

// Work items of N consecutive elements (4 or 1): all rotary pairs of all tokens, then all plain parts.
template <typename T, int N>
__global__ void __launch_bounds__(256) latent_query_kernel(const LatentQueryArgs p) {
  const int half = p.rot_dim >> 1, hv = half / N, dv = p.nope_out != nullptr ? p.dim / N : 0;
  const int per_head = hv + dv, hd = p.dim + p.rot_dim;
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  const int64_t th = i / per_head;
  const int e = static_cast<int>(i - th * per_head);
  const int64_t t = th / p.heads;
  const int h = static_cast<int>(th - t * p.heads);
  if (t >= p.T) return;
  const T* q = static_cast<const T*>(p.q) + t * p.ld + static_cast<int64_t>(h) * hd;
  if (e < hv) {
    int pos = p.positions[t];
    if (pos < 0 || pos >= p.max_pos) {
      report(p.status, kStatusIndexOutOfRange);
      pos = pos < 0 ? 0 : p.max_pos - 1;
    }
    const int j = e * N;
    const float* ct = p.cos_t + static_cast<int64_t>(pos) * half + j;
    const float* st = p.sin_t + static_cast<int64_t>(pos) * half + j;
    const T* src = q + p.dim + j;
    T* dst = static_cast<T*>(p.rope_out) + h * p.rope_hs + t * p.rope_ts + j;   // in place: one thread owns a pair
    if constexpr (N == 4) {
      float c[4], s[4], u[4], v[4], a[4], b[4];
      load4(ct, c); load4(st, s); load4(src, u); load4(src + half, v);
#pragma unroll
      for (int k = 0; k < 4; ++k) { a[k] = u[k] * c[k] - v[k] * s[k]; b[k] = v[k] * c[k] + u[k] * s[k]; }
      store4(dst, a);
      store4(dst + half, b);
    } else {
      const float u = to_f(src[0]), v = to_f(src[half]);
      dst[0] = from_f<T>(u * ct[0] - v * st[0]);
      dst[half] = from_f<T>(v * ct[0] + u * st[0]);
    }
  } else {
    const int j = (e - hv) * N;
    T* dst = static_cast<T*>(p.nope_out) + h * p.nope_hs + t * p.nope_ts + j;
    if constexpr (N == 4) { float f[4]; load4(q + j, f); store4(dst, f); }
    else dst[0] = q[j];
  }
}

// One warp per row.
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* __restrict__ cache, int64_t num_slots,
                                                            const int* __restrict__ slots, T* __restrict__ out, int64_t n,
                                                            int row, uint32_t* status) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (i >= n) return;
  const int64_t s = slots[i];
  const bool ok = s >= 0 && s < num_slots;
  if (!ok && lane == 0) report(status, kStatusIndexOutOfRange);
  const T* src = cache + (ok ? s : 0) * row;
  T* dst = out + i * row;
  if ((row * sizeof(T)) % 16 == 0) {
    const int nv = static_cast<int>(row * sizeof(T) / 16);
#pragma unroll 4
    for (int c = lane; c < nv; c += 32)
      reinterpret_cast<uint4*>(dst)[c] = ok ? reinterpret_cast<const uint4*>(src)[c] : make_uint4(0, 0, 0, 0);
  } else {
    for (int c = lane; c < row; c += 32) dst[c] = ok ? src[c] : from_f<T>(0.f);
  }
}

// ---- CUDA-core attention ---------------------------------------------------------------------------------------------
// A warp walks keys 32 at a time: lane i scores key i of the chunk, the softmax state is kept warp-wide, and the
// weighted sum is accumulated in shared memory (lanes over the value dimensions).

// prompts: one warp per (query, head)
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_simt_kernel(const LatentAttnArgs p) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.y;
  const int q0 = p.cu_q[b], nq = p.cu_q[b + 1] - q0;
  const int k0 = p.cu_k[b], nk = p.cu_k[b + 1] - k0;
  const int qi = blockIdx.x * 4 + warp;
  if (qi >= nq) return;
  const int hd = p.dim + p.rot_dim;
  float* sq = sm + warp * (hd + p.vdim);
  float* acc = sq + hd;
  const T* q = static_cast<const T*>(p.q) + static_cast<int64_t>(q0 + qi) * p.q_ld + static_cast<int64_t>(h) * hd;
  for (int i = lane; i < hd; i += 32) sq[i] = to_f(q[i]);
  for (int i = lane; i < p.vdim; i += 32) acc[i] = 0.f;
  __syncwarp();
  const int last = qi + nk - nq;                       // key index of the query itself
  int first = (p.window > 0 && last - p.window + 1 > 0) ? last - p.window + 1 : 0;
  const T* K = static_cast<const T*>(p.k) + static_cast<int64_t>(h) * p.dim;
  const T* V = static_cast<const T*>(p.v) + static_cast<int64_t>(h) * p.vdim;
  const T* R = static_cast<const T*>(p.kr);
  float m = -INFINITY, l = 0.f;
  for (int j0 = first; j0 <= last; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    if (j <= last) {
      const T* kp = K + static_cast<int64_t>(k0 + j) * p.k_ld;
      const T* rp = R + static_cast<int64_t>(k0 + j) * p.kr_ld;
      float d = 0.f;
      for (int i = 0; i < p.dim; ++i) d = fmaf(sq[i], to_f(kp[i]), d);
      for (int i = 0; i < p.rot_dim; ++i) d = fmaf(sq[p.dim + i], to_f(rp[i]), d);
      s = d * p.scale;
    }
    const float mn = fmaxf(m, warp_max(s));
    const float w = expf(s - mn), alpha = expf(m - mn);
    l = l * alpha + warp_sum(w);
    m = mn;
    const int n = min(32, last - j0 + 1);
    for (int i = lane; i < p.vdim; i += 32) acc[i] *= alpha;
    for (int k = 0; k < n; ++k) {
      const float wk = __shfl_sync(0xFFFFFFFFu, w, k);
      const T* vp = V + static_cast<int64_t>(k0 + j0 + k) * p.v_ld;
      for (int i = lane; i < p.vdim; i += 32) acc[i] = fmaf(wk, to_f(vp[i]), acc[i]);
    }
    __syncwarp();
  }
  float g = 1.f / l;
  if (p.gate != nullptr) {
    const float z = to_f(static_cast<const T*>(p.gate)[static_cast<int64_t>(q0 + qi) * p.gate_ld + h]);
    g *= 1.f / (1.f + expf(-z));
  }
  T* o = static_cast<T*>(p.o) + static_cast<int64_t>(q0 + qi) * p.o_ld + static_cast<int64_t>(h) * p.vdim;
  for (int i = lane; i < p.vdim; i += 32) o[i] = from_f<T>(acc[i] * g);
}

// decode: one block per (sequence, head); four warps take 32-key chunks in turn and are merged at the end
template <typename T>
__global__ void __launch_bounds__(128) latent_decode_simt_kernel(const LatentDecodeArgs p) {
  extern __shared__ float sm[];
  __shared__ float s_m[4], s_l[4];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, b = blockIdx.y;
  const int r = p.kv_rank, row = r + p.rot_dim;
  float* sq = sm;
  float* acc = sm + row + warp * r;
  int n = p.seq_lens[b];
  const int64_t cap = static_cast<int64_t>(p.max_blocks_per_seq) * p.block;
  if (n < 0 || n > cap) {
    if (threadIdx.x == 0) report(p.status, kStatusIndexOutOfRange);
    n = n < 0 ? 0 : static_cast<int>(cap);
  }
  const int64_t qrow = static_cast<int64_t>(h) * p.rows_pad + b;
  const T* q = static_cast<const T*>(p.q) + qrow * row;
  for (int i = threadIdx.x; i < row; i += 128) sq[i] = to_f(q[i]);
  for (int i = lane; i < r; i += 32) acc[i] = 0.f;
  __syncthreads();
  const int first = (p.window > 0 && n > p.window) ? n - p.window : 0;
  const T* cache = static_cast<const T*>(p.cache);
  const int* table = p.block_table + static_cast<int64_t>(b) * p.max_blocks_per_seq;
  float m = -1.0e30f, l = 0.f;
  for (int j0 = first + warp * 32; j0 < n; j0 += 128) {
    const int j = j0 + lane;
    int64_t slot = -1;
    float s = -INFINITY;
    if (j < n) {
      const int page = table[j / p.block];
      if (page >= 0 && page < p.num_blocks) slot = static_cast<int64_t>(page) * p.block + j % p.block;
      else report(p.status, kStatusIndexOutOfRange);
    }
    if (slot >= 0) {
      const T* kp = cache + slot * row;
      float d = 0.f;
      for (int i = 0; i < row; ++i) d = fmaf(sq[i], to_f(kp[i]), d);
      s = d * p.scale;
    }
    const float mn = fmaxf(m, warp_max(s));
    const float w = expf(s - mn), alpha = expf(m - mn);
    l = l * alpha + warp_sum(w);
    m = mn;
    for (int i = lane; i < r; i += 32) acc[i] *= alpha;
    const int cnt = min(32, n - j0);
    for (int k = 0; k < cnt; ++k) {
      const float wk = __shfl_sync(0xFFFFFFFFu, w, k);
      const int64_t sk = __shfl_sync(0xFFFFFFFFu, slot, k);
      if (sk < 0) continue;
      const T* vp = cache + sk * row;
      for (int i = lane; i < r; i += 32) acc[i] = fmaf(wk, to_f(vp[i]), acc[i]);
    }
    __syncwarp();
  }
  if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
  __syncthreads();
  const float M = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));
  float e[4], L = 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) { e[w] = expf(s_m[w] - M); L += s_l[w] * e[w]; }
  const float inv = L > 0.f ? 1.f / L : 0.f;
  T* o = static_cast<T*>(p.out) + qrow * r;
  for (int i = threadIdx.x; i < r; i += 128) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += sm[row + w * r + i] * e[w];
    o[i] = from_f<T>(v * inv);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) head_gate_kernel(const T* __restrict__ v, int64_t v_hs, int64_t v_ts,
                                                        const T* __restrict__ gate, int64_t gate_ld, T* __restrict__ out,
                                                        int64_t total, int heads, int vdim) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= total) return;
  const int j = static_cast<int>(i % vdim);
  const int64_t th = i / vdim;
  const int h = static_cast<int>(th % heads);
  const int64_t t = th / heads;
  float g = 1.f;
  if (gate != nullptr) g = 1.f / (1.f + expf(-to_f(gate[t * gate_ld + h])));
  out[i] = from_f<T>(to_f(v[h * v_hs + t * v_ts + j]) * g);
}

template <typename K>
int opt_in_smem(K kern, int bytes, PerDeviceInt& done) {
  if (bytes <= 48 * 1024 || done.cur() >= bytes) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return static_cast<int>(e);
  done.cur() = bytes;
  return 0;
}

constexpr int kMaxSmem = 227 * 1024;

}  // namespace

int launch_latent_prep(const LatentPrepArgs& a, cudaStream_t stream) {
  if (a.T <= 0) return 0;
  if (a.q_rank <= 0 || a.kv_rank <= 0 || a.rot_dim <= 0 || (a.rot_dim & 1) || a.max_pos <= 0) return -1;
  if (a.ld < a.q_rank + a.kv_rank + a.rot_dim || a.cq_ld < a.q_rank) return -2;
  if (a.cache != nullptr && a.slot_map == nullptr) return -3;
  const unsigned grid = static_cast<unsigned>(a.T);
  const int esz = a.dtype == 1 ? 4 : 2;
  auto al = [&](const void* p) { return (reinterpret_cast<uintptr_t>(p) % (4 * esz)) == 0; };
  const bool vec = ((a.q_rank | a.kv_rank | a.rot_dim) & 7) == 0 && ((a.ld | a.cq_ld) & 3) == 0 &&
                   a.q_rank <= 4 * kPrepVecs * kPrepThreads && a.kv_rank <= 4 * kPrepVecs * kPrepThreads && al(a.in) &&
                   al(a.cq) && al(a.rows) && al(a.cache) && al(a.w_q) && al(a.w_kv);
  if (vec && a.dtype == 1) latent_prep_vec_kernel<float><<<grid, kPrepThreads, 0, stream>>>(a);
  else if (vec) latent_prep_vec_kernel<__nv_bfloat16><<<grid, kPrepThreads, 0, stream>>>(a);
  else if (a.dtype == 1) latent_prep_kernel<float><<<grid, kPrepThreads, 0, stream>>>(a);
  else latent_prep_kernel<__nv_bfloat16><<<grid, kPrepThreads, 0, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

int launch_latent_query(const LatentQueryArgs& a, cudaStream_t stream) {
  if (a.T <= 0) return 0;
  if (a.heads <= 0 || a.dim < 0 || a.rot_dim <= 0 || (a.rot_dim & 1) || a.max_pos <= 0) return -1;
  const int esz = a.dtype == 1 ? 4 : 2;
  auto al = [&](const void* p) { return (reinterpret_cast<uintptr_t>(p) % (4 * esz)) == 0; };
  const bool vec = ((a.dim | (a.rot_dim >> 1)) & 3) == 0 && ((a.ld | a.nope_hs | a.nope_ts | a.rope_hs | a.rope_ts) & 3) == 0 &&
                   al(a.q) && al(a.nope_out) && al(a.rope_out);
  const int n = vec ? 4 : 1;
  const int64_t items = a.T * a.heads * ((a.rot_dim >> 1) / n + (a.nope_out != nullptr ? a.dim / n : 0));
  const unsigned grid = static_cast<unsigned>((items + 255) / 256);
  if (a.dtype == 1) {
    if (vec) latent_query_kernel<float, 4><<<grid, 256, 0, stream>>>(a);
    else latent_query_kernel<float, 1><<<grid, 256, 0, stream>>>(a);
  } else {
    if (vec) latent_query_kernel<__nv_bfloat16, 4><<<grid, 256, 0, stream>>>(a);
    else latent_query_kernel<__nv_bfloat16, 1><<<grid, 256, 0, stream>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

int launch_latent_gather(const void* cache, int64_t num_slots, const int* slots, void* out, int64_t n, int row,
                         int dtype, uint32_t* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  const unsigned grid = static_cast<unsigned>((n + 7) / 8);
  if (dtype == 1)
    latent_gather_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const float*>(cache), num_slots, slots,
                                                          static_cast<float*>(out), n, row, status);
  else
    latent_gather_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(static_cast<const __nv_bfloat16*>(cache), num_slots,
                                                                  slots, static_cast<__nv_bfloat16*>(out), n, row, status);
  return static_cast<int>(cudaGetLastError());
}

int launch_latent_attn(const LatentAttnArgs& a, cudaStream_t stream) {
  if (a.batch <= 0 || a.Tq <= 0) return 0;
  if (a.heads <= 0 || a.heads > 65535 || a.batch > 65535) return -1;
  if (!a.simt && latent_attn_on_tensor_cores(a)) return launch_latent_prefill_mma(a, stream);
  const int smem = 4 * 4 * (a.dim + a.rot_dim + a.vdim);
  if (smem > kMaxSmem) return -2;
  dim3 grid(static_cast<unsigned>((a.max_q + 3) / 4), static_cast<unsigned>(a.heads), static_cast<unsigned>(a.batch));
  int r;
  if (a.dtype == 1) {
    static PerDeviceInt done;
    if ((r = opt_in_smem(latent_attn_simt_kernel<float>, smem, done)) != 0) return r;
    latent_attn_simt_kernel<float><<<grid, 128, smem, stream>>>(a);
  } else {
    static PerDeviceInt done;
    if ((r = opt_in_smem(latent_attn_simt_kernel<__nv_bfloat16>, smem, done)) != 0) return r;
    latent_attn_simt_kernel<__nv_bfloat16><<<grid, 128, smem, stream>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

int launch_latent_decode(const LatentDecodeArgs& a, cudaStream_t stream) {
  if (a.batch <= 0) return 0;
  if (a.heads <= 0 || a.batch > 65535 || a.rows_pad < a.batch || a.block <= 0 || a.splits <= 0) return -1;
  if (!a.simt && latent_decode_on_tensor_cores(a)) return launch_latent_decode_mma(a, stream);
  const int smem = 4 * (a.kv_rank + a.rot_dim + 4 * a.kv_rank);
  if (smem > kMaxSmem) return -2;
  dim3 grid(static_cast<unsigned>(a.heads), static_cast<unsigned>(a.batch));
  int r;
  if (a.dtype == 1) {
    static PerDeviceInt done;
    if ((r = opt_in_smem(latent_decode_simt_kernel<float>, smem, done)) != 0) return r;
    latent_decode_simt_kernel<float><<<grid, 128, smem, stream>>>(a);
  } else {
    static PerDeviceInt done;
    if ((r = opt_in_smem(latent_decode_simt_kernel<__nv_bfloat16>, smem, done)) != 0) return r;
    latent_decode_simt_kernel<__nv_bfloat16><<<grid, 128, smem, stream>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

int launch_head_gate(const void* v, int64_t v_hs, int64_t v_ts, const void* gate, int64_t gate_ld, void* out,
                     int64_t T, int heads, int vdim, int dtype, cudaStream_t stream) {
  const int64_t total = T * heads * vdim;
  if (total <= 0) return 0;
  const unsigned grid = static_cast<unsigned>((total + 255) / 256);
  if (dtype == 1)
    head_gate_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const float*>(v), v_hs, v_ts,
                                                      static_cast<const float*>(gate), gate_ld, static_cast<float*>(out),
                                                      total, heads, vdim);
  else
    head_gate_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(
        static_cast<const __nv_bfloat16*>(v), v_hs, v_ts, static_cast<const __nv_bfloat16*>(gate), gate_ld,
        static_cast<__nv_bfloat16*>(out), total, heads, vdim);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace yv
