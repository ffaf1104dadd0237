// Grouped-query attention of layered models: keys and values in pages, query / key and value heads of sizes of their own.
//   prep     biases, head norms, partial rotation, query temperature and the cache append: one pass over the projection
//   prompts  attention of a portion of a prompt over the pages
//   decode   attention of one query per sequence over the pages, cut into key ranges that a merge kernel joins
// Prompts and decode have a tensor-core kernel for bf16 (portion_attention.cuh, attention_decode_mma.cuh) and one
// CUDA-core kernel here for fp32 and for sizes the tensor-core kernels do not take.
#include <cuda_bf16.h>
#include <math.h>

#include "attention_decode_mma.cuh"
#include "grouped_ops.h"
#include "portion_attention.cuh"

namespace yv {

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 t = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u); }
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}

__device__ __forceinline__ void report(uint32_t* status) {
  if (status != nullptr) atomicOr(status, kStatusIndexOutOfRange);
}

// ---- prep ------------------------------------------------------------------------------------------------------------
// One head of one token: where it is read, its bias, where it goes, and what is done to it.
template <typename T>
struct PrepUnit {
  const T* src;
  const T* bias;       // null = none
  T* dst;              // null = not stored
  int size;
  bool is_v, is_q;
};

// Unit u of token t: query heads, then key heads, then value heads.
template <typename T>
__device__ __forceinline__ PrepUnit<T> prep_unit(const GroupedPrepArgs& p, int64_t t, int u, bool lead) {
  PrepUnit<T> r;
  if (u < p.heads) {
    T* q = static_cast<T*>(p.q) + t * p.q_ld + static_cast<int64_t>(u) * p.dim;
    r.src = q; r.dst = q; r.size = p.dim; r.is_q = true; r.is_v = false;
    r.bias = p.bq != nullptr ? static_cast<const T*>(p.bq) + static_cast<int64_t>(u) * p.dim : nullptr;
    return r;
  }
  r.is_q = false;
  r.is_v = u >= p.heads + p.kv_heads;
  const int g = u - p.heads - (r.is_v ? p.kv_heads : 0);
  r.size = r.is_v ? p.vdim : p.dim;
  const int64_t at = static_cast<int64_t>(g) * r.size;
  r.src = static_cast<const T*>(r.is_v ? p.v : p.k) + t * (r.is_v ? p.v_ld : p.k_ld) + at;
  const void* b = r.is_v ? p.bv : p.bk;
  r.bias = b != nullptr ? static_cast<const T*>(b) + at : nullptr;
  const int64_t slot = p.slot_map != nullptr ? p.slot_map[t] : t;
  r.dst = nullptr;
  if (slot >= p.num_slots) { if (lead) report(p.status); }
  else if (slot >= 0) r.dst = static_cast<T*>(r.is_v ? p.v_pages : p.k_pages) + slot * p.kv_heads * r.size + at;
  return r;
}

// Row of the angle tables for a position; a position outside them is reported and clamped.
__device__ __forceinline__ int64_t angle_row(const GroupedPrepArgs& p, int pos, bool lead) {
  if (pos < 0 || pos >= p.max_pos) {
    if (lead) report(p.status);
    pos = pos < 0 ? 0 : p.max_pos - 1;
  }
  return static_cast<int64_t>(pos) * (p.rot_dims >> 1);
}

__device__ __forceinline__ float query_factor(const GroupedPrepArgs& p, int pos) {
  return 1.f + p.temp_coef * logf(static_cast<float>((pos + 1) / p.temp_every) + 1.f);
}

// LANES (8 or 16) lanes to a head of up to 8 LANES numbers, eight numbers to a lane (sizes, pitches and half the rotated
// part are multiples of 8).  The other number of a rotated pair sits half / 8 lanes away.
template <typename T, int LANES>
__global__ void __launch_bounds__(256) grouped_prep_vec_kernel(const GroupedPrepArgs p) {
  const int64_t t = blockIdx.x;
  int u = blockIdx.y * (256 / LANES) + threadIdx.x / LANES;
  const bool real = u < p.heads + 2 * p.kv_heads;               // whole warps stay together for the shuffles
  if (!real) u = 0;
  const int lane = threadIdx.x % LANES, c = lane * 8;
  const bool lead = real && lane == 0;
  const PrepUnit<T> w = prep_unit<T>(p, t, u, lead);
  const bool in = c < w.size;
  float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (in) {
    load8(w.src + c, f);
    if (w.bias != nullptr) {
      float b[8];
      load8(w.bias + c, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] += b[j];
    }
  }
  if (p.unit) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o, LANES);
    if (!w.is_v) {
      const float r = 1.f / sqrtf(ss / static_cast<float>(w.size) + p.eps);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= r;
    }
  }
  if (p.rot_dims > 0) {
    const int half = p.rot_dims >> 1, step = half >> 3;
    const bool low = c < half, turned = c < p.rot_dims && !w.is_v;
    const int peer = (low ? lane + step : lane - step) & (LANES - 1);
    float g[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) g[j] = __shfl_sync(0xFFFFFFFFu, f[j], peer, LANES);
    if (turned) {
      const int64_t row = angle_row(p, p.positions[t], lead) + (low ? c : c - half);
      float cs[8], sn[8];
      load8(p.cos_t + row, cs);
      load8(p.sin_t + row, sn);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = low ? f[j] * cs[j] - g[j] * sn[j] : f[j] * cs[j] + g[j] * sn[j];
    }
  }
  if (w.is_q && p.temp_every > 0) {
    const float s = query_factor(p, p.positions[t]);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= s;
  }
  if (real && in && w.dst != nullptr) store8(w.dst + c, f);
}

// One warp per head, any sizes; a lane owns whole pairs, so queries can be finished in place.
template <typename T>
__global__ void __launch_bounds__(256) grouped_prep_kernel(const GroupedPrepArgs p) {
  const int64_t t = blockIdx.x;
  const int u = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (u >= p.heads + 2 * p.kv_heads) return;
  const int lane = threadIdx.x & 31;
  const PrepUnit<T> w = prep_unit<T>(p, t, u, lane == 0);
  auto at = [&](int c) { return to_f(w.src[c]) + (w.bias != nullptr ? to_f(w.bias[c]) : 0.f); };
  float r = 1.f;
  if (p.unit && !w.is_v) {
    float ss = 0.f;
    for (int c = lane; c < w.size; c += 32) { const float f = at(c); ss += f * f; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    r = 1.f / sqrtf(ss / static_cast<float>(w.size) + p.eps);
  }
  if (w.dst == nullptr) return;
  const int pos = p.positions[t];
  const float s = w.is_q && p.temp_every > 0 ? query_factor(p, pos) : 1.f;
  const int rot = w.is_v ? 0 : p.rot_dims, half = rot >> 1;
  if (rot > 0) {
    const int64_t row = angle_row(p, pos, lane == 0);
    for (int c = lane; c < half; c += 32) {
      const float cs = p.cos_t[row + c], sn = p.sin_t[row + c];
      const float a = at(c) * r, b = at(c + half) * r;
      w.dst[c] = from_f<T>((a * cs - b * sn) * s);
      w.dst[c + half] = from_f<T>((b * cs + a * sn) * s);
    }
  }
  for (int c = rot + lane; c < w.size; c += 32) w.dst[c] = from_f<T>(at(c) * r * s);
}

// ---- CUDA-core attention ---------------------------------------------------------------------------------------------
// One block per (query, head, sequence); four warps take 32 keys at a time in turn (lane i scores key i of its chunk, the
// weighted sum is accumulated in shared memory, lanes over the value dimensions) and are merged at the end.
template <typename T>
__global__ void __launch_bounds__(128) grouped_attn_simt_kernel(const GroupedAttnArgs p) {
  extern __shared__ float sm[];
  __shared__ float s_m[4], s_l[4];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.y;
  const int q0 = p.cu_q != nullptr ? p.cu_q[b] : b;
  const int nq = p.cu_q != nullptr ? p.cu_q[b + 1] - q0 : 1;
  const int qi = blockIdx.x;
  if (qi >= nq) return;
  int n = p.table != nullptr ? p.lens[b] : nq;
  if (p.table != nullptr) {
    const int64_t cap = static_cast<int64_t>(p.table_width) * p.block;
    if (n < 0 || n > cap) {
      if (threadIdx.x == 0) report(p.status);
      n = n < 0 ? 0 : static_cast<int>(cap);
    }
  }
  float* sq = sm;
  float* acc = sm + p.dim + warp * p.vdim;
  const T* q = static_cast<const T*>(p.q) + static_cast<int64_t>(q0 + qi) * p.q_ld + static_cast<int64_t>(h) * p.dim;
  for (int i = threadIdx.x; i < p.dim; i += 128) sq[i] = to_f(q[i]);
  for (int i = lane; i < p.vdim; i += 32) acc[i] = 0.f;
  __syncthreads();
  const int last = qi + n - nq;                          // key index of the query itself
  const int kvh = h / (p.heads / p.kv_heads);
  const int64_t k_row = static_cast<int64_t>(p.kv_heads) * p.dim, v_row = static_cast<int64_t>(p.kv_heads) * p.vdim;
  const T* K = static_cast<const T*>(p.k) + static_cast<int64_t>(kvh) * p.dim;
  const T* V = static_cast<const T*>(p.v) + static_cast<int64_t>(kvh) * p.vdim;
  float m = -1.0e30f, l = 0.f;
  for (int j0 = warp * 32; j0 <= last; j0 += 128) {
    const int j = j0 + lane;
    int64_t slot = -1;
    float s = -INFINITY;
    if (j <= last) {
      if (p.table == nullptr) {
        slot = q0 + j;
      } else {
        const int page = p.table[static_cast<int64_t>(b) * p.table_width + j / p.block];
        if (page >= 0 && page < p.num_blocks) slot = static_cast<int64_t>(page) * p.block + j % p.block;
        else report(p.status);
      }
    }
    if (slot >= 0) {
      const T* kp = K + slot * k_row;
      float d = 0.f;
      for (int i = 0; i < p.dim; ++i) d = fmaf(sq[i], to_f(kp[i]), d);
      s = d * p.scale;
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, o));
    const float mn = fmaxf(m, mx);
    const float w = expf(s - mn), alpha = expf(m - mn);
    float sum = w;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, o);
    l = l * alpha + sum;
    m = mn;
    for (int i = lane; i < p.vdim; i += 32) acc[i] *= alpha;
    const int cnt = min(32, last - j0 + 1);
    for (int k = 0; k < cnt; ++k) {
      const float wk = __shfl_sync(0xFFFFFFFFu, w, k);
      const int64_t sk = __shfl_sync(0xFFFFFFFFu, slot, k);
      if (sk < 0) continue;
      const T* vp = V + sk * v_row;
      for (int i = lane; i < p.vdim; i += 32) acc[i] = fmaf(wk, to_f(vp[i]), acc[i]);
    }
    __syncwarp();
  }
  if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
  __syncthreads();
  float M = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));
  const float sink = p.sink != nullptr ? to_f(static_cast<const T*>(p.sink)[h]) : -INFINITY;
  M = fmaxf(M, sink);
  float e[4], L = p.sink != nullptr ? expf(sink - M) : 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) { e[w] = expf(s_m[w] - M); L += s_l[w] * e[w]; }
  const float inv = L > 0.f ? 1.f / L : 0.f;
  const T* gate = nullptr;
  if (p.gate != nullptr) gate = static_cast<const T*>(p.gate) + static_cast<int64_t>(q0 + qi) * p.gate_ld + static_cast<int64_t>(h) * p.gate_step;
  T* o = static_cast<T*>(p.o) + static_cast<int64_t>(q0 + qi) * p.o_ld + static_cast<int64_t>(h) * p.vdim;
  for (int i = threadIdx.x; i < p.vdim; i += 128) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += sm[p.dim + w * p.vdim + i] * e[w];
    float g = inv;
    if (gate != nullptr) g *= 1.f / (1.f + expf(-to_f(gate[p.gate_step > 1 ? i : 0])));
    o[i] = from_f<T>(v * g);
  }
}

// One block per (head, sequence): joins the key ranges of a decode step.
__global__ void __launch_bounds__(128) grouped_merge_kernel(const GroupedAttnArgs p) {
  const int h = blockIdx.x, b = blockIdx.y;
  const int64_t base = (static_cast<int64_t>(b) * p.heads + h) * p.splits;
  float m = -1.0e29f;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, p.partial_ml[(base + s) * 2]);
  float l = 0.f;
  for (int s = 0; s < p.splits; ++s) l += p.partial_ml[(base + s) * 2 + 1] * exp2f(p.partial_ml[(base + s) * 2] - m);
  if (p.sink != nullptr) l += exp2f(__bfloat162float(static_cast<const __nv_bfloat16*>(p.sink)[h]) * kDmLog2e - m);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int d = threadIdx.x; d < p.vdim; d += 128) {
    float v = 0.f;
#pragma unroll 4
    for (int s = 0; s < p.splits; ++s) v += p.partial_o[(base + s) * p.vdim + d] * exp2f(p.partial_ml[(base + s) * 2] - m);
    float f = inv;
    if (p.gate != nullptr) {
      const __nv_bfloat16* g = static_cast<const __nv_bfloat16*>(p.gate) + b * p.gate_ld + static_cast<int64_t>(h) * p.gate_step;
      f *= 1.f / (1.f + expf(-__bfloat162float(g[p.gate_step > 1 ? d : 0])));
    }
    static_cast<__nv_bfloat16*>(p.o)[b * p.o_ld + static_cast<int64_t>(h) * p.vdim + d] = __float2bfloat16(v * f);
  }
}

constexpr int kMaxSmem = 227 * 1024;

template <typename T>
int run_simt(const GroupedAttnArgs& a, int max_q, cudaStream_t stream) {
  const int smem = 4 * (a.dim + 4 * a.vdim);
  if (smem > kMaxSmem - 1024) return -2;
  if (smem > 48 * 1024) {
    static PerDeviceInt done;
    if (done.cur() < smem) {
      const cudaError_t e = cudaFuncSetAttribute(grouped_attn_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
      done.cur() = smem;
    }
  }
  dim3 grid(static_cast<unsigned>(max_q), static_cast<unsigned>(a.heads), static_cast<unsigned>(a.batch));
  grouped_attn_simt_kernel<T><<<grid, 128, smem, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

// The tensor-core kernels take bf16, heads of up to 128 numbers, sizes, pitches and offsets of whole 16-byte vectors,
// and a positive scale (the row maximum is taken before scaling).
bool on_tensor_cores(const GroupedAttnArgs& a) {
  const int64_t slots = static_cast<int64_t>(a.num_blocks) * a.block;
  return !a.simt && a.dtype == 0 && a.scale > 0.f && a.dim <= 128 && a.vdim <= 128 && ((a.dim | a.vdim) & 7) == 0 &&
         ((a.q_ld | a.o_ld) & 7) == 0 && al16(a.q) && al16(a.k) && al16(a.v) && al16(a.o) && slots < (1ll << 31) &&
         (a.gate == nullptr || a.gate_step == 1 || ((a.gate_ld & 7) == 0 && al16(a.gate)));
}

int check(const GroupedAttnArgs& a) {
  if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads != 0 || a.heads > 65535 || a.batch > 65535) return -1;
  if (a.dim <= 0 || a.vdim <= 0 || a.block <= 0 || (a.table != nullptr && (a.lens == nullptr || a.table_width <= 0))) return -1;
  return 0;
}

template <int NB>
int decode_mma(const PagedDecodeMmaParams& p, int g, dim3 grid, cudaStream_t stream) {
  switch (g) {
    case 1: return paged_decode_mma_run<1, NB>(p, grid, stream);
    case 2: return paged_decode_mma_run<2, NB>(p, grid, stream);
    case 4: return paged_decode_mma_run<4, NB>(p, grid, stream);
    case 8: return paged_decode_mma_run<8, NB>(p, grid, stream);
    default: return paged_decode_mma_run<16, NB>(p, grid, stream);
  }
}

}  // namespace

int launch_grouped_prep(const GroupedPrepArgs& a, cudaStream_t stream) {
  if (a.T <= 0) return 0;
  if (a.heads <= 0 || a.kv_heads <= 0 || a.dim <= 0 || a.vdim <= 0 || a.rot_dims < 0 || (a.rot_dims & 1) || a.rot_dims > a.dim) return -1;
  if (a.rot_dims > 0 && (a.cos_t == nullptr || a.sin_t == nullptr || a.max_pos <= 0)) return -2;
  if (a.temp_every < 0 || a.positions == nullptr) return -3;
  const int units = a.heads + 2 * a.kv_heads;
  if (a.T > 0x7FFFFFFFll || (units + 7) / 8 > 65535) return -4;
  bool vec = a.dim <= 128 && a.vdim <= 128 && ((a.dim | a.vdim | (a.rot_dims >> 1)) & 7) == 0 &&
             ((a.q_ld | a.k_ld | a.v_ld) & 7) == 0;
  for (const void* p : {static_cast<const void*>(a.q), a.k, a.v, a.bq, a.bk, a.bv, static_cast<const void*>(a.k_pages),
                        static_cast<const void*>(a.v_pages), static_cast<const void*>(a.cos_t), static_cast<const void*>(a.sin_t)})
    vec = vec && al16(p);
  const bool narrow = a.dim <= 64 && a.vdim <= 64;
  const int per_block = vec ? (narrow ? 32 : 16) : 8;
  const dim3 grid(static_cast<unsigned>(a.T), static_cast<unsigned>((units + per_block - 1) / per_block));
  if (vec && a.dtype == 1 && narrow) grouped_prep_vec_kernel<float, 8><<<grid, 256, 0, stream>>>(a);
  else if (vec && a.dtype == 1) grouped_prep_vec_kernel<float, 16><<<grid, 256, 0, stream>>>(a);
  else if (vec && narrow) grouped_prep_vec_kernel<__nv_bfloat16, 8><<<grid, 256, 0, stream>>>(a);
  else if (vec) grouped_prep_vec_kernel<__nv_bfloat16, 16><<<grid, 256, 0, stream>>>(a);
  else if (a.dtype == 1) grouped_prep_kernel<float><<<grid, 256, 0, stream>>>(a);
  else grouped_prep_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

int launch_grouped_attn(const GroupedAttnArgs& a, cudaStream_t stream) {
  if (a.batch <= 0 || a.Tq <= 0) return 0;
  if (check(a) != 0 || a.cu_q == nullptr) return -1;
  if (!on_tensor_cores(a) || (a.table != nullptr && a.block % 64 != 0))
    return a.dtype == 1 ? run_simt<float>(a, a.max_q, stream) : run_simt<__nv_bfloat16>(a, a.max_q, stream);
  PortionAttnParams p = {};
  const int64_t slots = static_cast<int64_t>(a.num_blocks) * a.block;
  int r = portion_head_map(&p.tma_qn, a.q, a.dim, a.heads, a.dim, a.Tq, a.q_ld, kLpBlock);
  if (r != 0) return -10 + r;
  r = portion_head_map(&p.tma_k, a.k, a.dim, a.kv_heads, a.dim, slots, static_cast<int64_t>(a.kv_heads) * a.dim, 64);
  if (r != 0) return -20 + r;
  r = portion_head_map(&p.tma_v, a.v, a.vdim, a.kv_heads, a.vdim, slots, static_cast<int64_t>(a.kv_heads) * a.vdim, 64);
  if (r != 0) return -30 + r;
  p.o = static_cast<__nv_bfloat16*>(a.o); p.o_ld = a.o_ld;
  p.gate = static_cast<const __nv_bfloat16*>(a.gate); p.gate_ld = a.gate_ld; p.gate_step = a.gate_step;
  p.sink = static_cast<const __nv_bfloat16*>(a.sink);
  p.cu_q = a.cu_q; p.cu_k = a.cu_q;
  p.table = a.table; p.lens = a.lens; p.table_width = a.table_width; p.block = a.block; p.num_blocks = a.num_blocks;
  p.dim = a.dim; p.vdim = a.vdim; p.group = a.heads / a.kv_heads;
  p.scale_log2 = a.scale * kLpLog2e;
  p.status = a.status;
  return portion_attn_dispatch<false>(p, a.max_q, a.heads, a.batch, stream);
}

int launch_grouped_decode(const GroupedAttnArgs& a, cudaStream_t stream) {
  if (a.batch <= 0) return 0;
  if (check(a) != 0 || a.table == nullptr || a.splits <= 0 || a.splits > 65535) return -1;
  if (!on_tensor_cores(a) || a.block != kDmBlock)
    return a.dtype == 1 ? run_simt<float>(a, 1, stream) : run_simt<__nv_bfloat16>(a, 1, stream);
  if (a.splits > 1 && (a.partial_o == nullptr || a.partial_ml == nullptr)) return -3;
  PagedDecodeMmaParams p = {};
  const int64_t slots = static_cast<int64_t>(a.num_blocks) * a.block;
  int r = paged_decode_map(&p.tma_k, a.k, a.dim, a.kv_heads, slots);
  if (r != 0) return -40 + r;
  r = paged_decode_map(&p.tma_v, a.v, a.vdim, a.kv_heads, slots);
  if (r != 0) return -50 + r;
  p.q = static_cast<const __nv_bfloat16*>(a.q); p.q_ld = a.q_ld;
  p.o = static_cast<__nv_bfloat16*>(a.o); p.o_ld = a.o_ld;
  p.sink = static_cast<const __nv_bfloat16*>(a.sink);
  p.gate = static_cast<const __nv_bfloat16*>(a.gate); p.gate_ld = a.gate_ld; p.gate_step = a.gate_step;
  p.partial_o = a.partial_o; p.partial_ml = a.partial_ml;
  p.block_table = a.table; p.seq_lens = a.lens;
  p.hq = a.heads; p.group = a.heads / a.kv_heads;
  int g = 1;                                           // query heads per CTA
  while (g < p.group && g < 16) g *= 2;
  p.chunks = (p.group + g - 1) / g;
  p.dim = a.dim; p.vdim = a.vdim; p.max_blocks_per_seq = a.table_width;
  p.splits = a.splits; p.num_blocks = a.num_blocks;
  p.scale_log2 = a.scale * kDmLog2e;
  p.status = a.status;
  dim3 grid(static_cast<unsigned>(a.kv_heads * p.chunks), static_cast<unsigned>(a.batch), static_cast<unsigned>(a.splits));
  r = a.dim <= 64 && a.vdim <= 64 ? decode_mma<1>(p, g, grid, stream) : decode_mma<2>(p, g, grid, stream);
  if (r != 0 || a.splits == 1) return r;
  grouped_merge_kernel<<<dim3(static_cast<unsigned>(a.heads), static_cast<unsigned>(a.batch)), 128, 0, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace yv
