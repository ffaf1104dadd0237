#pragma once
#include "latent_ops.h"
#include "sm100.cuh"
namespace yv {
inline int launch_latent_prefill_mma(const LatentAttnArgs&, cudaStream_t) { return -99; }
bool latent_attn_on_tensor_cores(const LatentAttnArgs&) { return false; }
}
