#pragma once
#include "latent_ops.h"
#include "sm100.cuh"
namespace yv {
inline int launch_latent_decode_mma(const LatentDecodeArgs&, cudaStream_t) { return -99; }
bool latent_decode_on_tensor_cores(const LatentDecodeArgs&) { return false; }
}
