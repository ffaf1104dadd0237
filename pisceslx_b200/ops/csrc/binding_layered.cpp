// The operators that serve a layered model, as a library of their own (``_yv_layered.so``): a process that replays a
// trace in a fresh checkout compiles these and nothing else.  ``_yv_ops.so`` holds the same operators, so a process
// loads one of the two.
#include "binding_gemm.inc"
#include "binding_latent.inc"

TORCH_LIBRARY(yv, m) {
  yv_register_gemm_schemas(m);
  yv_register_latent_schemas(m);
}

TORCH_LIBRARY_IMPL(yv, CUDA, m) {
  yv_register_gemm_impls(m);
  yv_register_latent_impls(m);
}
