// The operators that serve one family of layered models, as a library of its own (``_yv_layered_<mixers>.so``, see
// ops/build.py): a process that replays a trace in a fresh checkout compiles these and nothing else.  ``_yv_ops.so``
// holds all of them, so a process loads one library.
#include "binding_gemm.inc"
#include "binding_stream.inc"
#ifdef YV_FAMILY_LATENT_ATTENTION
#include "binding_latent.inc"
#endif
#ifdef YV_FAMILY_GROUPED_ATTENTION
#include "binding_grouped.inc"
#endif

TORCH_LIBRARY(yv, m) {
  yv_register_gemm_schemas(m);
  yv_register_stream_schemas(m);
#ifdef YV_FAMILY_LATENT_ATTENTION
  yv_register_latent_schemas(m);
#endif
#ifdef YV_FAMILY_GROUPED_ATTENTION
  yv_register_grouped_schemas(m);
#endif
}

TORCH_LIBRARY_IMPL(yv, CUDA, m) {
  yv_register_gemm_impls(m);
  yv_register_stream_impls(m);
#ifdef YV_FAMILY_LATENT_ATTENTION
  yv_register_latent_impls(m);
#endif
#ifdef YV_FAMILY_GROUPED_ATTENTION
  yv_register_grouped_impls(m);
#endif
}
