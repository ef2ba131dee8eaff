// Decode megakernel of the hybrid models, build for rotary and latent attention, gated units, convolutions, loops.
#define MKBH_FEATURES 2
#include "hybrid_decode.cu"
