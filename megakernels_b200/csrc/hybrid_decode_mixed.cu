// Decode megakernel of the hybrid models, build for all mechanisms.
#define MKBH_FEATURES 3
#include "hybrid_decode.cu"
