#include "hybrid_kernels.h"
#include "megakernel.cuh"

mpk::MegaKernel mpk::hybrid_kernel_bf16() { return mpk::mpk_megakernel<false, false, HYB_BF16>; }
