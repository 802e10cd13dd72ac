#include "hybrid_kernels.h"
#include "megakernel.cuh"

mpk::MegaKernel mpk::hybrid_kernel_bf16_wide() { return mpk::mpk_megakernel<true, false, HYB_BF16>; }
