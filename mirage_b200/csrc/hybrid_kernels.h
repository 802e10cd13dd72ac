// Megakernel instantiations of hybrid graphs, one per source file.
#pragma once
#include <cuda_runtime.h>

#include "runtime_types.h"

namespace mpk {
typedef void (*MegaKernel)(const KernelParams);
MegaKernel hybrid_kernel_bf16();        // up to 8 batched tokens
MegaKernel hybrid_kernel_bf16_wide();   // more: tcgen05 linears
MegaKernel hybrid_kernel_f32();
}  // namespace mpk
