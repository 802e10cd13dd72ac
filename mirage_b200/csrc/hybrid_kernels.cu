// Launch entry points of hybrid graphs (hybrid_tasks.cuh).  Their megakernel instantiations are in one source each, which nvcc
// compiles side by side: bf16 with the narrow linear body (up to 8 batched tokens), bf16 with the tcgen05 body (more), and 32-bit
// throughout.  Built as libmpk_b200_hybrid.so, loaded by the C ABI library when such a graph is compiled.
#include "hybrid_kernels.h"

static mpk::MegaKernel pick(int hybrid, int general) {
  if (hybrid == mpk::HYB_F32) return mpk::hybrid_kernel_f32();
  return general ? mpk::hybrid_kernel_bf16_wide() : mpk::hybrid_kernel_bf16();
}

extern "C" int mpk_family_prepare(int smem_bytes, int) {
  int dev = 0, limit = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e == cudaSuccess) e = cudaDeviceGetAttribute(&limit, cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
  if (e != cudaSuccess) return (int)e;
  if (smem_bytes > limit) return (int)cudaErrorInvalidValue;
  const mpk::MegaKernel all[3] = {pick(mpk::HYB_BF16, 0), pick(mpk::HYB_BF16, 1), pick(mpk::HYB_F32, 0)};
  for (mpk::MegaKernel k : all) {
    e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, limit);
    if (e != cudaSuccess) return (int)e;
  }
  return 0;
}

extern "C" int mpk_family_launch(const mpk::KernelParams *params, int smem_bytes, void *stream) {
  pick(params->hybrid, params->general_kernel)<<<params->num_workers, mpk::kBlockThreads, smem_bytes, (cudaStream_t)stream>>>(*params);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : (int)e;
}
