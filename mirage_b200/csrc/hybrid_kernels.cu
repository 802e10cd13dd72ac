// Megakernel instantiations of hybrid graphs (hybrid_tasks.cuh) and their launch entry points: bf16 with the narrow
// linear body (up to 8 batched tokens), bf16 with the tcgen05 body (more), and 32-bit throughout.  Built as
// libmpk_b200_hybrid.so, loaded by the C ABI library when such a graph is compiled.
#include "megakernel.cuh"

typedef void (*HybridKernel)(const mpk::KernelParams);
static HybridKernel pick(int hybrid, int general) {
  if (hybrid == mpk::HYB_F32) return mpk::mpk_megakernel<false, false, mpk::HYB_F32>;
  return general ? mpk::mpk_megakernel<true, false, mpk::HYB_BF16> : mpk::mpk_megakernel<false, false, mpk::HYB_BF16>;
}

extern "C" int mpk_family_prepare(int smem_bytes, int) {
  int dev = 0, limit = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e == cudaSuccess) e = cudaDeviceGetAttribute(&limit, cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
  if (e != cudaSuccess) return (int)e;
  if (smem_bytes > limit) return (int)cudaErrorInvalidValue;
  const HybridKernel all[3] = {pick(mpk::HYB_BF16, 0), pick(mpk::HYB_BF16, 1), pick(mpk::HYB_F32, 0)};
  for (HybridKernel k : all) {
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
