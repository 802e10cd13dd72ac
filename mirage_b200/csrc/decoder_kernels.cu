// Megakernel instantiations of transformer decoder graphs (bf16 / FP8 linears, paged GQA attention, MoE, MLA) and their
// launch entry points.  Built as libmpk_b200_decoder.so, loaded by the C ABI library when such a graph is compiled.
//
// The shared-memory limit is a property of the function on the current device, shared by every handle of the process:
// it is raised to the device's opt-in maximum (not to this handle's need), so that preparing a graph with a small
// footprint cannot lower it under a graph prepared earlier.
#include "megakernel.cuh"

extern "C" int mpk_family_prepare(int smem_bytes, int) {
  int dev = 0, limit = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e == cudaSuccess) e = cudaDeviceGetAttribute(&limit, cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
  if (e != cudaSuccess) return (int)e;
  if (smem_bytes > limit) return (int)cudaErrorInvalidValue;
  smem_bytes = limit;
  e = cudaFuncSetAttribute(mpk::mpk_megakernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_bytes);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(mpk::mpk_megakernel<false, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_bytes);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(mpk::mpk_megakernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_bytes);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(mpk::mpk_megakernel<true, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_bytes);
  return e == cudaSuccess ? 0 : (int)e;
}

extern "C" int mpk_family_launch(const mpk::KernelParams *params, int smem_bytes, void *stream) {
  if (params->general_kernel && params->world_size > 1)
    mpk::mpk_megakernel<true, true><<<params->num_workers, mpk::kBlockThreads, smem_bytes, (cudaStream_t)stream>>>(*params);
  else if (params->general_kernel)
    mpk::mpk_megakernel<true><<<params->num_workers, mpk::kBlockThreads, smem_bytes, (cudaStream_t)stream>>>(*params);
  else if (params->world_size > 1 && params->tp_extensions)
    mpk::mpk_megakernel<false, true><<<params->num_workers, mpk::kBlockThreads, smem_bytes, (cudaStream_t)stream>>>(*params);
  else
    mpk::mpk_megakernel<false><<<params->num_workers, mpk::kBlockThreads, smem_bytes, (cudaStream_t)stream>>>(*params);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : (int)e;
}
