// Row interleaving of weight tensors at compile time (mpk_shuffle_tensors / mpk_fuse_tensors).
#include <cuda_runtime.h>
#include <stdint.h>

__global__ void mpk_shuffle_rows_kernel(uint8_t *dst, const uint8_t *const *srcs, const int64_t *rows_per_group,
                                        const int64_t *prefix_rows, int n, int64_t group_rows_total,
                                        int64_t row_bytes, int64_t total_rows) {
  // dst row r: group g = r / group_rows_total, offset o within the group; tensor i with prefix[i] <= o < prefix[i+1]
  for (int64_t r = blockIdx.x; r < total_rows; r += gridDim.x) {
    const int64_t g = r / group_rows_total, o = r - g * group_rows_total;
    int i = 0;
    while (i + 1 < n && o >= prefix_rows[i + 1]) ++i;
    const uint8_t *src = srcs[i] + ((g * rows_per_group[i]) + (o - prefix_rows[i])) * row_bytes;
    uint8_t *d = dst + r * row_bytes;
    if (row_bytes % 16 == 0) {
      for (int64_t b = threadIdx.x * 16; b < row_bytes; b += blockDim.x * 16)
        *reinterpret_cast<uint4 *>(d + b) = *reinterpret_cast<const uint4 *>(src + b);
    } else {   // narrow rows (e.g. the packed scale words of a small weight): 4-byte words
      for (int64_t b = threadIdx.x * 4; b < row_bytes; b += blockDim.x * 4)
        *reinterpret_cast<uint32_t *>(d + b) = *reinterpret_cast<const uint32_t *>(src + b);
    }
  }
}

extern "C" int mpk_shuffle_rows_launch(void *dst, const void *const *srcs_dev, const int64_t *rows_per_group_dev,
                                       const int64_t *prefix_rows_dev, int n, int64_t group_rows_total,
                                       int64_t row_bytes, int64_t total_rows, void *stream) {
  mpk_shuffle_rows_kernel<<<1024, 256, 0, (cudaStream_t)stream>>>(
      (uint8_t *)dst, (const uint8_t *const *)srcs_dev, rows_per_group_dev, prefix_rows_dev, n, group_rows_total,
      row_bytes, total_rows);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : (int)e;
}
