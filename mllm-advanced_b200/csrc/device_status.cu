// The device status word of a library image and its host-side reader.
#include "device_common.cuh"
#include "../../include/mllmb200.h"

namespace mllmb200 {

__device__ unsigned int g_device_status = 0;

// Synchronizes the stream, reads and clears the word; *status = what it says.
cudaError_t read_device_status(cudaStream_t st, int* status) {
  cudaError_t e = cudaStreamSynchronize(st);
  unsigned int word = 0;
  if (e == cudaSuccess) e = cudaMemcpyFromSymbol(&word, g_device_status, sizeof(word));
  if (e == cudaSuccess && word != 0) {
    const unsigned int zero = 0;
    e = cudaMemcpyToSymbol(g_device_status, &zero, sizeof(zero));
  }
  *status = (word & kDevStatusTimeout) ? MLLMB200_TIMEOUT : (word & kDevStatusBadHeader) ? MLLMB200_BAD_BLOB : MLLMB200_OK;
  return e;
}

}  // namespace mllmb200
