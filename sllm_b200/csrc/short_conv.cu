// A slot's ring holds the inputs of a short causal convolution at the last `taps` positions of its sequence, row position mod
// taps.  Decode kernels store the row of their own token; after a prompt portion this kernel stores the last ones.
#include "short_conv.h"
#include "typed.cuh"

namespace sllm {

// grid (ceil(channels / 256), sequences).
template <typename T>
__global__ void __launch_bounds__(256)
conv_ring_kernel(const T* __restrict__ x, int ldx, float* __restrict__ ring, long long ring_stride, const int* __restrict__ row_off,
                 const int* __restrict__ slots, const int* __restrict__ positions, int channels, int taps) {
  pdl_wait();
  pdl_trigger();
  const int c = blockIdx.x * 256 + threadIdx.x, seq = blockIdx.y;
  if (c >= channels) return;
  const int r1 = row_off[seq + 1];
  for (int row = max(row_off[seq], r1 - taps); row < r1; ++row)
    ring[slots[seq] * ring_stride + static_cast<size_t>(positions[row] % taps) * channels + c] = ld_f(x + static_cast<size_t>(row) * ldx + c);
}

cudaError_t conv_ring_launch(const void* x, int ldx, bool fp32, float* ring, long long ring_stride, const int* row_off, const int* slots,
                             const int* positions, int channels, int taps, int sequences, cudaStream_t st) {
  const dim3 grid((channels + 255) / 256, sequences);
  if (fp32)
    return launch_kernel(conv_ring_kernel<float>, grid, dim3(256), 0, st, 1u, static_cast<const float*>(x), ldx, ring, ring_stride, row_off,
                         slots, positions, channels, taps);
  return launch_kernel(conv_ring_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, 1u, static_cast<const __nv_bfloat16*>(x), ldx, ring,
                       ring_stride, row_off, slots, positions, channels, taps);
}

}  // namespace sllm
