// Store of the inputs of a short causal convolution after a prompt portion (short_conv.cu).
#pragma once
#include <cuda_runtime.h>

namespace sllm {

// x: the inputs' columns of a flat batch [rows, ldx] (bf16, or fp32); ring: a slot's [taps][channels] at slot * ring_stride.
cudaError_t conv_ring_launch(const void* x, int ldx, bool fp32, float* ring, long long ring_stride, const int* row_off, const int* slots,
                             const int* positions, int channels, int taps, int sequences, cudaStream_t stream);

}  // namespace sllm
