// Plain tiled matrix product on the CUDA cores: Y[m, n] = act(sum_k X[m, k] W[n, k]) (+ residual), fp32 accumulation,
// bf16 or fp32 storage, any sizes and row strides.  It is the 32-bit product of models that run in fp32 (the tensor
// cores have no full-precision fp32 mode) and takes the bf16 shapes whose rows a TMA copy cannot address (K not a
// multiple of 8).
#include "typed.cuh"
#include "api.h"

#include <type_traits>

namespace sllm {

constexpr int kSgTile = 64, kSgK = 16, kSgThreads = 256;

template <typename T, typename TY>
__global__ void __launch_bounds__(kSgThreads)
gemm_simt_kernel(const T* __restrict__ x, const T* __restrict__ w, TY* __restrict__ y, const TY* __restrict__ residual, int m, int n,
                 int k, int ldx, int ldw, int ldy, int act, float act_arg) {
  pdl_wait();
  pdl_trigger();
  __shared__ float xs[kSgK][kSgTile + 4];
  __shared__ float ws[kSgK][kSgTile + 4];
  const int m0 = blockIdx.y * kSgTile, n0 = blockIdx.x * kSgTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += kSgK) {
#pragma unroll
    for (int e = threadIdx.x; e < kSgTile * kSgK; e += kSgThreads) {
      const int rr = e / kSgK, kk = e % kSgK;
      const bool kin = k0 + kk < k;
      xs[kk][rr] = kin && m0 + rr < m ? ld_f(x + static_cast<size_t>(m0 + rr) * ldx + k0 + kk) : 0.f;
      ws[kk][rr] = kin && n0 + rr < n ? ld_f(w + static_cast<size_t>(n0 + rr) * ldw + k0 + kk) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kSgK; ++kk) {
      float a[4], b[4];
      ld_vec<4>(&xs[kk][ty * 4], a);
      ld_vec<4>(&ws[kk][tx * 4], b);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = m0 + ty * 4 + i;
    if (r >= m) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tx * 4 + j;
      if (c >= n) continue;
      float v = acc[i][j];
      if (act == 1) v = v > 0.f ? v * v : 0.f;
      else if (act == 2) v = act_arg * tanhf(v / act_arg);
      const size_t idx = static_cast<size_t>(r) * ldy + c;
      if (residual) v += ld_f(residual + idx);
      st_f(y + idx, v);
    }
  }
}

}  // namespace sllm

using namespace sllm;

// act: 0 none, 1 square of relu, 2 soft cap act_arg * tanh(y / act_arg).  fp32: element type of x, w, y and residual (0 bf16,
// 1 fp32); out_fp32: y and residual are fp32 whatever x and w are.
SLLM_EXPORT int sllm_gemm_simt(const void* x, const void* w, void* y, const void* residual, int m, int n, int k, int ldx, int ldw,
                               int ldy, int act, float act_arg, int fp32, int out_fp32, void* stream) {
  if (!x || !w || !y || m <= 0 || n <= 0 || k <= 0 || ldx < k || ldw < k || ldy < n || act < 0 || act > 2 || (act == 2 && !(act_arg > 0.f)))
    return SLLM_ERR_INVALID_ARGUMENT;
  const dim3 grid((n + kSgTile - 1) / kSgTile, (m + kSgTile - 1) / kSgTile);
  if (grid.y > 65535) return SLLM_ERR_LIMIT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto* kernel, auto* xt, auto* yt) {
    using T = std::remove_pointer_t<decltype(xt)>;
    using TY = std::remove_pointer_t<decltype(yt)>;
    return launch_kernel(kernel, grid, dim3(kSgThreads), 0, st, 1u, static_cast<const T*>(x), static_cast<const T*>(w), static_cast<TY*>(y),
                         static_cast<const TY*>(residual), m, n, k, ldx, ldw, ldy, act, act_arg);
  };
  float* f = nullptr;
  __nv_bfloat16* h = nullptr;
  const cudaError_t e = fp32 ? go(gemm_simt_kernel<float, float>, f, f)
                             : out_fp32 ? go(gemm_simt_kernel<__nv_bfloat16, float>, h, f)
                                        : go(gemm_simt_kernel<__nv_bfloat16, __nv_bfloat16>, h, h);
  return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}
