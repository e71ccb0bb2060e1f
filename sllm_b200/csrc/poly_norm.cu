// Polynomial activation with normed powers: y = a N(z) + b N(z^2) + c N(z^3) + e, powers element by element, N(v) = v /
// sqrt(mean(v^2) + eps) over a row's values.  A row is read once: its 16-byte pieces stay in registers between the sums and
// the result (rows too long or not aligned for that are read twice).
#include "typed.cuh"
#include "api.h"

namespace sllm {

constexpr int kPnThreads = 256;

// kHeld: pieces per thread; 0: none held, element by element.  coef: {a, b, c, e}.
template <typename T, int kHeld>
__global__ void __launch_bounds__(kPnThreads)
poly_norm_kernel(const T* __restrict__ x, long long ldx, T* __restrict__ y, int n, const float* __restrict__ coef, float eps) {
  pdl_wait();
  pdl_trigger();
  constexpr int kV = kVec16<T>, kN = kHeld > 0 ? kHeld : 1;
  __shared__ float red[3][kPnThreads / 32];
  const T* src = x + blockIdx.x * ldx;
  T* dst = y + static_cast<size_t>(blockIdx.x) * n;
  float ss[3] = {0.f, 0.f, 0.f};
  auto add = [&](float z) {
    const float s = z * z, q = s * s;
    ss[0] += s;
    ss[1] += q;
    ss[2] = fmaf(q, s, ss[2]);
  };
  float v[kN][kV];
  if constexpr (kHeld > 0) {
#pragma unroll
    for (int u = 0; u < kHeld; ++u) {
      const int i = (u * kPnThreads + threadIdx.x) * kV;
      if (i < n) {
        ld16(src + i, v[u]);
      } else {
#pragma unroll
        for (int j = 0; j < kV; ++j) v[u][j] = 0.f;
      }
    }
#pragma unroll
    for (int u = 0; u < kHeld; ++u)
#pragma unroll
      for (int j = 0; j < kV; ++j) add(v[u][j]);
  } else {
    for (int i = threadIdx.x; i < n; i += kPnThreads) add(ld_f(src + i));
  }
#pragma unroll
  for (int m = 0; m < 3; ++m) {
    ss[m] = warp_sum(ss[m]);
    if ((threadIdx.x & 31) == 0) red[m][threadIdx.x >> 5] = ss[m];
  }
  __syncthreads();
  float f[3];
#pragma unroll
  for (int m = 0; m < 3; ++m) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < kPnThreads / 32; ++w) s += red[m][w];
    f[m] = coef[m] / sqrtf(s / static_cast<float>(n) + eps);
  }
  const float e = coef[3];
  auto value = [&](float z) { return fmaf(fmaf(fmaf(f[2], z, f[1]), z, f[0]), z, e); };
  if constexpr (kHeld > 0) {
#pragma unroll
    for (int u = 0; u < kHeld; ++u) {
      const int i = (u * kPnThreads + threadIdx.x) * kV;
      if (i >= n) break;
#pragma unroll
      for (int j = 0; j < kV; j += 4) {
        const float o[4] = {value(v[u][j]), value(v[u][j + 1]), value(v[u][j + 2]), value(v[u][j + 3])};
        st_vec<4>(dst + i + j, o);
      }
    }
  } else {
    for (int i = threadIdx.x; i < n; i += kPnThreads) st_f(dst + i, value(ld_f(src + i)));
  }
}

template <typename T>
static int poly_norm_launch(const void* x, long long ldx, void* y, int rows, int n, const float* coef, float eps, cudaStream_t st) {
  const bool vec = n % kVec16<T> == 0 && ldx % kVec16<T> == 0 && !((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y)) & 15);
  const int pieces = (n + kPnThreads * kVec16<T> - 1) / (kPnThreads * kVec16<T>);
  auto* kernel = !vec || pieces > 8 ? poly_norm_kernel<T, 0> : pieces > 6 ? poly_norm_kernel<T, 8> : pieces > 5 ? poly_norm_kernel<T, 6>
               : pieces > 4 ? poly_norm_kernel<T, 5> : pieces > 3 ? poly_norm_kernel<T, 4> : pieces > 2 ? poly_norm_kernel<T, 3>
               : pieces > 1 ? poly_norm_kernel<T, 2> : poly_norm_kernel<T, 1>;
  return launch_kernel(kernel, dim3(rows), dim3(kPnThreads), 0, st, 1u, static_cast<const T*>(x), ldx, static_cast<T*>(y), n, coef, eps) ==
                 cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

}  // namespace sllm

using namespace sllm;

// x [rows, ldx], y [rows, n], coef fp32 [4]; fp32: element type of x and y (0 bf16, 1 fp32).
SLLM_EXPORT int sllm_poly_norm(const void* x, long long ldx, void* y, int rows, int n, const float* coef, float eps, int fp32, void* stream) {
  if (!x || !y || !coef || rows <= 0 || n <= 0 || ldx < n) return SLLM_ERR_INVALID_ARGUMENT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return fp32 ? poly_norm_launch<float>(x, ldx, y, rows, n, coef, eps, st) : poly_norm_launch<__nv_bfloat16>(x, ldx, y, rows, n, coef, eps, st);
}
