// Grouped RMSNorm on a 32-bit residual stream, with the work around it in one launch.
//
// A vector of d channels is split into `groups` equal consecutive parts; each part is divided by its own
// sqrt(mean(part^2) + eps) and the whole is multiplied by the weight (fp32).  groups = 1 is the ordinary RMSNorm.
//
// One launch does, per row:
//   1. x  = table[id]                (embedding),  or
//      x += norm(y) * w_post         (sandwich: the sublayer's output is normalised before it joins the residual; y may be
//                                     the sum of several listed rows, the routed experts of a token), or
//      x  as it is, optionally of a gathered row
//   2. z  = norm(x) * w_out          (the next sublayer's input, in the activation type), or z = x without w_out
// so a decoder layer with norms before and after each sublayer costs one such launch per sublayer.
#include "typed.cuh"
#include "api.h"

namespace sllm {

constexpr int kGnThreads = 256;
constexpr int kGnWarps = kGnThreads / 32;

template <typename T>
struct GroupNormParams {
  const T* table;            // embedding mode: [vocab, d]
  const int* ids;
  int vocab;
  const T* y;                // sandwich mode: [rows, ldy]
  int ldy;
  const int* y_rows;         // sandwich mode: y is the sum of the rows y_rows[r * y_terms ..] >= 0 (null: row r)
  int y_terms;
  const float* w_post;       // [d]
  float* x;                  // residual [*, d]: written in the embedding and sandwich modes
  const long long* row_idx;  // read-only mode: z row r comes from x row row_idx[r] (null: row r)
  const float* w_out;        // [d], null: z is x itself
  T* z;                      // [rows, d], null: none
  int d, groups, parts;
  float eps;
};

// inv[g] = 1 / sqrt(mean of group g of v + eps); `parts` warps share a group.
__device__ __forceinline__ void group_inv_rms(const float* v, int gs, int groups, int parts, float eps, float* part, float* inv) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int u = warp; u < groups * parts; u += kGnWarps) {
    const int g = u / parts, p = u % parts;
    const int lo = g * gs + static_cast<int>(static_cast<long long>(gs) * p / parts);
    const int hi = g * gs + static_cast<int>(static_cast<long long>(gs) * (p + 1) / parts);
    float ss = 0.f;
    for (int i = lo + lane; i < hi; i += 32) ss += v[i] * v[i];
    ss = warp_sum(ss);
    if (lane == 0) part[u] = ss;
  }
  __syncthreads();
  for (int g = threadIdx.x; g < groups; g += kGnThreads) {
    float ss = 0.f;
    for (int p = 0; p < parts; ++p) ss += part[g * parts + p];
    inv[g] = 1.f / sqrtf(ss / static_cast<float>(gs) + eps);
  }
  __syncthreads();
}

// kV: channels per access (4 when the group size and the row strides allow it, else 1).
template <typename T, int kV>
__global__ void __launch_bounds__(kGnThreads) group_norm_kernel(const GroupNormParams<T> p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float sm[];
  float* row = sm;                                   // [d]
  float* inv = sm + ((p.d + 3) & ~3);                // [groups]
  float* part = inv + p.groups;                      // [groups * parts]
  const int r = blockIdx.x, d = p.d, gs = d / p.groups;
  auto load = [](const auto* src, float (&v)[kV]) {
    if constexpr (kV == 1) v[0] = ld_f(src);
    else ld_vec<kV>(src, v);
  };
  auto store = [](auto* dst, const float (&v)[kV]) {
    if constexpr (kV == 1) st_f(dst, v[0]);
    else st_vec<kV>(dst, v);
  };
  float* xr = p.x;
  if (p.table) {
    int id = p.ids[r];
    if (id < 0 || id >= p.vocab) id = 0;
    xr += static_cast<size_t>(r) * d;
    const T* src = p.table + static_cast<size_t>(id) * d;
    for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
      float v[kV];
      load(src + i, v);
      store(row + i, v);
      store(xr + i, v);
    }
  } else if (p.y) {
    xr += static_cast<size_t>(r) * d;
    if (p.y_rows) {
      const int* rows = p.y_rows + static_cast<size_t>(r) * p.y_terms;
      for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
        float v[kV] = {};
#pragma unroll 4
        for (int t = 0; t < p.y_terms; ++t) {
          const int src = rows[t];
          if (src < 0) continue;
          float a[kV];
          load(p.y + static_cast<size_t>(src) * p.ldy + i, a);
#pragma unroll
          for (int j = 0; j < kV; ++j) v[j] += a[j];
        }
        store(row + i, v);
      }
    } else {
      const T* src = p.y + static_cast<size_t>(r) * p.ldy;
      for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
        float v[kV];
        load(src + i, v);
        store(row + i, v);
      }
    }
    __syncthreads();
    group_inv_rms(row, gs, p.groups, p.parts, p.eps, part, inv);
    for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
      float v[kV], w[kV], x[kV];
      load(row + i, v);
      load(p.w_post + i, w);
      load(xr + i, x);
      const float s = inv[i / gs];
#pragma unroll
      for (int j = 0; j < kV; ++j) x[j] += v[j] * s * w[j];
      store(xr + i, x);
      store(row + i, x);
    }
  } else {
    const long long src = p.row_idx ? p.row_idx[r] : r;
    xr += static_cast<size_t>(src) * d;
    for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
      float v[kV];
      load(xr + i, v);
      store(row + i, v);
    }
  }
  if (!p.z) return;
  T* zr = p.z + static_cast<size_t>(r) * d;
  if (!p.w_out) {                                    // every thread reads back what it wrote
    for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
      float v[kV];
      load(row + i, v);
      store(zr + i, v);
    }
    return;
  }
  __syncthreads();
  group_inv_rms(row, gs, p.groups, p.parts, p.eps, part, inv);
  for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
    float v[kV], w[kV];
    load(row + i, v);
    load(p.w_out + i, w);
    const float s = inv[i / gs];
#pragma unroll
    for (int j = 0; j < kV; ++j) v[j] = v[j] * s * w[j];
    store(zr + i, v);
  }
}

template <typename T>
static int group_norm_launch(const void* table, const int* ids, int vocab, const void* y, int ldy, const int* y_rows, int y_terms,
                             const float* w_post, float* x, const long long* row_idx, const float* w_out, void* z, int rows, int d, int groups, float eps,
                             cudaStream_t st) {
  GroupNormParams<T> p = {};
  p.table = static_cast<const T*>(table); p.ids = ids; p.vocab = vocab;
  p.y = static_cast<const T*>(y); p.ldy = ldy; p.y_rows = y_rows; p.y_terms = y_terms; p.w_post = w_post; p.x = x; p.row_idx = row_idx;
  p.w_out = w_out; p.z = static_cast<T*>(z); p.d = d; p.groups = groups; p.eps = eps;
  p.parts = groups >= kGnWarps ? 1 : (kGnWarps + groups - 1) / groups;
  const size_t smem = sizeof(float) * (((d + 3) & ~3) + groups + static_cast<size_t>(groups) * p.parts);
  if (smem > 200 * 1024) return SLLM_ERR_UNSUPPORTED_SHAPE;
  const bool vec = (d / groups) % 4 == 0 && (!y || ldy % 4 == 0);
  auto* kernel = vec ? group_norm_kernel<T, 4> : group_norm_kernel<T, 1>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
    return SLLM_ERR_CUDA;
  return launch_kernel(kernel, dim3(rows), dim3(kGnThreads), smem, st, 1u, p) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

}  // namespace sllm

using namespace sllm;

// table + ids: embedding mode; y + w_post: sandwich mode; neither: x is read only (rows picked by row_idx when given).
// y_rows [rows, y_terms]: y is the sum of those rows of it.  z may be null (residual update alone), z without w_out is x in
// the element type.  fp32: element type of table, y and z (0 bf16, 1 fp32).
SLLM_EXPORT int sllm_group_norm(const void* table, const int* ids, int vocab, const void* y, int ldy, const int* y_rows,
                                int y_terms, const float* w_post, float* x, const long long* row_idx, const float* w_out, void* z, int rows, int d, int groups,
                                float eps, int fp32, void* stream) {
  if (!x || rows <= 0 || d <= 0 || groups <= 0 || d % groups) return SLLM_ERR_INVALID_ARGUMENT;
  if ((table && (!ids || vocab <= 0 || y)) || (y && !w_post) || (!z && w_out) || (y_rows && (!y || y_terms <= 0)) || (!z && !y && !table)) return SLLM_ERR_INVALID_ARGUMENT;
  if (row_idx && (table || y)) return SLLM_ERR_INVALID_ARGUMENT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return fp32 ? group_norm_launch<float>(table, ids, vocab, y, ldy, y_rows, y_terms, w_post, x, row_idx, w_out, z, rows, d, groups, eps, st)
              : group_norm_launch<__nv_bfloat16>(table, ids, vocab, y, ldy, y_rows, y_terms, w_post, x, row_idx, w_out, z, rows, d, groups, eps, st);
}
