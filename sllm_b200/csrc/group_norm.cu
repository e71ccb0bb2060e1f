// Grouped RMSNorm on a 32-bit residual stream, with the work around it in one launch.
//
// A vector of d channels is split into `groups` equal consecutive parts; each part is divided by its own
// sqrt(mean(part^2) + eps) and the whole is multiplied by the weight (fp32).  groups = 1 is the ordinary RMSNorm.
//
// One launch does, per row:
//   1. x  = table_scale table[id]    (embedding),  or
//      x += coef norm(y) * w_post    (the sublayer's output is normalised before it joins the residual, or joins as it is
//                                     without w_post; y may be the sum of several listed rows, the routed experts of a
//                                     token; a second output y2 with its own coefficient and weight may join as well), or
//      x  as it is, optionally of a gathered row
//   2. x += table_scale table[id] (with y) and x += step     (what a looped block adds before each of its passes)
//   3. z  = norm(x) * w_out          (the next sublayer's input, in the activation type), or z = x without w_out
// so a decoder layer costs one such launch per sublayer, whether its norms lie before or after the sublayers or both.
#include "typed.cuh"
#include "api.h"

#include <cstddef>

namespace sllm {

constexpr int kGnThreads = 256;
constexpr int kGnWarps = kGnThreads / 32;

template <typename T>
struct GroupNormParams {
  const T* table;            // [vocab, d]: becomes x, or with y joins it
  const int* ids;
  int vocab;
  float table_scale;
  const float* step;         // optional [d]: joins x
  const T* y;                // [rows, ldy]
  int ldy;
  const int* y_rows;         // y is the sum of the rows y_rows[r * y_terms ..] >= 0 (null: row r)
  int y_terms;
  const float* w_post;       // [d], null: y joins without a norm
  float coef;
  const T* y2;               // optional second summand [rows, ldy2] with its own weight and coefficient
  int ldy2;
  const float* w_post2;
  float coef2;
  float* x;                  // residual [*, d]: written in the embedding and summand modes
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
  const int dp = (p.d + 3) & ~3;
  float* row = sm;                                   // [d]
  float* row2 = sm + dp;                             // [d] with a second summand
  float* inv = row2 + (p.y2 ? dp : 0);               // [groups]
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
  const T* emb = nullptr;
  if (p.table) {
    int id = p.ids[r];
    if (id < 0 || id >= p.vocab) id = 0;
    emb = p.table + static_cast<size_t>(id) * d;
  }
  // channels i .. of x and what a pass of a loop adds to them
  auto with_extras = [&](int i, float (&x)[kV]) {
    if (emb) {
      float v[kV];
      load(emb + i, v);
#pragma unroll
      for (int j = 0; j < kV; ++j) x[j] = fmaf(v[j], p.table_scale, x[j]);
    }
    if (p.step) {
      float v[kV];
      load(p.step + i, v);
#pragma unroll
      for (int j = 0; j < kV; ++j) x[j] += v[j];
    }
  };
  if (p.table && !p.y) {
    xr += static_cast<size_t>(r) * d;
    for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
      float v[kV] = {};
      with_extras(i, v);
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
    if (p.y2) {
      const T* src = p.y2 + static_cast<size_t>(r) * p.ldy2;
      for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
        float v[kV];
        load(src + i, v);
        store(row2 + i, v);
      }
    }
    // x += coef v (every thread reads back what it wrote), or coef norm(v) * weight
    auto join = [&](float* from, const float* weight, float coef, bool last) {
      if (weight) {
        __syncthreads();
        group_inv_rms(from, gs, p.groups, p.parts, p.eps, part, inv);
      }
      for (int i = threadIdx.x * kV; i < d; i += kGnThreads * kV) {
        float v[kV], x[kV];
        load(from + i, v);
        load(xr + i, x);
        if (weight) {
          float w[kV];
          load(weight + i, w);
          const float s = inv[i / gs];
#pragma unroll
          for (int j = 0; j < kV; ++j) v[j] *= s * w[j];
        }
#pragma unroll
        for (int j = 0; j < kV; ++j) x[j] = fmaf(v[j], coef, x[j]);
        if (last) {
          with_extras(i, x);
          store(row + i, x);
        }
        store(xr + i, x);
      }
    };
    join(row, p.w_post, p.coef, !p.y2);
    if (p.y2) join(row2, p.w_post2, p.coef2, true);
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

}  // namespace sllm

using namespace sllm;

// Mirrored by ops/core.py (ctypes.Structure); checked by sllm_group_norm_abi.
struct SllmGroupNorm {
  const void* table;
  const int* ids;
  const float* step;
  const void* y;
  const int* y_rows;
  const float* w_post;
  const void* y2;
  const float* w_post2;
  float* x;
  const long long* row_idx;
  const float* w_out;
  void* z;
  int vocab, ldy, y_terms, ldy2, rows, d, groups, fp32;
  float table_scale, coef, coef2, eps;
};

SLLM_EXPORT int sllm_group_norm_abi(int* out, int n) {
  const int v[2] = {static_cast<int>(sizeof(SllmGroupNorm)), static_cast<int>(offsetof(SllmGroupNorm, eps))};
  for (int i = 0; i < n && i < 2; ++i) out[i] = v[i];
  return 2;
}

template <typename T>
static int group_norm_launch(const SllmGroupNorm* a, cudaStream_t st) {
  GroupNormParams<T> p = {};
  p.table = static_cast<const T*>(a->table); p.ids = a->ids; p.vocab = a->vocab; p.table_scale = a->table_scale; p.step = a->step;
  p.y = static_cast<const T*>(a->y); p.ldy = a->ldy; p.y_rows = a->y_rows; p.y_terms = a->y_terms; p.w_post = a->w_post;
  p.coef = a->coef; p.y2 = static_cast<const T*>(a->y2); p.ldy2 = a->ldy2; p.w_post2 = a->w_post2; p.coef2 = a->coef2;
  p.x = a->x; p.row_idx = a->row_idx; p.w_out = a->w_out; p.z = static_cast<T*>(a->z); p.d = a->d; p.groups = a->groups; p.eps = a->eps;
  p.parts = p.groups >= kGnWarps ? 1 : (kGnWarps + p.groups - 1) / p.groups;
  const size_t smem = sizeof(float) * (static_cast<size_t>((p.d + 3) & ~3) * (a->y2 ? 2 : 1) + p.groups + static_cast<size_t>(p.groups) * p.parts);
  if (smem > 200 * 1024) return SLLM_ERR_UNSUPPORTED_SHAPE;
  const bool vec = (p.d / p.groups) % 4 == 0 && (!a->y || a->ldy % 4 == 0) && (!a->y2 || a->ldy2 % 4 == 0);
  auto* kernel = vec ? group_norm_kernel<T, 4> : group_norm_kernel<T, 1>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
    return SLLM_ERR_CUDA;
  return launch_kernel(kernel, dim3(a->rows), dim3(kGnThreads), smem, st, 1u, p) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

// table + ids without y: embedding mode; y: summand mode (table and step join as well where given); neither: x is read only
// (rows picked by row_idx when given).  z may be null (residual update alone), z without w_out is x in the element type.
// fp32: element type of table, y, y2 and z (0 bf16, 1 fp32).
SLLM_EXPORT int sllm_group_norm(const SllmGroupNorm* a, void* stream) {
  if (!a || !a->x || a->rows <= 0 || a->d <= 0 || a->groups <= 0 || a->d % a->groups) return SLLM_ERR_INVALID_ARGUMENT;
  if ((a->table && (!a->ids || a->vocab <= 0)) || (a->y2 && (!a->y || a->ldy2 < a->d)) || (a->y && a->ldy < a->d) || (!a->z && a->w_out) ||
      (a->y_rows && (!a->y || a->y_terms <= 0)) || (!a->z && !a->y && !a->table) || (a->step && !a->y && !a->table))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->row_idx && (a->table || a->y)) return SLLM_ERR_INVALID_ARGUMENT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->fp32 ? group_norm_launch<float>(a, st) : group_norm_launch<__nv_bfloat16>(a, st);
}
