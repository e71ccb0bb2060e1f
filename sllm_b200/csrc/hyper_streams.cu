// A residual of several parallel streams (hyper-connections), 32-bit, with the work around it in one launch.
//
// x [rows, streams, d].  A sublayer reads a weighted sum of the streams, u = sum_s in[s] x_s, and what it returns flows back
// while the streams mix:  x_t <- sum_s mix[s][t] x_s + out[t] y, all streams from the old ones.
//
// One launch does, per row:
//   1. x_s = table_scale table[id] + pair[row of (previous id, id)]    (start; the pair table is optional), or
//      x_t = sum_s mix[s][t] x_s + out[t] (coef y + coef2 y2)          (after a sublayer), or
//      x as it is, optionally of a gathered row
//   2. z = norm(sum_s in[s] x_s) * w   (the next sublayer's input in the activation type; w a vector or one number)
// The pair table has buckets + 1 rows: (prev mul_prev + id mul_cur) mod buckets, the last for a sequence's first token.  The
// token before a portion's first comes from the sequence's state slot, where the portion's last one is left.
#include "typed.cuh"
#include "api.h"

#include <cstddef>

namespace sllm {

constexpr int kHsThreads = 256, kHsMaxStreams = 16;

template <typename T>
struct StreamParams {
  const T* table;            // [vocab, d]
  const T* pair;             // optional [buckets + 1, d]
  const int *ids, *positions, *seq_index, *row_off, *slots;
  float* last;               // a slot's token, slot s at s * last_stride
  long long last_stride, mul_prev, mul_cur;
  int vocab, buckets;
  float table_scale;
  const T *y, *y2;           // [rows, ldy], optional [rows, ldy2]
  int ldy, ldy2;
  float coef, coef2;
  const float *mix, *out;    // [streams][streams] (from, to), [streams]
  float* x;
  const long long* row_idx;
  const float* in;           // [streams], null: ones
  const float* w;            // [d] or (w_step 0) one number
  int w_step;
  T* z;                      // [rows, d], null: none
  int d, streams;
  float eps;
};

// kS: streams, rounded up; kV: channels per access.
template <typename T, int kS, int kV>
__global__ void __launch_bounds__(kHsThreads) hyper_stream_kernel(const StreamParams<T> p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float u_s[];       // [d]
  __shared__ float mix_s[kS * kS], out_s[kS], in_s[kS], red[kHsThreads / 32];
  __shared__ int pair_row;
  const int r = blockIdx.x, d = p.d, n = p.streams;
  for (int e = threadIdx.x; e < kS * kS; e += kHsThreads) {
    const int s = e / kS, t = e % kS;
    mix_s[e] = p.y && s < n && t < n ? p.mix[s * n + t] : 0.f;
    if (s == 0) {
      out_s[t] = p.y && t < n ? p.out[t] : 0.f;
      in_s[t] = t < n ? (p.in ? p.in[t] : 1.f) : 0.f;
    }
  }
  int id = 0;
  if (p.table) {
    id = p.ids[r];
    if (id < 0 || id >= p.vocab) id = 0;
    if (p.pair && threadIdx.x == 0) {
      const int seq = p.seq_index[r], first = p.row_off[seq];
      float* last = p.last + p.slots[seq] * p.last_stride;
      long long row = p.buckets;
      if (r > first || p.positions[r] > 0) {
        const long long prev = r > first ? p.ids[r - 1] : static_cast<int>(*last);
        row = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
        if (row < 0) row += p.buckets;
      }
      pair_row = static_cast<int>(row);
      if (r == first) *last = static_cast<float>(p.ids[p.row_off[seq + 1] - 1]);   // read above by this thread alone
    }
  }
  __syncthreads();
  auto load = [](const auto* src, float (&v)[kV]) {
    if constexpr (kV == 1) v[0] = ld_f(src);
    else ld_vec<kV>(src, v);
  };
  auto store = [](auto* dst, const float (&v)[kV]) {
    if constexpr (kV == 1) st_f(dst, v[0]);
    else st_vec<kV>(dst, v);
  };
  float* xr = p.x + static_cast<size_t>(p.row_idx ? p.row_idx[r] : r) * n * d;
  float ss = 0.f;
  for (int i = threadIdx.x * kV; i < d; i += kHsThreads * kV) {
    float u[kV] = {};
    if (p.table) {
      float v[kV];
      load(p.table + static_cast<size_t>(id) * d + i, v);
#pragma unroll
      for (int j = 0; j < kV; ++j) v[j] *= p.table_scale;
      if (p.pair) {
        float b[kV];
        load(p.pair + static_cast<size_t>(pair_row) * d + i, b);
#pragma unroll
        for (int j = 0; j < kV; ++j) v[j] += b[j];
      }
#pragma unroll
      for (int s = 0; s < kS; ++s) {
        if (s >= n) break;
        store(xr + static_cast<size_t>(s) * d + i, v);
#pragma unroll
        for (int j = 0; j < kV; ++j) u[j] = fmaf(in_s[s], v[j], u[j]);
      }
    } else {
      float x[kS][kV];
#pragma unroll
      for (int s = 0; s < kS; ++s) {
#pragma unroll
        for (int j = 0; j < kV; ++j) x[s][j] = 0.f;
        if (s < n) load(xr + static_cast<size_t>(s) * d + i, x[s]);
      }
      if (p.y) {
        float y[kV];
        load(p.y + static_cast<size_t>(r) * p.ldy + i, y);
#pragma unroll
        for (int j = 0; j < kV; ++j) y[j] *= p.coef;
        if (p.y2) {
          float b[kV];
          load(p.y2 + static_cast<size_t>(r) * p.ldy2 + i, b);
#pragma unroll
          for (int j = 0; j < kV; ++j) y[j] = fmaf(p.coef2, b[j], y[j]);
        }
#pragma unroll
        for (int t = 0; t < kS; ++t) {
          if (t >= n) break;
          float v[kV];
#pragma unroll
          for (int j = 0; j < kV; ++j) v[j] = out_s[t] * y[j];
#pragma unroll
          for (int s = 0; s < kS; ++s)
#pragma unroll
            for (int j = 0; j < kV; ++j) v[j] = fmaf(mix_s[s * kS + t], x[s][j], v[j]);
          store(xr + static_cast<size_t>(t) * d + i, v);
#pragma unroll
          for (int j = 0; j < kV; ++j) u[j] = fmaf(in_s[t], v[j], u[j]);
        }
      } else {
#pragma unroll
        for (int s = 0; s < kS; ++s)
#pragma unroll
          for (int j = 0; j < kV; ++j) u[j] = fmaf(in_s[s], x[s][j], u[j]);
      }
    }
    store(u_s + i, u);
#pragma unroll
    for (int j = 0; j < kV; ++j) ss += u[j] * u[j];
  }
  if (!p.z) return;
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kHsThreads / 32; ++i) ss += red[i];
  const float inv = 1.f / sqrtf(ss / static_cast<float>(d) + p.eps), one = p.w_step ? 1.f : *p.w;
  T* zr = p.z + static_cast<size_t>(r) * d;
  for (int i = threadIdx.x * kV; i < d; i += kHsThreads * kV) {   // every thread reads back what it wrote
    float v[kV], w[kV];
    load(u_s + i, v);
    if (p.w_step) load(p.w + i, w);
#pragma unroll
    for (int j = 0; j < kV; ++j) v[j] = v[j] * inv * (p.w_step ? w[j] : one);
    store(zr + i, v);
  }
}

}  // namespace sllm

using namespace sllm;

// Mirrored by ops/streams.py (ctypes.Structure); checked by sllm_streams_abi.
struct SllmStreams {
  const void *table, *pair, *ids, *positions, *seq_index, *row_off, *slots, *last, *y, *y2, *mix, *out, *x, *row_idx, *in, *w, *z;
  long long last_stride, mul_prev, mul_cur;
  int vocab, buckets, ldy, ldy2, w_step, rows, d, streams, fp32;
  float table_scale, coef, coef2, eps;
};

SLLM_EXPORT int sllm_streams_abi(int* out, int n) {
  const int v[2] = {static_cast<int>(sizeof(SllmStreams)), static_cast<int>(offsetof(SllmStreams, eps))};
  for (int i = 0; i < n && i < 2; ++i) out[i] = v[i];
  return 2;
}

template <typename T, int kS>
static cudaError_t streams_go(const StreamParams<T>& p, int rows, bool vec, cudaStream_t st) {
  const size_t smem = sizeof(float) * ((p.d + 3) & ~3);
  auto* kernel = vec ? hyper_stream_kernel<T, kS, 4> : hyper_stream_kernel<T, kS, 1>;
  if (smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
  }
  return launch_kernel(kernel, dim3(rows), dim3(kHsThreads), smem, st, 1u, p);
}

template <typename T>
static int streams_launch(const SllmStreams* a, cudaStream_t st) {
  StreamParams<T> p = {};
  auto t = [](const void* x) { return static_cast<T*>(const_cast<void*>(x)); };
  auto f = [](const void* x) { return static_cast<float*>(const_cast<void*>(x)); };
  auto n = [](const void* x) { return static_cast<const int*>(x); };
  p.table = t(a->table); p.pair = t(a->pair); p.ids = n(a->ids); p.positions = n(a->positions); p.seq_index = n(a->seq_index);
  p.row_off = n(a->row_off); p.slots = n(a->slots); p.last = f(a->last); p.last_stride = a->last_stride; p.mul_prev = a->mul_prev;
  p.mul_cur = a->mul_cur; p.vocab = a->vocab; p.buckets = a->buckets; p.table_scale = a->table_scale;
  p.y = t(a->y); p.y2 = t(a->y2); p.ldy = a->ldy; p.ldy2 = a->ldy2; p.coef = a->coef; p.coef2 = a->coef2; p.mix = f(a->mix); p.out = f(a->out);
  p.x = f(a->x); p.row_idx = static_cast<const long long*>(a->row_idx); p.in = f(a->in); p.w = f(a->w); p.w_step = a->w_step; p.z = t(a->z);
  p.d = a->d; p.streams = a->streams; p.eps = a->eps;
  const bool vec = ((p.d | (p.y ? p.ldy : 0) | (p.y2 ? p.ldy2 : 0)) & 3) == 0;
  cudaError_t e;
  switch (p.streams) {
    case 1: e = streams_go<T, 1>(p, a->rows, vec, st); break;
    case 2: e = streams_go<T, 2>(p, a->rows, vec, st); break;
    case 3: e = streams_go<T, 3>(p, a->rows, vec, st); break;
    case 4: e = streams_go<T, 4>(p, a->rows, vec, st); break;
    default: e = p.streams <= 8 ? streams_go<T, 8>(p, a->rows, vec, st) : streams_go<T, kHsMaxStreams>(p, a->rows, vec, st);
  }
  return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

// table: start; y: after a sublayer; neither: x is read only (rows picked by row_idx when given).  fp32: element type of the
// tables, y, y2 and z (0 bf16, 1 fp32).
SLLM_EXPORT int sllm_streams(const SllmStreams* a, void* stream) {
  if (!a || !a->x || a->rows <= 0 || a->d <= 0 || a->streams <= 0 || (a->z && !a->w) || (a->table && a->y) || (!a->z && !a->table && !a->y))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->table && (!a->ids || a->vocab <= 0 || a->row_idx)) return SLLM_ERR_INVALID_ARGUMENT;
  if (a->pair && (!a->table || a->buckets <= 0 || !a->positions || !a->seq_index || !a->row_off || !a->slots || !a->last))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->y && (a->ldy < a->d || !a->mix || !a->out || a->row_idx)) return SLLM_ERR_INVALID_ARGUMENT;
  if (a->y2 && (!a->y || a->ldy2 < a->d)) return SLLM_ERR_INVALID_ARGUMENT;
  if (a->streams > kHsMaxStreams || a->d > 48 * 1024) return SLLM_ERR_UNSUPPORTED_SHAPE;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->fp32 ? streams_launch<float>(a, st) : streams_launch<__nv_bfloat16>(a, st);
}
