// One step of a matrix-valued recurrent state, per head, S [dim keys, vdim values] in fp32:
//   S <- diag(w) S - au (u^T S) + k v^T,   o = S^T r          (kRemoval: with the removal term, kPlain: without it)
//   S <- g S;  S <- S + k (beta (v - S^T k))^T,   o = S^T q   (kGatedDelta: one decay g per head, beta v in place of v)
// Columns of S (value channels) never meet, so heads are cut into column tiles.  A thread keeps 16 keys x 2 or 4 columns of S
// in registers; kKL = 1 .. 32 lanes share a column.  All dot products of a token are taken from the OLD state in one sweep,
//   o = (w r)^T S - (u^T S) (au^T r) + v k^T r,     o = g q^T S + (k^T q) (beta v - beta g k^T S)
// so a token costs one shuffle reduction and no barrier.
#pragma once
#include "typed.cuh"
#include "state_scan.h"

namespace sllm {

constexpr int kDrKeys = 16;          // keys per thread

__host__ __device__ constexpr int state_pad(int dim) {   // padded head size: 16 x a power of two
  int kl = 1;
  while (kl * kDrKeys < dim) kl *= 2;
  return kl * kDrKeys;
}

// What the scan reads per (head, token): the vectors [pad] in this order (the last two with kRemoval only; kGatedDelta: q, k),
// v [value pad], and four scalars: au^T r, k^T r, -, - (kGatedDelta: g, beta g, k^T q, -).
enum StateVec { kVecWR = 0, kVecW = 1, kVecK = 2, kVecU = 3, kVecAU = 4 };
enum GatedVec { kVecGQ = 0, kVecGK = 1 };
__host__ __device__ constexpr int state_vecs(int step) { return step == kGatedDelta ? 2 : step == kRemoval ? 5 : 3; }
__host__ __device__ constexpr int state_vpad(int vdim) { return (vdim + 3) & ~3; }
__host__ __device__ constexpr int state_record(int step, int pad, int vdim) {   // floats
  return state_vecs(step) * pad + state_vpad(vdim) + 4;
}

// Lane l of a warp loads channels d0 = l kN .. + kN - 1 of a head; vec: widths and offsets allow 4-channel accesses.
template <typename T, int kN>
__device__ __forceinline__ void lane_load(const T* src, int d0, int dim, bool vec, float (&v)[kN]) {
  if constexpr (kN % 4 == 0) {
    if (vec) {
#pragma unroll
      for (int i = 0; i < kN; i += 4) {
        float x[4] = {0.f, 0.f, 0.f, 0.f};
        if (d0 + i < dim) ld_vec<4>(src + d0 + i, x);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[i + j] = x[j];
      }
      return;
    }
  }
#pragma unroll
  for (int i = 0; i < kN; ++i) v[i] = d0 + i < dim ? ld_f(src + d0 + i) : 0.f;
}

// Stores the lane's channels below `limit` (a multiple of 4) to 16-byte aligned shared or global floats.
template <int kN>
__device__ __forceinline__ void lane_store(float* dst, int d0, int limit, const float (&x)[kN]) {
  if constexpr (kN % 4 == 0) {
#pragma unroll
    for (int i = 0; i < kN; i += 4)
      if (d0 + i < limit) *reinterpret_cast<float4*>(dst + d0 + i) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < kN; ++i)
      if (d0 + i < limit) dst[d0 + i] = x[i];
  }
}

// The step with one decay per head: two vectors and three scalars.
template <int kKL, int kC>
__device__ __forceinline__ void gated_token(float (&S)[kDrKeys][kC], const float* vs, int kl, const float (&v)[kC], const float4& sc,
                                            float (&o)[kC]) {
  constexpr int pad = kKL * kDrKeys;
  float pc[2][kC], qc[2][kC];                        // two chains per column
#pragma unroll
  for (int c = 0; c < kC; ++c) pc[0][c] = pc[1][c] = qc[0][c] = qc[1][c] = 0.f;
  float ka[kDrKeys];
#pragma unroll
  for (int j = 0; j < kDrKeys / 4; ++j) {
    float qa[4], kv[4];
    ld_vec<4>(vs + kVecGQ * pad + (j * kKL + kl) * 4, qa);
    ld_vec<4>(vs + kVecGK * pad + (j * kKL + kl) * 4, kv);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      ka[j * 4 + e] = kv[e];
#pragma unroll
      for (int c = 0; c < kC; ++c) {
        pc[e & 1][c] = fmaf(kv[e], S[j * 4 + e][c], pc[e & 1][c]);
        qc[e & 1][c] = fmaf(qa[e], S[j * 4 + e][c], qc[e & 1][c]);
      }
    }
  }
  float p[kC], q[kC];
#pragma unroll
  for (int c = 0; c < kC; ++c) {
    p[c] = pc[0][c] + pc[1][c];
    q[c] = qc[0][c] + qc[1][c];
  }
#pragma unroll
  for (int x = kKL / 2; x > 0; x >>= 1)
#pragma unroll
    for (int c = 0; c < kC; ++c) {
      p[c] += __shfl_xor_sync(0xffffffffu, p[c], x);
      q[c] += __shfl_xor_sync(0xffffffffu, q[c], x);
    }
#pragma unroll
  for (int c = 0; c < kC; ++c) {
    p[c] = fmaf(-sc.y, p[c], v[c]);                  // what is written along k
    o[c] = fmaf(sc.x, q[c], sc.z * p[c]);
  }
#pragma unroll
  for (int e = 0; e < kDrKeys; ++e)
#pragma unroll
    for (int c = 0; c < kC; ++c) S[e][c] = fmaf(ka[e], p[c], sc.x * S[e][c]);
}

// One token on a thread's 16 keys x kC columns: S is updated, o holds the outputs on every lane of the columns.
// vs: the token's vectors in shared memory; sc: its scalars.  Key of S[j * 4 + e]: (j * kKL + kl) * 4 + e.
template <int kKL, int kC, int kStep>
__device__ __forceinline__ void state_token(float (&S)[kDrKeys][kC], const float* vs, int kl, const float (&v)[kC], const float4& sc,
                                            float (&o)[kC]) {
  constexpr int pad = kKL * kDrKeys;
  if constexpr (kStep == kGatedDelta) {
    gated_token<kKL, kC>(S, vs, kl, v, sc, o);
    return;
  }
  constexpr bool kDelta = kStep == kRemoval;
  float pc[2][kC], qc[2][kC];                        // two chains per column
#pragma unroll
  for (int c = 0; c < kC; ++c) pc[0][c] = pc[1][c] = qc[0][c] = qc[1][c] = 0.f;
#pragma unroll
  for (int j = 0; j < kDrKeys / 4; ++j) {
    const float4 wr = *reinterpret_cast<const float4*>(vs + kVecWR * pad + (j * kKL + kl) * 4);
    const float wa[4] = {wr.x, wr.y, wr.z, wr.w};
    float ua[4];
    if constexpr (kDelta) ld_vec<4>(vs + kVecU * pad + (j * kKL + kl) * 4, ua);
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int c = 0; c < kC; ++c) {
        if constexpr (kDelta) pc[e & 1][c] = fmaf(ua[e], S[j * 4 + e][c], pc[e & 1][c]);
        qc[e & 1][c] = fmaf(wa[e], S[j * 4 + e][c], qc[e & 1][c]);
      }
  }
  float p[kC], q[kC];
#pragma unroll
  for (int c = 0; c < kC; ++c) {
    p[c] = pc[0][c] + pc[1][c];
    q[c] = qc[0][c] + qc[1][c];
  }
#pragma unroll
  for (int x = kKL / 2; x > 0; x >>= 1)
#pragma unroll
    for (int c = 0; c < kC; ++c) {
      if constexpr (kDelta) p[c] += __shfl_xor_sync(0xffffffffu, p[c], x);
      q[c] += __shfl_xor_sync(0xffffffffu, q[c], x);
    }
#pragma unroll
  for (int j = 0; j < kDrKeys / 4; ++j) {
    float wa[4], aa[4], ka[4];
    ld_vec<4>(vs + kVecW * pad + (j * kKL + kl) * 4, wa);
    ld_vec<4>(vs + kVecK * pad + (j * kKL + kl) * 4, ka);
    if constexpr (kDelta) ld_vec<4>(vs + kVecAU * pad + (j * kKL + kl) * 4, aa);
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int c = 0; c < kC; ++c) {
        float x = wa[e] * S[j * 4 + e][c];
        if constexpr (kDelta) x = fmaf(-aa[e], p[c], x);
        S[j * 4 + e][c] = fmaf(ka[e], v[c], x);
      }
  }
#pragma unroll
  for (int c = 0; c < kC; ++c) o[c] = kDelta ? q[c] - p[c] * sc.x + v[c] * sc.y : fmaf(v[c], sc.y, q[c]);
}

template <int kKL, int kC, bool kStore>
__device__ __forceinline__ void state_io(float (&S)[kDrKeys][kC], float* st, int dim, int vdim, int kl, int col) {
  const bool whole = vdim % kC == 0;                 // col is a multiple of kC: its columns are one aligned access
#pragma unroll
  for (int j = 0; j < kDrKeys / 4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = (j * kKL + kl) * 4 + e;
      float* ptr = st + static_cast<size_t>(key) * vdim + col;
      float(&x)[kC] = S[j * 4 + e];
      const bool in = key < dim && col < vdim;
      if constexpr (kStore) {
        if (in && whole) {
          st_vec<kC>(ptr, x);
        } else if (in) {
#pragma unroll
          for (int c = 0; c < kC; ++c)
            if (col + c < vdim) ptr[c] = x[c];
        }
      } else {
#pragma unroll
        for (int c = 0; c < kC; ++c) x[c] = 0.f;
        if (in && whole) {
          ld_vec<kC>(ptr, x);
        } else if (in) {
#pragma unroll
          for (int c = 0; c < kC; ++c)
            if (col + c < vdim) x[c] = ptr[c];
        }
      }
    }
}

__device__ __forceinline__ float block_sum(float v, float* red, int warps) {
  v = warp_sum(v);
  __syncthreads();                                   // red may still be read from the previous sum
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < warps; ++i) s += red[i];
  return s;
}

}  // namespace sllm
