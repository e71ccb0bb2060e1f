// The recurrence of state_scan.cuh over the rows of a flat batch (rows of sequence s: row_off[s] .. row_off[s + 1], its state
// in slot slots[s]).  Everything that does not depend on the state comes in staged records, one per (head, token).
#include "state_scan.h"
#include "state_scan.cuh"

namespace sllm {

constexpr int kDrChunk = 8;          // tokens staged at a time
constexpr int kDrScanWarps = 4;

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// grid (heads, column tiles, sequences), 4 warps of (32 / kKL) groups of kC columns.
template <int kKL, int kC, int kStep>
__global__ void __launch_bounds__(kDrScanWarps * 32) state_scan_kernel(const ScanParams p) {
  pdl_wait();
  constexpr int pad = kKL * kDrKeys, nv = state_vecs(kStep);
  const int h = blockIdx.x, s = blockIdx.z, D = p.dim, V = p.vdim, vpad = state_vpad(V), rec = state_record(kStep, pad, V);
  extern __shared__ __align__(16) float buf[];       // [2][kDrChunk][rec]
  const int r0 = p.row_off[s], r1 = p.row_off[s + 1];
  if (r1 <= r0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % kKL;
  const int col = ((blockIdx.y * kDrScanWarps + warp) * (32 / kKL) + lane / kKL) * kC;
  float* st = p.state + static_cast<long long>(p.slots[s]) * p.slot_stride + static_cast<size_t>(h) * D * V;
  float S[kDrKeys][kC];
  state_io<kKL, kC, false>(S, st, D, V, kl, col);
  const float* vec = p.vec + static_cast<size_t>(h) * p.tokens * rec;
  auto stage = [&](int c0, int b) {
    const int n = min(kDrChunk, r1 - c0) * (rec / 4);
    for (int e = threadIdx.x; e < n; e += kDrScanWarps * 32)
      cp_async16(buf + b * kDrChunk * rec + e * 4, vec + static_cast<size_t>(c0) * rec + e * 4);
  };
  stage(r0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  int b = 0;
  for (int c0 = r0; c0 < r1; c0 += kDrChunk, b ^= 1) {
    if (c0 + kDrChunk < r1) stage(c0 + kDrChunk, b ^ 1);
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const int n = min(kDrChunk, r1 - c0);
    for (int i = 0; i < n; ++i) {
      const float* vs = buf + (b * kDrChunk + i) * rec;
      const float4 sc = *reinterpret_cast<const float4*>(vs + nv * pad + vpad);
      float v[kC], o[kC];
#pragma unroll
      for (int c = 0; c < kC; ++c) v[c] = col < vpad ? vs[nv * pad + col + c] : 0.f;
      state_token<kKL, kC, kStep>(S, vs, kl, v, sc, o);
      if (kl == 0) {
        float* dst = p.o_raw + (static_cast<size_t>(c0 + i) * p.heads + h) * V + col;
#pragma unroll
        for (int c = 0; c < kC; ++c)
          if (col + c < V) dst[c] = o[c];
      }
    }
    __syncthreads();                                 // the buffer is refilled by the next iteration's stage()
  }
  pdl_trigger();
  state_io<kKL, kC, true>(S, st, D, V, kl, col);
}

template <int kKL, int kC, int kStep>
static int scan_go(const ScanParams& p, int sequences, cudaStream_t st) {
  constexpr int cols = kDrScanWarps * (32 / kKL) * kC;
  const dim3 grid(p.heads, (p.vdim + cols - 1) / cols, sequences);
  size_t smem = sizeof(float) * 2 * kDrChunk * state_record(kStep, kKL * kDrKeys, p.vdim);
  // a grid that fits one CTA per SM asks for more than half of an SM's shared memory, so that no two share one
  if (static_cast<long long>(grid.x) * grid.y * grid.z <= 148 && smem < 116 * 1024) smem = 116 * 1024;
  if (smem > 227 * 1024) return SLLM_ERR_UNSUPPORTED_SHAPE;
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    if (cudaFuncSetAttribute(state_scan_kernel<kKL, kC, kStep>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) !=
        cudaSuccess)
      return SLLM_ERR_CUDA;
    configured = smem;
  }
  return launch_kernel(state_scan_kernel<kKL, kC, kStep>, grid, dim3(kDrScanWarps * 32), smem, st, 1u, p) == cudaSuccess ? SLLM_OK
                                                                                                                           : SLLM_ERR_CUDA;
}

// The scan is bound by its reads of the staged vectors: more columns per thread reuse them more often, fewer spread a small
// batch over more SMs.
template <int kKL, int kStep>
static int scan_columns(const ScanParams& p, int sequences, cudaStream_t st) {
  constexpr int cols = kDrScanWarps * (32 / kKL) * 2;
  if (static_cast<long long>(p.heads) * ((p.vdim + cols - 1) / cols) * sequences > 148) return scan_go<kKL, 4, kStep>(p, sequences, st);
  return scan_go<kKL, 2, kStep>(p, sequences, st);
}

template <int kStep>
static int scan_keys(const ScanParams& p, int sequences, cudaStream_t st) {
  switch (state_pad(p.dim) / kDrKeys) {
    case 1: return scan_columns<1, kStep>(p, sequences, st);
    case 2: return scan_columns<2, kStep>(p, sequences, st);
    case 4: return scan_columns<4, kStep>(p, sequences, st);
    case 8: return scan_columns<8, kStep>(p, sequences, st);
    case 16: return scan_columns<16, kStep>(p, sequences, st);
    case 32: return scan_columns<32, kStep>(p, sequences, st);
    default: return SLLM_ERR_UNSUPPORTED_SHAPE;
  }
}

int state_scan_launch(const ScanParams& p, int step, int sequences, cudaStream_t stream) {
  if (step == kGatedDelta) return scan_keys<kGatedDelta>(p, sequences, stream);
  return step == kRemoval ? scan_keys<kRemoval>(p, sequences, stream) : scan_keys<kPlain>(p, sequences, stream);
}

}  // namespace sllm
