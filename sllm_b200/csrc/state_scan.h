// Scan over matrix-valued recurrent states (state_scan.cu), driven by delta_rule.cu and linear_state.cu.
#pragma once
#include <cuda_runtime.h>

namespace sllm {

// What one token does to a state, see state_scan.cuh.
enum StateStep { kPlain = 0, kRemoval = 1, kGatedDelta = 2 };

// vec: [heads][tokens] records, see state_record in state_scan.cuh.  State of slot s, head h: state + s * slot_stride +
// h * dim * vdim, [dim keys][vdim values].  o_raw: [tokens, heads * vdim].
struct ScanParams {
  const float* vec;
  float* state;
  long long slot_stride;
  const int *row_off, *slots;
  float* o_raw;
  int heads, dim, vdim, tokens;
};

// step: a StateStep, which the records are made for.  Returns an SllmStatus.
int state_scan_launch(const ScanParams& p, int step, int sequences, cudaStream_t stream);

}  // namespace sllm
