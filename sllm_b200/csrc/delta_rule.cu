// Generalised delta rule with a decay and a removal rate per key channel:
//   S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T,   o_t = S_t^T r_t,
//   u = k / sqrt(sum k^2 + eps_u),  w = exp(-exp(-1/2) sigmoid(x)),  a = sigmoid(z)
// per head, S [dim keys, dim values] in fp32; then each head's o is divided by its root mean square, weighted and gated:
//   y = o / rms(o) * norm_w * sigmoid(g).
// The batch is flat (rows of sequence s: row_off[s] .. row_off[s + 1]) and sequence s owns state slot slots[s].
//
// Prompts: delta_pre_kernel computes everything that does not depend on the state in parallel over the tokens, the scan of
// state_scan.cu runs the recurrence, delta_post_kernel normalises and gates.  One-token batches (decode) take
// delta_decode_kernel, which does all of it, the low-rank decay projection included, in one launch.
#include <cstddef>
#include <type_traits>
#include "state_scan.cuh"
#include "state_scan.h"
#include "api.h"

namespace sllm {

constexpr int kDrDecodeThreads = 256;
constexpr float kDecayRate = 0.60653065971263342f;   // exp(-1/2)

template <typename T>
struct DeltaParams {
  const T* proj;           // [tokens, ldp]: r | k | v | a | g | low-rank decay input, columns off_*
  int ldp, off_r, off_k, off_v, off_a, off_g, off_w1, rank;
  const T* decay;          // prompt form: [tokens, ld_decay] second product of the decay projection
  int ld_decay;
  const T* w2;             // decode form: [heads * dim, ld_w2]
  int ld_w2;
  const float* w0;         // [heads * dim]
  const float* a_bias;     // [heads * dim]
  const float* norm_w;     // [heads * dim]
  float eps_u, eps;
  float* state;            // slot s, head h at state + s * slot_stride + h * dim * dim, [dim keys][dim values]
  long long slot_stride;
  const int* row_off;
  const int* slots;
  int heads, dim, tokens;
  float* vec;              // [heads][tokens] records of the scan
  float* o_raw;            // [tokens, heads * dim]
  T* out;                  // [tokens, heads * dim]
};

// ---------------------------------------------------------------- prompt form
// A warp per (token, head), lane l the channels l kN .. l kN + kN - 1 (kN = padded head size / 32, at least 1); vec: heads
// and offsets allow 4-channel accesses.
constexpr int kDrRowWarps = 8;       // (token, head) pairs per CTA of the row kernels

// No early trigger of the dependent launch here: the scan's few CTAs would become resident while this grid drains, several
// of them on the first SMs that run empty, and share those SMs' shared-memory bandwidth for their whole run.
template <typename T, int kN>
__global__ void __launch_bounds__(kDrRowWarps * 32) delta_pre_kernel(const DeltaParams<T> p, bool vec) {
  pdl_wait();
  const int lane = threadIdx.x & 31, D = p.dim, pad = state_pad(D), d0 = lane * kN;
  const long long unit = static_cast<long long>(blockIdx.x) * kDrRowWarps + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(p.tokens) * p.heads) return;
  const int t = static_cast<int>(unit / p.heads), h = static_cast<int>(unit % p.heads);
  const T* row = p.proj + static_cast<size_t>(t) * p.ldp + h * D;
  float r[kN], k[kN], v[kN], a[kN], w[kN], b0[kN], b1[kN];
  lane_load<T, kN>(row + p.off_r, d0, D, vec, r);
  lane_load<T, kN>(row + p.off_k, d0, D, vec, k);
  lane_load<T, kN>(row + p.off_v, d0, D, vec, v);
  lane_load<T, kN>(row + p.off_a, d0, D, vec, a);
  lane_load<T, kN>(p.decay + static_cast<size_t>(t) * p.ld_decay + h * D, d0, D, vec, w);
  lane_load<float, kN>(p.w0 + h * D, d0, D, vec, b0);
  lane_load<float, kN>(p.a_bias + h * D, d0, D, vec, b1);
  float kk = 0.f, s1 = 0.f, s2 = 0.f;
#pragma unroll
  for (int i = 0; i < kN; ++i) kk += k[i] * k[i];
  const float inv = 1.f / sqrtf(warp_sum(kk) + p.eps_u);
  float u[kN];
#pragma unroll
  for (int i = 0; i < kN; ++i) {
    const bool in = d0 + i < D;
    w[i] = in ? expf(-kDecayRate * sigmoid_f(w[i] + b0[i])) : 0.f;
    u[i] = k[i] * inv;
    a[i] = in ? sigmoid_f(a[i] + b1[i]) * u[i] : 0.f;
    s1 += a[i] * r[i];
    s2 += k[i] * r[i];
    r[i] *= w[i];
  }
  s1 = warp_sum(s1);
  s2 = warp_sum(s2);
  float* dst = p.vec + (static_cast<size_t>(h) * p.tokens + t) * state_record(kRemoval, pad, D);
  lane_store(dst + kVecWR * pad, d0, pad, r);
  lane_store(dst + kVecW * pad, d0, pad, w);
  lane_store(dst + kVecK * pad, d0, pad, k);
  lane_store(dst + kVecU * pad, d0, pad, u);
  lane_store(dst + kVecAU * pad, d0, pad, a);
  dst += state_vecs(kRemoval) * pad;
  lane_store(dst, d0, state_vpad(D), v);
  if (lane == 0) *reinterpret_cast<float2*>(dst + state_vpad(D)) = make_float2(s1, s2);
}

// A warp per (token, head), as in the first stage.
template <typename T, int kN>
__global__ void __launch_bounds__(kDrRowWarps * 32) delta_post_kernel(const DeltaParams<T> p, bool vec) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, D = p.dim, d0 = lane * kN;
  const long long unit = static_cast<long long>(blockIdx.x) * kDrRowWarps + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(p.tokens) * p.heads) return;
  const int t = static_cast<int>(unit / p.heads), h = static_cast<int>(unit % p.heads);
  const size_t idx = static_cast<size_t>(t) * p.heads * D + h * D;
  float o[kN], g[kN], w[kN];
  lane_load<float, kN>(p.o_raw + idx, d0, D, vec, o);
  lane_load<T, kN>(p.proj + static_cast<size_t>(t) * p.ldp + p.off_g + h * D, d0, D, vec, g);
  lane_load<float, kN>(p.norm_w + h * D, d0, D, vec, w);
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kN; ++i) ss += o[i] * o[i];
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(D) + p.eps);
#pragma unroll
  for (int i = 0; i < kN; ++i) o[i] = o[i] * inv * w[i] * sigmoid_f(g[i]);
  T* dst = p.out + idx + d0;
  if constexpr (kN % 4 == 0) {
    if (vec) {
#pragma unroll
      for (int i = 0; i < kN; i += 4) {
        const float x[4] = {o[i], o[i + 1], o[i + 2], o[i + 3]};
        if (d0 + i < D) st_vec<4>(dst + i, x);
      }
      return;
    }
  }
#pragma unroll
  for (int i = 0; i < kN; ++i)
    if (d0 + i < D) st_f(dst + i, o[i]);
}

// ---------------------------------------------------------------- decode form: exactly one row per sequence
// grid (heads, sequences), 256 threads; warps sweep the head's column tiles.
template <typename T, int kKL>
__global__ void __launch_bounds__(kDrDecodeThreads) delta_decode_kernel(const DeltaParams<T> p) {
  pdl_wait();
  pdl_trigger();
  constexpr int pad = kKL * kDrKeys;
  constexpr int kWarps = kDrDecodeThreads / 32;
  __shared__ __align__(16) float vs[(state_vecs(kRemoval) + 1) * pad];
  __shared__ float o_s[pad];
  __shared__ float red[kWarps];
  extern __shared__ float low[];                     // [rank] tanh of the low-rank decay input
  const int h = blockIdx.x, s = blockIdx.y, D = p.dim, t = p.row_off[s];
  if (p.row_off[s + 1] <= t) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % kKL;
  const T* row = p.proj + static_cast<size_t>(t) * p.ldp;
  float* st = p.state + static_cast<long long>(p.slots[s]) * p.slot_stride + static_cast<size_t>(h) * D * D;
  // the first tile of the state is requested before anything is computed
  int col = (warp * (32 / kKL) + lane / kKL) * 2;
  float S[kDrKeys][2];
  state_io<kKL, 2, false>(S, st, D, D, kl, col);
  for (int i = threadIdx.x; i < p.rank; i += kDrDecodeThreads) low[i] = tanhf(ld_f(row + p.off_w1 + i));
  __syncthreads();
  float kk = 0.f, kr = 0.f;
  for (int d = threadIdx.x; d < pad; d += kDrDecodeThreads) {
    const int c = h * D + d;
    float r = 0.f, k = 0.f, v = 0.f, w = 0.f, a = 0.f;
    if (d < D) {
      r = ld_f(row + p.off_r + c);
      k = ld_f(row + p.off_k + c);
      v = ld_f(row + p.off_v + c);
      a = sigmoid_f(ld_f(row + p.off_a + c) + p.a_bias[c]);
      const T* w2 = p.w2 + static_cast<size_t>(c) * p.ld_w2;
      float x = p.w0[c];
      if (p.ld_w2 % kVec16<T> == 0) {
        for (int i = 0; i < p.rank; i += kVec16<T>) {   // columns past the rank are zero
          float wv[kVec16<T>];
          ld16(w2 + i, wv);
#pragma unroll
          for (int j = 0; j < kVec16<T>; ++j) x = fmaf(wv[j], i + j < p.rank ? low[i + j] : 0.f, x);
        }
      } else {
        for (int i = 0; i < p.rank; ++i) x = fmaf(ld_f(w2 + i), low[i], x);
      }
      w = expf(-kDecayRate * sigmoid_f(x));
    }
    vs[kVecWR * pad + d] = w * r; vs[kVecW * pad + d] = w; vs[kVecAU * pad + d] = a; vs[kVecK * pad + d] = k; vs[5 * pad + d] = v;
    vs[kVecU * pad + d] = r;
    kk += k * k;
    kr += k * r;
  }
  kk = block_sum(kk, red, kWarps);
  const float s2 = block_sum(kr, red, kWarps);
  const float inv_u = 1.f / sqrtf(kk + p.eps_u);
  float s1 = 0.f;
  for (int d = threadIdx.x; d < pad; d += kDrDecodeThreads) {   // each thread rewrites only what it wrote above
    const float r = vs[kVecU * pad + d], u = vs[kVecK * pad + d] * inv_u, au = vs[kVecAU * pad + d] * u;
    s1 += au * r;
    vs[kVecU * pad + d] = u;
    vs[kVecAU * pad + d] = au;
  }
  s1 = block_sum(s1, red, kWarps);                   // its barriers also publish vs
  constexpr int kSweep = kWarps * (32 / kKL) * 2;    // columns per sweep of the CTA
  for (int base = 0; base < D; base += kSweep) {
    if (base > 0) {
      col += kSweep;
      state_io<kKL, 2, false>(S, st, D, D, kl, col);
    }
    float v[2] = {0.f, 0.f}, o[2];
    if (col < pad) { v[0] = vs[5 * pad + col]; v[1] = vs[5 * pad + col + 1]; }
    state_token<kKL, 2, kRemoval>(S, vs, kl, v, make_float4(s1, s2, 0.f, 0.f), o);
    state_io<kKL, 2, true>(S, st, D, D, kl, col);
    if (kl == 0 && col < pad) { o_s[col] = o[0]; o_s[col + 1] = o[1]; }
  }
  __syncthreads();
  float ss = 0.f;
  for (int d = threadIdx.x; d < D; d += kDrDecodeThreads) ss += o_s[d] * o_s[d];
  ss = block_sum(ss, red, kWarps);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(D) + p.eps);
  for (int d = threadIdx.x; d < D; d += kDrDecodeThreads) {
    const int c = h * D + d;
    st_f(p.out + static_cast<size_t>(t) * p.heads * D + c, o_s[d] * inv * p.norm_w[c] * sigmoid_f(ld_f(row + p.off_g + c)));
  }
}

// y[t, i] = tanh(x[t, i]) for i < n, 0 for n <= i < n_pad (the padded operand of the second decay product).
template <typename T>
__global__ void tanh_rows_kernel(const T* __restrict__ x, T* __restrict__ y, int ldx, int n, int n_pad) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  for (int i = threadIdx.x; i < n_pad; i += blockDim.x)
    st_f(y + static_cast<size_t>(t) * n_pad + i, i < n ? tanhf(ld_f(x + static_cast<size_t>(t) * ldx + i)) : 0.f);
}

template <typename T, int kN>
static cudaError_t delta_rows_launch(const DeltaParams<T>& p, bool pre, bool vec, cudaStream_t st) {
  const long long units = static_cast<long long>(p.tokens) * p.heads;
  const dim3 grid(static_cast<unsigned>((units + kDrRowWarps - 1) / kDrRowWarps));
  return launch_kernel(pre ? delta_pre_kernel<T, kN> : delta_post_kernel<T, kN>, grid, dim3(kDrRowWarps * 32), 0, st, 1u, p, vec);
}
template <typename T>
static cudaError_t delta_rows(const DeltaParams<T>& p, int pad, bool pre, cudaStream_t st) {
  const bool vec = ((p.dim | p.ldp | p.off_r | p.off_k | p.off_v | p.off_a | p.off_g | p.ld_decay) & 3) == 0;
  switch (pad / 32) {
    case 0: case 1: return delta_rows_launch<T, 1>(p, pre, vec, st);
    case 2: return delta_rows_launch<T, 2>(p, pre, vec, st);
    case 4: return delta_rows_launch<T, 4>(p, pre, vec, st);
    case 8: return delta_rows_launch<T, 8>(p, pre, vec, st);
    default: return delta_rows_launch<T, 16>(p, pre, vec, st);
  }
}

template <typename T>
static int delta_prompt_launch(DeltaParams<T> p, int sequences, cudaStream_t st) {
  const int pad = state_pad(p.dim);
  if (delta_rows<T>(p, pad, true, st) != cudaSuccess) return SLLM_ERR_CUDA;
  const ScanParams sp{p.vec, p.state, p.slot_stride, p.row_off, p.slots, p.o_raw, p.heads, p.dim, p.dim, p.tokens};
  const int rc = state_scan_launch(sp, kRemoval, sequences, st);
  if (rc != SLLM_OK) return rc;
  return delta_rows<T>(p, pad, false, st) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

template <typename T>
static int delta_decode_launch(const DeltaParams<T>& p, int sequences, cudaStream_t st) {
  const dim3 grid(p.heads, sequences), block(kDrDecodeThreads);
  const size_t smem = sizeof(float) * p.rank;
  cudaError_t e;
  switch (state_pad(p.dim) / kDrKeys) {
    case 1: e = launch_kernel(delta_decode_kernel<T, 1>, grid, block, smem, st, 1u, p); break;
    case 2: e = launch_kernel(delta_decode_kernel<T, 2>, grid, block, smem, st, 1u, p); break;
    case 4: e = launch_kernel(delta_decode_kernel<T, 4>, grid, block, smem, st, 1u, p); break;
    case 8: e = launch_kernel(delta_decode_kernel<T, 8>, grid, block, smem, st, 1u, p); break;
    case 16: e = launch_kernel(delta_decode_kernel<T, 16>, grid, block, smem, st, 1u, p); break;
    default: e = launch_kernel(delta_decode_kernel<T, 32>, grid, block, smem, st, 1u, p); break;
  }
  return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

}  // namespace sllm

using namespace sllm;

struct SllmDeltaArgs {     // host-side mirror passed by the Python layer (ctypes.Structure)
  const void* proj;
  const void* decay;
  const void* w2;
  const float* w0;
  const float* a_bias;
  const float* norm_w;
  float* state;
  const int* row_off;
  const int* slots;
  float* scratch;          // prompt form: heads * tokens * (5 * pad + dim padded to 4 + 4) + tokens * heads * dim floats, 16-byte aligned
  void* out;
  long long slot_stride, scratch_floats;
  int ldp, off_r, off_k, off_v, off_a, off_g, off_w1, rank, ld_decay, ld_w2, heads, dim, tokens, sequences, fp32, decode;
  float eps_u, eps;
};

// decode = 1: exactly one row per sequence (w2 and rank used); 0: any rows (decay and scratch used).
SLLM_EXPORT int sllm_general_delta(const SllmDeltaArgs* a, void* stream) {
  if (!a || !a->proj || !a->w0 || !a->a_bias || !a->norm_w || !a->state || !a->row_off || !a->slots || !a->out || a->heads <= 0 ||
      a->dim <= 0 || a->tokens <= 0 || a->sequences <= 0 || a->heads > 65535 || a->sequences > 65535)
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->dim > 512) return SLLM_ERR_UNSUPPORTED_SHAPE;
  const int pad = state_pad(a->dim);
  const long long nv = static_cast<long long>(a->heads) * a->tokens * state_record(kRemoval, pad, a->dim);
  const long long no = static_cast<long long>(a->tokens) * a->heads * a->dim;
  if (a->decode) {
    if (!a->w2 || a->rank <= 0 || a->ld_w2 < a->rank || a->rank > 8192) return SLLM_ERR_INVALID_ARGUMENT;
  } else {
    if (!a->decay || !a->scratch) return SLLM_ERR_INVALID_ARGUMENT;
    if (a->scratch_floats < nv + no) return SLLM_ERR_WORKSPACE_TOO_SMALL;
    if (reinterpret_cast<uintptr_t>(a->scratch) & 15) return SLLM_ERR_ALIGNMENT;
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto run = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    DeltaParams<T> p = {};
    p.proj = static_cast<const T*>(a->proj); p.ldp = a->ldp;
    p.off_r = a->off_r; p.off_k = a->off_k; p.off_v = a->off_v; p.off_a = a->off_a; p.off_g = a->off_g; p.off_w1 = a->off_w1;
    p.rank = a->rank; p.decay = static_cast<const T*>(a->decay); p.ld_decay = a->ld_decay;
    p.w2 = static_cast<const T*>(a->w2); p.ld_w2 = a->ld_w2; p.w0 = a->w0; p.a_bias = a->a_bias; p.norm_w = a->norm_w;
    p.eps_u = a->eps_u; p.eps = a->eps; p.state = a->state; p.slot_stride = a->slot_stride; p.row_off = a->row_off; p.slots = a->slots;
    p.heads = a->heads; p.dim = a->dim; p.tokens = a->tokens; p.out = static_cast<T*>(a->out);
    if (a->decode) return delta_decode_launch<T>(p, a->sequences, st);
    p.vec = a->scratch; p.o_raw = a->scratch + nv;
    return delta_prompt_launch<T>(p, a->sequences, st);
  };
  return a->fp32 ? run(static_cast<float*>(nullptr)) : run(static_cast<__nv_bfloat16*>(nullptr));
}

SLLM_EXPORT int sllm_tanh_rows(const void* x, void* y, int rows, int ldx, int n, int n_pad, int fp32, void* stream) {
  if (!x || !y || rows <= 0 || n <= 0 || n_pad < n || ldx < n) return SLLM_ERR_INVALID_ARGUMENT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 block(n_pad < 128 ? 64 : 128);
  const cudaError_t e =
      fp32 ? launch_kernel(tanh_rows_kernel<float>, dim3(rows), block, 0, st, 1u, static_cast<const float*>(x), static_cast<float*>(y),
                           ldx, n, n_pad)
           : launch_kernel(tanh_rows_kernel<__nv_bfloat16>, dim3(rows), block, 0, st, 1u, static_cast<const __nv_bfloat16*>(x),
                           static_cast<__nv_bfloat16*>(y), ldx, n, n_pad);
  return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

SLLM_EXPORT int sllm_delta_abi(int* out, int n) {
  if (!out || n < 2) return 0;
  out[0] = static_cast<int>(sizeof(SllmDeltaArgs));
  out[1] = static_cast<int>(offsetof(SllmDeltaArgs, eps));
  return 2;
}
