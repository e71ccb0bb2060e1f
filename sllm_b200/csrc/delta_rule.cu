// Generalised delta rule with a decay and a removal rate per key channel:
//   S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T,   o_t = S_t^T r_t,
//   u = k / sqrt(sum k^2 + eps_u),  w = exp(-exp(-1/2) sigmoid(x)),  a = sigmoid(z)
// per head, S [dim keys, dim values] in fp32; then each head's o is divided by its root mean square, weighted and gated:
//   y = o / rms(o) * norm_w * sigmoid(g).
// The batch is flat (rows of sequence s: row_off[s] .. row_off[s + 1]) and sequence s owns state slot slots[s].
//
// Columns of S (value channels) never meet: column j only needs p = u^T S_j, so heads are cut into column tiles.  A
// thread keeps 16 keys x 2 columns of S in registers; kKL = 1 .. 32 lanes share a column.  Both dot products of a token
// are taken from the OLD state in one sweep, because
//   o = S_t^T r = (w r)^T S_{t-1} - p (a u)^T r + v k^T r
// so a token costs one shuffle reduction and no barrier.
//
// Prompts: delta_pre_kernel computes everything that does not depend on the state in parallel over the tokens,
// delta_scan_kernel runs the recurrence, delta_post_kernel normalises and gates.  One-token batches (decode) take
// delta_decode_kernel, which does all of it, the low-rank decay projection included, in one launch.
#include <cstddef>
#include <type_traits>
#include "typed.cuh"
#include "api.h"

namespace sllm {

constexpr int kDrKeys = 16;          // keys per thread
constexpr int kDrVecs = 6;           // u, w r, w, a u, k, v
constexpr int kDrChunk = 8;          // tokens staged at a time by the scan
constexpr int kDrScanWarps = 4;
constexpr int kDrDecodeThreads = 256;
constexpr float kDecayRate = 0.60653065971263342f;   // exp(-1/2)

__host__ __device__ constexpr int delta_pad(int dim) {   // padded head size: 16 x a power of two
  int kl = 1;
  while (kl * kDrKeys < dim) kl *= 2;
  return kl * kDrKeys;
}

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
  float* vec;              // [heads][tokens][6][pad]
  float* sums;             // [heads][tokens][2]: (a u)^T r, k^T r
  float* o_raw;            // [tokens, heads * dim]
  T* out;                  // [tokens, heads * dim]
};

__device__ __forceinline__ float block_sum(float v, float* red, int warps) {
  v = warp_sum(v);
  __syncthreads();                                   // red may still be read from the previous sum
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < warps; ++i) s += red[i];
  return s;
}

// ---------------------------------------------------------------- prompt form
// grid (tokens, heads), block = padded head size (at least 32).
template <typename T>
__global__ void delta_pre_kernel(const DeltaParams<T> p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[16];
  const int t = blockIdx.x, h = blockIdx.y, d = threadIdx.x, D = p.dim, pad = delta_pad(D), warps = blockDim.x >> 5;
  const bool in = d < D;
  const int c = h * D + d;
  float r = 0.f, k = 0.f, v = 0.f, w = 0.f, a = 0.f;
  if (in) {
    const T* row = p.proj + static_cast<size_t>(t) * p.ldp;
    r = ld_f(row + p.off_r + c);
    k = ld_f(row + p.off_k + c);
    v = ld_f(row + p.off_v + c);
    a = sigmoid_f(ld_f(row + p.off_a + c) + p.a_bias[c]);
    w = expf(-kDecayRate * sigmoid_f(ld_f(p.decay + static_cast<size_t>(t) * p.ld_decay + c) + p.w0[c]));
  }
  const float kk = block_sum(k * k, red, warps);
  const float u = k / sqrtf(kk + p.eps_u);
  const float s1 = block_sum(a * u * r, red, warps);
  const float s2 = block_sum(k * r, red, warps);
  const size_t ht = static_cast<size_t>(h) * p.tokens + t;
  if (d < pad) {
    float* dst = p.vec + ht * kDrVecs * pad + d;
    dst[0] = u; dst[pad] = w * r; dst[2 * pad] = w; dst[3 * pad] = a * u; dst[4 * pad] = k; dst[5 * pad] = v;
  }
  if (d == 0) {
    p.sums[ht * 2] = s1;
    p.sums[ht * 2 + 1] = s2;
  }
}

// One token on a thread's 16 keys x 2 columns: S is updated, o[2] holds the outputs on every lane of the column.
// vs: the token's [6][pad] vectors in shared memory.  Key of S[j * 4 + e]: (j * kKL + kl) * 4 + e.
template <int kKL>
__device__ __forceinline__ void delta_token(float (&S)[kDrKeys][2], const float* vs, int kl, const float (&v)[2], float s1, float s2,
                                            float (&o)[2]) {
  constexpr int pad = kKL * kDrKeys;
  float p0 = 0.f, p1 = 0.f, q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int j = 0; j < kDrKeys / 4; ++j) {
    const float4 u = *reinterpret_cast<const float4*>(vs + (j * kKL + kl) * 4);
    const float4 wr = *reinterpret_cast<const float4*>(vs + pad + (j * kKL + kl) * 4);
    const float ua[4] = {u.x, u.y, u.z, u.w}, wa[4] = {wr.x, wr.y, wr.z, wr.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      p0 = fmaf(ua[e], S[j * 4 + e][0], p0);
      p1 = fmaf(ua[e], S[j * 4 + e][1], p1);
      q0 = fmaf(wa[e], S[j * 4 + e][0], q0);
      q1 = fmaf(wa[e], S[j * 4 + e][1], q1);
    }
  }
#pragma unroll
  for (int x = kKL / 2; x > 0; x >>= 1) {
    p0 += __shfl_xor_sync(0xffffffffu, p0, x);
    p1 += __shfl_xor_sync(0xffffffffu, p1, x);
    q0 += __shfl_xor_sync(0xffffffffu, q0, x);
    q1 += __shfl_xor_sync(0xffffffffu, q1, x);
  }
#pragma unroll
  for (int j = 0; j < kDrKeys / 4; ++j) {
    const float4 w = *reinterpret_cast<const float4*>(vs + 2 * pad + (j * kKL + kl) * 4);
    const float4 au = *reinterpret_cast<const float4*>(vs + 3 * pad + (j * kKL + kl) * 4);
    const float4 k = *reinterpret_cast<const float4*>(vs + 4 * pad + (j * kKL + kl) * 4);
    const float wa[4] = {w.x, w.y, w.z, w.w}, aa[4] = {au.x, au.y, au.z, au.w}, ka[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      S[j * 4 + e][0] = fmaf(ka[e], v[0], fmaf(-aa[e], p0, wa[e] * S[j * 4 + e][0]));
      S[j * 4 + e][1] = fmaf(ka[e], v[1], fmaf(-aa[e], p1, wa[e] * S[j * 4 + e][1]));
    }
  }
  o[0] = q0 - p0 * s1 + v[0] * s2;
  o[1] = q1 - p1 * s1 + v[1] * s2;
}

template <int kKL, bool kStore>
__device__ __forceinline__ void delta_state_io(float (&S)[kDrKeys][2], float* st, int dim, int kl, int col) {
  const bool pair = (dim & 1) == 0;                  // col is even: two columns are one aligned 8-byte access
#pragma unroll
  for (int j = 0; j < kDrKeys / 4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = (j * kKL + kl) * 4 + e;
      float* ptr = st + static_cast<size_t>(key) * dim + col;
      if constexpr (kStore) {
        if (key < dim && col < dim) {
          if (pair) {
            *reinterpret_cast<float2*>(ptr) = make_float2(S[j * 4 + e][0], S[j * 4 + e][1]);
          } else {
            ptr[0] = S[j * 4 + e][0];
            if (col + 1 < dim) ptr[1] = S[j * 4 + e][1];
          }
        }
      } else {
        float2 x = make_float2(0.f, 0.f);
        if (key < dim && col < dim) {
          if (pair) {
            x = *reinterpret_cast<const float2*>(ptr);
          } else {
            x.x = ptr[0];
            if (col + 1 < dim) x.y = ptr[1];
          }
        }
        S[j * 4 + e][0] = x.x;
        S[j * 4 + e][1] = x.y;
      }
    }
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// grid (heads, column tiles, sequences), 4 warps of (32 / kKL) column pairs.
template <typename T, int kKL>
__global__ void __launch_bounds__(kDrScanWarps * 32) delta_scan_kernel(const DeltaParams<T> p) {
  pdl_wait();
  pdl_trigger();
  constexpr int pad = kKL * kDrKeys;
  constexpr int kTok = kDrVecs * pad;                // floats per token
  extern __shared__ __align__(16) float buf[];       // [2][kDrChunk][kTok]
  const int h = blockIdx.x, s = blockIdx.z, D = p.dim;
  const int r0 = p.row_off[s], r1 = p.row_off[s + 1];
  if (r1 <= r0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % kKL;
  const int col = ((blockIdx.y * kDrScanWarps + warp) * (32 / kKL) + lane / kKL) * 2;
  float* st = p.state + static_cast<long long>(p.slots[s]) * p.slot_stride + static_cast<size_t>(h) * D * D;
  float S[kDrKeys][2];
  delta_state_io<kKL, false>(S, st, D, kl, col);
  const float* vec = p.vec + static_cast<size_t>(h) * p.tokens * kTok;
  const float* sums = p.sums + static_cast<size_t>(h) * p.tokens * 2;
  auto stage = [&](int c0, int b) {
    const int n = min(kDrChunk, r1 - c0) * (kTok / 4);
    for (int e = threadIdx.x; e < n; e += kDrScanWarps * 32)
      cp_async16(buf + b * kDrChunk * kTok + e * 4, vec + static_cast<size_t>(c0) * kTok + e * 4);
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
      const float* vs = buf + (b * kDrChunk + i) * kTok;
      const float2 s12 = *reinterpret_cast<const float2*>(sums + static_cast<size_t>(c0 + i) * 2);
      float v[2] = {0.f, 0.f}, o[2];
      if (col < pad) { v[0] = vs[5 * pad + col]; v[1] = vs[5 * pad + col + 1]; }
      delta_token<kKL>(S, vs, kl, v, s12.x, s12.y, o);
      if (kl == 0) {
        float* dst = p.o_raw + static_cast<size_t>(c0 + i) * p.heads * D + h * D + col;
        if (col < D) dst[0] = o[0];
        if (col + 1 < D) dst[1] = o[1];
      }
    }
    __syncthreads();                                 // the buffer is refilled by the next iteration's stage()
  }
  delta_state_io<kKL, true>(S, st, D, kl, col);
}

// grid (tokens, heads), block = padded head size (at least 32).
template <typename T>
__global__ void delta_post_kernel(const DeltaParams<T> p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[16];
  const int t = blockIdx.x, h = blockIdx.y, d = threadIdx.x, D = p.dim, warps = blockDim.x >> 5;
  const int c = h * D + d;
  const size_t idx = static_cast<size_t>(t) * p.heads * D + c;
  const float o = d < D ? p.o_raw[idx] : 0.f;
  const float ss = block_sum(o * o, red, warps);
  if (d < D) {
    const float g = ld_f(p.proj + static_cast<size_t>(t) * p.ldp + p.off_g + c);
    st_f(p.out + idx, o * (1.f / sqrtf(ss / static_cast<float>(D) + p.eps)) * p.norm_w[c] * sigmoid_f(g));
  }
}

// ---------------------------------------------------------------- decode form: exactly one row per sequence
// grid (heads, sequences), 256 threads; warps sweep the head's column tiles.
template <typename T, int kKL>
__global__ void __launch_bounds__(kDrDecodeThreads) delta_decode_kernel(const DeltaParams<T> p) {
  pdl_wait();
  pdl_trigger();
  constexpr int pad = kKL * kDrKeys;
  constexpr int kWarps = kDrDecodeThreads / 32;
  __shared__ __align__(16) float vs[kDrVecs * pad];
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
  delta_state_io<kKL, false>(S, st, D, kl, col);
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
    vs[pad + d] = w * r; vs[2 * pad + d] = w; vs[3 * pad + d] = a; vs[4 * pad + d] = k; vs[5 * pad + d] = v;
    vs[d] = r;
    kk += k * k;
    kr += k * r;
  }
  kk = block_sum(kk, red, kWarps);
  const float s2 = block_sum(kr, red, kWarps);
  const float inv_u = 1.f / sqrtf(kk + p.eps_u);
  float s1 = 0.f;
  for (int d = threadIdx.x; d < pad; d += kDrDecodeThreads) {   // each thread rewrites only what it wrote above
    const float r = vs[d], u = vs[4 * pad + d] * inv_u, au = vs[3 * pad + d] * u;
    s1 += au * r;
    vs[d] = u;
    vs[3 * pad + d] = au;
  }
  s1 = block_sum(s1, red, kWarps);                   // its barriers also publish vs
  constexpr int kSweep = kWarps * (32 / kKL) * 2;    // columns per sweep of the CTA
  for (int base = 0; base < D; base += kSweep) {
    if (base > 0) {
      col += kSweep;
      delta_state_io<kKL, false>(S, st, D, kl, col);
    }
    float v[2] = {0.f, 0.f}, o[2];
    if (col < pad) { v[0] = vs[5 * pad + col]; v[1] = vs[5 * pad + col + 1]; }
    delta_token<kKL>(S, vs, kl, v, s1, s2, o);
    delta_state_io<kKL, true>(S, st, D, kl, col);
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

template <typename T, int kKL>
static int delta_scan_launch(const DeltaParams<T>& p, int sequences, cudaStream_t st) {
  constexpr size_t smem = sizeof(float) * 2 * kDrChunk * kDrVecs * kKL * kDrKeys;
  static bool cfg = false;
  if (!cfg && smem > 48 * 1024) {
    if (cudaFuncSetAttribute(delta_scan_kernel<T, kKL>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
      return SLLM_ERR_CUDA;
    cfg = true;
  }
  constexpr int cols = kDrScanWarps * (32 / kKL) * 2;
  return launch_kernel(delta_scan_kernel<T, kKL>, dim3(p.heads, (p.dim + cols - 1) / cols, sequences), dim3(kDrScanWarps * 32), smem,
                       st, 1u, p) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

template <typename T>
static int delta_prompt_launch(DeltaParams<T> p, int sequences, cudaStream_t st) {
  const int pad = delta_pad(p.dim), block = pad < 32 ? 32 : pad;
  if (launch_kernel(delta_pre_kernel<T>, dim3(p.tokens, p.heads), dim3(block), 0, st, 1u, p) != cudaSuccess) return SLLM_ERR_CUDA;
  int rc;
  switch (pad / kDrKeys) {
    case 1: rc = delta_scan_launch<T, 1>(p, sequences, st); break;
    case 2: rc = delta_scan_launch<T, 2>(p, sequences, st); break;
    case 4: rc = delta_scan_launch<T, 4>(p, sequences, st); break;
    case 8: rc = delta_scan_launch<T, 8>(p, sequences, st); break;
    case 16: rc = delta_scan_launch<T, 16>(p, sequences, st); break;
    default: rc = delta_scan_launch<T, 32>(p, sequences, st); break;
  }
  if (rc != SLLM_OK) return rc;
  return launch_kernel(delta_post_kernel<T>, dim3(p.tokens, p.heads), dim3(block), 0, st, 1u, p) == cudaSuccess ? SLLM_OK
                                                                                                              : SLLM_ERR_CUDA;
}

template <typename T>
static int delta_decode_launch(const DeltaParams<T>& p, int sequences, cudaStream_t st) {
  const dim3 grid(p.heads, sequences), block(kDrDecodeThreads);
  const size_t smem = sizeof(float) * p.rank;
  cudaError_t e;
  switch (delta_pad(p.dim) / kDrKeys) {
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
  float* scratch;          // prompt form: heads * tokens * (6 * pad + 2) + tokens * heads * dim floats, 16-byte aligned
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
  const int pad = delta_pad(a->dim);
  const long long nv = static_cast<long long>(a->heads) * a->tokens * kDrVecs * pad, ns = static_cast<long long>(a->heads) * a->tokens * 2;
  const long long no = static_cast<long long>(a->tokens) * a->heads * a->dim;
  if (a->decode) {
    if (!a->w2 || a->rank <= 0 || a->ld_w2 < a->rank || a->rank > 8192) return SLLM_ERR_INVALID_ARGUMENT;
  } else {
    if (!a->decay || !a->scratch) return SLLM_ERR_INVALID_ARGUMENT;
    if (a->scratch_floats < nv + ns + no) return SLLM_ERR_WORKSPACE_TOO_SMALL;
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
    p.vec = a->scratch; p.sums = a->scratch + nv; p.o_raw = p.sums + ns;
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
