// Linear attention with a matrix-valued state per head, S [dim keys, vdim values] in fp32, in four forms:
//   gated linear    S <- diag(g_t) S + k v^T,  g = sigmoid(z + bias)^(1 / tau),  z a low-rank product of the input
//   fixed decay     S <- g_h S + k v^T  (retention)
//   channel delta   S <- diag(g_t) S;  S <- S + k (beta (v - S^T k))^T,  g = exp(-rate_h softplus(z + bias)); q, k and v pass a
//                   short causal convolution and SiLU, q and k become unit vectors, beta = sigmoid(b); a head uses the query and
//                   key of its group
//   head delta      the same with one decay per head, g = exp(-rate_h softplus(a + bias_h)), a a column of the projection
// then o = S^T q, o / rms(o) (* norm weight) and the output gate: SiLU of a projection, in the channel form the sigmoid of a
// low-rank product.  q and k are scaled as given.  With u = g k and beta v for v the channel form is the removal step of
// state_scan.cuh; the first two are that step without its removal term, the last has a step of its own.
//
// The batch is flat (rows of sequence s: row_off[s] .. row_off[s + 1]) and sequence s owns state slot slots[s].
// Prompts: linear_pre_kernel computes everything that does not depend on the state in parallel over the tokens, the scan of
// state_scan.cu runs the recurrence, linear_post_kernel normalises and gates; the two low-rank products' second factors are
// GEMMs of the caller.  One-token batches (decode) take linear_decode_kernel, which does all of it in one launch.
#include <cstddef>
#include <type_traits>
#include "state_scan.cuh"
#include "state_scan.h"
#include "short_conv.h"
#include "api.h"

namespace sllm {

enum StateForm { kGatedLinear = 0, kFixedDecay = 1, kChannelDelta = 2, kHeadDelta = 3 };

__host__ __device__ constexpr bool form_delta(int form) { return form == kChannelDelta || form == kHeadDelta; }   // convolutions, unit keys
__host__ __device__ constexpr bool form_low_decay(int form) { return form == kGatedLinear || form == kChannelDelta; }   // low-rank decay
__host__ __device__ constexpr int form_step(int form) { return form == kHeadDelta ? kGatedDelta : form == kChannelDelta ? kRemoval : kPlain; }

constexpr int kLsRowWarps = 8;       // (token, head) pairs per CTA of the row kernels
constexpr int kLsDecodeThreads = 256;

template <typename T>
struct LinearStateParams {
  const T* proj;             // [tokens, ldp], columns off_*: q | k | v (consecutive in the delta forms), output gate (its low-rank input
  int ldp, off_q, off_k, off_v, off_g, off_a, off_b;   // in the channel form), decay (its low-rank input), write strengths
  const float* decay;        // prompt form: [tokens, ld_decay] second product of the decay, without bias
  int ld_decay;
  const T* gate;             // prompt form, channel delta: [tokens, ld_gate] second product of the gate
  int ld_gate;
  const T *w_a, *w_g;        // decode form: [heads * dim, ld_wa], [heads * vdim, ld_wg]; columns past the rank are zero
  int ld_wa, ld_wg, rank_a, rank_g;
  const float* bias;         // [heads * dim], in the head form [heads]
  const float* rate;         // [heads]: decay (fixed form), rate (delta forms)
  const float* conv_w;       // [taps, channels], last row: the current token
  float* ring;               // slot s at s * ring_stride: [taps][channels]
  long long ring_stride;
  int taps;
  const float* norm_w;       // optional [vdim]
  float inv_tau, q_scale, k_scale, unit_eps, eps;
  float* state;              // slot s, head h at state + s * slot_stride + h * dim * vdim
  long long slot_stride;
  const int *row_off, *slots, *positions, *seq_index;
  int heads, kv_heads, dim, vdim, tokens;
  float* vec;                // records of the scan
  float* o_raw;              // [tokens, heads * vdim]
  T* out;                    // [tokens, heads * vdim]
};

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float silu_f(float x) { return x * sigmoid_f(x); }

template <int kForm>
__device__ __forceinline__ float channel_decay(float z, float rate, float inv_tau) {
  if constexpr (kForm == kGatedLinear) return expf(-softplus_f(-z) * inv_tau);
  else if constexpr (kForm == kChannelDelta) return expf(-rate * softplus_f(z));
  else return rate;
}

// ---------------------------------------------------------------- prompt form
// SiLU of the convolution over a lane's channels: `col` their first column of proj's q | k | v and of the filter.
template <typename T, int kN>
__device__ __forceinline__ void conv_lane(const LinearStateParams<T>& p, int t, int pos, int first, const float* ring, int channels, int col,
                                          int d0, int width, bool vec, float (&y)[kN]) {
  float acc[kN];
#pragma unroll
  for (int i = 0; i < kN; ++i) acc[i] = 0.f;
  for (int b = 0; b < p.taps; ++b) {
    if (pos - b < 0) break;
    float x[kN], w[kN];
    if (t - b >= first) lane_load<T, kN>(p.proj + static_cast<size_t>(t - b) * p.ldp + p.off_q + col, d0, width, vec, x);
    else lane_load<float, kN>(ring + static_cast<size_t>((pos - b) % p.taps) * channels + col, d0, width, vec, x);
    lane_load<float, kN>(p.conv_w + static_cast<size_t>(p.taps - 1 - b) * channels + col, d0, width, vec, w);
#pragma unroll
    for (int i = 0; i < kN; ++i) acc[i] = fmaf(w[i], x[i], acc[i]);
  }
#pragma unroll
  for (int i = 0; i < kN; ++i) y[i] = silu_f(acc[i]);
}

// A warp per (token, head), lane l the channels l kN .. l kN + kN - 1 of its keys and of its values.  No early trigger of the
// dependent launch: the scan's few CTAs would become resident while this grid drains and share the first empty SMs.
template <typename T, int kN, int kForm>
__global__ void __launch_bounds__(kLsRowWarps * 32) linear_pre_kernel(const LinearStateParams<T> p, bool vec) {
  pdl_wait();
  constexpr bool kDelta = form_delta(kForm);
  constexpr int kStep = form_step(kForm);
  const int lane = threadIdx.x & 31, D = p.dim, V = p.vdim, pad = state_pad(D), d0 = lane * kN;
  const long long unit = static_cast<long long>(blockIdx.x) * kLsRowWarps + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(p.tokens) * p.heads) return;
  const int t = static_cast<int>(unit / p.heads), h = static_cast<int>(unit % p.heads), kvh = h / (p.heads / p.kv_heads);
  const T* row = p.proj + static_cast<size_t>(t) * p.ldp;
  float q[kN], k[kN], v[kN], w[kN];
  float q_scale = p.q_scale, k_scale = p.k_scale, beta = 0.f;
  if constexpr (kDelta) {
    const int seq = p.seq_index[t], pos = p.positions[t], first = p.row_off[seq];
    const float* ring = p.ring + p.slots[seq] * p.ring_stride;
    const int channels = 2 * p.kv_heads * D + p.heads * V;
    conv_lane<T, kN>(p, t, pos, first, ring, channels, kvh * D, d0, D, vec, q);
    conv_lane<T, kN>(p, t, pos, first, ring, channels, (p.kv_heads + kvh) * D, d0, D, vec, k);
    conv_lane<T, kN>(p, t, pos, first, ring, channels, 2 * p.kv_heads * D + h * V, d0, V, vec, v);
    float qq = 0.f, kk = 0.f;
#pragma unroll
    for (int i = 0; i < kN; ++i) {
      qq += q[i] * q[i];
      kk += k[i] * k[i];
    }
    q_scale /= sqrtf(warp_sum(qq) + p.unit_eps);
    k_scale /= sqrtf(warp_sum(kk) + p.unit_eps);
    beta = sigmoid_f(ld_f(row + p.off_b + h));
  } else {
    lane_load<T, kN>(row + p.off_q + kvh * D, d0, D, vec, q);
    lane_load<T, kN>(row + p.off_k + kvh * D, d0, D, vec, k);
    lane_load<T, kN>(row + p.off_v + h * V, d0, V, vec, v);
  }
  const float rate = kForm == kGatedLinear ? 0.f : p.rate[h];
  if constexpr (form_low_decay(kForm)) {
    float b[kN];
    lane_load<float, kN>(p.decay + static_cast<size_t>(t) * p.ld_decay + h * D, d0, D, vec, w);
    lane_load<float, kN>(p.bias + h * D, d0, D, vec, b);
#pragma unroll
    for (int i = 0; i < kN; ++i) w[i] += b[i];
  }
  float kq = 0.f, u[kN], au[kN];
  float* dst = p.vec + (static_cast<size_t>(h) * p.tokens + t) * state_record(kStep, pad, V);
  if constexpr (kStep == kGatedDelta) {
#pragma unroll
    for (int i = 0; i < kN; ++i) {
      q[i] *= q_scale;
      k[i] *= k_scale;
      kq += k[i] * q[i];
      v[i] *= beta;
    }
    kq = warp_sum(kq);
    const float g = expf(-rate * softplus_f(ld_f(row + p.off_a + h) + p.bias[h]));
    lane_store(dst + kVecGQ * pad, d0, pad, q);
    lane_store(dst + kVecGK * pad, d0, pad, k);
    dst += state_vecs(kStep) * pad;
    lane_store(dst, d0, state_vpad(V), v);
    if (lane == 0) *reinterpret_cast<float4*>(dst + state_vpad(V)) = make_float4(g, beta * g, kq, 0.f);
  } else {
#pragma unroll
    for (int i = 0; i < kN; ++i) {
      w[i] = d0 + i < D ? channel_decay<kForm>(w[i], rate, p.inv_tau) : 0.f;
      q[i] *= q_scale;
      k[i] *= k_scale;
      kq += k[i] * q[i];
      q[i] *= w[i];
      u[i] = w[i] * k[i];
      au[i] = beta * k[i];
      if constexpr (kDelta) v[i] *= beta;
    }
    kq = warp_sum(kq);
    lane_store(dst + kVecWR * pad, d0, pad, q);
    lane_store(dst + kVecW * pad, d0, pad, w);
    lane_store(dst + kVecK * pad, d0, pad, k);
    if constexpr (kDelta) {
      lane_store(dst + kVecU * pad, d0, pad, u);
      lane_store(dst + kVecAU * pad, d0, pad, au);
    }
    dst += state_vecs(kStep) * pad;
    lane_store(dst, d0, state_vpad(V), v);
    if (lane == 0) *reinterpret_cast<float2*>(dst + state_vpad(V)) = make_float2(beta * kq, kq);
  }
}

// A warp per (token, head), as in the first stage.
template <typename T, int kN, int kForm>
__global__ void __launch_bounds__(kLsRowWarps * 32) linear_post_kernel(const LinearStateParams<T> p, bool vec) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, V = p.vdim, d0 = lane * kN;
  const long long unit = static_cast<long long>(blockIdx.x) * kLsRowWarps + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(p.tokens) * p.heads) return;
  const int t = static_cast<int>(unit / p.heads), h = static_cast<int>(unit % p.heads);
  const size_t idx = (static_cast<size_t>(t) * p.heads + h) * V;
  float o[kN], g[kN], w[kN];
  lane_load<float, kN>(p.o_raw + idx, d0, V, vec, o);
  if constexpr (kForm == kChannelDelta) lane_load<T, kN>(p.gate + static_cast<size_t>(t) * p.ld_gate + h * V, d0, V, vec, g);
  else lane_load<T, kN>(p.proj + static_cast<size_t>(t) * p.ldp + p.off_g + h * V, d0, V, vec, g);
#pragma unroll
  for (int i = 0; i < kN; ++i) w[i] = 1.f;
  if (p.norm_w) lane_load<float, kN>(p.norm_w, d0, V, vec, w);
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kN; ++i) ss += o[i] * o[i];
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(V) + p.eps);
#pragma unroll
  for (int i = 0; i < kN; ++i) o[i] = o[i] * inv * w[i] * (kForm == kChannelDelta ? sigmoid_f(g[i]) : silu_f(g[i]));
  T* dst = p.out + idx + d0;
  if constexpr (kN % 4 == 0) {
    if (vec) {
#pragma unroll
      for (int i = 0; i < kN; i += 4) {
        const float x[4] = {o[i], o[i + 1], o[i + 2], o[i + 3]};
        if (d0 + i < V) st_vec<4>(dst + i, x);
      }
      return;
    }
  }
#pragma unroll
  for (int i = 0; i < kN; ++i)
    if (d0 + i < V) st_f(dst + i, o[i]);
}

// ---------------------------------------------------------------- decode form: exactly one row per sequence
// Row `w` of a low-rank product's second factor times its input, ranks in shared memory (zero past the rank up to 8).
template <typename T>
__device__ __forceinline__ float low_rank_dot(const T* w, int ld, int rank, const float* low) {
  float x = 0.f;
  if (ld % kVec16<T> == 0) {
#pragma unroll 4
    for (int i = 0; i < rank; i += kVec16<T>) {
      float wv[kVec16<T>];
      ld16(w + i, wv);
#pragma unroll
      for (int j = 0; j < kVec16<T>; ++j) x = fmaf(wv[j], low[i + j], x);
    }
  } else {
    for (int i = 0; i < rank; ++i) x = fmaf(ld_f(w + i), low[i], x);
  }
  return x;
}

__host__ __device__ constexpr int rank_pad(int r) { return (r + 7) & ~7; }

// grid (heads, sequences), 256 threads; warps sweep the head's column tiles.
template <typename T, int kKL, int kForm>
__global__ void __launch_bounds__(kLsDecodeThreads, 2) linear_decode_kernel(const LinearStateParams<T> p) {
  pdl_wait();
  pdl_trigger();
  constexpr bool kDelta = form_delta(kForm);
  constexpr int kStep = form_step(kForm), pad = kKL * kDrKeys, nv = state_vecs(kStep), kWarps = kLsDecodeThreads / 32;
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[3][kWarps];
  const int h = blockIdx.x, s = blockIdx.y, D = p.dim, V = p.vdim, vpad = state_vpad(V), t = p.row_off[s];
  if (p.row_off[s + 1] <= t) return;
  float* vs = sm;                                    // [nv][pad], then v [vpad]
  float* o_s = vs + nv * pad + vpad;                 // [vpad]
  float* gate = o_s + vpad;                          // [vpad]
  float* low_a = gate + vpad;                        // [rank_a padded]
  float* low_g = low_a + rank_pad(p.rank_a);         // [rank_g padded]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % kKL, kvh = h / (p.heads / p.kv_heads);
  const T* row = p.proj + static_cast<size_t>(t) * p.ldp;
  float* st = p.state + static_cast<long long>(p.slots[s]) * p.slot_stride + static_cast<size_t>(h) * D * V;
  // the first tile of the state is requested before anything is computed
  int col = (warp * (32 / kKL) + lane / kKL) * 2;
  float S[kDrKeys][2];
  state_io<kKL, 2, false>(S, st, D, V, kl, col);
  if constexpr (form_low_decay(kForm)) {
    for (int i = threadIdx.x; i < rank_pad(p.rank_a); i += kLsDecodeThreads) low_a[i] = i < p.rank_a ? ld_f(row + p.off_a + i) : 0.f;
    if constexpr (kForm == kChannelDelta)
      for (int i = threadIdx.x; i < rank_pad(p.rank_g); i += kLsDecodeThreads) low_g[i] = i < p.rank_g ? ld_f(row + p.off_g + i) : 0.f;
    __syncthreads();
  }
  const float rate = kForm == kGatedLinear ? 0.f : p.rate[h];
  const int channels = 2 * p.kv_heads * D + p.heads * V, pos = kDelta ? p.positions[t] : 0;
  float* ring = kDelta ? p.ring + p.slots[s] * p.ring_stride : nullptr;
  // input of column c of q | k | v: in the delta forms SiLU of its convolution; `keep` stores it in the ring
  auto input = [&](int c, bool keep) {
    const float x = ld_f(row + p.off_q + c);
    float a = p.conv_w[static_cast<size_t>(p.taps - 1) * channels + c] * x;
    for (int b = 1; b < p.taps && pos - b >= 0; ++b)
      a = fmaf(p.conv_w[static_cast<size_t>(p.taps - 1 - b) * channels + c], ring[static_cast<size_t>((pos - b) % p.taps) * channels + c], a);
    if (keep) ring[static_cast<size_t>(pos % p.taps) * channels + c] = x;
    return silu_f(a);
  };
  float qq = 0.f, kk = 0.f, kq = 0.f;
  for (int e = threadIdx.x; e < pad + vpad; e += kLsDecodeThreads) {
    if (e < pad) {
      float q = 0.f, k = 0.f, w = 0.f;
      if (e < D) {
        if constexpr (kDelta) {
          const bool keep = h % (p.heads / p.kv_heads) == 0;   // one head of a group stores the group's rows
          q = input(kvh * D + e, keep);
          k = input((p.kv_heads + kvh) * D + e, keep);
        } else {
          q = ld_f(row + p.off_q + kvh * D + e);
          k = ld_f(row + p.off_k + kvh * D + e);
        }
        if constexpr (form_low_decay(kForm))
          w = low_rank_dot(p.w_a + static_cast<size_t>(h * D + e) * p.ld_wa, p.ld_wa, p.rank_a, low_a) + p.bias[h * D + e];
        if constexpr (kForm != kHeadDelta) w = channel_decay<kForm>(w, rate, p.inv_tau);
      }
      if constexpr (kStep == kGatedDelta) {
        vs[kVecGQ * pad + e] = q;
        vs[kVecGK * pad + e] = k;
      } else {
        vs[kVecWR * pad + e] = q;
        vs[kVecW * pad + e] = w;
        vs[kVecK * pad + e] = k;
      }
      qq += q * q;
      kk += k * k;
      kq += k * q;
    } else {
      const int d = e - pad;
      float v = 0.f, g = 0.f;
      if (d < V) {
        if constexpr (kDelta) {
          v = input(2 * p.kv_heads * D + h * V + d, true);
          if constexpr (kForm == kHeadDelta) g = silu_f(ld_f(row + p.off_g + h * V + d));
          else g = sigmoid_f(low_rank_dot(p.w_g + static_cast<size_t>(h * V + d) * p.ld_wg, p.ld_wg, p.rank_g, low_g));
        } else {
          v = ld_f(row + p.off_v + h * V + d);
          g = silu_f(ld_f(row + p.off_g + h * V + d));
        }
      }
      vs[nv * pad + d] = v;
      gate[d] = g;
    }
  }
  qq = warp_sum(qq);
  kk = warp_sum(kk);
  kq = warp_sum(kq);
  if (lane == 0) {
    red[0][warp] = qq;
    red[1][warp] = kk;
    red[2][warp] = kq;
  }
  __syncthreads();
  qq = kk = kq = 0.f;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) {
    qq += red[0][i];
    kk += red[1][i];
    kq += red[2][i];
  }
  const float beta = kDelta ? sigmoid_f(ld_f(row + p.off_b + h)) : 0.f;
  const float qs = kDelta ? p.q_scale / sqrtf(qq + p.unit_eps) : p.q_scale, ks = kDelta ? p.k_scale / sqrtf(kk + p.unit_eps) : p.k_scale;
  kq *= qs * ks;
  float4 sc = make_float4(beta * kq, kq, 0.f, 0.f);
  if constexpr (kStep == kGatedDelta) {
    const float g = expf(-rate * softplus_f(ld_f(row + p.off_a + h) + p.bias[h]));
    sc = make_float4(g, beta * g, kq, 0.f);
  }
  for (int e = threadIdx.x; e < pad + vpad; e += kLsDecodeThreads) {   // each thread rewrites only what it wrote above
    if (kStep == kGatedDelta && e < pad) {
      vs[kVecGQ * pad + e] *= qs;
      vs[kVecGK * pad + e] *= ks;
    } else if (e < pad) {
      const float w = vs[kVecW * pad + e], k = vs[kVecK * pad + e] * ks;
      vs[kVecWR * pad + e] *= w * qs;
      vs[kVecK * pad + e] = k;
      if constexpr (kDelta) {
        vs[kVecU * pad + e] = w * k;
        vs[kVecAU * pad + e] = beta * k;
      }
    } else if (kDelta) {
      vs[nv * pad + e - pad] *= beta;
    }
  }
  __syncthreads();
  constexpr int kSweep = kWarps * (32 / kKL) * 2;    // columns per sweep of the CTA
  for (int base = 0; base < V; base += kSweep) {
    if (base > 0) {
      col += kSweep;
      state_io<kKL, 2, false>(S, st, D, V, kl, col);
    }
    float v[2] = {0.f, 0.f}, o[2];
    if (col < vpad) { v[0] = vs[nv * pad + col]; v[1] = vs[nv * pad + col + 1]; }
    state_token<kKL, 2, kStep>(S, vs, kl, v, sc, o);
    state_io<kKL, 2, true>(S, st, D, V, kl, col);
    if (kl == 0 && col < vpad) { o_s[col] = o[0]; o_s[col + 1] = o[1]; }
  }
  __syncthreads();
  float ss = 0.f;
  for (int d = threadIdx.x; d < V; d += kLsDecodeThreads) ss += o_s[d] * o_s[d];
  ss = block_sum(ss, red[0], kWarps);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(V) + p.eps);
  for (int d = threadIdx.x; d < V; d += kLsDecodeThreads)
    st_f(p.out + (static_cast<size_t>(t) * p.heads + h) * V + d, o_s[d] * inv * (p.norm_w ? p.norm_w[d] : 1.f) * gate[d]);
}

// ---------------------------------------------------------------- launches
template <typename T, int kN, int kForm>
static cudaError_t linear_rows_launch(const LinearStateParams<T>& p, bool pre, bool vec, cudaStream_t st) {
  const long long units = static_cast<long long>(p.tokens) * p.heads;
  const dim3 grid(static_cast<unsigned>((units + kLsRowWarps - 1) / kLsRowWarps));
  return launch_kernel(pre ? linear_pre_kernel<T, kN, kForm> : linear_post_kernel<T, kN, kForm>, grid, dim3(kLsRowWarps * 32), 0, st, 1u, p,
                       vec);
}

template <typename T, int kForm>
static cudaError_t linear_rows(const LinearStateParams<T>& p, bool pre, bool vec, cudaStream_t st) {
  const int pd = state_pad(p.dim), pv = state_pad(p.vdim), wide = pre && pd > pv ? pd : pv;
  switch (wide / 32) {
    case 0: case 1: return linear_rows_launch<T, 1, kForm>(p, pre, vec, st);
    case 2: return linear_rows_launch<T, 2, kForm>(p, pre, vec, st);
    case 4: return linear_rows_launch<T, 4, kForm>(p, pre, vec, st);
    case 8: return linear_rows_launch<T, 8, kForm>(p, pre, vec, st);
    default: return linear_rows_launch<T, 16, kForm>(p, pre, vec, st);
  }
}

template <typename T, int kKL, int kForm>
static cudaError_t linear_decode_go(const LinearStateParams<T>& p, int sequences, cudaStream_t st) {
  const size_t smem = sizeof(float) * (state_vecs(form_step(kForm)) * kKL * kDrKeys + 3 * state_vpad(p.vdim) + rank_pad(p.rank_a) +
                                       rank_pad(p.rank_g));
  return launch_kernel(linear_decode_kernel<T, kKL, kForm>, dim3(p.heads, sequences), dim3(kLsDecodeThreads), smem, st, 1u, p);
}

template <typename T, int kForm>
static int linear_form(LinearStateParams<T> p, int decode, int sequences, bool vec, cudaStream_t st) {
  if (decode) {
    cudaError_t e;
    switch (state_pad(p.dim) / kDrKeys) {
      case 1: e = linear_decode_go<T, 1, kForm>(p, sequences, st); break;
      case 2: e = linear_decode_go<T, 2, kForm>(p, sequences, st); break;
      case 4: e = linear_decode_go<T, 4, kForm>(p, sequences, st); break;
      case 8: e = linear_decode_go<T, 8, kForm>(p, sequences, st); break;
      case 16: e = linear_decode_go<T, 16, kForm>(p, sequences, st); break;
      default: e = linear_decode_go<T, 32, kForm>(p, sequences, st); break;
    }
    return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
  }
  constexpr bool kDelta = form_delta(kForm);
  if (linear_rows<T, kForm>(p, true, vec, st) != cudaSuccess) return SLLM_ERR_CUDA;
  if (kDelta && p.taps > 1 &&
      conv_ring_launch(p.proj + p.off_q, p.ldp, std::is_same_v<T, float>, p.ring, p.ring_stride, p.row_off, p.slots, p.positions,
                       2 * p.kv_heads * p.dim + p.heads * p.vdim, p.taps, sequences, st) != cudaSuccess)
    return SLLM_ERR_CUDA;
  const ScanParams sp{p.vec, p.state, p.slot_stride, p.row_off, p.slots, p.o_raw, p.heads, p.dim, p.vdim, p.tokens};
  const int rc = state_scan_launch(sp, form_step(kForm), sequences, st);
  if (rc != SLLM_OK) return rc;
  return linear_rows<T, kForm>(p, false, vec, st) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

}  // namespace sllm

using namespace sllm;

struct SllmLinearState {   // host-side mirror passed by the Python layer (ctypes.Structure)
  const void *proj, *decay, *gate, *w_a, *w_g, *bias, *rate, *conv_w, *ring, *norm_w, *state, *row_off, *slots, *positions, *seq_index,
      *scratch, *out;      // scratch, prompt form: sllm_linear_state_floats floats, 16-byte aligned
  long long ring_stride, slot_stride, scratch_floats;
  int form, ldp, off_q, off_k, off_v, off_g, off_a, off_b, ld_decay, ld_gate, ld_wa, ld_wg, rank_a, rank_g, taps, heads, kv_heads, dim, vdim,
      tokens, sequences, fp32, decode;
  float inv_tau, q_scale, k_scale, unit_eps, eps;
};

SLLM_EXPORT int sllm_linear_state_abi(int* out, int n) {
  const int v[2] = {static_cast<int>(sizeof(SllmLinearState)), static_cast<int>(offsetof(SllmLinearState, eps))};
  for (int i = 0; i < n && i < 2; ++i) out[i] = v[i];
  return 2;
}

// Scratch of the prompt form.
SLLM_EXPORT long long sllm_linear_state_floats(int form, int heads, int dim, int vdim, int tokens) {
  return static_cast<long long>(heads) * tokens * (state_record(form_step(form), state_pad(dim), vdim) + vdim);
}

// decode = 1: exactly one row per sequence (w_a, w_g used); 0: any rows (decay, gate and scratch used).
SLLM_EXPORT int sllm_linear_state(const SllmLinearState* a, void* stream) {
  if (!a || !a->proj || !a->state || !a->row_off || !a->slots || !a->out || a->form < kGatedLinear || a->form > kHeadDelta ||
      a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 || a->tokens <= 0 || a->sequences <= 0 ||
      a->heads > 65535 || a->sequences > 65535 || a->rank_a < 0 || a->rank_g < 0)
    return SLLM_ERR_INVALID_ARGUMENT;
  const bool delta = form_delta(a->form), low = form_low_decay(a->form), low_gate = a->form == kChannelDelta;
  if ((a->form != kGatedLinear && !a->rate) || (low && (!a->bias || a->rank_a <= 0)) || (a->form == kHeadDelta && !a->bias) ||
      (low_gate && a->rank_g <= 0) ||
      (delta && (!a->conv_w || !a->ring || a->taps < 1 || !a->positions || !a->seq_index ||
                 a->off_k != a->off_q + a->kv_heads * a->dim || a->off_v != a->off_k + a->kv_heads * a->dim)))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->dim > 512 || a->vdim > 512 || a->rank_a > 2048 || a->rank_g > 2048) return SLLM_ERR_UNSUPPORTED_SHAPE;
  if (a->decode) {
    if ((low && (!a->w_a || a->ld_wa < a->rank_a)) || (low_gate && (!a->w_g || a->ld_wg < a->rank_g)) || a->tokens != a->sequences)
      return SLLM_ERR_INVALID_ARGUMENT;
  } else {
    if ((low && !a->decay) || (low_gate && !a->gate) || !a->scratch) return SLLM_ERR_INVALID_ARGUMENT;
    if (a->scratch_floats < sllm_linear_state_floats(a->form, a->heads, a->dim, a->vdim, a->tokens)) return SLLM_ERR_WORKSPACE_TOO_SMALL;
    if (reinterpret_cast<uintptr_t>(a->scratch) & 15) return SLLM_ERR_ALIGNMENT;
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int odd = a->dim | a->vdim | a->ldp | a->off_q | a->off_k | a->off_v | a->off_g | (low ? a->ld_decay : 0) | (low_gate ? a->ld_gate : 0);
  if (delta) odd |= static_cast<int>(a->ring_stride & 3);
  const bool vec = (odd & 3) == 0;
  auto run = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    auto t = [](const void* x) { return static_cast<T*>(const_cast<void*>(x)); };
    auto f = [](const void* x) { return static_cast<float*>(const_cast<void*>(x)); };
    auto n = [](const void* x) { return static_cast<const int*>(x); };
    LinearStateParams<T> p = {};
    p.proj = t(a->proj); p.ldp = a->ldp; p.off_q = a->off_q; p.off_k = a->off_k; p.off_v = a->off_v; p.off_g = a->off_g; p.off_a = a->off_a;
    p.off_b = a->off_b; p.decay = f(a->decay); p.ld_decay = a->ld_decay; p.gate = t(a->gate); p.ld_gate = a->ld_gate; p.w_a = t(a->w_a);
    p.w_g = t(a->w_g); p.ld_wa = a->ld_wa; p.ld_wg = a->ld_wg; p.rank_a = low ? a->rank_a : 0; p.rank_g = low_gate ? a->rank_g : 0;
    p.bias = f(a->bias); p.rate = f(a->rate); p.conv_w = f(a->conv_w); p.ring = f(a->ring); p.ring_stride = a->ring_stride; p.taps = a->taps;
    p.norm_w = f(a->norm_w); p.inv_tau = a->inv_tau; p.q_scale = a->q_scale; p.k_scale = a->k_scale; p.unit_eps = a->unit_eps; p.eps = a->eps;
    p.state = f(a->state); p.slot_stride = a->slot_stride; p.row_off = n(a->row_off); p.slots = n(a->slots); p.positions = n(a->positions);
    p.seq_index = n(a->seq_index); p.heads = a->heads; p.kv_heads = a->kv_heads; p.dim = a->dim; p.vdim = a->vdim; p.tokens = a->tokens;
    p.out = t(a->out); p.vec = f(a->scratch);
    if (!a->decode)
      p.o_raw = p.vec + static_cast<long long>(a->heads) * a->tokens * state_record(form_step(a->form), state_pad(a->dim), a->vdim);
    if (a->form == kGatedLinear) return linear_form<T, kGatedLinear>(p, a->decode, a->sequences, vec, st);
    if (a->form == kFixedDecay) return linear_form<T, kFixedDecay>(p, a->decode, a->sequences, vec, st);
    if (a->form == kHeadDelta) return linear_form<T, kHeadDelta>(p, a->decode, a->sequences, vec, st);
    return linear_form<T, kChannelDelta>(p, a->decode, a->sequences, vec, st);
  };
  return a->fp32 ? run(static_cast<float*>(nullptr)) : run(static_cast<__nv_bfloat16*>(nullptr));
}
