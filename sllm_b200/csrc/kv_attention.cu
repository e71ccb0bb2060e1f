// Attention over paged keys and values whose widths differ (dim, vdim), with the work between the input projection and the
// scores in one launch.
//
//   kv_prepare_kernel   per (token, head): bias or short causal convolution of the q / k / v columns, optional RMS norm of
//                       q and k (per head or over all heads, weighted or not) and of v, values mixed with another layer's,
//                       rotation of the first channels in pairs (2i, 2i+1) or (i, i + half), page write of k and v; q goes to
//                       [T, heads, q_pad].  In a decode step the kernel also stores the conv inputs; short_conv.cu has the
//                       prompt form of that store
//   kv_gather_kernel    pages -> contiguous [context rows, all heads' keys | all heads' values] for the tensor-core prompt
//                       kernel (latent_prefill.cu)
//   kv_attention_kernel any sizes, bf16 or fp32: one warp per (row, query head); sinks, windows with kept first tokens,
//                       chunks, distance slopes, distance biases and output gate
//
// Pages of a layer: keys [num_pages, kv_heads, page, ld_k], values [num_pages, kv_heads, page, ld_v].
#include "typed.cuh"
#include "api.h"
#include "attention_common.cuh"
#include "short_conv.h"

#include <cstddef>
#include <type_traits>

namespace sllm {

constexpr int kKpThreads = 256, kKpRun = 8;

template <typename T>
struct KvPrepareParams {
  const T* proj;             // [T, ldp]: q | k | v columns from 0
  const float* conv_w;       // [taps, channels], null: no convolution
  const float* bias;         // optional [channels], joins the columns first
  const float *q_norm, *k_norm;   // optional weights of the norms: [dim], over all heads [heads * dim], [kv_heads * dim]
  const T* v_other;          // optional [T, ld_other]: values that v is mixed with, v <- (1 - v_mix) v + v_mix v_other
  float v_mix;
  int ld_other, v_norm;
  float* ring;               // [slots (ring_stride)][taps][channels]
  const float* inv_freq;     // [rot_dims / 2]
  const int *row_off, *slots, *positions, *seq_index, *block_table;
  T *q, *k_pages, *v_pages;
  long long ring_stride;
  int ldp, max_blocks, heads, kv_heads, dim, vdim, q_pad, ld_k, ld_v, rot_dims, taps, page_size, tokens, run, norm, decode,
      interleaved;
  float eps;
};

enum KvNorm { kNormNone = 0, kNormHead = 1, kNormAll = 2 };   // of q and k: per head, over all heads at once

// kNP: channel pairs per lane; kTaps: filter length after padding; kVec: every pair is one aligned access.  grid (ceil(T / run), <= ceil(all heads / 8)); a warp takes
// every (8 gridDim.y)-th head.
template <typename T, int kNP, int kTaps, bool kVec>
__global__ void __launch_bounds__(kKpThreads) kv_prepare_kernel(const KvPrepareParams<T> p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float2 cs[];                        // [run][rot_dims / 2]
  __shared__ __align__(8) float swap_s[8][kNP * 64];    // a warp's head, where rotary pairs lie in different lanes
  __shared__ float part[2][8], inv_all[2][kKpRun];      // norms over all heads: sums of squares, 1 / rms of q and k
  __shared__ int m_pos[kKpRun], m_seq[kKpRun], m_first[kKpRun], m_slot[kKpRun], m_page[kKpRun];
  const int r0 = blockIdx.x * p.run, n = min(p.run, p.tokens - r0), half = p.rot_dims >> 1;
  if (threadIdx.x < n) {
    const int row = r0 + threadIdx.x, seq = p.seq_index[row], pos = p.positions[row];
    m_pos[threadIdx.x] = pos;
    m_seq[threadIdx.x] = seq;
    m_first[threadIdx.x] = p.decode ? row : p.row_off[seq];
    m_slot[threadIdx.x] = p.slots[seq];
    m_page[threadIdx.x] = p.kv_heads > 0 ? p.block_table[static_cast<size_t>(seq) * p.max_blocks + pos / p.page_size] : 0;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < n * half; e += kKpThreads) {
    float sn, c;
    sincosf(static_cast<float>(m_pos[e / half]) * p.inv_freq[e % half], &sn, &c);
    cs[e] = make_float2(c, sn);
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, all = p.heads + 2 * p.kv_heads;
  if (p.norm == kNormAll) {                             // 8 / run warps share a token
    const int parts = 8 / p.run, i = warp / parts, pt = warp % parts;
    float ss[2] = {0.f, 0.f};
    if (i < n) {
      const T* src = p.proj + static_cast<size_t>(r0 + i) * p.ldp;
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const int c0 = m ? p.heads * p.dim : 0, c1 = c0 + (m ? p.kv_heads : p.heads) * p.dim;
        if constexpr (kVec) {
#pragma unroll 4
          for (int c = c0 + 2 * (pt * 32 + lane); c < c1; c += 64 * parts) {
            float x[2];
            ld_vec<2>(src + c, x);
            if (p.bias) {
              x[0] += p.bias[c];
              x[1] += p.bias[c + 1];
            }
            ss[m] += x[0] * x[0] + x[1] * x[1];
          }
        } else {
          for (int c = c0 + pt * 32 + lane; c < c1; c += 32 * parts) {
            const float x = ld_f(src + c) + (p.bias ? p.bias[c] : 0.f);
            ss[m] += x * x;
          }
        }
      }
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      ss[m] = warp_sum(ss[m]);
      if (lane == 0) part[m][warp] = ss[m];
    }
    __syncthreads();
    if (threadIdx.x < 2 * n) {
      const int m = threadIdx.x / n, t = threadIdx.x % n;
      float s = 0.f;
      for (int j = 0; j < parts; ++j) s += part[m][t * parts + j];
      inv_all[m][t] = 1.f / sqrtf(s / static_cast<float>((m ? p.kv_heads : p.heads) * p.dim) + p.eps);
    }
    __syncthreads();
  }
  for (int head = blockIdx.y * 8 + warp; head < all; head += gridDim.y * 8) {
    const bool is_q = head < p.heads, is_v = head >= p.heads + p.kv_heads;
    const int kvh = is_v ? head - p.heads - p.kv_heads : head - p.heads;
    const int width = is_v ? p.vdim : p.dim;
    const int col = is_v ? (p.heads + p.kv_heads) * p.dim + kvh * p.vdim : head * p.dim;
    const int channels = (p.heads + p.kv_heads) * p.dim + p.kv_heads * p.vdim;
    auto ld2 = [&](const auto* src, int c, float (&v)[2]) {
      if constexpr (kVec) {
        v[0] = v[1] = 0.f;
        if (c < width) ld_vec<2>(src + c, v);
      } else {
        v[0] = c < width ? ld_f(src + c) : 0.f;
        v[1] = c + 1 < width ? ld_f(src + c + 1) : 0.f;
      }
    };
    auto st2 = [&](auto* dst, int c, int w, const float (&v)[2]) {
      if constexpr (kVec) {
        if (c < w) st_vec<2>(dst + c, v);
      } else {
        if (c < w) st_f(dst + c, v[0]);
        if (c + 1 < w) st_f(dst + c + 1, v[1]);
      }
    };
    float w[kTaps][kNP][2];
#pragma unroll
    for (int t = 0; t < kTaps; ++t)
#pragma unroll
      for (int s = 0; s < kNP; ++s) {
        w[t][s][0] = w[t][s][1] = 0.f;
        if (!p.conv_w) w[t][s][0] = w[t][s][1] = t == kTaps - 1 ? 1.f : 0.f;
        else if (t >= kTaps - p.taps)
          ld2(p.conv_w + static_cast<size_t>(t - (kTaps - p.taps)) * channels + col, 2 * (lane + 32 * s), w[t][s]);
      }
    float nw[kNP][2], bias[kNP][2];                       // norm weight and bias of the lane's channels
#pragma unroll
    for (int s = 0; s < kNP; ++s) {
      nw[s][0] = nw[s][1] = 1.f;
      bias[s][0] = bias[s][1] = 0.f;
      const float* src = is_v ? nullptr : is_q ? p.q_norm : p.k_norm;
      if (src && p.norm == kNormAll) src += (is_q ? head : kvh) * p.dim;
      if (src) ld2(src, 2 * (lane + 32 * s), nw[s]);
      if (p.bias) ld2(p.bias + col, 2 * (lane + 32 * s), bias[s]);
    }
    float win[kTaps > 1 ? kTaps - 1 : 1][kNP][2];         // win[b - 1]: the input b positions back
    // the next token's inputs are requested a token early, and kept as they come until they are used
    constexpr bool kAhead = kVec && kTaps == 1;
    using Pair = std::conditional_t<std::is_same_v<T, float>, float2, __nv_bfloat162>;
    Pair ahead[kNP];
    auto request = [&](const T* src) {
#pragma unroll
      for (int s = 0; s < kNP; ++s) {
        const int c = 2 * (lane + 32 * s);
        ahead[s] = c < width ? *reinterpret_cast<const Pair*>(src + c) : Pair();
      }
    };
    if constexpr (kAhead) request(p.proj + static_cast<size_t>(r0) * p.ldp + col);
    int prev = -1;
    for (int i = 0; i < n; ++i) {
      const int row = r0 + i, pos = m_pos[i], seq = m_seq[i];
      const T* src = p.proj + static_cast<size_t>(row) * p.ldp + col;
      float* ring = p.ring + m_slot[i] * p.ring_stride + col;
      if (seq != prev) {
#pragma unroll
        for (int b = 1; b < kTaps; ++b)
#pragma unroll
          for (int s = 0; s < kNP; ++s) {
            win[b - 1][s][0] = win[b - 1][s][1] = 0.f;
            if (b < p.taps && pos - b >= 0) {
              if (row - b >= m_first[i]) ld2(src - static_cast<size_t>(b) * p.ldp, 2 * (lane + 32 * s), win[b - 1][s]);
              else ld2(ring + static_cast<size_t>((pos - b) % p.taps) * channels, 2 * (lane + 32 * s), win[b - 1][s]);
            }
          }
        prev = seq;
      }
      float y[kNP][2];
      float ss = 0.f;
      Pair now[kNP];
      if constexpr (kAhead) {
#pragma unroll
        for (int s = 0; s < kNP; ++s) now[s] = ahead[s];
        if (i + 1 < n) request(src + p.ldp);
      }
#pragma unroll
      for (int s = 0; s < kNP; ++s) {
        const int c = 2 * (lane + 32 * s);
        float x[2];
        if constexpr (kAhead) {
          x[0] = static_cast<float>(now[s].x);
          x[1] = static_cast<float>(now[s].y);
        } else {
          ld2(src, c, x);
        }
        x[0] += bias[s][0];
        x[1] += bias[s][1];
        if (p.decode && p.ring) st2(ring + static_cast<size_t>(pos % p.taps) * channels, c, width, x);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          float a = w[kTaps - 1][s][j] * x[j];
#pragma unroll
          for (int b = 1; b < kTaps; ++b) a = fmaf(w[kTaps - 1 - b][s][j], win[b - 1][s][j], a);
          y[s][j] = a;
        }
        if constexpr (kTaps > 1) {
#pragma unroll
          for (int b = kTaps - 1; b > 1; --b)
#pragma unroll
            for (int j = 0; j < 2; ++j) win[b - 1][s][j] = win[b - 2][s][j];
#pragma unroll
          for (int j = 0; j < 2; ++j) win[0][s][j] = x[j];
        }
        ss += y[s][0] * y[s][0] + y[s][1] * y[s][1];
      }
      if (is_v ? p.v_norm : p.norm) {                     // (an unweighted norm and the rotation commute)
        const float inv = !is_v && p.norm == kNormAll ? inv_all[is_q ? 0 : 1][i]
                                                      : 1.f / sqrtf(warp_sum(ss) / static_cast<float>(width) + p.eps);
#pragma unroll
        for (int s = 0; s < kNP; ++s) {
          y[s][0] *= inv * nw[s][0];
          y[s][1] *= inv * nw[s][1];
        }
      }
      if (is_v && p.v_other) {
        const T* other = p.v_other + static_cast<size_t>(row) * p.ld_other + kvh * p.vdim;
#pragma unroll
        for (int s = 0; s < kNP; ++s) {
          float x[2];
          ld2(other, 2 * (lane + 32 * s), x);
#pragma unroll
          for (int j = 0; j < 2; ++j) y[s][j] = (1.f - p.v_mix) * y[s][j] + p.v_mix * x[j];
        }
      }
      if (!is_v && p.interleaved) {
#pragma unroll
        for (int s = 0; s < kNP; ++s) {
          const int c = 2 * (lane + 32 * s);
          if (c < p.rot_dims) {
            const float2 a = cs[i * half + (c >> 1)];
            const float u = y[s][0], v = y[s][1];
            y[s][0] = u * a.x - v * a.y;
            y[s][1] = v * a.x + u * a.y;
          }
        }
      } else if (!is_v && half > 0) {
        float* sw = swap_s[warp];
#pragma unroll
        for (int s = 0; s < kNP; ++s) *reinterpret_cast<float2*>(sw + 2 * (lane + 32 * s)) = make_float2(y[s][0], y[s][1]);
        __syncwarp();
#pragma unroll
        for (int s = 0; s < kNP; ++s)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int c = 2 * (lane + 32 * s) + j;
            if (c < half) {
              const float2 a = cs[i * half + c];
              y[s][j] = y[s][j] * a.x - sw[c + half] * a.y;
            } else if (c < p.rot_dims) {
              const float2 a = cs[i * half + c - half];
              y[s][j] = y[s][j] * a.x + sw[c - half] * a.y;
            }
          }
        __syncwarp();
      }
      T* dst;
      int w_out;
      if (is_q) {
        dst = p.q + (static_cast<size_t>(row) * p.heads + head) * p.q_pad;
        w_out = p.q_pad;                                  // channels past dim are zero
      } else {
        const size_t slot = (static_cast<size_t>(m_page[i]) * p.kv_heads + kvh) * p.page_size + pos % p.page_size;
        dst = is_v ? p.v_pages + slot * p.ld_v : p.k_pages + slot * p.ld_k;
        w_out = width;
      }
#pragma unroll
      for (int s = 0; s < kNP; ++s) st2(dst, 2 * (lane + 32 * s), w_out, y[s]);
    }
  }
}

// spans: [sequences][4] = {row of the block table, first context position, context rows, first gathered row}.
// grid (ceil(longest context / 8), sequences), 8 warps: a warp per row.
__global__ void __launch_bounds__(256)
kv_gather_kernel(const __nv_bfloat16* __restrict__ k_pages, const __nv_bfloat16* __restrict__ v_pages, int page_size,
                 const int* __restrict__ block_table, int max_blocks, const int* __restrict__ spans, __nv_bfloat16* __restrict__ out,
                 int kv_heads, int dim, int vdim) {
  pdl_wait();
  pdl_trigger();
  const int* sp = spans + 4 * blockIdx.y;
  const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= sp[2]) return;
  const int pos = sp[1] + i;
  const size_t page = static_cast<size_t>(block_table[static_cast<size_t>(sp[0]) * max_blocks + pos / page_size]) * kv_heads;
  __nv_bfloat16* dst = out + (static_cast<size_t>(sp[3]) + i) * kv_heads * (dim + vdim);
  const int ku = dim >> 3, vu = vdim >> 3, off = pos % page_size;
  for (int e = lane; e < kv_heads * (ku + vu); e += 32) {
    const bool is_v = e >= kv_heads * ku;
    const int f = is_v ? e - kv_heads * ku : e, u = is_v ? vu : ku, h = f / u, c = (f - h * u) * 8;
    const size_t slot = (page + h) * page_size + off;
    const __nv_bfloat16* src = is_v ? v_pages + slot * vdim + c : k_pages + slot * dim + c;
    *reinterpret_cast<uint4*>(dst + (is_v ? kv_heads * dim + h * vdim : h * dim) + c) = *reinterpret_cast<const uint4*>(src);
  }
}

template <typename T>
struct KvAttentionParams {
  const T *q, *k_pages, *v_pages, *gate;
  const float* sinks;
  const int *block_table, *seq_index, *kv_lens;
  T* out;
  const float* slopes;
  DistanceBias dist;
  long long ld_gate;
  int max_blocks, heads, kv_heads, dim, vdim, q_pad, ld_k, ld_v, page_size, window, keep_first, chunk, gate_heads;
  float scale;
};

// grid (rows, ceil(heads / 4)), 128 threads; kNV: value channels per lane.
template <typename T, int kNV>
__global__ void __launch_bounds__(128) kv_attention_kernel(const KvAttentionParams<T> p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float q_all[];                      // [4][dim]
  const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y * 4 + warp;
  if (head >= p.heads) return;
  float* q = q_all + warp * p.dim;
  const int kvh = head / (p.heads / p.kv_heads), len = p.kv_lens[r];
  const VisibleKeys keys(len, p.window, p.keep_first, p.chunk);
  const float slope = p.slopes ? p.slopes[head] : 0.f;
  const float* dist = p.dist.table ? p.dist.head(head) : nullptr;
  const int* bt = p.block_table + static_cast<size_t>(p.seq_index[r]) * p.max_blocks;
  for (int c = lane; c < p.dim; c += 32) q[c] = ld_f(p.q + (static_cast<size_t>(r) * p.heads + head) * p.q_pad + c) * p.scale;
  __syncwarp();
  float m = -INFINITY, l = 0.f, o[kNV];
#pragma unroll
  for (int j = 0; j < kNV; ++j) o[j] = 0.f;
  for (int base = 0; base < keys.n; base += 32) {
    const bool live = base + lane < keys.n;
    long long slot = 0;
    float s = -INFINITY;
    if (live) {
      const int tok = keys.position(base + lane);
      slot = (static_cast<long long>(bt[tok / p.page_size]) * p.kv_heads + kvh) * p.page_size + tok % p.page_size;
      const T* k = p.k_pages + slot * p.ld_k;
      s = 0.f;
      for (int c = 0; c < p.dim; ++c) s = fmaf(q[c], ld_f(k + c), s);
      s = fmaf(-slope, static_cast<float>(len - 1 - tok), s);
      if (dist) s += dist[min(len - 1 - tok, p.dist.n - 1)];
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float pr = live ? expf(s - m_new) : 0.f;
    const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
    l = l * alpha + warp_sum(pr);
    m = m_new;
#pragma unroll
    for (int j = 0; j < kNV; ++j) o[j] *= alpha;
    const int cnt = min(32, keys.n - base);
    for (int i = 0; i < cnt; ++i) {
      const float pi = __shfl_sync(0xffffffffu, pr, i);
      const T* v = p.v_pages + __shfl_sync(0xffffffffu, slot, i) * p.ld_v;
#pragma unroll
      for (int j = 0; j < kNV; ++j)
        if (lane + 32 * j < p.vdim) o[j] = fmaf(pi, ld_f(v + lane + 32 * j), o[j]);
    }
  }
  if (p.sinks) {                                        // a score that joins the denominator only
    const float sk = p.sinks[head], m2 = fmaxf(m, sk), f = m == -INFINITY ? 0.f : expf(m - m2);
    l = l * f + expf(sk - m2);
#pragma unroll
    for (int j = 0; j < kNV; ++j) o[j] *= f;
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
  for (int j = 0; j < kNV; ++j) {
    const int c = lane + 32 * j;
    if (c < p.vdim) {
      float v = o[j] * inv;
      if (p.gate) v *= sigmoid_f(ld_f(p.gate + r * p.ld_gate + (p.gate_heads ? head : head * p.vdim + c)));
      st_f(p.out + (static_cast<size_t>(r) * p.heads + head) * p.vdim + c, v);
    }
  }
}

}  // namespace sllm

using namespace sllm;

// Mirrored by ops/kv_attention.py (ctypes.Structure); checked by sllm_kv_abi.
struct SllmKvPrepare {
  const void *proj, *conv_w, *bias, *q_norm, *k_norm, *ring, *inv_freq, *row_off, *slots, *positions, *seq_index, *block_table, *q,
      *k_pages, *v_pages, *v_other;
  long long ring_stride;
  int ldp, max_blocks, heads, kv_heads, dim, vdim, q_pad, ld_k, ld_v, rot_dims, taps, page_size, tokens, sequences, norm, decode, fp32,
      interleaved, ld_other, v_norm;
  float v_mix, eps;
};

SLLM_EXPORT int sllm_kv_abi(int* out, int n) {
  const int v[2] = {static_cast<int>(sizeof(SllmKvPrepare)), static_cast<int>(offsetof(SllmKvPrepare, eps))};
  for (int i = 0; i < n && i < 2; ++i) out[i] = v[i];
  return 2;
}

template <typename T, int kTaps, bool kVec>
static cudaError_t kv_prepare_go(const KvPrepareParams<T>& p, int by, size_t smem, cudaStream_t st) {
  const int wide = p.q_pad > p.vdim ? p.q_pad : p.vdim;
  auto* kernel = wide <= 64 ? kv_prepare_kernel<T, 1, kTaps, kVec> : wide <= 128 ? kv_prepare_kernel<T, 2, kTaps, kVec>
                                                                                  : kv_prepare_kernel<T, 4, kTaps, kVec>;
  return launch_kernel(kernel, dim3((p.tokens + p.run - 1) / p.run, by), dim3(kKpThreads), smem, st, 1u, p);
}

template <typename T>
static int kv_prepare_launch(const SllmKvPrepare* a, cudaStream_t st) {
  KvPrepareParams<T> p = {};
  auto n = [](const void* x) { return static_cast<const int*>(x); };
  auto t = [](const void* x) { return static_cast<T*>(const_cast<void*>(x)); };
  p.bias = static_cast<const float*>(a->bias); p.q_norm = static_cast<const float*>(a->q_norm);
  p.k_norm = static_cast<const float*>(a->k_norm); p.interleaved = a->interleaved;
  p.proj = t(a->proj); p.conv_w = static_cast<const float*>(a->conv_w); p.ring = static_cast<float*>(const_cast<void*>(a->ring));
  p.inv_freq = static_cast<const float*>(a->inv_freq); p.row_off = n(a->row_off); p.slots = n(a->slots);
  p.positions = n(a->positions); p.seq_index = n(a->seq_index); p.block_table = n(a->block_table);
  p.q = t(a->q); p.k_pages = t(a->k_pages); p.v_pages = t(a->v_pages); p.ring_stride = a->ring_stride;
  p.ldp = a->ldp; p.max_blocks = a->max_blocks; p.heads = a->heads; p.kv_heads = a->kv_heads; p.dim = a->dim; p.vdim = a->vdim;
  p.q_pad = a->q_pad; p.ld_k = a->ld_k; p.ld_v = a->ld_v; p.rot_dims = a->rot_dims; p.taps = a->taps; p.page_size = a->page_size;
  p.v_other = t(a->v_other); p.v_mix = a->v_mix; p.ld_other = a->ld_other; p.v_norm = a->v_norm;
  p.tokens = a->tokens; p.norm = a->norm; p.decode = a->decode; p.eps = a->eps;
  const bool vec = !((p.ldp | p.dim | p.vdim | p.q_pad | p.ld_k | p.ld_v) & 1) && !(a->ring_stride & 1) &&
          !((reinterpret_cast<uintptr_t>(a->proj) | reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->v_other)) & 7) &&
          !(p.ld_other & 1);
  int by = (p.heads + 2 * p.kv_heads + 7) / 8;
  if (p.norm == kNormAll && p.tokens >= 296) by = 1;    // a CTA's sums over a token's row serve all of its heads
  p.run = kKpRun;
  while (p.run > 1 && (p.decode || static_cast<long long>((p.tokens + p.run - 1) / p.run) * by < 296)) p.run >>= 1;
  const size_t smem = sizeof(float2) * p.run * (p.rot_dims / 2 + 1);
  cudaError_t e;
  if (p.taps == 1) e = vec ? kv_prepare_go<T, 1, true>(p, by, smem, st) : kv_prepare_go<T, 1, false>(p, by, smem, st);
  else if (p.taps <= 4) e = vec ? kv_prepare_go<T, 4, true>(p, by, smem, st) : kv_prepare_go<T, 4, false>(p, by, smem, st);
  else e = vec ? kv_prepare_go<T, 8, true>(p, by, smem, st) : kv_prepare_go<T, 8, false>(p, by, smem, st);
  if (e != cudaSuccess) return SLLM_ERR_CUDA;
  if (p.decode || p.taps < 2 || !p.conv_w) return SLLM_OK;
  const int channels = (p.heads + p.kv_heads) * p.dim + p.kv_heads * p.vdim;
  return conv_ring_launch(p.proj, p.ldp, std::is_same_v<T, float>, p.ring, p.ring_stride, p.row_off, p.slots, p.positions, channels,
                          p.taps, a->sequences, st) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

// kv_heads 0: a layer without keys and values of its own (queries only).
SLLM_EXPORT int sllm_kv_prepare(const SllmKvPrepare* a, void* stream) {
  if (!a || !a->proj || (a->conv_w && !a->ring) || (!a->conv_w && a->taps != 1) || (a->bias && a->conv_w) || !a->slots || !a->positions || !a->seq_index || !a->q || a->heads <= 0 ||
      a->kv_heads < 0 || a->dim <= 0 || a->vdim <= 0 || a->q_pad < a->dim || a->taps <= 0 || a->tokens <= 0 || a->sequences <= 0 ||
      a->rot_dims < 0 || a->rot_dims > a->dim || (a->rot_dims & 1) || (a->rot_dims > 0 && !a->inv_freq) || (!a->decode && !a->row_off) ||
      (a->decode && a->tokens != a->sequences))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->norm < kNormNone || a->norm > kNormAll || (a->norm == kNormAll && a->conv_w) ||
      (a->v_other && (a->kv_heads <= 0 || a->ld_other < a->kv_heads * a->vdim)))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->kv_heads > 0 && (!a->k_pages || !a->v_pages || !a->block_table || a->page_size <= 0 || a->ld_k < a->dim || a->ld_v < a->vdim))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (a->taps > 8 || a->q_pad > 256 || a->vdim > 256 || a->sequences > 65535) return SLLM_ERR_UNSUPPORTED_SHAPE;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->fp32 ? kv_prepare_launch<float>(a, st) : kv_prepare_launch<__nv_bfloat16>(a, st);
}

SLLM_EXPORT int sllm_kv_gather(const void* k_pages, const void* v_pages, int page_size, const int* block_table, int max_blocks,
                               const int* spans, int sequences, int longest, void* out, int kv_heads, int dim, int vdim,
                               void* stream) {
  if (!k_pages || !v_pages || !block_table || !spans || !out || sequences <= 0 || longest <= 0 || page_size <= 0 || kv_heads <= 0 ||
      dim <= 0 || vdim <= 0)
    return SLLM_ERR_INVALID_ARGUMENT;
  if ((dim & 7) || (vdim & 7) || sequences > 65535) return SLLM_ERR_UNSUPPORTED_SHAPE;
  if ((reinterpret_cast<uintptr_t>(k_pages) | reinterpret_cast<uintptr_t>(v_pages) | reinterpret_cast<uintptr_t>(out)) & 15)
    return SLLM_ERR_ALIGNMENT;
  return launch_kernel(kv_gather_kernel, dim3((longest + 7) / 8, sequences), dim3(256), 0, static_cast<cudaStream_t>(stream), 1u,
                       static_cast<const __nv_bfloat16*>(k_pages), static_cast<const __nv_bfloat16*>(v_pages), page_size, block_table,
                       max_blocks, spans, static_cast<__nv_bfloat16*>(out), kv_heads, dim, vdim) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

template <typename T>
static int kv_attention_launch(const KvAttentionParams<T>& p, int rows, cudaStream_t st) {
  const dim3 grid(rows, (p.heads + 3) / 4);
  const size_t smem = sizeof(float) * 4 * p.dim;
  cudaError_t e;
  if (p.vdim <= 64) e = launch_kernel(kv_attention_kernel<T, 2>, grid, dim3(128), smem, st, 1u, p);
  else if (p.vdim <= 128) e = launch_kernel(kv_attention_kernel<T, 4>, grid, dim3(128), smem, st, 1u, p);
  else e = launch_kernel(kv_attention_kernel<T, 8>, grid, dim3(128), smem, st, 1u, p);
  return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

// q [rows, heads, q_pad]; gate: optional logits [rows, ld_gate], one per output channel (gate_heads: per head); keep_first,
// chunk: see VisibleKeys; slopes: optional [heads]; dist: see DistanceBias; out [rows, heads * vdim].
SLLM_EXPORT int sllm_kv_attention(const void* q, const void* k_pages, const void* v_pages, const void* gate, long long ld_gate,
                                  const float* sinks, const int* block_table, int max_blocks, const int* seq_index, const int* kv_lens,
                                  int rows, int heads, int kv_heads, int dim, int vdim, int q_pad, int ld_k, int ld_v, int page_size,
                                  int window, int keep_first, int chunk, const float* slopes, const float* dist, int n_dist, int ld_dist,
                                  int gate_heads, float scale, void* out, int fp32, void* stream) {
  if (!q || !k_pages || !v_pages || !block_table || !seq_index || !kv_lens || !out || rows <= 0 || heads <= 0 || kv_heads <= 0 ||
      heads % kv_heads || dim <= 0 || vdim <= 0 || q_pad < dim || ld_k < dim || ld_v < vdim || page_size <= 0 || window < 0 || keep_first < 0 ||
      chunk < 0 || (keep_first > 0 && window == 0) || (chunk > 0 && window > 0))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (dist && (n_dist < 1 || ld_dist < kDistFront + n_dist)) return SLLM_ERR_INVALID_ARGUMENT;
  if (vdim > 256 || dim > 2048) return SLLM_ERR_UNSUPPORTED_SHAPE;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto fill = [&](auto* p) {
    using T = std::remove_const_t<std::remove_pointer_t<decltype(p->q)>>;
    p->q = static_cast<const T*>(q); p->k_pages = static_cast<const T*>(k_pages); p->v_pages = static_cast<const T*>(v_pages);
    p->gate = static_cast<const T*>(gate); p->ld_gate = ld_gate; p->sinks = sinks; p->block_table = block_table;
    p->max_blocks = max_blocks; p->seq_index = seq_index; p->kv_lens = kv_lens; p->out = static_cast<T*>(out);
    p->heads = heads; p->kv_heads = kv_heads; p->dim = dim; p->vdim = vdim; p->q_pad = q_pad; p->ld_k = ld_k; p->ld_v = ld_v;
    p->page_size = page_size; p->window = window; p->keep_first = keep_first; p->chunk = chunk; p->slopes = slopes; p->dist = {dist, n_dist, ld_dist}; p->gate_heads = gate_heads; p->scale = scale;
  };
  if (fp32) {
    KvAttentionParams<float> p = {};
    fill(&p);
    return kv_attention_launch(p, rows, st);
  }
  KvAttentionParams<__nv_bfloat16> p = {};
  fill(&p);
  return kv_attention_launch(p, rows, st);
}
