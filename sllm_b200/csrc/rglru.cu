// Gated linear recurrence with a short convolution in front of it, per channel:
//
//   u   = conv(x + bias_x) + conv_b                    causal, `taps` inputs per channel
//   r,i = sigmoid(block-diagonal products of u + biases)
//   a   = exp(decay * r)                               decay = -c softplus(lambda), negative, per channel
//   S   = a S + sqrt(1 - a^2) i u                      fp32, carried per sequence slot
//   out = S gelu_tanh(y + bias_y)
//
// y and x are column slices of one projection.  Rows of a sequence are consecutive in the flat batch.  The conv inputs of
// the last `taps` positions live in a ring per slot, row (position mod taps), fp32: a decoded token reads taps - 1 rows and
// writes another one, so CTAs that share a channel do not race.
//
//   rglru_tile_kernel    gates on tcgen05: D[channel, token] of both gates for 64 tokens, weights resident in shared memory
//                        for all tiles of the CTA, u built there by the producer warps.  A thread of the epilogue owns one
//                        channel and walks over the tokens.  Decode form: a token is a sequence, the kernel finishes it.
//                        Prompt form: the recurrence within the tile, from the slot's state in a sequence's first tile and
//                        from zero in the others, with the running product of a.
//   rglru_finish_kernel  prompt form: carry over the earlier tiles of the sequence, output gate, state and ring
//   rglru_terms_kernel / rglru_scan_kernel    the same in fp32 or bf16 for any sizes on the CUDA cores
#include "typed.cuh"
#include "api.h"
#include "tmap.h"

#include <cstddef>

namespace sllm {

constexpr int kRgTokens = 64;            // tokens of a tile (prompt form)
constexpr int kRgDecodeRows = 16;        // tokens of a tile (decode form)
constexpr int kRgChannels = 128;         // channels of a tile
constexpr int kRgTaps = 4;               // taps of the tile kernel (shorter filters are padded)
constexpr int kRgMaxChunks = 4;          // 64-channel chunks of a block

struct RglruParams {
  const void* proj;        // [T, ldp]
  const float *bias_y, *bias_x, *conv_w, *conv_b, *bias_r, *bias_i, *decay;   // [W]; conv_w [taps, W]
  const void *gate_r, *gate_i;   // any-size form: [blocks, bs, bs] (out, in); tile form: through the tensor map
  float *state, *ring;     // slot strides below
  const int *row_off, *slots, *positions, *seq_index, *tiles;
  float *h, *prod;         // [T, W] prompt form (terms form: a in prod, the input term in h)
  void* out;               // [T, W]
  int* status;
  long long state_stride, ring_stride;
  int ldp, off_y, off_x, width, blocks, bs, taps, tokens, sequences, n_tiles, ct, kc;
};

__device__ __forceinline__ float rg_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rg_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rg_sqrt(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float kLog2e = 1.4426950408889634f;
// gelu_tanh(z) = z sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3))
__device__ __forceinline__ float rg_gelu(float z) {
  const float u = 1.5957691216057308f * (z + 0.044715f * z * z * z);
  return z * rg_rcp(1.f + rg_ex2(-kLog2e * u));
}
__device__ __forceinline__ float rg_gelu_exact(float z) {
  const float u = 1.5957691216057308f * (z + 0.044715f * z * z * z);
  return z / (1.f + expf(-u));
}
// (a, sqrt(1 - a^2) * gate) from gate logits; decay2 = decay * log2(e)
__device__ __forceinline__ void rg_terms(float zr, float zi, float decay2, float& a, float& m) {
  const float r = rg_rcp(1.f + rg_ex2(-kLog2e * zr));
  const float i = rg_rcp(1.f + rg_ex2(-kLog2e * zi));
  const float la = decay2 * r;                              // log2 a
  a = rg_ex2(la);
  // 1 - a^2 = 1 - exp(-x): directly, or by its series where that would cancel
  const float x = -1.3862943611198906f * la;                // -2 ln a
  const float series = x * (1.f - x * (0.5f - x * (0.16666667f - x * 0.041666667f)));
  const float one = x < 0.06f ? series : fmaf(-a, a, 1.f);
  m = rg_sqrt(one) * i;
}

// Eight channels of one conv input row (x + bias), fp32.
__device__ __forceinline__ void rg_row8(const __nv_bfloat16* p, const float (&bias)[8], float (&v)[8]) {
  ld16(p, v);
#pragma unroll
  for (int j = 0; j < 8; ++j) v[j] += bias[j];
}
__device__ __forceinline__ void rg_ld8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}

struct __align__(16) RglruShared {
  uint64_t w_full, mma_done[2], free_[2];
  uint32_t tmem_base;
  int abort_flag;
};

// grid (blocks * ct, CTAs per channel tile), 256 threads: warps 0-3 build u and issue the products, warps 4-7 finish.
// TMEM columns of buffer b: gate r at 128 b, gate i 64 further.
template <bool kDecode>
__global__ void __launch_bounds__(256, 1)
rglru_tile_kernel(const __grid_constant__ CUtensorMap tm_w, const RglruParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int kN = kDecode ? kRgDecodeRows : kRgTokens;
  constexpr int kWChunk = kRgChannels * 128, kUChunk = kN * 128;
  uint8_t* w_s = smem;                                  // [2 gates][kc] chunks
  uint8_t* u_s = smem + 2 * p.kc * kWChunk;             // [2 buffers][kc] chunks
  RglruShared* sh = reinterpret_cast<RglruShared*>(u_s + 2 * p.kc * kUChunk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blk = blockIdx.x / p.ct, ct = blockIdx.x % p.ct;
  volatile int* abort_flag = &sh->abort_flag;
  if (threadIdx.x == 0) {
    mbar_init(&sh->w_full, 1);
    for (int b = 0; b < 2; ++b) {
      mbar_init(&sh->mma_done[b], 1);
      mbar_init(&sh->free_[b], 128);
    }
    sh->abort_flag = 0;
    mbar_fence_init();
    mbar_expect_tx(&sh->w_full, 2 * p.kc * kWChunk);    // the weights are constant: no need to wait for earlier kernels
    for (int g = 0; g < 2; ++g)
      for (int c = 0; c < p.kc; ++c)
        tma_load_2d(w_s + (g * p.kc + c) * kWChunk, &tm_w, &sh->w_full, c * 64, (blockIdx.x * 2 + g) * kRgChannels);
  }
  if (warp == 4) {
    tmem_alloc(&sh->tmem_base, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = sh->tmem_base;
  pdl_wait();
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj);
  const int W = p.width;

  if (warp < 4) {
    const int tid = threadIdx.x, cgs = p.kc * 8, tgs = 128 / cgs, per = (kN + tgs - 1) / tgs;
    const int k0 = (tid % cgs) * 8, tg = tid / cgs;
    const bool active = tg < tgs, real = active && k0 < p.bs;
    const int ch = blk * p.bs + k0;                     // first of this thread's eight channels
    float cw[kRgTaps][8], cb[8], bx[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      cb[j] = real ? p.conv_b[ch + j] : 0.f;
      bx[j] = real ? p.bias_x[ch + j] : 0.f;
    }
#pragma unroll
    for (int t = 0; t < kRgTaps; ++t) {
      const int tap = t - (kRgTaps - p.taps);
#pragma unroll
      for (int j = 0; j < 8; ++j) cw[t][j] = real && tap >= 0 ? p.conv_w[static_cast<size_t>(tap) * W + ch + j] : 0.f;
    }
    const bool owner = real && k0 >= ct * kRgChannels && k0 < (ct + 1) * kRgChannels;
    bool ok = true;
    int it = 0;
    for (int tile = blockIdx.y; tile < p.n_tiles; tile += gridDim.y, ++it) {
      const int buf = it & 1;
      int row0, rows, seq = 0, pos0 = 0, first = 0;
      if (kDecode) {
        row0 = tile * kN;
        rows = min(kN, p.tokens - row0);
      } else {
        const int4 tl = reinterpret_cast<const int4*>(p.tiles)[tile];
        row0 = tl.x; rows = tl.y; seq = tl.z;
        first = p.row_off[seq];
        pos0 = p.positions[row0];
      }
      if (ok && it >= 2) ok = mbar_wait(&sh->free_[buf], ((it >> 1) - 1) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMEM_EMPTY);
      if (active) {
        uint8_t* dst = u_s + (buf * p.kc + (k0 >> 6)) * kUChunk;
        const int unit = (k0 & 63) >> 3;
        const int t_lo = tg * per, t_hi = min(kN, t_lo + per);
        auto put = [&](int t, const float (&x)[8], const float (&win)[kRgTaps - 1][8]) {   // win[b - 1]: b positions back
          float acc[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[j] = fmaf(cw[kRgTaps - 1][j], x[j], cb[j]);
#pragma unroll
          for (int b = 1; b < kRgTaps; ++b)
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[j] = fmaf(cw[kRgTaps - 1 - b][j], win[b - 1][j], acc[j]);
          uint4 o;
          __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
          for (int j = 0; j < 4; ++j) h2[j] = __floats2bfloat162_rn(acc[2 * j], acc[2 * j + 1]);
          *reinterpret_cast<uint4*>(dst + t * 128 + ((unit ^ (t & 7)) << 4)) = o;
        };
        auto zero = [&](int t) { *reinterpret_cast<uint4*>(dst + t * 128 + ((unit ^ (t & 7)) << 4)) = make_uint4(0, 0, 0, 0); };
        constexpr int kBatch = kDecode ? 4 : 8;         // rows whose loads are in flight together
        if constexpr (kDecode) {
          for (int t0 = t_lo; t0 < t_hi; t0 += kBatch) {
            int pos[kBatch], slot[kBatch];
            uint4 raw[kBatch];
            float win[kBatch][kRgTaps - 1][8];
#pragma unroll
            for (int i = 0; i < kBatch; ++i) {
              const bool in = real && t0 + i < t_hi && t0 + i < rows;
              pos[i] = in ? p.positions[row0 + t0 + i] : -1;
              slot[i] = in ? p.slots[row0 + t0 + i] : 0;
              raw[i] = in ? *reinterpret_cast<const uint4*>(proj + static_cast<size_t>(row0 + t0 + i) * p.ldp + p.off_x + ch) : make_uint4(0, 0, 0, 0);
            }
#pragma unroll
            for (int i = 0; i < kBatch; ++i)
#pragma unroll
              for (int b = 1; b < kRgTaps; ++b) {
#pragma unroll
                for (int j = 0; j < 8; ++j) win[i][b - 1][j] = 0.f;
                if (b < p.taps && pos[i] - b >= 0)
                  rg_ld8(p.ring + slot[i] * p.ring_stride + static_cast<size_t>((pos[i] - b) % p.taps) * W + ch, win[i][b - 1]);
              }
#pragma unroll
            for (int i = 0; i < kBatch; ++i) {
              if (t0 + i >= t_hi) break;
              if (pos[i] < 0) {
                zero(t0 + i);
                continue;
              }
              float x[8];
              rg_row8(reinterpret_cast<const __nv_bfloat16*>(&raw[i]), bx, x);
              if (owner) {
                float* d = p.ring + slot[i] * p.ring_stride + static_cast<size_t>(pos[i] % p.taps) * W + ch;
                *reinterpret_cast<float4*>(d) = make_float4(x[0], x[1], x[2], x[3]);
                *reinterpret_cast<float4*>(d + 4) = make_float4(x[4], x[5], x[6], x[7]);
              }
              put(t0 + i, x, win[i]);
            }
          }
        } else {
          const int n = real ? min(t_hi, rows) : t_lo;  // rows [t_lo, n) are real
          const __nv_bfloat16* src = proj + static_cast<size_t>(row0) * p.ldp + p.off_x + ch;
          float win[kRgTaps - 1][8];
          if (t_lo < n) {
            const float* ring = p.ring + p.slots[seq] * p.ring_stride;
#pragma unroll
            for (int b = 1; b < kRgTaps; ++b) {
              const int t = t_lo - b, pos = pos0 + t;
#pragma unroll
              for (int j = 0; j < 8; ++j) win[b - 1][j] = 0.f;
              if (b < p.taps && pos >= 0) {
                if (row0 + t >= first) rg_row8(src + static_cast<long long>(t) * p.ldp, bx, win[b - 1]);
                else rg_ld8(ring + static_cast<size_t>(pos % p.taps) * W + ch, win[b - 1]);
              }
            }
          }
          for (int t0 = t_lo; t0 < n; t0 += kBatch) {
            uint4 raw[kBatch];
#pragma unroll
            for (int i = 0; i < kBatch; ++i)
              raw[i] = t0 + i < n ? *reinterpret_cast<const uint4*>(src + static_cast<size_t>(t0 + i) * p.ldp) : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int i = 0; i < kBatch; ++i) {
              if (t0 + i >= n) break;
              float x[8];
              rg_row8(reinterpret_cast<const __nv_bfloat16*>(&raw[i]), bx, x);
              put(t0 + i, x, win);
#pragma unroll
              for (int b = kRgTaps - 1; b > 1; --b)
#pragma unroll
                for (int j = 0; j < 8; ++j) win[b - 1][j] = win[b - 2][j];
#pragma unroll
              for (int j = 0; j < 8; ++j) win[0][j] = x[j];
            }
          }
          for (int t = max(n, t_lo); t < t_hi; ++t) zero(t);
        }
      }
      fence_proxy_async_smem();
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (tid == 0) {
        if (ok && it == 0) ok = mbar_wait(&sh->w_full, 0, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMA_FULL);
        if (ok) {
          tc_fence_after();
          constexpr uint32_t idesc = make_idesc(kFmtBf16, kRgChannels, kN, 0, 0);
          for (int g = 0; g < 2; ++g)
            for (int c = 0; c < p.kc; ++c) {
              const uint64_t da = make_smem_desc_sw128(smem_u32(w_s + (g * p.kc + c) * kWChunk));
              const uint64_t db = make_smem_desc_sw128(smem_u32(u_s + (buf * p.kc + c) * kUChunk));
#pragma unroll
              for (int k = 0; k < 4; ++k)
                umma_f16(tmem_base + buf * 128 + g * 64, da + 2 * k, db + 2 * k, idesc, (c | k) != 0);
            }
          tc_commit(&sh->mma_done[buf]);
        }
      }
    }
    if (tid == 0) {
      int dummy = 0;                                    // the weight copies have landed before the CTA leaves
      mbar_wait(&sh->w_full, 0, &dummy, p.status, SLLM_DEV_TIMEOUT_DRAIN, 200000000LL);
    }
  } else {
    const int qd = warp & 3;
    const int kch = ct * kRgChannels + qd * 32 + lane;  // channel within the block
    const bool valid = kch < p.bs;
    const int ch = blk * p.bs + (valid ? kch : 0);
    const float rb = p.bias_r[ch], ib = p.bias_i[ch], dec2 = p.decay[ch] * kLog2e, by = p.bias_y[ch];
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(qd * 32) << 16);
    const uint32_t u_col = ((static_cast<uint32_t>(valid ? kch : 0) & 63) >> 3), u_byte = (kch & 7) * 2;
    bool ok = true;
    int it = 0;
    for (int tile = blockIdx.y; tile < p.n_tiles; tile += gridDim.y, ++it) {
      const int buf = it & 1;
      const uint8_t* u_t = u_s + (buf * p.kc + ((valid ? kch : 0) >> 6)) * kUChunk + u_byte;
      int row0, rows, slot = 0, chunk = 0;
      if (kDecode) {
        row0 = tile * kN;
        rows = min(kN, p.tokens - row0);
      } else {
        const int4 tl = reinterpret_cast<const int4*>(p.tiles)[tile];
        row0 = tl.x; rows = tl.y; slot = p.slots[tl.z]; chunk = tl.w & 0xffffff;
      }
      float S = 0.f, A = 1.f;
      if (!kDecode && chunk == 0 && valid) S = p.state[slot * p.state_stride + ch];
      for (int c = 0; c < kN / 16; ++c) {
        float st[16], yv[16];
        int sl[16];
        if (kDecode) {
          // the states and gates of 16 rows are requested together, the first ones before the products are there
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const int t = c * 16 + i;
            sl[i] = t < rows ? p.slots[row0 + t] : 0;
          }
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const int t = c * 16 + i;
            const bool in = t < rows && valid;
            st[i] = in ? p.state[sl[i] * p.state_stride + ch] : 0.f;
            yv[i] = in ? __bfloat162float(proj[static_cast<size_t>(row0 + t) * p.ldp + p.off_y + ch]) : 0.f;
          }
        }
        if (c == 0) {
          if (ok) ok = mbar_wait(&sh->mma_done[buf], (it >> 1) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMEM_FULL);
          ok = __all_sync(0xffffffffu, ok);
          tc_fence_after();
        }
        if (c * 16 >= rows || !ok) break;
        uint32_t zr[16], zi[16];
        tmem_ld16(lane_addr + buf * 128 + c * 16, zr);
        tmem_ld16(lane_addr + buf * 128 + 64 + c * 16, zi);
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int t = c * 16 + i;
          const float u = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(u_t + t * 128 + ((u_col ^ (t & 7)) << 4)));
          float a, m;
          rg_terms(__uint_as_float(zr[i]) + rb, __uint_as_float(zi[i]) + ib, dec2, a, m);
          if (kDecode) {
            const float s = fmaf(a, st[i], m * u);
            if (t < rows && valid) {
              p.state[sl[i] * p.state_stride + ch] = s;
              static_cast<__nv_bfloat16*>(p.out)[static_cast<size_t>(row0 + t) * W + ch] = __float2bfloat16_rn(s * rg_gelu(yv[i] + by));
            }
          } else {
            S = fmaf(a, S, m * u);
            A *= a;
            if (t < rows && valid) {
              const size_t idx = static_cast<size_t>(row0 + t) * W + ch;
              p.h[idx] = S;
              p.prod[idx] = A;
            }
          }
        }
      }
      tc_fence_before();
      mbar_arrive(&sh->free_[buf]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 4) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 256);
  }
}

// grid (ceil(W / 256), tiles), 256 threads: 64 groups of 4 channels x 4 runs of 16 tokens.
__global__ void __launch_bounds__(256) rglru_finish_kernel(const RglruParams p) {
  pdl_wait();
  const int4 tl = reinterpret_cast<const int4*>(p.tiles)[blockIdx.y];
  const int row0 = tl.x, rows = tl.y, seq = tl.z, chunk = tl.w & 0xffffff;
  const bool last = (tl.w >> 24) != 0;
  const int ch = blockIdx.x * 256 + (threadIdx.x & 63) * 4, run = threadIdx.x >> 6, W = p.width;
  if (ch >= W) return;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj);
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  const size_t tail = static_cast<size_t>(row0 - chunk * kRgTokens + kRgTokens - 1) * W + ch;   // last row of the first tile
#pragma unroll 4
  for (int j = 0; j < chunk; ++j) {
    const size_t idx = tail + static_cast<size_t>(j) * kRgTokens * W;
    const float4 h = *reinterpret_cast<const float4*>(p.h + idx), a = *reinterpret_cast<const float4*>(p.prod + idx);
    S.x = fmaf(a.x, S.x, h.x); S.y = fmaf(a.y, S.y, h.y); S.z = fmaf(a.z, S.z, h.z); S.w = fmaf(a.w, S.w, h.w);
  }
  const float4 by = *reinterpret_cast<const float4*>(p.bias_y + ch);
  const int t_hi = min(rows, run * 16 + 16);
#pragma unroll 4
  for (int t = run * 16; t < t_hi; ++t) {
    const size_t idx = static_cast<size_t>(row0 + t) * W + ch;
    const float4 h = *reinterpret_cast<const float4*>(p.h + idx), a = *reinterpret_cast<const float4*>(p.prod + idx);
    float y[4];
    ld_vec<4>(proj + static_cast<size_t>(row0 + t) * p.ldp + p.off_y + ch, y);
    const float4 s = make_float4(fmaf(a.x, S.x, h.x), fmaf(a.y, S.y, h.y), fmaf(a.z, S.z, h.z), fmaf(a.w, S.w, h.w));
    const float o[4] = {s.x * rg_gelu(y[0] + by.x), s.y * rg_gelu(y[1] + by.y), s.z * rg_gelu(y[2] + by.z), s.w * rg_gelu(y[3] + by.w)};
    st_vec<4>(static_cast<__nv_bfloat16*>(p.out) + idx, o);
    if (last && t == rows - 1) *reinterpret_cast<float4*>(p.state + p.slots[seq] * p.state_stride + ch) = s;
  }
  if (last && run == 0) {
    const float4 bx = *reinterpret_cast<const float4*>(p.bias_x + ch);
    const int end = row0 + rows;
    for (int row = max(p.row_off[seq], end - p.taps); row < end; ++row) {
      float x[4];
      ld_vec<4>(proj + static_cast<size_t>(row) * p.ldp + p.off_x + ch, x);
      *reinterpret_cast<float4*>(p.ring + p.slots[seq] * p.ring_stride + static_cast<size_t>(p.positions[row] % p.taps) * W + ch) =
          make_float4(x[0] + bx.x, x[1] + bx.y, x[2] + bx.z, x[3] + bx.w);
    }
  }
}

// ---------------------------------------------------------------- any sizes
constexpr int kRgRows = 8;

// grid (ceil(T / 8), blocks), 128 threads.
template <typename T>
__global__ void __launch_bounds__(128) rglru_terms_kernel(const RglruParams p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float u[];                          // [8][bs]
  const int r0 = blockIdx.x * kRgRows, n = min(kRgRows, p.tokens - r0), base = blockIdx.y * p.bs, W = p.width;
  const T* proj = static_cast<const T*>(p.proj);
  for (int e = threadIdx.x; e < n * p.bs; e += 128) {
    const int row = r0 + e / p.bs, ch = base + e % p.bs, seq = p.seq_index[row], pos = p.positions[row];
    float acc = p.conv_b[ch];
    for (int b = 0; b < p.taps && b <= pos; ++b) {
      const float x = row - b >= p.row_off[seq]
                          ? ld_f(proj + static_cast<size_t>(row - b) * p.ldp + p.off_x + ch) + p.bias_x[ch]
                          : p.ring[p.slots[seq] * p.ring_stride + static_cast<size_t>((pos - b) % p.taps) * W + ch];
      acc = fmaf(p.conv_w[static_cast<size_t>(p.taps - 1 - b) * W + ch], x, acc);
    }
    u[e] = acc;
  }
  __syncthreads();
  const T* gr = static_cast<const T*>(p.gate_r) + static_cast<size_t>(base) * p.bs;
  const T* gi = static_cast<const T*>(p.gate_i) + static_cast<size_t>(base) * p.bs;
  for (int o = threadIdx.x; o < p.bs; o += 128) {
    float zr[kRgRows], zi[kRgRows];
#pragma unroll
    for (int t = 0; t < kRgRows; ++t) {
      zr[t] = p.bias_r[base + o];
      zi[t] = p.bias_i[base + o];
    }
    for (int k = 0; k < p.bs; ++k) {
      const float wr = ld_f(gr + static_cast<size_t>(o) * p.bs + k), wi = ld_f(gi + static_cast<size_t>(o) * p.bs + k);
#pragma unroll
      for (int t = 0; t < kRgRows; ++t) {
        const float x = t < n ? u[t * p.bs + k] : 0.f;
        zr[t] = fmaf(wr, x, zr[t]);
        zi[t] = fmaf(wi, x, zi[t]);
      }
    }
#pragma unroll
    for (int t = 0; t < kRgRows; ++t) {
      if (t < n) {
        const float la = p.decay[base + o] * sigmoid_f(zr[t]);
        const size_t idx = static_cast<size_t>(r0 + t) * W + base + o;
        p.prod[idx] = expf(la);
        p.h[idx] = sqrtf(-expm1f(2.f * la)) * sigmoid_f(zi[t]) * u[t * p.bs + o];
      }
    }
  }
}

// grid (ceil(W / 128), sequences), 128 threads.
template <typename T>
__global__ void __launch_bounds__(128) rglru_scan_kernel(const RglruParams p) {
  pdl_wait();
  pdl_trigger();
  const int ch = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y, W = p.width;
  if (ch >= W) return;
  const int r0 = p.row_off[seq], r1 = p.row_off[seq + 1];
  if (r1 <= r0) return;
  const T* proj = static_cast<const T*>(p.proj);
  float* st = p.state + p.slots[seq] * p.state_stride + ch;
  float S = *st;
  for (int row = r0; row < r1; ++row) {
    const size_t idx = static_cast<size_t>(row) * W + ch;
    S = fmaf(p.prod[idx], S, p.h[idx]);
    st_f(static_cast<T*>(p.out) + idx, S * rg_gelu_exact(ld_f(proj + static_cast<size_t>(row) * p.ldp + p.off_y + ch) + p.bias_y[ch]));
  }
  *st = S;
  for (int row = max(r0, r1 - p.taps); row < r1; ++row)
    p.ring[p.slots[seq] * p.ring_stride + static_cast<size_t>(p.positions[row] % p.taps) * W + ch] =
        ld_f(proj + static_cast<size_t>(row) * p.ldp + p.off_x + ch) + p.bias_x[ch];
}

}  // namespace sllm

using namespace sllm;

// Mirrored by ops/rglru.py (ctypes.Structure); checked by sllm_rglru_abi.
struct SllmRglru {
  const void *proj, *bias_y, *bias_x, *conv_w, *conv_b, *bias_r, *bias_i, *decay, *gate_r, *gate_i, *gate_tiles;
  void *state, *ring;
  const void *row_off, *slots, *positions, *seq_index, *tiles;
  void *h, *prod, *out, *status;
  long long state_stride, ring_stride;
  int ldp, off_y, off_x, width, blocks, bs, taps, tokens, sequences, n_tiles, fp32, decode;
};

SLLM_EXPORT int sllm_rglru_abi(int* out, int n) {
  const int v[2] = {static_cast<int>(sizeof(SllmRglru)), static_cast<int>(offsetof(SllmRglru, decode))};
  for (int i = 0; i < n && i < 2; ++i) out[i] = v[i];
  return 2;
}

static int rglru_params(const SllmRglru* a, RglruParams* p) {
  if (!a || !a->proj || !a->bias_y || !a->bias_x || !a->conv_w || !a->conv_b || !a->bias_r || !a->bias_i || !a->decay || !a->state ||
      !a->ring || !a->slots || !a->positions || !a->out || a->width <= 0 || a->blocks <= 0 || a->bs <= 0 || a->taps <= 0 ||
      a->tokens <= 0 || a->sequences <= 0 || a->blocks * a->bs != a->width || a->off_y < 0 || a->off_x < 0 ||
      a->ldp < a->off_x + a->width || a->ldp < a->off_y + a->width)
    return SLLM_ERR_INVALID_ARGUMENT;
  *p = {};
  auto f = [](const void* x) { return static_cast<const float*>(x); };
  auto n = [](const void* x) { return static_cast<const int*>(x); };
  p->proj = a->proj; p->bias_y = f(a->bias_y); p->bias_x = f(a->bias_x); p->conv_w = f(a->conv_w); p->conv_b = f(a->conv_b);
  p->bias_r = f(a->bias_r); p->bias_i = f(a->bias_i); p->decay = f(a->decay); p->gate_r = a->gate_r; p->gate_i = a->gate_i;
  p->state = static_cast<float*>(a->state); p->ring = static_cast<float*>(a->ring);
  p->row_off = n(a->row_off); p->slots = n(a->slots); p->positions = n(a->positions); p->seq_index = n(a->seq_index);
  p->tiles = n(a->tiles); p->h = static_cast<float*>(a->h); p->prod = static_cast<float*>(a->prod); p->out = a->out;
  p->status = static_cast<int*>(a->status); p->state_stride = a->state_stride; p->ring_stride = a->ring_stride;
  p->ldp = a->ldp; p->off_y = a->off_y; p->off_x = a->off_x; p->width = a->width; p->blocks = a->blocks; p->bs = a->bs;
  p->taps = a->taps; p->tokens = a->tokens; p->sequences = a->sequences; p->n_tiles = a->n_tiles;
  return SLLM_OK;
}

// Tensor-core form (bf16; gate_tiles: [blocks, ceil(bs / 128), 2 gates, 128 rows, ceil(bs / 64) * 64], zero padded).
// decode: one row per sequence.  Otherwise tiles is int32 [n_tiles][4] = {first row, rows, sequence, tile number within the
// sequence | last << 24}, in order within each sequence, and h / prod hold [tokens, width] floats.
SLLM_EXPORT int sllm_rglru(const SllmRglru* a, void* stream) {
  RglruParams p;
  int rc = rglru_params(a, &p);
  if (rc != SLLM_OK) return rc;
  if (a->fp32 || !a->gate_tiles || (a->bs & 7) || a->bs > kRgMaxChunks * 64 || a->taps > kRgTaps || (a->ldp & 7) || (a->off_x & 7) ||
      (a->off_y & 7) || (a->state_stride & 3) || (a->ring_stride & 3))
    return SLLM_ERR_UNSUPPORTED_SHAPE;
  if ((reinterpret_cast<uintptr_t>(a->proj) | reinterpret_cast<uintptr_t>(a->ring) | reinterpret_cast<uintptr_t>(a->state) |
       reinterpret_cast<uintptr_t>(a->bias_y) | reinterpret_cast<uintptr_t>(a->bias_x) | reinterpret_cast<uintptr_t>(a->out)) & 15)
    return SLLM_ERR_ALIGNMENT;
  if (a->decode) {
    if (a->tokens != a->sequences) return SLLM_ERR_INVALID_ARGUMENT;
    p.n_tiles = (a->tokens + kRgDecodeRows - 1) / kRgDecodeRows;
  } else if (!a->tiles || a->n_tiles <= 0 || !a->h || !a->prod || !a->row_off) {
    return SLLM_ERR_INVALID_ARGUMENT;
  }
  p.ct = (a->bs + kRgChannels - 1) / kRgChannels;
  p.kc = (a->bs + 63) / 64;
  const int units = p.blocks * p.ct;
  CUtensorMap tm;
  rc = cached_kmajor_tmap(&tm, a->gate_tiles, 2, static_cast<long long>(units) * 2 * kRgChannels, p.kc * 64, p.kc * 128, kRgChannels);
  if (rc != SLLM_OK) return rc;
  const size_t smem = static_cast<size_t>(p.kc) * (2 * kRgChannels + 2 * (a->decode ? kRgDecodeRows : kRgTokens)) * 128 + sizeof(RglruShared) + 1024;
  static size_t cfg[2] = {0, 0};
  auto* kernel = a->decode ? rglru_tile_kernel<true> : rglru_tile_kernel<false>;
  if (smem > cfg[a->decode ? 1 : 0]) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
      return SLLM_ERR_CUDA;
    cfg[a->decode ? 1 : 0] = smem;
  }
  int gy = 148 / units;                              // one CTA per SM, each with its share of the tiles
  if (gy < 1) gy = 1;
  if (gy > p.n_tiles) gy = p.n_tiles;
  if (gy > 65535 || p.n_tiles > 65535) return SLLM_ERR_LIMIT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (launch_kernel(kernel, dim3(units, gy), dim3(256), smem, st, 1u, tm, p) != cudaSuccess) return SLLM_ERR_CUDA;
  if (a->decode) return SLLM_OK;
  return launch_kernel(rglru_finish_kernel, dim3((p.width + 255) / 256, p.n_tiles), dim3(256), 0, st, 1u, p) == cudaSuccess
             ? SLLM_OK : SLLM_ERR_CUDA;
}

// Any-size form on the CUDA cores: gate_r / gate_i [blocks, bs, bs] in the type of proj; h / prod [tokens, width] floats.
SLLM_EXPORT int sllm_rglru_simt(const SllmRglru* a, void* stream) {
  RglruParams p;
  const int rc = rglru_params(a, &p);
  if (rc != SLLM_OK) return rc;
  if (!a->gate_r || !a->gate_i || !a->h || !a->prod || !a->row_off || !a->seq_index) return SLLM_ERR_INVALID_ARGUMENT;
  const size_t smem = sizeof(float) * kRgRows * a->bs;
  if (smem > 48 * 1024 || a->blocks > 65535 || a->sequences > 65535) return SLLM_ERR_UNSUPPORTED_SHAPE;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 g1((p.tokens + kRgRows - 1) / kRgRows, p.blocks), g2((p.width + 127) / 128, p.sequences);
  cudaError_t e = a->fp32 ? launch_kernel(rglru_terms_kernel<float>, g1, dim3(128), smem, st, 1u, p)
                          : launch_kernel(rglru_terms_kernel<__nv_bfloat16>, g1, dim3(128), smem, st, 1u, p);
  if (e != cudaSuccess) return SLLM_ERR_CUDA;
  e = a->fp32 ? launch_kernel(rglru_scan_kernel<float>, g2, dim3(128), 0, st, 1u, p)
              : launch_kernel(rglru_scan_kernel<__nv_bfloat16>, g2, dim3(128), 0, st, 1u, p);
  return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}
