// Latent attention of long prompt portions in the expanded form, on the 5th-generation tensor cores.
//
// The latents that a portion's queries may see (its own tokens and, for a later portion, the earlier ones from the pages)
// are gathered into contiguous rows, one GEMM expands them to every head's keys and values, and a flash-attention kernel
// runs over the expanded rows: 2 (dim + rot_dim) + 2 vdim flops per (query, key, head) instead of the absorbed form's
// 2 (kv_rank + rot_dim) + 2 kv_rank.
//
//   latent_gather_kernel   pages -> [context rows, kv_rank] and [context rows, rotated part padded to 64]
//   latent_pack_q_kernel   q -> [tokens, heads, unrotated padded to 64 | rotated padded to 64], rotation applied; the
//                          padding is zero, so key columns that a 64-wide box reads beyond a head's own do not count
//   latent_prefill_kernel  see below; it also serves ordinary keys and values gathered from their pages (kv_attention.cu),
//                          with fewer key / value heads than query heads, attention sinks and a gate per output channel
#include "typed.cuh"
#include "attention_common.cuh"
#include "api.h"
#include "tmap.h"

namespace sllm {

// ---------------------------------------------------------------- gather
// spans: [sequences][4] = {row of the block table, first context position, context rows, first gathered row}.
// grid (ceil(longest context / 8), sequences), 8 warps: a warp per row.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const __nv_bfloat16* __restrict__ pages, int ld, int page_size, const int* __restrict__ block_table,
                     int max_blocks, const int* __restrict__ spans, __nv_bfloat16* __restrict__ c_out,
                     __nv_bfloat16* __restrict__ r_out, int kv_rank, int rot_dim, int rot_pad) {
  pdl_wait();
  pdl_trigger();
  const int* sp = spans + 4 * blockIdx.y;
  const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= sp[2]) return;
  const int pos = sp[1] + i;
  const __nv_bfloat16* src =
      pages + (static_cast<size_t>(block_table[static_cast<size_t>(sp[0]) * max_blocks + pos / page_size]) * page_size + pos % page_size) * ld;
  const size_t row = static_cast<size_t>(sp[3]) + i;
  for (int e = lane * 8; e < kv_rank; e += 256) *reinterpret_cast<uint4*>(c_out + row * kv_rank + e) = *reinterpret_cast<const uint4*>(src + e);
  for (int e = lane; e < rot_pad; e += 32) r_out[row * rot_pad + e] = e < rot_dim ? src[kv_rank + e] : __float2bfloat16_rn(0.f);
}

// ---------------------------------------------------------------- query packing
// grid (tokens), 256 threads; a token's angles are computed once for all heads.  dim, dim_pad and rot_pad are multiples of 8.
__global__ void __launch_bounds__(256)
latent_pack_q_kernel(const __nv_bfloat16* __restrict__ q, long long ldq, __nv_bfloat16* __restrict__ out, int heads, int dim,
                     int rot_dim, int dim_pad, int rot_pad, const int* __restrict__ positions, const float* __restrict__ inv_freq,
                     int rot_dims, int interleaved, int vec) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float2 cs[];                     // [rot_dims / 2] = {cos, sin}
  const int t = blockIdx.x, half = rot_dims >> 1, width = dim_pad + rot_pad;
  const float pos = static_cast<float>(positions[t]);
  for (int i = threadIdx.x; i < half; i += 256) {
    float sn, c;
    sincosf(pos * inv_freq[i], &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  const __nv_bfloat16* src = q + t * ldq;
  __nv_bfloat16* dst = out + static_cast<size_t>(t) * heads * width;
  const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);
  const int pieces = dim_pad >> 3;
  for (int e = threadIdx.x; e < heads * pieces; e += 256) {
    const int h = e / pieces, i = (e - h * pieces) * 8;
    const __nv_bfloat16* s = src + h * (dim + rot_dim) + i;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (i < dim) {
      if (vec) {
        v = *reinterpret_cast<const uint4*>(s);
      } else {
        __nv_bfloat16* x = reinterpret_cast<__nv_bfloat16*>(&v);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = s[j];
      }
    }
    *reinterpret_cast<uint4*>(dst + h * width + i) = v;
  }
  __syncthreads();
  const int pairs = rot_pad >> 1;                    // pairs of neighbouring output channels
  for (int e = threadIdx.x; e < heads * pairs; e += 256) {
    const int h = e / pairs, i = (e - h * pairs) * 2;
    const __nv_bfloat16* s = src + h * (dim + rot_dim) + dim;
    __nv_bfloat162 o;
    if (interleaved && i < rot_dims) {
      const float u = __bfloat162float(s[i]), v = __bfloat162float(s[i + 1]);
      const float2 c = cs[i >> 1];
      o = __floats2bfloat162_rn(u * c.x - v * c.y, v * c.x + u * c.y);
    } else {
      __nv_bfloat16 x[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int k = i + j;
        if (k >= rot_dims) {
          x[j] = k < rot_dim ? s[k] : zero;
        } else {
          const int fi = k < half ? k : k - half;
          const float u = __bfloat162float(s[fi]), v = __bfloat162float(s[fi + half]);
          x[j] = __float2bfloat16_rn(k < half ? u * cs[fi].x - v * cs[fi].y : v * cs[fi].x + u * cs[fi].y);
        }
      }
      o = __halves2bfloat162(x[0], x[1]);
    }
    *reinterpret_cast<__nv_bfloat162*>(dst + h * width + dim_pad + i) = o;
  }
}

// ---------------------------------------------------------------- attention
// One CTA = (128-row query tile, head); 384 threads:
//   warp 0      TMA producer: Q once, then per 128-key tile the K chunks (a head's unrotated columns of the expanded rows,
//               then the shared rotated part) and the V chunks; chunks are [128 rows x 64 channels], 128-byte swizzle
//   warps 1, 2  S = Q K^T of even / odd key tiles, each with its own K stage and TMEM accumulator, so the next scores are
//               computed while the softmax works on the current ones (warp 1 also owns the TMEM)
//   warp 3      PV = P V
//   warps 4-11  softmax: two threads per query row, 64 keys each; row maxima meet in shared memory, P goes to shared
//               memory as the bf16 K-major operand, each thread folds half of the value columns into registers
// Causal with any offset between queries and context, optional sliding window (key tiles outside it are not visited).
// kRich adds chunks of positions, distance slopes, distance biases (a head's table in shared memory where it fits), and windows whose first `keep_first` positions stay visible: a tile that
// lies past those walks two runs of key tiles, the kept positions and the window.
constexpr int kLpThreads = 384;
constexpr int kLpTile = 128;
constexpr int kLpChunk = kLpTile * 128;

struct LatentPrefillParams {
  const int* tiles;          // [tiles][8]: query row, rows, position of the first row, context row, its position, context row
                             // of position 0 (with kept positions), -, -
  int heads, kv_heads, dim, vdim, dim_chunks, v_stages, window, keep_first, chunk;
  float scale_log2;
  const float* slopes;       // optional [heads]: taken off a score per position of distance
  DistanceBias dist;         // what joins a score by its distance
  int dist_smem;             // bytes of a head's table in shared memory (0: it is read where it is)
  const float* sinks;        // optional [heads]: scores that join the denominator only
  const __nv_bfloat16* gate; // optional logits [tokens, ld_gate], one per head or (gate_channels) per output channel
  long long ld_gate;
  int gate_channels;
  __nv_bfloat16* out;        // [tokens, heads * vdim]
  int* status;
};

struct __align__(16) LatentPrefillShared {
  uint64_t q_full;
  uint64_t k_full[2];
  uint64_t k_empty[2];
  uint64_t v_full[2];
  uint64_t v_empty[2];
  uint64_t s_full[2];
  uint64_t p_ready[2];
  uint64_t o_full[2];
  uint32_t tmem_base;
  int abort_flag;
  float red[2][2][kLpTile];
};

// MN-major operand: rows = K index, 128-byte rows of 64 contiguous MN elements, MN blocks `mn_block_stride` bytes apart.
__device__ __forceinline__ uint64_t lp_desc_mn(uint32_t smem_addr, uint32_t mn_block_stride) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>((mn_block_stride >> 4) & 0x3FFF) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
__device__ __forceinline__ float lp_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void lp_bar_softmax() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// kNQ: 64-channel chunks of a query / key row; kNV: of a value row.
template <int kNQ, int kNV, bool kRich>
__global__ void __launch_bounds__(kLpThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv,
                      const __grid_constant__ CUtensorMap tm_r, const LatentPrefillParams p) {
  pdl_wait();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;
  uint8_t* p_s = q_s + kNQ * kLpChunk;
  uint8_t* k_s = p_s + 2 * kLpChunk;                 // [2][kNQ]
  uint8_t* v_s = k_s + 2 * kNQ * kLpChunk;           // [v_stages][kNV]
  LatentPrefillShared* sh = reinterpret_cast<LatentPrefillShared*>(v_s + p.v_stages * kNV * kLpChunk);
  float* dist_s = reinterpret_cast<float*>(sh + 1);
  constexpr uint32_t kTmemCols = 512;                // S at columns 0 and 128, PV at 256
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y, kvh = head / (p.heads / p.kv_heads);
  const int* tile = p.tiles + 8 * blockIdx.x;
  const int q_row = tile[0], rows = tile[1], q0 = tile[2], k_lo = tile[4];
  // first visible position of the tile's rows; with kept positions, those below `kept` take `kept_tiles` key tiles of their own
  int first = p.window > 0 ? max(k_lo, q0 - p.window + 1) : kRich && p.chunk > 0 ? max(k_lo, q0 / p.chunk * p.chunk) : k_lo;
  int kept = 0;
  if (kRich && p.keep_first > 0) {
    if (first > p.keep_first) kept = p.keep_first;
    else first = k_lo;                               // 0: the rows are gathered from the start
  }
  const int kept_tiles = kRich ? (kept + kLpTile - 1) / kLpTile : 0, kept_row = tile[5];
  const int c_row = tile[3] + first - k_lo - kept_tiles * kLpTile;
  const int nt = kept_tiles + (q0 + rows - first + kLpTile - 1) / kLpTile;
  volatile int* abort_flag = &sh->abort_flag;
  if (threadIdx.x == 0) {
    mbar_init(&sh->q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&sh->k_full[s], 1);
      mbar_init(&sh->k_empty[s], 1);
      mbar_init(&sh->v_full[s], 1);
      mbar_init(&sh->v_empty[s], 1);
      mbar_init(&sh->s_full[s], 1);
      mbar_init(&sh->p_ready[s], 256);
      mbar_init(&sh->o_full[s], 1);
    }
    sh->abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_kv);
    tma_prefetch_desc(&tm_r);
  }
  if (warp == 1) {
    tmem_alloc(&sh->tmem_base, kTmemCols);
    tmem_relinquish();
  }
  if constexpr (kRich) {
    if (p.dist_smem > 0) {
      const float* src = p.dist.head(head) - kDistFront;
      for (int i = threadIdx.x; i < p.dist_smem / 4; i += kLpThreads) dist_s[i] = src[i];
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = sh->tmem_base;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(&sh->q_full, kNQ * kLpChunk);
      for (int c = 0; c < kNQ; ++c)
        tma_load_2d(q_s + c * kLpChunk, &tm_q, &sh->q_full, (head * kNQ + c) * 64, q_row);
      int ks = 0, vs = 0;
      for (int j = 0; j < nt; ++j) {
        const int y = (j < kept_tiles ? kept_row : c_row) + j * kLpTile, st = j & 1, sv = j % p.v_stages;
        if (!mbar_wait(&sh->k_empty[st], ((j >> 1) & 1) ^ 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_SMEM_EMPTY)) break;
        mbar_expect_tx(&sh->k_full[st], kNQ * kLpChunk);
        for (int c = 0; c < kNQ; ++c) {
          uint8_t* dst = k_s + (st * kNQ + c) * kLpChunk;
          if (c < p.dim_chunks) tma_load_2d(dst, &tm_kv, &sh->k_full[st], kvh * p.dim + c * 64, y);
          else tma_load_2d(dst, &tm_r, &sh->k_full[st], (c - p.dim_chunks) * 64, y);
        }
        ks = j + 1;
        if (!mbar_wait(&sh->v_empty[sv], ((j / p.v_stages) & 1) ^ 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_SMEM_EMPTY)) break;
        mbar_expect_tx(&sh->v_full[sv], kNV * kLpChunk);
        for (int c = 0; c < kNV; ++c)
          tma_load_2d(v_s + (sv * kNV + c) * kLpChunk, &tm_kv, &sh->v_full[sv], p.kv_heads * p.dim + kvh * p.vdim + c * 64, y);
        vs = j + 1;
      }
      // every copy has landed before the CTA may leave
      int dummy = 0;
      mbar_wait(&sh->q_full, 0, &dummy, p.status, SLLM_DEV_TIMEOUT_DRAIN, 200000000LL);
      for (int j = max(0, ks - 2); j < ks; ++j)
        mbar_wait(&sh->k_full[j & 1], (j >> 1) & 1, &dummy, p.status, SLLM_DEV_TIMEOUT_DRAIN, 200000000LL);
      for (int j = max(0, vs - p.v_stages); j < vs; ++j)
        mbar_wait(&sh->v_full[j % p.v_stages], (j / p.v_stages) & 1, &dummy, p.status, SLLM_DEV_TIMEOUT_DRAIN, 200000000LL);
    }
  } else if (warp == 1 || warp == 2) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(kFmtBf16, 128, 128, 0, 0);
      const int par = warp - 1;
      const uint32_t q_addr = smem_u32(q_s), k_addr = smem_u32(k_s + par * kNQ * kLpChunk);
      bool ok = mbar_wait(&sh->q_full, 0, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMA_FULL);
      for (int j = par; ok && j < nt; j += 2) {
        if (!mbar_wait(&sh->k_full[par], (j >> 1) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMA_FULL)) break;
        // the accumulator is free once the softmax has read S(j - 2), which it does before p_ready(j - 2)
        if (j >= 2 && !mbar_wait(&sh->p_ready[par], ((j - 2) >> 1) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMEM_EMPTY)) break;
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < kNQ; ++c)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_f16(tmem_base + par * 128, make_smem_desc_sw128(q_addr + c * kLpChunk) + 2 * k,
                     make_smem_desc_sw128(k_addr + c * kLpChunk) + 2 * k, idesc, (c | k) != 0);
        tc_commit(&sh->s_full[par]);
        tc_commit(&sh->k_empty[par]);
      }
    }
  } else if (warp == 3) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(kFmtBf16, 128, kNV * 64, 0, 1);
      const uint32_t p_addr = smem_u32(p_s);
      for (int j = 0; j < nt; ++j) {
        const int sv = j % p.v_stages;
        if (!mbar_wait(&sh->v_full[sv], (j / p.v_stages) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMA_FULL)) break;
        if (!mbar_wait(&sh->p_ready[j & 1], (j >> 1) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMEM_EMPTY)) break;
        tc_fence_after();
        const uint32_t v_addr = smem_u32(v_s + sv * kNV * kLpChunk);
#pragma unroll
        for (int c = 0; c < 2; ++c)          // P chunk c holds keys [64 c, 64 c + 64)
#pragma unroll
          for (int k = 0; k < 4; ++k)        // 16 keys per MMA
            umma_f16(tmem_base + 256, make_smem_desc_sw128(p_addr + c * kLpChunk) + 2 * k,
                     lp_desc_mn(v_addr + (c * 64 + k * 16) * 128, kLpChunk), idesc, (c | k) != 0);
        tc_commit(&sh->o_full[j & 1]);
        tc_commit(&sh->v_empty[sv]);
      }
    }
  } else {
    const int qd = warp & 3, half = (warp - 4) >> 2;
    const int r = qd * 32 + lane, qpos = q0 + r;
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(qd * 32) << 16);
    constexpr int kO = kNV * 32;                     // value columns of this thread
    float o[kO];
#pragma unroll
    for (int i = 0; i < kO; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f, alpha_prev = 0.f;
    bool ok = true;
    const float slope = kRich && p.slopes ? p.slopes[head] * 1.4426950408889634f : 0.f;
    const float mul = kRich && (p.slopes || p.dist.table) ? 1.f : p.scale_log2;   // scores that something joins are scaled before the mask
    const float* dist = !kRich || !p.dist.table ? nullptr : p.dist_smem > 0 ? dist_s + kDistFront : p.dist.head(head);
    auto fold = [&](int j) {                         // o <- o * alpha(j) + PV(j)
      if (ok) ok = mbar_wait(&sh->o_full[j & 1], (j >> 1) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMEM_FULL);
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < kO / 16; ++c) {
        uint32_t v[16];
        tmem_ld16(lane_addr + 256 + half * kO + c * 16, v);
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) o[c * 16 + i] = fmaf(o[c * 16 + i], alpha_prev, __uint_as_float(v[i]));
      }
      tc_fence_before();
    };
    for (int j = 0; j < nt; ++j) {
      // a thread that gives up keeps in step with the barriers of the other softmax threads
      if (ok) ok = mbar_wait(&sh->s_full[j & 1], (j >> 1) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMEM_FULL);
      tc_fence_after();
      float s[64];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t v[16];
        tmem_ld16(lane_addr + (j & 1) * 128 + half * 64 + c * 16, v);
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) s[c * 16 + i] = __uint_as_float(v[i]);
      }
      const int k0 = (j < kept_tiles ? 0 : first - kept_tiles * kLpTile) + j * kLpTile;
      if constexpr (kRich) {
        if (p.slopes) {
          const float d0 = static_cast<float>(k0 + half * 64 - qpos);
#pragma unroll
          for (int i = 0; i < 64; ++i) s[i] = fmaf(s[i], p.scale_log2, slope * (d0 + static_cast<float>(i)));
        }
        if (dist) {                                  // entries outside the row belong to keys that are masked below
          const float* b = dist + min(q0 - k0, p.dist.n - 1 + kLpTile) + r - half * 64;
#pragma unroll
          for (int i = 0; i < 64; ++i) s[i] = fmaf(s[i], p.scale_log2, b[-i] * 1.4426950408889634f);
        }
        // keys [lo, hi] of this thread's 64 are visible, and those before `head_keys`
        int hi = 64, lo = 0, head_keys = 0;
        if (j < kept_tiles) {
          hi = kept - 1 - (k0 + half * 64);          // all kept positions precede the tile's rows
        } else {
          hi = qpos - (k0 + half * 64);
          lo = p.window > 0 ? hi - p.window + 1 : p.chunk > 0 ? hi - qpos % p.chunk : 0;
          if (kept == 0) head_keys = p.keep_first - (k0 + half * 64);
        }
        if (hi < 63 || lo > 0) {
#pragma unroll
          for (int i = 0; i < 64; ++i) s[i] = i > hi || (i < lo && i >= head_keys) ? -INFINITY : s[i];
        }
      } else if (k0 + kLpTile - 1 > q0 || (p.window > 0 && k0 <= q0 + kLpTile - 1 - p.window)) {
        const int hi = qpos - (k0 + half * 64);      // keys [lo, hi] of this thread's 64 are visible
        const int lo = p.window > 0 ? hi - p.window + 1 : 0;
#pragma unroll
        for (int i = 0; i < 64; ++i) s[i] = i > hi || i < lo ? -INFINITY : s[i];
      }
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 64; ++i) mx[i & 3] = fmaxf(mx[i & 3], s[i]);
      const float tmax = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
      sh->red[j & 1][half][r] = tmax;
      lp_bar_softmax();
      const float m_new = fmaxf(m, fmaxf(tmax, sh->red[j & 1][half ^ 1][r]) * mul);
      const float m_use = m_new == -INFINITY ? 0.f : m_new;
      const float alpha = m == -INFINITY ? 0.f : lp_ex2(m - m_use);
      if (j > 0) fold(j - 1);                        // P(j - 1) has been consumed: its buffer is free
      float sum[2] = {0.f, 0.f};
      uint8_t* rowp = p_s + half * kLpChunk + r * 128;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        uint32_t w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const __nv_bfloat162 h = __floats2bfloat162_rn(lp_ex2(fmaf(s[u * 8 + 2 * i], mul, -m_use)),
                                                         lp_ex2(fmaf(s[u * 8 + 2 * i + 1], mul, -m_use)));
          // the normaliser sums the rounded values, which are what the product multiplies
          sum[0] += __bfloat162float(h.x);
          sum[1] += __bfloat162float(h.y);
          w[i] = *reinterpret_cast<const uint32_t*>(&h);
        }
        *reinterpret_cast<uint4*>(rowp + ((u ^ (r & 7)) << 4)) = make_uint4(w[0], w[1], w[2], w[3]);
      }
      l = l * alpha + sum[0] + sum[1];
      m = m_new;
      alpha_prev = alpha;
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(&sh->p_ready[j & 1]);
    }
    fold(nt - 1);
    sh->red[nt & 1][half][r] = l;                    // the other parity's buffer was last read before tile nt - 1's barrier
    lp_bar_softmax();
    float total = l + sh->red[nt & 1][half ^ 1][r];
    if (p.sinks) total += lp_ex2(p.sinks[head] * 1.4426950408889634f - m);
    if (ok && r < rows) {
      float inv = total > 0.f ? 1.f / total : 0.f;
      const long long t = q_row + r;
      const bool per_channel = p.gate && p.gate_channels;
      if (p.gate && !p.gate_channels) inv *= sigmoid_f(__bfloat162float(p.gate[t * p.ld_gate + head]));
      const __nv_bfloat16* gate = p.gate + t * p.ld_gate + head * p.vdim;
      __nv_bfloat16* dst = p.out + (t * p.heads + head) * p.vdim;
#pragma unroll
      for (int i = 0; i < kO; i += 8) {
        if (half * kO + i < p.vdim) {
          uint4 w;
          __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&w);
          float g[8];
          if (per_channel) ld16(gate + half * kO + i, g);
#pragma unroll
          for (int k = 0; k < 8; ++k) g[k] = per_channel ? inv / (1.f + __expf(-g[k])) : inv;
#pragma unroll
          for (int k = 0; k < 4; ++k) h[k] = __floats2bfloat162_rn(o[i + 2 * k] * g[2 * k], o[i + 2 * k + 1] * g[2 * k + 1]);
          *reinterpret_cast<uint4*>(dst + half * kO + i) = w;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

template <int kNQ, int kNV, bool kRich>
static int latent_prefill_go(const CUtensorMap& tq, const CUtensorMap& tkv, const CUtensorMap& tr, LatentPrefillParams p,
                                 int tiles, cudaStream_t st) {
  // two V stages where they fit; at least 120 KB, so that one CTA (which takes the whole TMEM) is on an SM at a time
  p.v_stages = (3 * kNQ + 2 + 2 * kNV) * kLpChunk <= 208 * 1024 ? 2 : 1;
  size_t smem = static_cast<size_t>(3 * kNQ + 2 + p.v_stages * kNV) * kLpChunk + sizeof(LatentPrefillShared) + 1024;
  if (kRich && p.dist.table) {                       // distances up to the window's, and what a tile reads beyond
    const int n = p.window > 0 && p.keep_first == 0 && p.window < p.dist.n ? p.window : p.dist.n;
    const int bytes = (kDistFront + n + kDistBack) * 4;
    if (smem + bytes <= 227 * 1024) {
      p.dist_smem = bytes;
      smem += bytes;
    }
  }
  if (smem < 120 * 1024) smem = 120 * 1024;
  static size_t configured = 0;
  if (smem > configured) {
    if (cudaFuncSetAttribute(latent_prefill_kernel<kNQ, kNV, kRich>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) !=
        cudaSuccess)
      return SLLM_ERR_CUDA;
    configured = smem;
  }
  return launch_kernel(latent_prefill_kernel<kNQ, kNV, kRich>, dim3(tiles, p.heads), dim3(kLpThreads), smem, st, 1u, tq, tkv, tr, p) ==
                 cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

template <int kNQ, int kNV>
static int latent_prefill_launch(const CUtensorMap& tq, const CUtensorMap& tkv, const CUtensorMap& tr, const LatentPrefillParams& p,
                                 int tiles, cudaStream_t st) {
  return p.keep_first > 0 || p.chunk > 0 || p.slopes || p.dist.table ? latent_prefill_go<kNQ, kNV, true>(tq, tkv, tr, p, tiles, st)
                                                     : latent_prefill_go<kNQ, kNV, false>(tq, tkv, tr, p, tiles, st);
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_latent_gather(const void* pages, int ld, int page_size, const int* block_table, int max_blocks, const int* spans,
                                   int sequences, int longest, void* c_out, void* r_out, int kv_rank, int rot_dim, int rot_pad,
                                   void* stream) {
  if (!pages || !block_table || !spans || !c_out || !r_out || sequences <= 0 || longest <= 0 || page_size <= 0 || kv_rank <= 0 ||
      rot_dim < 0 || rot_pad < rot_dim)
    return SLLM_ERR_INVALID_ARGUMENT;
  if ((kv_rank & 7) || (ld & 7) || sequences > 65535) return SLLM_ERR_UNSUPPORTED_SHAPE;
  if ((reinterpret_cast<uintptr_t>(pages) | reinterpret_cast<uintptr_t>(c_out)) & 15) return SLLM_ERR_ALIGNMENT;
  return launch_kernel(latent_gather_kernel, dim3((longest + 7) / 8, sequences), dim3(256), 0, static_cast<cudaStream_t>(stream), 1u,
                       static_cast<const __nv_bfloat16*>(pages), ld, page_size, block_table, max_blocks, spans,
                       static_cast<__nv_bfloat16*>(c_out), static_cast<__nv_bfloat16*>(r_out), kv_rank, rot_dim, rot_pad) ==
                 cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

SLLM_EXPORT int sllm_latent_pack_q(const void* q, long long ldq, void* out, int tokens, int heads, int dim, int rot_dim, int dim_pad,
                                   int rot_pad, const int* positions, const float* inv_freq, int rot_dims, int interleaved,
                                   void* stream) {
  if (!q || !out || !positions || tokens <= 0 || heads <= 0 || heads > 65535 || dim <= 0 || rot_dim < 0 || dim_pad < dim ||
      rot_pad < rot_dim || rot_dims > rot_dim || (rot_dims & 1) || (rot_dims > 0 && !inv_freq))
    return SLLM_ERR_INVALID_ARGUMENT;
  if ((dim & 7) || (dim_pad & 7) || (rot_pad & 7) || rot_dims > 4096) return SLLM_ERR_UNSUPPORTED_SHAPE;
  const int vec = (ldq & 7) == 0 && (rot_dim & 7) == 0 && (reinterpret_cast<uintptr_t>(q) & 15) == 0;
  return launch_kernel(latent_pack_q_kernel, dim3(tokens), dim3(256), sizeof(float2) * (rot_dims / 2 + 1), static_cast<cudaStream_t>(stream),
                       1u, static_cast<const __nv_bfloat16*>(q), ldq, static_cast<__nv_bfloat16*>(out), heads, dim, rot_dim, dim_pad,
                       rot_pad, positions, inv_freq, rot_dims, interleaved, vec) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

static int latent_prefill_impl(const void* q, int tokens, const void* kv, const void* r, int context, const int* tiles, int num_tiles,
                               int rot_dim, LatentPrefillParams p, cudaStream_t st) {
  const int dim = p.dim, vdim = p.vdim;
  const int nd = (dim + 63) / 64, nr = (rot_dim + 63) / 64, nq = nd + nr, nv = (vdim + 63) / 64;
  if (nq < 1 || nq > 3 || nv > 2 || (dim & 7) || (vdim & 7)) return SLLM_ERR_UNSUPPORTED_SHAPE;
  if (reinterpret_cast<uintptr_t>(p.out) & 15) return SLLM_ERR_ALIGNMENT;
  const long long wq = static_cast<long long>(p.heads) * nq * 64, wkv = static_cast<long long>(p.kv_heads) * (dim + vdim);
  CUtensorMap tq, tkv, tr;
  int rc = cached_kmajor_tmap(&tq, q, 2, tokens, wq, wq * 2, kLpTile);
  if (rc == SLLM_OK) rc = cached_kmajor_tmap(&tkv, kv, 2, context, wkv, wkv * 2, kLpTile);
  if (rc == SLLM_OK) rc = nr > 0 ? cached_kmajor_tmap(&tr, r, 2, context, nr * 64, nr * 128, kLpTile) : (tr = tkv, SLLM_OK);
  if (rc != SLLM_OK) return rc;
  p.tiles = tiles; p.dim_chunks = nd;
  switch (nq * 2 + nv - 1) {
    case 2: return latent_prefill_launch<1, 1>(tq, tkv, tr, p, num_tiles, st);
    case 3: return latent_prefill_launch<1, 2>(tq, tkv, tr, p, num_tiles, st);
    case 4: return latent_prefill_launch<2, 1>(tq, tkv, tr, p, num_tiles, st);
    case 5: return latent_prefill_launch<2, 2>(tq, tkv, tr, p, num_tiles, st);
    case 6: return latent_prefill_launch<3, 1>(tq, tkv, tr, p, num_tiles, st);
    default: return latent_prefill_launch<3, 2>(tq, tkv, tr, p, num_tiles, st);
  }
}

// q: packed [tokens, heads, (dim chunks + rot chunks) * 64]; kv: [context rows, heads * (dim + vdim)] (all heads' keys, then
// all heads' values); r: [context rows, rot chunks * 64]; tiles: [num_tiles][8], see LatentPrefillParams; gate per head.
SLLM_EXPORT int sllm_latent_prefill(const void* q, int tokens, const void* kv, const void* r, int context, const int* tiles,
                                    int num_tiles, int heads, int dim, int rot_dim, int vdim, int window, float scale,
                                    const void* gate, long long ld_gate, void* out, int* status, void* stream) {
  if (!q || !kv || !r || !tiles || !out || tokens <= 0 || context <= 0 || num_tiles <= 0 || heads <= 0 || heads > 65535 || dim <= 0 ||
      rot_dim < 0 || vdim <= 0 || window < 0)
    return SLLM_ERR_INVALID_ARGUMENT;
  LatentPrefillParams p = {};
  p.heads = p.kv_heads = heads; p.dim = dim; p.vdim = vdim; p.window = window; p.scale_log2 = scale * 1.4426950408889634f;
  p.gate = static_cast<const __nv_bfloat16*>(gate); p.ld_gate = ld_gate; p.out = static_cast<__nv_bfloat16*>(out); p.status = status;
  return latent_prefill_impl(q, tokens, kv, r, context, tiles, num_tiles, rot_dim, p, static_cast<cudaStream_t>(stream));
}

// The same kernel over ordinary keys and values: q [tokens, heads, dim padded to 64 with zeros]; kv [context rows, kv_heads *
// (dim + vdim)]; sinks, slopes: optional [heads]; dist: see DistanceBias, its back part included; gate: optional logits [tokens, ld_gate], one per output channel
// (gate_heads: per head).
SLLM_EXPORT int sllm_kv_prefill(const void* q, int tokens, const void* kv, int context, const int* tiles, int num_tiles, int heads,
                                int kv_heads, int dim, int vdim, int window, int keep_first, int chunk, const float* slopes,
                                const float* dist, int n_dist, int ld_dist, float scale, const float* sinks, const void* gate,
                                long long ld_gate, int gate_heads, void* out, int* status, void* stream) {
  if (!q || !kv || !tiles || !out || tokens <= 0 || context <= 0 || num_tiles <= 0 || heads <= 0 || heads > 65535 || kv_heads <= 0 ||
      heads % kv_heads || dim <= 0 || vdim <= 0 || window < 0 || keep_first < 0 || chunk < 0 || (keep_first > 0 && window == 0) ||
      (chunk > 0 && window > 0))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (dist && (slopes || n_dist < 1 || ld_dist < kDistFront + n_dist + kDistBack)) return SLLM_ERR_INVALID_ARGUMENT;
  if (gate && !gate_heads && ((ld_gate & 7) || (reinterpret_cast<uintptr_t>(gate) & 15))) return SLLM_ERR_ALIGNMENT;
  LatentPrefillParams p = {};
  p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.window = window; p.scale_log2 = scale * 1.4426950408889634f;
  p.sinks = sinks; p.gate = static_cast<const __nv_bfloat16*>(gate); p.ld_gate = ld_gate; p.gate_channels = !gate_heads;
  p.keep_first = keep_first; p.chunk = chunk; p.slopes = slopes; p.dist = {dist, n_dist, ld_dist};
  p.out = static_cast<__nv_bfloat16*>(out); p.status = status;
  return latent_prefill_impl(q, tokens, kv, nullptr, context, tiles, num_tiles, 0, p, static_cast<cudaStream_t>(stream));
}
