// Routed experts with bf16 (or fp32) weights: one product over the rows of every expert, rows grouped by expert
// (tok_off, moe_permute), with the expert's activation or the routing weight in the epilogue.
//
//   mode 0   y[p, f] = g sigmoid(alpha g) (u + shift),  g = min(gate row f . x, limit),  u = clamp(up row f . x, +-limit)
//   mode 1   y[p, n] = row_w[p] (row n . x)
//
// Weights are [experts * n_rows, K]; in mode 0 rows come in blocks of 128: 64 gate rows, then the up rows of the same 64
// features (zero rows pad the last block), so that both meet in one output tile.
//
//   grouped_gemm_kernel        tcgen05, bf16: D[token, weight row]; A = rows of x in tiles of kRows tokens, B = weights.
//                              kRows 32: decode batches (a tile of A is a quarter of the operand, the other rows of D are
//                              not read), kRows 128: prompts.  One thread of the epilogue owns one token.
//   grouped_gemm_simt_kernel   fp32, or rows that a TMA copy cannot address; reads its rows through `src`
//
// The tile -> (expert, rows) map is derived from tok_off in every CTA: the launch covers the largest number of tiles that
// the rows can form, CTAs past the last tile leave at once.
#include "typed.cuh"
#include "api.h"
#include "tmap.h"

namespace sllm {

constexpr int kGgThreads = 192, kGgMaxStages = 8;

struct GroupedParams {
  const int* tok_off;        // [experts + 1]
  const int* src;            // simt: row of x of every permuted row (null: the row itself)
  const float* row_w;        // mode 1: [rows]
  const void *x, *w;         // simt
  void* y;
  int* status;
  int experts, n_rows, k, kb, stages, mode, ldy, ldx, features;   // features: output columns
  float limit, alpha, shift;
};

struct __align__(16) GroupedShared {
  uint64_t full[kGgMaxStages], empty[kGgMaxStages], done;
  uint32_t tmem_base;
  int abort_flag;
  int expert, row0, rows;
};

// Warp-wide: tile number -> expert, first row and rows of the tile (rows 0: past the last tile).
__device__ __forceinline__ void grouped_find(const int* tok_off, int experts, int tile, int per, int lane, int& expert, int& row0,
                                             int& rows) {
  const int each = (experts + 31) / 32, e0 = lane * each;
  int count = 0;
  for (int e = e0; e < min(experts, e0 + each); ++e) count += (tok_off[e + 1] - tok_off[e] + per - 1) / per;
  int before = count;
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= o) before += v;
  }
  before -= count;
  int fe = -1, fr = 0, fn = 0;
  if (tile >= before && tile < before + count) {
    int at = before;
    for (int e = e0; e < min(experts, e0 + each); ++e) {
      const int n = tok_off[e + 1] - tok_off[e], t = (n + per - 1) / per;
      if (tile < at + t) {
        fe = e;
        fr = tok_off[e] + (tile - at) * per;
        fn = min(per, n - (tile - at) * per);
        break;
      }
      at += t;
    }
  }
  const unsigned who = __ballot_sync(0xffffffffu, fe >= 0);
  const int from = who ? __ffs(who) - 1 : 0;
  expert = __shfl_sync(0xffffffffu, fe, from);
  row0 = __shfl_sync(0xffffffffu, fr, from);
  rows = who ? __shfl_sync(0xffffffffu, fn, from) : 0;
}

__device__ __forceinline__ float gated_clamp(float g, float u, float limit, float alpha, float shift) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return __fdividef(g, 1.f + __expf(-alpha * g)) * (u + shift);      // 0 where the exponential overflows
}

template <int BN, int kRows>
__global__ void __launch_bounds__(kGgThreads)
grouped_gemm_kernel(const __grid_constant__ CUtensorMap tm_x, const __grid_constant__ CUtensorMap tm_w, const GroupedParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  // with 32-row tiles the operand's other rows are whatever follows in the stage; their sums are never read
  constexpr int kABytes = kRows * 128, kStage = kABytes + BN * 128;
  GroupedShared* sh = reinterpret_cast<GroupedShared*>(smem + p.stages * kStage);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  volatile int* abort_flag = &sh->abort_flag;
  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(&sh->full[s], 1);
      mbar_init(&sh->empty[s], 1);
    }
    mbar_init(&sh->done, 1);
    sh->abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_x);
    tma_prefetch_desc(&tm_w);
  }
  if (warp == 1) {
    tmem_alloc(&sh->tmem_base, BN);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_trigger();
  if (warp == 0) {
    int e, r, n;
    grouped_find(p.tok_off, p.experts, blockIdx.y, kRows, lane, e, r, n);
    if (lane == 0) {
      sh->expert = e;
      sh->row0 = r;
      sh->rows = n;
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = sh->tmem_base;
  const int rows = sh->rows, row0 = sh->row0, expert = sh->expert;
  if (rows > 0) {
    if (warp == 0) {
      if (lane == 0) {
        const int wy = expert * p.n_rows + blockIdx.x * BN;
        for (int i = 0; i < p.kb; ++i) {
          const int s = i % p.stages;
          if (i >= p.stages &&
              !mbar_wait(&sh->empty[s], ((i / p.stages) & 1) ^ 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_SMEM_EMPTY))
            break;
          uint8_t* st = smem + s * kStage;
          mbar_expect_tx(&sh->full[s], kStage);
#pragma unroll
          for (int b = 0; b < BN / 128; ++b) tma_load_2d(st + kABytes + b * 128 * 128, &tm_w, &sh->full[s], i * 64, wy + b * 128);
          tma_load_2d(st, &tm_x, &sh->full[s], i * 64, row0);
        }
        // the MMA issuer waits for every stage that was filled; when it gave up, drain here
        if (*abort_flag) {
          int dummy = 0;
          for (int s = 0; s < p.stages && s < p.kb; ++s)
            mbar_wait(&sh->full[s], ((p.kb - 1 - s) / p.stages) & 1, &dummy, p.status, SLLM_DEV_TIMEOUT_DRAIN, 200000000LL);
        }
      }
    } else if (warp == 1) {
      if (lane == 0) {
        constexpr uint32_t idesc = make_idesc(kFmtBf16, 128, BN);
        bool ok = true;
        for (int i = 0; i < p.kb; ++i) {
          const int s = i % p.stages;
          ok = mbar_wait(&sh->full[s], (i / p.stages) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMA_FULL);
          if (!ok) break;
          tc_fence_after();
          const uint32_t st = smem_u32(smem + s * kStage);
          const uint64_t da = make_smem_desc_sw128(st), db = make_smem_desc_sw128(st + kABytes);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16(tmem_base, da + 2 * k, db + 2 * k, idesc, (i | k) != 0);
          tc_commit(&sh->empty[s]);
        }
        if (ok) tc_commit(&sh->done);
      }
    } else if ((warp & 3) * 32 < kRows) {
      const int qd = warp & 3, r = qd * 32 + lane;
      const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(qd * 32) << 16);
      const float rw = p.mode == 1 && r < rows ? p.row_w[row0 + r] : 0.f;
      bool ok = mbar_wait(&sh->done, 0, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        tc_fence_after();
        __nv_bfloat16* y = static_cast<__nv_bfloat16*>(p.y) + static_cast<size_t>(row0 + r) * p.ldy;
        const bool in = r < rows;
        if (p.mode == 0) {
#pragma unroll
          for (int b = 0; b < BN / 128; ++b) {
            const int f0 = (blockIdx.x * (BN / 128) + b) * 64;
            if (f0 >= p.features) break;
#pragma unroll 1
            for (int c = 0; c < 64; c += 16) {
              uint32_t g[16], u[16];
              tmem_ld16(lane_addr + b * 128 + c, g);
              tmem_ld16(lane_addr + b * 128 + 64 + c, u);
              tmem_wait_ld();
              uint32_t o[8];
#pragma unroll
              for (int j = 0; j < 8; ++j) {
                const __nv_bfloat162 h = __floats2bfloat162_rn(
                    gated_clamp(__uint_as_float(g[2 * j]), __uint_as_float(u[2 * j]), p.limit, p.alpha, p.shift),
                    gated_clamp(__uint_as_float(g[2 * j + 1]), __uint_as_float(u[2 * j + 1]), p.limit, p.alpha, p.shift));
                o[j] = *reinterpret_cast<const uint32_t*>(&h);
              }
              if (in) {
                *reinterpret_cast<uint4*>(y + f0 + c) = make_uint4(o[0], o[1], o[2], o[3]);
                *reinterpret_cast<uint4*>(y + f0 + c + 8) = make_uint4(o[4], o[5], o[6], o[7]);
              }
            }
          }
        } else {
#pragma unroll 1
          for (int c = 0; c < BN; c += 16) {
            const int n0 = blockIdx.x * BN + c;
            if (n0 >= p.features) break;
            uint32_t v[16];
            tmem_ld16(lane_addr + c, v);
            tmem_wait_ld();
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              uint32_t o[4];
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                const __nv_bfloat162 x2 = __floats2bfloat162_rn(__uint_as_float(v[h * 8 + 2 * j]) * rw, __uint_as_float(v[h * 8 + 2 * j + 1]) * rw);
                o[j] = *reinterpret_cast<const uint32_t*>(&x2);
              }
              if (in && n0 + h * 8 < p.features) *reinterpret_cast<uint4*>(y + n0 + h * 8) = make_uint4(o[0], o[1], o[2], o[3]);
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, BN);
  }
}

// 64 rows x 64 weight rows (mode 0: 32 features) per CTA; 256 threads.
template <typename T>
__global__ void __launch_bounds__(256) grouped_gemm_simt_kernel(const GroupedParams p) {
  pdl_wait();
  pdl_trigger();
  constexpr int kT = 64, kK = 16;
  __shared__ float xs[kK][kT + 4], ws[kK][kT + 4];
  int expert, row0, rows;
  grouped_find(p.tok_off, p.experts, blockIdx.y, kT, threadIdx.x & 31, expert, row0, rows);
  if (rows == 0) return;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* w = static_cast<const T*>(p.w) + static_cast<size_t>(expert) * p.n_rows * p.k;
  auto weight_row = [&](int j) {                        // tile column -> weight row (-1: none)
    if (p.mode == 1) return static_cast<int>(blockIdx.x) * kT + j < p.n_rows ? static_cast<int>(blockIdx.x) * kT + j : -1;
    const int f = blockIdx.x * 32 + (j & 31);
    return f < p.features ? (f / 64) * 128 + f % 64 + (j >= 32 ? 64 : 0) : -1;
  };
  float acc[4][4] = {};                                 // rows ty * 4 + i, columns tx + 16 j
  for (int k0 = 0; k0 < p.k; k0 += kK) {
    for (int e = threadIdx.x; e < kT * kK; e += 256) {
      const int rr = e / kK, kk = e % kK, wr = weight_row(rr);
      const bool kin = k0 + kk < p.k;
      float xv = 0.f;
      if (kin && rr < rows) {
        const int row = p.src ? p.src[row0 + rr] : row0 + rr;
        xv = ld_f(static_cast<const T*>(p.x) + static_cast<size_t>(row) * p.ldx + k0 + kk);
      }
      xs[kk][rr] = xv;
      ws[kk][rr] = kin && wr >= 0 ? ld_f(w + static_cast<size_t>(wr) * p.k + k0 + kk) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kK; ++kk) {
      float a[4];
      ld_vec<4>(&xs[kk][ty * 4], a);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float b = ws[kk][tx + 16 * j];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i][j] = fmaf(a[i], b, acc[i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= rows) continue;
    T* y = static_cast<T*>(p.y) + static_cast<size_t>(row0 + r) * p.ldy;
    if (p.mode == 0) {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int f = blockIdx.x * 32 + tx + 16 * j;
        if (f < p.features) {
          const float g = fminf(acc[i][j], p.limit), u = fminf(fmaxf(acc[i][j + 2], -p.limit), p.limit);
          st_f(y + f, g * sigmoid_f(p.alpha * g) * (u + p.shift));
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = blockIdx.x * kT + tx + 16 * j;
        if (n < p.features) st_f(y + n, acc[i][j] * p.row_w[row0 + r]);
      }
    }
  }
}

template <int BN, int kRows>
static int grouped_launch(const CUtensorMap& tx, const CUtensorMap& tw, GroupedParams p, int max_rows, cudaStream_t st) {
  constexpr int kStage = (kRows + BN) * 128;
  // the operand of a 32-row tile is read as 128 rows: 16 KB from the start of the last stage stay inside the buffer
  static_assert(kStage >= 128 * 128, "a stage holds a full operand");
  p.stages = BN == 256 ? 4 : kRows == 32 ? 5 : 3;
  const size_t smem = static_cast<size_t>(p.stages) * kStage + sizeof(GroupedShared) + 1024;
  static bool cfg = false;
  if (!cfg) {
    if (cudaFuncSetAttribute(grouped_gemm_kernel<BN, kRows>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) !=
        cudaSuccess)
      return SLLM_ERR_CUDA;
    cfg = true;
  }
  const int tiles = (max_rows < p.experts ? max_rows : p.experts) + max_rows / kRows;
  const dim3 grid((p.n_rows + BN - 1) / BN, tiles);
  if (tiles > 65535) return SLLM_ERR_LIMIT;
  return launch_kernel(grouped_gemm_kernel<BN, kRows>, grid, dim3(kGgThreads), smem, st, 1u, tx, tw, p) == cudaSuccess ? SLLM_OK
                                                                                                                       : SLLM_ERR_CUDA;
}

static int grouped_params(GroupedParams* p, const int* tok_off, int experts, int n_rows, int k, int mode, const float* row_w,
                          float limit, float alpha, float shift, void* y, int ldy, int features, int rows) {
  if (!tok_off || !y || experts <= 0 || n_rows <= 0 || k <= 0 || mode < 0 || mode > 1 || (mode == 1 && !row_w) || features <= 0 ||
      ldy < features || rows <= 0 || (mode == 0 && (n_rows % 128 || features != n_rows / 2)) || (mode == 1 && features != n_rows))
    return SLLM_ERR_INVALID_ARGUMENT;
  if (experts > 32 * 64) return SLLM_ERR_UNSUPPORTED_SHAPE;
  *p = {};
  p->tok_off = tok_off; p->experts = experts; p->n_rows = n_rows; p->k = k; p->mode = mode; p->row_w = row_w; p->limit = limit;
  p->alpha = alpha; p->shift = shift; p->y = y; p->ldy = ldy; p->features = features;
  return SLLM_OK;
}

}  // namespace sllm

using namespace sllm;

// x: bf16 [rows, k] permuted rows (k a multiple of 8), w: bf16 [experts * n_rows, k], y: bf16 [rows, ldy].  tile_rows 32 or
// 128, bn 128 or 256 (256 with 128-row tiles).
SLLM_EXPORT int sllm_moe_grouped(const void* x, const void* w, const int* tok_off, int experts, int n_rows, int k, int mode,
                                 const float* row_w, float limit, float alpha, float shift, void* y, int ldy, int features, int rows,
                                 int tile_rows, int bn, int* status, void* stream) {
  GroupedParams p;
  int rc = grouped_params(&p, tok_off, experts, n_rows, k, mode, row_w, limit, alpha, shift, y, ldy, features, rows);
  if (rc != SLLM_OK) return rc;
  if (!x || !w || (tile_rows != 32 && tile_rows != 128) || (bn != 128 && bn != 256) || (bn == 256 && tile_rows != 128))
    return SLLM_ERR_INVALID_ARGUMENT;
  if ((k & 7) || (ldy & 7) || (features & 7)) return SLLM_ERR_UNSUPPORTED_SHAPE;
  if (reinterpret_cast<uintptr_t>(y) & 15) return SLLM_ERR_ALIGNMENT;
  p.kb = (k + 63) / 64;
  p.status = status;
  CUtensorMap tx, tw;
  rc = cached_kmajor_tmap(&tx, x, 2, rows, k, static_cast<long long>(k) * 2, tile_rows);
  if (rc == SLLM_OK) rc = cached_kmajor_tmap(&tw, w, 2, static_cast<long long>(experts) * n_rows, k, static_cast<long long>(k) * 2, 128);
  if (rc != SLLM_OK) return rc;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (tile_rows == 32) return grouped_launch<128, 32>(tx, tw, p, rows, st);
  return bn == 256 ? grouped_launch<256, 128>(tx, tw, p, rows, st) : grouped_launch<128, 128>(tx, tw, p, rows, st);
}

// Any sizes; x rows are read through src (null: already permuted).  fp32: element type of x, w and y.
SLLM_EXPORT int sllm_moe_grouped_simt(const void* x, int ldx, const int* src, const void* w, const int* tok_off, int experts, int n_rows,
                                      int k, int mode, const float* row_w, float limit, float alpha, float shift, void* y, int ldy,
                                      int features, int rows, int fp32, void* stream) {
  GroupedParams p;
  const int rc = grouped_params(&p, tok_off, experts, n_rows, k, mode, row_w, limit, alpha, shift, y, ldy, features, rows);
  if (rc != SLLM_OK) return rc;
  if (!x || !w || ldx < k) return SLLM_ERR_INVALID_ARGUMENT;
  p.x = x; p.w = w; p.src = src; p.ldx = ldx;
  const int tiles = (rows < experts ? rows : experts) + rows / 64, cols = mode == 0 ? (features + 31) / 32 : (features + 63) / 64;
  if (tiles > 65535) return SLLM_ERR_LIMIT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const cudaError_t e = fp32 ? launch_kernel(grouped_gemm_simt_kernel<float>, dim3(cols, tiles), dim3(256), 0, st, 1u, p)
                             : launch_kernel(grouped_gemm_simt_kernel<__nv_bfloat16>, dim3(cols, tiles), dim3(256), 0, st, 1u, p);
  return e == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}
