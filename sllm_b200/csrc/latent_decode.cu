// Attention of absorbed query rows over bf16 latent pages, for decode steps and short prompt portions: the memory-bound
// form.  A cache row [latent | rotated part] is key and value of every head at once, so a CTA takes up to 32 heads of a
// query row and reads each page once.
//
// Tiles of 64 keys x width are brought in by TMA ({64 channels, one page} boxes, 128-byte swizzle) through a ring of five
// half tiles while the previous tile is being worked on.  Per tile:
//   scores   8 warps = 4 channel quarters x 2 key halves; the query fragments of a warp's quarter stay in registers for
//            the whole kernel, so every key byte is read from shared memory once; the four partial sums meet in shared
//            memory (fp32)
//   softmax  warp w owns heads 4 w .. 4 w + 3, lane l keys l and l + 32; fp32 running maximum and sum
//   values   warp w accumulates its 16-column strips of the latent, P (bf16) x page rows, fp32 registers
// KV splits of a row leave (maximum, sum, weighted sum) in a workspace and are merged by a second small launch: one SM
// alone would need longer to read the partials of 20 heads x 512 channels than all of them need for the keys.
//
// The products are m16n8k16 warp MMAs on purpose: with one tile of latents filling a third of the shared memory and only
// 16 to 32 rows of queries per page byte the kernel is bound by HBM, and the 5th-generation MMA's fixed 128 accumulator
// rows would pad the queries fourfold (or, with keys as rows, need 128-key tiles of which a single one fits).
#include "common.cuh"
#include "api.h"
#include "tmap.h"

namespace sllm {

constexpr int kLdTile = 64;                 // keys per tile
constexpr int kLdHeads = 32;                // heads per CTA (two 16-row MMA tiles)
constexpr int kLdWarps = 8;
constexpr int kLdThreads = kLdWarps * 32;
constexpr int kLdSlotKeys = 32;             // keys per ring slot: a tile is two slots
constexpr int kLdSlots = 5;
constexpr int kLdMaxChunks = 9;             // width <= 576
constexpr int kLdMaxStrips = 4;             // kv_rank <= 512
constexpr int kLdChunkBytes = kLdSlotKeys * 128;
constexpr int kLdSc = 72;                   // row stride of the score partials (floats) and of P (bf16 elements)

struct LatentDecodeParams {
  const __nv_bfloat16* q;   // [rows, heads, width]
  int page_size, max_blocks;
  const int* block_table;
  const int* seq_index;
  const int* kv_lens;
  int heads, kv_rank, width, window, chunks;
  float scale_log2;
  __nv_bfloat16* out;       // [rows, heads, kv_rank]
  float* ws_o;              // [units, splits, 32, kv_rank]
  float* ws_ml;             // [units, splits, 32, 2]
  int* status;
};

struct __align__(16) LatentDecodeShared {
  uint64_t full[kLdSlots];
  int abort_flag;
  float alpha[kLdHeads];
  float inv_l[kLdHeads];
  alignas(16) __nv_bfloat16 p[kLdHeads][kLdSc];
  alignas(16) float s[4][kLdHeads][kLdSc];
};

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void bar_compute() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// Byte offset inside a slot of the 16-byte unit that holds channels [col, col + 8) of key `key` (0 .. 31).
__device__ __forceinline__ uint32_t slot_unit(int key, int col) {
  return static_cast<uint32_t>((col >> 6) * kLdChunkBytes + key * 128 + ((((col & 63) >> 3) ^ (key & 7)) << 4));
}

// kSteps: 16-channel MMA steps of a warp's quarter (width <= 64 kSteps); kMt: 16-head MMA tiles (1 or 2).
template <int kSteps, int kMt>
__global__ void __launch_bounds__(kLdThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm, const LatentDecodeParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int slot_bytes = p.chunks * kLdChunkBytes;
  LatentDecodeShared* sh = reinterpret_cast<LatentDecodeShared*>(smem + kLdSlots * slot_bytes);
  const int r = blockIdx.x, h0 = blockIdx.y * kLdHeads, split = blockIdx.z, splits = gridDim.z;
  const int nh = min(kLdHeads, p.heads - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  volatile int* abort_flag = &sh->abort_flag;
  if (threadIdx.x == 0) {
    for (int s = 0; s < kLdSlots; ++s) mbar_init(&sh->full[s], 1);
    sh->abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm);
  }
  __syncthreads();
  pdl_wait();
  pdl_trigger();
  const int kv_len = p.kv_lens[r];
  const int first = p.window > 0 && kv_len > p.window ? kv_len - p.window : 0;
  const int base0 = first / p.page_size * p.page_size;
  int chunk = (kv_len - base0 + splits - 1) / splits;
  chunk = (chunk + kLdTile - 1) / kLdTile * kLdTile;
  const int begin = base0 + split * chunk;
  const int end = min(begin + chunk, kv_len);
  const int nt = end > begin ? (end - begin + kLdTile - 1) / kLdTile : 0;

  // Page boxes are issued by warp 0, lane i the boxes i, i + 32, .. of a slot.  Every such box of a lane lies in the same
  // page of the slot, whose table entry is read one slot ahead.
  const int* bt = p.block_table + static_cast<size_t>(p.seq_index[r]) * p.max_blocks;
  const int pps = kLdSlotKeys / p.page_size;           // pages per slot
  const int boxes = pps * p.chunks, my_pg = lane % pps;
  const int nslots = 2 * nt, last_page = (kv_len - 1) / p.page_size;
  auto page_row = [&](int u) {                         // pages past the last one that holds keys repeat it (masked keys)
    return bt[min((begin + u * kLdSlotKeys) / p.page_size + my_pg, last_page)] * p.page_size;
  };
  auto fill = [&](int u, int row) {                    // slot-sized piece u into slot u % kLdSlots
    const int s = u % kLdSlots;
    if (lane == 0) mbar_expect_tx(&sh->full[s], static_cast<uint32_t>(slot_bytes));
    __syncwarp();
    for (int b = lane; b < boxes; b += 32)
      tma_load_2d(smem + s * slot_bytes + (b / pps) * kLdChunkBytes + my_pg * p.page_size * 128, &tm, &sh->full[s], (b / pps) * 64,
                  row);
  };
  int filled = 0, row_next = 0;                        // warp 0: pieces requested, table entry of piece `filled`
  if (warp == 0 && nslots > 0) {
    int rows0[kLdSlots];
#pragma unroll
    for (int u = 0; u < kLdSlots; ++u) rows0[u] = u < nslots ? page_row(u) : 0;
#pragma unroll
    for (int u = 0; u < kLdSlots; ++u)
      if (u < nslots) {
        fill(u, rows0[u]);
        filled = u + 1;
      }
    if (filled < nslots) row_next = page_row(filled);
  }
  {
    const int kq = warp & 3, nb = warp >> 2;           // channel quarter, key half of the score product
    const int total_steps = (p.width + 15) >> 4;
    const int per = (total_steps + 3) >> 2;            // steps per quarter (<= kSteps)
    const int step0 = kq * per;
    const int nsteps = max(0, min(per, total_steps - step0));
    // query fragments (rows = heads, zero beyond the heads and the width)
    uint32_t qa[kSteps][kMt][4];
    const __nv_bfloat16* qrow = p.q + (static_cast<size_t>(r) * p.heads + h0) * p.width;
#pragma unroll
    for (int i = 0; i < kSteps; ++i)
#pragma unroll
      for (int mt = 0; mt < kMt; ++mt)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int head = mt * 16 + (lane >> 2) + (x & 1) * 8;
          const int col = (step0 + i) * 16 + (lane & 3) * 2 + (x >> 1) * 8;
          qa[i][mt][x] = i < nsteps && head < nh && col < p.width
                             ? *reinterpret_cast<const uint32_t*>(qrow + static_cast<size_t>(head) * p.width + col) : 0u;
        }
    float o[kMt][kLdMaxStrips][2][4];
#pragma unroll
    for (int mt = 0; mt < kMt; ++mt)
#pragma unroll
      for (int i = 0; i < kLdMaxStrips; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int x = 0; x < 4; ++x) o[mt][i][h][x] = 0.f;
    constexpr int kOwn = 2 * kMt;                      // heads whose softmax a warp keeps
    float m[kOwn], l[kOwn];
#pragma unroll
    for (int g = 0; g < kOwn; ++g) { m[g] = -INFINITY; l[g] = 0.f; }
    bool ok = true;
    for (int j = 0; j < nt; ++j) {
      const int u0 = 2 * j;
      const uint32_t slot[2] = {smem_u32(smem + (u0 % kLdSlots) * slot_bytes), smem_u32(smem + ((u0 + 1) % kLdSlots) * slot_bytes)};
      // a warp scores the keys of one slot; one that gives up stays in step with the CTA barriers
      if (ok)
        ok = mbar_wait(&sh->full[(u0 + nb) % kLdSlots], ((u0 + nb) / kLdSlots) & 1, abort_flag, p.status, SLLM_DEV_TIMEOUT_TMA_FULL);
      // ---- scores of 32 keys over this warp's quarter of the channels
      float sc[kMt][4][4];
#pragma unroll
      for (int mt = 0; mt < kMt; ++mt)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int x = 0; x < 4; ++x) sc[mt][n][x] = 0.f;
#pragma unroll
      for (int i = 0; i < kSteps; ++i) {
        if (i < nsteps) {
          const int col = (step0 + i) * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
          for (int n2 = 0; n2 < 2; ++n2) {
            const int key = n2 * 16 + ((lane >> 4) << 3) + (lane & 7);
            uint32_t b[4];
            ldsm_x4((nb ? slot[1] : slot[0]) + slot_unit(key, col), b);
#pragma unroll
            for (int mt = 0; mt < kMt; ++mt) {
              mma_bf16(sc[mt][2 * n2], qa[i][mt], b[0], b[1]);
              mma_bf16(sc[mt][2 * n2 + 1], qa[i][mt], b[2], b[3]);
            }
          }
        }
      }
#pragma unroll
      for (int mt = 0; mt < kMt; ++mt)
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const int head = mt * 16 + (lane >> 2), key = nb * 32 + n * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(&sh->s[kq][head][key]) = make_float2(sc[mt][n][0], sc[mt][n][1]);
          *reinterpret_cast<float2*>(&sh->s[kq][head + 8][key]) = make_float2(sc[mt][n][2], sc[mt][n][3]);
        }
      bar_compute();
      // every warp is past the previous tile's values: its two slots take the next pieces
      if (warp == 0) {
#pragma unroll
        for (int k = 0; k < 2; ++k)
          if (filled < nslots && filled < u0 + kLdSlots) {
            fill(filled, row_next);
            ++filled;
            if (filled < nslots) row_next = page_row(filled);
          }
      }
      // ---- softmax of this warp's heads
      {
        const int tok = begin + j * kLdTile + lane;
        const bool v0 = tok >= first && tok < end, v1 = tok + 32 >= first && tok + 32 < end;
#pragma unroll
        for (int g = 0; g < kOwn; ++g) {
          const int head = warp * kOwn + g;
          float s0 = 0.f, s1 = 0.f;
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            s0 += sh->s[k][head][lane];
            s1 += sh->s[k][head][lane + 32];
          }
          s0 = v0 ? s0 * p.scale_log2 : -INFINITY;
          s1 = v1 ? s1 * p.scale_log2 : -INFINITY;
          const float m_new = fmaxf(m[g], warp_max_redux(fmaxf(s0, s1)));
          const float m_use = m_new == -INFINITY ? 0.f : m_new;
          const float alpha = m[g] == -INFINITY ? 0.f : ex2_approx(m[g] - m_use);
          const __nv_bfloat16 p0 = __float2bfloat16_rn(ex2_approx(s0 - m_use)), p1 = __float2bfloat16_rn(ex2_approx(s1 - m_use));
          // the normaliser sums the values that the product multiplies
          l[g] = l[g] * alpha + __bfloat162float(p0) + __bfloat162float(p1);
          m[g] = m_new;
          sh->p[head][lane] = p0;
          sh->p[head][lane + 32] = p1;
          if (lane == 0) sh->alpha[head] = alpha;
        }
      }
      // the other slot's data: each warp observes its barrier itself before reading it below
      if (ok)
        ok = mbar_wait(&sh->full[(u0 + 1 - nb) % kLdSlots], ((u0 + 1 - nb) / kLdSlots) & 1, abort_flag, p.status,
                       SLLM_DEV_TIMEOUT_TMA_FULL);
      bar_compute();
      // ---- values: strips of 16 latent channels
#pragma unroll
      for (int mt = 0; mt < kMt; ++mt) {
        const float a0 = sh->alpha[mt * 16 + (lane >> 2)], a1 = sh->alpha[mt * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int i = 0; i < kLdMaxStrips; ++i)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            o[mt][i][h][0] *= a0; o[mt][i][h][1] *= a0;
            o[mt][i][h][2] *= a1; o[mt][i][h][3] *= a1;
          }
      }
#pragma unroll
      for (int k = 0; k < kLdTile / 16; ++k) {
        uint32_t pa[kMt][4];
#pragma unroll
        for (int mt = 0; mt < kMt; ++mt)
          ldsm_x4(smem_u32(&sh->p[mt * 16 + (lane & 15)][k * 16 + ((lane >> 4) << 3)]), pa[mt]);
        const int key = (k & 1) * 16 + (lane & 15);
#pragma unroll
        for (int i = 0; i < kLdMaxStrips; ++i) {
          const int col0 = (warp + kLdWarps * i) * 16;
          if (col0 < p.kv_rank) {
            uint32_t b[4];
            ldsm_x4_t(slot[k >> 1] + slot_unit(key, col0 + ((lane >> 4) << 3)), b);
#pragma unroll
            for (int mt = 0; mt < kMt; ++mt) {
              mma_bf16(o[mt][i][0], pa[mt], b[0], b[1]);
              mma_bf16(o[mt][i][1], pa[mt], b[2], b[3]);
            }
          }
        }
      }
    }
    // every piece requested has been waited for by all warps, so no copy is in flight here - unless a wait gave up
    if (!ok && warp == 0 && lane == 0) {
      int dummy = 0;
      for (int u = max(0, filled - kLdSlots); u < filled; ++u)
        mbar_wait(&sh->full[u % kLdSlots], (u / kLdSlots) & 1, &dummy, p.status, SLLM_DEV_TIMEOUT_DRAIN, 200000000LL);
    }
    // ---- results: this split's (maximum, sum, weighted sum), or the output itself without splits
    const size_t unit = static_cast<size_t>(r) * gridDim.y + blockIdx.y;
#pragma unroll
    for (int g = 0; g < kOwn; ++g) {
      const float ls = warp_sum(l[g]);
      if (lane == 0) {
        const int head = warp * kOwn + g;
        sh->inv_l[head] = ls > 0.f ? 1.f / ls : 0.f;
        if (splits > 1) {
          float* ml = p.ws_ml + ((unit * splits + split) * kLdHeads + head) * 2;
          ml[0] = m[g];
          ml[1] = ls;
        }
      }
    }
    bar_compute();
#pragma unroll
    for (int mt = 0; mt < kMt; ++mt)
#pragma unroll
      for (int rr = 0; rr < 2; ++rr) {
        const int head = mt * 16 + (lane >> 2) + rr * 8;
        if (head >= nh) continue;
        const float inv = sh->inv_l[head];
#pragma unroll
        for (int i = 0; i < kLdMaxStrips; ++i)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int col = (warp + kLdWarps * i) * 16 + h * 8 + (lane & 3) * 2;
            if (col >= p.kv_rank) continue;
            const float x0 = o[mt][i][h][rr * 2], x1 = o[mt][i][h][rr * 2 + 1];
            if (splits > 1)
              *reinterpret_cast<float2*>(p.ws_o + ((unit * splits + split) * kLdHeads + head) * p.kv_rank + col) = make_float2(x0, x1);
            else
              *reinterpret_cast<__nv_bfloat162*>(p.out + (static_cast<size_t>(r) * p.heads + h0 + head) * p.kv_rank + col) =
                  __floats2bfloat162_rn(x0 * inv, x1 * inv);
          }
      }
  }
  __syncthreads();
}

// Merges the KV splits of a row: grid (rows, heads), a thread per 4 latent channels.
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentDecodeParams p, int splits, int groups) {
  __shared__ float fac[32];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, h = blockIdx.y, head = h % kLdHeads;
  const size_t unit = static_cast<size_t>(r) * groups + h / kLdHeads;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    float2 ml = make_float2(-INFINITY, 0.f);
    if (lane < splits) ml = *reinterpret_cast<const float2*>(p.ws_ml + ((unit * splits + lane) * kLdHeads + head) * 2);
    const float mx = warp_max_redux(ml.x);
    const float f = ml.x == -INFINITY ? 0.f : ex2_approx(ml.x - mx);
    const float sum = warp_sum(f * ml.y);
    fac[lane] = sum > 0.f ? f / sum : 0.f;
  }
  __syncthreads();
  const size_t stride = static_cast<size_t>(kLdHeads) * p.kv_rank;
  for (int col = threadIdx.x * 4; col < p.kv_rank; col += 512) {
    const float* src = p.ws_o + (unit * splits * kLdHeads + head) * p.kv_rank + col;
    float x[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s0 = 0; s0 < splits; s0 += 8) {
      float4 v[8];
#pragma unroll
      for (int k = 0; k < 8; ++k)
        v[k] = s0 + k < splits ? *reinterpret_cast<const float4*>(src + (s0 + k) * stride) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float f = s0 + k < splits ? fac[s0 + k] : 0.f;
        x[0] = fmaf(f, v[k].x, x[0]); x[1] = fmaf(f, v[k].y, x[1]);
        x[2] = fmaf(f, v[k].z, x[2]); x[3] = fmaf(f, v[k].w, x[3]);
      }
    }
    __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(p.out + (static_cast<size_t>(r) * p.heads + h) * p.kv_rank + col);
    dst[0] = __floats2bfloat162_rn(x[0], x[1]);
    dst[1] = __floats2bfloat162_rn(x[2], x[3]);
  }
}

template <int kSteps, int kMt>
static int latent_decode_launch(const CUtensorMap& tm, const LatentDecodeParams& p, dim3 grid, size_t smem, cudaStream_t st) {
  static size_t configured = 0;
  if (smem > configured) {
    if (cudaFuncSetAttribute(latent_decode_kernel<kSteps, kMt>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) !=
        cudaSuccess)
      return SLLM_ERR_CUDA;
    configured = smem;
  }
  if (launch_kernel(latent_decode_kernel<kSteps, kMt>, grid, dim3(kLdThreads), smem, st, 1u, tm, p) != cudaSuccess) return SLLM_ERR_CUDA;
  if (grid.z == 1) return SLLM_OK;
  return launch_kernel(latent_combine_kernel, dim3(grid.x, p.heads), dim3(128), 0, st, 1u, p, static_cast<int>(grid.z),
                       static_cast<int>(grid.y)) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

}  // namespace sllm

using namespace sllm;

// Floats of workspace for a launch with this many KV splits (0 without splits).
SLLM_EXPORT long long sllm_latent_decode_workspace_floats(int rows, int heads, int kv_rank, int splits) {
  if (splits <= 1) return 0;
  const long long units = static_cast<long long>(rows) * ((heads + kLdHeads - 1) / kLdHeads);
  return units * splits * kLdHeads * (static_cast<long long>(kv_rank) + 2);
}

// bf16 pages [num_pages * page_size, ld]; width <= 576, kv_rank <= 512 and a multiple of 8, ld a multiple of 8, pages of
// 8, 16 or 32 rows.
SLLM_EXPORT int sllm_latent_decode(const void* q, const void* pages, long long page_rows, int ld, int page_size, int max_blocks,
                                   const int* block_table, const int* seq_index, const int* kv_lens, int rows, int heads,
                                   int kv_rank, int width, int window, float scale, void* out, int splits, float* ws,
                                   long long ws_floats, int* status, void* stream) {
  if (!q || !pages || !block_table || !seq_index || !kv_lens || !out || rows <= 0 || heads <= 0 || width < kv_rank || ld < width ||
      max_blocks <= 0 || page_rows <= 0 || splits < 1 || splits > 32)
    return SLLM_ERR_INVALID_ARGUMENT;
  if (kv_rank <= 0 || kv_rank > kLdMaxStrips * kLdWarps * 16 || (kv_rank & 7) || width > kLdMaxChunks * 64 || (width & 1) || (ld & 7) ||
      (page_size != 8 && page_size != 16 && page_size != 32))
    return SLLM_ERR_UNSUPPORTED_SHAPE;
  if ((reinterpret_cast<uintptr_t>(q) & 3) || (reinterpret_cast<uintptr_t>(out) & 3)) return SLLM_ERR_ALIGNMENT;
  const int groups = (heads + kLdHeads - 1) / kLdHeads;
  LatentDecodeParams p = {};
  p.q = static_cast<const __nv_bfloat16*>(q); p.page_size = page_size; p.max_blocks = max_blocks;
  p.block_table = block_table; p.seq_index = seq_index; p.kv_lens = kv_lens; p.heads = heads; p.kv_rank = kv_rank; p.width = width;
  p.window = window; p.scale_log2 = scale * 1.4426950408889634f; p.out = static_cast<__nv_bfloat16*>(out); p.status = status;
  // value strips read whole 16-channel units: the staged tile covers them (columns past the row are zero)
  const int need = ((kv_rank + 15) / 16 * 16 > width) ? (kv_rank + 15) / 16 * 16 : width;
  p.chunks = (need + 63) / 64;
  if (p.chunks > kLdMaxChunks) return SLLM_ERR_UNSUPPORTED_SHAPE;
  if (splits > 1) {
    const long long units = static_cast<long long>(rows) * groups;
    if (!ws || ws_floats < sllm_latent_decode_workspace_floats(rows, heads, kv_rank, splits))
      return SLLM_ERR_WORKSPACE_TOO_SMALL;
    p.ws_o = ws;
    p.ws_ml = ws + units * splits * kLdHeads * kv_rank;
  }
  CUtensorMap tm;
  const int rc = cached_kmajor_tmap(&tm, pages, 2, page_rows, width, static_cast<long long>(ld) * 2, page_size);
  if (rc != SLLM_OK) return rc;
  const size_t smem = static_cast<size_t>(kLdSlots) * p.chunks * kLdChunkBytes + sizeof(LatentDecodeShared) + 1024;
  const dim3 grid(rows, groups, splits);
  if (groups > 65535) return SLLM_ERR_LIMIT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int per = ((width + 15) / 16 + 3) / 4;
  const bool one = heads <= 16;
  if (per <= 3) return one ? latent_decode_launch<3, 1>(tm, p, grid, smem, st) : latent_decode_launch<3, 2>(tm, p, grid, smem, st);
  if (per <= 5) return one ? latent_decode_launch<5, 1>(tm, p, grid, smem, st) : latent_decode_launch<5, 2>(tm, p, grid, smem, st);
  return one ? latent_decode_launch<9, 1>(tm, p, grid, smem, st) : latent_decode_launch<9, 2>(tm, p, grid, smem, st);
}
