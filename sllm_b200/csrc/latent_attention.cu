// Latent attention over a paged cache of latents, the parts that are not matrix products over the whole batch.
//
// Cache row of a token (one per layer, shared by all heads): [latent c (kv_rank) | rotated key part (rot_dim)], row
// stride ld (padded to 16 bytes).  Keys and values of a head are linear images of c:
//   k_h = W_uk[h] c,  v_h = W_uv[h] c
// so a query row can be carried into latent space once, q_h W_uk[h] (kv_rank wide), scored against the cache row
// directly, and the weighted sum of latents carried back by W_uv[h] afterwards ("absorbed" form).  Every row of a
// batch - a decoded token, a row of a prompt portion - is served by it; long prompt portions take the expanded form
// (latent_prefill.cu).
//
//   latent_append_kernel    per token: RMSNorm of the query latent, RMSNorm of the key latent and rotation of the shared
//                           key part, written straight into the page
//   head_matmul_kernel      per head: out[t, h, :] = in[t, h, :] M[h] (absorb: M = W_uk as stored; values: M = W_uv^T)
//                           with the rotation of the query's rotated part or the sigmoid output gate riding along
//   latent_attention_kernel CUDA-core attention of absorbed rows, any sizes, fp32 or bf16 pages
#include <type_traits>
#include "typed.cuh"
#include "api.h"

namespace sllm {

// Rotation of a pair (u, v) at angle pos * freq.
__device__ __forceinline__ void rotate_pair(float& u, float& v, float pos, float freq) {
  float sn, cs;
  sincosf(pos * freq, &sn, &cs);
  const float a = u * cs - v * sn, b = v * cs + u * sn;
  u = a;
  v = b;
}
// Channel i of a rotated vector from its values v[] (fp32); interleaved: pairs (2i, 2i+1), else (i, i + dims / 2).
__device__ __forceinline__ float rotated_channel(const float* v, int i, int dims, int interleaved, const float* inv_freq, float pos) {
  if (i >= dims) return v[i];
  const int half = dims >> 1;
  const int fi = interleaved ? i >> 1 : (i < half ? i : i - half);
  const int iu = interleaved ? 2 * fi : fi, iv = interleaved ? 2 * fi + 1 : fi + half;
  float a = v[iu], b = v[iv];
  rotate_pair(a, b, pos, inv_freq[fi]);
  return i == iu ? a : b;
}

struct LatentRot {
  const float* inv_freq;   // [dims / 2]
  int dims, interleaved;
};

// ---------------------------------------------------------------- projections -> normed query latent, cache row
template <typename T>
struct LatentAppendParams {
  const T* proj;           // [tokens, ldp]
  int ldp, off_q, off_kv;  // columns of the query latent and of [key latent | rotated part]
  int q_rank, kv_rank, rot_dim;
  const float* q_norm;     // [q_rank]
  const float* kv_norm;    // [kv_rank]
  float eps;
  T* q_out;                // [tokens, q_rank]
  T* pages;                // [num_pages * page, ld]
  int ld, page_size, max_blocks;
  const int* positions;
  const int* seq_index;
  const int* block_table;
  LatentRot rot;
};

// grid (tokens, 1 or 2), 128 threads: y = 0 the cache row, y = 1 the query latent.
template <typename T>
__global__ void __launch_bounds__(128) latent_append_kernel(const LatentAppendParams<T> p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float vals[];
  __shared__ float red[4];
  const int t = blockIdx.x;
  const bool q = blockIdx.y == 1;
  const T* src = p.proj + static_cast<size_t>(t) * p.ldp + (q ? p.off_q : p.off_kv);
  const int n = q ? p.q_rank : p.kv_rank;
  const int total = q ? n : n + p.rot_dim;
  float ss = 0.f;
  for (int i = threadIdx.x; i < total; i += 128) {
    const float v = ld_f(src + i);
    vals[i] = v;
    if (i < n) ss += v * v;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float inv = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / static_cast<float>(n) + p.eps);
  if (q) {
    T* dst = p.q_out + static_cast<size_t>(t) * n;
    for (int i = threadIdx.x; i < n; i += 128) st_f(dst + i, vals[i] * inv * p.q_norm[i]);
    return;
  }
  const int pos = p.positions[t];
  const int blk = p.block_table[static_cast<size_t>(p.seq_index[t]) * p.max_blocks + pos / p.page_size];
  T* dst = p.pages + (static_cast<size_t>(blk) * p.page_size + pos % p.page_size) * p.ld;
  for (int i = threadIdx.x; i < total; i += 128) {
    const float v = i < n ? vals[i] * inv * p.kv_norm[i]
                          : rotated_channel(vals + n, i - n, p.rot.dims, p.rot.interleaved, p.rot.inv_freq, static_cast<float>(pos));
    st_f(dst + i, v);
  }
}

// ---------------------------------------------------------------- per-head matrix product
template <typename T>
struct HeadMatmulParams {
  const T* in;             // [rows, ...]: head h of row r at in + r * ld_in + h * hs_in, K elements
  long long ld_in;
  int hs_in;
  const T* m;              // [heads, K, N]
  T* out;                  // head h of row r at out + r * ld_out + h * hs_out, N elements
  long long ld_out;
  int hs_out;
  int rows, k, n;
  const T* gate;           // optional [rows, ld_gate]: the result is multiplied by sigmoid(gate[r, h])
  long long ld_gate;
  // optional: the input's rot_dim channels behind the first K are rotated and copied behind the N results
  int rot_dim;
  const int* positions;
  LatentRot rot;
};

constexpr int kHmRows = 8, kHmThreads = 256;

// grid (ceil(N / (kLanes * VEC)), heads, ceil(rows / 8)): a CTA covers 8 rows and kLanes * VEC columns of one head; its
// 256 / kLanes K slices read 16-byte pieces of the matrix and are summed through shared memory.
// kAligned: N is a multiple of the 16-byte vector (and so every piece is aligned).
template <typename T, int kLanes, bool kAligned>
__global__ void __launch_bounds__(kHmThreads) head_matmul_kernel(const HeadMatmulParams<T> p) {
  pdl_wait();
  pdl_trigger();
  constexpr int V = kVec16<T>;
  constexpr int kCols = kLanes * V, kSlices = kHmThreads / kLanes;
  extern __shared__ __align__(16) float sm[];
  float* in_s = sm;                                   // [K][kHmRows]
  float* red = sm + p.k * kHmRows;                    // [kSlices][kHmRows][kCols]
  const int h = blockIdx.y, r0 = blockIdx.z * kHmRows, c0 = blockIdx.x * kCols;
  const int nr = min(kHmRows, p.rows - r0);
  {
    // lane <-> row fastest: the transposed stores are conflict free, and a row's pieces stay in the cache
    const int r = threadIdx.x & (kHmRows - 1);
    const T* src = p.in + (r0 + r) * p.ld_in + static_cast<long long>(h) * p.hs_in;
    for (int k = threadIdx.x / kHmRows; k < p.k; k += kHmThreads / kHmRows) in_s[k * kHmRows + r] = r < nr ? ld_f(src + k) : 0.f;
  }
  __syncthreads();
  const int lane = threadIdx.x % kLanes, slice = threadIdx.x / kLanes;
  const int col = c0 + lane * V;
  float acc[kHmRows][V];
#pragma unroll
  for (int r = 0; r < kHmRows; ++r)
#pragma unroll
    for (int v = 0; v < V; ++v) acc[r][v] = 0.f;
  const T* mh = p.m + static_cast<size_t>(h) * p.k * p.n;
  if (col < p.n) {
#pragma unroll 8
    for (int k = slice; k < p.k; k += kSlices) {
      float w[V];
      const T* src = mh + static_cast<size_t>(k) * p.n + col;
      if constexpr (kAligned) {
        ld16(src, w);
      } else {
#pragma unroll
        for (int v = 0; v < V; ++v) w[v] = col + v < p.n ? ld_f(src + v) : 0.f;
      }
      const float4 a = *reinterpret_cast<const float4*>(in_s + k * kHmRows);
      const float4 b = *reinterpret_cast<const float4*>(in_s + k * kHmRows + 4);
      const float x[kHmRows] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
      for (int r = 0; r < kHmRows; ++r)
#pragma unroll
        for (int v = 0; v < V; ++v) acc[r][v] = fmaf(x[r], w[v], acc[r][v]);
    }
  }
#pragma unroll
  for (int r = 0; r < kHmRows; ++r)
#pragma unroll
    for (int v = 0; v < V; v += 4) {
      const float q[4] = {acc[r][v], acc[r][v + 1], acc[r][v + 2], acc[r][v + 3]};
      st_vec<4>(red + (slice * kHmRows + r) * kCols + lane * V + v, q);
    }
  __syncthreads();
  for (int e = threadIdx.x; e < nr * kCols; e += kHmThreads) {
    const int r = e / kCols, c = e % kCols;
    if (c0 + c >= p.n) continue;
    float a = 0.f;
#pragma unroll
    for (int s = 0; s < kSlices; ++s) a += red[(s * kHmRows + r) * kCols + c];
    if (p.gate) a *= sigmoid_f(ld_f(p.gate + (r0 + r) * p.ld_gate + h));
    st_f(p.out + (r0 + r) * p.ld_out + static_cast<long long>(h) * p.hs_out + c0 + c, a);
  }
  if (p.rot_dim > 0 && blockIdx.x == 0) {
    __syncthreads();
    for (int e = threadIdx.x; e < nr * p.rot_dim; e += kHmThreads) {
      const int r = e / p.rot_dim, i = e % p.rot_dim;
      red[e] = ld_f(p.in + (r0 + r) * p.ld_in + static_cast<long long>(h) * p.hs_in + p.k + i);
    }
    __syncthreads();
    for (int e = threadIdx.x; e < nr * p.rot_dim; e += kHmThreads) {
      const int r = e / p.rot_dim, i = e % p.rot_dim;
      const float v = rotated_channel(red + r * p.rot_dim, i, p.rot.dims, p.rot.interleaved, p.rot.inv_freq,
                                      static_cast<float>(p.positions[r0 + r]));
      st_f(p.out + (r0 + r) * p.ld_out + static_cast<long long>(h) * p.hs_out + p.n + i, v);
    }
  }
}

// ---------------------------------------------------------------- attention of absorbed rows (CUDA cores)
template <typename T>
struct LatentAttnParams {
  const T* q;              // [rows, heads, width] absorbed queries, width = kv_rank + rot_dim
  const T* pages;          // [num_pages * page, ld]
  int ld, page_size, max_blocks;
  const int* block_table;
  const int* seq_index;    // [rows]
  const int* kv_lens;      // [rows]
  int heads, kv_rank, width, window;
  float scale;
  T* out;                  // [rows, heads, kv_rank]
};

constexpr int kLaThreads = 256, kLaHeads = 4, kLaKeys = 32, kLaChunks = 8;   // kv_rank <= 256 * kLaChunks

// grid (rows, ceil(heads / 4)).  32 keys at a time in shared memory (fp32); lane <-> key for the scores (two warps per
// head, half the channels each), thread <-> channel for the weighted sum.
template <typename T>
__global__ void __launch_bounds__(kLaThreads) latent_attention_kernel(const LatentAttnParams<T> p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float sm[];
  const int W = p.width, ldk = W | 1;                // odd row stride: lane <-> key reads hit different banks
  float* q_s = sm;                                   // [4][W]
  float* k_s = q_s + kLaHeads * W;                   // [32][ldk]
  float* s_s = k_s + kLaKeys * ldk;                  // [2][4][32] partial scores
  float* p_s = s_s + 2 * kLaHeads * kLaKeys;         // [4][32]
  float* a_s = p_s + kLaHeads * kLaKeys;             // [4] rescale factors
  float* l_s = a_s + kLaHeads;                       // [4]
  const int r = blockIdx.x, h0 = blockIdx.y * kLaHeads;
  const int nh = min(kLaHeads, p.heads - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kv_len = p.kv_lens[r];
  const int first = p.window > 0 && kv_len > p.window ? kv_len - p.window : 0;
  const int* bt = p.block_table + static_cast<size_t>(p.seq_index[r]) * p.max_blocks;
  const T* q = p.q + (static_cast<size_t>(r) * p.heads + h0) * W;
  for (int e = threadIdx.x; e < kLaHeads * W; e += kLaThreads) q_s[e] = e < nh * W ? ld_f(q + e) * p.scale : 0.f;
  float acc[kLaHeads][kLaChunks];
#pragma unroll
  for (int g = 0; g < kLaHeads; ++g)
#pragma unroll
    for (int c = 0; c < kLaChunks; ++c) acc[g][c] = 0.f;
  float m = -INFINITY, l = 0.f;                      // warps 0..3: running state of head `warp`
  for (int base = first; base < kv_len; base += kLaKeys) {
    const int cnt = min(kLaKeys, kv_len - base);
    __syncthreads();
    for (int j = warp; j < cnt; j += kLaThreads / 32) {
      const int tok = base + j;
      const T* src = p.pages + (static_cast<size_t>(bt[tok / p.page_size]) * p.page_size + tok % p.page_size) * p.ld;
      for (int i = lane; i < W; i += 32) k_s[j * ldk + i] = ld_f(src + i);
    }
    __syncthreads();
    {
      const int g = warp & 3, half = warp >> 2, mid = W >> 1;
      const int lo = half ? mid : 0, hi = half ? W : mid;
      float s0 = 0.f, s1 = 0.f;
      if (lane < cnt) {
        const float* kr = k_s + lane * ldk;
        const float* qr = q_s + g * W;
        int i = lo;
        for (; i + 1 < hi; i += 2) {
          s0 = fmaf(qr[i], kr[i], s0);
          s1 = fmaf(qr[i + 1], kr[i + 1], s1);
        }
        if (i < hi) s0 = fmaf(qr[i], kr[i], s0);
      }
      s_s[(half * kLaHeads + g) * kLaKeys + lane] = s0 + s1;
    }
    __syncthreads();
    if (warp < kLaHeads) {
      const float s = lane < cnt ? s_s[warp * kLaKeys + lane] + s_s[(kLaHeads + warp) * kLaKeys + lane] : -INFINITY;
      const float m_new = fmaxf(m, warp_max(s));
      const float pr = lane < cnt ? expf(s - m_new) : 0.f;
      const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
      l = l * alpha + warp_sum(pr);
      m = m_new;
      p_s[warp * kLaKeys + lane] = pr;
      if (lane == 0) a_s[warp] = alpha;
    }
    __syncthreads();
#pragma unroll
    for (int g = 0; g < kLaHeads; ++g) {
      const float alpha = a_s[g];
#pragma unroll
      for (int c = 0; c < kLaChunks; ++c) acc[g][c] *= alpha;
    }
    for (int j = 0; j < cnt; ++j) {
      float pj[kLaHeads];
#pragma unroll
      for (int g = 0; g < kLaHeads; ++g) pj[g] = p_s[g * kLaKeys + j];
#pragma unroll
      for (int c = 0; c < kLaChunks; ++c) {
        const int ch = c * kLaThreads + threadIdx.x;
        if (ch < p.kv_rank) {
          const float kv = k_s[j * ldk + ch];
#pragma unroll
          for (int g = 0; g < kLaHeads; ++g) acc[g][c] = fmaf(pj[g], kv, acc[g][c]);
        }
      }
    }
  }
  if (warp < kLaHeads && lane == 0) l_s[warp] = l;
  __syncthreads();
  for (int g = 0; g < nh; ++g) {
    const float inv = l_s[g] > 0.f ? 1.f / l_s[g] : 0.f;
    T* dst = p.out + (static_cast<size_t>(r) * p.heads + h0 + g) * p.kv_rank;
#pragma unroll
    for (int c = 0; c < kLaChunks; ++c) {
      const int ch = c * kLaThreads + threadIdx.x;
      float v = 0.f;
#pragma unroll
      for (int gg = 0; gg < kLaHeads; ++gg) v = gg == g ? acc[gg][c] : v;
      if (ch < p.kv_rank) st_f(dst + ch, v * inv);
    }
  }
}

template <typename K>
static int opt_in_smem(K* kernel, size_t smem) {
  if (smem > 227 * 1024) return SLLM_ERR_UNSUPPORTED_SHAPE;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
    return SLLM_ERR_CUDA;
  return SLLM_OK;
}

template <typename T>
static int append_launch(const void* proj, int ldp, int off_q, int off_kv, int q_rank, int kv_rank, int rot_dim, const float* q_norm,
                         const float* kv_norm, float eps, void* q_out, void* pages, int ld, int page_size, int max_blocks,
                         const int* positions, const int* seq_index, const int* block_table, LatentRot rot, int tokens,
                         cudaStream_t st) {
  LatentAppendParams<T> p = {};
  p.proj = static_cast<const T*>(proj); p.ldp = ldp; p.off_q = off_q; p.off_kv = off_kv;
  p.q_rank = q_rank; p.kv_rank = kv_rank; p.rot_dim = rot_dim; p.q_norm = q_norm; p.kv_norm = kv_norm; p.eps = eps;
  p.q_out = static_cast<T*>(q_out); p.pages = static_cast<T*>(pages); p.ld = ld; p.page_size = page_size;
  p.max_blocks = max_blocks; p.positions = positions; p.seq_index = seq_index; p.block_table = block_table; p.rot = rot;
  const int widest = q_rank > kv_rank + rot_dim ? q_rank : kv_rank + rot_dim;
  const size_t smem = sizeof(float) * widest;
  const int rc = opt_in_smem(latent_append_kernel<T>, smem);
  if (rc != SLLM_OK) return rc;
  return launch_kernel(latent_append_kernel<T>, dim3(tokens, q_rank > 0 ? 2 : 1), dim3(128), smem, st, 1u, p) == cudaSuccess
             ? SLLM_OK : SLLM_ERR_CUDA;
}

template <typename T, int kLanes>
static int head_matmul_launch_l(const HeadMatmulParams<T>& p, int heads, cudaStream_t st) {
  constexpr int kCols = kLanes * kVec16<T>;
  const bool al = p.n % kVec16<T> == 0 && (reinterpret_cast<uintptr_t>(p.m) & 15) == 0;
  auto* kernel = al ? head_matmul_kernel<T, kLanes, true> : head_matmul_kernel<T, kLanes, false>;
  size_t red = static_cast<size_t>(kHmThreads / kLanes) * kHmRows * kCols;
  if (static_cast<size_t>(kHmRows) * p.rot_dim > red) red = static_cast<size_t>(kHmRows) * p.rot_dim;
  const size_t smem = sizeof(float) * (static_cast<size_t>(p.k) * kHmRows + red);
  const int rc = opt_in_smem(kernel, smem);
  if (rc != SLLM_OK) return rc;
  const dim3 grid((p.n + kCols - 1) / kCols, heads, (p.rows + kHmRows - 1) / kHmRows);
  if (grid.z > 65535 || grid.y > 65535) return SLLM_ERR_LIMIT;
  return launch_kernel(kernel, grid, dim3(kHmThreads), smem, st, 1u, p) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

template <typename T>
static int head_matmul_launch(const HeadMatmulParams<T>& p, int heads, cudaStream_t st) {
  const int pieces = (p.n + kVec16<T> - 1) / kVec16<T>;
  if (pieces >= 32) return head_matmul_launch_l<T, 32>(p, heads, st);
  if (pieces >= 16) return head_matmul_launch_l<T, 16>(p, heads, st);
  return head_matmul_launch_l<T, 8>(p, heads, st);
}

template <typename T>
static int latent_attention_launch(const void* q, const void* pages, int ld, int page_size, int max_blocks, const int* block_table,
                                   const int* seq_index, const int* kv_lens, int rows, int heads, int kv_rank, int width, int window,
                                   float scale, void* out, cudaStream_t st) {
  LatentAttnParams<T> p = {};
  p.q = static_cast<const T*>(q); p.pages = static_cast<const T*>(pages); p.ld = ld; p.page_size = page_size;
  p.max_blocks = max_blocks; p.block_table = block_table; p.seq_index = seq_index; p.kv_lens = kv_lens;
  p.heads = heads; p.kv_rank = kv_rank; p.width = width; p.window = window; p.scale = scale; p.out = static_cast<T*>(out);
  const size_t smem = sizeof(float) * (kLaHeads * width + kLaKeys * (width | 1) + 3 * kLaHeads * kLaKeys + 2 * kLaHeads);
  const int rc = opt_in_smem(latent_attention_kernel<T>, smem);
  if (rc != SLLM_OK) return rc;
  return launch_kernel(latent_attention_kernel<T>, dim3(rows, (heads + kLaHeads - 1) / kLaHeads), dim3(kLaThreads), smem, st, 1u,
                       p) == cudaSuccess ? SLLM_OK : SLLM_ERR_CUDA;
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_latent_append(const void* proj, int ldp, int off_q, int off_kv, int q_rank, int kv_rank, int rot_dim,
                                   const float* q_norm, const float* kv_norm, float eps, void* q_out, void* pages, int ld,
                                   int page_size, int max_blocks, const int* positions, const int* seq_index, const int* block_table,
                                   const float* inv_freq, int rot_dims, int interleaved, int tokens, int fp32, void* stream) {
  if (!proj || !kv_norm || !pages || !positions || !seq_index || !block_table || tokens <= 0 || kv_rank <= 0 || rot_dim < 0 ||
      q_rank < 0 || (q_rank > 0 && (!q_norm || !q_out)) || ld < kv_rank + rot_dim || page_size <= 0 || rot_dims > rot_dim ||
      (rot_dims & 1) || (rot_dims > 0 && !inv_freq))
    return SLLM_ERR_INVALID_ARGUMENT;
  const LatentRot rot = {inv_freq, rot_dims, interleaved};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return fp32 ? append_launch<float>(proj, ldp, off_q, off_kv, q_rank, kv_rank, rot_dim, q_norm, kv_norm, eps, q_out, pages, ld,
                                     page_size, max_blocks, positions, seq_index, block_table, rot, tokens, st)
              : append_launch<__nv_bfloat16>(proj, ldp, off_q, off_kv, q_rank, kv_rank, rot_dim, q_norm, kv_norm, eps, q_out, pages,
                                             ld, page_size, max_blocks, positions, seq_index, block_table, rot, tokens, st);
}

SLLM_EXPORT int sllm_head_matmul(const void* in, long long ld_in, int hs_in, const void* m, void* out, long long ld_out, int hs_out,
                                 int rows, int heads, int k, int n, const void* gate, long long ld_gate, int rot_dim,
                                 const int* positions, const float* inv_freq, int rot_dims, int interleaved, int fp32, void* stream) {
  if (!in || !m || !out || rows <= 0 || heads <= 0 || k <= 0 || n <= 0 || rot_dim < 0 || rot_dims > rot_dim || (rot_dims & 1) ||
      (rot_dim > 0 && !positions) || (rot_dims > 0 && !inv_freq))
    return SLLM_ERR_INVALID_ARGUMENT;
  const LatentRot rot = {inv_freq, rot_dims, interleaved};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    HeadMatmulParams<T> p = {};
    p.in = static_cast<const T*>(in); p.ld_in = ld_in; p.hs_in = hs_in; p.m = static_cast<const T*>(m);
    p.out = static_cast<T*>(out); p.ld_out = ld_out; p.hs_out = hs_out; p.rows = rows; p.k = k; p.n = n;
    p.gate = static_cast<const T*>(gate); p.ld_gate = ld_gate; p.rot_dim = rot_dim; p.positions = positions; p.rot = rot;
    return head_matmul_launch<T>(p, heads, st);
  };
  return fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}

SLLM_EXPORT int sllm_latent_attention(const void* q, const void* pages, int ld, int page_size, int max_blocks, const int* block_table,
                                      const int* seq_index, const int* kv_lens, int rows, int heads, int kv_rank, int width,
                                      int window, float scale, void* out, int fp32, void* stream) {
  if (!q || !pages || !block_table || !seq_index || !kv_lens || !out || rows <= 0 || heads <= 0 || kv_rank <= 0 || width < kv_rank ||
      ld < width || page_size <= 0)
    return SLLM_ERR_INVALID_ARGUMENT;
  if (kv_rank > kLaThreads * kLaChunks) return SLLM_ERR_UNSUPPORTED_SHAPE;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return fp32 ? latent_attention_launch<float>(q, pages, ld, page_size, max_blocks, block_table, seq_index, kv_lens, rows, heads,
                                               kv_rank, width, window, scale, out, st)
              : latent_attention_launch<__nv_bfloat16>(q, pages, ld, page_size, max_blocks, block_table, seq_index, kv_lens, rows,
                                                       heads, kv_rank, width, window, scale, out, st);
}
