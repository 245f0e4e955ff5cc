// Multi-head latent attention over a paged cache. Per token and layer the cache holds one row [c: R | k_r: D_r | 0 ..]
// (W = R + D_r rounded up to 16 columns, rows W + 8 apart): the normed latent and one rotated key part shared by all heads. With per-head
// up-projections W_uk (D_n x R) and W_uv (D_v x R), head h scores  (q_n . W_uk c + q_r . k_r) * scale  and reads out
// W_uv (sum_j p_j c_j).
//
// Short portions (decode) move W_uk to the query side: q_l = W_uk^T q_n once per token and head, then every head attends
// to the cached rows themselves (keys: all W columns, values: the first R), so a step streams the cache once for all
// heads:
//   latent_prep_kernel      norm of the latent, rotation of k_r and of the queries' rotated part (or norm of the latent that
//                           the queries come from), cache append
//   latent_absorb_kernel    [q_l | q_r | 0] rows of width W (q_r turned here where the queries come from a latent)
//   latent_attn_mma_kernel  bf16, split over key pages: 16 or 32 (token, head) rows share each 64-key page in shared
//                           memory; S by mma.sync with keys and row quarters cut over the warps (query fragments stay in
//                           registers), P V with the columns cut over the warps
//   latent_attn_row_kernel  any type and size, one (token, head) row per CTA (fp32 models)
//   latent_up_kernel        joins the splits and applies W_uv
// Longer portions expand keys and values of the visible rows with one GEMM and run the flash-attention kernels of
// attention_tc.cu; latent_gather_kernel / latent_assemble_kernel lay out their operands (128 channels per head, zero
// padded).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math_constants.h>
#include <stdint.h>
#include "common.cuh"
#include "elem.cuh"
#include "host_util.cuh"
#include "mma_sync.cuh"
#include "pdl.cuh"
#include "pmetal_b200.h"

namespace pm {

constexpr int kPage = 64;
constexpr int kRowPad = 8;            // cache rows are W + 8 apart: a page copied as one block has conflict-free rows in shared memory

// One element, or two neighbours at an even offset.
template <int V>
__device__ __forceinline__ void load_pair(const float* p, float (&v)[V]) {
  if constexpr (V == 2) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[1] = f.y;
  } else {
    v[0] = p[0];
  }
}
template <int V>
__device__ __forceinline__ void load_pair(const __nv_bfloat16* p, float (&v)[V]) {
  if constexpr (V == 2) {
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    v[0] = f.x; v[1] = f.y;
  } else {
    v[0] = to_f(p[0]);
  }
}

// One CTA per token. qd [tokens, ld]: H heads of [D_n | D_r] or (lead > 0, H = 0) a query latent of `lead` channels, which is
// normed in place; then (own != 0) the down-projection [R | D_r].
// V: elements per access of the norms.
template <typename T, int V>
__device__ __forceinline__ void latent_norm_row(const T* src, T* dst, const float* __restrict__ w, int n, float eps) {
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
    float v[V];
    load_vec<V>(src + i, v);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
  }
  const float r = 1.f / sqrtf(block_sum(ss) / static_cast<float>(n) + eps);
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
    float v[V], ww[V];
    load_vec<V>(src + i, v);
    load_vec<V>(w + i, ww);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= r * ww[e];
    store_vec<V>(dst + i, v);
  }
}

template <typename T, int V>
__global__ void latent_prep_kernel(T* __restrict__ qd, long long ld, const float* __restrict__ norm_w, float eps,
                                   const float* __restrict__ cs, const float* __restrict__ sn, int H, int dn, int dr, int rank,
                                   int own, T* __restrict__ cache, int W, const long long* __restrict__ slots, int lead,
                                   const float* __restrict__ lead_w) {
  const long long t = blockIdx.x;
  T* row = qd + t * ld;
  const int half = dr / 2;
  const float* c = cs + t * half;
  const float* s = sn + t * half;
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, j = i - h * half;
    T* p = row + h * (dn + dr) + dn + 2 * j;
    const float a = to_f(p[0]), b = to_f(p[1]);
    put(p, a * c[j] - b * s[j]);
    put(p + 1, b * c[j] + a * s[j]);
  }
  if (lead > 0) latent_norm_row<T, V>(row, row, lead_w, lead, eps);
  if (!own) return;
  const T* d = row + H * (dn + dr) + lead;
  T* dst = cache + slots[t] * (W + kRowPad);
  latent_norm_row<T, V>(d, dst, norm_w, rank, eps);
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    const float a = to_f(d[rank + 2 * j]), b = to_f(d[rank + 2 * j + 1]);
    put(dst + rank + 2 * j, a * c[j] - b * s[j]);
    put(dst + rank + 2 * j + 1, b * c[j] + a * s[j]);
  }
}

// grid (column tiles of 128 plus one, H, groups of kAbsTok tokens), 256 threads. The CTA computes 128 columns of q_l for
// kAbsTok tokens of one head (compact token i is row rows[i] of qd): 128 / V threads side by side own the columns, the
// groups of threads behind them cut the unrotated dimensions and meet in shared memory. The last column tile copies the
// rotated part and zeroes the rest.
constexpr int kAbsTok = 8;
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const T* __restrict__ qd, long long ld, const T* __restrict__ wuk,
                                                            int H, int dn, int dr, int rank, int W, const int* __restrict__ rows,
                                                            int n, T* __restrict__ out, const T* __restrict__ wuv,
                                                            unsigned wuv_bytes, const float* __restrict__ cs,
                                                            const float* __restrict__ sn) {
  extern __shared__ __align__(16) float abs_q[];           // [dn][kAbsTok], then [groups][kAbsTok][128]
  constexpr int kCols = 128 / V, kGroups = 256 / kCols;
  const int h = blockIdx.y, t0 = blockIdx.z * kAbsTok, n_tok = min(kAbsTok, n - t0);
  if (blockIdx.x == gridDim.x - 1) {
    const int tail = W - rank;
    if (blockIdx.z == 0 && wuv_bytes) {                    // latent_up_kernel will want this head's value weights in L2
      const char* v = reinterpret_cast<const char*>(wuv) + static_cast<size_t>(h) * wuv_bytes;
      for (unsigned o = threadIdx.x * 4096u; o < wuv_bytes; o += blockDim.x * 4096u) l2_prefetch_bulk(v + o, min(4096u, wuv_bytes - o));
    }
    for (int i = threadIdx.x; i < n_tok * tail; i += blockDim.x) {
      const int t = i / tail, j = i - t * tail;
      float v = 0.f;
      if (j < dr) {
        const T* q = qd + rows[t0 + t] * ld + h * (dn + dr) + dn;
        v = to_f(q[j]);
        if (cs) {
          const long long f = static_cast<long long>(rows[t0 + t]) * (dr / 2) + j / 2;
          const float w = to_f(q[j ^ 1]);
          v = fmaf(v, cs[f], j & 1 ? w * sn[f] : -w * sn[f]);
        }
      }
      put(out + (static_cast<long long>(t0 + t) * H + h) * W + rank + j, v);
    }
    return;
  }
  float* red = abs_q + dn * kAbsTok;
  {
    const int t = threadIdx.x >> 5;                        // one warp per token
    const T* q = qd + (t < n_tok ? rows[t0 + t] : 0) * ld + h * (dn + dr);
    for (int j = threadIdx.x & 31; j < dn; j += 32) abs_q[j * kAbsTok + t] = t < n_tok ? to_f(q[j]) : 0.f;
  }
  const int col = (threadIdx.x % kCols) * V, grp = threadIdx.x / kCols, c = blockIdx.x * 128 + col;
  const int per = (dn + kGroups - 1) / kGroups, j0 = grp * per, j1 = min(dn, j0 + per);
  float acc[kAbsTok][V];
#pragma unroll
  for (int t = 0; t < kAbsTok; ++t)
#pragma unroll
    for (int e = 0; e < V; ++e) acc[t][e] = 0.f;
  __syncthreads();
  if (c < rank) {
    const T* w = wuk + static_cast<long long>(h) * dn * rank + c;
#pragma unroll 16
    for (int j = j0; j < j1; ++j) {
      float wv[V], qa[kAbsTok];
      load_pair<V>(w + static_cast<long long>(j) * rank, wv);
      load_vec<kAbsTok>(abs_q + j * kAbsTok, qa);
#pragma unroll
      for (int t = 0; t < kAbsTok; ++t)
#pragma unroll
        for (int e = 0; e < V; ++e) acc[t][e] = fmaf(qa[t], wv[e], acc[t][e]);
    }
  }
#pragma unroll
  for (int t = 0; t < kAbsTok; ++t)
#pragma unroll
    for (int e = 0; e < V; ++e) red[(grp * kAbsTok + t) * 128 + col + e] = acc[t][e];
  __syncthreads();
  for (int i = threadIdx.x; i < n_tok * 128; i += 256) {
    const int t = i >> 7, k = i & 127, cc = blockIdx.x * 128 + k;
    if (cc >= rank) continue;
    float v = 0.f;
#pragma unroll
    for (int g = 0; g < kGroups; ++g) v += red[(g * kAbsTok + t) * 128 + k];
    put(out + (static_cast<long long>(t0 + t) * H + h) * W + cc, v);
  }
}

struct LatentParams {
  const void* q;             // [compact tokens, H, W]
  const void* cache;         // [pages, 64, W + 8]
  const int* block_table;
  const int* seq_lens;
  const int* c_start;        // first row of each sequence in the compact buffers (q, part_o, part_ml)
  const int* q_lens;
  float* part_o;             // [split][compact tokens * H][rank], not normalised
  float* part_ml;            // [split][compact tokens * H][2]: maximum (log2 domain), sum
  int max_blocks, H, W, rank, n_split, row_tiles;
  long long rows;            // compact tokens * H
  float scale_log2;          // scale * log2(e)
  int* status;               // set when a bounded wait runs out
};

// One (token, head) row per CTA, all keys, any type. grid (rows of the longest portion, sequences).
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_row_kernel(const LatentParams p) {
  extern __shared__ __align__(16) float lr_smem[];
  float* sq = lr_smem;               // [W]
  float* so = sq + p.W;              // [rank]
  float* ss = so + p.rank;           // [64]
  const int seq = blockIdx.y, len = p.q_lens[seq], r = blockIdx.x;
  if (r >= len * p.H) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long row = static_cast<long long>(p.c_start[seq]) * p.H + r;
  const int n_keys = p.seq_lens[seq] - len + r / p.H + 1;
  const T* q = static_cast<const T*>(p.q) + row * p.W;
  for (int i = threadIdx.x; i < p.W; i += 128) sq[i] = to_f(q[i]) * p.scale_log2;
  for (int i = threadIdx.x; i < p.rank; i += 128) so[i] = 0.f;
  float m = -CUDART_INF_F, l = 0.f;
  for (int j0 = 0; j0 < n_keys; j0 += kPage) {
    const int n = min(kPage, n_keys - j0);
    const T* page = static_cast<const T*>(p.cache) +
                    static_cast<long long>(p.block_table[static_cast<long long>(seq) * p.max_blocks + j0 / kPage]) * kPage * (p.W + kRowPad);
    __syncthreads();
    for (int k = warp; k < n; k += 4) {
      float v = 0.f;
      for (int i = lane; i < p.W; i += 32) v = fmaf(sq[i], to_f(page[static_cast<long long>(k) * (p.W + kRowPad) + i]), v);
      v = warp_sum(v);
      if (lane == 0) ss[k] = v;
    }
    __syncthreads();
    const float a = lane < n ? ss[lane] : -CUDART_INF_F, b = lane + 32 < n ? ss[lane + 32] : -CUDART_INF_F;
    float mx = fmaxf(a, b);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float m_new = fmaxf(m, mx);
    const float corr = exp2f(m - m_new), pa = exp2f(a - m_new), pb = exp2f(b - m_new);
    l = l * corr + warp_sum(pa + pb);
    m = m_new;
    __syncthreads();
    if (warp == 0) {
      ss[lane] = pa;
      ss[lane + 32] = pb;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.rank; i += 128) {
      float o = so[i] * corr;
#pragma unroll 4
      for (int k = 0; k < n; ++k) o = fmaf(ss[k], to_f(page[static_cast<long long>(k) * (p.W + kRowPad) + i]), o);
      so[i] = o;
    }
  }
  for (int i = threadIdx.x; i < p.rank; i += 128) p.part_o[row * p.rank + i] = so[i];
  if (threadIdx.x == 0) {
    p.part_ml[row * 2] = m;
    p.part_ml[row * 2 + 1] = l;
  }
}

// 16 warps. MT: 16-row tiles of (token, head) rows; KS: 16-column steps of a quarter of the row; NT: 8-column tiles of the
// latent per warp. For the scores a warp owns one row tile, one column quarter (its query fragments stay in registers for all
// pages) and 32 (MT = 2) or 16 (MT = 1) keys of a page; the softmax adds the four partial scores of a key. For P V warp w
// owns columns 8 (w + 16 j).
constexpr int kMmaThreads = 512;
constexpr int kLdS = kPage + 8, kLdP = kPage + 8;
template <int MT, int KS, int NT>
__global__ void __launch_bounds__(kMmaThreads) latent_attn_mma_kernel(const LatentParams p) {
  extern __shared__ __align__(16) uint8_t lm_smem[];
  constexpr int RT = 16 * MT;
  const int ld = p.W + kRowPad;
  __nv_bfloat16* sKV = reinterpret_cast<__nv_bfloat16*>(lm_smem);           // [2][64][ld]
  __nv_bfloat16* sQ = sKV + kPage * ld;                                      // [RT][ld], before the second page is loaded
  __nv_bfloat16* sP = sKV + 2 * kPage * ld;                                  // [RT][kLdP]
  float* sS = reinterpret_cast<float*>(sP + RT * kLdP);                      // [4][RT][kLdS]
  float* sCorr = sS + 4 * RT * kLdS;                                         // [RT]
  __shared__ uint64_t full[2];                                               // a page has arrived in its buffer
  __shared__ int abort_flag;
  const int seq = blockIdx.x / p.row_tiles, row0 = (blockIdx.x % p.row_tiles) * RT, split = blockIdx.y;
  const int len = p.q_lens[seq], n_rows = len * p.H;
  if (row0 >= n_rows) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, t4 = lane & 3;
  const int prior = p.seq_lens[seq] - len;
  const int last_row = min(row0 + RT, n_rows) - 1;
  const int n_keys = prior + last_row / p.H + 1;                             // keys the last row of the tile sees
  const int n_blocks = (n_keys + kPage - 1) / kPage;
  const int per = (n_blocks + p.n_split - 1) / p.n_split;
  const int b0 = split * per, b1 = min(n_blocks, b0 + per);
  const long long base_row = static_cast<long long>(p.c_start[seq]) * p.H + row0;
  const long long part_base = split * p.rows + base_row;
  if (b0 >= b1) {
    for (int i = threadIdx.x; i < RT && row0 + i < n_rows; i += kMmaThreads) {
      p.part_ml[(part_base + i) * 2] = -CUDART_INF_F;
      p.part_ml[(part_base + i) * 2 + 1] = 0.f;
    }
    return;
  }
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.cache);
  const int* bt = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  const int chunks = p.W / 8;
  // One bulk copy brings the rows of a page that a query of the tile sees; the others are zeroed: what lies there may belong
  // to anyone.
  auto load_page = [&](int b, int buf) {
    __nv_bfloat16* dst = sKV + buf * kPage * ld;
    const int valid = min(kPage, n_keys - b * kPage);
    if (threadIdx.x == 0) {
      const uint32_t bytes = static_cast<uint32_t>(valid * ld) * 2;
      mbar_expect_tx(&full[buf], bytes);
      ms_bulk_copy(ms_addr(dst), cache + static_cast<long long>(bt[b]) * kPage * ld, bytes, &full[buf]);
    }
    for (int i = valid * ld / 8 + threadIdx.x; i < kPage * ld / 8; i += kMmaThreads)
      reinterpret_cast<uint4*>(dst)[i] = make_uint4(0u, 0u, 0u, 0u);
  };
  if (threadIdx.x == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    abort_flag = 0;
    mbar_init_fence();
  }
  __syncthreads();
  load_page(b0, 0);
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + base_row * p.W;
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int r = warp + 16 * i;
      const bool ok = row0 + r < n_rows;
      for (int c = lane; c < chunks; c += 32)
        ms_cp16(ms_addr(sQ + r * ld + c * 8), q + static_cast<long long>(ok ? r : 0) * p.W + c * 8, ok);
    }
    ms_commit();
  }
  constexpr int kGroups = 4 / MT, kTiles = 2 * MT;         // groups of keys and 8-key tiles per group
  const int kg = warp & (kGroups - 1), slice = (warp / kGroups) & 3, row_tile = warp / (4 * kGroups);
  const int steps = p.W / 16, per_slice = (steps + 3) / 4, s0 = slice * per_slice, n_steps = max(0, min(per_slice, steps - s0));
  uint32_t qf[KS][4];
  ms_wait<0>();
  __syncthreads();
#pragma unroll
  for (int k = 0; k < KS; ++k)
    if (k < n_steps) ms_ldsm4(ms_a_at(ms_addr(sQ), ld, row_tile * 16, (s0 + k) * 16, lane), qf[k]);
  float acc[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  constexpr int kRows = MT;                      // softmax rows of this warp
  float m_run[kRows], l_run[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i) { m_run[i] = -CUDART_INF_F; l_run[i] = 0.f; }
  const uint32_t aP = ms_addr(sP);
  const int n8 = (p.rank + 7) / 8;
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  __syncthreads();                               // the query tile may be overwritten by a bulk copy

  for (int b = b0; b < b1; ++b) {
    const int buf = (b - b0) & 1;
    if (b + 1 < b1) load_page(b + 1, buf ^ 1);
    if (!mbar_wait(&full[buf], ((b - b0) >> 1) & 1, &abort_flag, p.status, kTimeoutProducer)) abort_flag = 1;
    __syncthreads();
    if (abort_flag) break;                       // every thread sees the same value here
    const uint32_t aK = ms_addr(sKV + buf * kPage * ld);
    float s[kTiles][4];
#pragma unroll
    for (int j = 0; j < kTiles; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
#pragma unroll
    for (int k = 0; k < KS; ++k)
      if (k < n_steps) {
#pragma unroll
        for (int np = 0; np < MT; ++np) {
          uint32_t fb[4];
          ms_ldsm4(ms_b_nt_at(aK, ld, (kg * MT + np) * 16, (s0 + k) * 16, lane), fb);
          ms_mma(s[2 * np], qf[k], fb[0], fb[1]);
          ms_mma(s[2 * np + 1], qf[k], fb[2], fb[3]);
        }
      }
#pragma unroll
    for (int j = 0; j < kTiles; ++j)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf)
        *reinterpret_cast<float2*>(sS + (slice * RT + row_tile * 16 + g4 + 8 * hf) * kLdS + kg * MT * 16 + j * 8 + 2 * t4) =
            make_float2(s[j][2 * hf], s[j][2 * hf + 1]);
    __syncthreads();
    float x[kRows][2], mx[kRows];
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int r = warp * kRows + i, lim = prior + (row0 + r) / p.H;        // last key this row sees
      float2 v = make_float2(0.f, 0.f);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 w = *reinterpret_cast<const float2*>(sS + (q * RT + r) * kLdS + 2 * lane);
        v.x += w.x;
        v.y += w.y;
      }
      const int j = b * kPage + 2 * lane;
      x[i][0] = j <= lim ? v.x * p.scale_log2 : -CUDART_INF_F;
      x[i][1] = j + 1 <= lim ? v.y * p.scale_log2 : -CUDART_INF_F;
      mx[i] = fmaxf(x[i][0], x[i][1]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int i = 0; i < kRows; ++i) mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], o));
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int r = warp * kRows + i;
      const float m_new = fmaxf(m_run[i], mx[i]), m_use = m_new == -CUDART_INF_F ? 0.f : m_new;
      const float corr = exp2f(m_run[i] - m_use), e0 = exp2f(x[i][0] - m_use), e1 = exp2f(x[i][1] - m_use);
      l_run[i] = l_run[i] * corr + e0 + e1;      // this lane's keys; the lanes meet at the end
      m_run[i] = m_new;
      *reinterpret_cast<uint32_t*>(sP + r * kLdP + 2 * lane) = pack_bf16(e0, e1);
      if (lane == 0) sCorr[r] = corr;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const float c0 = sCorr[i * 16 + g4], c1 = sCorr[i * 16 + g4 + 8];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        acc[i][j][0] *= c0; acc[i][j][1] *= c0;
        acc[i][j][2] *= c1; acc[i][j][3] *= c1;
      }
    }
#pragma unroll
    for (int kk = 0; kk < kPage; kk += 16) {
      uint32_t fp[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ms_ldsm4(ms_a_at(aP, kLdP, i * 16, kk, lane), fp[i]);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {      // column tiles j and j + 1 in one load where both exist
        const int tile = warp + 16 * j, next = NT > 1 && tile + 16 < n8 ? tile + 16 : tile;
        if (tile < n8) {
          uint32_t fb[4];
          ms_ldsm4_t(aK + static_cast<uint32_t>(((kk + (lane & 15)) * ld + (lane < 16 ? tile : next) * 8) * 2), fb);
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            ms_mma(acc[i][j], fp[i], fb[0], fb[1]);
            if (NT > 1 && next != tile) ms_mma(acc[i][j + (NT > 1 ? 1 : 0)], fp[i], fb[2], fb[3]);
          }
        }
      }
    }
    __syncthreads();                  // the page buffer, scores and probabilities may be overwritten
  }
  if (abort_flag) {                   // abandoned wait: the copies in flight get one more limit to land before the CTA leaves
    __syncthreads();
    if (threadIdx.x == 0) {
      const unsigned long long t0 = globaltimer_ns();
      while (globaltimer_ns() - t0 < kWaitLimitNs) {}
    }
    __syncthreads();
    return;
  }
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const int r = warp * kRows + i;
    const float l = warp_sum(l_run[i]);
    if (lane == 0 && row0 + r < n_rows) {
      p.part_ml[(part_base + r) * 2] = m_run[i];
      p.part_ml[(part_base + r) * 2 + 1] = l;
    }
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int r = i * 16 + g4 + 8 * hf, c = (warp + 16 * j) * 8 + 2 * t4;
        if (row0 + r >= n_rows || c >= p.rank) continue;
        float* dst = p.part_o + (part_base + r) * p.rank + c;
        if (p.rank % 2 == 0) {
          *reinterpret_cast<float2*>(dst) = make_float2(acc[i][j][2 * hf], acc[i][j][2 * hf + 1]);
        } else {
          dst[0] = acc[i][j][2 * hf];
          if (c + 1 < p.rank) dst[1] = acc[i][j][2 * hf + 1];
        }
      }
}

// out[rows[i], h, v] = W_uv[h, v, :] . (joined splits of row (i, h)). grid (H, groups of kUpTok tokens, chunks of value
// channels); a CTA joins the rows of its tokens and shares the weight rows between them. V: elements per weight load.
constexpr int kUpTok = 4;
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_up_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                        const T* __restrict__ wuv, const int* __restrict__ rows, int n, int H,
                                                        int dv, int rank, int n_split, T* __restrict__ out, long long ldo) {
  extern __shared__ __align__(16) float up_o[];            // [kUpTok][rank]
  __shared__ float coef[kUpTok][64];
  const int h = blockIdx.x, t0 = blockIdx.y * kUpTok, n_tok = min(kUpTok, n - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long part_rows = static_cast<long long>(n) * H;
  if (warp < n_tok) {                        // n_split <= 64: two splits per lane
    const float* ml = part_ml + (static_cast<long long>(t0 + warp) * H + h) * 2;
    float m0 = -CUDART_INF_F, m1 = -CUDART_INF_F, l0 = 0.f, l1 = 0.f;
    if (lane < n_split) { m0 = ml[lane * part_rows * 2]; l0 = ml[lane * part_rows * 2 + 1]; }
    if (lane + 32 < n_split) { m1 = ml[(lane + 32) * part_rows * 2]; l1 = ml[(lane + 32) * part_rows * 2 + 1]; }
    float mx = fmaxf(m0, m1);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float e0 = l0 > 0.f ? exp2f(m0 - mx) : 0.f, e1 = l1 > 0.f ? exp2f(m1 - mx) : 0.f;
    const float inv = 1.f / warp_sum(e0 * l0 + e1 * l1);
    coef[warp][lane] = e0 * inv;
    coef[warp][lane + 32] = e1 * inv;
  }
  __syncthreads();
  constexpr int JV = V >= 4 ? 4 : 1;
  for (int i = threadIdx.x * JV; i < kUpTok * rank; i += 256 * JV) {
    const int t = i / rank, c = i - t * rank;
    float v[JV];
#pragma unroll
    for (int e = 0; e < JV; ++e) v[e] = 0.f;
    if (t < n_tok) {
      const float* src = part_o + (static_cast<long long>(t0 + t) * H + h) * rank + c;
#pragma unroll 8
      for (int s = 0; s < n_split; ++s) {    // an empty split left its rows unwritten: read those of the first one
        const float w = coef[t][s];
        float x[JV];
        load_vec<JV>(src + (w != 0.f ? s : 0) * part_rows * rank, x);
#pragma unroll
        for (int e = 0; e < JV; ++e) v[e] = fmaf(w, x[e], v[e]);
      }
    }
    store_vec<JV>(up_o + i, v);
  }
  __syncthreads();
  const int per = (dv + gridDim.z - 1) / gridDim.z, r1 = min(dv, (static_cast<int>(blockIdx.z) + 1) * per);
  for (int r = blockIdx.z * per + warp; r < r1; r += 16) {         // rows r and r + 8
    const bool two = r + 8 < r1;
    const T* w = wuv + (static_cast<long long>(h) * dv + r) * rank;
    const T* w2 = two ? w + 8ll * rank : w;
    float acc[2][kUpTok];
#pragma unroll
    for (int t = 0; t < kUpTok; ++t) acc[0][t] = acc[1][t] = 0.f;
#pragma unroll 2
    for (int c = lane * V; c < rank; c += 32 * V) {
      float wv[V], wv2[V];
      load_vec<V>(w + c, wv);
      load_vec<V>(w2 + c, wv2);
#pragma unroll
      for (int t = 0; t < kUpTok; ++t) {
        float x[V];
        load_vec<V>(up_o + t * rank + c, x);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          acc[0][t] = fmaf(wv[e], x[e], acc[0][t]);
          acc[1][t] = fmaf(wv2[e], x[e], acc[1][t]);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < 2; ++k)
#pragma unroll
      for (int t = 0; t < kUpTok; ++t) acc[k][t] = warp_sum(acc[k][t]);
    const int t = lane & (kUpTok - 1), k = lane / kUpTok;          // lane (k, t) writes row r + 8 k of token t
    if (t < n_tok && (k == 0 || (k == 1 && two))) {
      float v = 0.f;
#pragma unroll
      for (int kk = 0; kk < 2; ++kk)
#pragma unroll
        for (int tt = 0; tt < kUpTok; ++tt)
          if (k == kk && t == tt) v = acc[kk][tt];
      put(out + rows[t0 + t] * ldo + h * dv + r + 8 * k, v);
    }
  }
}

// ------------------------------------------------------------------------------------------- expanded keys and values
// lat [n, R8] (R8 >= rank, zero padded) = latents of the n cache rows in `slots` (page * 64 + offset).
__global__ void latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const long long* __restrict__ slots, int n, int W,
                                     int rank, int r8, __nv_bfloat16* __restrict__ lat) {
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < static_cast<long long>(n) * r8;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int j = static_cast<int>(i / r8), c = static_cast<int>(i - static_cast<long long>(j) * r8);
    const __nv_bfloat16* src = cache + slots[j] * (W + kRowPad);
    lat[i] = c < rank ? src[c] : __float2bfloat16(0.f);
  }
}
__global__ void latent_gather8_kernel(const __nv_bfloat16* __restrict__ cache, const long long* __restrict__ slots, int n, int W,
                                      int rank, __nv_bfloat16* __restrict__ lat) {
  const int per = rank / 8;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < static_cast<long long>(n) * per;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int j = static_cast<int>(i / per), c = static_cast<int>(i - static_cast<long long>(j) * per) * 8;
    const __nv_bfloat16* src = cache + slots[j] * (W + kRowPad);
    *reinterpret_cast<uint4*>(lat + static_cast<long long>(j) * rank + c) = *reinterpret_cast<const uint4*>(src + c);
  }
}

// Query / key / value operands of the 128-channel attention kernels, zero padded. kv [n, ldkv]: H heads of D_n key
// channels, then H heads of D_v value channels. blockIdx.y: 0 = queries (n_q rows of qd), 1 = keys, 2 = values.
// A thread writes 8 channels. Operands without a destination are left out.
__global__ void latent_assemble_kernel(const __nv_bfloat16* __restrict__ qd, long long ldq, int n_q,
                                       const __nv_bfloat16* __restrict__ kv, long long ldkv, int n,
                                       const __nv_bfloat16* __restrict__ cache, const long long* __restrict__ slots, int W, int rank,
                                       int H, int dn, int dr, int dv, __nv_bfloat16* __restrict__ q128,
                                       __nv_bfloat16* __restrict__ k128, __nv_bfloat16* __restrict__ v128) {
  const int what = blockIdx.y;
  __nv_bfloat16* to = what == 0 ? q128 : (what == 1 ? k128 : v128);
  if (!to) return;
  const long long rows = static_cast<long long>(what == 0 ? n_q : n) * H;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < rows * 16;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i >> 4;
    const int c0 = static_cast<int>(i & 15) * 8, h = static_cast<int>(r % H);
    const long long t = r / H;
    __nv_bfloat16* dst = to + r * 128 + c0;
    const __nv_bfloat16 *a, *b = nullptr;      // channels [0, na) from a, [na, nb) from b
    int na, nb;
    if (what == 0) {
      a = qd + t * ldq + h * (dn + dr);
      na = nb = dn + dr;
    } else if (what == 1) {
      a = kv + t * ldkv + h * dn;
      b = cache + slots[t] * (W + kRowPad) + rank;
      na = dn;
      nb = dn + dr;
    } else {
      a = kv + t * ldkv + static_cast<long long>(H) * dn + h * dv;
      na = nb = dv;
    }
    uint32_t w[4];
    const bool from_a = c0 + 8 <= na, from_b = b && c0 >= na && c0 + 8 <= nb;
    const __nv_bfloat16* src = from_a ? a + c0 : b + (c0 - na);
    if ((from_a || from_b) && !(reinterpret_cast<uintptr_t>(src) & 15)) {
      *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
      continue;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float v[2];
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int c = c0 + 2 * e + f;
        v[f] = c < na ? __bfloat162float(a[c]) : (c < nb ? __bfloat162float(b[c - na]) : 0.f);
      }
      w[e] = pack_bf16(v[0], v[1]);
    }
    *reinterpret_cast<uint4*>(dst) = make_uint4(w[0], w[1], w[2], w[3]);
  }
}

// Rows of [n, H, 128] back to [n, H * dv] (row stride ldo).
__global__ void latent_take_kernel(const __nv_bfloat16* __restrict__ o128, int n, int H, int dv, __nv_bfloat16* __restrict__ out,
                                   long long ldo) {
  const long long total = static_cast<long long>(n) * H * dv;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int c = static_cast<int>(i % dv);
    const long long r = i / dv;
    out[(r / H) * ldo + (r % H) * dv + c] = o128[r * 128 + c];
  }
}

static size_t latent_mma_smem(int mt, int W) {
  const size_t rt = 16 * mt, ld = W + 8;
  return (2 * kPage * ld + rt * kLdP) * 2 + (4 * rt * kLdS + rt) * 4;
}
static int latent_mma_tiles(int H, int W) {      // 16-row tiles per CTA, 0: not covered
  if (H > 16 && latent_mma_smem(2, W) <= 220 * 1024) return 2;
  return latent_mma_smem(1, W) <= 220 * 1024 ? 1 : 0;
}

template <int MT, int KS, int NT>
static int latent_mma_launch(const LatentParams& p, dim3 grid, size_t smem, cudaStream_t st) {
  static DeviceMax configured;
  if (smem > configured.get()) {
    const cudaError_t e = cudaFuncSetAttribute(latent_attn_mma_kernel<MT, KS, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.set(smem);
  }
  latent_attn_mma_kernel<MT, KS, NT><<<grid, kMmaThreads, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int latent_absorb_launch(const void* qd, long long ld, const void* wuk, int H, int dn, int dr, int rank, int W,
                                const int* rows, int n, int tiles, size_t smem, void* out, const void* wuv, int dv,
                                const float* cs, const float* sn, cudaStream_t st) {
  const dim3 grid((rank + 127) / 128 + 1, H, tiles);
  const T *q = static_cast<const T*>(qd), *w = static_cast<const T*>(wuk), *v = static_cast<const T*>(wuv);
  // bulk prefetches take whole 16-byte pieces
  const size_t head = static_cast<size_t>(dv) * rank * sizeof(T);
  const unsigned bytes = head % 16 == 0 && !(reinterpret_cast<uintptr_t>(v) & 15) ? static_cast<unsigned>(head) : 0;
  if (rank % 2 == 0) latent_absorb_kernel<T, 2><<<grid, 256, smem, st>>>(q, ld, w, H, dn, dr, rank, W, rows, n, static_cast<T*>(out), v, bytes, cs, sn);
  else latent_absorb_kernel<T, 1><<<grid, 256, smem, st>>>(q, ld, w, H, dn, dr, rank, W, rows, n, static_cast<T*>(out), v, bytes, cs, sn);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int latent_up_launch(const float* part_o, const float* part_ml, const void* wuv, const int* rows, int n, int H, int dv,
                            int rank, int n_split, dim3 grid, size_t smem, void* out, long long ldo, cudaStream_t st) {
  const T* w = static_cast<const T*>(wuv);
  T* o = static_cast<T*>(out);
  // whole 16-byte pieces need aligned weight rows (the value weights may lie behind the keys' in one allocation)
  const int v = rank % 8 == 0 && !(reinterpret_cast<uintptr_t>(w) & 15) ? 8 : 1;
  if (v == 8) latent_up_kernel<T, 8><<<grid, 256, smem, st>>>(part_o, part_ml, w, rows, n, H, dv, rank, n_split, o, ldo);
  else latent_up_kernel<T, 1><<<grid, 256, smem, st>>>(part_o, part_ml, w, rows, n, H, dv, rank, n_split, o, ldo);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace pm

using namespace pm;

// qd [n, ld]: the queries' rotated parts are turned in place; with cache != null the down-projection behind the queries is
// normed / rotated and written to row slots[t] of cache [.., W + 8]. cs / sn [n, dr / 2]. lead > 0 (with H = 0): qd begins with
// a query latent of that many channels, which is normed in place with the weight lead_w (fp32).
extern "C" int pm_latent_prep(void* qd, int f32, long long ld, const float* norm_w, float eps, const float* cs,
                              const float* sn, int n, int H, int dn, int dr, int rank, void* cache, int W,
                              const long long* slots, int lead, const float* lead_w, cudaStream_t st) {
  if (n < 0 || H < 0 || lead < 0 || (H == 0) != (lead > 0) || (lead && !lead_w) || dn < 0 || dr < 0 || (dr & 1) || rank < 1 || W < rank + dr) return -1;
  if (ld < static_cast<long long>(H) * (dn + dr) + lead + (cache ? rank + dr : 0)) return -2;
  if (n == 0) return 0;
  const int own = cache != nullptr;
  if (f32) {
    latent_prep_kernel<float, 1><<<n, 128, 0, st>>>(static_cast<float*>(qd), ld, norm_w, eps, cs, sn, H, dn, dr, rank, own,
                                                    static_cast<float*>(cache), W, slots, lead, lead_w);
  } else {
    const bool vec = ((H * (dn + dr)) | lead | (own ? rank : 0) | static_cast<int>(ld % 8)) % 8 == 0 && reinterpret_cast<uintptr_t>(qd) % 16 == 0;
    const auto kernel = vec ? latent_prep_kernel<__nv_bfloat16, 8> : latent_prep_kernel<__nv_bfloat16, 1>;
    kernel<<<n, 128, 0, st>>>(static_cast<__nv_bfloat16*>(qd), ld, norm_w, eps, cs, sn, H, dn, dr, rank, own,
                              static_cast<__nv_bfloat16*>(cache), W, slots, lead, lead_w);
  }
  return static_cast<int>(cudaGetLastError());
}

// Whether the tensor-core kernel covers H heads over rows of W columns with `rank` value columns.
extern "C" int pm_latent_mma_supported(int H, int W, int rank) {
  return W % 16 == 0 && W <= 640 && rank <= 512 && latent_mma_tiles(H, W) > 0;
}

// Attention of short portions in the latent space. qd as pm_latent_prep leaves it, wuk [H * dn, rank], wuv [H * dv, rank],
// cache [pages, 64, W + 8]. The n_tok tokens of the listed sequences are counted through: sequence i covers compact tokens
// c_start[i] .. of the work buffers q_lat [n_tok, H, W], part_o [n_split, n_tok * H, rank] fp32 and part_ml [n_split,
// n_tok * H, 2] fp32, and compact token j is row tok_rows[j] of qd and out. out [.., ldo]: H * dv columns. max_q: longest of
// q_lens. cs / sn (nullable) [.., dr / 2]: the queries' rotated parts are still to be turned. n_split <= 64 (1 for fp32 and for sizes that the tensor-core kernel does not cover).
extern "C" int pm_latent_attn(const void* qd, int f32, long long ld, const void* wuk, const void* wuv, const void* cache,
                              const int* block_table, const int* seq_lens, const int* c_start, const int* q_lens,
                              const int* tok_rows, int n_seq, int max_blocks, int n_tok, int max_q, int H, int dn, int dr,
                              int dv, int rank, int W, int n_split, float scale, void* q_lat, float* part_o, float* part_ml,
                              void* out, long long ldo, const float* cs, const float* sn, int* status, cudaStream_t st) {
  if (H < 1 || rank < 1 || W < rank + dr || dv < 1 || n_split < 1 || n_split > 64 || ldo < static_cast<long long>(H) * dv)
    return -1;
  if (n_seq < 1 || max_q < 1 || n_tok < 1) return 0;
  const bool mma = !f32 && pm_latent_mma_supported(H, W, rank);
  if (!mma && n_split != 1) return -2;
  const size_t sm_abs = static_cast<size_t>(kAbsTok) * (dn + 512) * 4, sm_row = (static_cast<size_t>(W) + rank + kPage) * 4,
               sm_up = static_cast<size_t>(kUpTok) * rank * 4;
  if (sm_abs > 48 * 1024 || (!mma && sm_row > 48 * 1024) || sm_up > 46 * 1024) return -3;
  const int abs_tiles = (n_tok + kAbsTok - 1) / kAbsTok, up_tiles = (n_tok + kUpTok - 1) / kUpTok;
  if (abs_tiles > 65535 || up_tiles > 65535) return -4;
  int rc = f32 ? latent_absorb_launch<float>(qd, ld, wuk, H, dn, dr, rank, W, tok_rows, n_tok, abs_tiles, sm_abs, q_lat, wuv, dv, cs, sn, st)
               : latent_absorb_launch<__nv_bfloat16>(qd, ld, wuk, H, dn, dr, rank, W, tok_rows, n_tok, abs_tiles, sm_abs, q_lat, wuv, dv, cs, sn, st);
  if (rc) return rc;
  LatentParams p{};
  p.q = q_lat; p.cache = cache; p.block_table = block_table; p.seq_lens = seq_lens; p.c_start = c_start; p.q_lens = q_lens;
  p.part_o = part_o; p.part_ml = part_ml; p.max_blocks = max_blocks; p.H = H; p.W = W; p.rank = rank; p.n_split = n_split;
  p.rows = static_cast<long long>(n_tok) * H;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = status;
  if (mma) {
    const int mt = latent_mma_tiles(H, W), rt = 16 * mt;
    p.row_tiles = (max_q * H + rt - 1) / rt;
    const dim3 grid(p.row_tiles * n_seq, n_split);
    const size_t smem = latent_mma_smem(mt, W);
    // (steps per quarter, column tiles per warp): the smallest instance that holds both
    const int size = W <= 128 && rank <= 128 ? 0 : (W <= 320 && rank <= 256 ? 1 : 2);
    if (mt == 1)
      rc = size == 0 ? latent_mma_launch<1, 2, 1>(p, grid, smem, st) : size == 1 ? latent_mma_launch<1, 5, 2>(p, grid, smem, st)
                                                                                 : latent_mma_launch<1, 10, 4>(p, grid, smem, st);
    else
      rc = size == 0 ? latent_mma_launch<2, 2, 1>(p, grid, smem, st) : size == 1 ? latent_mma_launch<2, 5, 2>(p, grid, smem, st)
                                                                                 : latent_mma_launch<2, 10, 4>(p, grid, smem, st);
    if (rc) return rc;
  } else {
    const dim3 grid(max_q * H, n_seq);
    if (f32) latent_attn_row_kernel<float><<<grid, 128, sm_row, st>>>(p);
    else latent_attn_row_kernel<__nv_bfloat16><<<grid, 128, sm_row, st>>>(p);
    const cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  // few heads and tokens: the value channels are cut so that the launch still fills the machine
  int cut = (2 * num_sms() + H * up_tiles - 1) / (H * up_tiles);
  const int most = (dv + 7) / 8;
  if (cut > most) cut = most;
  const dim3 g_up(H, up_tiles, cut);
  return f32 ? latent_up_launch<float>(part_o, part_ml, wuv, tok_rows, n_tok, H, dv, rank, n_split, g_up, sm_up, out, ldo, st)
             : latent_up_launch<__nv_bfloat16>(part_o, part_ml, wuv, tok_rows, n_tok, H, dv, rank, n_split, g_up, sm_up, out, ldo, st);
}

// lat [n, r8] bf16 = latents of the n cache rows in `slots` (page * 64 + offset; zero padded).
extern "C" int pm_latent_gather(const void* cache, const long long* slots, int n, int W, int rank, int r8, void* lat,
                                cudaStream_t st) {
  if (n < 0 || rank < 1 || r8 < rank || W < rank) return -1;
  if (n == 0) return 0;
  const bool vec = rank == r8 && rank % 8 == 0 && W % 8 == 0;
  long long grid = (static_cast<long long>(n) * (vec ? rank / 8 : r8) + 255) / 256;
  if (grid > num_sms() * 16) grid = num_sms() * 16;
  if (vec)
    latent_gather8_kernel<<<static_cast<int>(grid), 256, 0, st>>>(static_cast<const __nv_bfloat16*>(cache), slots, n, W, rank,
                                                                  static_cast<__nv_bfloat16*>(lat));
  else
    latent_gather_kernel<<<static_cast<int>(grid), 256, 0, st>>>(static_cast<const __nv_bfloat16*>(cache), slots, n, W, rank,
                                                                 r8, static_cast<__nv_bfloat16*>(lat));
  return static_cast<int>(cudaGetLastError());
}

// Operands [.., H, 128] bf16 of the flash-attention kernels for n_q queries and the n keys in `slots`; dn + dr <= 128,
// dv <= 128. qd: the first query row; kv [n, ldkv] = [keys: H * dn | values: H * dv].
extern "C" int pm_latent_assemble(const void* qd, long long ldq, int n_q, const void* kv, long long ldkv, int n,
                                  const void* cache, const long long* slots, int W, int rank, int H, int dn, int dr, int dv,
                                  void* q128, void* k128, void* v128, cudaStream_t st) {
  if (n_q < 1 || n < 1 || H < 1 || dn + dr > 128 || dv > 128 || W < rank + dr) return -1;
  long long grid = (static_cast<long long>(n > n_q ? n : n_q) * H * 16 + 255) / 256;
  if (grid > num_sms() * 16) grid = num_sms() * 16;
  latent_assemble_kernel<<<dim3(static_cast<int>(grid), 3), 256, 0, st>>>(
      static_cast<const __nv_bfloat16*>(qd), ldq, n_q, static_cast<const __nv_bfloat16*>(kv), ldkv, n,
      static_cast<const __nv_bfloat16*>(cache), slots, W, rank, H, dn, dr, dv, static_cast<__nv_bfloat16*>(q128),
      static_cast<__nv_bfloat16*>(k128), static_cast<__nv_bfloat16*>(v128));
  return static_cast<int>(cudaGetLastError());
}

// out [n, ldo] (H * dv columns) = the first dv channels of every head of o128 [n, H, 128].
extern "C" int pm_latent_take(const void* o128, int n, int H, int dv, void* out, long long ldo, cudaStream_t st) {
  if (n < 1 || H < 1 || dv < 1 || dv > 128) return -1;
  long long grid = (static_cast<long long>(n) * H * dv + 255) / 256;
  if (grid > num_sms() * 16) grid = num_sms() * 16;
  latent_take_kernel<<<static_cast<int>(grid), 256, 0, st>>>(static_cast<const __nv_bfloat16*>(o128), n, H, dv,
                                                             static_cast<__nv_bfloat16*>(out), ldo);
  return static_cast<int>(cudaGetLastError());
}
