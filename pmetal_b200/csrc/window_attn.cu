// Grouped-query attention over a paged cache for heads of any size, with an optional sliding window: position i sees the keys
// j with 0 <= i - j < window (every j <= i when window is 0). Per token and layer the cache holds one row
// [head 0: k | v, head 1: k | v, ..] with D8 channels each (the head size D rounded up to 8, zeros behind it).
//
//   window_prep_kernel  rotation of queries and keys on their first R channels, optional division by their root mean square
//                       over the head, cache append. Values are the keys as projected, or columns of their own.
//   window_mma_kernel   bf16, mma.sync on 64-key pages in shared memory (two in flight), online softmax in base 2. Rows are
//                       (query token, head of the group) pairs of one (sequence, key/value head). Prefill: 64 rows, a warp
//                       owns 16 of them. Decode: 16 rows, the four warps share them and split the keys of every page, and
//                       CTAs split the pages; the parts are merged in shared memory and by window_combine_kernel. Pages
//                       outside every row's window are not visited.
//   window_row_kernel   any type and size, one (token, head) per CTA (fp32 models, heads beyond 256 channels)
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math_constants.h>
#include <stdint.h>
#include "elem.cuh"
#include "host_util.cuh"
#include "mma_sync.cuh"
#include "pmetal_b200.h"

namespace pm {

constexpr int kWinPage = 64;
constexpr int kWinMaxHead = 1024;

template <typename T>
struct WindowPrepParams {
  const T* u;                // [tokens, ldu]: q [H D], k [G D] (, v [G D])
  long long ldu;
  const float* cs;           // [tokens, R / 2]
  const float* sn;
  T* q;                      // [tokens, H, D8]
  T* pages;                  // [block][64][G][2][D8]
  const long long* slots;    // page * 64 + offset of every token
  int n_tok, H, G, D, D8, R, pairs, normed, own_v;
  float eps;
};

// One warp per (token, head of q or k).
template <typename T>
__global__ void __launch_bounds__(256) window_prep_kernel(const WindowPrepParams<T> p) {
  const int heads = p.H + p.G, lane = threadIdx.x & 31;
  const long long item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const long long t = item / heads;
  if (t >= p.n_tok) return;
  const int h = static_cast<int>(item - t * heads);
  const bool key = h >= p.H;
  const T* src = p.u + t * p.ldu + static_cast<long long>(h) * p.D;
  float scale = 1.f;
  if (p.normed) {            // a rotation keeps the sum of squares
    float ss = 0.f;
    for (int c = lane; c < p.D; c += 32) {
      const float v = to_f(src[c]);
      ss = fmaf(v, v, ss);
    }
    scale = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.D) + p.eps);
  }
  T* row = p.pages + (p.slots[t] * p.G + (h - p.H)) * 2 * p.D8;
  T* dst = key ? row : p.q + (t * p.H + h) * p.D8;
  const int half = p.R / 2;
  const float* cs = p.cs + t * half;
  const float* sn = p.sn + t * half;
  const T* vsrc = p.own_v ? src + static_cast<long long>(p.G) * p.D : src;
  for (int c = lane; c < p.D8; c += 32) {
    float v = 0.f;
    if (c < p.D) {
      v = to_f(src[c]);
      if (c < p.R) {
        const bool second = p.pairs ? (c & 1) : c >= half;
        const int f = p.pairs ? c >> 1 : (second ? c - half : c);
        const float w = to_f(src[p.pairs ? c ^ 1 : (second ? c - half : c + half)]);
        v = fmaf(v, cs[f], second ? w * sn[f] : -w * sn[f]);
      }
      v *= scale;
    }
    put(dst + c, v);
    if (key) put(row + p.D8 + c, c < p.D ? to_f(vsrc[c]) : 0.f);
  }
}

// The same for heads in 8-channel pieces (bf16, D <= 256): a lane owns 8 channels of a head, gs lanes a head (gs: power of two).
__global__ void __launch_bounds__(256) window_prep_vec_kernel(const WindowPrepParams<__nv_bfloat16> p, int gs) {
  const int heads = p.H + p.G, lane = threadIdx.x & 31, per = 32 / gs;
  const long long item = (blockIdx.x * 8ll + (threadIdx.x >> 5)) * per + lane / gs;
  const long long t = item / heads;
  const bool live = t < p.n_tok;
  const int h = live ? static_cast<int>(item - t * heads) : 0, c = (lane % gs) * 8;
  const bool key = h >= p.H, mine = live && c < p.D;
  const __nv_bfloat16* src = p.u + (live ? t : 0) * p.ldu + static_cast<long long>(h) * p.D;
  float v[8], raw[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) raw[e] = 0.f;
  if (mine) load_vec<8>(src + c, raw);
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    v[e] = raw[e];
    ss = fmaf(v[e], v[e], ss);
  }
  for (int o = gs / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float scale = p.normed ? 1.f / sqrtf(ss / static_cast<float>(p.D) + p.eps) : 1.f;
  if (!mine) return;
  const int half = p.R / 2;
  const float* cs = p.cs + t * half;
  const float* sn = p.sn + t * half;
  if (c < p.R) {
    if (p.pairs) {
      float a[4], b[4];
      load_vec<4>(cs + c / 2, a);
      load_vec<4>(sn + c / 2, b);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[2 * i] = fmaf(raw[2 * i], a[i], -raw[2 * i + 1] * b[i]);
        v[2 * i + 1] = fmaf(raw[2 * i + 1], a[i], raw[2 * i] * b[i]);
      }
    } else {
      const bool second = c >= half;
      float a[8], b[8], w[8];
      load_vec<8>(src + (second ? c - half : c + half), w);
      load_vec<8>(cs + (second ? c - half : c), a);
      load_vec<8>(sn + (second ? c - half : c), b);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = fmaf(raw[e], a[e], second ? w[e] * b[e] : -w[e] * b[e]);
    }
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] *= scale;
  if (!key) {
    store_vec<8>(p.q + (t * p.H + h) * p.D8 + c, v);
    return;
  }
  __nv_bfloat16* row = p.pages + (p.slots[t] * p.G + (h - p.H)) * 2 * p.D8 + c;
  store_vec<8>(row, v);
  if (p.own_v) load_vec<8>(src + static_cast<long long>(p.G) * p.D + c, raw);
  store_vec<8>(row + p.D8, raw);
}

template <typename T>
struct WindowParams {
  const T* q;                // [tokens, H, D8]
  const T* pages;
  T* out;                    // [tokens, ldo], head h at column h D
  long long ldo;
  const int* block_table;
  const int* seq_lens;
  const int* q_start;
  const int* q_lens;
  float* po;                 // [n_split][n_tok][H][D8] and [n_split][n_tok][H][2], n_split > 1
  float* pml;
  int n_tok, max_blocks, H, G, rep, D, D8, window, n_split;
  float scale;
};

// First visible key of the query at position pos.
__device__ __forceinline__ int window_first(int pos, int window) { return window > 0 ? max(0, pos - window + 1) : 0; }

// KD: 16-channel steps of the head. KEYW: warps that share 16 rows and split the keys of a page (1 or 4).
template <int KD, int KEYW>
__global__ void __launch_bounds__(128) window_mma_kernel(const WindowParams<__nv_bfloat16> p) {
  extern __shared__ __align__(16) uint8_t win_smem[];
  constexpr int kRows = 64 / KEYW, DP = KD * 16, LD = DP + 8, NT = 8 / KEYW;      // NT: 8-key tiles per warp
  constexpr int kTile = kWinPage * LD;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(win_smem);        // [kRows][LD]
  __nv_bfloat16* sK = sQ + kRows * LD;                                   // [2][64][LD]
  __nv_bfloat16* sV = sK + 2 * kTile;                                    // [2][64][LD]
  const int g = blockIdx.y, seq = blockIdx.z / p.n_split, split = blockIdx.z % p.n_split;
  const int len = p.q_lens[seq], r0 = blockIdx.x * kRows, n_rows = min(kRows, len * p.rep - r0);
  if (n_rows <= 0) return;
  const int q0 = p.q_start[seq], base = p.seq_lens[seq] - len;           // position of the first new token
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p_lo = base + r0 / p.rep, p_hi = base + (r0 + n_rows - 1) / p.rep;      // positions of the first and last row
  const int b_all = window_first(p_lo, p.window) / kWinPage, n_all = p_hi / kWinPage + 1 - b_all;
  const int per = (n_all + p.n_split - 1) / p.n_split;
  const int b0 = b_all + split * per, b1 = min(b0 + per, b_all + n_all);

  const int vec = p.D8 / 8;                                              // 16-byte pieces of a row that exist
  for (int i = threadIdx.x; i < kRows * KD * 2; i += 128) {
    const int r = i / (KD * 2), c = i % (KD * 2);
    const bool ok = r < n_rows && c < vec;
    const int row = r0 + (ok ? r : 0);
    const __nv_bfloat16* src = p.q + (static_cast<long long>(q0 + row / p.rep) * p.H + g * p.rep + row % p.rep) * p.D8 + (ok ? c * 8 : 0);
    ms_cp16(ms_addr(sQ + r * LD + c * 8), src, ok);
  }
  const int* table = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  auto load_page = [&](int b, int buf) {
    const __nv_bfloat16* src = p.pages + (static_cast<long long>(table[b]) * kWinPage * p.G + g) * 2 * p.D8;
    for (int i = threadIdx.x; i < kWinPage * KD * 2; i += 128) {
      const int r = i / (KD * 2), c = i % (KD * 2);
      const bool ok = c < vec;
      const __nv_bfloat16* at = src + static_cast<long long>(r) * p.G * 2 * p.D8 + (ok ? c * 8 : 0);
      ms_cp16(ms_addr(sK + buf * kTile + r * LD + c * 8), at, ok);
      ms_cp16(ms_addr(sV + buf * kTile + r * LD + c * 8), at + p.D8, ok);
    }
  };
  if (b0 < b1) load_page(b0, 0);
  ms_commit();

  const int wr = KEYW == 1 ? warp * 16 : 0, wk = KEYW == 1 ? 0 : warp * (kWinPage / KEYW);     // this warp's rows and keys
  const int g4 = lane >> 2, t4 = lane & 3;
  int pos[2], first[2];
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = wr + g4 + 8 * hf;
    pos[hf] = r < n_rows ? base + (r0 + r) / p.rep : -1;                 // rows that do not exist see nothing
    first[hf] = window_first(pos[hf], p.window);
  }
  float o[2 * KD][4], m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2 * KD; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  const float a2 = p.scale * 1.4426950408889634f;
  const uint32_t aQ = ms_addr(sQ);
  const bool idle = wr >= n_rows;

  for (int b = b0; b < b1; ++b) {
    const int buf = (b - b0) & 1;
    if (b + 1 < b1) load_page(b + 1, buf ^ 1);
    ms_commit();
    ms_wait<1>();
    __syncthreads();
    if (!idle) {
      const uint32_t aK = ms_addr(sK + buf * kTile), aV = ms_addr(sV + buf * kTile);
      float s[NT][4];
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
#pragma unroll
      for (int k = 0; k < KD; ++k) {
        uint32_t fa[4];
        ms_ldsm4(ms_a_at(aQ, LD, wr, k * 16, lane), fa);
#pragma unroll
        for (int n = 0; n < NT / 2; ++n) {
          uint32_t fb[4];
          ms_ldsm4(ms_b_nt_at(aK, LD, wk + n * 16, k * 16, lane), fb);
          ms_mma(s[2 * n], fa, fb[0], fb[1]);
          ms_mma(s[2 * n + 1], fa, fb[2], fb[3]);
        }
      }
      const int j0 = b * kWinPage + wk + 2 * t4;
      const bool whole = b * kWinPage + kWinPage - 1 <= p_lo && b * kWinPage >= window_first(p_hi, p.window) && n_rows == kRows;
      float mx[2] = {m[0], m[1]};
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int hf = e >> 1, j = j0 + n * 8 + (e & 1);
          s[n][e] = whole || (j <= pos[hf] && j >= first[hf]) ? s[n][e] * a2 : -CUDART_INF_F;
          mx[hf] = fmaxf(mx[hf], s[n][e]);
        }
      float keep[2], at[2];
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 1));
        mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 2));
        at[hf] = mx[hf] == -CUDART_INF_F ? 0.f : mx[hf];
        keep[hf] = exp2f(m[hf] - at[hf]);
        m[hf] = mx[hf];
        l[hf] *= keep[hf];
      }
#pragma unroll
      for (int i = 0; i < 2 * KD; ++i) {
        o[i][0] *= keep[0]; o[i][1] *= keep[0];
        o[i][2] *= keep[1]; o[i][3] *= keep[1];
      }
#pragma unroll
      for (int n = 0; n < NT / 2; ++n) {
        uint32_t fp[4];
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            const float e0 = exp2f(s[2 * n + q][2 * hf] - at[hf]), e1 = exp2f(s[2 * n + q][2 * hf + 1] - at[hf]);
            l[hf] += e0 + e1;
            fp[2 * q + hf] = pack_bf16(e0, e1);
          }
#pragma unroll
        for (int c = 0; c < KD; ++c) {
          uint32_t fv[4];
          ms_ldsm4_t(ms_b_nn_at(aV, LD, wk + n * 16, c * 16, lane), fv);
          ms_mma(o[2 * c], fp, fv[0], fv[1]);
          ms_mma(o[2 * c + 1], fp, fv[2], fv[3]);
        }
      }
    }
    __syncthreads();                       // the page is free for the load after the next
  }
  ms_wait<0>();
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    l[hf] += __shfl_xor_sync(0xffffffffu, l[hf], 1);
    l[hf] += __shfl_xor_sync(0xffffffffu, l[hf], 2);
  }
  if (KEYW > 1) {                          // merge the warps' parts of the 16 rows; warp 0 keeps the result
    __syncthreads();
    float* so = reinterpret_cast<float*>(sK);                            // [3][16][DP]
    float* sml = so + (KEYW - 1) * 16 * DP;                              // [4][16][2]
#pragma unroll
    for (int hf = 0; hf < 2; ++hf)
      if (t4 == 0) {
        sml[(warp * 16 + g4 + 8 * hf) * 2] = m[hf];
        sml[(warp * 16 + g4 + 8 * hf) * 2 + 1] = l[hf];
      }
    if (warp > 0)
#pragma unroll
      for (int i = 0; i < 2 * KD; ++i)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf)
          *reinterpret_cast<float2*>(so + ((warp - 1) * 16 + g4 + 8 * hf) * DP + i * 8 + 2 * t4) = make_float2(o[i][2 * hf], o[i][2 * hf + 1]);
    __syncthreads();
    if (warp > 0) return;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int r = g4 + 8 * hf;
      float mm = m[hf];
#pragma unroll
      for (int w = 1; w < KEYW; ++w) mm = fmaxf(mm, sml[(w * 16 + r) * 2]);
      const float at = mm == -CUDART_INF_F ? 0.f : mm;
      float f = exp2f(m[hf] - at), ll = l[hf] * f;
#pragma unroll
      for (int i = 0; i < 2 * KD; ++i) { o[i][2 * hf] *= f; o[i][2 * hf + 1] *= f; }
#pragma unroll
      for (int w = 1; w < KEYW; ++w) {
        f = exp2f(sml[(w * 16 + r) * 2] - at);
        ll = fmaf(sml[(w * 16 + r) * 2 + 1], f, ll);
#pragma unroll
        for (int i = 0; i < 2 * KD; ++i) {
          const float2 v = *reinterpret_cast<const float2*>(so + ((w - 1) * 16 + r) * DP + i * 8 + 2 * t4);
          o[i][2 * hf] = fmaf(v.x, f, o[i][2 * hf]);
          o[i][2 * hf + 1] = fmaf(v.y, f, o[i][2 * hf + 1]);
        }
      }
      m[hf] = mm;
      l[hf] = ll;
    }
  }
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = wr + g4 + 8 * hf;
    if (r >= n_rows) continue;
    const int row = r0 + r, h = g * p.rep + row % p.rep;
    const long long t = q0 + row / p.rep;
    if (p.n_split > 1) {
      const long long at = (static_cast<long long>(split) * p.n_tok + t) * p.H + h;
      if (t4 == 0) {
        p.pml[at * 2] = m[hf];
        p.pml[at * 2 + 1] = l[hf];
      }
#pragma unroll
      for (int i = 0; i < 2 * KD; ++i) {
        const int c = i * 8 + 2 * t4;
        if (c < p.D8) *reinterpret_cast<float2*>(p.po + at * p.D8 + c) = make_float2(o[i][2 * hf], o[i][2 * hf + 1]);
      }
      continue;
    }
    const float inv = l[hf] > 0.f ? 1.f / l[hf] : 0.f;
    __nv_bfloat16* dst = p.out + t * p.ldo + static_cast<long long>(h) * p.D;
    const bool even = (p.D | static_cast<int>(p.ldo)) % 2 == 0;
#pragma unroll
    for (int i = 0; i < 2 * KD; ++i) {
      const int c = i * 8 + 2 * t4;
      const float v0 = o[i][2 * hf] * inv, v1 = o[i][2 * hf + 1] * inv;
      if (c + 1 < p.D && even) {
        *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(v0, v1);
      } else {
        if (c < p.D) dst[c] = __float2bfloat16(v0);
        if (c + 1 < p.D) dst[c + 1] = __float2bfloat16(v1);
      }
    }
  }
}

// Joins the splits (at most 32): one warp per (token, head) of the sequences in q_start / q_lens. grid (tokens of the longest portion,
// heads / 4, sequences).
__global__ void __launch_bounds__(128) window_combine_kernel(const WindowParams<__nv_bfloat16> p) {
  const int seq = blockIdx.z, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (static_cast<int>(blockIdx.x) >= p.q_lens[seq] || h >= p.H) return;
  const long long t = p.q_start[seq] + blockIdx.x, step = static_cast<long long>(p.n_tok) * p.H, at = t * p.H + h;
  const float ms = lane < p.n_split ? p.pml[(at + lane * step) * 2] : -CUDART_INF_F;         // lane s: split s
  const float ls = lane < p.n_split ? p.pml[(at + lane * step) * 2 + 1] : 0.f;
  float m = ms;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  float f = exp2f(ms - m);
  f /= warp_sum(ls * f);
  for (int c0 = 0; c0 < p.D; c0 += 128) {
    float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int s = 0; s < p.n_split; ++s) {
      const float fs = __shfl_sync(0xffffffffu, f, s);
      const float* src = p.po + (at + s * step) * p.D8 + c0 + lane;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c0 + lane + 32 * i < p.D) v[i] = fmaf(src[32 * i], fs, v[i]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (c0 + lane + 32 * i < p.D) p.out[t * p.ldo + static_cast<long long>(h) * p.D + c0 + lane + 32 * i] = __float2bfloat16(v[i]);
  }
}

// One CTA of four warps per (token, head): the warps take every fourth group of four keys, the lanes the channels.
template <typename T, int NC>
__global__ void __launch_bounds__(128) window_row_kernel(const WindowParams<T> p) {
  const int seq = blockIdx.z, h = blockIdx.y, i = blockIdx.x, len = p.q_lens[seq];
  if (i >= len) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / p.rep;
  const long long t = p.q_start[seq] + i;
  const int pos = p.seq_lens[seq] - len + i;
  const int* table = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  const T* qr = p.q + (t * p.H + h) * p.D8;
  float q[NC], o[NC], m = -CUDART_INF_F, l = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    q[c] = c * 32 + lane < p.D ? to_f(qr[c * 32 + lane]) * p.scale : 0.f;
    o[c] = 0.f;
  }
  for (int j0 = window_first(pos, p.window) + warp * 4; j0 <= pos; j0 += 16) {
    float s[4];
    const T* row[4];
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      const int j = min(j0 + a, pos);
      row[a] = p.pages + ((static_cast<long long>(table[j / kWinPage]) * kWinPage + j % kWinPage) * p.G + g) * 2 * p.D8;
      s[a] = 0.f;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (c * 32 + lane < p.D) s[a] = fmaf(q[c], to_f(row[a][c * 32 + lane]), s[a]);
    }
    float mx = m;
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      s[a] = warp_sum(s[a]);
      if (j0 + a > pos) s[a] = -CUDART_INF_F;
      mx = fmaxf(mx, s[a]);
    }
    const float keep = expf(m - mx);
    m = mx;
    l *= keep;
#pragma unroll
    for (int c = 0; c < NC; ++c) o[c] *= keep;
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      const float w = expf(s[a] - m);
      l += w;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (c * 32 + lane < p.D) o[c] = fmaf(w, to_f(row[a][p.D8 + c * 32 + lane]), o[c]);
    }
  }
  __shared__ float sm[4], sl[4], so[4][32];
  if (lane == 0) { sm[warp] = m; sl[warp] = l; }
  __syncthreads();
  const float mm = fmaxf(fmaxf(sm[0], sm[1]), fmaxf(sm[2], sm[3]));
  float ll = 0.f;
  for (int w = 0; w < 4; ++w) ll = fmaf(sl[w], expf(sm[w] - mm), ll);
  const float f = expf(m - mm);
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    __syncthreads();
    so[warp][lane] = o[c] * f;
    __syncthreads();
    if (warp == 0 && c * 32 + lane < p.D)
      put(p.out + t * p.ldo + static_cast<long long>(h) * p.D + c * 32 + lane,
          (so[0][lane] + so[1][lane] + so[2][lane] + so[3][lane]) / ll);
  }
}

template <int KD, int KEYW>
static int window_mma_launch(const WindowParams<__nv_bfloat16>& p, int n_seq, int max_q, cudaStream_t st) {
  constexpr int kRows = 64 / KEYW, LD = KD * 16 + 8;
  const size_t smem = (kRows + 4 * kWinPage) * LD * sizeof(__nv_bfloat16);
  static DeviceOnce once;
  if (once.pending()) {
    const cudaError_t e = cudaFuncSetAttribute(window_mma_kernel<KD, KEYW>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    once.mark();
  }
  const dim3 grid((max_q * p.rep + kRows - 1) / kRows, p.G, n_seq * p.n_split);
  window_mma_kernel<KD, KEYW><<<grid, 128, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <int KEYW>
static int window_mma_any(const WindowParams<__nv_bfloat16>& p, int n_seq, int max_q, cudaStream_t st) {
  if (p.D8 <= 32) return window_mma_launch<2, KEYW>(p, n_seq, max_q, st);
  if (p.D8 <= 64) return window_mma_launch<4, KEYW>(p, n_seq, max_q, st);
  if (p.D8 <= 96) return window_mma_launch<6, KEYW>(p, n_seq, max_q, st);
  if (p.D8 <= 128) return window_mma_launch<8, KEYW>(p, n_seq, max_q, st);
  if (p.D8 <= 192) return window_mma_launch<12, KEYW>(p, n_seq, max_q, st);
  return window_mma_launch<16, KEYW>(p, n_seq, max_q, st);
}

template <typename T>
static int window_row_launch(const WindowParams<T>& p, int n_seq, int max_q, cudaStream_t st) {
  const dim3 grid(max_q, p.H, n_seq);
  if (p.D <= 64) window_row_kernel<T, 2><<<grid, 128, 0, st>>>(p);
  else if (p.D <= 128) window_row_kernel<T, 4><<<grid, 128, 0, st>>>(p);
  else if (p.D <= 256) window_row_kernel<T, 8><<<grid, 128, 0, st>>>(p);
  else window_row_kernel<T, 32><<<grid, 128, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int window_prep_launch(const void* u, long long ldu, const float* cs, const float* sn, int n_tok, int H, int G, int D, int R,
                              int pairs, int normed, float eps, int own_v, void* q, void* pages, const long long* slots, cudaStream_t st) {
  const WindowPrepParams<T> p{static_cast<const T*>(u), ldu, cs, sn, static_cast<T*>(q), static_cast<T*>(pages), slots, n_tok, H, G,
                              D, (D + 7) / 8 * 8, R, pairs, normed, own_v, eps};
  const long long items = static_cast<long long>(n_tok) * (H + G);
  const int unit = pairs ? R : R / 2;
  if constexpr (sizeof(T) == 2) {
    if (D % 8 == 0 && D <= 256 && ldu % 8 == 0 && unit % 8 == 0 && reinterpret_cast<uintptr_t>(u) % 16 == 0) {
      int gs = 1;
      while (gs * 8 < D) gs *= 2;
      const long long warps = (items + 32 / gs - 1) / (32 / gs);
      window_prep_vec_kernel<<<static_cast<unsigned>((warps + 7) / 8), 256, 0, st>>>(p, gs);
      return static_cast<int>(cudaGetLastError());
    }
  }
  window_prep_kernel<T><<<static_cast<unsigned>((items + 7) / 8), 256, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace pm

using namespace pm;

static bool window_bad_dims(int H, int G, int D) { return H < 1 || G < 1 || H % G || D < 1 || D > kWinMaxHead || G > 65535 || H > 65535; }

// u [n_tok, ldu]: q [H D], k [G D] and, own_v 1, v [G D] (else the values are the keys before rotation and norm). q_out
// [n_tok, H, D8] and the cache rows pages[slot] get rotated (first R channels; pairs 1: (2 i, 2 i + 1), else (i, i + R / 2);
// cs / sn fp32 [n_tok, R / 2]) and, normed 1, normalised vectors.
extern "C" int pm_window_prep(const void* u, int f32, long long ldu, const float* cs, const float* sn, int n_tok, int H, int G,
                              int D, int R, int pairs, int normed, float eps, int own_v, void* q_out, void* pages,
                              const long long* slots, cudaStream_t st) {
  if (window_bad_dims(H, G, D) || R < 0 || R > D || R % 2) return -1;
  if (ldu < static_cast<long long>(H + (own_v ? 2 : 1) * G) * D) return -2;
  if (n_tok < 1) return 0;
  return f32 ? window_prep_launch<float>(u, ldu, cs, sn, n_tok, H, G, D, R, pairs, normed, eps, own_v, q_out, pages, slots, st)
             : window_prep_launch<__nv_bfloat16>(u, ldu, cs, sn, n_tok, H, G, D, R, pairs, normed, eps, own_v, q_out, pages, slots, st);
}

// Attention of the new tokens q_start[i] .. + q_lens[i] - 1 of n_seq sequences (rows of q [n_tok, H, D8] and out [.., ldo])
// over their cached keys; sequence i has seq_lens[i] keys behind row i of block_table. few 1: decode tiles (a few rows per
// sequence), which take n_split > 1 with work buffers po [n_split][n_tok][H][D8] and pml [n_split][n_tok][H][2].
extern "C" int pm_window_attn(const void* q, int f32, const void* pages, const int* block_table, const int* seq_lens,
                              const int* q_start, const int* q_lens, int n_seq, int max_blocks, int n_tok, int max_q, int H,
                              int G, int D, int window, float scale, int few, int n_split, float* po, float* pml, void* out,
                              long long ldo, cudaStream_t st) {
  if (window_bad_dims(H, G, D) || window < 0 || n_split < 1 || n_split > 32 || (n_split > 1 && (!few || !po || !pml))) return -1;
  if (n_seq < 1 || max_q < 1) return 0;
  if (static_cast<long long>(n_seq) * n_split > 65535) return -2;
  const int D8 = (D + 7) / 8 * 8;
  if (f32) {
    const WindowParams<float> p{static_cast<const float*>(q), static_cast<const float*>(pages), static_cast<float*>(out), ldo,
                                block_table, seq_lens, q_start, q_lens, nullptr, nullptr, n_tok, max_blocks, H, G, H / G, D, D8,
                                window, 1, scale};
    return window_row_launch<float>(p, n_seq, max_q, st);
  }
  const WindowParams<__nv_bfloat16> p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(pages),
                                      static_cast<__nv_bfloat16*>(out), ldo, block_table, seq_lens, q_start, q_lens, po, pml, n_tok,
                                      max_blocks, H, G, H / G, D, D8, window, D8 <= 256 ? n_split : 1, scale};
  if (D8 > 256) return window_row_launch<__nv_bfloat16>(p, n_seq, max_q, st);
  if (!few) return window_mma_any<1>(p, n_seq, max_q, st);
  const int rc = window_mma_any<4>(p, n_seq, max_q, st);
  if (rc || n_split == 1) return rc;
  window_combine_kernel<<<dim3(max_q, (H + 3) / 4, n_seq), 128, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}
