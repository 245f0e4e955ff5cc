// Grouped-query attention over a paged cache for heads of any size: position i sees the keys j with 0 <= i - j < window (every
// j <= i when window is 0) or, chunked, those of its own chunk (j <= i, the same j / window). Key and value sizes may differ, a head
// may have several attention maps over the same values, scores may be capped (cap tanh(s / cap)), and the softmax may have a sink
// per head (a score without a value). Instead of a softmax the weights may be sigmoids of score + a number per head, which nothing
// is divided by. Per token and layer the
// cache holds one row [head 0: k of map 0 | .. | v, head 1: ..] with D8 channels per key and DV8 per value (the sizes D and DV
// rounded up to 8, zeros behind them).
//
//   window_prep_kernel  rotation of queries and keys on their first R channels, optional division by their root mean square
//                       over the head with a weight, query factor that grows with the position, cache append. Values are the
//                       keys as projected, or columns of their own.
//   window_mma_kernel   bf16, mma.sync on 64-key pages in shared memory (two in flight), online softmax in base 2. Rows are
//                       (query token, head of the group, map) of one (sequence, key/value head). Prefill: 64 rows of one map, a
//                       warp owns 16 of them. Decode: 16 rows of all maps (a query has zeros at the other maps' channels, so
//                       that a page is read once), the four warps share them and split the keys of every page, and CTAs split
//                       the pages; the parts are merged in shared memory and by window_finish_kernel. Pages outside every row's
//                       window are not visited.
//   window_row_kernel   any type and size, one (token, head, map) per CTA (fp32 models, heads beyond 256 channels)
//   window_expand_kernel  keys (all maps side by side) and values of cached tokens in rows of 128 channels, for long portions on the
//                       tcgen05 kernel of attention_tc.cu; queries then lie in rows of 128, at their map's channels
//   window_finish_kernel  joins the parts of split pages; with two maps a_1 - lambda a_2, its RMS norm over the head and a
//                       factor; one sigmoid gate per head
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
  const T* u;                // [tokens, ldu]: q [H M D] from column 0, k [G M D] from k_at, v [G DV] from v_at
  long long ldu;
  const float* cs;           // [tokens, R / 2]
  const float* sn;
  T* q;                      // [tokens, H M, QP], channels of map i from i QM on, zeros elsewhere
  T* pages;                  // [block][64][G][M D8 + DV8]; null: queries alone
  const long long* slots;    // page * 64 + offset of every token
  const float* qw;           // [D], nullable: weights of the norms
  const float* kw;
  const int* pos;            // position of every token (temp_every > 0)
  int n_tok, H, G, M, D, D8, DV, DV8, QP, QM, k_at, v_at, R, pairs, normed, temp_every;
  float eps, temp_coef;
};

// Factor of the queries at a position.
template <typename T>
__device__ __forceinline__ float window_query_factor(const WindowPrepParams<T>& p, long long t) {
  if (p.temp_every <= 0) return 1.f;
  return 1.f + p.temp_coef * logf(static_cast<float>((p.pos[t] + 1) / p.temp_every + 1));
}

// One warp per (token, head and map of q or k, or value head).
template <typename T>
__global__ void __launch_bounds__(256) window_prep_kernel(const WindowPrepParams<T> p) {
  const int nq = p.H * p.M, nk = p.pages ? p.G * p.M : 0, items = nq + nk + (p.pages ? p.G : 0), lane = threadIdx.x & 31;
  const long long item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const long long t = item / items;
  if (t >= p.n_tok) return;
  const int h = static_cast<int>(item - t * items), kv = p.M * p.D8 + p.DV8;
  const T* u = p.u + t * p.ldu;
  if (h >= nq + nk) {
    const int g = h - nq - nk;
    T* dst = p.pages + (p.slots[t] * p.G + g) * kv + p.M * p.D8;
    for (int c = lane; c < p.DV8; c += 32) put(dst + c, c < p.DV ? to_f(u[p.v_at + g * p.DV + c]) : 0.f);
    return;
  }
  const bool key = h >= nq;
  const int hk = h - nq;
  const T* src = u + (key ? p.k_at + hk * p.D : h * p.D);
  float scale = key ? 1.f : window_query_factor(p, t);
  if (p.normed) {            // a rotation keeps the sum of squares
    float ss = 0.f;
    for (int c = lane; c < p.D; c += 32) {
      const float v = to_f(src[c]);
      ss = fmaf(v, v, ss);
    }
    scale /= sqrtf(warp_sum(ss) / static_cast<float>(p.D) + p.eps);
  }
  T* dst = key ? p.pages + (p.slots[t] * p.G + hk / p.M) * kv + (hk % p.M) * p.D8 : p.q + (t * nq + h) * p.QP + (h % p.M) * p.QM;
  if (!key)
    for (int c = lane; c < p.QP; c += 32)
      if (c < h % p.M * p.QM || c >= h % p.M * p.QM + p.D8) put(p.q + (t * nq + h) * p.QP + c, 0.f);
  const float* w = key ? p.kw : p.qw;
  const int half = p.R / 2;
  const float* cs = p.cs + t * half;
  const float* sn = p.sn + t * half;
  for (int c = lane; c < p.D8; c += 32) {
    float v = 0.f;
    if (c < p.D) {
      v = to_f(src[c]);
      if (w) v *= w[c];
      if (c < p.R) {
        const bool second = p.pairs ? (c & 1) : c >= half;
        const int f = p.pairs ? c >> 1 : (second ? c - half : c);
        const int o = p.pairs ? c ^ 1 : (second ? c - half : c + half);
        const float x = to_f(src[o]) * (w ? w[o] : 1.f);
        v = fmaf(v, cs[f], second ? x * sn[f] : -x * sn[f]);
      }
      v *= scale;
    }
    put(dst + c, v);
  }
}

// The same for heads in 8-channel pieces (bf16, D and DV <= 256, all columns at multiples of 8): a lane owns 8 channels of a
// head, gs lanes a head (gs: power of two).
__global__ void __launch_bounds__(256) window_prep_vec_kernel(const WindowPrepParams<__nv_bfloat16> p, int gs) {
  const int nq = p.H * p.M, nk = p.pages ? p.G * p.M : 0, items = nq + nk + (p.pages ? p.G : 0);
  const int lane = threadIdx.x & 31, per = 32 / gs, kv = p.M * p.D8 + p.DV8;
  const long long item = (blockIdx.x * 8ll + (threadIdx.x >> 5)) * per + lane / gs;
  const long long t = item / items;
  const bool live = t < p.n_tok;
  const int h = live ? static_cast<int>(item - t * items) : 0, c = (lane % gs) * 8;
  const bool value = h >= nq + nk, key = !value && h >= nq, mine = live && c < (value ? p.DV : p.D);
  const int hk = value ? h - nq - nk : h - nq;
  const __nv_bfloat16* src = p.u + (live ? t : 0) * p.ldu + (value ? p.v_at + hk * p.DV : key ? p.k_at + hk * p.D : h * p.D);
  float v[8], raw[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) raw[e] = 0.f;
  if (mine) load_vec<8>(src + c, raw);
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) ss = fmaf(raw[e], raw[e], ss);
  for (int o = gs / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!mine) return;
  if (value) {
    store_vec<8>(p.pages + (p.slots[t] * p.G + hk) * kv + p.M * p.D8 + c, raw);
    return;
  }
  float scale = key ? 1.f : window_query_factor(p, t);
  if (p.normed) scale /= sqrtf(ss / static_cast<float>(p.D) + p.eps);
  const float* w = key ? p.kw : p.qw;
  if (w) {
    float a[8];
    load_vec<8>(w + c, a);
#pragma unroll
    for (int e = 0; e < 8; ++e) raw[e] *= a[e];
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = raw[e];
  const int half = p.R / 2;
  if (c < p.R) {
    const float* cs = p.cs + t * half;
    const float* sn = p.sn + t * half;
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
      const int at = second ? c - half : c, other = second ? c - half : c + half;
      float a[8], b[8], x[8];
      load_vec<8>(src + other, x);
      load_vec<8>(cs + at, a);
      load_vec<8>(sn + at, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        if (w) x[e] *= w[other + e];
        v[e] = fmaf(raw[e], a[e], second ? x[e] * b[e] : -x[e] * b[e]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] *= scale;
  if (key) {
    store_vec<8>(p.pages + (p.slots[t] * p.G + hk / p.M) * kv + (hk % p.M) * p.D8 + c, v);
    return;
  }
  __nv_bfloat16* q = p.q + (t * nq + h) * p.QP;
  const int at = h % p.M * p.QM;
  store_vec<8>(q + at + c, v);
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = 0.f;
  for (int z = c; z < p.QP - p.D; z += p.D) store_vec<8>(q + (z < at ? z : z + p.D), v);      // the lanes own D channels at a time
}

template <typename T>
struct WindowParams {
  const T* q;                // [tokens, H M, QP], channels of map i from i QM on
  const T* pages;
  T* out;                    // [tokens, ldo], (head, map) n at column n DV
  long long ldo;
  const int* block_table;
  const int* seq_lens;
  const int* q_start;
  const int* q_lens;
  float* po;                 // null, or [n_split][n_tok][H M][DV8] and [n_split][n_tok][H M][2]: parts instead of out
  float* pml;
  const float* sink;         // [H], nullable
  const T* gate;             // [tokens, ldg], nullable: logits of the heads' gates
  long long ldg;
  int n_tok, max_blocks, H, G, rep, M, KM, D, D8, DV, DV8, QP, QM, window, n_split;      // KM: maps of a CTA, 1 or M
  float scale, softcap;      // softcap 0: none
  int chunked;               // window is the size of chunks counted from position 0
  const float* wbias;        // [H], nullable: sigmoid weights, added to the scores
  float out_scale;           // factor of the result
};

constexpr float kLog2e = 1.4426950408889634f;

// tanh with a small absolute and, near zero (odd series), relative error.
__device__ __forceinline__ float window_tanh(float x) {
  const float a = fabsf(x), e = exp2f(-2.f * kLog2e * a), x2 = x * x;
  return a < 0.1f ? x * fmaf(x2, fmaf(x2, 2.f / 15.f, -1.f / 3.f), 1.f) : copysignf(__fdividef(1.f - e, 1.f + e), x);
}

// First visible key of the query at position pos.
__device__ __forceinline__ int window_first(int pos, int window, int chunked) {
  if (chunked) return pos - pos % window;
  return window > 0 ? max(0, pos - window + 1) : 0;
}

// KK: 16-channel steps of a key row, 0: counted at run time. KD: 16-channel steps of the values. KEYW: warps that share 16 rows
// and split the keys of a page (1 or 4).
template <int KK, int KD, int KEYW>
__global__ void __launch_bounds__(128) window_mma_kernel(const WindowParams<__nv_bfloat16> p) {
  extern __shared__ __align__(16) uint8_t win_smem[];
  constexpr int kRows = 64 / KEYW, DP = KD * 16, LD = DP + 8, NT = 8 / KEYW;      // NT: 8-key tiles per warp
  const int steps = KK ? KK : (p.KM * p.D8 + 15) / 16, ldk = steps * 16 + 8;
  const int ktile = kWinPage * ldk;
  constexpr int kTile = kWinPage * LD;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(win_smem);        // [kRows][ldk]
  __nv_bfloat16* sK = sQ + kRows * ldk;                                  // [2][64][ldk]
  __nv_bfloat16* sV = sK + 2 * ktile;                                    // [2][64][LD]
  const int parts = p.M / p.KM, g = blockIdx.y / parts, map0 = blockIdx.y % parts * p.KM, rpt = p.rep * p.KM;
  const int seq = blockIdx.z / p.n_split, split = blockIdx.z % p.n_split;
  const int len = p.q_lens[seq], r0 = blockIdx.x * kRows, n_rows = min(kRows, len * rpt - r0);
  if (n_rows <= 0) return;
  const int q0 = p.q_start[seq], base = p.seq_lens[seq] - len;           // position of the first new token
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p_lo = base + r0 / rpt, p_hi = base + (r0 + n_rows - 1) / rpt;      // positions of the first and last row
  const int b_all = window_first(p_lo, p.window, p.chunked) / kWinPage, n_all = p_hi / kWinPage + 1 - b_all;
  const int per = (n_all + p.n_split - 1) / p.n_split;
  const int b0 = b_all + split * per, b1 = min(b0 + per, b_all + n_all);

  const int kvec = p.D8 / 8, vec = p.DV8 / 8, kw = steps * 2, kcat = p.KM * kvec;      // 16-byte pieces: of a key, a value, a tile row
  for (int i = threadIdx.x; i < kRows * kw; i += 128) {
    const int r = i / kw, c = i - r * kw, row = r0 + r, own = row % p.KM, at = c - own * kvec;
    const bool ok = r < n_rows && at >= 0 && at < kvec;                  // zeros at the channels of the other maps
    const __nv_bfloat16* src = p.q;
    if (ok) src += ((static_cast<long long>(q0 + row / rpt) * p.H + g * p.rep + row % rpt / p.KM) * p.M + map0 + own) * p.QP + (map0 + own) * p.QM + at * 8;
    ms_cp16(ms_addr(sQ + r * ldk + c * 8), src, ok);
  }
  const int* table = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  const int kv = p.M * p.D8 + p.DV8;                                     // cache row of one key/value head
  auto load_page = [&](int b, int buf) {
    const __nv_bfloat16* src = p.pages + (static_cast<long long>(table[b]) * kWinPage * p.G + g) * kv;
    for (int i = threadIdx.x; i < kWinPage * kw; i += 128) {
      const int r = i / kw, c = i - r * kw;
      const bool ok = c < kcat;
      ms_cp16(ms_addr(sK + buf * ktile + r * ldk + c * 8), src + static_cast<long long>(r) * p.G * kv + map0 * p.D8 + (ok ? c * 8 : 0), ok);
    }
    for (int i = threadIdx.x; i < kWinPage * KD * 2; i += 128) {
      const int r = i / (KD * 2), c = i % (KD * 2);
      const bool ok = c < vec;
      ms_cp16(ms_addr(sV + buf * kTile + r * LD + c * 8), src + static_cast<long long>(r) * p.G * kv + p.M * p.D8 + (ok ? c * 8 : 0), ok);
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
    pos[hf] = r < n_rows ? base + (r0 + r) / rpt : -1;                 // rows that do not exist see nothing
    first[hf] = window_first(pos[hf], p.window, p.chunked);
  }
  float o[2 * KD][4], m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2 * KD; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  const bool capped = p.softcap > 0.f, plain = p.wbias != nullptr;       // plain: sigmoid weights, m stays 0
  float wb2[2] = {0.f, 0.f};
  if (plain) {
    m[0] = m[1] = 0.f;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf)
      if (wr + g4 + 8 * hf < n_rows) wb2[hf] = p.wbias[g * p.rep + (r0 + wr + g4 + 8 * hf) % rpt / p.KM] * kLog2e;
  }
  const float a2 = capped ? p.scale / p.softcap : p.scale * kLog2e, cap2 = p.softcap * kLog2e;
  const uint32_t aQ = ms_addr(sQ);
  const bool idle = wr >= n_rows;

  for (int b = b0; b < b1; ++b) {
    const int buf = (b - b0) & 1;
    if (b + 1 < b1) load_page(b + 1, buf ^ 1);
    ms_commit();
    ms_wait<1>();
    __syncthreads();
    if (!idle) {
      const uint32_t aK = ms_addr(sK + buf * ktile), aV = ms_addr(sV + buf * kTile);
      float s[NT][4];
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
#pragma unroll (KK ? KK : 2)
      for (int k = 0; k < steps; ++k) {
        uint32_t fa[4];
        ms_ldsm4(ms_a_at(aQ, ldk, wr, k * 16, lane), fa);
#pragma unroll
        for (int n = 0; n < NT / 2; ++n) {
          uint32_t fb[4];
          ms_ldsm4(ms_b_nt_at(aK, ldk, wk + n * 16, k * 16, lane), fb);
          ms_mma(s[2 * n], fa, fb[0], fb[1]);
          ms_mma(s[2 * n + 1], fa, fb[2], fb[3]);
        }
      }
      const int j0 = b * kWinPage + wk + 2 * t4;
      const bool whole = b * kWinPage + kWinPage - 1 <= p_lo && b * kWinPage >= window_first(p_hi, p.window, p.chunked) && n_rows == kRows;
      float mx[2] = {m[0], m[1]};
      if (plain) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int hf = e >> 1, j = j0 + n * 8 + (e & 1);
            const float w = __fdividef(1.f, 1.f + exp2f(-fmaf(s[n][e], a2, wb2[hf])));
            s[n][e] = !whole && (j > pos[hf] || j < first[hf]) ? 0.f : w;
          }
      } else if (capped) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[n][e] = cap2 * window_tanh(s[n][e] * a2);
      } else {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[n][e] *= a2;
      }
      float keep[2], at[2] = {0.f, 0.f};
      if (!plain) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int hf = e >> 1, j = j0 + n * 8 + (e & 1);
            if (!whole && (j > pos[hf] || j < first[hf])) s[n][e] = -CUDART_INF_F;
            mx[hf] = fmaxf(mx[hf], s[n][e]);
          }
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
      }
#pragma unroll
      for (int n = 0; n < NT / 2; ++n) {
        uint32_t fp[4];
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            float e0 = s[2 * n + q][2 * hf], e1 = s[2 * n + q][2 * hf + 1];
            if (!plain) {
              e0 = exp2f(e0 - at[hf]);
              e1 = exp2f(e1 - at[hf]);
            }
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
    const int row = r0 + r, h = g * p.rep + row % rpt / p.KM, hm = h * p.M + map0 + row % p.KM;
    const long long t = q0 + row / rpt;
    if (p.po) {
      const long long at = (static_cast<long long>(split) * p.n_tok + t) * p.H * p.M + hm;
      if (t4 == 0) {
        p.pml[at * 2] = m[hf];
        p.pml[at * 2 + 1] = l[hf];
      }
#pragma unroll
      for (int i = 0; i < 2 * KD; ++i) {
        const int c = i * 8 + 2 * t4;
        if (c < p.DV8) *reinterpret_cast<float2*>(p.po + at * p.DV8 + c) = make_float2(o[i][2 * hf], o[i][2 * hf + 1]);
      }
      continue;
    }
    float f = 1.f, ll = l[hf];
    if (p.sink) {
      const float s2 = p.sink[h] * kLog2e, mm = fmaxf(m[hf], s2);
      f = exp2f(m[hf] - mm);
      ll = fmaf(ll, f, exp2f(s2 - mm));
    }
    float inv = plain ? 1.f : (ll > 0.f ? f / ll : 0.f);
    inv *= p.out_scale;
    if (p.gate) inv *= sigmoid_fast(to_f(p.gate[t * p.ldg + h]));
    __nv_bfloat16* dst = p.out + t * p.ldo + static_cast<long long>(hm) * p.DV;
    const bool even = (p.DV | static_cast<int>(p.ldo)) % 2 == 0;
#pragma unroll
    for (int i = 0; i < 2 * KD; ++i) {
      const int c = i * 8 + 2 * t4;
      const float v0 = o[i][2 * hf] * inv, v1 = o[i][2 * hf + 1] * inv;
      if (c + 1 < p.DV && even) {
        *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(v0, v1);
      } else {
        if (c < p.DV) dst[c] = __float2bfloat16(v0);
        if (c + 1 < p.DV) dst[c + 1] = __float2bfloat16(v1);
      }
    }
  }
}

template <typename T>
struct WindowFinishParams {
  const float* po;           // parts as in WindowParams, or
  const float* pml;
  const T* o;                // [n_tok, H M, OP]
  T* out;                    // [tokens, ldo], head h at column h DV
  long long ldo;
  const int* q_start;
  const int* q_lens;
  const float* sink;
  const T* gate;
  long long ldg;
  const float* lambda;       // M = 2: one number
  float keep, eps;           // M = 2: factor behind the norm
  int n_tok, H, M, DV, DV8, OP, n_split;
  int plain;                 // parts are added up as they are
  float out_scale;
};

// One warp per (token, head) of the sequences in q_start / q_lens, NC * 32 channels. grid (tokens of the longest portion,
// heads / 4, sequences). At most 32 splits.
template <typename T, int NC>
__global__ void __launch_bounds__(128) window_finish_kernel(const WindowFinishParams<T> p) {
  const int seq = blockIdx.z, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (static_cast<int>(blockIdx.x) >= p.q_lens[seq] || h >= p.H) return;
  const long long t = p.q_start[seq] + blockIdx.x, step = static_cast<long long>(p.n_tok) * p.H * p.M;
  float v[NC];
#pragma unroll
  for (int i = 0; i < NC; ++i) v[i] = 0.f;
  for (int map = 0; map < p.M; ++map) {
    const long long at = (t * p.H + h) * p.M + map;
    const float w = map ? -*p.lambda : 1.f;
    if (p.o) {
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (lane + 32 * i < p.DV) v[i] = fmaf(w, to_f(p.o[at * p.OP + lane + 32 * i]), v[i]);
      continue;
    }
    const float ms = lane < p.n_split ? p.pml[(at + lane * step) * 2] : -CUDART_INF_F;       // lane s: split s
    const float ls = lane < p.n_split ? p.pml[(at + lane * step) * 2 + 1] : 0.f;
    const float s2 = p.sink ? p.sink[h] * kLog2e : -CUDART_INF_F;
    float m = fmaxf(ms, s2);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    float f = 1.f;
    if (!p.plain) {
      f = exp2f(ms - m);
      f *= w / (warp_sum(ls * f) + exp2f(s2 - m));
    }
#pragma unroll 8
    for (int s = 0; s < p.n_split; ++s) {
      const float fs = __shfl_sync(0xffffffffu, f, s);
      const float* src = p.po + (at + s * step) * p.DV8 + lane;
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (lane + 32 * i < p.DV) v[i] = fmaf(src[32 * i], fs, v[i]);
    }
  }
  float f = p.out_scale;
  if (p.M > 1) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) ss = fmaf(v[i], v[i], ss);
    f *= p.keep / sqrtf(warp_sum(ss) / static_cast<float>(p.DV) + p.eps);
  }
  if (p.gate) f *= sigmoid_f(to_f(p.gate[t * p.ldg + h]));
#pragma unroll
  for (int i = 0; i < NC; ++i)
    if (lane + 32 * i < p.DV) put(p.out + t * p.ldo + static_cast<long long>(h) * p.DV + lane + 32 * i, v[i] * f);
}

// One CTA of four warps per (token, head, map): the warps take every fourth group of four keys, the lanes the channels.
template <typename T, int NC>
__global__ void __launch_bounds__(128) window_row_kernel(const WindowParams<T> p) {
  const int seq = blockIdx.z, hm = blockIdx.y, i = blockIdx.x, len = p.q_lens[seq];
  if (i >= len) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = hm / p.M, g = h / p.rep;
  const long long t = p.q_start[seq] + i;
  const int pos = p.seq_lens[seq] - len + i;
  const int* table = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  const T* qr = p.q + (t * p.H * p.M + hm) * p.QP + hm % p.M * p.QM;
  const int kv = p.M * p.D8 + p.DV8, k_at = hm % p.M * p.D8, v_at = p.M * p.D8;
  const bool plain = p.wbias != nullptr;
  const float wb = plain ? p.wbias[h] : 0.f;
  float q[NC], o[NC], m = plain ? 0.f : -CUDART_INF_F, l = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    q[c] = c * 32 + lane < p.D ? to_f(qr[c * 32 + lane]) * p.scale : 0.f;
    o[c] = 0.f;
  }
  for (int j0 = window_first(pos, p.window, p.chunked) + warp * 4; j0 <= pos; j0 += 16) {
    float s[4];
    const T* row[4];
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      const int j = min(j0 + a, pos);
      row[a] = p.pages + ((static_cast<long long>(table[j / kWinPage]) * kWinPage + j % kWinPage) * p.G + g) * kv;
      s[a] = 0.f;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (c * 32 + lane < p.D) s[a] = fmaf(q[c], to_f(row[a][k_at + c * 32 + lane]), s[a]);
    }
    float mx = m;
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      s[a] = warp_sum(s[a]);
      if (p.softcap > 0.f) s[a] = p.softcap * tanhf(s[a] / p.softcap);
      if (plain) s[a] = sigmoid_f(s[a] + wb);
      if (j0 + a > pos) s[a] = plain ? 0.f : -CUDART_INF_F;
      if (!plain) mx = fmaxf(mx, s[a]);
    }
    const float keep = expf(m - mx);
    m = mx;
    l *= keep;
#pragma unroll
    for (int c = 0; c < NC; ++c) o[c] *= keep;
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      const float w = plain ? s[a] : expf(s[a] - m);
      l += w;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (c * 32 + lane < p.DV) o[c] = fmaf(w, to_f(row[a][v_at + c * 32 + lane]), o[c]);
    }
  }
  __shared__ float sm[4], sl[4], so[4][32];
  if (lane == 0) { sm[warp] = m; sl[warp] = l; }
  __syncthreads();
  float mm = fmaxf(fmaxf(sm[0], sm[1]), fmaxf(sm[2], sm[3]));
  if (p.sink) mm = fmaxf(mm, p.sink[h]);
  float ll = p.sink ? expf(p.sink[h] - mm) : 0.f;
  for (int w = 0; w < 4; ++w) ll = fmaf(sl[w], expf(sm[w] - mm), ll);
  if (plain) ll = 1.f;
  const float f = expf(m - mm), gate = (p.gate ? sigmoid_f(to_f(p.gate[t * p.ldg + h])) : 1.f) * p.out_scale;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    __syncthreads();
    so[warp][lane] = o[c] * f;
    __syncthreads();
    if (warp == 0 && c * 32 + lane < p.DV)
      put(p.out + t * p.ldo + static_cast<long long>(hm) * p.DV + c * 32 + lane,
          (so[0][lane] + so[1][lane] + so[2][lane] + so[3][lane]) / ll * gate);
  }
}

// k128 [n, G, 128] and v128 [n, G, 128] of the n cache rows in `slots`, zeros behind their channels. A thread writes 8 channels.
__global__ void window_expand_kernel(const __nv_bfloat16* __restrict__ pages, const long long* __restrict__ slots, int n, int G, int keys,
                                     int values, __nv_bfloat16* __restrict__ k128, __nv_bfloat16* __restrict__ v128) {
  const long long total = static_cast<long long>(n) * G * 32;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long row = i >> 5;                        // (position, head)
    const int c = static_cast<int>(i & 15) * 8, j = static_cast<int>(row / G), g = static_cast<int>(row - static_cast<long long>(j) * G);
    const bool value = i & 16;
    const __nv_bfloat16* src = pages + (slots[j] * G + g) * (keys + values);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (c < (value ? values : keys)) v = *reinterpret_cast<const uint4*>(src + (value ? keys : 0) + c);
    *reinterpret_cast<uint4*>((value ? v128 : k128) + row * 128 + c) = v;
  }
}

constexpr size_t kWinSmem = 220 * 1024;
static size_t window_mma_smem(int key_steps, int value_steps, int rows) {
  return (static_cast<size_t>(rows + 2 * kWinPage) * (key_steps * 16 + 8) + 2 * kWinPage * (value_steps * 16 + 8)) * sizeof(__nv_bfloat16);
}
// 16-channel steps that the kernel instances have for this many channels (at most 256).
static int window_steps(int channels) {
  for (const int s : {2, 4, 6, 8, 12})
    if (channels <= s * 16) return s;
  return 16;
}

template <int KK, int KD, int KEYW>
static int window_mma_launch(const WindowParams<__nv_bfloat16>& p, int n_seq, int max_q, cudaStream_t st) {
  constexpr int kRows = 64 / KEYW;
  const size_t smem = window_mma_smem(KK ? KK : (p.KM * p.D8 + 15) / 16, KD, kRows);
  static DeviceMax configured;
  if (smem > configured.get()) {
    const cudaError_t e = cudaFuncSetAttribute(window_mma_kernel<KK, KD, KEYW>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.set(smem);
  }
  const dim3 grid((max_q * p.rep * p.KM + kRows - 1) / kRows, p.G * (p.M / p.KM), n_seq * p.n_split);
  window_mma_kernel<KK, KD, KEYW><<<grid, 128, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <int KD, int KEYW>
static int window_mma_keys(const WindowParams<__nv_bfloat16>& p, int n_seq, int max_q, cudaStream_t st) {
  const int keys = p.KM * p.D8;
  if (keys <= KD * 16 && keys > (KD - 2) * 16) return window_mma_launch<KD, KD, KEYW>(p, n_seq, max_q, st);
  return window_mma_launch<0, KD, KEYW>(p, n_seq, max_q, st);
}

template <int KEYW>
static int window_mma_any(const WindowParams<__nv_bfloat16>& p, int n_seq, int max_q, cudaStream_t st) {
  switch (window_steps(p.DV8)) {
    case 2: return window_mma_keys<2, KEYW>(p, n_seq, max_q, st);
    case 4: return window_mma_keys<4, KEYW>(p, n_seq, max_q, st);
    case 6: return window_mma_keys<6, KEYW>(p, n_seq, max_q, st);
    case 8: return window_mma_keys<8, KEYW>(p, n_seq, max_q, st);
    case 12: return window_mma_keys<12, KEYW>(p, n_seq, max_q, st);
    default: return window_mma_keys<16, KEYW>(p, n_seq, max_q, st);
  }
}

template <typename T>
static int window_row_launch(const WindowParams<T>& p, int n_seq, int max_q, cudaStream_t st) {
  const dim3 grid(max_q, p.H * p.M, n_seq);
  const int most = p.D > p.DV ? p.D : p.DV;
  if (most <= 64) window_row_kernel<T, 2><<<grid, 128, 0, st>>>(p);
  else if (most <= 128) window_row_kernel<T, 4><<<grid, 128, 0, st>>>(p);
  else if (most <= 256) window_row_kernel<T, 8><<<grid, 128, 0, st>>>(p);
  else window_row_kernel<T, 32><<<grid, 128, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int window_finish_launch(const WindowFinishParams<T>& p, int n_seq, int max_q, cudaStream_t st) {
  const dim3 grid(max_q, (p.H + 3) / 4, n_seq);
  if (p.DV <= 128) window_finish_kernel<T, 4><<<grid, 128, 0, st>>>(p);
  else if (p.DV <= 256) window_finish_kernel<T, 8><<<grid, 128, 0, st>>>(p);
  else window_finish_kernel<T, 32><<<grid, 128, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int window_prep_launch(WindowPrepParams<T> p, cudaStream_t st) {
  const long long items = static_cast<long long>(p.n_tok) * (p.H * p.M + (p.pages ? p.G * (p.M + 1) : 0));
  const int unit = p.pairs ? p.R : p.R / 2, most = p.D > p.DV ? p.D : p.DV;
  if constexpr (sizeof(T) == 2) {
    if (p.D % 8 == 0 && p.DV % 8 == 0 && most <= 256 && p.ldu % 8 == 0 && unit % 8 == 0 && p.k_at % 8 == 0 && p.v_at % 8 == 0 &&
        reinterpret_cast<uintptr_t>(p.u) % 16 == 0) {
      int gs = 1;
      while (gs * 8 < most) gs *= 2;
      const long long warps = (items + 32 / gs - 1) / (32 / gs);
      window_prep_vec_kernel<<<static_cast<unsigned>((warps + 7) / 8), 256, 0, st>>>(p, gs);
      return static_cast<int>(cudaGetLastError());
    }
  }
  window_prep_kernel<T><<<static_cast<unsigned>((items + 7) / 8), 256, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static WindowPrepParams<T> window_prep_params(const void* u, long long ldu, const float* cs, const float* sn, int n_tok, int H, int G, int M,
                                              int D, int DV, int wide, int k_at, int v_at, int R, int pairs, int normed, float eps,
                                              const float* qw, const float* kw, const int* pos, float temp_coef, int temp_every,
                                              void* q, void* pages, const long long* slots) {
  return {static_cast<const T*>(u), ldu, cs, sn, static_cast<T*>(q), static_cast<T*>(pages), slots, qw, kw, pos, n_tok, H, G, M,
          D, (D + 7) / 8 * 8, DV, (DV + 7) / 8 * 8, wide ? wide : (D + 7) / 8 * 8, wide ? (D + 7) / 8 * 8 : 0, k_at, v_at, R, pairs, normed, temp_every, eps, temp_coef};
}

template <typename T>
static int window_attn_launch(WindowParams<T> p, int n_seq, int max_q, int few, void* o, const float* lambda, float keep, float eps,
                              cudaStream_t st) {
  constexpr bool low = sizeof(T) == 2;
  WindowFinishParams<T> f{p.po, p.pml, nullptr, p.out, p.ldo, p.q_start, p.q_lens, p.sink, p.gate, p.ldg, lambda, keep, eps,
                          p.n_tok, p.H, p.M, p.DV, p.DV8, p.DV, p.n_split, p.wbias != nullptr, p.out_scale};
  if (!p.po && p.M > 1) {                 // results of the maps, then their difference
    if (!o) return -3;
    f.o = static_cast<const T*>(o);
    p.out = static_cast<T*>(o);
    p.ldo = static_cast<long long>(p.H) * p.M * p.DV;
    p.gate = nullptr;
    p.out_scale = 1.f;
  }
  int rc;
  if constexpr (low) {
    if (p.D8 > 256 || p.DV8 > 256) {
      if (p.po) return -4;
      rc = window_row_launch<T>(p, n_seq, max_q, st);
    } else if (few) {
      p.KM = window_mma_smem((p.M * p.D8 + 15) / 16, window_steps(p.DV8), 16) <= kWinSmem ? p.M : 1;
      rc = window_mma_any<4>(p, n_seq, max_q, st);
    } else {
      rc = window_mma_any<1>(p, n_seq, max_q, st);
    }
  } else {
    if (p.po) return -4;
    rc = window_row_launch<T>(p, n_seq, max_q, st);
  }
  if (rc || (!p.po && p.M == 1)) return rc;
  return window_finish_launch<T>(f, n_seq, max_q, st);
}

}  // namespace pm

using namespace pm;

static bool window_bad_dims(int H, int G, int M, int D, int DV) {
  return H < 1 || G < 1 || H % G || D < 1 || D > kWinMaxHead || DV < 1 || DV > kWinMaxHead || M < 1 || M > 2 || G * M > 65535 || H * M > 65535;
}

// u [n_tok, ldu]: queries [H][M][D] from column 0 and, with pages, keys [G][M][D] from column k_at and values [G][DV] from
// column v_at (k_at again: the values are the keys before rotation and norm). q_out [n_tok, H M, D8] (wide > 0: rows of that many
// channels, those of map i from i D8 on, zeros elsewhere) and the cache rows
// pages[slot] get rotated (first R channels; pairs 1: (2 i, 2 i + 1), else (i, i + R / 2); cs / sn fp32 [n_tok, R / 2]) and,
// normed 1, normalised vectors times qw / kw (fp32 [D], nullable). temp_every > 0: queries at position p = pos[t] are multiplied
// by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1).
extern "C" int pm_window_prep(const void* u, int f32, long long ldu, const float* cs, const float* sn, int n_tok, int H, int G, int M,
                              int D, int DV, int wide, int k_at, int v_at, int R, int pairs, int normed, float eps, const float* qw,
                              const float* kw, const int* pos, float temp_coef, int temp_every, void* q_out, void* pages,
                              const long long* slots, cudaStream_t st) {
  if (window_bad_dims(H, G, M, D, DV) || R < 0 || R > D || R % 2 || temp_every < 0 || (temp_every && !pos) ||
      (wide && (wide % 8 || wide < M * ((D + 7) / 8 * 8)))) return -1;
  if (ldu < static_cast<long long>(H) * M * D || (pages && (k_at < 0 || v_at < 0 || ldu < k_at + static_cast<long long>(G) * M * D ||
                                                            ldu < v_at + static_cast<long long>(G) * DV))) return -2;
  if (n_tok < 1) return 0;
  return f32 ? window_prep_launch(window_prep_params<float>(u, ldu, cs, sn, n_tok, H, G, M, D, DV, wide, k_at, v_at, R, pairs, normed, eps, qw,
                                                            kw, pos, temp_coef, temp_every, q_out, pages, slots), st)
             : window_prep_launch(window_prep_params<__nv_bfloat16>(u, ldu, cs, sn, n_tok, H, G, M, D, DV, wide, k_at, v_at, R, pairs, normed,
                                                                    eps, qw, kw, pos, temp_coef, temp_every, q_out, pages, slots), st);
}

// Attention of the new tokens q_start[i] .. + q_lens[i] - 1 of n_seq sequences (rows of q as pm_window_prep leaves them and out [.., ldo])
// over their cached keys; sequence i has seq_lens[i] keys behind row i of block_table. Scores times scale, capped when
// softcap > 0; sink (fp32 [H], M = 1) adds exp(sink) to a head's softmax sum; gate [.., ldg] multiplies head h by the sigmoid of
// column h. M = 2: the result of a head is a_1 - lambda[0] a_2 over its root mean square (eps inside), times keep; it takes o
// [n_tok, H M, DV] in the compute type unless parts are given. few 1: decode tiles (a few rows per sequence), which take work
// buffers po [n_split][n_tok][H M][DV8] and pml [n_split][n_tok][H M][2] (both or none; needed for n_split > 1). chunked 1: a position
// sees the keys of its own chunk of `window` positions. wbias (fp32 [H], nullable, M = 1, without sink): the weight of a key is the
// sigmoid of its score + wbias, not divided by their sum. out_scale multiplies the result.
extern "C" int pm_window_attn(const void* q, int f32, const void* pages, const int* block_table, const int* seq_lens,
                              const int* q_start, const int* q_lens, int n_seq, int max_blocks, int n_tok, int max_q, int H,
                              int G, int M, int D, int DV, int wide, int window, float scale, float softcap, const float* sink, const void* gate,
                              long long ldg, const float* lambda, float keep, float eps, int few, int n_split, float* po, float* pml,
                              void* o, void* out, long long ldo, int chunked, const float* wbias, float out_scale, cudaStream_t st) {
  if (window_bad_dims(H, G, M, D, DV) || window < 0 || n_split < 1 || n_split > 32 || (n_split > 1 && (!few || !po)) ||
      (!po != !pml) || (M > 1 && (!lambda || sink)) || softcap < 0.f || (chunked && window < 1) || (wbias && (M > 1 || sink || softcap > 0.f)))
    return -1;
  if (n_seq < 1 || max_q < 1) return 0;
  if (static_cast<long long>(n_seq) * n_split > 65535) return -2;
  const int D8 = (D + 7) / 8 * 8, DV8 = (DV + 7) / 8 * 8;
  if (f32)
    return window_attn_launch<float>({static_cast<const float*>(q), static_cast<const float*>(pages), static_cast<float*>(out), ldo,
                                      block_table, seq_lens, q_start, q_lens, po, pml, sink, static_cast<const float*>(gate), ldg,
                                      n_tok, max_blocks, H, G, H / G, M, 1, D, D8, DV, DV8, wide ? wide : D8, wide ? D8 : 0, window, n_split, scale, softcap, chunked, wbias, out_scale},
                                     n_seq, max_q, few, o, lambda, keep, eps, st);
  return window_attn_launch<__nv_bfloat16>({static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(pages),
                                            static_cast<__nv_bfloat16*>(out), ldo, block_table, seq_lens, q_start, q_lens, po, pml,
                                            sink, static_cast<const __nv_bfloat16*>(gate), ldg, n_tok, max_blocks, H, G, H / G, M, 1,
                                            D, D8, DV, DV8, wide ? wide : D8, wide ? D8 : 0, window, n_split, scale, softcap, chunked,
                                            wbias, out_scale},
                                           n_seq, max_q, few, o, lambda, keep, eps, st);
}

// k128 / v128 [n, G, 128] bf16 = the cached keys (M maps of D8 channels side by side) and values (DV8) of the n cache rows in `slots`
// (page * 64 + offset), zero padded. M D8 <= 128 and DV8 <= 128.
extern "C" int pm_window_expand(const void* pages, const long long* slots, int n, int G, int M, int D, int DV, void* k128, void* v128,
                                cudaStream_t st) {
  const int keys = M * ((D + 7) / 8 * 8), values = (DV + 7) / 8 * 8;
  if (n < 1 || window_bad_dims(G, G, M, D, DV) || keys > 128 || values > 128) return -1;
  long long grid = (static_cast<long long>(n) * G * 32 + 255) / 256;
  if (grid > num_sms() * 16) grid = num_sms() * 16;
  window_expand_kernel<<<static_cast<int>(grid), 256, 0, st>>>(static_cast<const __nv_bfloat16*>(pages), slots, n, G, keys, values,
                                                               static_cast<__nv_bfloat16*>(k128), static_cast<__nv_bfloat16*>(v128));
  return static_cast<int>(cudaGetLastError());
}

// The last step of pm_window_attn by itself, for the tokens of n_seq sequences: o [n_tok, H M, OP] (bf16, DV channels per row) -> out
// [.., ldo]: the difference of two maps with its norm (M = 2: lambda, keep, eps) and the heads' gates (nullable).
extern "C" int pm_window_finish(const void* o, int n_tok, int H, int M, int DV, int OP, const int* q_start, const int* q_lens, int n_seq,
                                int max_q, const float* lambda, float keep, float eps, const void* gate, long long ldg, void* out,
                                long long ldo, cudaStream_t st) {
  if (window_bad_dims(H, H, M, 1, DV) || OP < DV || (M > 1 && !lambda)) return -1;
  if (n_seq < 1 || max_q < 1) return 0;
  const WindowFinishParams<__nv_bfloat16> f{nullptr, nullptr, static_cast<const __nv_bfloat16*>(o), static_cast<__nv_bfloat16*>(out),
                                            ldo, q_start, q_lens, nullptr, static_cast<const __nv_bfloat16*>(gate), ldg, lambda, keep,
                                            eps, n_tok, H, M, DV, (DV + 7) / 8 * 8, OP, 1, 0, 1.f};
  return window_finish_launch(f, n_seq, max_q, st);
}
