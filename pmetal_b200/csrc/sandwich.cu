// Pieces of decoders whose sublayers have a norm before and a norm after them, on an fp32 stream:
//   * token embedding + a row chosen by the pair (previous token, token) + a learned row of the position; the previous token of a
//     sequence's first new token lies in its slot
//   * norm of a sublayer's result, residual sum and the norm in front of the next sublayer:
//         v = x + r / rms(r) (base + wb),  r = y + bias;     h = v / rms(v) (base + wn)
//     and, where every sequence brings one token, the input convolution of the next layer behind it
//   * causal convolution over the last inputs of a layer, added to them:  out_t = h_t + sum_j w_j h_{t - taps + 1 + j}. The inputs
//     before a step lie in a ring per sequence, [slot][taps - 1][width], position p in row p mod (taps - 1); inputs before a
//     sequence's start are zeros whatever the ring holds.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include "elem.cuh"
#include "host_util.cuh"
#include "pmetal_b200.h"

namespace pm {

struct PairEmbedParams {
  const long long* ids;
  const void* table;           // [vocab, width] compute type
  const void* pairs;           // [buckets + 1, width]; the last row is the first token's
  const void* pos_table;       // [max_pos, width]
  const int* pos;              // position of every token
  const int* seq_of;
  const int* q_start;
  const int* q_lens;
  const int* slots;
  int* last;                   // [slots] last token of every sequence
  long long buckets, mul_prev, mul_cur;
  int n, width, max_pos;
  float* xf;                   // [n, width]
  void* xc;                    // nullable: the same in the compute type, rows ldc apart
  long long ldc;
};

// One CTA per token.
template <typename T, int V>
__global__ void pair_embed_kernel(const PairEmbedParams p) {
  __shared__ long long row;
  const int t = blockIdx.x;
  const long long tok = p.ids[t];
  const int pos = p.pos[t];
  if (threadIdx.x == 0) {
    const int seq = p.seq_of[t], q0 = p.q_start[seq], slot = p.slots[seq];
    long long r = p.buckets;
    if (pos > 0) {
      const long long prev = t > q0 ? p.ids[t - 1] : p.last[slot];
      r = (prev * p.mul_prev + tok * p.mul_cur) % p.buckets;
    }
    row = r;
    if (t == q0) p.last[slot] = static_cast<int>(p.ids[q0 + p.q_lens[seq] - 1]);      // behind this token's read
  }
  __syncthreads();
  const T* a = static_cast<const T*>(p.table) + tok * p.width;
  const T* b = static_cast<const T*>(p.pairs) + row * p.width;
  const T* c = static_cast<const T*>(p.pos_table) + static_cast<long long>(min(pos, p.max_pos - 1)) * p.width;
  T* xc = static_cast<T*>(p.xc);
  for (int k = threadIdx.x * V; k < p.width; k += blockDim.x * V) {
    float v[V], u[V], w[V];
    load_vec<V>(a + k, v);
    load_vec<V>(b + k, u);
    load_vec<V>(c + k, w);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = v[e] + u[e] + w[e];
    store_vec<V>(p.xf + static_cast<long long>(t) * p.width + k, v);
    if (xc) store_vec<V>(xc + t * p.ldc + k, v);
  }
}

struct BranchNormParams {
  const float* x;              // [.., width]
  const void* y;               // nullable, [.., ldy] compute type
  long long ldy;
  const float* bias;           // nullable
  const float* wb;             // weight of the norm of r (with y)
  const float* wn;             // nullable: weight of the norm of v, else oc = v
  float base, eps;
  const long long* rows;       // nullable: input rows
  float* of;                   // nullable: v (may be x when rows is null)
  void* oc;                    // nullable, rows ldo apart
  long long ldo;
  const float* conv;           // nullable: [taps][width], one token per sequence; oc = h + convolution
  int taps;
  void* ring;                  // [slot][taps - 1][width]
  const int* slots;
  const int* pos;
  int width;
};

// One CTA per row, the row in registers: width <= NV V blockDim.x.
template <typename T, int V, int NV>
__global__ void branch_norm_kernel(const BranchNormParams p) {
  const long long o = blockIdx.x, r = p.rows ? p.rows[o] : o;
  const T* y = static_cast<const T*>(p.y);
  const float inv = 1.f / static_cast<float>(p.width);
  float v[NV][V];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = (i * blockDim.x + threadIdx.x) * V;
    if (k < p.width) load_vec<V>(p.x + r * p.width + k, v[i]);
  }
  if (y) {
    float s[NV][V], ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int k = (i * blockDim.x + threadIdx.x) * V;
      if (k >= p.width) continue;
      load_vec<V>(y + r * p.ldy + k, s[i]);
      if (p.bias) {
        float c[V];
        load_vec<V>(p.bias + k, c);
#pragma unroll
        for (int e = 0; e < V; ++e) s[i][e] += c[e];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(s[i][e], s[i][e], ss);
    }
    const float scale = 1.f / sqrtf(block_sum(ss) * inv + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int k = (i * blockDim.x + threadIdx.x) * V;
      if (k >= p.width) continue;
      float w[V];
      load_vec<V>(p.wb + k, w);
#pragma unroll
      for (int e = 0; e < V; ++e) v[i][e] = fmaf(s[i][e] * scale, p.base + w[e], v[i][e]);
      if (p.of) store_vec<V>(p.of + o * p.width + k, v[i]);
    }
  }
  if (!p.oc) return;
  T* oc = static_cast<T*>(p.oc) + o * p.ldo;
  if (!p.wn) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int k = (i * blockDim.x + threadIdx.x) * V;
      if (k < p.width) store_vec<V>(oc + k, v[i]);
    }
    return;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = (i * blockDim.x + threadIdx.x) * V;
    if (k < p.width)
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[i][e], v[i][e], ss);
  }
  const float scale = 1.f / sqrtf(block_sum(ss) * inv + p.eps);
  const int last = p.taps - 1, pos = p.conv ? p.pos[o] : 0;
  T* ring = p.conv ? static_cast<T*>(p.ring) + static_cast<long long>(p.slots[o]) * last * p.width : nullptr;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = (i * blockDim.x + threadIdx.x) * V;
    if (k >= p.width) continue;
    float w[V], h[V];
    load_vec<V>(p.wn + k, w);
#pragma unroll
    for (int e = 0; e < V; ++e) h[e] = v[i][e] * scale * (p.base + w[e]);
    if (p.conv) {
      float a[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {      // as the next steps will read it
        T c;
        put(&c, h[e]);
        h[e] = to_f(c);
      }
      load_vec<V>(p.conv + static_cast<long long>(last) * p.width + k, w);
#pragma unroll
      for (int e = 0; e < V; ++e) a[e] = fmaf(w[e], h[e], h[e]);
      for (int j = 0; j < last; ++j) {
        const int at = pos - last + j;
        if (at < 0) continue;
        float g[V];
        load_vec<V>(ring + static_cast<long long>(at % last) * p.width + k, g);
        load_vec<V>(p.conv + static_cast<long long>(j) * p.width + k, w);
#pragma unroll
        for (int e = 0; e < V; ++e) a[e] = fmaf(w[e], g[e], a[e]);
      }
      if (last > 0) store_vec<V>(ring + static_cast<long long>(pos % last) * p.width + k, h);
      store_vec<V>(oc + k, a);
    } else {
      store_vec<V>(oc + k, h);
    }
  }
}

struct CanonParams {
  const void* h;               // [tokens, width]
  const float* w;              // [taps][width]
  int taps;
  void* ring;
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  void* out;                   // [tokens, width], not h
  int width;
};

constexpr int kCanonTokens = 16;

// V channels of 16 tokens per thread; grid (token tiles of the longest portion, channel blocks, sequences). TAPS 0: p.taps. The thread
// with a portion's first tokens writes the ring once it has read it.
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(128) canon_kernel(const CanonParams p) {
  const int seq = blockIdx.z, len = p.q_lens[seq], t0 = blockIdx.x * kCanonTokens, k = (blockIdx.y * 128 + threadIdx.x) * V;
  if (t0 >= len || k >= p.width) return;
  const int taps = TAPS ? TAPS : p.taps, last = taps - 1;
  const long long q0 = p.q_start[seq];
  const int start = p.seq_lens[seq] - len;                 // position of the first new token
  const T* h = static_cast<const T*>(p.h) + q0 * p.width + k;
  T* out = static_cast<T*>(p.out) + q0 * p.width + k;
  T* ring = static_cast<T*>(p.ring) + static_cast<long long>(p.slots[seq]) * last * p.width + k;
  auto input = [&](int t, float (&v)[V]) {                 // input of new token t (negative: before the step)
    if (t >= 0) {
      load_vec<V>(h + static_cast<long long>(t) * p.width, v);
    } else if (start + t >= 0) {
      load_vec<V>(ring + static_cast<long long>((start + t) % last) * p.width, v);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = 0.f;
    }
  };
  const int n = min(kCanonTokens, len - t0);
  if constexpr (TAPS > 1) {
    float w[TAPS][V], past[TAPS - 1][V];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_vec<V>(p.w + static_cast<long long>(j) * p.width + k, w[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(t0 - last + j, past[j]);
    for (int i = 0; i < n; ++i) {
      float v[V], a[V];
      load_vec<V>(h + static_cast<long long>(t0 + i) * p.width, v);
#pragma unroll
      for (int e = 0; e < V; ++e) a[e] = fmaf(w[TAPS - 1][e], v[e], v[e]);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) a[e] = fmaf(w[j][e], past[j][e], a[e]);
      store_vec<V>(out + static_cast<long long>(t0 + i) * p.width, a);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) past[j][e] = j + 1 < TAPS - 1 ? past[j + 1][e] : v[e];
    }
  } else {
    for (int i = 0; i < n; ++i) {
      float v[V], a[V], w[V];
      load_vec<V>(h + static_cast<long long>(t0 + i) * p.width, v);
      load_vec<V>(p.w + static_cast<long long>(last) * p.width + k, w);
#pragma unroll
      for (int e = 0; e < V; ++e) a[e] = fmaf(w[e], v[e], v[e]);
      for (int j = 0; j < last; ++j) {
        input(t0 + i - last + j, v);
        load_vec<V>(p.w + static_cast<long long>(j) * p.width + k, w);
#pragma unroll
        for (int e = 0; e < V; ++e) a[e] = fmaf(w[e], v[e], a[e]);
      }
      store_vec<V>(out + static_cast<long long>(t0 + i) * p.width, a);
    }
  }
  if (t0 > 0) return;
  // later tiles have at least 16 tokens of the step before them and never read the ring (taps <= 17)
  for (int t = max(0, len - last); t < len; ++t) {
    float v[V];
    load_vec<V>(h + static_cast<long long>(t) * p.width, v);
    store_vec<V>(ring + static_cast<long long>((start + t) % last) * p.width, v);
  }
}

template <typename T, int V>
static int branch_launch_v(const BranchNormParams& p, int n, cudaStream_t st) {
  const int vecs = (p.width + V - 1) / V;
  int nv = 1;                                  // few rows: one pass; many: several vectors per thread
  const int want = n < 2 * num_sms() ? 1 : 4;
  while (nv < want && vecs > 64 * nv) nv *= 2;
  while ((vecs + nv - 1) / nv > 1024) nv *= 2;
  const int threads = ((vecs + nv - 1) / nv + 31) / 32 * 32;
  switch (nv) {
    case 1: branch_norm_kernel<T, V, 1><<<n, threads, 0, st>>>(p); break;
    case 2: branch_norm_kernel<T, V, 2><<<n, threads, 0, st>>>(p); break;
    case 4: branch_norm_kernel<T, V, 4><<<n, threads, 0, st>>>(p); break;
    case 8: branch_norm_kernel<T, V, 8><<<n, threads, 0, st>>>(p); break;
    default: return -3;
  }
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int branch_launch(const BranchNormParams& p, int n, cudaStream_t st) {
  const bool vec = p.width % 4 == 0 && p.ldy % 4 == 0 && p.ldo % 4 == 0;
  return vec ? branch_launch_v<T, 4>(p, n, st) : branch_launch_v<T, 1>(p, n, st);
}

template <typename T, int V>
static int canon_launch_v(const CanonParams& p, int n_seq, int max_q, cudaStream_t st) {
  const dim3 grid((max_q + kCanonTokens - 1) / kCanonTokens, (p.width / V + 127) / 128, n_seq);
  switch (p.taps) {
    case 2: canon_kernel<T, V, 2><<<grid, 128, 0, st>>>(p); break;
    case 3: canon_kernel<T, V, 3><<<grid, 128, 0, st>>>(p); break;
    case 4: canon_kernel<T, V, 4><<<grid, 128, 0, st>>>(p); break;
    default: canon_kernel<T, V, 0><<<grid, 128, 0, st>>>(p); break;
  }
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int pair_embed_launch(const PairEmbedParams& p, cudaStream_t st) {
  const bool vec = p.width % 4 == 0 && p.ldc % 4 == 0;
  int threads = (p.width / (vec ? 4 : 1) + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
  if (vec) pair_embed_kernel<T, 4><<<p.n, threads, 0, st>>>(p);
  else pair_embed_kernel<T, 1><<<p.n, threads, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace pm

using namespace pm;

// xf [n, width] fp32 = table[id] + pairs[row] + pos_table[position], xc (nullable, rows ldc apart) the same in the tables' type; row =
// (previous id * mul_prev + id * mul_cur) mod buckets, `buckets` itself for a sequence's first token. Sequence i brings the tokens
// q_start[i] .. + q_lens[i] - 1; last[slots[i]] (int32) holds its latest token, read and written. Positions lie below max_pos.
extern "C" int pm_pair_embed(const long long* ids, const void* table, const void* pairs, const void* pos_table, int f32, const int* pos,
                             const int* seq_of, const int* q_start, const int* q_lens, const int* slots, int* last, long long buckets,
                             long long mul_prev, long long mul_cur, int n, int width, int max_pos, float* xf, void* xc, long long ldc,
                             cudaStream_t st) {
  if (n < 0 || width < 1 || buckets < 1 || max_pos < 1 || mul_prev < 0 || mul_cur < 0) return -1;
  if (n == 0) return 0;
  const PairEmbedParams p{ids, table, pairs, pos_table, pos, seq_of, q_start, q_lens, slots, last, buckets, mul_prev, mul_cur, n, width,
                          max_pos, xf, xc, ldc};
  return f32 ? pair_embed_launch<float>(p, st) : pair_embed_launch<__nv_bfloat16>(p, st);
}

// v = x + r / rms(r) (base + wb), r = y + bias (y nullable: v = x), for the n rows listed in `rows` (nullable: row i); of [n, width]
// fp32 (nullable, written when there is a y; may be x when rows is null) = v, oc (nullable, compute type, rows ldo apart) =
// v / rms(v) (base + wn), without wn v itself. conv (nullable, [taps][width] fp32, with wn and without rows): row i is the only new
// token of a sequence, at position pos[i] with the ring of slot slots[i]; oc = h + sum_j conv[j] h_(taps - 1 - j tokens earlier).
extern "C" int pm_branch_norm(const float* x, const void* y, int f32, long long ldy, const float* bias, const float* wb, const float* wn,
                              float base, float eps, const long long* rows, float* of, void* oc, long long ldo, const float* conv,
                              int taps, void* ring, const int* slots, const int* pos, int n, int width, cudaStream_t st) {
  if (n < 0 || width < 1 || width > 8192 || (rows && of == x) || (y && !wb) ||
      (conv && (!wn || rows || !oc || taps < 1 || (taps > 1 && !ring) || !slots || !pos)))
    return -1;
  if (n == 0) return 0;
  const BranchNormParams p{x, y, ldy, bias, wb, wn, base, eps, rows, of, oc, ldo, conv, taps, ring, slots, pos, width};
  return f32 ? branch_launch<float>(p, n, st) : branch_launch<__nv_bfloat16>(p, n, st);
}

// out [tokens, width] = h + causal convolution of h with w [taps][width] fp32 along every sequence; h and out in the compute type,
// two buffers. ring [slot][taps - 1][width] (compute type) holds the sequences' earlier inputs, read and written. taps <= 17.
extern "C" int pm_canon(const void* h, int f32, const float* w, int taps, void* ring, const int* slots, const int* q_start,
                        const int* q_lens, const int* seq_lens, int n_seq, int max_q, int width, void* out, cudaStream_t st) {
  if (taps < 1 || taps > kCanonTokens + 1 || width < 1 || h == out || (taps > 1 && !ring) || n_seq > 65535) return -1;
  if (n_seq < 1 || max_q < 1) return 0;
  const CanonParams p{h, w, taps, ring, slots, q_start, q_lens, seq_lens, out, width};
  if (f32) return width % 4 ? canon_launch_v<float, 1>(p, n_seq, max_q, st) : canon_launch_v<float, 4>(p, n_seq, max_q, st);
  if (width % 8 == 0) return canon_launch_v<__nv_bfloat16, 8>(p, n_seq, max_q, st);
  return width % 4 ? canon_launch_v<__nv_bfloat16, 1>(p, n_seq, max_q, st) : canon_launch_v<__nv_bfloat16, 4>(p, n_seq, max_q, st);
}
