// Routed experts, two forms: a gated unit whose routing weight multiplies the expert's input, y = sum over a token's experts of
// down(silu(G w h) * (U w h)), and plain units y = sum of w down(gelu(U h)), whose weights the caller applies to the rows.
// The (token, slot) pairs come sorted by expert (moe_quant.cu); pairs behind the last expert (offsets off[E] ..) are left alone:
//   router_logits_kernel   fp32 logits of a few experts for many tokens
//   expert_gather_kernel   rows w h (or h) in sorted order, or in a layout whose slabs start at multiples of `align` rows (zero rows
//                          between them), for the grouped tensor-core GEMMs (grouped_gemm.cu)
//   expert_gemv_kernel     a few rows per expert (decode, bf16): every weight row is read once by one warp and multiplied with
//                          all rows of its expert; fp32 sums, the routing weight applied to them, activation inside
//   expert_rows_kernel     products of sorted rows with their experts' matrices on the CUDA cores, fp32 sums, any size and
//                          type: fp32 models, and sizes that the GEMMs cannot copy in 16-byte pieces
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <type_traits>
#include "elem.cuh"
#include "host_util.cuh"
#include "mma_sync.cuh"
#include "pmetal_b200.h"

namespace pm {

// out [T, n] fp32 = h W^T for n <= 8 NT outputs: a CTA takes 16 tokens, its eight warps cut K into pieces of 32 in turn and meet in
// shared memory. A lane loads 8 consecutive values of a row: the order of K inside a piece is the same for both operands, so it
// need not be the one of the fragment layout.
constexpr int kRouterWarps = 8;
template <int NT>
__global__ void __launch_bounds__(kRouterWarps * 32) router_logits_kernel(const __nv_bfloat16* __restrict__ h, long long ldh,
                                                                          const __nv_bfloat16* __restrict__ W, int T, int n, int K,
                                                                          float* __restrict__ out) {
  __shared__ float part[kRouterWarps][16][8 * NT + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, t4 = lane & 3, t0 = blockIdx.x * 16;
  const __nv_bfloat16* a0 = h + static_cast<long long>(min(t0 + g4, T - 1)) * ldh + t4 * 8;
  const __nv_bfloat16* a1 = h + static_cast<long long>(min(t0 + g4 + 8, T - 1)) * ldh + t4 * 8;
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll 2
  for (int k = warp * 32; k < K; k += kRouterWarps * 32) {
    const uint4 x = *reinterpret_cast<const uint4*>(a0 + k), y = *reinterpret_cast<const uint4*>(a1 + k);
    const uint32_t fa[4] = {x.x, y.x, x.y, y.y}, fb[4] = {x.z, y.z, x.w, y.w};
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const uint4 w = __ldg(reinterpret_cast<const uint4*>(W + static_cast<long long>(min(i * 8 + g4, n - 1)) * K + t4 * 8 + k));
      ms_mma(acc[i], fa, w.x, w.y);
      ms_mma(acc[i], fb, w.z, w.w);
    }
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) part[warp][g4 + 8 * (e >> 1)][i * 8 + 2 * t4 + (e & 1)] = acc[i][e];
  __syncthreads();
  for (int i = threadIdx.x; i < 16 * n; i += kRouterWarps * 32) {
    const int r = i / n, c = i - r * n;
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < kRouterWarps; ++w) v += part[w][r][c];
    if (t0 + r < T) out[static_cast<long long>(t0 + r) * n + c] = v;
  }
}

// Largest e with off[e] <= row (off non-decreasing, row < off[E]).
__device__ __forceinline__ int expert_at(const int* __restrict__ off, int E, int row) {
  int lo = 0, hi = E;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (off[mid] <= row) lo = mid; else hi = mid;
  }
  return lo;
}

// One CTA per row of xs. Plain layout: row = sorted position. Padded layout (align > 0): every CTA derives the padded
// offsets itself; CTA 0 writes them, and the rows write dest[pair] = padded row.
template <typename T, int V>
__global__ void __launch_bounds__(128) expert_gather_kernel(const T* __restrict__ h, long long ldh, const int* __restrict__ perm,
                                                            const float* __restrict__ w, const int* __restrict__ off, int E,
                                                            int k, int align, int width, T* __restrict__ xs,
                                                            int* __restrict__ off_pad, int* __restrict__ dest) {
  extern __shared__ int s_pad[];                  // [E + 1]
  const int row = blockIdx.x;
  int pos = row;
  if (align > 0) {
    const int lane = threadIdx.x & 31;
    if (threadIdx.x < 32) {
      int base = 0;
      for (int e0 = 0; e0 < E; e0 += 32) {
        const int e = e0 + lane;
        int c = e < E ? (off[e + 1] - off[e] + align - 1) / align * align : 0;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const int up = __shfl_up_sync(0xffffffffu, c, o);
          if (lane >= o) c += up;
        }
        if (e < E) s_pad[e + 1] = base + c;
        base += __shfl_sync(0xffffffffu, c, 31);
      }
      if (lane == 0) s_pad[0] = 0;
    }
    __syncthreads();
    if (row == 0)
      for (int e = threadIdx.x; e <= E; e += blockDim.x) off_pad[e] = s_pad[e];
    pos = -1;
    if (row >= s_pad[E]) return;                  // past the last slab: never read
    const int e = expert_at(s_pad, E, row);
    const int in = row - s_pad[e];
    if (in < off[e + 1] - off[e]) pos = off[e] + in;
  }
  const int pair = pos >= 0 ? perm[pos] : 0;
  const float f = pos < 0 ? 0.f : w ? w[pair] : 1.f;
  if (align > 0 && pos >= 0 && threadIdx.x == 0) dest[pair] = row;
  const T* src = h + static_cast<long long>(pair / k) * ldh;
  T* dst = xs + static_cast<long long>(row) * width;
  for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
    float v[V];
    if (pos >= 0) {
      load_vec<V>(src + c, v);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] *= f;
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = 0.f;
    }
    store_vec<V>(dst + c, v);
  }
}

enum ExpertAct { kActNone = 0, kActSwiglu = 1, kActGelu = 2 };

struct ExpertGemvParams {
  const __nv_bfloat16* x;      // kActNone: sorted rows; else token rows [.., ldx]
  long long ldx;
  const __nv_bfloat16* W;      // [E][N or 2 N][K]
  const int* perm;             // pair of every sorted position, its token row is pair / k
  const float* w;              // kActSwiglu: weight of every pair
  const int* off;
  __nv_bfloat16* out;          // [n, N] in sorted order
  int n, E, k, N, K;
};

// grid (channel tiles, sorted positions): the position that begins an expert's slab works for the whole slab. A warp owns four
// weight rows: two gate / up pairs (GLU) or four output channels.
template <int ACT>
__global__ void __launch_bounds__(128) expert_gemv_kernel(const ExpertGemvParams p) {
  constexpr bool GLU = ACT == kActSwiglu;
  const int pos0 = blockIdx.y, e = expert_at(p.off, p.E, pos0);
  if (p.off[e] != pos0) return;
  const int n_rows = p.off[e + 1] - pos0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int kPer = GLU ? 2 : 4;
  const int c0 = (blockIdx.x * 4 + warp) * kPer;
  if (c0 >= p.N) return;
  const __nv_bfloat16* mat = p.W + static_cast<long long>(e) * (GLU ? 2 * p.N : p.N) * p.K;
  const __nv_bfloat16* wr[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int c = min(c0 + (GLU ? i >> 1 : i), p.N - 1) + (GLU && (i & 1) ? p.N : 0);
    wr[i] = mat + static_cast<long long>(c) * p.K;
  }
  auto pass = [&](auto rows_tag, int r0) {
    constexpr int R = decltype(rows_tag)::value;
    const __nv_bfloat16* xr[R];
    float acc[4][R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int pos = pos0 + min(r0 + r, n_rows - 1);
      xr[r] = p.x + static_cast<long long>(ACT != kActNone ? p.perm[pos] / p.k : pos) * p.ldx;
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i][r] = 0.f;
    }
#pragma unroll 2
    for (int c = lane * 8; c < p.K; c += 256) {
      uint4 raw[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) raw[i] = __ldg(reinterpret_cast<const uint4*>(wr[i] + c));
#pragma unroll
      for (int r = 0; r < R; ++r) {
        float xv[8];
        load_vec<8>(xr[r] + c, xv);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const uint32_t q[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            acc[i][r] = fmaf(__uint_as_float(q[j] << 16), xv[2 * j], acc[i][r]);
            acc[i][r] = fmaf(__uint_as_float(q[j] & 0xffff0000u), xv[2 * j + 1], acc[i][r]);
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i][r] = warp_sum(acc[i][r]);
      if (lane == 0 && r0 + r < n_rows) {
        const int pos = pos0 + r0 + r;
        __nv_bfloat16* dst = p.out + static_cast<long long>(pos) * p.N + c0;
        const float f = GLU ? p.w[p.perm[pos]] : 1.f;
#pragma unroll
        for (int i = 0; i < kPer; ++i)
          if (c0 + i < p.N)
            dst[i] = __float2bfloat16(GLU ? silu_fast(acc[2 * i % 4][r] * f) * (acc[(2 * i + 1) % 4][r] * f)
                                          : ACT == kActGelu ? gelu_fast(acc[i][r]) : acc[i][r]);
      }
    }
  };
  for (int r0 = 0; r0 < n_rows;) {
    const int left = n_rows - r0;
    if (left > 2) {
      pass(std::integral_constant<int, 4>{}, r0);
      r0 += 4;
    } else if (left == 2) {
      pass(std::integral_constant<int, 2>{}, r0);
      r0 += 2;
    } else {
      pass(std::integral_constant<int, 1>{}, r0);
      r0 += 1;
    }
  }
}

constexpr int kRowTile = 8;

// x [rows, K] sorted, W [E][M][K] -> out [rows, N]: M = N (plain or gelu), or with kActSwiglu M = 2 N (gate rows above up rows)
// and out = silu(gate) * up. CTA: 8 rows; warp: one output channel at a time.
template <typename T>
__global__ void __launch_bounds__(256) expert_rows_kernel(const T* __restrict__ x, int rows, const T* __restrict__ W,
                                                          const int* __restrict__ off, int E, int N, int K, int act,
                                                          T* __restrict__ out) {
  const int r0 = blockIdx.y * kRowTile, n_rows = min(kRowTile, min(rows, off[E]) - r0);
  const bool glu = act == kActSwiglu;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long mat = static_cast<long long>(glu ? 2 * N : N) * K;
  for (int n = blockIdx.x * 8 + warp; n < N; n += gridDim.x * 8) {
    for (int a = 0; a < n_rows;) {
      const int e = expert_at(off, E, r0 + a);
      const int b = max(a + 1, min(n_rows, off[e + 1] - r0));          // rows a .. b - 1 belong to expert e
      const T* wg = W + e * mat + static_cast<long long>(n) * K;
      const T* wu = wg + static_cast<long long>(N) * K;
      float g[kRowTile], u[kRowTile];
#pragma unroll
      for (int i = 0; i < kRowTile; ++i) g[i] = u[i] = 0.f;
      for (int c = lane; c < K; c += 32) {
        const float fg = to_f(wg[c]), fu = glu ? to_f(wu[c]) : 0.f;
#pragma unroll
        for (int i = 0; i < kRowTile; ++i)
          if (a + i < b) {
            const float v = to_f(x[static_cast<long long>(r0 + a + i) * K + c]);
            g[i] = fmaf(fg, v, g[i]);
            u[i] = fmaf(fu, v, u[i]);
          }
      }
#pragma unroll
      for (int i = 0; i < kRowTile; ++i)
        if (a + i < b) {
          const float sg = warp_sum(g[i]), su = glu ? warp_sum(u[i]) : 0.f;
          if (lane == 0) put(out + static_cast<long long>(r0 + a + i) * N + n, glu ? silu_f(sg) * su : act == kActGelu ? gelu_f(sg) : sg);
        }
      a = b;
    }
  }
}

template <typename T>
static int gather_launch(const void* h, long long ldh, const int* perm, const float* w, const int* off, int E, int k, int align,
                         int rows, int width, void* xs, int* off_pad, int* dest, cudaStream_t st) {
  const size_t smem = align > 0 ? sizeof(int) * (E + 1) : 0;
  const T* src = static_cast<const T*>(h);
  T* dst = static_cast<T*>(xs);
  if (width % 8 == 0 && ldh % 8 == 0)
    expert_gather_kernel<T, 8><<<rows, 128, smem, st>>>(src, ldh, perm, w, off, E, k, align, width, dst, off_pad, dest);
  else
    expert_gather_kernel<T, 1><<<rows, 128, smem, st>>>(src, ldh, perm, w, off, E, k, align, width, dst, off_pad, dest);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace pm

using namespace pm;

// out [T, n] fp32 = h [T, K] W^T (bf16, W [>= n, K]) for at most 64 outputs; K a multiple of 32, ldh of 8.
extern "C" int pm_router_logits(const void* h, long long ldh, const void* W, int T, int n, int K, float* out, cudaStream_t st) {
  if (n < 1 || n > 64 || K < 32 || K % 32 || ldh % 8 || ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(W)) & 15)) return -1;
  if (T < 1) return 0;
  const auto kernel = n <= 16 ? router_logits_kernel<2> : n <= 32 ? router_logits_kernel<4> : router_logits_kernel<8>;
  kernel<<<(T + 15) / 16, kRouterWarps * 32, 0, st>>>(static_cast<const __nv_bfloat16*>(h), ldh, static_cast<const __nv_bfloat16*>(W),
                                                      T, n, K, out);
  return static_cast<int>(cudaGetLastError());
}

// xs [rows, width] = w[pair] * h[pair / k] (w null: h) for the pairs perm[0 .. n) sorted by expert (off [E + 1]). align 0: rows = n in
// sorted order. align > 0: every expert's slab starts at a multiple of align (off_pad [E + 1]), dest [n] is the row of each
// pair, rows between slabs are zero; rows must be at least n + (align - 1) per expert with pairs.
extern "C" int pm_expert_gather(const void* h, int f32, long long ldh, const int* perm, const float* w, const int* off, int E,
                                int k, int align, int rows, int width, void* xs, int* off_pad, int* dest, cudaStream_t st) {
  if (E < 1 || E > 1024 || k < 1 || align < 0 || width < 1 || (align > 0 && (!off_pad || !dest))) return -1;
  if (rows < 1) return 0;
  return f32 ? gather_launch<float>(h, ldh, perm, w, off, E, k, align, rows, width, xs, off_pad, dest, st)
             : gather_launch<__nv_bfloat16>(h, ldh, perm, w, off, E, k, align, rows, width, xs, off_pad, dest, st);
}

// Both bf16 products of a step with few rows per expert. act 1: out [n, N] = silu(w G_e h) * (w U_e h) for the n sorted pairs
// perm, h [.., ldx] token rows, w [n] weights by pair, W [E][2 N][K]. act 2: out = gelu(W_e h) for the same pairs, W [E][N][K].
// act 0: out = x W_e^T for sorted rows x. K, ldx and W in 16-byte pieces.
extern "C" int pm_expert_gemv(const void* x, long long ldx, const void* W, const int* perm, const float* w, const int* off, int n,
                              int E, int k, int N, int K, int act, void* out, cudaStream_t st) {
  if (E < 1 || k < 1 || N < 1 || K < 8 || K % 8 || ldx % 8 || n > 65535 || act < 0 || act > 2 || (act && !perm) || (act == 1 && !w)) return -1;
  if (n < 1) return 0;
  const ExpertGemvParams p{static_cast<const __nv_bfloat16*>(x), ldx, static_cast<const __nv_bfloat16*>(W), perm, w, off,
                           static_cast<__nv_bfloat16*>(out), n, E, k, N, K};
  if (act == kActSwiglu) expert_gemv_kernel<kActSwiglu><<<dim3((N + 7) / 8, n), 128, 0, st>>>(p);
  else if (act == kActGelu) expert_gemv_kernel<kActGelu><<<dim3((N + 15) / 16, n), 128, 0, st>>>(p);
  else expert_gemv_kernel<kActNone><<<dim3((N + 15) / 16, n), 128, 0, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// x [rows, K] sorted by expert (off [E + 1]; rows behind off[E] are skipped), W [E][N or, act 1, 2 N][K] -> out [rows, N] =
// x W_e^T, act 1: silu(x G_e^T) * (x U_e^T) (gate rows above up rows), act 2: gelu(x W_e^T).
extern "C" int pm_expert_rows(const void* x, int f32, int rows, const void* W, const int* off, int E, int N, int K, int act,
                              void* out, cudaStream_t st) {
  if (E < 1 || N < 1 || K < 1 || act < 0 || act > 2) return -1;
  if (rows < 1) return 0;
  const int tiles = (rows + kRowTile - 1) / kRowTile;
  if (tiles > 65535) return -2;
  const int want = (16 * num_sms() + tiles - 1) / tiles, cols = (N + 7) / 8;
  const dim3 grid(want < cols ? (want < 1 ? 1 : want) : cols, tiles);
  if (f32)
    expert_rows_kernel<float><<<grid, 256, 0, st>>>(static_cast<const float*>(x), rows, static_cast<const float*>(W), off, E, N, K,
                                                    act, static_cast<float*>(out));
  else
    expert_rows_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(x), rows,
                                                            static_cast<const __nv_bfloat16*>(W), off, E, N, K, act,
                                                            static_cast<__nv_bfloat16*>(out));
  return static_cast<int>(cudaGetLastError());
}
