// Selective state-space layers with one decay per head (Mamba-2). Per sequence and head h of group g, with channels
// x [P], B and C [N] after the short causal convolution and silu, and the step size dt > 0:
//
//     S <- exp(-exp(A_h) dt) S + dt B x^T,      y = S^T C + D_h x                        S: [N, P], fp32
//
// The projection row of a token is u = [z: inner | x: inner | B: G N | C: G N | dt: H], inner = H P. What a sequence
// carries from step to step lies in slots: S as [slot][H][N][P4] fp32 (P4 = P rounded up to 4) and the convolution's
// latest inputs as a ring [slot][R][inner + 2 G N], position p in row p % R, with R = taps, so that a step of one token
// writes a row that nobody reads in that step. A sequence whose first token of the step is position 0 starts from zeros
// whatever the slot holds.
//
//   ssm_scan_kernel   any number of tokens, one after the other, convolution included; one CTA per (sequence, head,
//                     slice of P), the state in registers. Decode, short portions, fp32 models.
//   ssm_conv_kernel   convolution + silu and softplus of the step sizes for all tokens of longer portions.
//   ssd_segment_kernel / ssd_chunk_kernel  the recurrence of longer portions in blocks of 64 tokens on the tensor cores,
//                     segments of several blocks in parallel (the first kernel sums what each segment adds to the state,
//                     the second starts every segment from the decayed sum of the earlier ones):
//                     y_i = sum_{j <= i} (C_i.B_j) exp(a_i - a_j) dt_j x_j + exp(a_i) S^T C_i + D x_i (a: running sum of
//                     the log decays), S <- exp(a_63) S + sum_j exp(a_63 - a_j) dt_j B_j x_j^T. x, B and C are bf16
//                     activations; every fp32 factor (decayed scores, state, decayed B) enters the products as the sum
//                     of two bf16 terms, so the recurrence keeps about 16 bits in its operands and fp32 in its sums.
//   ssm_gate_norm_kernel  y * silu(z), RMS norm over equal parts of the row, weight; it also moves the last inputs of
//                     the convolution into the ring (it runs after every reader of the ring).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <type_traits>
#include "elem.cuh"
#include "host_util.cuh"
#include "mma_sync.cuh"
#include "pmetal_b200.h"

namespace pm {

struct SsmDims {
  int H, P, N, G, taps;
  int inner, conv;      // H P, inner + 2 G N
  int P4;               // stored width of a state row
};

static SsmDims make_dims(int H, int P, int N, int G, int taps) {
  SsmDims d;
  d.H = H; d.P = P; d.N = N; d.G = G; d.taps = taps;
  d.inner = H * P;
  d.conv = d.inner + 2 * G * N;
  d.P4 = (P + 3) / 4 * 4;
  return d;
}

template <typename T>
struct ScanParams {
  const T* u;
  long long ldu;
  const float* conv_w;     // [taps][conv]
  const float* conv_b;
  const float* dt_bias;
  const float* a_log;
  const float* dskip;
  const T* ring;
  float* state;
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  T* y;                    // [tokens, inner]
  SsmDims d;
  int pw;                  // channels of P per CTA (multiple of 4)
};

constexpr int kScanThreads = 256;

// E: state rows per thread (float4 each).
template <typename T, int E>
__global__ void __launch_bounds__(kScanThreads, E <= 8 ? 4 : 2) ssm_scan_kernel(const ScanParams<T> p) {
  extern __shared__ __align__(16) float scan_smem[];
  const SsmDims& d = p.d;
  const int seq = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * p.pw;
  const int len = p.q_lens[seq];
  if (len <= 0) return;
  const int cols = p.pw / 4, groups = kScanThreads / cols;
  float* sx = scan_smem;                     // [pw]
  float* sb = sx + p.pw;                     // [N]
  float* sc = sb + d.N;                      // [N]
  float* part = sx + (p.pw + 2 * d.N + 3) / 4 * 4;     // [groups][pw]
  const int q0 = p.q_start[seq], start = p.seq_lens[seq] - len;
  const long long slot = p.slots[seq];
  const int g = h / (d.H / d.G);
  const int cx = h * d.P, cb = d.inner + g * d.N, cc = d.inner + (d.G + g) * d.N;     // first channels of x, B, C
  const int col = threadIdx.x % cols, grp = threadIdx.x / cols;
  const bool owner = grp < groups && p0 + col * 4 < d.P4;
  float4 S[E];
  float* st = p.state + ((slot * d.H + h) * d.N) * d.P4 + p0 + col * 4;
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const int n = grp + i * groups;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (owner && start > 0 && n < d.N) S[i] = *reinterpret_cast<const float4*>(st + static_cast<long long>(n) * d.P4);
  }
  const float a = -expf(p.a_log[h]), skip = p.dskip[h], bias_dt = p.dt_bias[h];
  for (int t = 0; t < len; ++t) {
    const int pos = start + t;
    const T* row = p.u + static_cast<long long>(q0 + t) * p.ldu;
    const int turn = pos % d.taps;
    __syncthreads();                          // the previous token's readers are done
    for (int i = threadIdx.x; i < p.pw + 2 * d.N; i += kScanThreads) {
      int c;
      if (i < p.pw) {
        c = p0 + i < d.P ? cx + p0 + i : -1;
      } else {
        c = i < p.pw + d.N ? cb + (i - p.pw) : cc + (i - p.pw - d.N);
      }
      float v = 0.f;
      if (c >= 0) {
        v = p.conv_b[c];
        for (int j0 = 0; j0 < d.taps; j0 += 4) {           // four independent loads at a time
          float w[4], in[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int j = j0 + k, back = d.taps - 1 - j, src = pos - back;
            const bool ok = j < d.taps && src >= 0;
            const T* at = t >= back ? row + d.inner + c - static_cast<long long>(back) * p.ldu
                                    : p.ring + (slot * d.taps + (back > turn ? turn - back + d.taps : turn - back)) * d.conv + c;
            w[k] = ok ? p.conv_w[static_cast<long long>(j) * d.conv + c] : 0.f;
            in[k] = ok ? to_f(*at) : 0.f;
          }
#pragma unroll
          for (int k = 0; k < 4; ++k) v = fmaf(w[k], in[k], v);
        }
        v = silu_f(v);
      }
      scan_smem[i] = v;
    }
    const float dt = softplus_f(to_f(row[d.inner + d.conv + h]) + bias_dt);
    const float decay = expf(a * dt);
    __syncthreads();
    if (owner) {
      float4 x = *reinterpret_cast<const float4*>(sx + col * 4);
      x.x *= dt; x.y *= dt; x.z *= dt; x.w *= dt;
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < E; ++i) {
        const int n = grp + i * groups;
        if (n < d.N) {
          const float b = sb[n], c = sc[n];
          S[i].x = fmaf(decay, S[i].x, b * x.x); y.x = fmaf(c, S[i].x, y.x);
          S[i].y = fmaf(decay, S[i].y, b * x.y); y.y = fmaf(c, S[i].y, y.y);
          S[i].z = fmaf(decay, S[i].z, b * x.z); y.z = fmaf(c, S[i].z, y.z);
          S[i].w = fmaf(decay, S[i].w, b * x.w); y.w = fmaf(c, S[i].w, y.w);
        }
      }
      *reinterpret_cast<float4*>(part + grp * p.pw + col * 4) = y;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.pw; i += kScanThreads) {
      if (p0 + i >= d.P) continue;
      float v = 0.f;
      for (int k = 0; k < groups; ++k) v += part[k * p.pw + i];
      put(p.y + static_cast<long long>(q0 + t) * d.inner + cx + p0 + i, fmaf(skip, sx[i], v));
    }
  }
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const int n = grp + i * groups;
    if (owner && n < d.N) *reinterpret_cast<float4*>(st + static_cast<long long>(n) * d.P4) = S[i];
  }
}

// ------------------------------------------------------------------------------------------- longer portions (bf16)
constexpr int kConvTokens = 8;

struct ConvParams {
  const __nv_bfloat16* u;
  long long ldu;
  const float* conv_w;     // [taps][conv]
  const float* conv_b;
  const float* dt_bias;
  const __nv_bfloat16* ring;
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  __nv_bfloat16* act;      // [tokens, conv]
  float* dt;               // [tokens, H]
  SsmDims d;
};

// grid (tiles of 8 tokens, sequences, channel tiles + 1): a thread owns V channels of 8 consecutive tokens; the last
// channel tile computes the step sizes. TAPS = 0: any number of taps.
template <int V, int TAPS>
__global__ void __launch_bounds__(128) ssm_conv_kernel(const ConvParams p) {
  const SsmDims& d = p.d;
  const int seq = blockIdx.y, len = p.q_lens[seq], t0 = blockIdx.x * kConvTokens;
  if (t0 >= len) return;
  const int q0 = p.q_start[seq], start = p.seq_lens[seq] - len, n_tok = min(kConvTokens, len - t0);
  if (blockIdx.z == gridDim.z - 1) {
    for (int i = threadIdx.x; i < n_tok * d.H; i += blockDim.x) {
      const int t = i / d.H, h = i - t * d.H;
      const long long r = q0 + t0 + t;
      p.dt[r * d.H + h] = softplus_f(__bfloat162float(p.u[r * p.ldu + d.inner + d.conv + h]) + p.dt_bias[h]);
    }
    return;
  }
  const int c = (blockIdx.z * 128 + threadIdx.x) * V;
  if (c >= d.conv) return;
  const long long slot = p.slots[seq];
  float acc[kConvTokens][V], b[V];
  load_vec<V>(p.conv_b + c, b);
#pragma unroll
  for (int t = 0; t < kConvTokens; ++t)
#pragma unroll
    for (int e = 0; e < V; ++e) acc[t][e] = b[e];
  auto input = [&](int t, float (&in)[V]) {               // input of token t0 + t (t may be negative), zeros before the start
    const int src = start + t0 + t;
    if (src < 0) {
#pragma unroll
      for (int e = 0; e < V; ++e) in[e] = 0.f;
    } else if (t0 + t >= 0) {
      load_vec<V>(p.u + static_cast<long long>(q0 + t0 + t) * p.ldu + d.inner + c, in);
    } else {
      load_vec<V>(p.ring + (slot * d.taps + src % d.taps) * d.conv + c, in);
    }
  };
  if (TAPS > 0) {
    float w[TAPS > 0 ? TAPS : 1][V];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_vec<V>(p.conv_w + static_cast<long long>(j) * d.conv + c, w[j]);
    // all rows are requested before the first is used
    using Raw = typename std::conditional<V == 4, uint2, __nv_bfloat16>::type;
    Raw raw[kConvTokens + TAPS];
    bool have[kConvTokens + TAPS];
    const int turn = (start + t0 + d.taps) % d.taps;       // ring row of position start + t0
#pragma unroll
    for (int r = 1 - TAPS; r < kConvTokens; ++r) {
      const int back = -r;                                 // only positions before this portion lie in the ring
      const __nv_bfloat16* at = t0 + r >= 0 ? p.u + static_cast<long long>(q0 + t0 + r) * p.ldu + d.inner + c
                                            : p.ring + (slot * d.taps + (back > turn ? turn - back + d.taps : turn - back)) * d.conv + c;
      have[r + TAPS - 1] = r < n_tok && start + t0 + r >= 0;
      if (have[r + TAPS - 1]) raw[r + TAPS - 1] = *reinterpret_cast<const Raw*>(at);
    }
#pragma unroll
    for (int r = 1 - TAPS; r < kConvTokens; ++r) {
      float in[V];
      if (have[r + TAPS - 1]) {
        load_vec<V>(reinterpret_cast<const __nv_bfloat16*>(&raw[r + TAPS - 1]), in);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) in[e] = 0.f;
      }
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int t = r + TAPS - 1 - j;                    // row r is tap j of token t
        if (t >= 0 && t < kConvTokens)
#pragma unroll
          for (int e = 0; e < V; ++e) acc[t][e] = fmaf(w[j][e], in[e], acc[t][e]);
      }
    }
  } else {
    for (int j = 0; j < d.taps; ++j) {
      float w[V];
      load_vec<V>(p.conv_w + static_cast<long long>(j) * d.conv + c, w);
#pragma unroll
      for (int t = 0; t < kConvTokens; ++t) {
        if (t >= n_tok) break;
        float in[V];
        input(t - (d.taps - 1 - j), in);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[t][e] = fmaf(w[e], in[e], acc[t][e]);
      }
    }
  }
#pragma unroll
  for (int t = 0; t < kConvTokens; ++t) {
    if (t >= n_tok) break;
#pragma unroll
    for (int e = 0; e < V; ++e) acc[t][e] = silu_fast(acc[t][e]);
    store_vec<V>(p.act + static_cast<long long>(q0 + t0 + t) * d.conv + c, acc[t]);
  }
}

struct ChunkParams {
  const __nv_bfloat16* act;   // [tokens, conv]
  const float* dt;            // [tokens, H]
  const float* a_log;
  const float* dskip;
  float* state;
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  __nv_bfloat16* y;           // [tokens, inner]
  // segments: seg_state [seq][n_seg][H][N][P4] (0: the state a sequence starts from, k > 0: what segment k - 1 adds to it),
  // seg_decay [seq][n_seg][H] (decay of the state over segment k)
  float* seg_state;
  float* seg_decay;
  int n_seg, seg_chunks;      // segments of the longest portion, blocks per segment
  SsmDims d;
  int n16;                    // N rounded up to 16
  int aligned;                // rows can be copied 16 bytes at a time
};

constexpr int kChunk = 64;
constexpr int kSlice = 32;            // channels of P per CTA
constexpr int kLdX = kSlice + 8;
constexpr float kLog2e = 1.4426950408889634f;

// Rows t0 .. t0 + 63 of `act`, `width` columns from c0 (multiple of 8, zero filled beyond valid_w and beyond the portion).
__device__ __forceinline__ void ssd_load_rows(const ChunkParams& p, __nv_bfloat16* dst, int ld, int width, int valid_w, int c0,
                                              long long q0, int t0, int len) {
  if (p.aligned) {
    const int per = width / 8, dr = 128 / per, dc = 128 - dr * per;
    int r = threadIdx.x / per, c = threadIdx.x - r * per;
    for (; r < kChunk; r += dr, c += dc) {
      if (c >= per) {
        c -= per;
        if (++r >= kChunk) break;
      }
      const bool ok = t0 + r < len && c * 8 < valid_w;
      const __nv_bfloat16* src = p.act + (q0 + (ok ? t0 + r : 0)) * p.d.conv + c0 + (ok ? c * 8 : 0);
      ms_cp16(ms_addr(dst + r * ld + c * 8), src, ok);
    }
  } else {
    for (int i = threadIdx.x; i < kChunk * width; i += 128) {
      const int r = i / width, c = i - r * width;
      const bool ok = t0 + r < len && c < valid_w;
      dst[r * ld + c] = ok ? p.act[(q0 + t0 + r) * p.d.conv + c0 + c] : __float2bfloat16(0.f);
    }
  }
}

// One warp's copy of the block's running log2 decays and of the weights with which its tokens enter the state; returns the
// log2 decay over the block.
__device__ __forceinline__ float ssd_decays(const float* dts, float a2, float* cum, float* wgt, int lane) {
  const float d0 = dts[2 * lane], d1 = dts[2 * lane + 1];
  float run = a2 * d0 + a2 * d1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += up;
  }
  const float total = __shfl_sync(0xffffffffu, run, 31);
  const float c1 = run, c0 = run - a2 * d1;
  __syncwarp();
  *reinterpret_cast<float2*>(cum + 2 * lane) = make_float2(c0, c1);
  *reinterpret_cast<float2*>(wgt + 2 * lane) = make_float2(exp2f(total - c0) * d0, exp2f(total - c1) * d1);
  __syncwarp();
  return total;
}

// S (rows of this warp) <- keep * S + sum_j wgt_j B_j x_j^T
template <int NI>
__device__ __forceinline__ void ssd_update(float (&S)[NI][4][4], float keep, const float* wgt, uint32_t aB, uint32_t aX, int ldn,
                                           int n16, int warp, int lane) {
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][nt][e] *= keep;
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    uint32_t fx[2][4];
#pragma unroll
    for (int np = 0; np < 2; ++np) ms_ldsm4_t(ms_b_nn_at(aX, kLdX, kk * 16, np * 16, lane), fx[np]);
    const int j = kk * 16 + 2 * (lane & 3);
    const float2 wa = *reinterpret_cast<const float2*>(wgt + j), wb = *reinterpret_cast<const float2*>(wgt + j + 8);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int n0 = (warp + 4 * i) * 16;
      if (n0 >= n16) continue;
      uint32_t fb[4], fh[4], fl[4];
      ms_ldsm4_t(ms_a_t_at(aB, ldn, kk * 16, n0, lane), fb);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float lo = __uint_as_float(fb[q] << 16), hi = __uint_as_float(fb[q] & 0xffff0000u);
        ms_split(lo * (q & 2 ? wb.x : wa.x), hi * (q & 2 ? wb.y : wa.y), fh[q], fl[q]);
      }
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        ms_mma(S[i][2 * np], fh, fx[np][0], fx[np][1]);
        ms_mma(S[i][2 * np + 1], fh, fx[np][2], fx[np][3]);
        ms_mma(S[i][2 * np], fl, fx[np][0], fx[np][1]);
        ms_mma(S[i][2 * np + 1], fl, fx[np][2], fx[np][3]);
      }
    }
  }
}

// Calls f(fragment pair, row n, channel c) for this thread's accumulator pairs (channels c, c + 1).
template <int NI, typename F>
__device__ __forceinline__ void ssd_each(float (&S)[NI][4][4], int n, int pw, int warp, int lane, F f) {
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int row = (warp + 4 * i) * 16 + (lane >> 2) + 8 * hf, c = nt * 8 + 2 * (lane & 3);
        if (row < n && c < pw) f(S[i][nt][2 * hf], S[i][nt][2 * hf + 1], row, c);
      }
}

// What every segment but the last adds to the state, with segment-parallel CTAs. grid (slices * n_seg, H, sequences).
template <int NI>
__global__ void __launch_bounds__(128) ssd_segment_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) uint8_t ssd_smem[];
  const SsmDims& d = p.d;
  const int slices = gridDim.x / p.n_seg;
  const int seq = blockIdx.z, h = blockIdx.y, p0 = (blockIdx.x % slices) * kSlice, seg = blockIdx.x / slices;
  const int len = p.q_lens[seq];
  const int n_chunks = (len + kChunk - 1) / kChunk;
  if ((seg + 1) * p.seg_chunks >= n_chunks) return;            // the last segment is summed by the main kernel
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ldn = p.n16 + 8, tile_n = kChunk * ldn, tile_x = kChunk * kLdX;
  __nv_bfloat16* sB = reinterpret_cast<__nv_bfloat16*>(ssd_smem);        // [2][64][ldn]
  __nv_bfloat16* sX = sB + 2 * tile_n;                                   // [2][64][kLdX]
  float* sDt = reinterpret_cast<float*>(sX + 2 * tile_x);                // [2][64]
  float* cum = sDt + 2 * kChunk + warp * kChunk;                         // [4 warps][64]
  float* wgt = sDt + 6 * kChunk + warp * kChunk;                         // [4 warps][64]
  const long long q0 = p.q_start[seq];
  const int start = p.seq_lens[seq] - len;
  const int g = h / (d.H / d.G);
  const int cx = h * d.P + p0, cb = d.inner + g * d.N, pw = min(kSlice, d.P - p0);
  const float a2 = -expf(p.a_log[h]) * kLog2e;
  const long long mat = static_cast<long long>(d.N) * d.P4;
  auto slot_of = [&](int k) { return (static_cast<long long>(seq) * p.n_seg + k) * d.H + h; };
  auto load_chunk = [&](int ch, int buf) {
    const int t0 = ch * kChunk;
    ssd_load_rows(p, sB + buf * tile_n, ldn, p.n16, d.N, cb, q0, t0, len);
    ssd_load_rows(p, sX + buf * tile_x, kLdX, kSlice, pw, cx, q0, t0, len);
    if (threadIdx.x < kChunk) sDt[buf * kChunk + threadIdx.x] = p.dt[(q0 + t0 + threadIdx.x) * d.H + h];
    ms_commit();
  };
  float S[NI][4][4];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][nt][e] = 0.f;
  const int c0 = seg * p.seg_chunks;
  load_chunk(c0, 0);
  if (seg == 0) {                                              // the starting state, before the main kernel overwrites it
    const float* st = p.state + (static_cast<long long>(p.slots[seq]) * d.H + h) * mat + p0;
    float* dst = p.seg_state + slot_of(0) * mat + p0;
    ssd_each<NI>(S, d.N, pw, warp, lane, [&](float&, float&, int n, int c) {
      const long long o = static_cast<long long>(n) * d.P4 + c;
      *reinterpret_cast<float2*>(dst + o) = start > 0 ? *reinterpret_cast<const float2*>(st + o) : make_float2(0.f, 0.f);
    });
  }
  float sum = 0.f;
  for (int k = 0; k < p.seg_chunks; ++k) {
    const int buf = k & 1;
    ms_wait<0>();
    __syncthreads();
    if (k + 1 < p.seg_chunks) load_chunk(c0 + k + 1, buf ^ 1);
    const float total = ssd_decays(sDt + buf * kChunk, a2, cum, wgt, lane);
    sum += total;
    ssd_update<NI>(S, exp2f(total), wgt, ms_addr(sB + buf * tile_n), ms_addr(sX + buf * tile_x), ldn, p.n16, warp, lane);
  }
  float* dst = p.seg_state + slot_of(seg + 1) * mat + p0;
  ssd_each<NI>(S, d.N, pw, warp, lane, [&](float& v0, float& v1, int n, int c) {
    *reinterpret_cast<float2*>(dst + static_cast<long long>(n) * d.P4 + c) = make_float2(v0, v1);
  });
  if (threadIdx.x == 0 && p0 == 0) p.seg_decay[slot_of(seg)] = exp2f(sum);
}

// NI: state row tiles (16 rows) per warp; 4 warps cover N <= 64 NI. Same grid as ssd_segment_kernel.
template <int NI>
__global__ void __launch_bounds__(128) ssd_chunk_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) uint8_t ssd_smem[];
  const SsmDims& d = p.d;
  const int slices = gridDim.x / p.n_seg;
  const int seq = blockIdx.z, h = blockIdx.y, p0 = (blockIdx.x % slices) * kSlice, seg = blockIdx.x / slices;
  const int len = p.q_lens[seq];
  const int n_chunks = (len + kChunk - 1) / kChunk, ch0 = seg * p.seg_chunks, ch1 = min(n_chunks, ch0 + p.seg_chunks);
  if (ch0 >= ch1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, t4 = lane & 3;
  const int ldn = p.n16 + 8, tile_n = kChunk * ldn, tile_x = kChunk * kLdX;
  __nv_bfloat16* sC = reinterpret_cast<__nv_bfloat16*>(ssd_smem);        // [64][ldn]
  __nv_bfloat16* sB = sC + tile_n;                                       // [64][ldn]
  __nv_bfloat16* sX = sB + tile_n;                                       // [64][kLdX]
  __nv_bfloat16* sSh = sX + tile_x;                                      // [n16][kLdX]
  __nv_bfloat16* sSl = sSh + p.n16 * kLdX;                               // [n16][kLdX]
  float* sDt = reinterpret_cast<float*>(sSl + p.n16 * kLdX);             // [64]
  float* cum = sDt + kChunk + warp * kChunk;                             // [4 warps][64]
  float* wgt = sDt + 5 * kChunk + warp * kChunk;                         // [4 warps][64]

  const long long q0 = p.q_start[seq];
  const int start = p.seq_lens[seq] - len;
  const int g = h / (d.H / d.G);
  const int cx = h * d.P + p0, cb = d.inner + g * d.N, cc = d.inner + (d.G + g) * d.N;
  const int pw = min(kSlice, d.P - p0);
  const float a2 = -expf(p.a_log[h]) * kLog2e, skip = p.dskip[h];
  const long long mat = static_cast<long long>(d.N) * d.P4;
  float* st = p.state + (static_cast<long long>(p.slots[seq]) * d.H + h) * mat + p0;

  auto load_chunk = [&](int ch) {
    const int t0 = ch * kChunk;
    ssd_load_rows(p, sC, ldn, p.n16, d.N, cc, q0, t0, len);
    ssd_load_rows(p, sB, ldn, p.n16, d.N, cb, q0, t0, len);
    ssd_load_rows(p, sX, kLdX, kSlice, pw, cx, q0, t0, len);
    if (threadIdx.x < kChunk)
      sDt[threadIdx.x] = t0 + static_cast<int>(threadIdx.x) < len ? p.dt[(q0 + t0 + threadIdx.x) * d.H + h] : 0.f;
    ms_commit();
  };
  load_chunk(ch0);

  // this warp's rows of the state at the start of the segment, accumulator layout
  float S[NI][4][4];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][nt][e] = 0.f;
  if (n_chunks <= p.seg_chunks) {
    if (start > 0)
      ssd_each<NI>(S, d.N, pw, warp, lane, [&](float& v0, float& v1, int n, int c) {
        const float2 v = *reinterpret_cast<const float2*>(st + static_cast<long long>(n) * d.P4 + c);
        v0 = v.x;
        v1 = v.y;
      });
  } else {
    for (int k = 0; k <= seg; ++k) {
      const long long o = (static_cast<long long>(seq) * p.n_seg + k) * d.H + h;
      const float* src = p.seg_state + o * mat + p0;
      const float keep = k > 0 ? p.seg_decay[o - d.H] : 0.f;
      ssd_each<NI>(S, d.N, pw, warp, lane, [&](float& v0, float& v1, int n, int c) {
        const float2 v = *reinterpret_cast<const float2*>(src + static_cast<long long>(n) * d.P4 + c);
        v0 = fmaf(keep, v0, v.x);
        v1 = fmaf(keep, v1, v.y);
      });
    }
  }
  auto publish = [&]() {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int r0 = (warp + 4 * i) * 16;
      if (r0 >= p.n16) continue;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          uint32_t hi, lo;
          ms_split(S[i][nt][2 * hf], S[i][nt][2 * hf + 1], hi, lo);
          const int off = (r0 + g4 + 8 * hf) * kLdX + nt * 8 + 2 * t4;
          *reinterpret_cast<uint32_t*>(sSh + off) = hi;
          *reinterpret_cast<uint32_t*>(sSl + off) = lo;
        }
    }
  };
  publish();
  const uint32_t aC = ms_addr(sC), aB = ms_addr(sB), aX = ms_addr(sX), aSh = ms_addr(sSh), aSl = ms_addr(sSl);
  const int r0 = warp * 16;

  for (int ch = ch0; ch < ch1; ++ch) {
    ms_wait<0>();
    __syncthreads();                       // the block's rows and the published state are visible
    const float total = ssd_decays(sDt, a2, cum, wgt, lane);
    float s[8][4], yi[4][4], y[4][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) yi[i][e] = y[i][e] = 0.f;
    // scores C B^T of the causal part, and the state's contribution, in one pass over C
    for (int k = 0; k < p.n16; k += 16) {
      uint32_t fa[4];
      ms_ldsm4(ms_a_at(aC, ldn, r0, k, lane), fa);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (np <= warp) {
          uint32_t fb[4];
          ms_ldsm4(ms_b_nt_at(aB, ldn, np * 16, k, lane), fb);
          ms_mma(s[2 * np], fa, fb[0], fb[1]);
          ms_mma(s[2 * np + 1], fa, fb[2], fb[3]);
        }
      }
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t fh[4], fl[4];
        ms_ldsm4_t(ms_b_nn_at(aSh, kLdX, k, np * 16, lane), fh);
        ms_ldsm4_t(ms_b_nn_at(aSl, kLdX, k, np * 16, lane), fl);
        ms_mma(yi[2 * np], fa, fh[0], fh[1]);
        ms_mma(yi[2 * np + 1], fa, fh[2], fh[3]);
        ms_mma(yi[2 * np], fa, fl[0], fl[1]);
        ms_mma(yi[2 * np + 1], fa, fl[2], fl[3]);
      }
    }
    const float ci[2] = {cum[r0 + g4], cum[r0 + g4 + 8]};
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk > warp) break;
      float m[2][4];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int j0 = kk * 16 + q * 8 + 2 * t4;
        const float2 cj = *reinterpret_cast<const float2*>(cum + j0), dj = *reinterpret_cast<const float2*>(sDt + j0);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const bool seen = kk < warp || j0 + (e & 1) <= r0 + g4 + ((e & 2) ? 8 : 0);
          m[q][e] = seen ? s[2 * kk + q][e] * exp2f(ci[e >> 1] - ((e & 1) ? cj.y : cj.x)) * ((e & 1) ? dj.y : dj.x) : 0.f;
        }
      }
      uint32_t fh[4], fl[4];
      ms_split(m[0][0], m[0][1], fh[0], fl[0]);
      ms_split(m[0][2], m[0][3], fh[1], fl[1]);
      ms_split(m[1][0], m[1][1], fh[2], fl[2]);
      ms_split(m[1][2], m[1][3], fh[3], fl[3]);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t fx[4];
        ms_ldsm4_t(ms_b_nn_at(aX, kLdX, kk * 16, np * 16, lane), fx);
        ms_mma(y[2 * np], fh, fx[0], fx[1]);
        ms_mma(y[2 * np + 1], fh, fx[2], fx[3]);
        ms_mma(y[2 * np], fl, fx[0], fx[1]);
        ms_mma(y[2 * np + 1], fl, fx[2], fx[3]);
      }
    }
    // y of this warp's 16 tokens
    const float ei[2] = {exp2f(ci[0]), exp2f(ci[1])};
    const int t0 = ch * kChunk;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = r0 + g4 + 8 * hf, c = nt * 8 + 2 * t4;
        if (t0 + i >= len || c >= pw) continue;
        const float2 xf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sX + i * kLdX + c));
        const float v0 = fmaf(skip, xf.x, fmaf(ei[hf], yi[nt][2 * hf], y[nt][2 * hf]));
        const float v1 = fmaf(skip, xf.y, fmaf(ei[hf], yi[nt][2 * hf + 1], y[nt][2 * hf + 1]));
        __nv_bfloat16* dst = p.y + (q0 + t0 + i) * d.inner + cx + c;
        if (p.aligned) {
          *reinterpret_cast<uint32_t*>(dst) = pack_bf16(v0, v1);
        } else {
          dst[0] = __float2bfloat16(v0);
          if (c + 1 < pw) dst[1] = __float2bfloat16(v1);
        }
      }
    if (ch + 1 < ch1 || ch1 == n_chunks)
      ssd_update<NI>(S, exp2f(total), wgt, aB, aX, ldn, p.n16, warp, lane);
    __syncthreads();                       // everyone has read this block's rows and the published state
    if (ch + 1 < ch1) {
      load_chunk(ch + 1);
      publish();
    }
  }
  if (ch1 == n_chunks)
    ssd_each<NI>(S, d.N, pw, warp, lane, [&](float& v0, float& v1, int n, int c) {
      *reinterpret_cast<float2*>(st + static_cast<long long>(n) * d.P4 + c) = make_float2(v0, v1);
    });
}

// ------------------------------------------------------------------------------------------- gate, norm, ring
template <typename T, int V>
__global__ void ssm_gate_norm_kernel(const T* __restrict__ y, const T* __restrict__ u, long long ldu,
                                     const float* __restrict__ w, float eps, int parts, T* __restrict__ out,
                                     T* __restrict__ ring, const int* __restrict__ slots, const int* __restrict__ seq_of,
                                     const int* __restrict__ pos, const int* __restrict__ seq_lens, SsmDims d) {
  extern __shared__ __align__(16) float part_row[];
  const long long t = blockIdx.x;
  const int part = blockIdx.y, width = d.inner / parts, c0 = part * width;
  // the last taps - 1 inputs of the convolution stay with the sequence
  const int seq = seq_of[t], ps = pos[t];
  if (seq_lens[seq] - ps < d.taps) {
    T* dst = ring + (static_cast<long long>(slots[seq]) * d.taps + ps % d.taps) * d.conv;
    const T* src = u + t * ldu + d.inner;
    for (int c = part * blockDim.x + threadIdx.x; c < d.conv; c += parts * blockDim.x) dst[c] = src[c];
  }
  float ss = 0.f;
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V) {
    float v[V], z[V];
    load_vec<V>(y + t * d.inner + c0 + k, v);
    load_vec<V>(u + t * ldu + c0 + k, z);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      v[e] *= silu_f(z[e]);
      part_row[k + e] = v[e];
      ss = fmaf(v[e], v[e], ss);
    }
  }
  const float r = 1.f / sqrtf(block_sum(ss) / static_cast<float>(width) + eps);
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V) {
    float v[V], g[V];
    load_vec<V>(w + c0 + k, g);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = part_row[k + e] * r * g[e];
    store_vec<V>(out + t * d.inner + c0 + k, v);
  }
}

// The same with one warp per (token, part) and the part in registers: widths up to 256 IT, rows copied in 8-element vectors.
template <typename T, int IT>
__global__ void __launch_bounds__(256) ssm_gate_norm_warp_kernel(const T* __restrict__ y, const T* __restrict__ u, long long ldu,
                                                                 const float* __restrict__ w, float eps, int parts,
                                                                 T* __restrict__ out, T* __restrict__ ring,
                                                                 const int* __restrict__ slots, const int* __restrict__ seq_of,
                                                                 const int* __restrict__ pos, const int* __restrict__ seq_lens,
                                                                 int n_tok, SsmDims d) {
  const long long item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  const long long t = item / parts;
  if (t >= n_tok) return;
  const int part = static_cast<int>(item - t * parts), width = d.inner / parts, c0 = part * width;
  float v[IT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int k = (i * 32 + lane) * 8;
    if (k < width) {
      float z[8];
      load_vec<8>(y + t * d.inner + c0 + k, v[i]);
      load_vec<8>(u + t * ldu + c0 + k, z);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        v[i][e] *= sizeof(T) == 2 ? silu_fast(z[e]) : silu_f(z[e]);
        ss = fmaf(v[i][e], v[i][e], ss);
      }
    }
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(width) + eps);
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int k = (i * 32 + lane) * 8;
    if (k < width) {
      float g[8];
      load_vec<8>(w + c0 + k, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] *= r * g[e];
      store_vec<8>(out + t * d.inner + c0 + k, v[i]);
    }
  }
  const int seq = seq_of[t], ps = pos[t];
  if (seq_lens[seq] - ps < d.taps) {
    T* dst = ring + (static_cast<long long>(slots[seq]) * d.taps + ps % d.taps) * d.conv;
    const T* src = u + t * ldu + d.inner;
    for (int c = (part * 32 + lane) * 8; c < d.conv; c += parts * 256) {
      float x[8];
      load_vec<8>(src + c, x);
      store_vec<8>(dst + c, x);
    }
  }
}

template <typename T>
static int scan_launch(ScanParams<T> p, int n_seq, cudaStream_t st) {
  const SsmDims& d = p.d;
  // widest slice of P whose state fits in 16 float4 per thread
  int pw = d.P4;
  auto rows = [&](int w) { const int groups = kScanThreads / (w / 4); return groups < 1 ? 1 << 30 : (d.N + groups - 1) / groups; };
  while (pw > 4 && rows(pw) > 16) pw = (pw / 2 + 3) / 4 * 4;
  if (rows(pw) > 16) return -3;
  p.pw = pw;
  const int groups = kScanThreads / (pw / 4), e = rows(pw);
  const size_t smem = static_cast<size_t>((pw + 2 * d.N + 3) / 4 * 4 + groups * pw) * sizeof(float);
  if (smem > 48 * 1024) return -3;
  const dim3 grid(n_seq, d.H, (d.P4 + pw - 1) / pw);
  if (e <= 1) ssm_scan_kernel<T, 1><<<grid, kScanThreads, smem, st>>>(p);
  else if (e <= 2) ssm_scan_kernel<T, 2><<<grid, kScanThreads, smem, st>>>(p);
  else if (e <= 4) ssm_scan_kernel<T, 4><<<grid, kScanThreads, smem, st>>>(p);
  else if (e <= 8) ssm_scan_kernel<T, 8><<<grid, kScanThreads, smem, st>>>(p);
  else ssm_scan_kernel<T, 16><<<grid, kScanThreads, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static ScanParams<T> scan_params(const void* u, long long ldu, const float* conv_w, const float* conv_b,
                                 const float* dt_bias, const float* a_log, const float* dskip, const void* ring,
                                 float* state, const int* slots, const int* q_start, const int* q_lens,
                                 const int* seq_lens, void* y, const SsmDims& d) {
  ScanParams<T> p{};
  p.u = static_cast<const T*>(u); p.ldu = ldu; p.conv_w = conv_w; p.conv_b = conv_b; p.dt_bias = dt_bias;
  p.a_log = a_log; p.dskip = dskip; p.ring = static_cast<const T*>(ring); p.state = state; p.slots = slots;
  p.q_start = q_start; p.q_lens = q_lens; p.seq_lens = seq_lens; p.y = static_cast<T*>(y); p.d = d;
  return p;
}

template <typename T, int IT>
static int gate_norm_warp_launch(const void* y, const void* u, long long ldu, const float* w, float eps, int parts, void* out,
                                 void* ring, const int* slots, const int* seq_of, const int* pos, const int* seq_lens, int n_tok,
                                 const SsmDims& d, cudaStream_t st) {
  const long long items = static_cast<long long>(n_tok) * parts;
  ssm_gate_norm_warp_kernel<T, IT><<<static_cast<unsigned>((items + 7) / 8), 256, 0, st>>>(
      static_cast<const T*>(y), static_cast<const T*>(u), ldu, w, eps, parts, static_cast<T*>(out), static_cast<T*>(ring),
      slots, seq_of, pos, seq_lens, n_tok, d);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int V>
static int gate_norm_launch(const void* y, const void* u, long long ldu, const float* w, float eps, int parts, void* out,
                            void* ring, const int* slots, const int* seq_of, const int* pos, const int* seq_lens, int n_tok,
                            const SsmDims& d, cudaStream_t st) {
  const int width = d.inner / parts;
  const size_t smem = static_cast<size_t>(width) * sizeof(float);
  static DeviceMax configured;
  if (smem > 40 * 1024 && smem > configured.get()) {
    const cudaError_t e = cudaFuncSetAttribute(ssm_gate_norm_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.set(200 * 1024);
  }
  int threads = (width / V + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
  ssm_gate_norm_kernel<T, V><<<dim3(n_tok, parts), threads, smem, st>>>(
      static_cast<const T*>(y), static_cast<const T*>(u), ldu, w, eps, parts, static_cast<T*>(out), static_cast<T*>(ring),
      slots, seq_of, pos, seq_lens, d);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace pm

using namespace pm;

static bool ssm_bad_dims(int H, int P, int N, int G, int taps) {
  return H < 1 || P < 1 || N < 1 || G < 1 || taps < 1 || H % G;
}

// Token-by-token recurrence with the convolution inside. u [tokens, ldu]; conv_w [taps][conv], conv_b, dt_bias, a_log,
// dskip fp32; ring [slots][taps][conv] in u's type; state [slots][H][N][P4] fp32, read and written; y [tokens, H P].
// Sequence i covers tokens q_start[i] .. + q_lens[i] - 1 and ends at position seq_lens[i] - 1.
extern "C" int pm_ssm_scan(const void* u, int f32, long long ldu, const float* conv_w, const float* conv_b,
                           const float* dt_bias, const float* a_log, const float* dskip, const void* ring, float* state,
                           const int* slots, const int* q_start, const int* q_lens, const int* seq_lens, int n_seq, int H,
                           int P, int N, int G, int taps, void* y, cudaStream_t st) {
  if (ssm_bad_dims(H, P, N, G, taps)) return -1;
  if (n_seq < 1) return 0;
  const SsmDims d = make_dims(H, P, N, G, taps);
  if (ldu < d.inner + d.conv + H) return -2;
  if (f32)
    return scan_launch(scan_params<float>(u, ldu, conv_w, conv_b, dt_bias, a_log, dskip, ring, state, slots, q_start,
                                          q_lens, seq_lens, y, d), n_seq, st);
  return scan_launch(scan_params<__nv_bfloat16>(u, ldu, conv_w, conv_b, dt_bias, a_log, dskip, ring, state, slots, q_start,
                                                q_lens, seq_lens, y, d), n_seq, st);
}

// Whether pm_ssm_chunk covers a state of N rows.
extern "C" int pm_ssm_chunk_supported(int N) { return N >= 1 && N <= 128; }

// The same for longer portions of bf16 models: act [tokens, conv] bf16, dt [tokens, H], seg_state [n_seq][max_seg][H][N][P4]
// and seg_decay [n_seq][max_seg][H] fp32 are work buffers, max_q is the longest of q_lens. A portion is cut into at most
// max_seg segments that run in parallel (fewer when sequences and heads fill the machine by themselves).
extern "C" int pm_ssm_chunk(const void* u, long long ldu, const float* conv_w, const float* conv_b, const float* dt_bias,
                            const float* a_log, const float* dskip, const void* ring, float* state, const int* slots,
                            const int* q_start, const int* q_lens, const int* seq_lens, int n_seq, int max_q, int H, int P,
                            int N, int G, int taps, void* act, float* dt, float* seg_state, float* seg_decay,
                            int max_seg, void* y, cudaStream_t st) {
  if (ssm_bad_dims(H, P, N, G, taps) || !pm_ssm_chunk_supported(N) || max_seg < 1) return -1;
  if (n_seq < 1 || max_q < 1) return 0;
  const SsmDims d = make_dims(H, P, N, G, taps);
  if (ldu < d.inner + d.conv + H) return -2;
  ConvParams c{};
  c.u = static_cast<const __nv_bfloat16*>(u); c.ldu = ldu; c.conv_w = conv_w; c.conv_b = conv_b; c.dt_bias = dt_bias;
  c.ring = static_cast<const __nv_bfloat16*>(ring); c.slots = slots; c.q_start = q_start; c.q_lens = q_lens;
  c.seq_lens = seq_lens; c.act = static_cast<__nv_bfloat16*>(act); c.dt = dt; c.d = d;
  const int tiles = (max_q + kConvTokens - 1) / kConvTokens;
  const int v = d.conv % 4 == 0 && d.inner % 4 == 0 && ldu % 4 == 0 ? 4 : 1;
  const dim3 g_conv(tiles, n_seq, (d.conv / v + 127) / 128 + 1);
  if (v == 4 && taps == 4) ssm_conv_kernel<4, 4><<<g_conv, 128, 0, st>>>(c);
  else if (v == 4) ssm_conv_kernel<4, 0><<<g_conv, 128, 0, st>>>(c);
  else ssm_conv_kernel<1, 0><<<g_conv, 128, 0, st>>>(c);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return static_cast<int>(e);
  ChunkParams p{};
  p.act = c.act; p.dt = dt; p.a_log = a_log; p.dskip = dskip; p.state = state; p.slots = slots; p.q_start = q_start;
  p.q_lens = q_lens; p.seq_lens = seq_lens; p.y = static_cast<__nv_bfloat16*>(y); p.d = d;
  p.n16 = (N + 15) / 16 * 16;
  p.aligned = d.conv % 8 == 0 && d.inner % 8 == 0 && N % 8 == 0 && P % 8 == 0;
  // enough CTAs to keep three on every SM for a few rounds
  const int slices = (P + kSlice - 1) / kSlice, n_chunks = (max_q + kChunk - 1) / kChunk;
  const long long base = static_cast<long long>(slices) * H * n_seq;
  long long want = (6ll * num_sms() + base - 1) / base;
  if (want > max_seg) want = max_seg;
  if (want > n_chunks) want = n_chunks;
  p.seg_chunks = (n_chunks + static_cast<int>(want) - 1) / static_cast<int>(want);
  p.n_seg = (n_chunks + p.seg_chunks - 1) / p.seg_chunks;
  p.seg_state = seg_state;
  p.seg_decay = seg_decay;
  const size_t tile_n = static_cast<size_t>(kChunk) * (p.n16 + 8), tile_x = static_cast<size_t>(kChunk) * kLdX;
  const size_t smem = (2 * tile_n + tile_x + 2 * static_cast<size_t>(p.n16) * kLdX) * 2 + 9 * kChunk * 4;
  const size_t smem_seg = (2 * tile_n + 2 * tile_x) * 2 + 10 * kChunk * 4;
  static DeviceOnce once;
  if (once.pending()) {
    e = cudaFuncSetAttribute(ssd_chunk_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(ssd_chunk_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(ssd_segment_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(ssd_segment_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    once.mark();
  }
  const dim3 grid(slices * p.n_seg, H, n_seq);
  if (p.n_seg > 1) {
    if (p.n16 <= 64) ssd_segment_kernel<1><<<grid, 128, smem_seg, st>>>(p);
    else ssd_segment_kernel<2><<<grid, 128, smem_seg, st>>>(p);
    e = cudaGetLastError();
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  if (p.n16 <= 64) ssd_chunk_kernel<1><<<grid, 128, smem, st>>>(p);
  else ssd_chunk_kernel<2><<<grid, 128, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// out [tokens, H P] = RMS norm over `parts` equal parts of y * silu(z) (z: the first H P columns of u), times w; the last
// taps - 1 convolution inputs of every sequence go to the ring. seq_of / pos [tokens]: sequence index and position.
extern "C" int pm_ssm_gate_norm(const void* y, const void* u, int f32, long long ldu, const float* w, float eps, int parts,
                                void* out, void* ring, const int* slots, const int* seq_of, const int* pos,
                                const int* seq_lens, int n_tok, int H, int P, int N, int G, int taps, cudaStream_t st) {
  if (ssm_bad_dims(H, P, N, G, taps) || parts < 1 || (H * P) % parts) return -1;
  if (n_tok < 1) return 0;
  const SsmDims d = make_dims(H, P, N, G, taps);
  const int width = d.inner / parts;
  if (static_cast<size_t>(width) * 4 > 200 * 1024) return -2;
  if (!f32 && width % 8 == 0 && ldu % 8 == 0 && d.conv % 8 == 0 && width <= 1024) {
    if (width <= 256)
      return gate_norm_warp_launch<__nv_bfloat16, 1>(y, u, ldu, w, eps, parts, out, ring, slots, seq_of, pos, seq_lens, n_tok, d, st);
    if (width <= 512)
      return gate_norm_warp_launch<__nv_bfloat16, 2>(y, u, ldu, w, eps, parts, out, ring, slots, seq_of, pos, seq_lens, n_tok, d, st);
    return gate_norm_warp_launch<__nv_bfloat16, 4>(y, u, ldu, w, eps, parts, out, ring, slots, seq_of, pos, seq_lens, n_tok, d, st);
  }
  const bool vec = width % 4 == 0 && ldu % 4 == 0;
  if (f32)
    return vec ? gate_norm_launch<float, 4>(y, u, ldu, w, eps, parts, out, ring, slots, seq_of, pos, seq_lens, n_tok, d, st)
               : gate_norm_launch<float, 1>(y, u, ldu, w, eps, parts, out, ring, slots, seq_of, pos, seq_lens, n_tok, d, st);
  return vec ? gate_norm_launch<__nv_bfloat16, 4>(y, u, ldu, w, eps, parts, out, ring, slots, seq_of, pos, seq_lens, n_tok, d, st)
             : gate_norm_launch<__nv_bfloat16, 1>(y, u, ldu, w, eps, parts, out, ring, slots, seq_of, pos, seq_lens, n_tok, d, st);
}
