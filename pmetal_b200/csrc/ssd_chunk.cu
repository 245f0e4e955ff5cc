// The decayed recurrence in blocks of 64 tokens on the tensor cores, segments of several blocks in parallel: the first kernel
// sums what each segment adds to the state, the second starts every segment from the decayed sum of the earlier ones:
//
//     y_i = sum_{j <= i} (C_i.B_j) exp(a_i - a_j) dt_j x_j + exp(a_i) S^T C_i + D x_i     (a: running sum of the log decays)
//     S  <- exp(a_63) S + sum_j exp(a_63 - a_j) dt_j B_j x_j^T
//
// State-space layers (ssm.cu) have step sizes dt per token and B, C shared by groups of heads; linear attention
// (linear_attn.cu) has keys and queries per head as B and C, values as x, steps of 1 and a fixed decay. The matrix memory
// (gated_linear.cu) has decays and weights per token and a normaliser beside the state, kept in fp32; layers with a decay per
// state row bring the scores within the blocks and B, C with the decays inside. x, B and C are bf16 activations (or, SPLIT, B and
// C the sums of two bf16 terms); every fp32 factor (decayed scores, state, decayed B) enters the products as the sum of two bf16
// terms, so the recurrence keeps about 16 bits in its operands and fp32 in its sums.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include "elem.cuh"
#include "host_util.cuh"
#include "mma_sync.cuh"
#include "ssd_chunk.cuh"

namespace pm {

constexpr int kChunk = 64;
constexpr int kSlice = 32;            // channels of P per group of four warps
constexpr int kLdX = kSlice + 8;
constexpr int kLdA = kChunk + 8;
constexpr float kLog2e = 1.4426950408889634f;

// Rows t0 .. t0 + 63 of `act` (lda apart), `width` columns from c0 (multiple of 8, zero filled beyond valid_w and beyond the portion), by
// NT threads, of which this is number tid.
template <int NT>
__device__ __forceinline__ void ssd_load_rows(int tid, const __nv_bfloat16* act, long long lda, bool aligned, __nv_bfloat16* dst, int ld,
                                              int width, int valid_w, int c0, long long q0, int t0, int len) {
  if (aligned) {
    const int per = width / 8, dr = NT / per, dc = NT - dr * per;
    int r = tid / per, c = tid - r * per;
    for (; r < kChunk; r += dr, c += dc) {
      if (c >= per) {
        c -= per;
        if (++r >= kChunk) break;
      }
      const bool ok = t0 + r < len && c * 8 < valid_w;
      const __nv_bfloat16* src = act + (q0 + (ok ? t0 + r : 0)) * lda + c0 + (ok ? c * 8 : 0);
      ms_cp16(ms_addr(dst + r * ld + c * 8), src, ok);
    }
  } else {
    for (int i = tid; i < kChunk * width; i += NT) {
      const int r = i / width, c = i - r * width;
      const bool ok = t0 + r < len && c < valid_w;
      dst[r * ld + c] = ok ? act[(q0 + t0 + r) * lda + c0 + c] : __float2bfloat16(0.f);
    }
  }
}

// log2 of the decay over a unit step.
__device__ __forceinline__ float ssd_rate(const SsdParams& p, int h) {
  return p.log2_decay ? p.log2_decay[h] : -expf(p.a_log[h]) * kLog2e;
}

// One warp's copy of the block's running log2 decays and of the weights with which its tokens enter the state; returns the
// log2 decay over the block. A token's log2 decay is lds[.] or, where that is null, a2 times its step.
__device__ __forceinline__ float ssd_decays(const float* dts, const float* lds, float a2, float* cum, float* wgt, int lane) {
  const float d0 = dts[2 * lane], d1 = dts[2 * lane + 1];
  const float l0 = lds ? lds[2 * lane] : a2 * d0, l1 = lds ? lds[2 * lane + 1] : a2 * d1;
  float run = l0 + l1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += up;
  }
  const float total = __shfl_sync(0xffffffffu, run, 31);
  const float c1 = run, c0 = run - l1;
  __syncwarp();
  *reinterpret_cast<float2*>(cum + 2 * lane) = make_float2(c0, c1);
  *reinterpret_cast<float2*>(wgt + 2 * lane) = make_float2(exp2f(total - c0) * d0, exp2f(total - c1) * d1);
  __syncwarp();
  return total;
}

// S (rows of this warp) <- keep * S + sum_j wgt_j B_j x_j^T; SPLIT: B = tile at aB + tile at aBl. CHANNEL: keeps[row] in place of
// keep, and B is taken as it is.
template <int NI, bool SPLIT, bool CHANNEL>
__device__ __forceinline__ void ssd_update(float (&S)[NI][4][4], float keep, const float* keeps, const float* wgt, uint32_t aB,
                                           uint32_t aBl, uint32_t aX, int ldn, int n16, int warp, int lane) {
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    float k0 = keep, k1 = keep;
    if (CHANNEL) {
      const int row = (warp + 4 * i) * 16 + (lane >> 2);
      k0 = row < n16 ? keeps[row] : 0.f;
      k1 = row < n16 ? keeps[row + 8] : 0.f;
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][nt][e] *= e & 2 ? k1 : k0;
  }
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    uint32_t fx[2][4];
#pragma unroll
    for (int np = 0; np < 2; ++np) ms_ldsm4_t(ms_b_nn_at(aX, kLdX, kk * 16, np * 16, lane), fx[np]);
    const int j = kk * 16 + 2 * (lane & 3);
    float2 wa, wb;
    if (!CHANNEL) {
      wa = *reinterpret_cast<const float2*>(wgt + j);
      wb = *reinterpret_cast<const float2*>(wgt + j + 8);
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int n0 = (warp + 4 * i) * 16;
      if (n0 >= n16) continue;
      uint32_t fb[4], fbl[4], fh[4], fl[4];
      ms_ldsm4_t(ms_a_t_at(aB, ldn, kk * 16, n0, lane), fb);
      if (SPLIT) ms_ldsm4_t(ms_a_t_at(aBl, ldn, kk * 16, n0, lane), fbl);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        if (CHANNEL) {
          fh[q] = fb[q];
          fl[q] = fbl[q];
          continue;
        }
        float lo = __uint_as_float(fb[q] << 16), hi = __uint_as_float(fb[q] & 0xffff0000u);
        if (SPLIT) {
          lo += __uint_as_float(fbl[q] << 16);
          hi += __uint_as_float(fbl[q] & 0xffff0000u);
        }
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

// n (rows threadIdx.x and threadIdx.x + 128) <- keep n + sum_j wgt_j B_j, in fp32.
__device__ __forceinline__ void ssd_norm_add(float (&n)[2], float keep, const float* wgt, const __nv_bfloat16* B, int ldn, int N) {
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = threadIdx.x + 128 * i;
    if (row >= N) continue;
    float v = n[i] * keep;
#pragma unroll 8
    for (int j = 0; j < kChunk; ++j) v = fmaf(wgt[j], __bfloat162float(B[j * ldn + row]), v);
    n[i] = v;
  }
}

// What every segment but the last adds to the state, with segment-parallel CTAs. A CTA has WG groups of four warps, each with a slice
// of P, on the same B. grid (slices / WG * n_seg, H, sequences).
template <int NI, bool SPLIT, int KIND, int WG>
__global__ void __launch_bounds__(128 * WG) ssd_segment_kernel(const SsdParams p) {
  constexpr int NT = 128 * WG;
  constexpr bool MEMORY = KIND == kSsdMemory, CHANNEL = KIND == kSsdChannel;
  extern __shared__ __align__(16) uint8_t ssd_smem[];
  const SsdParams& d = p;
  const int slices = gridDim.x / p.n_seg, grp = threadIdx.x >> 7, gt = threadIdx.x & 127;
  const int seq = blockIdx.z, h = blockIdx.y, p0 = (blockIdx.x % slices * WG + grp) * kSlice, seg = blockIdx.x / slices;
  const int len = p.q_lens[seq];
  const int n_chunks = (len + kChunk - 1) / kChunk;
  if ((seg + 1) * p.seg_chunks >= n_chunks) return;            // the last segment is summed by the main kernel
  const int warp = gt >> 5, lane = threadIdx.x & 31;
  const int ldn = p.n16 + 8, tile_n = kChunk * ldn, tile_x = kChunk * kLdX;
  __nv_bfloat16* sB = reinterpret_cast<__nv_bfloat16*>(ssd_smem);        // [2][64][ldn]
  __nv_bfloat16* sBl = sB + 2 * tile_n;                                  // [2][64][ldn] (SPLIT)
  __nv_bfloat16* sX = sB + (SPLIT ? 4 : 2) * tile_n + grp * 2 * tile_x;  // [WG][2][64][kLdX]
  float* sDt = reinterpret_cast<float*>(sB + (SPLIT ? 4 : 2) * tile_n + WG * 2 * tile_x);      // [2][64]
  float* cum = sDt + 2 * kChunk + (threadIdx.x >> 5) * kChunk;           // [4 WG warps][64]
  float* wgt = cum + 4 * WG * kChunk;                                    // [4 WG warps][64]
  float* sLd = sDt + (2 + 8 * WG) * kChunk;                              // [2][64] (MEMORY) or the blocks' decays [2][n16] (CHANNEL)
  const long long q0 = p.q_start[seq];
  const int start = p.seq_lens[seq] - len;
  const int g = h / (d.H / d.G);
  const int cx = h * d.P + p0, cb = d.b0 + g * d.NB, pw = max(0, min(kSlice, d.P - p0));
  const float a2 = KIND == kSsdPlain ? ssd_rate(p, h) : 0.f;
  const bool norm = MEMORY && p0 == 0;                                   // this CTA keeps the head's normaliser
  const long long mat = static_cast<long long>(d.N) * d.P4;
  auto slot_of = [&](int k) { return (static_cast<long long>(seq) * p.n_seg + k) * d.H + h; };
  auto load_chunk = [&](int ch, int buf) {
    const int t0 = ch * kChunk;
    ssd_load_rows<NT>(threadIdx.x, p.act, p.ld, p.aligned, sB + buf * tile_n, ldn, p.n16, d.N, cb, q0, t0, len);
    if (SPLIT) ssd_load_rows<NT>(threadIdx.x, p.act, p.ld, p.aligned, sBl + buf * tile_n, ldn, p.n16, d.N, cb + d.lo, q0, t0, len);
    ssd_load_rows<128>(gt, p.x, p.ldx, p.aligned_x, sX + buf * tile_x, kLdX, kSlice, pw, cx, q0, t0, len);
    if (CHANNEL) {
      const long long block = p.c_start[seq] / kChunk + seq + ch;
      for (int n = threadIdx.x; n < p.n16; n += NT) sLd[buf * p.n16 + n] = p.block_decay[(block * d.H + h) * d.NB + n];
    } else if (threadIdx.x < kChunk) {
      sDt[buf * kChunk + threadIdx.x] = p.dt ? p.dt[(q0 + t0 + threadIdx.x) * d.H + h] : 1.f;
      if (MEMORY) sLd[buf * kChunk + threadIdx.x] = p.ldec[(q0 + t0 + threadIdx.x) * d.H + h];
    }
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
    if (norm)
      for (int n = threadIdx.x; n < d.N; n += 128)
        p.seg_n[slot_of(0) * d.N + n] = start > 0 ? p.nstate[(static_cast<long long>(p.slots[seq]) * d.H + h) * d.N + n] : 0.f;
  }
  float sum = 0.f, nacc[2] = {0.f, 0.f}, ndec[2] = {1.f, 1.f};       // CHANNEL: ndec, the decays of this thread's rows
  for (int k = 0; k < p.seg_chunks; ++k) {
    const int buf = k & 1;
    ms_wait<0>();
    __syncthreads();
    if (k + 1 < p.seg_chunks) load_chunk(c0 + k + 1, buf ^ 1);
    float total = 0.f;
    if (!CHANNEL) total = ssd_decays(sDt + buf * kChunk, MEMORY ? sLd + buf * kChunk : nullptr, a2, cum, wgt, lane);
    sum += total;
    ssd_update<NI, SPLIT, CHANNEL>(S, exp2f(total), sLd + buf * p.n16, wgt, ms_addr(sB + buf * tile_n), ms_addr(sBl + buf * tile_n),
                                   ms_addr(sX + buf * tile_x), ldn, p.n16, warp, lane);
    if (norm) ssd_norm_add(nacc, exp2f(total), wgt, sB + buf * tile_n, ldn, d.N);
    if (CHANNEL)
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (static_cast<int>(threadIdx.x) + 128 * i < d.N) ndec[i] *= sLd[buf * p.n16 + threadIdx.x + 128 * i];
  }
  float* dst = p.seg_state + slot_of(seg + 1) * mat + p0;
  ssd_each<NI>(S, d.N, pw, warp, lane, [&](float& v0, float& v1, int n, int c) {
    *reinterpret_cast<float2*>(dst + static_cast<long long>(n) * d.P4 + c) = make_float2(v0, v1);
  });
  if (CHANNEL && p0 == 0) {
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (static_cast<int>(threadIdx.x) + 128 * i < d.N) p.seg_decay[slot_of(seg) * d.N + threadIdx.x + 128 * i] = ndec[i];
  } else if (threadIdx.x == 0 && p0 == 0) {
    p.seg_decay[slot_of(seg)] = exp2f(sum);
  }
  if (norm)
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (static_cast<int>(threadIdx.x) + 128 * i < d.N) p.seg_n[slot_of(seg + 1) * d.N + threadIdx.x + 128 * i] = nacc[i];
}

// NI: state row tiles (16 rows) per warp; 4 warps cover N <= 64 NI. Same grid as ssd_segment_kernel. The next block's C, scores and x are
// copied while the state is updated, its B (which the scores need unless they come from the caller) behind that.
template <int NI, bool SPLIT, int KIND, int WG>
__global__ void __launch_bounds__(128 * WG) ssd_chunk_kernel(const SsdParams p) {
  constexpr int NT = 128 * WG;
  constexpr bool MEMORY = KIND == kSsdMemory, CHANNEL = KIND == kSsdChannel;
  extern __shared__ __align__(16) uint8_t ssd_smem[];
  const SsdParams& d = p;
  const int slices = gridDim.x / p.n_seg, grp = threadIdx.x >> 7, gt = threadIdx.x & 127;
  const int seq = blockIdx.z, h = blockIdx.y, p0 = (blockIdx.x % slices * WG + grp) * kSlice, seg = blockIdx.x / slices;
  const int len = p.q_lens[seq];
  const int n_chunks = (len + kChunk - 1) / kChunk, ch0 = seg * p.seg_chunks, ch1 = min(n_chunks, ch0 + p.seg_chunks);
  if (ch0 >= ch1) return;
  const int warp = gt >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, t4 = lane & 3;
  const int ldn = p.n16 + 8, tile_n = kChunk * ldn, tile_x = kChunk * kLdX;
  __nv_bfloat16* sC = reinterpret_cast<__nv_bfloat16*>(ssd_smem);        // [64][ldn]
  __nv_bfloat16* sB = sC + tile_n;                                       // [64][ldn]
  __nv_bfloat16* sCl = sB + tile_n;                                      // [64][ldn] (SPLIT)
  __nv_bfloat16* sBl = sCl + tile_n;                                     // [64][ldn] (SPLIT)
  const int own = 2 * tile_x + 2 * p.n16 * kLdX;                         // what a group keeps by itself
  __nv_bfloat16* sX = sB + (SPLIT ? 3 : 1) * tile_n + grp * own;         // [2][64][kLdX]
  __nv_bfloat16* sSh = sX + 2 * tile_x;                                  // [n16][kLdX]
  __nv_bfloat16* sSl = sSh + p.n16 * kLdX;                               // [n16][kLdX]
  __nv_bfloat16* sA = sB + (SPLIT ? 3 : 1) * tile_n + WG * own;          // [2][64][kLdA] (CHANNEL)
  float* sDt = reinterpret_cast<float*>(sA + (CHANNEL ? 2 * kChunk * kLdA : 0));      // [64]
  float* cum = sDt + kChunk + (threadIdx.x >> 5) * kChunk;               // [4 WG warps][64]
  float* wgt = cum + 4 * WG * kChunk;                                    // [4 WG warps][64]
  float* sLd = sDt + (1 + 8 * WG) * kChunk;                              // [64] (MEMORY) or the block's decays [n16] (CHANNEL)
  float* sN = sLd + kChunk;                                              // [n16] (MEMORY)

  const long long q0 = p.q_start[seq];
  const int start = p.seq_lens[seq] - len;
  const int g = h / (d.H / d.G);
  const int cx = h * d.P + p0, cb = d.b0 + g * d.NB, cc = d.c0 + g * d.NB;
  const int pw = max(0, min(kSlice, d.P - p0));
  const float a2 = KIND == kSsdPlain ? ssd_rate(p, h) : 0.f, skip = p.dskip ? p.dskip[h] : 0.f;
  const bool norm = MEMORY && p0 == 0;                                   // this CTA keeps the head's normaliser
  const long long mat = static_cast<long long>(d.N) * d.P4;
  float* st = p.state + (static_cast<long long>(p.slots[seq]) * d.H + h) * mat + p0;

  auto load_c = [&](int ch) {               // C, scores, x (the buffer of the block's parity), steps and decays of the tokens
    const int t0 = ch * kChunk;
    ssd_load_rows<NT>(threadIdx.x, p.act, p.ld, p.aligned, sC, ldn, p.n16, d.N, cc, q0, t0, len);
    if (SPLIT) ssd_load_rows<NT>(threadIdx.x, p.act, p.ld, p.aligned, sCl, ldn, p.n16, d.N, cc + d.lo, q0, t0, len);
    ssd_load_rows<128>(gt, p.x, p.ldx, p.aligned_x, sX + (ch & 1) * tile_x, kLdX, kSlice, pw, cx, q0, t0, len);
    if (CHANNEL) {
      ssd_load_rows<NT>(threadIdx.x, p.score, 2ll * kChunk * d.H, true, sA, kLdA, kChunk, kChunk, h * 2 * kChunk, q0, t0, len);
      ssd_load_rows<NT>(threadIdx.x, p.score, 2ll * kChunk * d.H, true, sA + kChunk * kLdA, kLdA, kChunk, kChunk, (h * 2 + 1) * kChunk, q0,
                        t0, len);
    } else if (threadIdx.x < kChunk) {
      const bool ok = t0 + static_cast<int>(threadIdx.x) < len;
      sDt[threadIdx.x] = ok ? (p.dt ? p.dt[(q0 + t0 + threadIdx.x) * d.H + h] : 1.f) : 0.f;
      if (MEMORY) sLd[threadIdx.x] = ok ? p.ldec[(q0 + t0 + threadIdx.x) * d.H + h] : 0.f;
    }
    ms_commit();
  };
  auto load_b = [&](int ch) {
    const int t0 = ch * kChunk;
    ssd_load_rows<NT>(threadIdx.x, p.act, p.ld, p.aligned, sB, ldn, p.n16, d.N, cb, q0, t0, len);
    if (SPLIT) ssd_load_rows<NT>(threadIdx.x, p.act, p.ld, p.aligned, sBl, ldn, p.n16, d.N, cb + d.lo, q0, t0, len);
    if (CHANNEL) {
      const long long block = p.c_start[seq] / kChunk + seq + ch;
      for (int n = threadIdx.x; n < p.n16; n += NT) sLd[n] = p.block_decay[(block * d.H + h) * d.NB + n];
    }
    ms_commit();
  };
  load_c(ch0);
  load_b(ch0);

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
    if (norm)
      for (int n = threadIdx.x; n < p.n16; n += 128)
        sN[n] = start > 0 && n < d.N ? p.nstate[(static_cast<long long>(p.slots[seq]) * d.H + h) * d.N + n] : 0.f;
  } else {
    float nv[2] = {0.f, 0.f};
    for (int k = 0; k <= seg; ++k) {
      const long long o = (static_cast<long long>(seq) * p.n_seg + k) * d.H + h;
      const float* src = p.seg_state + o * mat + p0;
      const float keep = k > 0 && !CHANNEL ? p.seg_decay[o - d.H] : 0.f;
      const float* keeps = p.seg_decay + (o - d.H) * d.N;              // CHANNEL, k > 0
      ssd_each<NI>(S, d.N, pw, warp, lane, [&](float& v0, float& v1, int n, int c) {
        const float2 v = *reinterpret_cast<const float2*>(src + static_cast<long long>(n) * d.P4 + c);
        const float f = CHANNEL ? (k > 0 ? keeps[n] : 0.f) : keep;
        v0 = fmaf(f, v0, v.x);
        v1 = fmaf(f, v1, v.y);
      });
      if (norm)
#pragma unroll
        for (int i = 0; i < 2; ++i)
          if (static_cast<int>(threadIdx.x) + 128 * i < d.N) nv[i] = fmaf(keep, nv[i], p.seg_n[o * d.N + threadIdx.x + 128 * i]);
    }
    if (norm)
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (static_cast<int>(threadIdx.x) + 128 * i < p.n16) sN[threadIdx.x + 128 * i] = nv[i];
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
  const uint32_t aC = ms_addr(sC), aB = ms_addr(sB), aSh = ms_addr(sSh), aSl = ms_addr(sSl);
  const uint32_t aCl = ms_addr(sCl), aBl = ms_addr(sBl);
  const int r0 = warp * 16;

  for (int ch = ch0; ch < ch1; ++ch) {
    if (CHANNEL) ms_wait<1>();
    else ms_wait<0>();
    __syncthreads();                       // the block's rows (CHANNEL: without B) and the published state are visible
    const __nv_bfloat16* sXb = sX + (ch & 1) * tile_x;
    const uint32_t aX = ms_addr(sXb);
    float total = 0.f;
    if (!CHANNEL) total = ssd_decays(sDt, MEMORY ? sLd : nullptr, a2, cum, wgt, lane);
    float s[8][4], yi[4][4], y[4][4], rows[2] = {0.f, 0.f};
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
      uint32_t fa[4], fal[4];
      ms_ldsm4(ms_a_at(aC, ldn, r0, k, lane), fa);
      if (SPLIT) ms_ldsm4(ms_a_at(aCl, ldn, r0, k, lane), fal);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (!CHANNEL && np <= warp) {
          uint32_t fb[4];
          ms_ldsm4(ms_b_nt_at(aB, ldn, np * 16, k, lane), fb);
          ms_mma(s[2 * np], fa, fb[0], fb[1]);
          ms_mma(s[2 * np + 1], fa, fb[2], fb[3]);
          if (SPLIT) {
            ms_mma(s[2 * np], fal, fb[0], fb[1]);
            ms_mma(s[2 * np + 1], fal, fb[2], fb[3]);
            ms_ldsm4(ms_b_nt_at(aBl, ldn, np * 16, k, lane), fb);
            ms_mma(s[2 * np], fa, fb[0], fb[1]);
            ms_mma(s[2 * np + 1], fa, fb[2], fb[3]);
          }
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
        if (SPLIT) {
          ms_mma(yi[2 * np], fal, fh[0], fh[1]);
          ms_mma(yi[2 * np + 1], fal, fh[2], fh[3]);
        }
      }
    }
    float ci[2] = {0.f, 0.f};
    if (!CHANNEL) {
      ci[0] = cum[r0 + g4];
      ci[1] = cum[r0 + g4 + 8];
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk > warp) break;
      uint32_t fh[4], fl[4];
      if (CHANNEL) {
        ms_ldsm4(ms_a_at(ms_addr(sA), kLdA, r0, kk * 16, lane), fh);
        ms_ldsm4(ms_a_at(ms_addr(sA + kChunk * kLdA), kLdA, r0, kk * 16, lane), fl);
      }
      float m[2][4];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        if (CHANNEL) break;
        const int j0 = kk * 16 + q * 8 + 2 * t4;
        const float2 cj = *reinterpret_cast<const float2*>(cum + j0), dj = *reinterpret_cast<const float2*>(sDt + j0);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const bool seen = kk < warp || j0 + (e & 1) <= r0 + g4 + ((e & 2) ? 8 : 0);
          m[q][e] = seen ? s[2 * kk + q][e] * exp2f(ci[e >> 1] - ((e & 1) ? cj.y : cj.x)) * ((e & 1) ? dj.y : dj.x) : 0.f;
          if (MEMORY) rows[e >> 1] += m[q][e];
        }
      }
      if (!CHANNEL) {
        ms_split(m[0][0], m[0][1], fh[0], fl[0]);
        ms_split(m[0][2], m[0][3], fh[1], fl[1]);
        ms_split(m[1][0], m[1][1], fh[2], fl[2]);
        ms_split(m[1][2], m[1][3], fh[3], fl[3]);
      }
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
    if (norm) {                            // n . c of the rows: the block's part from the scores, the rest from the normaliser at its start
      float at_start = 0.f;
      const int per = p.n16 / 2, from = (lane >> 4) * per;
      for (int k = from; k < from + per; k += 8) {
        float v[8];
        load_vec<8>(sC + (r0 + (lane & 15)) * ldn + k, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) at_start = fmaf(v[e], sN[k + e], at_start);
      }
      at_start += __shfl_xor_sync(0xffffffffu, at_start, 16);
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        rows[hf] += __shfl_xor_sync(0xffffffffu, rows[hf], 1);
        rows[hf] += __shfl_xor_sync(0xffffffffu, rows[hf], 2);
        const float nq = fmaf(ei[hf], __shfl_sync(0xffffffffu, at_start, g4 + 8 * hf), rows[hf]) * p.yscale;
        const int i = r0 + g4 + 8 * hf;
        if (t4 == 0 && t0 + i < len) {
          const long long at = (q0 + t0 + i) * d.H + h;
          p.den[at] = fmaxf(fabsf(nq), expf(-p.mrun[at])) + p.den_eps;
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = r0 + g4 + 8 * hf, c = nt * 8 + 2 * t4;
        if (t0 + i >= len || c >= pw) continue;
        const float2 xf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sXb + i * kLdX + c));
        float v0 = fmaf(skip, xf.x, fmaf(ei[hf], yi[nt][2 * hf], y[nt][2 * hf]));
        float v1 = fmaf(skip, xf.y, fmaf(ei[hf], yi[nt][2 * hf + 1], y[nt][2 * hf + 1]));
        if (MEMORY) {
          v0 *= p.yscale;
          v1 *= p.yscale;
        }
        __nv_bfloat16* dst = p.y + (q0 + t0 + i) * (d.H * d.P) + cx + c;
        if (d.P % 2 == 0) {
          *reinterpret_cast<uint32_t*>(dst) = pack_bf16(v0, v1);
        } else {
          dst[0] = __float2bfloat16(v0);
          if (c + 1 < pw) dst[1] = __float2bfloat16(v1);
        }
      }
    if (CHANNEL) ms_wait<0>();
    __syncthreads();                       // C, scores and steps have been read; CHANNEL: B is visible
    if (ch + 1 < ch1) load_c(ch + 1);
    float nv[2] = {0.f, 0.f};
    if (ch + 1 < ch1 || ch1 == n_chunks) {
      ssd_update<NI, SPLIT, CHANNEL>(S, exp2f(total), sLd, wgt, aB, aBl, aX, ldn, p.n16, warp, lane);
      if (norm) {
#pragma unroll
        for (int i = 0; i < 2; ++i)
          if (static_cast<int>(threadIdx.x) + 128 * i < d.N) nv[i] = sN[threadIdx.x + 128 * i];
        ssd_norm_add(nv, exp2f(total), wgt, sB, ldn, d.N);
      }
    }
    __syncthreads();                       // everyone has read B and the published state
    if (norm && (ch + 1 < ch1 || ch1 == n_chunks))
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (static_cast<int>(threadIdx.x) + 128 * i < d.N) sN[threadIdx.x + 128 * i] = nv[i];
    if (ch + 1 < ch1) {
      load_b(ch + 1);
      publish();
    }
  }
  if (ch1 == n_chunks) {
    ssd_each<NI>(S, d.N, pw, warp, lane, [&](float& v0, float& v1, int n, int c) {
      *reinterpret_cast<float2*>(st + static_cast<long long>(n) * d.P4 + c) = make_float2(v0, v1);
    });
    if (norm)                              // every thread reads what it wrote
      for (int n = threadIdx.x; n < d.N; n += 128) p.nstate[(static_cast<long long>(p.slots[seq]) * d.H + h) * d.N + n] = sN[n];
  }
}

static size_t ssd_bytes(const SsdParams& p, bool split, int kind, int wg) {
  const size_t tile_n = static_cast<size_t>(kChunk) * (p.n16 + 8), tile_x = static_cast<size_t>(kChunk) * kLdX;
  const size_t scores = kind == kSsdChannel ? 2 * static_cast<size_t>(kChunk) * kLdA : 0;
  const size_t more = kind == kSsdPlain ? 0 : (kind == kSsdMemory ? kChunk + p.n16 : p.n16);
  return ((split ? 4 : 2) * tile_n + wg * (2 * tile_x + 2 * static_cast<size_t>(p.n16) * kLdX) + scores) * 2 + ((1 + 8 * wg) * kChunk + more) * 4;
}
static size_t ssd_bytes_segment(const SsdParams& p, bool split, int kind, int wg) {
  const size_t tile_n = static_cast<size_t>(kChunk) * (p.n16 + 8), tile_x = static_cast<size_t>(kChunk) * kLdX;
  const size_t more = kind == kSsdPlain ? 0 : 2 * (kind == kSsdMemory ? kChunk : p.n16);
  return ((split ? 4 : 2) * tile_n + wg * 2 * tile_x) * 2 + ((2 + 8 * wg) * kChunk + more) * 4;
}
constexpr size_t kSsdSmem = 224 * 1024;

template <int NI, bool SPLIT, int KIND, int WG>
static int ssd_launch_as(const SsdParams& p, dim3 grid, cudaStream_t st) {
  const size_t smem = ssd_bytes(p, SPLIT, KIND, WG), smem_seg = ssd_bytes_segment(p, SPLIT, KIND, WG);
  if (smem > kSsdSmem || smem_seg > kSsdSmem) return -4;
  static DeviceOnce once;
  if (once.pending()) {
    cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<NI, SPLIT, KIND, WG>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSsdSmem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(ssd_segment_kernel<NI, SPLIT, KIND, WG>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSsdSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    once.mark();
  }
  if (p.n_seg > 1) {
    ssd_segment_kernel<NI, SPLIT, KIND, WG><<<grid, 128 * WG, smem_seg, st>>>(p);
    const cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  ssd_chunk_kernel<NI, SPLIT, KIND, WG><<<grid, 128 * WG, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <bool SPLIT, int KIND>
static int ssd_launch_any(SsdParams p, int n_seq, int n_chunks, int max_seg, cudaStream_t st) {
  // groups of warps on the same B and C: as many as there are slices, while registers and shared memory last
  const int slices = (p.P + kSlice - 1) / kSlice;
  int wg = 1;
  if (KIND != kSsdPlain) {
    wg = slices >= 3 ? 4 : slices;
    if (p.n16 > 128 && wg > 2) wg = 2;
    while (wg > 1 && ssd_bytes(p, SPLIT, KIND, wg) > kSsdSmem) wg /= 2;
  }
  // enough CTAs to keep three single groups on every SM for a few rounds, or one of several for a round
  const int ctas = (slices + wg - 1) / wg;
  const long long base = static_cast<long long>(ctas) * p.H * n_seq, rounds = wg == 1 ? 6 : (wg == 2 ? 2 : 1);
  long long want = wg == 1 ? (rounds * num_sms() + base - 1) / base : rounds * num_sms() / base;
  if (want < 1) want = 1;
  if (want > max_seg) want = max_seg;
  if (want > n_chunks) want = n_chunks;
  p.seg_chunks = (n_chunks + static_cast<int>(want) - 1) / static_cast<int>(want);
  p.n_seg = (n_chunks + p.seg_chunks - 1) / p.seg_chunks;
  const dim3 grid(ctas * p.n_seg, p.H, n_seq);
  if constexpr (KIND != kSsdPlain) {
    if (wg == 4)
      return p.n16 <= 64 ? ssd_launch_as<1, SPLIT, KIND, 4>(p, grid, st) : ssd_launch_as<2, SPLIT, KIND, 4>(p, grid, st);
    if (wg == 2)
      return p.n16 <= 64 ? ssd_launch_as<1, SPLIT, KIND, 2>(p, grid, st)
                         : (p.n16 <= 128 ? ssd_launch_as<2, SPLIT, KIND, 2>(p, grid, st) : ssd_launch_as<4, SPLIT, KIND, 2>(p, grid, st));
  }
  return p.n16 <= 64 ? ssd_launch_as<1, SPLIT, KIND, 1>(p, grid, st)
                     : (p.n16 <= 128 ? ssd_launch_as<2, SPLIT, KIND, 1>(p, grid, st) : ssd_launch_as<4, SPLIT, KIND, 1>(p, grid, st));
}

int ssd_chunk_launch(SsdParams p, int n_seq, int max_q, int max_seg, cudaStream_t st) {
  if (p.N < 1 || p.N > kSsdMaxState || max_seg < 1) return -1;
  if (n_seq < 1 || max_q < 1) return 0;
  p.n16 = (p.N + 15) / 16 * 16;
  if (!p.x) {
    p.x = p.act;
    p.ldx = p.ld;
  }
  if (!p.NB) p.NB = p.N;
  const auto whole = [](const void* a) { return reinterpret_cast<uintptr_t>(a) % 16 == 0; };
  p.aligned = p.ld % 8 == 0 && p.b0 % 8 == 0 && p.c0 % 8 == 0 && p.lo % 8 == 0 && p.N % 8 == 0 && p.NB % 8 == 0 && whole(p.act);
  p.aligned_x = p.ldx % 8 == 0 && p.P % 8 == 0 && whole(p.x);
  const int n_chunks = (max_q + kChunk - 1) / kChunk;
  if (p.kind == kSsdMemory) return ssd_launch_any<false, kSsdMemory>(p, n_seq, n_chunks, max_seg, st);
  if (p.kind == kSsdChannel) return ssd_launch_any<true, kSsdChannel>(p, n_seq, n_chunks, max_seg, st);
  return p.lo > 0 ? ssd_launch_any<true, kSsdPlain>(p, n_seq, n_chunks, max_seg, st)
                  : ssd_launch_any<false, kSsdPlain>(p, n_seq, n_chunks, max_seg, st);
}

}  // namespace pm
