// Linear attention whose decays come from the tokens. Per sequence and head, S [N, P] in fp32 and starting from zeros:
//
//   channel gates (HGRN2)   f = l + (1 - l) sigmoid(z + b) per channel of N;   S <- diag(f) S + (1 - f) v^T,   y = S^T silu(q)
//   matrix memory (mLSTM)   i = cap tanh((z_i + b_i) / cap), f = log sigmoid(cap tanh((z_f + b_f) / cap)) per head;
//                           m' = max(f + m, i) with m = 0 at the start;  S <- exp(f + m - m') S + exp(i - m') k v^T, n the same
//                           with k alone;  y = S^T q c, den = max(|n . q c|, exp(-m')) + eps, the result is y / den
//
// q, k and v are columns of a projection row (bf16 or fp32), the gates' logits z fp32 columns of their own. S lives in slots as
// [slot][H][N][P4] (P4 = P rounded up to 4), n as [slot][H][N], m as [slot][H][P4 / 4] (the same number for every four channels:
// CTAs that share a head by channels read and write their own). A sequence whose first token of the step is position 0 starts from
// zeros whatever the slot holds.
//
//   gated_scan_kernel    any number of tokens one after the other, one CTA per (sequence, head, slice of P), S in registers.
//                        Decode, short portions, fp32 models.
//   memory_gates_kernel  decays exp(f + m - m'), weights exp(i - m') and m' of all tokens of longer portions, by a scan over
//                        (sum of f, largest i + later f): in these the recurrence is linear and runs in the blocks of ssd_chunk.cu
//   channel_block_kernel the same for channel gates, one CTA per (block of 64 tokens, head): running sums c of log2 f, q 2^c and
//                        (1 - f) 2^(c_63 - c) as sums of two bf16 terms, and the scores sum_n q_i 2^(c_i - c_j) (1 - f_j) of the
//                        block on the tensor cores. Keys are taken relative to the middle of their eight tokens, queries relative
//                        to that of the keys they meet, so that no factor of a causal pair overflows; a step's decay is held at
//                        2^-24 or more, below which nothing is left of the old state in fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math_constants.h>
#include <stdint.h>
#include "elem.cuh"
#include "host_util.cuh"
#include "mma_sync.cuh"
#include "pmetal_b200.h"
#include "ssd_chunk.cuh"

namespace pm {

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kMinLog2 = -24.f;

// f and 1 - f, each without cancellation.
__device__ __forceinline__ void channel_gate(float z, float lower, float& f, float& g) {
  const float e = expf(-fabsf(z)), big = 1.f / (1.f + e), small = e * big;
  f = fmaf(1.f - lower, z >= 0.f ? big : small, lower);
  g = (1.f - lower) * (z >= 0.f ? small : big);
}

__device__ __forceinline__ float log2_gate(float f, float g) {
  return fmaxf(f < 0.5f ? log2f(f) : log1pf(-g) * kLog2e, kMinLog2);
}

__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

template <typename T>
struct GatedScanParams {
  const T* q;              // head 0 of row 0; rows ldu apart
  const T* k;              // matrix memory
  const T* v;
  long long ldu;
  const float* z;          // [tokens, ldz]: H N channel gates, or H input gates and H forget gates
  long long ldz;
  const float* bias;       // [H N] or [2 H]
  const float* lower;      // [H N], channel gates
  float cap, qscale, den_eps;      // matrix memory
  float* state;
  float* nstate;
  float* mstate;
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  T* y;                    // [tokens, H P]
  float* den;              // [tokens, H]
  int H, N, P, P4;
  int pw;                  // channels of P per CTA (multiple of 4)
};

constexpr int kScanThreads = 256;

// E: state rows per thread (float4 each).
template <typename T, int E, bool MEMORY>
__global__ void __launch_bounds__(kScanThreads, E <= 4 ? 4 : (E <= 8 ? 3 : 2)) gated_scan_kernel(const GatedScanParams<T> p) {
  extern __shared__ __align__(16) float gs_smem[];
  const int seq = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * p.pw;
  const int len = p.q_lens[seq];
  if (len <= 0) return;
  const int cols = p.pw / 4, groups = kScanThreads / cols;
  float* sv = gs_smem;                       // [pw]
  float* sk = sv + p.pw;                     // [N] keys, or 1 - f
  float* sq = sk + p.N;                      // [N]
  float* sx = sq + p.N;                      // [N] f, or the normaliser
  float* part = sv + (p.pw + 3 * p.N + 3) / 4 * 4;     // [groups][pw]
  const int q0 = p.q_start[seq], start = p.seq_lens[seq] - len;
  const long long slot = p.slots[seq];
  const int col = threadIdx.x % cols, grp = threadIdx.x / cols;
  const bool owner = grp < groups && p0 + col * 4 < p.P4, norm = MEMORY && p0 == 0;
  float4 S[E];
  float* st = p.state + ((slot * p.H + h) * p.N) * p.P4 + p0 + col * 4;
  float* ms = p.mstate + (slot * p.H + h) * (p.P4 / 4) + p0 / 4;
  float* ns = p.nstate + (slot * p.H + h) * p.N;
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const int n = grp + i * groups;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (owner && start > 0 && n < p.N) S[i] = *reinterpret_cast<const float4*>(st + static_cast<long long>(n) * p.P4);
  }
  float m = 0.f;
  if (MEMORY && start > 0) m = ms[0];
  if (norm)
    for (int n = threadIdx.x; n < p.N; n += kScanThreads) sx[n] = start > 0 ? ns[n] : 0.f;
  for (int t = 0; t < len; ++t) {
    const long long r = q0 + t, u = r * p.ldu;
    float keep = 1.f, put_ = 1.f;
    if (MEMORY) {
      const float* z = p.z + r * p.ldz;
      const float ig = soft_cap(z[h] + p.bias[h], p.cap);
      const float fg = log_sigmoid(soft_cap(z[p.H + h] + p.bias[p.H + h], p.cap));
      const float next = fmaxf(fg + m, ig);
      keep = expf(fg + m - next);
      put_ = expf(ig - next);
      m = next;
    }
    __syncthreads();                          // the previous token's readers are done; first token: m has been read
    for (int i = threadIdx.x; i < p.pw + 2 * p.N; i += kScanThreads) {
      if (i < p.pw) {
        sv[i] = p0 + i < p.P ? to_f(p.v[u + h * p.P + p0 + i]) : 0.f;
      } else if (i < p.pw + p.N) {
        const int n = i - p.pw, c = h * p.N + n;
        if (MEMORY) sk[n] = to_f(p.k[u + c]) * put_;
        else channel_gate(p.z[r * p.ldz + c] + p.bias[c], p.lower[c], sx[n], sk[n]);
      } else {
        const int n = i - p.pw - p.N;
        const float v = to_f(p.q[u + h * p.N + n]);
        sq[n] = MEMORY ? v * p.qscale : silu_f(v);
      }
    }
    __syncthreads();
    if (owner) {
      const float4 x = *reinterpret_cast<const float4*>(sv + col * 4);
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < E; ++i) {
        const int n = grp + i * groups;
        if (n < p.N) {
          const float f = MEMORY ? keep : sx[n], b = sk[n], c = sq[n];
          S[i].x = fmaf(f, S[i].x, b * x.x); y.x = fmaf(c, S[i].x, y.x);
          S[i].y = fmaf(f, S[i].y, b * x.y); y.y = fmaf(c, S[i].y, y.y);
          S[i].z = fmaf(f, S[i].z, b * x.z); y.z = fmaf(c, S[i].z, y.z);
          S[i].w = fmaf(f, S[i].w, b * x.w); y.w = fmaf(c, S[i].w, y.w);
        }
      }
      *reinterpret_cast<float4*>(part + grp * p.pw + col * 4) = y;
    }
    if (norm) {
      float nq = 0.f;
      for (int n = threadIdx.x; n < p.N; n += kScanThreads) {
        sx[n] = fmaf(keep, sx[n], sk[n]);
        nq = fmaf(sx[n], sq[n], nq);
      }
      nq = block_sum(nq);
      if (threadIdx.x == 0) p.den[r * p.H + h] = fmaxf(fabsf(nq), expf(-m)) + p.den_eps;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.pw; i += kScanThreads) {
      if (p0 + i >= p.P) continue;
      float v = 0.f;
      for (int k = 0; k < groups; ++k) v += part[k * p.pw + i];
      put(p.y + r * (p.H * p.P) + h * p.P + p0 + i, v);
    }
  }
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const int n = grp + i * groups;
    if (owner && n < p.N) *reinterpret_cast<float4*>(st + static_cast<long long>(n) * p.P4) = S[i];
  }
  if (MEMORY)
    for (int i = threadIdx.x; i < cols; i += kScanThreads)
      if (p0 / 4 + i < p.P4 / 4) ms[i] = m;
  if (norm)
    for (int n = threadIdx.x; n < p.N; n += kScanThreads) ns[n] = sx[n];
}

// ------------------------------------------------------------------------------------------- longer portions (bf16)
struct MemoryGateParams {
  const float* z;
  long long ldz;
  const float* bias;
  float cap;
  float* mstate;
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  float* ldec;             // [tokens, H] log2 of the decay
  float* weight;           // [tokens, H]
  float* mrun;             // [tokens, H]
  int H, P4;
};

constexpr int kGateThreads = 256, kGateTokens = 16;

// One CTA per (head, sequence), 16 consecutive tokens per thread.
__global__ void __launch_bounds__(kGateThreads) memory_gates_kernel(const MemoryGateParams p) {
  __shared__ float wsum[8], wmax[8], carry;
  const int h = blockIdx.x, seq = blockIdx.y, len = p.q_lens[seq], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (len <= 0) return;
  const long long q0 = p.q_start[seq];
  float* ms = p.mstate + (static_cast<long long>(p.slots[seq]) * p.H + h) * (p.P4 / 4);
  float m0 = p.seq_lens[seq] > len ? ms[0] : 0.f;
  const float bi = p.bias[h], bf = p.bias[p.H + h];
  for (int base = 0; base < len; base += kGateThreads * kGateTokens) {
    const int t0 = base + threadIdx.x * kGateTokens;
    float ig[kGateTokens], fg[kGateTokens];
#pragma unroll
    for (int e = 0; e < kGateTokens; ++e) {
      const bool ok = t0 + e < len;
      const float* z = p.z + (q0 + (ok ? t0 + e : 0)) * p.ldz;
      ig[e] = ok ? z[h] : 0.f;
      fg[e] = ok ? z[p.H + h] : 0.f;
    }
    float sum = 0.f, top = -CUDART_INF_F;      // m behind the tokens is max(sum + m before them, top)
#pragma unroll
    for (int e = 0; e < kGateTokens; ++e) {
      const bool ok = t0 + e < len;
      ig[e] = ok ? soft_cap(ig[e] + bi, p.cap) : -CUDART_INF_F;
      fg[e] = ok ? log_sigmoid(soft_cap(fg[e] + bf, p.cap)) : 0.f;
      top = fmaxf(top + fg[e], ig[e]);
      sum += fg[e];
    }
    float is = sum, it = top;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float us = __shfl_up_sync(0xffffffffu, is, o), ut = __shfl_up_sync(0xffffffffu, it, o);
      if (lane >= o) {
        it = fmaxf(ut + is, it);
        is += us;
      }
    }
    if (lane == 31) {
      wsum[warp] = is;
      wmax[warp] = it;
    }
    __syncthreads();
    float m = m0;
    for (int w = 0; w < warp; ++w) m = fmaxf(wsum[w] + m, wmax[w]);
    const float ps = __shfl_up_sync(0xffffffffu, is, 1), pt = __shfl_up_sync(0xffffffffu, it, 1);
    if (lane > 0) m = fmaxf(ps + m, pt);
#pragma unroll
    for (int e = 0; e < kGateTokens; ++e) {
      if (t0 + e >= len) break;
      const float next = fmaxf(fg[e] + m, ig[e]);
      const long long at = (q0 + t0 + e) * p.H + h;
      p.ldec[at] = (fg[e] + m - next) * kLog2e;
      p.weight[at] = expf(ig[e] - next);
      p.mrun[at] = next;
      m = next;
    }
    if (threadIdx.x == kGateThreads - 1) carry = m;
    __syncthreads();
    m0 = carry;
  }
  // threads behind the last token carried m through unchanged
  for (int i = threadIdx.x; i < p.P4 / 4; i += kGateThreads) ms[i] = m0;
}

struct ChannelBlockParams {
  const __nv_bfloat16* q;
  long long ldu;
  const float* z;
  long long ldz;
  const float* bias;
  const float* lower;
  const int* q_start;
  const int* q_lens;
  const int* c_start;
  __nv_bfloat16* act;      // [tokens, 4 H n16]: C, its second terms, B, its second terms
  __nv_bfloat16* score;    // [tokens, H, 128]
  float* block_decay;      // [block][H][n16]
  int H, N, n16;
};

constexpr int kBlockTokens = 64, kBlockThreads = 256, kBlockCols = 128;

// 2^x, small results flushed to zero
__device__ __forceinline__ float pow2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// channel_gate through the fast exponential and division, for sums of bf16 terms, and log2 f (no less than kMinLog2): close to one by
// the series of log(1 - g).
__device__ __forceinline__ float channel_gate_fast(float z, float lower, float& g) {
  const float e = __expf(-fabsf(z)), big = __fdividef(1.f, 1.f + e), small = e * big;
  const float f = fmaf(1.f - lower, z >= 0.f ? big : small, lower);
  g = (1.f - lower) * (z >= 0.f ? small : big);
  const float near = -g * kLog2e * fmaf(g, fmaf(g, fmaf(g, fmaf(g, fmaf(g, 1.f / 6.f, 0.2f), 0.25f), 1.f / 3.f), 0.5f), 1.f);
  return fmaxf(g < 0.0625f ? near : __log2f(f), kMinLog2);
}

// Four consecutive elements from element n of a row; those from `end` on are zero.
template <bool VEC, typename T>
__device__ __forceinline__ void load_four(const T* row, int n, int end, float (&v)[4]) {
  if (VEC) {
    load_vec<4>(row + n, v);
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = n + e < end ? to_f(row[n + e]) : 0.f;
  }
}

// grid (blocks of the longest portion, H, sequences). A warp forms the operands of 8 tokens, 4 channels per lane and pass. VEC: heads
// are whole 16-byte pieces of all rows.
template <bool VEC>
__global__ void __launch_bounds__(kBlockThreads) channel_block_kernel(const ChannelBlockParams p) {
  extern __shared__ __align__(16) uint8_t cb_smem[];
  const int seq = blockIdx.z, h = blockIdx.y, t0 = blockIdx.x * kBlockTokens, len = p.q_lens[seq] - t0;
  if (len <= 0) return;
  const int n16 = p.n16, ldc = n16 + 8, ldq = n16 + 8, ldk = 4 * n16 + 16;              // ldk: bytes
  float* sc = reinterpret_cast<float*>(cb_smem);                                        // [64][ldc] running sums of log2 f
  float* sT = sc + kBlockTokens * ldc;                                                  // [8][128] their growth over 8 tokens
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(sT + 8 * kBlockCols);            // [64][ldq]
  uint8_t* sK = reinterpret_cast<uint8_t*>(sQ + kBlockTokens * ldq);                    // [64][ldk]: keys, their second terms
  const long long row0 = p.q_start[seq] + t0;
  const int col0 = h * p.N, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, HN = p.H * n16;
  for (int n0 = 0; n0 < n16; n0 += kBlockCols) {
    const int n = n0 + lane * 4;
    const bool live = n < p.N;
    float bias[4] = {}, lower[4] = {}, c[8][4], g[8][4], run[4] = {};
    if (live) {
      load_four<VEC>(p.bias + col0, n, p.N, bias);
      load_four<VEC>(p.lower + col0, n, p.N, lower);
    }
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const int j = warp * 8 + r;
      float z[4];
      const bool ok = live && j < len;
      if (ok) load_four<VEC>(p.z + (row0 + j) * p.ldz + col0, n, p.N, z);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        g[r][e] = 0.f;
        if (ok && (VEC || n + e < p.N)) run[e] += channel_gate_fast(z[e] + bias[e], lower[e], g[r][e]);
        c[r][e] = run[e];
      }
    }
    *reinterpret_cast<float4*>(sT + warp * kBlockCols + lane * 4) = make_float4(run[0], run[1], run[2], run[3]);
    __syncthreads();
    float before[4] = {}, total[4] = {};
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      const float4 t = *reinterpret_cast<const float4*>(sT + w * kBlockCols + lane * 4);
      const float v[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (w < warp) before[e] += v[e];
        total[e] += v[e];
      }
    }
    __syncthreads();                                         // sT may be written again
    if (n >= n16) continue;
    if (warp == 0) {
      const long long block = p.c_start[seq] / kBlockTokens + seq + blockIdx.x;
      *reinterpret_cast<float4*>(p.block_decay + (block * p.H + h) * n16 + n) = make_float4(pow2(total[0]), pow2(total[1]), pow2(total[2]), pow2(total[3]));
    }
    const float mid[4] = {c[3][0], c[3][1], c[3][2], c[3][3]};
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const int j = warp * 8 + r;
      float q[4] = {}, v[4];
      if (live && j < len) load_four<VEC>(p.q + (row0 + j) * p.ldu + col0, n, p.N, q);
#pragma unroll
      for (int e = 0; e < 4; ++e) q[e] = silu_fast(q[e]);
      const uint2 qb = make_uint2(pack_bf16(q[0], q[1]), pack_bf16(q[2], q[3]));
      q[0] = __uint_as_float(qb.x << 16); q[1] = __uint_as_float(qb.x & 0xffff0000u);
      q[2] = __uint_as_float(qb.y << 16); q[3] = __uint_as_float(qb.y & 0xffff0000u);
      uint2 hi, lo;
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = g[r][e] * pow2(mid[e] - c[r][e]);
      ms_split(v[0], v[1], hi.x, lo.x);
      ms_split(v[2], v[3], hi.y, lo.y);
      *reinterpret_cast<uint2*>(sQ + j * ldq + n) = qb;
      *reinterpret_cast<uint2*>(sK + j * ldk + n * 2) = hi;
      *reinterpret_cast<uint2*>(sK + j * ldk + (n16 + n) * 2) = lo;
#pragma unroll
      for (int e = 0; e < 4; ++e) c[r][e] += before[e];
      *reinterpret_cast<float4*>(sc + j * ldc + n) = make_float4(c[r][0], c[r][1], c[r][2], c[r][3]);
      if (j >= len) continue;
      __nv_bfloat16* dst = p.act + (row0 + j) * 4 * HN + h * n16 + n;
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = q[e] * pow2(c[r][e]);
      ms_split(v[0], v[1], hi.x, lo.x);
      ms_split(v[2], v[3], hi.y, lo.y);
      *reinterpret_cast<uint2*>(dst) = hi;
      *reinterpret_cast<uint2*>(dst + HN) = lo;
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = g[r][e] * pow2(total[e] - c[r][e]);
      ms_split(v[0], v[1], hi.x, lo.x);
      ms_split(v[2], v[3], hi.y, lo.y);
      *reinterpret_cast<uint2*>(dst + 2 * HN) = hi;
      *reinterpret_cast<uint2*>(dst + 3 * HN) = lo;
    }
  }
  __syncthreads();

  // scores: a warp owns 16 queries and every second tile of 8 keys
  const int g4 = lane >> 2, t4 = lane & 3, I = warp & 3, par = warp >> 2, r0 = I * 16;
  if (r0 >= len) return;
  const uint32_t aK = ms_addr(sK);
  float s[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
  for (int k0 = 0; k0 < n16; k0 += 16) {
    // elements 2 a and 2 a + 1: row r0 + g4 + 8 (a & 1), channels k0 + 2 t4 + 8 (a >> 1) and the next
    float q[8], c[8], ci[4], qd[8];
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      const int row = r0 + g4 + 8 * (a & 1), n = k0 + 2 * t4 + 8 * (a >> 1);
      const uint32_t qb = *reinterpret_cast<const uint32_t*>(sQ + row * ldq + n);
      q[2 * a] = __uint_as_float(qb << 16);
      q[2 * a + 1] = __uint_as_float(qb & 0xffff0000u);
      const float2 v = *reinterpret_cast<const float2*>(sc + row * ldc + n);
      c[2 * a] = v.x;
      c[2 * a + 1] = v.y;
    }
#pragma unroll
    for (int a = 0; a < 2; ++a) {
      float2 v = make_float2(0.f, 0.f);
      if (I > 0) v = *reinterpret_cast<const float2*>(sc + (r0 - 1) * ldc + k0 + 2 * t4 + 8 * a);
      ci[2 * a] = v.x;
      ci[2 * a + 1] = v.y;
    }
#pragma unroll
    for (int a = 0; a < 8; ++a) qd[a] = q[a] * pow2(c[a] - ci[(a >> 2) * 2 + (a & 1)]);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int J = 2 * i + par;
      if (i > I) break;
      float mid[4], v[8];
#pragma unroll
      for (int a = 0; a < 2; ++a) {
        const float2 m2 = *reinterpret_cast<const float2*>(sc + (8 * J + 3) * ldc + k0 + 2 * t4 + 8 * a);
        mid[2 * a] = m2.x;
        mid[2 * a + 1] = m2.y;
      }
      if (i < I) {
        float f[4];
#pragma unroll
        for (int a = 0; a < 4; ++a) f[a] = pow2(ci[a] - mid[a]);
#pragma unroll
        for (int a = 0; a < 8; ++a) v[a] = qd[a] * f[(a >> 2) * 2 + (a & 1)];
      } else {
#pragma unroll
        for (int a = 0; a < 8; ++a) v[a] = q[a] * pow2(c[a] - mid[(a >> 2) * 2 + (a & 1)]);
      }
      uint32_t fh[4], fl[4], kb[4];
#pragma unroll
      for (int a = 0; a < 4; ++a) ms_split(v[2 * a], v[2 * a + 1], fh[a], fl[a]);
      // lanes 0 - 15: the keys' halves of 16 channels, 16 - 31: those of the second terms
      ms_ldsm4(aK + static_cast<uint32_t>((8 * J + (lane & 7)) * ldk + (k0 + ((lane >> 3) & 1) * 8 + (lane >> 4) * n16) * 2), kb);
      ms_mma(s[i], fh, kb[0], kb[1]);
      ms_mma(s[i], fl, kb[0], kb[1]);
      ms_mma(s[i], fh, kb[2], kb[3]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (i > I) break;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int row = r0 + g4 + 8 * hf, j = (2 * i + par) * 8 + 2 * t4;
      if (row >= len) continue;
      uint32_t hi, lo;
      ms_split(j <= row ? s[i][2 * hf] : 0.f, j + 1 <= row ? s[i][2 * hf + 1] : 0.f, hi, lo);
      __nv_bfloat16* dst = p.score + ((row0 + row) * p.H + h) * 128 + j;
      *reinterpret_cast<uint32_t*>(dst) = hi;
      *reinterpret_cast<uint32_t*>(dst + 64) = lo;
    }
  }
}

template <typename T, bool MEMORY>
static int gated_scan_launch(GatedScanParams<T> p, int n_seq, cudaStream_t st) {
  // widest slice of P whose state fits in 16 float4 per thread; narrower while that leaves most of the machine idle
  int pw = p.P4;
  auto rows = [&](int w) { const int groups = kScanThreads / (w / 4); return groups < 1 ? 1 << 30 : (p.N + groups - 1) / groups; };
  while (pw > 4 && rows(pw) > 16) pw = (pw / 2 + 3) / 4 * 4;
  if (rows(pw) > 16) return -3;
  while (pw >= 64 && pw % 8 == 0 && static_cast<long long>(n_seq) * p.H * ((p.P4 + pw - 1) / pw) < num_sms()) pw /= 2;
  p.pw = pw;
  const int groups = kScanThreads / (pw / 4), e = rows(pw);
  const size_t smem = static_cast<size_t>((pw + 3 * p.N + 3) / 4 * 4 + groups * pw) * sizeof(float);
  if (smem > 48 * 1024) return -3;
  const dim3 grid(n_seq, p.H, (p.P4 + pw - 1) / pw);
  if (e <= 1) gated_scan_kernel<T, 1, MEMORY><<<grid, kScanThreads, smem, st>>>(p);
  else if (e <= 2) gated_scan_kernel<T, 2, MEMORY><<<grid, kScanThreads, smem, st>>>(p);
  else if (e <= 4) gated_scan_kernel<T, 4, MEMORY><<<grid, kScanThreads, smem, st>>>(p);
  else if (e <= 8) gated_scan_kernel<T, 8, MEMORY><<<grid, kScanThreads, smem, st>>>(p);
  else gated_scan_kernel<T, 16, MEMORY><<<grid, kScanThreads, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

static bool gated_bad_dims(int H, int N, int P) { return H < 1 || N < 1 || P < 1 || H > 65535 || N > 2048; }

}  // namespace pm

using namespace pm;

// Channel gates token by token. q / v: head 0's first column in row 0 of rows ldu apart, z fp32 rows of H N logits ldz apart, bias
// and lower fp32 [H N]; state [slots][H][N][P4] fp32, read and written; y [tokens, H P]. Sequence i covers tokens q_start[i] ..
// + q_lens[i] - 1 and ends at position seq_lens[i] - 1.
extern "C" int pm_channel_scan(const void* q, const void* v, int f32, long long ldu, const float* z, long long ldz, const float* bias,
                               const float* lower, float* state, const int* slots, const int* q_start, const int* q_lens,
                               const int* seq_lens, int n_seq, int H, int N, int P, void* y, cudaStream_t st) {
  if (gated_bad_dims(H, N, P)) return -1;
  if (n_seq < 1) return 0;
  const int P4 = (P + 3) / 4 * 4;
  if (f32)
    return gated_scan_launch<float, false>({static_cast<const float*>(q), nullptr, static_cast<const float*>(v), ldu, z, ldz, bias, lower,
                                            0.f, 1.f, 0.f, state, nullptr, nullptr, slots, q_start, q_lens, seq_lens,
                                            static_cast<float*>(y), nullptr, H, N, P, P4, 0}, n_seq, st);
  return gated_scan_launch<__nv_bfloat16, false>({static_cast<const __nv_bfloat16*>(q), nullptr, static_cast<const __nv_bfloat16*>(v), ldu,
                                                  z, ldz, bias, lower, 0.f, 1.f, 0.f, state, nullptr, nullptr, slots, q_start, q_lens,
                                                  seq_lens, static_cast<__nv_bfloat16*>(y), nullptr, H, N, P, P4, 0}, n_seq, st);
}

// Matrix memory token by token. q / k / v as above, z fp32 rows of H input gates and H forget gates, bias fp32 [2 H]; nstate
// [slots][H][N] and mstate [slots][H][P4 / 4] fp32 beside the state; y [tokens, H P] without, den fp32 [tokens, H] with the
// normaliser: the result is y / den.
extern "C" int pm_memory_scan(const void* q, const void* k, const void* v, int f32, long long ldu, const float* z, long long ldz,
                              const float* bias, float cap, float qscale, float den_eps, float* state, float* nstate, float* mstate,
                              const int* slots, const int* q_start, const int* q_lens, const int* seq_lens, int n_seq, int H, int N,
                              int P, void* y, float* den, cudaStream_t st) {
  if (gated_bad_dims(H, N, P) || !(cap > 0.f)) return -1;
  if (n_seq < 1) return 0;
  const int P4 = (P + 3) / 4 * 4;
  if (f32)
    return gated_scan_launch<float, true>({static_cast<const float*>(q), static_cast<const float*>(k), static_cast<const float*>(v), ldu, z,
                                           ldz, bias, nullptr, cap, qscale, den_eps, state, nstate, mstate, slots, q_start, q_lens,
                                           seq_lens, static_cast<float*>(y), den, H, N, P, P4, 0}, n_seq, st);
  return gated_scan_launch<__nv_bfloat16, true>({static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k),
                                                 static_cast<const __nv_bfloat16*>(v), ldu, z, ldz, bias, nullptr, cap, qscale, den_eps,
                                                 state, nstate, mstate, slots, q_start, q_lens, seq_lens,
                                                 static_cast<__nv_bfloat16*>(y), den, H, N, P, P4, 0}, n_seq, st);
}

// pm_channel_scan for longer portions of bf16 models, N <= 256, n16 = N rounded up to 16. Work buffers over all rows of the step: act
// bf16 [tokens, 4 H n16], score bf16 [tokens, H, 128]; block_decay fp32 [n_tok / 64 + n_seq + 1][H][n16]; seg_state
// [n_seq][max_seg][H][N][P4] and seg_decay [n_seq][max_seg][H][N] fp32. c_start: first token of every sequence, counted over these
// sequences alone; max_q: the longest of q_lens.
extern "C" int pm_channel_chunk(const void* q, const void* v, long long ldu, const float* z, long long ldz, const float* bias,
                                const float* lower, float* state, const int* slots, const int* q_start, const int* q_lens,
                                const int* seq_lens, const int* c_start, int n_seq, int max_q, int H, int N, int P, void* act,
                                void* score, float* block_decay, float* seg_state, float* seg_decay, int max_seg, void* y,
                                cudaStream_t st) {
  if (gated_bad_dims(H, N, P) || N > kSsdMaxState) return -1;
  if (n_seq < 1 || max_q < 1) return 0;
  const int n16 = (N + 15) / 16 * 16;
  const ChannelBlockParams b{static_cast<const __nv_bfloat16*>(q), ldu, z, ldz, bias, lower, q_start, q_lens, c_start,
                             static_cast<__nv_bfloat16*>(act), static_cast<__nv_bfloat16*>(score), block_decay, H, N, n16};
  const size_t smem = static_cast<size_t>(kBlockTokens) * ((n16 + 8) * (4 + 2) + 4 * n16 + 16) + 8 * kBlockCols * sizeof(float);
  const bool vec = N % 4 == 0 && ldu % 4 == 0 && ldz % 4 == 0 && reinterpret_cast<uintptr_t>(q) % 8 == 0 &&
                   (reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(lower)) % 16 == 0;
  const auto kernel = vec ? channel_block_kernel<true> : channel_block_kernel<false>;
  static DeviceMax configured[2];
  if (smem > configured[vec].get()) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[vec].set(smem);
  }
  kernel<<<dim3((max_q + kBlockTokens - 1) / kBlockTokens, H, n_seq), kBlockThreads, smem, st>>>(b);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return static_cast<int>(e);
  SsdParams p{};
  p.kind = kSsdChannel;
  p.act = b.act; p.ld = 4 * H * n16; p.c0 = 0; p.b0 = 2 * H * n16; p.lo = H * n16; p.NB = n16;
  p.x = static_cast<const __nv_bfloat16*>(v); p.ldx = static_cast<int>(ldu);
  p.score = b.score; p.block_decay = block_decay; p.c_start = c_start;
  p.state = state; p.slots = slots; p.q_start = q_start; p.q_lens = q_lens; p.seq_lens = seq_lens;
  p.y = static_cast<__nv_bfloat16*>(y); p.seg_state = seg_state; p.seg_decay = seg_decay;
  p.H = H; p.P = P; p.N = N; p.G = H; p.P4 = (P + 3) / 4 * 4;
  return ssd_chunk_launch(p, n_seq, max_q, max_seg, st);
}

// pm_memory_scan for longer portions of bf16 models, N <= 256. u: rows ldu apart with the keys of head 0 at column k_at and the
// queries at q_at; work buffers gates fp32 [3][tokens, H], seg_state [n_seq][max_seg][H][N][P4], seg_decay [n_seq][max_seg][H] and
// seg_n [n_seq][max_seg][H][N] fp32.
extern "C" int pm_memory_chunk(const void* u, int q_at, int k_at, const void* v, long long ldu, const float* z, long long ldz,
                               const float* bias, float cap, float qscale, float den_eps, float* state, float* nstate, float* mstate,
                               const int* slots, const int* q_start, const int* q_lens, const int* seq_lens, int n_seq, int n_tok,
                               int max_q, int H, int N, int P, float* gates, float* seg_state, float* seg_decay, float* seg_n,
                               int max_seg, void* y, float* den, cudaStream_t st) {
  if (gated_bad_dims(H, N, P) || N > kSsdMaxState || !(cap > 0.f)) return -1;
  if (n_seq < 1 || max_q < 1 || n_tok < 1) return 0;
  const long long step = static_cast<long long>(n_tok) * H;
  const int P4 = (P + 3) / 4 * 4;
  const MemoryGateParams g{z, ldz, bias, cap, mstate, slots, q_start, q_lens, seq_lens, gates, gates + step, gates + 2 * step, H, P4};
  memory_gates_kernel<<<dim3(H, n_seq), kGateThreads, 0, st>>>(g);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return static_cast<int>(e);
  SsdParams p{};
  p.kind = kSsdMemory;
  p.act = static_cast<const __nv_bfloat16*>(u); p.ld = static_cast<int>(ldu); p.b0 = k_at; p.c0 = q_at;
  p.x = static_cast<const __nv_bfloat16*>(v); p.ldx = static_cast<int>(ldu);
  p.ldec = g.ldec; p.dt = g.weight; p.mrun = g.mrun; p.nstate = nstate; p.seg_n = seg_n; p.den = den;
  p.yscale = qscale; p.den_eps = den_eps;
  p.state = state; p.slots = slots; p.q_start = q_start; p.q_lens = q_lens; p.seq_lens = seq_lens;
  p.y = static_cast<__nv_bfloat16*>(y); p.seg_state = seg_state; p.seg_decay = seg_decay;
  p.H = H; p.P = P; p.N = N; p.G = H; p.P4 = P4;
  return ssd_chunk_launch(p, n_seq, max_q, max_seg, st);
}
