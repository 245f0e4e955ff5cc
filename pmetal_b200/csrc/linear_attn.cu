// Linear attention with one fixed decay per head and no normaliser. Per sequence and head, with queries and keys of N
// channels and values of P:
//
//     S <- decay_h S + k v^T,      o = S^T q                                             S: [N, P], fp32
//
// The projection row of a token is u = [q: H N | k: H N | v: H P | g: H P]. q, k and v pass through an activation (silu,
// or none); q and k may be rotated on their first R channels, pairs (i, i + R / 2) or (2 i, 2 i + 1), and k carries a
// factor. S lives in slots as [slot][H][N][P4] fp32 (P4 = P rounded up to 4); a sequence whose first token of the step is
// position 0 starts from zeros whatever the slot holds.
//
//   linear_scan_kernel  any number of tokens, one after the other; one CTA per (sequence, head, slice of P), the state in
//                       registers, activation and rotation on the way in. Decode, short portions, fp32 models.
//   linear_prep_kernel  activation, rotation and factor for all tokens of longer portions (bf16). Activations are bf16;
//                       rotated queries and keys are fp32 values and leave as sums of two bf16 terms. The recurrence then
//                       runs in blocks of 64 tokens on the tensor cores (ssd_chunk.cu).
//   norm_gate_*_kernel  RMS norm over equal parts of the row (the whole row, or every head), optional weight, times the
//                       sigmoid or silu of g.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include "elem.cuh"
#include "host_util.cuh"
#include "pmetal_b200.h"
#include "ssd_chunk.cuh"

namespace pm {

enum : int { kRotNone = 0, kRotHalf = 1, kRotPairs = 2 };

struct LinearDims {
  int H, N, P, P4;
  int R, rot;           // rotated channels, kRot*
  int act;              // 1: silu on q, k and v
  float kscale;
};

template <typename T>
struct LinearScanParams {
  const T* u;
  long long ldu;
  const float* cs;         // [tokens, R / 2]
  const float* sn;
  const float* decay;      // [H]
  float* state;
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  T* y;                    // [tokens, H P]
  LinearDims d;
  int pw;                  // channels of P per CTA (multiple of 4)
};

// Channel i of a query or key row (head's first channel at `row`) after activation and rotation.
template <typename T>
__device__ __forceinline__ float linear_channel(const T* row, int i, const LinearDims& d, const float* cs, const float* sn) {
  float v = to_f(row[i]);
  if (d.act) v = silu_f(v);
  if (i < d.R) {
    const int half = d.R / 2;
    const bool second = d.rot == kRotHalf ? i >= half : (i & 1);
    const int f = d.rot == kRotHalf ? (second ? i - half : i) : i >> 1;
    const int j = d.rot == kRotHalf ? (second ? i - half : i + half) : i ^ 1;
    float w = to_f(row[j]);
    if (d.act) w = silu_f(w);
    v = second ? fmaf(v, cs[f], w * sn[f]) : fmaf(v, cs[f], -w * sn[f]);
  }
  return v;
}

constexpr int kLinThreads = 256;

// E: state rows per thread (float4 each).
template <typename T, int E>
__global__ void __launch_bounds__(kLinThreads, E <= 4 ? 4 : (E <= 8 ? 3 : 2)) linear_scan_kernel(const LinearScanParams<T> p) {
  extern __shared__ __align__(16) float lin_smem[];
  const LinearDims& d = p.d;
  const int seq = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * p.pw;
  const int len = p.q_lens[seq];
  if (len <= 0) return;
  const int cols = p.pw / 4, groups = kLinThreads / cols;
  float* sv = lin_smem;                      // [pw]
  float* sk = sv + p.pw;                     // [N]
  float* sq = sk + d.N;                      // [N]
  float* part = sv + (p.pw + 2 * d.N + 3) / 4 * 4;     // [groups][pw]
  const int q0 = p.q_start[seq], start = p.seq_lens[seq] - len;
  const long long slot = p.slots[seq];
  const int cq = h * d.N, ck = (d.H + h) * d.N, cv = 2 * d.H * d.N + h * d.P;
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
  const float decay = p.decay[h];
  const int half = d.R / 2;
  for (int t = 0; t < len; ++t) {
    const long long r = q0 + t;
    const T* row = p.u + r * p.ldu;
    const float* cs = p.cs + r * half;
    const float* sn = p.sn + r * half;
    __syncthreads();                          // the previous token's readers are done
    for (int i = threadIdx.x; i < p.pw + 2 * d.N; i += kLinThreads) {
      float v = 0.f;
      if (i < p.pw) {
        if (p0 + i < d.P) {
          v = to_f(row[cv + p0 + i]);
          if (d.act) v = silu_f(v);
        }
      } else if (i < p.pw + d.N) {
        v = linear_channel(row + ck, i - p.pw, d, cs, sn) * d.kscale;
      } else {
        v = linear_channel(row + cq, i - p.pw - d.N, d, cs, sn);
      }
      lin_smem[i] = v;
    }
    __syncthreads();
    if (owner) {
      const float4 x = *reinterpret_cast<const float4*>(sv + col * 4);
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < E; ++i) {
        const int n = grp + i * groups;
        if (n < d.N) {
          const float b = sk[n], c = sq[n];
          S[i].x = fmaf(decay, S[i].x, b * x.x); y.x = fmaf(c, S[i].x, y.x);
          S[i].y = fmaf(decay, S[i].y, b * x.y); y.y = fmaf(c, S[i].y, y.y);
          S[i].z = fmaf(decay, S[i].z, b * x.z); y.z = fmaf(c, S[i].z, y.z);
          S[i].w = fmaf(decay, S[i].w, b * x.w); y.w = fmaf(c, S[i].w, y.w);
        }
      }
      *reinterpret_cast<float4*>(part + grp * p.pw + col * 4) = y;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.pw; i += kLinThreads) {
      if (p0 + i >= d.P) continue;
      float v = 0.f;
      for (int k = 0; k < groups; ++k) v += part[k * p.pw + i];
      put(p.y + r * (d.H * d.P) + h * d.P + p0 + i, v);
    }
  }
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const int n = grp + i * groups;
    if (owner && n < d.N) *reinterpret_cast<float4*>(st + static_cast<long long>(n) * d.P4) = S[i];
  }
}

// ------------------------------------------------------------------------------------------- longer portions (bf16)
// act row: [v: H P | k: H N | q: H N], then, when `split`, the second terms of k and q in the same order.
struct LinearPrepParams {
  const __nv_bfloat16* u;
  long long ldu;
  const float* cs;
  const float* sn;
  __nv_bfloat16* act;
  int ld, n_tok, split;
  LinearDims d;
};

// V consecutive channels of one head per thread (V divides the head sizes and, for rotated channels, R or R / 2).
template <int V>
__global__ void __launch_bounds__(256) linear_prep_kernel(const LinearPrepParams p) {
  const LinearDims& d = p.d;
  const int HN = d.H * d.N, HP = d.H * d.P, per_row = (2 * HN + HP) / V;
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  const long long t = i / per_row;
  if (t >= p.n_tok) return;
  const int c = static_cast<int>(i - t * per_row) * V;            // column of u
  const __nv_bfloat16* src = p.u + t * p.ldu + c;
  __nv_bfloat16* row = p.act + t * p.ld;
  float v[V];
  load_vec<V>(src, v);
  if (d.act)
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = silu_fast(v[e]);
  if (c >= 2 * HN) {
    store_vec<V>(row + c - 2 * HN, v);
    return;
  }
  const bool key = c >= HN;
  const int hc = c % d.N;                                          // channel within the head
  const float* cs = p.cs + t * (d.R / 2);
  const float* sn = p.sn + t * (d.R / 2);
  if (hc < d.R) {
    if (d.rot == kRotHalf) {
      const int half = d.R / 2;
      const bool second = hc >= half;
      float w[V], a[V], b[V];
      load_vec<V>(second ? src - half : src + half, w);
      load_vec<V>(cs + (second ? hc - half : hc), a);
      load_vec<V>(sn + (second ? hc - half : hc), b);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        if (d.act) w[e] = silu_fast(w[e]);
        v[e] = fmaf(v[e], a[e], second ? w[e] * b[e] : -w[e] * b[e]);
      }
    } else if (V > 1) {
#pragma unroll
      for (int e = 0; e + 1 < V; e += 2) {
        const float a = cs[(hc + e) >> 1], b = sn[(hc + e) >> 1], x = v[e], w = v[e + 1];
        v[e] = fmaf(x, a, -w * b);
        v[e + 1] = fmaf(w, a, x * b);
      }
    } else {
      float w = __bfloat162float(hc & 1 ? src[-1] : src[1]);
      if (d.act) w = silu_fast(w);
      const float a = cs[hc >> 1], b = sn[hc >> 1];
      v[0] = fmaf(v[0], a, hc & 1 ? w * b : -w * b);
    }
  }
  if (key)
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= d.kscale;
  __nv_bfloat16* dst = row + HP + (key ? c - HN : c + HN);
  store_vec<V>(dst, v);
  if (p.split) {
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] -= __bfloat162float(__float2bfloat16(v[e]));
    store_vec<V>(dst + 2 * HN, v);
  }
}

// ------------------------------------------------------------------------------------------- norm and gate
enum : int { kGateSigmoid = 0, kGateSilu = 1, kGateNone = 2 };

template <int kGate, bool kFast>
__device__ __forceinline__ float gate_of(float g) {
  if (kGate == kGateNone) return 1.f;
  if (kGate == kGateSilu) return kFast ? silu_fast(g) : silu_f(g);
  return kFast ? sigmoid_fast(g) : sigmoid_f(g);
}

// What the norm kernels take beside y and the gate.
struct NormGateExtra {
  const float* w;          // nullable; [parts * width], shared: [width] for every part
  const float* den;        // [tokens, parts], nullable: y is divided by it before the norm
  int shared;
  float scale;             // factor of the result
  long long ldo;
};

// One warp per (token, part) with the part in registers: widths up to 256 IT, 8-element vectors.
template <typename T, int GATE, int IT>
__global__ void __launch_bounds__(256) norm_gate_warp_kernel(const T* __restrict__ y, const T* __restrict__ gate, long long ldg,
                                                             const NormGateExtra x, float eps, int parts, int width,
                                                             T* __restrict__ out, int n_tok) {
  const long long item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  const long long t = item / parts;
  if (t >= n_tok) return;
  const int c0 = static_cast<int>(item - t * parts) * width;
  const long long row = t * parts * width;
  float v[IT][8], z[IT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int k = (i * 32 + lane) * 8;
    if (k < width) {
      load_vec<8>(y + row + c0 + k, v[i]);
      if (GATE != kGateNone) load_vec<8>(gate + t * ldg + c0 + k, z[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[i][e], v[i][e], ss);
    }
  }
  // y / den over its root mean square: y times r / den with the mean of squares over den^2
  const float by = x.den ? 1.f / x.den[item] : 1.f;
  const float r = x.scale * by / sqrtf(warp_sum(ss) * by * by / static_cast<float>(width) + eps);
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int k = (i * 32 + lane) * 8;
    if (k < width) {
      float g[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) g[e] = 1.f;
      if (x.w) load_vec<8>(x.w + (x.shared ? 0 : c0) + k, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] *= r * g[e] * gate_of<GATE, sizeof(T) == 2>(z[i][e]);
      store_vec<8>(out + t * x.ldo + c0 + k, v[i]);
    }
  }
}

// One CTA per (token, part), any width that shared memory holds.
template <typename T, int GATE, int V>
__global__ void norm_gate_kernel(const T* __restrict__ y, const T* __restrict__ gate, long long ldg, const NormGateExtra x,
                                 float eps, int width, T* __restrict__ out) {
  extern __shared__ __align__(16) float ng_row[];
  const long long t = blockIdx.x, row = t * gridDim.y * width;
  const int c0 = blockIdx.y * width;
  float ss = 0.f;
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V) {
    float v[V];
    load_vec<V>(y + row + c0 + k, v);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      ng_row[k + e] = v[e];
      ss = fmaf(v[e], v[e], ss);
    }
  }
  const float by = x.den ? 1.f / x.den[t * gridDim.y + blockIdx.y] : 1.f;
  const float r = x.scale * by / sqrtf(block_sum(ss) * by * by / static_cast<float>(width) + eps);
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V) {
    float v[V], z[V], g[V];
    if (GATE != kGateNone) load_vec<V>(gate + t * ldg + c0 + k, z);
#pragma unroll
    for (int e = 0; e < V; ++e) g[e] = 1.f;
    if (x.w) load_vec<V>(x.w + (x.shared ? 0 : c0) + k, g);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = ng_row[k + e] * r * g[e] * gate_of<GATE, sizeof(T) == 2>(z[e]);
    store_vec<V>(out + t * x.ldo + c0 + k, v);
  }
}

template <typename T>
static int linear_scan_launch(LinearScanParams<T> p, int n_seq, cudaStream_t st) {
  const LinearDims& d = p.d;
  // widest slice of P whose state fits in 16 float4 per thread; narrower while that leaves most of the machine idle
  int pw = d.P4;
  auto rows = [&](int w) { const int groups = kLinThreads / (w / 4); return groups < 1 ? 1 << 30 : (d.N + groups - 1) / groups; };
  while (pw > 4 && rows(pw) > 16) pw = (pw / 2 + 3) / 4 * 4;
  if (rows(pw) > 16) return -3;
  while (pw >= 64 && pw % 8 == 0 && static_cast<long long>(n_seq) * d.H * ((d.P4 + pw - 1) / pw) < num_sms()) pw /= 2;
  p.pw = pw;
  const int groups = kLinThreads / (pw / 4), e = rows(pw);
  const size_t smem = static_cast<size_t>((pw + 2 * d.N + 3) / 4 * 4 + groups * pw) * sizeof(float);
  if (smem > 48 * 1024) return -3;
  const dim3 grid(n_seq, d.H, (d.P4 + pw - 1) / pw);
  if (e <= 1) linear_scan_kernel<T, 1><<<grid, kLinThreads, smem, st>>>(p);
  else if (e <= 2) linear_scan_kernel<T, 2><<<grid, kLinThreads, smem, st>>>(p);
  else if (e <= 4) linear_scan_kernel<T, 4><<<grid, kLinThreads, smem, st>>>(p);
  else if (e <= 8) linear_scan_kernel<T, 8><<<grid, kLinThreads, smem, st>>>(p);
  else linear_scan_kernel<T, 16><<<grid, kLinThreads, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int GATE>
static int norm_gate_launch(const void* y, const void* gate, long long ldg, const NormGateExtra& x, float eps, int parts, int width,
                            void* out, int n_tok, cudaStream_t st) {
  const T* yy = static_cast<const T*>(y);
  const T* gg = static_cast<const T*>(gate);
  T* oo = static_cast<T*>(out);
  const bool v8 = width % 8 == 0 && ldg % 8 == 0 && x.ldo % 8 == 0 &&
                  (reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) % (8 * sizeof(T)) == 0;
  // a warp per part pays when there are parts enough to fill the machine
  if (v8 && width <= 1024 && (width <= 256 || static_cast<long long>(n_tok) * parts >= 8ll * num_sms())) {
    const unsigned grid = static_cast<unsigned>((static_cast<long long>(n_tok) * parts + 7) / 8);
    if (width <= 256) norm_gate_warp_kernel<T, GATE, 1><<<grid, 256, 0, st>>>(yy, gg, ldg, x, eps, parts, width, oo, n_tok);
    else if (width <= 512) norm_gate_warp_kernel<T, GATE, 2><<<grid, 256, 0, st>>>(yy, gg, ldg, x, eps, parts, width, oo, n_tok);
    else norm_gate_warp_kernel<T, GATE, 4><<<grid, 256, 0, st>>>(yy, gg, ldg, x, eps, parts, width, oo, n_tok);
    return static_cast<int>(cudaGetLastError());
  }
  const size_t smem = static_cast<size_t>(width) * sizeof(float);
  static DeviceOnce once;
  if (once.pending()) {
    cudaError_t e = cudaFuncSetAttribute(norm_gate_kernel<T, GATE, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(norm_gate_kernel<T, GATE, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    once.mark();
  }
  const int v = v8 ? 8 : 1;
  int threads = (width / v + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 512 ? 512 : threads);
  if (v8) norm_gate_kernel<T, GATE, 8><<<dim3(n_tok, parts), threads, smem, st>>>(yy, gg, ldg, x, eps, width, oo);
  else norm_gate_kernel<T, GATE, 1><<<dim3(n_tok, parts), threads, smem, st>>>(yy, gg, ldg, x, eps, width, oo);
  return static_cast<int>(cudaGetLastError());
}

static bool linear_dims(LinearDims* d, int H, int N, int P, int R, int rot, int act, float kscale) {
  if (H < 1 || N < 1 || P < 1 || rot < kRotNone || rot > kRotPairs || R < 0 || R > N || R % 2 || (rot == kRotNone && R)) return false;
  *d = LinearDims{H, N, P, (P + 3) / 4 * 4, R, rot, act, kscale};
  return true;
}

}  // namespace pm

using namespace pm;

// Token-by-token recurrence. u [tokens, ldu]; cs / sn fp32 [tokens, R / 2] (unused when R is 0); rot: 1 pairs (i, i + R / 2),
// 2 pairs (2 i, 2 i + 1); act: 1 silu on q, k, v; decay fp32 [H]; state [slots][H][N][P4] fp32, read and written;
// y [tokens, H P]. Sequence i covers tokens q_start[i] .. + q_lens[i] - 1 and ends at position seq_lens[i] - 1.
extern "C" int pm_linear_scan(const void* u, int f32, long long ldu, const float* cs, const float* sn, const float* decay,
                              float kscale, float* state, const int* slots, const int* q_start, const int* q_lens,
                              const int* seq_lens, int n_seq, int H, int N, int P, int R, int rot, int act, void* y,
                              cudaStream_t st) {
  LinearDims d;
  if (!linear_dims(&d, H, N, P, R, rot, act, kscale)) return -1;
  if (ldu < 2ll * H * N + static_cast<long long>(H) * P) return -2;
  if (n_seq < 1) return 0;
  if (f32) {
    LinearScanParams<float> p{static_cast<const float*>(u), ldu, cs, sn, decay, state, slots, q_start, q_lens, seq_lens,
                              static_cast<float*>(y), d, 0};
    return linear_scan_launch(p, n_seq, st);
  }
  LinearScanParams<__nv_bfloat16> p{static_cast<const __nv_bfloat16*>(u), ldu, cs, sn, decay, state, slots, q_start, q_lens,
                                    seq_lens, static_cast<__nv_bfloat16*>(y), d, 0};
  return linear_scan_launch(p, n_seq, st);
}

// Whether pm_linear_chunk covers keys of N channels.
extern "C" int pm_linear_chunk_supported(int N) { return N >= 1 && N <= kSsdMaxState; }

// The same for longer portions of bf16 models (act bf16 [n_tok, H P + 2 H N], twice the key and query columns when R > 0:
// work buffer over all n_tok rows of the step; log2_decay fp32 [H]; seg_state [n_seq][max_seg][H][N][P4] and seg_decay
// [n_seq][max_seg][H] fp32 work buffers; max_q: the longest of q_lens).
extern "C" int pm_linear_chunk(const void* u, long long ldu, const float* cs, const float* sn, const float* log2_decay,
                               float kscale, float* state, const int* slots, const int* q_start, const int* q_lens,
                               const int* seq_lens, int n_seq, int n_tok, int max_q, int H, int N, int P, int R, int rot,
                               int act, void* act_buf, float* seg_state, float* seg_decay, int max_seg, void* y,
                               cudaStream_t st) {
  LinearPrepParams a{};
  if (!linear_dims(&a.d, H, N, P, R, rot, act, kscale) || !pm_linear_chunk_supported(N)) return -1;
  const int HN = H * N, HP = H * P;
  if (ldu < 2ll * HN + HP) return -2;
  if (n_seq < 1 || max_q < 1 || n_tok < 1) return 0;
  a.split = R > 0;
  a.ld = HP + (a.split ? 4 : 2) * HN;
  a.u = static_cast<const __nv_bfloat16*>(u); a.ldu = ldu; a.cs = cs; a.sn = sn;
  a.act = static_cast<__nv_bfloat16*>(act_buf); a.n_tok = n_tok;
  const int unit = R > 0 ? (rot == kRotHalf ? R / 2 : R) : 8;
  const int v = N % 8 == 0 && P % 8 == 0 && unit % 8 == 0 && ldu % 8 == 0 ? 8 : 1;
  const long long items = static_cast<long long>(n_tok) * ((2 * HN + HP) / v);
  const unsigned grid = static_cast<unsigned>((items + 255) / 256);
  if (v == 8) linear_prep_kernel<8><<<grid, 256, 0, st>>>(a);
  else linear_prep_kernel<1><<<grid, 256, 0, st>>>(a);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return static_cast<int>(e);
  SsdParams p{};
  p.act = a.act; p.log2_decay = log2_decay; p.state = state; p.slots = slots; p.q_start = q_start; p.q_lens = q_lens;
  p.seq_lens = seq_lens; p.y = static_cast<__nv_bfloat16*>(y); p.seg_state = seg_state; p.seg_decay = seg_decay;
  p.H = H; p.P = P; p.N = N; p.G = H; p.P4 = a.d.P4;
  p.ld = a.ld; p.b0 = HP; p.c0 = HP + HN; p.lo = a.split ? 2 * HN : 0;
  return ssd_chunk_launch(p, n_seq, max_q, max_seg, st);
}

template <typename T>
static int norm_gate_any(const void* y, const void* gate, long long ldg, const NormGateExtra& x, float eps, int parts, int width, int silu,
                         void* out, int n_tok, cudaStream_t st) {
  if (!gate) return norm_gate_launch<T, kGateNone>(y, nullptr, 0, x, eps, parts, width, out, n_tok, st);
  return silu ? norm_gate_launch<T, kGateSilu>(y, gate, ldg, x, eps, parts, width, out, n_tok, st)
              : norm_gate_launch<T, kGateSigmoid>(y, gate, ldg, x, eps, parts, width, out, n_tok, st);
}

// out [tokens, ldo] = RMS norm over every part of y [tokens, parts * width], times w (fp32 [parts * width], shared 1: [width] for every
// part, or null), times sigmoid(gate) or, silu 1, silu(gate), times scale; gate rows are ldg apart (null: no gate). den (fp32
// [tokens, parts], nullable): y is divided by it first.
extern "C" int pm_norm_gate(const void* y, const void* gate, int f32, long long ldg, const float* w, float eps, int parts,
                            int width, int silu, void* out, int n_tok, const float* den, int shared, float scale, long long ldo,
                            cudaStream_t st) {
  if (parts < 1 || width < 1 || static_cast<size_t>(width) * 4 > 200 * 1024 || parts > 65535 || ldo < static_cast<long long>(parts) * width)
    return -1;
  if (n_tok < 1) return 0;
  const NormGateExtra x{w, den, shared, scale, ldo};
  return f32 ? norm_gate_any<float>(y, gate, ldg, x, eps, parts, width, silu, out, n_tok, st)
             : norm_gate_any<__nv_bfloat16>(y, gate, ldg, x, eps, parts, width, silu, out, n_tok, st);
}
