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
//   the recurrence of longer portions runs in blocks of 64 tokens on the tensor cores (ssd_chunk.cu).
//   ssm_gate_norm_kernel  y * silu(z), RMS norm over equal parts of the row, weight; it also moves the last inputs of
//                     the convolution into the ring (it runs after every reader of the ring).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <type_traits>
#include "elem.cuh"
#include "host_util.cuh"
#include "pmetal_b200.h"
#include "ssd_chunk.cuh"

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
  SsdParams p{};
  p.act = c.act; p.dt = dt; p.a_log = a_log; p.dskip = dskip; p.state = state; p.slots = slots; p.q_start = q_start;
  p.q_lens = q_lens; p.seq_lens = seq_lens; p.y = static_cast<__nv_bfloat16*>(y);
  p.seg_state = seg_state; p.seg_decay = seg_decay;
  p.H = H; p.P = P; p.N = N; p.G = G; p.P4 = d.P4;
  p.ld = d.conv; p.b0 = d.inner; p.c0 = d.inner + G * N;
  return ssd_chunk_launch(p, n_seq, max_q, max_seg, st);
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
