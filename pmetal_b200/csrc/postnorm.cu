// Pieces of decoders whose residual stream is kept in fp32:
//   * token embedding times a factor, written as the fp32 stream and as the compute-type copy the projections read
//   * residual sum + layer norm:  x <- LN(alpha * x + y (+ bias)) * w + b, statistics in fp32 over the row held in
//     shared memory (the variance is the mean of squared deviations, taken in a second pass)
//   * residual sum of parallel sublayers + RMS norm of the next layer:  x <- x + y + (sum of a token's expert rows) + x0,
//     h = x / rms(x) * w; every term but x is optional
//   * norm of a sublayer's result ahead of the residual sum:  x <- x + r / rms(r) * w,  r = y + (weighted sum of a token's expert
//     rows, where a choice may stand for x itself)
//   * exact gelu of rows
//   * clamped gated unit:  g = min(g, limit), u = clamp(u, -limit, limit), out = g * sigmoid(beta g) * (u + shift)
//   * rotation table whose angles are formed and reduced in fp64, so that far positions keep fp32-accurate angles
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include "elem.cuh"
#include "host_util.cuh"
#include "pmetal_b200.h"

namespace pm {

template <typename T, int V>
__global__ void embed_scale_kernel(const long long* __restrict__ ids, const T* __restrict__ table, float scale, int width,
                                   float* __restrict__ xf, T* __restrict__ xc) {
  const long long t = blockIdx.x;
  const T* src = table + ids[t] * static_cast<long long>(width);
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V) {
    float v[V];
    load_vec<V>(src + k, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= scale;
    store_vec<V>(xf + t * width + k, v);
    if (xc) store_vec<V>(xc + t * width + k, v);
  }
}

// One CTA per output row; `rows` (nullable) picks the input row. Outputs are nullable.
template <typename T, int V>
__global__ void post_layernorm_kernel(const float* x, const T* __restrict__ y, long long ldy,
                                      const float* __restrict__ bias, float alpha, const float* __restrict__ w,
                                      const float* __restrict__ b, float eps, int width, const long long* __restrict__ rows,
                                      float* of, T* __restrict__ oc) {
  extern __shared__ __align__(16) float row_buf[];
  const long long o = blockIdx.x, r = rows ? rows[o] : o;
  float sum = 0.f;
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V) {
    float v[V];
    load_vec<V>(x + r * width + k, v);
    if (y) {
      float s[V];
      load_vec<V>(y + r * ldy + k, s);
      if (bias) {
        float c[V];
        load_vec<V>(bias + k, c);
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] += c[e];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = fmaf(alpha, v[e], s[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      row_buf[k + e] = v[e];
      sum += v[e];
    }
  }
  const float mean = block_sum(sum) / static_cast<float>(width);
  float dev = 0.f;
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V)
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float d = row_buf[k + e] - mean;
      dev = fmaf(d, d, dev);
    }
  const float rstd = 1.f / sqrtf(block_sum(dev) / static_cast<float>(width) + eps);
  for (int k = threadIdx.x * V; k < width; k += blockDim.x * V) {
    float v[V], ww[V], bb[V];
    load_vec<V>(w + k, ww);
    load_vec<V>(b + k, bb);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = fmaf((row_buf[k + e] - mean) * rstd, ww[e], bb[e]);
    if (of) store_vec<V>(of + o * width + k, v);
    if (oc) store_vec<V>(oc + o * width + k, v);
  }
}

struct AddRmsParams {
  const float* x;
  const void* y;               // [.., ldy] compute type
  long long ldy;
  const void* z;               // [.., width] compute type: rows inv[t * k] .. inv[t * k + k - 1] belong to token t
  const int* inv;
  int k;
  const float* x0;
  const float* w;
  float w_base, eps;
  int width;
  const long long* rows;
  float* of;
  void* oc;
};

// One CTA per output row; `rows` (nullable) picks the input row. of may be x.
template <typename T, int V>
__global__ void add_rmsnorm_kernel(const AddRmsParams p) {
  extern __shared__ __align__(16) float row_buf[];
  const long long o = blockIdx.x, r = p.rows ? p.rows[o] : o;
  const T* y = static_cast<const T*>(p.y);
  const T* z = static_cast<const T*>(p.z);
  float ss = 0.f;
  for (int k = threadIdx.x * V; k < p.width; k += blockDim.x * V) {
    float v[V], s[V];
    load_vec<V>(p.x + r * p.width + k, v);
#pragma unroll
    for (int e = 0; e < V; ++e) s[e] = 0.f;
    if (y) load_vec<V>(y + r * p.ldy + k, s);
    if (z)
      for (int j = 0; j < p.k; ++j) {
        float c[V];
        load_vec<V>(z + static_cast<long long>(p.inv[r * p.k + j]) * p.width + k, c);
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] += c[e];
      }
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] += s[e];
    if (p.x0) {
      float c[V];
      load_vec<V>(p.x0 + r * p.width + k, c);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += c[e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      row_buf[k + e] = v[e];
      ss = fmaf(v[e], v[e], ss);
    }
    if (p.of) store_vec<V>(p.of + o * p.width + k, v);
  }
  const float scale = 1.f / sqrtf(block_sum(ss) / static_cast<float>(p.width) + p.eps);
  T* oc = static_cast<T*>(p.oc);
  for (int k = threadIdx.x * V; k < p.width; k += blockDim.x * V) {
    float v[V], ww[V];
    load_vec<V>(p.w + k, ww);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = row_buf[k + e] * scale * (p.w_base + ww[e]);
    store_vec<V>(oc + o * p.width + k, v);
  }
}

struct AddNormedParams {
  const float* x;
  const void* y;               // [.., ldy] compute type
  long long ldy;
  const void* z;               // [.., width] compute type: row[t * k + j] is the row of token t's choice j
  const int* row;
  const int* ids;              // the choices; from n_experts on they stand for x
  const float* wt;             // their weights
  int k, n_experts;
  const float* w;
  float w_base, eps;
  int width;
  float* of;
  void* oc;
};

// One CTA per row. of may be x.
template <typename T, int V>
__global__ void add_normed_kernel(const AddNormedParams p) {
  extern __shared__ __align__(16) float row_buf[];
  const long long t = blockIdx.x;
  const T* y = static_cast<const T*>(p.y);
  const T* z = static_cast<const T*>(p.z);
  const float* x = p.x + t * p.width;
  float own = 0.f;             // weight of x itself
  for (int j = 0; j < p.k; ++j)
    if (p.ids[t * p.k + j] >= p.n_experts) own += p.wt[t * p.k + j];
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < p.width; c += blockDim.x * V) {
    float r[V], s[V];
    load_vec<V>(x + c, r);
#pragma unroll
    for (int e = 0; e < V; ++e) r[e] *= own;
    if (y) {
      load_vec<V>(y + t * p.ldy + c, s);
#pragma unroll
      for (int e = 0; e < V; ++e) r[e] += s[e];
    }
    for (int j = 0; j < p.k; ++j) {
      if (p.ids[t * p.k + j] >= p.n_experts) continue;
      const float f = p.wt[t * p.k + j];
      load_vec<V>(z + static_cast<long long>(p.row[t * p.k + j]) * p.width + c, s);
#pragma unroll
      for (int e = 0; e < V; ++e) r[e] = fmaf(f, s[e], r[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      row_buf[c + e] = r[e];
      ss = fmaf(r[e], r[e], ss);
    }
  }
  const float scale = 1.f / sqrtf(block_sum(ss) / static_cast<float>(p.width) + p.eps);
  T* oc = static_cast<T*>(p.oc);
  for (int c = threadIdx.x * V; c < p.width; c += blockDim.x * V) {
    float v[V], ww[V];
    load_vec<V>(x + c, v);
    load_vec<V>(p.w + c, ww);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = fmaf(row_buf[c + e] * scale, p.w_base + ww[e], v[e]);
    store_vec<V>(p.of + t * p.width + c, v);
    if (oc) store_vec<V>(oc + t * p.width + c, v);
  }
}

// May run in place (out = x, ldo = ldx).
template <typename T, int V>
__global__ void gelu_kernel(const T* x, long long ldx, int cols, T* out, long long ldo, long long n_vec) {
  const int per_row = cols / V;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n_vec;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / per_row;
    const int c = static_cast<int>(i - t * per_row) * V;
    float v[V];
    load_vec<V>(x + t * ldx + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = sizeof(T) == 2 ? gelu_fast(v[e]) : gelu_f(v[e]);
    store_vec<V>(out + t * ldo + c, v);
  }
}

template <typename T, int V>
__global__ void clamped_glu_kernel(const T* __restrict__ gu, long long ld, const float* __restrict__ bias, int ff,
                                   float limit, float beta, float shift, T* __restrict__ out, long long n_vec) {
  const int per_row = ff / V;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n_vec;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / per_row;
    const int k = static_cast<int>(i - t * per_row) * V;
    float g[V], u[V];
    load_vec<V>(gu + t * ld + k, g);
    load_vec<V>(gu + t * ld + ff + k, u);
    if (bias) {
      float a[V], c[V];
      load_vec<V>(bias + k, a);
      load_vec<V>(bias + ff + k, c);
#pragma unroll
      for (int e = 0; e < V; ++e) { g[e] += a[e]; u[e] += c[e]; }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) g[e] = clamped_glu<sizeof(T) == 2>(g[e], u[e], limit, beta, shift);
    store_vec<V>(out + t * ff + k, g);
  }
}

__global__ void rope_table_f64_kernel(const int* __restrict__ pos, const double* __restrict__ freq, int n, int half,
                                      float* __restrict__ cs, float* __restrict__ sn) {
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n * half; i += gridDim.x * blockDim.x) {
    const int t = i / half, j = i - t * half;
    const double two_pi = 6.283185307179586476925286766559;
    double a = static_cast<double>(pos[t]) * freq[j];
    a -= rint(a / two_pi) * two_pi;
    float s, c;
    sincosf(static_cast<float>(a), &s, &c);
    cs[i] = c;
    sn[i] = s;
  }
}

static int row_threads(int width, int v) {
  const int want = (width / v + 31) / 32 * 32;
  return want < 32 ? 32 : (want > 256 ? 256 : want);
}

template <typename T>
static int embed_launch(const long long* ids, const void* table, float scale, int n, int width, float* xf, void* xc,
                        cudaStream_t st) {
  const T* tab = static_cast<const T*>(table);
  T* out = static_cast<T*>(xc);
  if (width % 4 == 0) embed_scale_kernel<T, 4><<<n, row_threads(width, 4), 0, st>>>(ids, tab, scale, width, xf, out);
  else embed_scale_kernel<T, 1><<<n, row_threads(width, 1), 0, st>>>(ids, tab, scale, width, xf, out);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int V>
static int postnorm_launch(const float* x, const void* y, long long ldy, const float* bias, float alpha, const float* w,
                           const float* b, float eps, int n, int width, const long long* rows, float* of, void* oc,
                           cudaStream_t st) {
  const size_t smem = static_cast<size_t>(width) * sizeof(float);
  static DeviceMax configured;
  if (smem > 40 * 1024 && smem > configured.get()) {
    const cudaError_t e = cudaFuncSetAttribute(post_layernorm_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.set(200 * 1024);
  }
  post_layernorm_kernel<T, V><<<n, row_threads(width, V), smem, st>>>(x, static_cast<const T*>(y), ldy, bias, alpha, w, b,
                                                                      eps, width, rows, of, static_cast<T*>(oc));
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int V>
static int add_rms_launch(const AddRmsParams& p, int n, cudaStream_t st) {
  const size_t smem = static_cast<size_t>(p.width) * sizeof(float);
  static DeviceMax configured;
  if (smem > 40 * 1024 && smem > configured.get()) {
    const cudaError_t e = cudaFuncSetAttribute(add_rmsnorm_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.set(200 * 1024);
  }
  int threads = row_threads(p.width, V);
  if (n < 2 * num_sms() && p.width >= 512 * V) threads = 512;       // few rows: one pass over each
  add_rmsnorm_kernel<T, V><<<n, threads, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int V>
static int add_normed_launch(const AddNormedParams& p, int n, cudaStream_t st) {
  const size_t smem = static_cast<size_t>(p.width) * sizeof(float);
  static DeviceMax configured;
  if (smem > 40 * 1024 && smem > configured.get()) {
    const cudaError_t e = cudaFuncSetAttribute(add_normed_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured.set(200 * 1024);
  }
  int threads = row_threads(p.width, V);
  if (n < 2 * num_sms() && p.width >= 512 * V) threads = 512;       // few rows: one pass over each
  add_normed_kernel<T, V><<<n, threads, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int gelu_launch(const void* x, long long ldx, int n, int cols, void* out, long long ldo, cudaStream_t st) {
  const int v = cols % 8 == 0 && ldx % 8 == 0 && ldo % 8 == 0 ? 8 : 1;
  const long long n_vec = static_cast<long long>(n) * (cols / v);
  long long grid = (n_vec + 255) / 256;
  if (grid > num_sms() * 16) grid = num_sms() * 16;
  const T* src = static_cast<const T*>(x);
  T* dst = static_cast<T*>(out);
  if (v == 8) gelu_kernel<T, 8><<<static_cast<int>(grid), 256, 0, st>>>(src, ldx, cols, dst, ldo, n_vec);
  else gelu_kernel<T, 1><<<static_cast<int>(grid), 256, 0, st>>>(src, ldx, cols, dst, ldo, n_vec);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int glu_launch(const void* gu, long long ld, const float* bias, int n, int ff, float limit, float beta, float shift,
                      void* out, cudaStream_t st) {
  const int v = ff % 8 == 0 && ld % 8 == 0 ? 8 : (ff % 4 == 0 && ld % 4 == 0 ? 4 : 1);
  const long long n_vec = static_cast<long long>(n) * (ff / v);
  long long grid = (n_vec + 255) / 256;
  if (grid > num_sms() * 16) grid = num_sms() * 16;
  const T* src = static_cast<const T*>(gu);
  if (v == 8) clamped_glu_kernel<T, 8><<<static_cast<int>(grid), 256, 0, st>>>(src, ld, bias, ff, limit, beta, shift, static_cast<T*>(out), n_vec);
  else if (v == 4) clamped_glu_kernel<T, 4><<<static_cast<int>(grid), 256, 0, st>>>(src, ld, bias, ff, limit, beta, shift, static_cast<T*>(out), n_vec);
  else clamped_glu_kernel<T, 1><<<static_cast<int>(grid), 256, 0, st>>>(src, ld, bias, ff, limit, beta, shift, static_cast<T*>(out), n_vec);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace pm

using namespace pm;

// xf [n, width] fp32 = table[ids] * scale, xc the same in the table's type (nullable). f32: the table is fp32, else bf16.
extern "C" int pm_embed_scale(const long long* ids, const void* table, int f32, float scale, int n, int width, float* xf,
                              void* xc, cudaStream_t st) {
  if (n < 0 || width < 1) return -1;
  if (n == 0) return 0;
  return f32 ? embed_launch<float>(ids, table, scale, n, width, xf, xc, st)
             : embed_launch<__nv_bfloat16>(ids, table, scale, n, width, xf, xc, st);
}

// of / oc [n, width] (fp32 / compute type, each nullable) = LN(alpha * x + y + bias) * w + b for the n rows listed in
// `rows` (nullable: row i). y [.., ldy] and bias are nullable; without y the row is x itself. of may be x when rows is
// null.
extern "C" int pm_post_layernorm(const float* x, const void* y, int f32, long long ldy, const float* bias, float alpha,
                                 const float* w, const float* b, float eps, int n, int width, const long long* rows,
                                 float* of, void* oc, cudaStream_t st) {
  if (n < 0 || width < 1 || static_cast<size_t>(width) * 4 > 200 * 1024 || (rows && of == x)) return -1;
  if (n == 0) return 0;
  const bool vec = width % 4 == 0 && ldy % 4 == 0;
  if (f32)
    return vec ? postnorm_launch<float, 4>(x, y, ldy, bias, alpha, w, b, eps, n, width, rows, of, oc, st)
               : postnorm_launch<float, 1>(x, y, ldy, bias, alpha, w, b, eps, n, width, rows, of, oc, st);
  return vec ? postnorm_launch<__nv_bfloat16, 4>(x, y, ldy, bias, alpha, w, b, eps, n, width, rows, of, oc, st)
             : postnorm_launch<__nv_bfloat16, 1>(x, y, ldy, bias, alpha, w, b, eps, n, width, rows, of, oc, st);
}

// v = x + y + sum_j z[inv[t * k + j]] + x0 for the n rows listed in `rows` (nullable: row i); of [n, width] fp32 (nullable, may
// be x when rows is null) = v, oc [n, width] in the compute type = v / rms(v) * (w_base + w). y [.., ldy], z [.., width] (compute type,
// inv int32 per token and j < k) and x0 (fp32) are nullable.
extern "C" int pm_add_rmsnorm(const float* x, const void* y, int f32, long long ldy, const void* z, const int* inv, int k,
                              const float* x0, const float* w, float w_base, float eps, int n, int width, const long long* rows,
                              float* of, void* oc, cudaStream_t st) {
  if (n < 0 || width < 1 || static_cast<size_t>(width) * 4 > 200 * 1024 || (rows && of == x) || (z && (!inv || k < 1))) return -1;
  if (n == 0) return 0;
  const AddRmsParams p{x, y, ldy, z, inv, k, x0, w, w_base, eps, width, rows, of, oc};
  const bool vec = width % 4 == 0 && ldy % 4 == 0;
  if (f32) return vec ? add_rms_launch<float, 4>(p, n, st) : add_rms_launch<float, 1>(p, n, st);
  return vec ? add_rms_launch<__nv_bfloat16, 4>(p, n, st) : add_rms_launch<__nv_bfloat16, 1>(p, n, st);
}

// v = x + r / rms(r) * (w_base + w) with r = y + sum over j < k of wt[t, j] * (ids[t, j] < n_experts ? z[row[t, j]] : x[t]); of
// [n, width] fp32 = v (may be x), oc the same in the compute type (nullable). y [.., ldy] is nullable, k may be 0.
extern "C" int pm_add_normed(const float* x, const void* y, int f32, long long ldy, const void* z, const int* row, const int* ids,
                             const float* wt, int k, int n_experts, const float* w, float w_base, float eps, int n, int width,
                             float* of, void* oc, cudaStream_t st) {
  if (n < 0 || width < 1 || static_cast<size_t>(width) * 4 > 200 * 1024 || k < 0 || (k > 0 && (!z || !row || !ids || !wt)) || !of) return -1;
  if (n == 0) return 0;
  const AddNormedParams p{x, y, ldy, z, row, ids, wt, k, n_experts, w, w_base, eps, width, of, oc};
  const bool vec = width % 4 == 0 && ldy % 4 == 0;
  if (f32) return vec ? add_normed_launch<float, 4>(p, n, st) : add_normed_launch<float, 1>(p, n, st);
  return vec ? add_normed_launch<__nv_bfloat16, 4>(p, n, st) : add_normed_launch<__nv_bfloat16, 1>(p, n, st);
}

// out [n, ldo] = exact gelu of x [n, ldx] on the first `cols` columns; out may be x.
extern "C" int pm_gelu(const void* x, int f32, long long ldx, int n, int cols, void* out, long long ldo, cudaStream_t st) {
  if (n < 0 || cols < 1 || ldx < cols || ldo < cols) return -1;
  if (n == 0) return 0;
  return f32 ? gelu_launch<float>(x, ldx, n, cols, out, ldo, st) : gelu_launch<__nv_bfloat16>(x, ldx, n, cols, out, ldo, st);
}

// gu [n, ld]: gate columns [0, ff), up columns [ff, 2 ff); bias fp32 [2 ff] or null -> out [n, ff].
extern "C" int pm_clamped_glu(const void* gu, int f32, long long ld, const float* bias, int n, int ff, float limit,
                              float beta, float shift, void* out, cudaStream_t st) {
  if (n < 0 || ff < 1 || ld < 2ll * ff) return -1;
  if (n == 0) return 0;
  return f32 ? glu_launch<float>(gu, ld, bias, n, ff, limit, beta, shift, out, st)
             : glu_launch<__nv_bfloat16>(gu, ld, bias, n, ff, limit, beta, shift, out, st);
}

// cos / sin [n, half] fp32 of pos * freq (freq fp64 [half] on the device).
extern "C" int pm_rope_table_f64(const int* pos, const double* freq, int n, int half, float* cs, float* sn,
                                 cudaStream_t st) {
  if (n < 0 || half < 1) return -1;
  if (n == 0) return 0;
  int grid = (n * half + 255) / 256;
  if (grid > num_sms() * 8) grid = num_sms() * 8;
  rope_table_f64_kernel<<<grid, 256, 0, st>>>(pos, freq, n, half, cs, sn);
  return static_cast<int>(cudaGetLastError());
}
