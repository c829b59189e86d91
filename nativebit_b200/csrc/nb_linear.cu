// Dense pieces of the layered decoders: embedding lookup with a scale, the residual chain (norm after a sublayer, add,
// norm before the next), the fp32 matrix product, and the decode matvec over bf16 weights with the chain folded in.
#include <cuda_runtime.h>
#include <cuda_bf16.h>

#include <algorithm>

#include "nb_layered.cuh"

namespace nb {

__global__ void __launch_bounds__(256) embed_scaled_kernel(const bf16* __restrict__ table, const long long* __restrict__ token,
                                                           float* __restrict__ x, int V, int C, float scale, int streams) {
  pdl_enter();
  long long t = token[blockIdx.x];
  t = t < 0 ? 0 : (t >= V ? V - 1 : t);
  const bf16* row = table + (size_t)t * C;
  for (int i = threadIdx.x; i < C; i += 256) {
    const float v = __bfloat162float(row[i]) * scale;
    for (int s = 0; s < streams; ++s) x[((size_t)blockIdx.x * streams + s) * C + i] = v;
  }
}

// One CTA per row; the row stays in shared memory between the passes (a thread rereads only what it wrote).
constexpr int kChainThreads = 256, kChainWarps = kChainThreads / 32;

template <typename TH>
__global__ void __launch_bounds__(kChainThreads) residual_norm_kernel(float* __restrict__ x, const float* __restrict__ y,
                                                                      const float* __restrict__ wy, const float* __restrict__ w, int kind,
                                                                      float eps, TH* __restrict__ h, int ldh, int C) {
  extern __shared__ __align__(16) float row_s[];
  __shared__ float red[4 * kChainWarps];
  pdl_enter();
  float* xr = x + (size_t)blockIdx.x * C;
  const int tid = threadIdx.x;
  auto each = [&](auto f) {
    for (int i = tid; i < C; i += kChainThreads) f(row_s[i]);
  };
  float mean, inv;
  if (y) {
    const float* yr = y + (size_t)blockIdx.x * C;
    for (int i = tid; i < C; i += kChainThreads) row_s[i] = yr[i];
    norm_stats<kChainWarps>(kind, C, eps, red, each, mean, inv);
    for (int i = tid; i < C; i += kChainThreads) {
      const float v = xr[i] + (row_s[i] - mean) * inv * wy[i];
      xr[i] = v;
      row_s[i] = v;
    }
  } else {
    for (int i = tid; i < C; i += kChainThreads) row_s[i] = xr[i];
  }
  if (h) {
    norm_stats<kChainWarps>(kind, C, eps, red + 2 * kChainWarps, each, mean, inv);
    TH* hr = h + (size_t)blockIdx.x * ldh;
    for (int i = tid; i < C; i += kChainThreads) hr[i] = from_f<TH>((row_s[i] - mean) * inv * w[i]);
  }
}

// The same with the row in registers, four values per thread and load: C <= 1024 * NV, a multiple of 4.
__device__ __forceinline__ void store4(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void store4(bf16* p, float a, float b, float c, float d) {
  const __nv_bfloat162 x = __floats2bfloat162_rn(a, b), y = __floats2bfloat162_rn(c, d);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&x), *reinterpret_cast<const uint32_t*>(&y));
}

// Statistics of a row held as NV float4 per thread (zero past the row's end, `in(i)` tells which are inside).
template <int kWarps, int NV, typename In>
__device__ __forceinline__ void norm_stats4(int kind, int C, float eps, float* red, const float4 (&v)[NV], In in, float& mean, float& inv) {
  mean = 0.f;
  if (kind == NB_NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    mean = block_sum<kWarps>(s, red) / (float)C;
  }
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (in(i)) {
      const float a = v[i].x - mean, b = v[i].y - mean, c = v[i].z - mean, d = v[i].w - mean;
      q += (a * a + b * b) + (c * c + d * d);
    }
  inv = 1.0f / sqrtf(block_sum<kWarps>(q, red + kWarps) / (float)C + eps);
}

template <typename TH, int NV>
__global__ void __launch_bounds__(kChainThreads) residual_norm_vec_kernel(float* __restrict__ x, const float* __restrict__ y,
                                                                          const float* __restrict__ wy, const float* __restrict__ w, int kind,
                                                                          float eps, TH* __restrict__ h, int ldh, int C) {
  __shared__ float red[4 * kChainWarps];
  pdl_enter();
  const int tid = threadIdx.x;
  float* xr = x + (size_t)blockIdx.x * C;
  const float* yr = y ? y + (size_t)blockIdx.x * C : nullptr;
  auto at = [&](int i) { return (i * kChainThreads + tid) * 4; };
  auto in = [&](int i) { return at(i) < C; };
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 v[NV];
  float mean, inv;
#pragma unroll
  for (int i = 0; i < NV; ++i) v[i] = in(i) ? *reinterpret_cast<const float4*>(xr + at(i)) : zero;
  if (yr) {
    float4 d[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) d[i] = in(i) ? *reinterpret_cast<const float4*>(yr + at(i)) : zero;
    norm_stats4<kChainWarps, NV>(kind, C, eps, red, d, in, mean, inv);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (in(i)) {
        const float4 g = __ldg(reinterpret_cast<const float4*>(wy + at(i)));
        v[i].x += (d[i].x - mean) * inv * g.x; v[i].y += (d[i].y - mean) * inv * g.y;
        v[i].z += (d[i].z - mean) * inv * g.z; v[i].w += (d[i].w - mean) * inv * g.w;
        *reinterpret_cast<float4*>(xr + at(i)) = v[i];
      }
  }
  if (h) {
    norm_stats4<kChainWarps, NV>(kind, C, eps, red + 2 * kChainWarps, v, in, mean, inv);
    TH* hr = h + (size_t)blockIdx.x * ldh;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (in(i)) {
        const float4 g = __ldg(reinterpret_cast<const float4*>(w + at(i)));
        store4(hr + at(i), (v[i].x - mean) * inv * g.x, (v[i].y - mean) * inv * g.y, (v[i].z - mean) * inv * g.z, (v[i].w - mean) * inv * g.w);
      }
  }
}

template <typename TH>
static int launch_residual_norm(float* x, const float* y, const float* wy, const float* w, int norm, float eps, TH* h, int ldh, int rows, int C,
                                cudaStream_t st) {
  const dim3 grid(rows), block(kChainThreads);
  const bool vec = C % 4 == 0 && ldh % 4 == 0 && C <= 8 * 1024 && (uintptr_t)x % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)wy % 16 == 0 &&
                   (uintptr_t)w % 16 == 0 && (uintptr_t)h % 16 == 0;
  if (!vec) return launch_pdl(residual_norm_kernel<TH>, grid, block, (size_t)C * 4, st, x, y, wy, w, norm, eps, h, ldh, C);
  if (C <= 1024) return launch_pdl(residual_norm_vec_kernel<TH, 1>, grid, block, 0, st, x, y, wy, w, norm, eps, h, ldh, C);
  if (C <= 2048) return launch_pdl(residual_norm_vec_kernel<TH, 2>, grid, block, 0, st, x, y, wy, w, norm, eps, h, ldh, C);
  if (C <= 4096) return launch_pdl(residual_norm_vec_kernel<TH, 4>, grid, block, 0, st, x, y, wy, w, norm, eps, h, ldh, C);
  return launch_pdl(residual_norm_vec_kernel<TH, 8>, grid, block, 0, st, x, y, wy, w, norm, eps, h, ldh, C);
}

// ---- hyper-connections (see nb_stream_args).  The coefficients sit in shared memory, in coef's order.
constexpr int kMaxCoef = 2 * NB_MAX_STREAMS + 1 + NB_MAX_STREAMS * NB_MAX_STREAMS;

struct StreamCoef {
  const float *read, *share, *mix;
  float direct;
  __device__ StreamCoef(const float* c, int S) : read(c), share(c + S + 1), mix(c + 2 * S + 1), direct(c[S]) {}
};

__device__ __forceinline__ float4 fma4(float a, const float4& b, const float4& c) {
  return make_float4(fmaf(a, b.x, c.x), fmaf(a, b.y, c.y), fmaf(a, b.z, c.z), fmaf(a, b.w, c.w));
}

// y = (y0 - mean0) inv0 w0 (+ the second branch) for one element or four.
__device__ __forceinline__ float branch(float y, float mean, float inv, float w) { return (y - mean) * inv * w; }
__device__ __forceinline__ float4 branch4(const float4& y, float mean, float inv, const float4& w) {
  return make_float4(branch(y.x, mean, inv, w.x), branch(y.y, mean, inv, w.y), branch(y.z, mean, inv, w.z), branch(y.w, mean, inv, w.w));
}

template <typename TH, int NV, int kS>   // C <= 1024 * NV, a multiple of 4; at most kS streams
__global__ void __launch_bounds__(kChainThreads) stream_norm_vec_kernel(const nb_stream_args p, TH* __restrict__ h, int ldh) {
  __shared__ float red[6 * kChainWarps], cf[kMaxCoef];
  const int tid = threadIdx.x, C = p.C, S = p.streams;
  for (int i = tid; i < 2 * S + 1 + S * S; i += kChainThreads) cf[i] = p.coef[i];
  pdl_enter();
  const float* x = p.x + (size_t)blockIdx.x * S * C;
  auto at = [&](int i) { return (i * kChainThreads + tid) * 4; };
  auto in = [&](int i) { return at(i) < C; };
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 v[kS][NV], y[NV];
#pragma unroll
  for (int s = 0; s < kS; ++s)
#pragma unroll
    for (int i = 0; i < NV; ++i) v[s][i] = s < S && in(i) ? *reinterpret_cast<const float4*>(x + (size_t)s * C + at(i)) : zero;
#pragma unroll
  for (int i = 0; i < NV; ++i) y[i] = zero;
  float mean, inv;
  auto add_branch = [&](const float* yr, const float* w, float* r) {
    float4 d[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) d[i] = in(i) ? *reinterpret_cast<const float4*>(yr + (size_t)blockIdx.x * C + at(i)) : zero;
    mean = 0.f; inv = 1.f;
    if (p.y_norm >= 0) norm_stats4<kChainWarps, NV>(p.y_norm, C, p.eps, r, d, in, mean, inv);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (in(i)) {
        const float4 b = branch4(d[i], mean, inv, __ldg(reinterpret_cast<const float4*>(w + at(i))));
        y[i].x += b.x; y[i].y += b.y; y[i].z += b.z; y[i].w += b.w;
      }
  };
  if (p.y0) add_branch(p.y0, p.w0, red);
  if (p.y1) add_branch(p.y1, p.w1, red + 2 * kChainWarps);
  __syncthreads();                       // the coefficients
  const StreamCoef c(cf, S);
  if (p.y0 && p.x_out) {
    float* xo = p.x_out + (size_t)blockIdx.x * S * C;
#pragma unroll
    for (int t = 0; t < kS; ++t)
      if (t < S) {
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (in(i)) {
            float4 r = make_float4(c.share[t] * y[i].x, c.share[t] * y[i].y, c.share[t] * y[i].z, c.share[t] * y[i].w);
#pragma unroll
            for (int s = 0; s < kS; ++s)
              if (s < S) r = fma4(c.mix[s * S + t], v[s][i], r);
            *reinterpret_cast<float4*>(xo + (size_t)t * C + at(i)) = r;
          }
      }
  }
  float4 u[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    u[i] = p.y0 ? make_float4(c.direct * y[i].x, c.direct * y[i].y, c.direct * y[i].z, c.direct * y[i].w) : zero;
#pragma unroll
    for (int s = 0; s < kS; ++s)
      if (s < S) u[i] = fma4(c.read[s], v[s][i], u[i]);
  }
  norm_stats4<kChainWarps, NV>(p.norm, C, p.eps, red + 4 * kChainWarps, u, in, mean, inv);
  TH* hr = h + (size_t)blockIdx.x * ldh;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (in(i)) {
      const float4 r = branch4(u[i], mean, inv, __ldg(reinterpret_cast<const float4*>(p.norm_w + at(i))));
      store4(hr + at(i), r.x, r.y, r.z, r.w);
    }
}

// The scalar form shared by the row kernel and the decode product: y in ys, then what the next sublayer reads, normed, through
// put(k, value).  Elements k are visited by the same thread throughout; us holds u.  Writes the streams of elements that
// `owns(k)`.  red: 6 * kWarps floats.
template <int kWarps, typename At, typename Owns, typename Put>
__device__ __forceinline__ void stream_row(const nb_stream_args& p, const float* x, float* xo, const float* y0, const float* y1, const float* cf,
                                           float* us, At at, float* ys, float* red, Owns owns, Put put) {
  const int C = p.C, S = p.streams, tid = threadIdx.x;
  const StreamCoef c(cf, S);
  float mean, inv;
  for (int k = tid; k < C; k += kWarps * 32) ys[k] = 0.f;
  for (int b = 0; b < 2; ++b) {
    const float *yr = b ? y1 : y0, *w = b ? p.w1 : p.w0;
    if (!yr) continue;
    mean = 0.f; inv = 1.f;
    if (p.y_norm >= 0)
      norm_stats<kWarps>(p.y_norm, C, p.eps, red + 2 * b * kWarps, [&](auto f) { for (int k = tid; k < C; k += kWarps * 32) f(yr[k]); }, mean, inv);
    for (int k = tid; k < C; k += kWarps * 32) ys[k] += branch(yr[k], mean, inv, w[k]);
  }
  for (int k = tid; k < C; k += kWarps * 32) {
    float v[NB_MAX_STREAMS], u = y0 ? c.direct * ys[k] : 0.f;
    for (int s = 0; s < S; ++s) { v[s] = x[(size_t)s * C + k]; u = fmaf(c.read[s], v[s], u); }
    if (y0 && xo && owns(k))
      for (int t = 0; t < S; ++t) {
        float r = c.share[t] * ys[k];
        for (int s = 0; s < S; ++s) r = fmaf(c.mix[s * S + t], v[s], r);
        xo[(size_t)t * C + k] = r;
      }
    us[at(k)] = u;
  }
  norm_stats<kWarps>(p.norm, C, p.eps, red + 4 * kWarps, [&](auto f) { for (int k = tid; k < C; k += kWarps * 32) f(us[at(k)]); }, mean, inv);
  for (int k = tid; k < C; k += kWarps * 32) put(k, branch(us[at(k)], mean, inv, p.norm_w[k]));
}

template <typename TH> __global__ void __launch_bounds__(kChainThreads) stream_norm_kernel(const nb_stream_args p, TH* __restrict__ h, int ldh) {
  extern __shared__ __align__(16) float row_s[];
  __shared__ float red[6 * kChainWarps], cf[kMaxCoef];
  const int S = p.streams, C = p.C;
  const size_t row = blockIdx.x;
  for (int i = threadIdx.x; i < 2 * S + 1 + S * S; i += kChainThreads) cf[i] = p.coef[i];
  pdl_enter();
  __syncthreads();
  stream_row<kChainWarps>(p, p.x + row * S * C, p.x_out ? p.x_out + row * S * C : nullptr, p.y0 ? p.y0 + row * C : nullptr,
                          p.y1 ? p.y1 + row * C : nullptr, cf, row_s, [](int k) { return k; }, row_s + C, red, [](int) { return true; },
                          [&](int k, float v) { h[row * ldh + k] = from_f<TH>(v); });
}

template <typename TH, int kS> static int launch_stream_norm_vec(const nb_stream_args& s, TH* h, int ldh, int rows, cudaStream_t st) {
  if (s.C <= 1024) return launch_pdl(stream_norm_vec_kernel<TH, 1, kS>, dim3(rows), dim3(kChainThreads), 0, st, s, h, ldh);
  if (s.C <= 2048) return launch_pdl(stream_norm_vec_kernel<TH, 2, kS>, dim3(rows), dim3(kChainThreads), 0, st, s, h, ldh);
  return launch_pdl(stream_norm_vec_kernel<TH, 4, kS>, dim3(rows), dim3(kChainThreads), 0, st, s, h, ldh);
}

template <typename TH> static int launch_stream_norm(const nb_stream_args& s, TH* h, int ldh, int rows, cudaStream_t st) {
  const uintptr_t ptrs = (uintptr_t)s.x | (uintptr_t)s.x_out | (uintptr_t)s.y0 | (uintptr_t)s.w0 | (uintptr_t)s.y1 | (uintptr_t)s.w1 |
                         (uintptr_t)s.norm_w | (uintptr_t)h;
  if (s.C % 4 == 0 && ldh % 4 == 0 && s.C <= 4096 && s.streams <= 4 && ptrs % 16 == 0)
    return s.streams <= 2 ? launch_stream_norm_vec<TH, 2>(s, h, ldh, rows, st) : launch_stream_norm_vec<TH, 4>(s, h, ldh, rows, st);
  return launch_pdl(stream_norm_kernel<TH>, dim3(rows), dim3(kChainThreads), (size_t)s.C * 8, st, s, h, ldh);
}

// ---- fp32 product: 64 x 64 output tile per CTA, 16 x 16 threads with 4 x 4 outputs each, k in steps of 16.
constexpr int kFT = 64, kFKS = 16;

__global__ void __launch_bounds__(256) linear_f32_kernel(const float* __restrict__ x, int ldx, const bf16* __restrict__ w, int ldw,
                                                         const float* __restrict__ bias, int act, float alpha, float limit, int M, int N,
                                                         int K, float* __restrict__ y, int ldy) {
  __shared__ float xs[kFKS][kFT + 4], ws[kFKS][kFT + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int m0 = blockIdx.y * kFT, n0 = blockIdx.x * kFT;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kFKS) {
    for (int i = tid; i < kFT * kFKS; i += 256) {
      const int r = i / kFKS, k = i % kFKS;
      xs[k][r] = (m0 + r < M && k0 + k < K) ? x[(size_t)(m0 + r) * ldx + k0 + k] : 0.f;
      ws[k][r] = (n0 + r < N && k0 + k < K) ? __bfloat162float(w[(size_t)(n0 + r) * ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFKS; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
  const int n = n0 + tx * 4;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = acc[i][j] + ((bias && n + j < N) ? bias[n + j] : 0.f);
    if (act != NB_ACT_NONE) {
#pragma unroll
      for (int j = 0; j < 4; j += 2)
        if (n + j + 1 < N) y[(size_t)m * ldy + ((n + j) >> 1)] = glu_f(act, alpha, limit, v[j], v[j + 1]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (n + j < N) y[(size_t)m * ldy + n + j] = v[j];
    }
  }
}

// ---- decode matvec.  A CTA owns a contiguous range of rows; the range, cut into items of one row x 256 columns (512
// bytes, 16 per lane), is dealt to the CTA's warps in equal contiguous runs, so every SM and every warp streams the
// same number of bytes whatever N and K are.  A row that lies in one run is finished by its warp; the parts of a row
// that runs share are added in warp order after a barrier: no atomics, bit-identical from run to run.  Each warp keeps
// 8 - 16 items in flight in registers and requests the first ones before the dependency wait.  (Eight warps per CTA, so that the next
// launch's CTA fits beside it, measured slower: too few bytes in flight.)
constexpr int kMvWarps = 16, kMvThreads = kMvWarps * 32, kMvBatch = 8;

struct MatvecParams {
  const uint4* w;
  const float *bias, *x, *delta, *delta_w, *norm_w;
  float *y, *x_out;
  float eps, alpha, limit;
  int N, K, ldw8;        // ldw8: row stride in 16-byte units
  short act, norm;
};

__device__ __forceinline__ uint4 ld_stream(const uint4* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// Hyper-connections in front of a decode product: h of one row into xs; every CTA computes the row, the streams behind the
// sublayer are written in equal shares.  ysm: C floats (NV = 0 only).
template <int NV, typename Slot>
__device__ __forceinline__ void stream_prologue(const nb_stream_args& p, float* xs, float* ysm, int padded, int bid, int ctas, Slot slot) {
  __shared__ float sred[6 * kMvWarps], cf[kMaxCoef];
  const int tid = threadIdx.x, C = p.C, S = p.streams;
  for (int i = tid; i < 2 * S + 1 + S * S; i += kMvThreads) cf[i] = p.coef[i];
  if constexpr (NV > 0) {
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto at = [&](int i) { return (i * kMvThreads + tid) * 4; };
    auto in = [&](int i) { return at(i) < C; };
    auto ld = [&](const float* q, int i) { return q && in(i) ? __ldg(reinterpret_cast<const float4*>(q + at(i))) : zero; };
    float4 nw[NV], w0[NV], w1[NV];
    if constexpr (NV <= 2) {
#pragma unroll
      for (int i = 0; i < NV; ++i) { nw[i] = ld(p.norm_w, i); w0[i] = ld(p.w0, i); w1[i] = ld(p.w1, i); }
    }
    pdl_enter();
    float4 a[NV], b[NV], u[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      a[i] = p.y0 && in(i) ? *reinterpret_cast<const float4*>(p.y0 + at(i)) : zero;
      b[i] = p.y1 && in(i) ? *reinterpret_cast<const float4*>(p.y1 + at(i)) : zero;
      u[i] = in(i) ? *reinterpret_cast<const float4*>(p.x + at(i)) : zero;
    }
    if constexpr (NV > 2) {
#pragma unroll
      for (int i = 0; i < NV; ++i) { nw[i] = ld(p.norm_w, i); w0[i] = ld(p.w0, i); w1[i] = ld(p.w1, i); }
    }
    __syncthreads();                   // the coefficients
    const StreamCoef c(cf, S);
#pragma unroll
    for (int i = 0; i < NV; ++i) u[i] = make_float4(c.read[0] * u[i].x, c.read[0] * u[i].y, c.read[0] * u[i].z, c.read[0] * u[i].w);
    for (int s = 1; s < S; ++s)
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (in(i)) u[i] = fma4(c.read[s], *reinterpret_cast<const float4*>(p.x + (size_t)s * C + at(i)), u[i]);
    float mean = 0.f, inv = 1.f;
    if (p.y0) {
      if (p.y_norm >= 0) norm_stats4<kMvWarps, NV>(p.y_norm, C, p.eps, sred, a, in, mean, inv);
#pragma unroll
      for (int i = 0; i < NV; ++i) a[i] = branch4(a[i], mean, inv, w0[i]);
      if (p.y1) {
        mean = 0.f; inv = 1.f;
        if (p.y_norm >= 0) norm_stats4<kMvWarps, NV>(p.y_norm, C, p.eps, sred + 2 * kMvWarps, b, in, mean, inv);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const float4 t = branch4(b[i], mean, inv, w1[i]);
          a[i].x += t.x; a[i].y += t.y; a[i].z += t.z; a[i].w += t.w;
        }
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        u[i] = fma4(c.direct, a[i], u[i]);
        if (in(i) && (i * kMvThreads + tid) % ctas == bid)
          for (int t = 0; t < S; ++t) {
            float4 r = make_float4(c.share[t] * a[i].x, c.share[t] * a[i].y, c.share[t] * a[i].z, c.share[t] * a[i].w);
            for (int s = 0; s < S; ++s) r = fma4(c.mix[s * S + t], *reinterpret_cast<const float4*>(p.x + (size_t)s * C + at(i)), r);
            *reinterpret_cast<float4*>(p.x_out + (size_t)t * C + at(i)) = r;
          }
      }
    }
    norm_stats4<kMvWarps, NV>(p.norm, C, p.eps, sred + 4 * kMvWarps, u, in, mean, inv);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (at(i) < padded) *reinterpret_cast<float4*>(xs + slot(at(i))) = in(i) ? branch4(u[i], mean, inv, nw[i]) : zero;
  } else {
    pdl_enter();
    for (int k = C + tid; k < padded; k += kMvThreads) xs[slot(k)] = 0.f;
    __syncthreads();
    stream_row<kMvWarps>(p, p.x, p.x_out, p.y0, p.y1, cf, xs, slot, ysm, sred, [&](int k) { return k % ctas == bid; },
                         [&](int k, float v) { xs[slot(k)] = v; });
  }
}

// NV: float4 of the row per thread in the prologue (K <= 2048 * NV, a multiple of 4), 0: any K.  The CTA is number `bid` of
// `ctas` on this product.  `sp`: hyper-connections in front (else not read).
template <int NV, bool kStreams>
__device__ __forceinline__ void matvec_body(const MatvecParams& p, const nb_stream_args& sp, const int bid, const int ctas) {
  extern __shared__ __align__(16) float mv_smem[];
  __shared__ float red[4 * kMvWarps], part_v[2 * kMvWarps];
  __shared__ int part_r[2 * kMvWarps];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int KC = (p.K + 255) >> 8;
  const int unit = p.act != NB_ACT_NONE ? 2 : 1;
  const int NU = p.N / unit;
  const int r0 = (int)((long long)NU * bid / ctas) * unit, r1 = (int)((long long)NU * (bid + 1) / ctas) * unit;
  const int R = r1 - r0, items = R * KC;
  const int i0 = (int)((long long)items * warp / kMvWarps), i1 = (int)((long long)items * (warp + 1) / kMvWarps);
  float* xs = mv_smem;                                  // per 256 columns: first halves of the lanes' eight values, then second halves
  float* ysum = xs + KC * 256;

  int lr = i0 / KC, lc = i0 - lr * KC, li = i0;         // next item to request
  const uint4* wp = p.w + (size_t)(r0 + lr) * p.ldw8;   // its row
  auto request = [&]() -> uint4 {
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (li < i1) {
      const int c8 = lc * 32 + lane;
      if (c8 < p.ldw8) v = ld_stream(wp + c8);
      ++li;
      if (++lc == KC) { lc = 0; wp += p.ldw8; }
    }
    return v;
  };
  uint4 cur[kMvBatch];
#pragma unroll
  for (int u = 0; u < kMvBatch; ++u) cur[u] = request();
  for (int r = tid; r < R; r += kMvThreads) ysum[r] = 0.f;
  if (tid < 2 * kMvWarps) part_r[tid] = -1;

  auto slot = [](int k) { return (k & ~255) + ((k & 4) << 5) + ((k & 255) >> 3) * 4 + (k & 3); };
  float mean, inv;
  if constexpr (kStreams) {
    stream_prologue<NV>(sp, xs, ysum + R, KC * 256, bid, ctas, slot);
  } else if constexpr (NV > 0) {
    // weights of the norms ahead of the wait, the vectors all at once behind it
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto at = [&](int i) { return (i * kMvThreads + tid) * 4; };
    auto in = [&](int i) { return at(i) < p.K; };
    float4 nw[NV], dw[NV], v[NV], d[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      nw[i] = (p.norm_w && in(i)) ? __ldg(reinterpret_cast<const float4*>(p.norm_w + at(i))) : zero;
      dw[i] = (p.delta && in(i)) ? __ldg(reinterpret_cast<const float4*>(p.delta_w + at(i))) : zero;
    }
    pdl_enter();
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      v[i] = in(i) ? *reinterpret_cast<const float4*>(p.x + at(i)) : zero;
      d[i] = (p.delta && in(i)) ? *reinterpret_cast<const float4*>(p.delta + at(i)) : zero;
    }
    if (p.delta) {
      norm_stats4<kMvWarps, NV>(p.norm, p.K, p.eps, red, d, in, mean, inv);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (in(i)) {
          v[i].x += (d[i].x - mean) * inv * dw[i].x; v[i].y += (d[i].y - mean) * inv * dw[i].y;
          v[i].z += (d[i].z - mean) * inv * dw[i].z; v[i].w += (d[i].w - mean) * inv * dw[i].w;
          if (bid == 0) *reinterpret_cast<float4*>(p.x_out + at(i)) = v[i];
        }
    }
    if (p.norm_w) {
      norm_stats4<kMvWarps, NV>(p.norm, p.K, p.eps, red + 2 * kMvWarps, v, in, mean, inv);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        v[i] = make_float4((v[i].x - mean) * inv * nw[i].x, (v[i].y - mean) * inv * nw[i].y, (v[i].z - mean) * inv * nw[i].z,
                           (v[i].w - mean) * inv * nw[i].w);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (at(i) < KC * 256) *reinterpret_cast<float4*>(xs + slot(at(i))) = in(i) ? v[i] : zero;
  } else {
    pdl_enter();
    auto each = [&](auto f) {
      for (int k = tid; k < p.K; k += kMvThreads) f(xs[slot(k)]);
    };
    for (int k = p.K + tid; k < KC * 256; k += kMvThreads) xs[slot(k)] = 0.f;
    if (p.delta) {
      for (int k = tid; k < p.K; k += kMvThreads) xs[slot(k)] = p.delta[k];
      norm_stats<kMvWarps>(p.norm, p.K, p.eps, red, each, mean, inv);
      for (int k = tid; k < p.K; k += kMvThreads) {
        const float v = p.x[k] + (xs[slot(k)] - mean) * inv * p.delta_w[k];
        if (bid == 0) p.x_out[k] = v;
        xs[slot(k)] = v;
      }
    } else {
      for (int k = tid; k < p.K; k += kMvThreads) xs[slot(k)] = p.x[k];
    }
    if (p.norm_w) {
      norm_stats<kMvWarps>(p.norm, p.K, p.eps, red + 2 * kMvWarps, each, mean, inv);
      for (int k = tid; k < p.K; k += kMvThreads) xs[slot(k)] = (xs[slot(k)] - mean) * inv * p.norm_w[k];
    }
  }
  __syncthreads();

  int ur = i0 / KC, uc = i0 - ur * KC;                  // next item to multiply
  int recs = 0;
  bool whole = uc == 0;                                 // the current row began in this run
  float acc = 0.f;
  for (int i = i0; i < i1; i += kMvBatch) {
    uint4 nxt[kMvBatch];
#pragma unroll
    for (int u = 0; u < kMvBatch; ++u) nxt[u] = request();
#pragma unroll
    for (int u = 0; u < kMvBatch; ++u) {
      if (i + u < i1) {
        const float4 a = *reinterpret_cast<const float4*>(xs + uc * 256 + lane * 4);
        const float4 b = *reinterpret_cast<const float4*>(xs + uc * 256 + 128 + lane * 4);
        const uint4 t = cur[u];
        acc = fmaf(bf_lo(t.x), a.x, acc); acc = fmaf(bf_hi(t.x), a.y, acc);
        acc = fmaf(bf_lo(t.y), a.z, acc); acc = fmaf(bf_hi(t.y), a.w, acc);
        acc = fmaf(bf_lo(t.z), b.x, acc); acc = fmaf(bf_hi(t.z), b.y, acc);
        acc = fmaf(bf_lo(t.w), b.z, acc); acc = fmaf(bf_hi(t.w), b.w, acc);
        const bool end_row = ++uc == KC;
        if (end_row || i + u + 1 == i1) {
          const float s = warp_sum(acc);
          if (lane == 0) {
            if (end_row && whole) {
              ysum[ur] = s;
            } else {                                    // at most the first and the last row of a run
              part_v[2 * warp + recs] = s;
              part_r[2 * warp + recs] = ur;
            }
          }
          if (!(end_row && whole)) ++recs;
          acc = 0.f;
          whole = true;
          if (end_row) { uc = 0; ++ur; }
        }
      }
    }
#pragma unroll
    for (int u = 0; u < kMvBatch; ++u) cur[u] = nxt[u];
  }
  __syncthreads();
  auto row_value = [&](int r) {
    float v = ysum[r];
#pragma unroll
    for (int j = 0; j < 2 * kMvWarps; ++j)
      if (part_r[j] == r) v += part_v[j];
    return v + (p.bias ? p.bias[r0 + r] : 0.f);
  };
  if (unit == 2) {
    for (int c = tid; c < R / 2; c += kMvThreads) p.y[(r0 >> 1) + c] = glu_f(p.act, p.alpha, p.limit, row_value(2 * c), row_value(2 * c + 1));
  } else {
    for (int r = tid; r < R; r += kMvThreads) p.y[r0 + r] = row_value(r);
  }
}

template <int NV> __global__ void __launch_bounds__(kMvThreads, 1) matvec_kernel(const MatvecParams p) {
  matvec_body<NV, false>(p, nb_stream_args{}, blockIdx.x, gridDim.x);
}
template <int NV> __global__ void __launch_bounds__(kMvThreads, 1) matvec_streams_kernel(const MatvecParams p, const nb_stream_args sp) {
  matvec_body<NV, true>(p, sp, blockIdx.x, gridDim.x);
}
// The first g0 CTAs work on one product, the others on the second.
template <int NV> __global__ void __launch_bounds__(kMvThreads, 1) matvec_pair_kernel(const MatvecParams a, const MatvecParams b, int g0) {
  const bool first = (int)blockIdx.x < g0;
  const MatvecParams p = first ? a : b;
  matvec_body<NV, false>(p, nb_stream_args{}, first ? blockIdx.x : blockIdx.x - g0, first ? g0 : gridDim.x - g0);
}

constexpr size_t kMvMaxSmem = 200 * 1024;

template <typename... KArgs, typename... Args> static int launch_matvec(void (*kernel)(KArgs...), bool (&done)[64], int G, size_t smem,
                                                                        cudaStream_t st, Args... args) {
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMvMaxSmem)) return record_cuda_error(e);
    done[dev & 63] = true;
  }
  return launch_pdl(kernel, dim3(G), dim3(kMvThreads), smem, st, args...);
}

// Argument checks and launch parameters of one product on at most `ctas` CTAs; smem: shared memory it needs.
static int matvec_params(const nb_matvec_args* a, int ctas, MatvecParams& p, int& G, size_t& smem) {
  if (!a || !a->w || !a->y || a->N < 1 || a->K < 1 || a->ldw < a->K) return NB_ERR_ARG;
  if (a->act < NB_ACT_NONE || a->act > NB_ACT_CLAMPED_GLU_PAIRS) return NB_ERR_ARG;
  const int unit = a->act != NB_ACT_NONE ? 2 : 1;
  if (a->N % unit) return NB_ERR_SHAPE;
  if ((uintptr_t)a->w % 16 || a->ldw % 8) return NB_ERR_ALIGN;
  G = std::min(ctas, a->N / unit);
  const int rows = ((a->N / unit + G - 1) / G) * unit, kc = (a->K + 255) / 256;
  smem = ((size_t)kc * 256 + rows) * 4;
  p.w = reinterpret_cast<const uint4*>(a->w);
  p.bias = a->bias; p.x = a->x; p.delta = a->delta; p.delta_w = a->delta_w; p.norm_w = a->norm_w;
  p.y = a->y; p.x_out = a->x_out;
  p.eps = a->eps; p.alpha = a->alpha; p.limit = a->limit; p.N = a->N; p.K = a->K; p.ldw8 = a->ldw / 8;
  p.act = (short)a->act; p.norm = (short)a->norm;
  return smem > kMvMaxSmem ? NB_ERR_SHAPE : NB_OK;
}

static bool aligned16(const void* a, const void* b = nullptr, const void* c = nullptr, const void* d = nullptr, const void* e = nullptr,
                      const void* f = nullptr, const void* g = nullptr) {
  return ((uintptr_t)a | (uintptr_t)b | (uintptr_t)c | (uintptr_t)d | (uintptr_t)e | (uintptr_t)f | (uintptr_t)g) % 16 == 0;
}

static int stream_check(const nb_stream_args* s) {
  if (!s || !s->x || !s->coef || !s->norm_w || s->C < 1 || s->streams < 1 || (s->y0 && !s->w0) || (s->y1 && (!s->w1 || !s->y0))) return NB_ERR_ARG;
  if (s->y_norm < -1 || s->y_norm > NB_NORM_LAYER || s->norm < NB_NORM_RMS || s->norm > NB_NORM_LAYER) return NB_ERR_ARG;
  return s->streams > NB_MAX_STREAMS ? NB_ERR_SHAPE : NB_OK;
}

}  // namespace nb

using namespace nb;

extern "C" int nb_embed_scaled(const void* table_bf16, const int64_t* token, int rows, int V, int C, float scale, int streams, float* x,
                               void* stream) {
  if (!table_bf16 || !token || !x || rows < 1 || V < 1 || C < 1 || streams < 1) return NB_ERR_ARG;
  if (int rc = check_device()) return rc;
  return launch_pdl(embed_scaled_kernel, dim3(rows), dim3(256), 0, (cudaStream_t)stream, reinterpret_cast<const bf16*>(table_bf16),
                    reinterpret_cast<const long long*>(token), x, V, C, scale, streams);
}

extern "C" int nb_residual_norm(float* x, const float* y, const float* wy, const float* w, int norm, float eps, void* h, int h_dtype,
                                int ldh, int rows, int C, void* stream) {
  if (!x || (y && !wy) || (h && !w) || (!y && !h) || rows < 1 || C < 1 || (h && ldh < C)) return NB_ERR_ARG;
  if ((norm != NB_NORM_RMS && norm != NB_NORM_LAYER) || (h_dtype != NB_BF16 && h_dtype != NB_F32)) return NB_ERR_ARG;
  if (C > 12 * 1024) return NB_ERR_SHAPE;   // the row sits in shared memory
  if (int rc = check_device()) return rc;
  return h_dtype == NB_BF16
             ? launch_residual_norm(x, y, wy, w, norm, eps, reinterpret_cast<bf16*>(h), ldh, rows, C, (cudaStream_t)stream)
             : launch_residual_norm(x, y, wy, w, norm, eps, reinterpret_cast<float*>(h), ldh, rows, C, (cudaStream_t)stream);
}

extern "C" int nb_linear_f32(const float* x, int ldx, const void* w, int ldw, const float* bias, int act, float alpha, float limit, int M,
                             int N, int K, float* y, int ldy, void* stream) {
  if (!x || !w || !y || M < 1 || N < 1 || K < 1 || ldx < K || ldw < K) return NB_ERR_ARG;
  if (act < NB_ACT_NONE || act > NB_ACT_CLAMPED_GLU_PAIRS) return NB_ERR_ARG;
  if (act != NB_ACT_NONE && N % 2) return NB_ERR_SHAPE;
  if (ldy < (act != NB_ACT_NONE ? N / 2 : N)) return NB_ERR_ARG;
  if ((M + kFT - 1) / kFT > 65535) return NB_ERR_SHAPE;
  if (int rc = check_device()) return rc;
  linear_f32_kernel<<<dim3((N + kFT - 1) / kFT, (M + kFT - 1) / kFT), 256, 0, (cudaStream_t)stream>>>(
      x, ldx, reinterpret_cast<const bf16*>(w), ldw, bias, act, alpha, limit, M, N, K, y, ldy);
  return check_launch();
}

extern "C" int nb_stream_norm(const nb_stream_args* s, void* h, int h_dtype, int ldh, int rows, void* stream) {
  if (int rc = stream_check(s)) return rc;
  if (!h || rows < 1 || ldh < s->C || (h_dtype != NB_BF16 && h_dtype != NB_F32)) return NB_ERR_ARG;
  if (s->C > 6 * 1024) return NB_ERR_SHAPE;   // two rows sit in shared memory
  if (int rc = check_device()) return rc;
  return h_dtype == NB_BF16 ? launch_stream_norm(*s, reinterpret_cast<bf16*>(h), ldh, rows, (cudaStream_t)stream)
                            : launch_stream_norm(*s, reinterpret_cast<float*>(h), ldh, rows, (cudaStream_t)stream);
}

extern "C" int nb_matvec_bf16(const nb_matvec_args* a, void* stream) {
  if (!a || !a->x) return NB_ERR_ARG;
  if (a->delta && (!a->delta_w || !a->x_out || !a->norm_w || a->x_out == a->x)) return NB_ERR_ARG;
  if (a->norm != NB_NORM_RMS && a->norm != NB_NORM_LAYER) return NB_ERR_ARG;
  MatvecParams p;
  int G;
  size_t smem;
  if (int rc = matvec_params(a, 1 << 30, p, G, smem); rc && rc != NB_ERR_SHAPE) return rc;   // arguments, before a device is asked for
  if (a->act != NB_ACT_NONE && a->N % 2) return NB_ERR_SHAPE;
  if (int rc = check_device()) return rc;
  if (int rc = matvec_params(a, sm_count(), p, G, smem)) return rc;
  const cudaStream_t st = (cudaStream_t)stream;
  const bool vec = a->K % 4 == 0 && aligned16(a->x, a->delta, a->delta_w, a->norm_w, a->x_out);
  static bool done[4][64] = {};
  if (vec && a->K <= 2048) return launch_matvec(matvec_kernel<1>, done[0], G, smem, st, p);
  if (vec && a->K <= 4096) return launch_matvec(matvec_kernel<2>, done[1], G, smem, st, p);
  if (vec && a->K <= 8192) return launch_matvec(matvec_kernel<4>, done[2], G, smem, st, p);
  return launch_matvec(matvec_kernel<0>, done[3], G, smem, st, p);
}

extern "C" int nb_matvec_streams(const nb_matvec_args* a, const nb_stream_args* s, void* stream) {
  if (int rc = stream_check(s)) return rc;
  MatvecParams p;
  int G;
  size_t smem;
  if (int rc = matvec_params(a, 1 << 30, p, G, smem); rc && rc != NB_ERR_SHAPE) return rc;
  if (s->C != a->K || s->x_out == s->x || (s->y0 && !s->x_out)) return NB_ERR_ARG;
  if (a->act != NB_ACT_NONE && a->N % 2) return NB_ERR_SHAPE;
  if (int rc = check_device()) return rc;
  if (int rc = matvec_params(a, sm_count(), p, G, smem)) return rc;
  const cudaStream_t st = (cudaStream_t)stream;
  const bool vec = a->K % 4 == 0 && aligned16(s->x, s->x_out, s->y0, s->w0, s->y1, s->w1, s->norm_w);
  static bool done[4][64] = {};
  if (vec && a->K <= 2048) return launch_matvec(matvec_streams_kernel<1>, done[0], G, smem, st, p, *s);
  if (vec && a->K <= 4096) return launch_matvec(matvec_streams_kernel<2>, done[1], G, smem, st, p, *s);
  if (vec && a->K <= 8192) return launch_matvec(matvec_streams_kernel<4>, done[2], G, smem, st, p, *s);
  smem += (size_t)a->K * 4;            // the sublayer's result, beside the row
  if (smem > kMvMaxSmem) return NB_ERR_SHAPE;
  return launch_matvec(matvec_streams_kernel<0>, done[3], G, smem, st, p, *s);
}

extern "C" int nb_matvec_pair(const nb_matvec_args* a, const nb_matvec_args* b, void* stream) {
  MatvecParams pa, pb;
  int ga, gb;
  size_t sa, sb;
  for (const nb_matvec_args* q : {a, b}) {
    if (!q || !q->x || q->delta || q->norm_w) return NB_ERR_ARG;
    if (int rc = matvec_params(q, 1 << 30, pa, ga, sa); rc && rc != NB_ERR_SHAPE) return rc;
    if (q->act != NB_ACT_NONE && q->N % 2) return NB_ERR_SHAPE;
  }
  if (int rc = check_device()) return rc;
  // CTAs in proportion to the bytes
  const int sms = sm_count();
  const double wa = (double)a->N * a->ldw, wb = (double)b->N * b->ldw;
  const int first = std::max(1, std::min(sms - 1, (int)(sms * wa / (wa + wb) + 0.5)));
  if (int rc = matvec_params(a, first, pa, ga, sa)) return rc;
  if (int rc = matvec_params(b, sms - first, pb, gb, sb)) return rc;
  const cudaStream_t st = (cudaStream_t)stream;
  const size_t smem = std::max(sa, sb);
  const int K = std::max(a->K, b->K), G = ga + gb;
  const bool vec = a->K % 4 == 0 && b->K % 4 == 0 && aligned16(a->x, b->x);
  static bool done[4][64] = {};
  if (vec && K <= 2048) return launch_matvec(matvec_pair_kernel<1>, done[0], G, smem, st, pa, pb, ga);
  if (vec && K <= 4096) return launch_matvec(matvec_pair_kernel<2>, done[1], G, smem, st, pa, pb, ga);
  if (vec && K <= 8192) return launch_matvec(matvec_pair_kernel<4>, done[2], G, smem, st, pa, pb, ga);
  return launch_matvec(matvec_pair_kernel<0>, done[3], G, smem, st, pa, pb, ga);
}
