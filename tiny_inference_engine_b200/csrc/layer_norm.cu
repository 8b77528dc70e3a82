// Norms that add a sum of sublayer outputs to the residual stream on their way (with mean and variance, or by the root mean
// square), and sums into the stream outside a norm.
//
//   add_layer_norm   x += the terms (float, in place, added in order; up to four, each a tensor in the compute type or the
//                    partial sums of a split product, times a factor), then
//                    out = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b in the compute type. With `rows`, out[i]
//                    comes from row rows[i] and x is left as it is. One block a row: the row stays in registers between
//                    the sum of the terms, the mean and the squared deviations.
//   add_terms_rmsnorm  the same without a mean and a bias: out = x / sqrt(mean(x^2) + eps) * w.
//   stream_add       x += the terms, then + other (float rows), then + vec (one float row for every row); any may be absent.
#include <math.h>

#include "terms.cuh"

namespace tie {

// CENTER: with mean and bias; otherwise the root mean square alone.
template <typename T, int NV, bool CENTER>
__global__ void __launch_bounds__(1024) add_layer_norm_vec4_kernel(float* __restrict__ x, Terms terms, const int* __restrict__ rows,
                                                                   const float* __restrict__ w, const float* __restrict__ bias, float eps,
                                                                   T* __restrict__ out, int D) {
  pdl_sync();
  __shared__ float scratch[33];
  const long long r = rows ? rows[blockIdx.x] : blockIdx.x;
  float v[NV][4];
  float sum = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (threadIdx.x + i * blockDim.x) * 4;
    if (d < D) {
      load4(x + r * D + d, v[i]);
      for (int k = 0; k < terms.n; ++k) term_add4<T>(terms.t[k], r * D + d, v[i]);
      if (rows == nullptr && terms.n > 0) store4(x + r * D + d, v[i]);
      if constexpr (CENTER) sum += (v[i][0] + v[i][1]) + (v[i][2] + v[i][3]);
    }
  }
  const float mean = CENTER ? block_sum(sum, scratch) / static_cast<float>(D) : 0.0f;
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    if ((threadIdx.x + i * blockDim.x) * 4 < D) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if constexpr (CENTER) v[i][e] -= mean;
        ss = fmaf(v[i][e], v[i][e], ss);
      }
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(D) + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (threadIdx.x + i * blockDim.x) * 4;
    if (d < D) {
      float ww[4], bb[4], o[4];
      load4(w + d, ww);
      if constexpr (CENTER) load4(bias + d, bb);
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] = CENTER ? fmaf(v[i][e] * inv, ww[e], bb[e]) : (v[i][e] * inv) * ww[e];
      store4(out + static_cast<long long>(blockIdx.x) * D + d, o);
    }
  }
}

// Any width: the row waits in shared memory.
template <typename T, bool CENTER>
__global__ void __launch_bounds__(256) add_layer_norm_kernel(float* __restrict__ x, Terms terms, const int* __restrict__ rows,
                                                             const float* __restrict__ w, const float* __restrict__ bias, float eps,
                                                             T* __restrict__ out, int D) {
  pdl_sync();
  __shared__ float scratch[33];
  extern __shared__ float row[];
  const long long r = rows ? rows[blockIdx.x] : blockIdx.x;
  float sum = 0.0f;
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    float v = x[r * D + d];
    for (int k = 0; k < terms.n; ++k) v += term_at<T>(terms.t[k], r * D + d);
    if (rows == nullptr && terms.n > 0) x[r * D + d] = v;
    row[d] = v;
    sum += v;
  }
  const float mean = CENTER ? block_sum(sum, scratch) / static_cast<float>(D) : 0.0f;
  float ss = 0.0f;
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    const float v = row[d] - mean;
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(D) + eps);
  for (int d = threadIdx.x; d < D; d += blockDim.x)
    st(out + static_cast<long long>(blockIdx.x) * D + d, CENTER ? fmaf((row[d] - mean) * inv, w[d], bias[d]) : (row[d] * inv) * w[d]);
}

template <typename T>
__global__ void __launch_bounds__(256) stream_add_kernel(float* __restrict__ x, Terms terms, const float* __restrict__ other,
                                                         const float* __restrict__ vec, long long total, int D) {
  pdl_sync();
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    float v = x[i];
    for (int k = 0; k < terms.n; ++k) v += term_at<T>(terms.t[k], i);
    if (other != nullptr) v += other[i];
    if (vec != nullptr) v += vec[i % D];
    x[i] = v;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) stream_add_vec4_kernel(float* __restrict__ x, Terms terms, const float* __restrict__ other,
                                                              const float* __restrict__ vec, long long total4, int D) {
  pdl_sync();
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total4;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long at = i * 4;
    float v[4], o[4] = {0.0f, 0.0f, 0.0f, 0.0f}, w[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    load4(x + at, v);
    if (other != nullptr) load4(other + at, o);
    if (vec != nullptr) load4(vec + at % D, w);
    for (int k = 0; k < terms.n; ++k) term_add4<T>(terms.t[k], at, v);
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = (v[e] + o[e]) + w[e];
    store4(x + at, v);
  }
}

}  // namespace tie

using namespace tie;

// A term travels as (tensor, partial sums, stride, splits, factor); kMaxTerms of them, absent ones all zero.
#define TIE_TERM(k) const void *t##k, const float *p##k, long long s##k, int z##k, float c##k
#define TIE_TERMS TIE_TERM(0), TIE_TERM(1), TIE_TERM(2), TIE_TERM(3)

static Terms pack_terms(TIE_TERMS) {
  const Term all[kMaxTerms] = {{t0, p0, s0, z0, c0}, {t1, p1, s1, z1, c1}, {t2, p2, s2, z2, c2}, {t3, p3, s3, z3, c3}};
  Terms terms{};
  for (const Term& t : all)
    if (t.tensor != nullptr || t.partial != nullptr) terms.t[terms.n++] = t;
  return terms;
}

template <typename T, bool CENTER>
static int launch_add_layer_norm(float* x, const Terms& terms, const int* rows, const float* w, const float* bias, float eps, void* out,
                                 int n, int D, cudaStream_t s) {
  T* o = static_cast<T*>(out);
  auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (D % 4 == 0 && D <= 16384 && on16(x) && on16(w) && on16(bias) && on16(out) && terms_on16(terms)) {
    const int pieces = D / 4;
    int threads = n <= 512 ? 1024 : 256;      // few rows (decode): many threads a row keep the latency short
    while (threads < 1024 && pieces > 4 * threads) threads *= 2;
    while (threads > 32 && threads / 2 >= pieces) threads /= 2;
    const int nv = (pieces + threads - 1) / threads;
    if (nv <= 1) TIE_LAUNCH((add_layer_norm_vec4_kernel<T, 1, CENTER>), n, threads, 0, s, x, terms, rows, w, bias, eps, o, D);
    else if (nv <= 2) TIE_LAUNCH((add_layer_norm_vec4_kernel<T, 2, CENTER>), n, threads, 0, s, x, terms, rows, w, bias, eps, o, D);
    else TIE_LAUNCH((add_layer_norm_vec4_kernel<T, 4, CENTER>), n, threads, 0, s, x, terms, rows, w, bias, eps, o, D);
    TIE_RETURN_LAUNCH("add_layer_norm");
  }
  const size_t smem = static_cast<size_t>(D) * sizeof(float);
  TIE_REQUIRE(smem <= 200 * 1024, "add_layer_norm: a row of %d exceeds the kernel's shared memory", D);
  if (smem > 48 * 1024) {
    if (cudaFuncSetAttribute(add_layer_norm_kernel<T, CENTER>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess) {
      set_error("add_layer_norm: cannot reserve %zu bytes of shared memory", smem);
      return kCudaError;
    }
  }
  TIE_LAUNCH((add_layer_norm_kernel<T, CENTER>), n, 256, smem, s, x, terms, rows, w, bias, eps, o, D);
  TIE_RETURN_LAUNCH("add_layer_norm");
}

TIE_API int tie_add_layer_norm(int dtype, float* x, TIE_TERMS, const int* rows, const float* w, const float* bias, float eps, void* out,
                               int n, int D, cudaStream_t s) {
  TIE_REQUIRE(n >= 0 && D > 0, "add_layer_norm: bad sizes n=%d D=%d", n, D);
  if (n == 0) return kOk;
  const Terms terms = pack_terms(t0, p0, s0, z0, c0, t1, p1, s1, z1, c1, t2, p2, s2, z2, c2, t3, p3, s3, z3, c3);
  if (dtype == TIE_F32) return launch_add_layer_norm<float, true>(x, terms, rows, w, bias, eps, out, n, D, s);
  if (dtype == TIE_BF16) return launch_add_layer_norm<__nv_bfloat16, true>(x, terms, rows, w, bias, eps, out, n, D, s);
  set_error("unknown dtype code %d", dtype);
  return kBadArgument;
}

TIE_API int tie_add_terms_rmsnorm(int dtype, float* x, TIE_TERMS, const int* rows, const float* w, float eps, void* out, int n, int D,
                                  cudaStream_t s) {
  TIE_REQUIRE(n >= 0 && D > 0, "add_terms_rmsnorm: bad sizes n=%d D=%d", n, D);
  if (n == 0) return kOk;
  const Terms terms = pack_terms(t0, p0, s0, z0, c0, t1, p1, s1, z1, c1, t2, p2, s2, z2, c2, t3, p3, s3, z3, c3);
  if (dtype == TIE_F32) return launch_add_layer_norm<float, false>(x, terms, rows, w, nullptr, eps, out, n, D, s);
  if (dtype == TIE_BF16) return launch_add_layer_norm<__nv_bfloat16, false>(x, terms, rows, w, nullptr, eps, out, n, D, s);
  set_error("unknown dtype code %d", dtype);
  return kBadArgument;
}

TIE_API int tie_stream_add(int dtype, float* x, TIE_TERMS, const float* other, const float* vec, int n, int D, cudaStream_t s) {
  TIE_REQUIRE(n >= 0 && D > 0, "stream_add: bad sizes n=%d D=%d", n, D);
  if (n == 0) return kOk;
  const Terms terms = pack_terms(t0, p0, s0, z0, c0, t1, p1, s1, z1, c1, t2, p2, s2, z2, c2, t3, p3, s3, z3, c3);
  const long long total = static_cast<long long>(n) * D;
  const int blocks = static_cast<int>(min(static_cast<long long>(148 * 8), (total + 255) / 256));
  auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (D % 4 == 0 && on16(x) && on16(other) && on16(vec) && terms_on16(terms) && (dtype == TIE_F32 || dtype == TIE_BF16)) {
    const int threads = total / 4 < 148 * 256 ? 64 : 256;      // few rows: spread them over the SMs
    const int blocks4 = static_cast<int>(min(static_cast<long long>(148 * 8), (total / 4 + threads - 1) / threads));
    if (dtype == TIE_F32) TIE_LAUNCH((stream_add_vec4_kernel<float>), blocks4, threads, 0, s, x, terms, other, vec, total / 4, D);
    else TIE_LAUNCH((stream_add_vec4_kernel<__nv_bfloat16>), blocks4, threads, 0, s, x, terms, other, vec, total / 4, D);
    TIE_RETURN_LAUNCH("stream_add");
  }
  if (dtype == TIE_F32) {
    TIE_LAUNCH((stream_add_kernel<float>), blocks, 256, 0, s, x, terms, other, vec, total, D);
  } else if (dtype == TIE_BF16) {
    TIE_LAUNCH((stream_add_kernel<__nv_bfloat16>), blocks, 256, 0, s, x, terms, other, vec, total, D);
  } else {
    set_error("unknown dtype code %d", dtype);
    return kBadArgument;
  }
  TIE_RETURN_LAUNCH("stream_add");
}
