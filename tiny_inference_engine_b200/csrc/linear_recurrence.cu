// What stands around the recurrence S <- diag(decay) S + k u^T, o = S^T q (delta_rule.cu in its plain mode) for two
// mixers that have no delta correction:
//
//   gated linear attention   q, k, v straight from their projections (q scaled), a decay per head and key channel,
//                            decay = sigmoid(z)^(1/tau) = exp(-softplus(-z) / tau), z the decay projection plus its bias;
//                            read-out: o / rms(o) * w * act(gate) per head.
//   state-space duality      x, B and C behind a short causal convolution with bias and SiLU; a step size per head,
//                            dt = softplus(raw + bias); decay = exp(-exp(A_log) dt) for the whole head; the write is
//                            dt * B x^T; read-out: (o + D x) * silu(z), normed in equal parts of the row, times w.
//
// Kernels (float inside; T is the storage type of the projections and of the outputs that feed a product):
//   gla_prep      one block per token.
//   act_split     q, k, v behind an activation as float rows (linear attention with constant decays).
//   rope_split    q and k rotated, k times a factor, and v, as float rows (one block per token; a token's angles are formed once).
//   ssd_prep      one block per (token, unit): units are the heads of C, of B and of x, and one for the step sizes.
//                 The convolution's first taps - 1 inputs come from the rows ahead in the step or from the tail that
//                 the sequence's state slot keeps behind S (channels in the order C, B, x).
//   head_norm_gate  one warp per (token, head).
//   ssd_out       one block per (token, part of the row).
#include <math.h>

#include "rotation.cuh"

namespace tie {

__device__ __forceinline__ float lr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float lr_softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

template <typename T>
__global__ void __launch_bounds__(256) gla_prep_kernel(const T* __restrict__ proj, long long stride, int q_off, int k_off,
                                                       int v_off, int nqk, int nv, float q_scale, float inv_tau,
                                                       const float* __restrict__ z_bias, float* __restrict__ qn,
                                                       float* __restrict__ kn, float* __restrict__ vn,
                                                       float* __restrict__ decay, long long decay_stride) {
  pdl_sync();
  const long long t = blockIdx.x;
  const T* row = proj + t * stride;
  for (int c = threadIdx.x; c < nqk; c += blockDim.x) {
    qn[t * nqk + c] = ld(row + q_off + c) * q_scale;
    kn[t * nqk + c] = ld(row + k_off + c);
    float* a = decay + t * decay_stride + c;
    const float z = *a + (z_bias ? z_bias[c] : 0.0f);
    *a = expf(-lr_softplus(-z) * inv_tau);
  }
  for (int c = threadIdx.x; c < nv; c += blockDim.x) vn[t * nv + c] = ld(row + v_off + c);
}

// q, k and v behind an activation (1: the SiLU), as float rows.
template <typename T>
__global__ void __launch_bounds__(256) act_split_kernel(const T* __restrict__ proj, long long stride, int q_off, int k_off, int v_off,
                                                        int nqk, int nv, int act, float* __restrict__ qn, float* __restrict__ kn,
                                                        float* __restrict__ vn, long long total) {
  pdl_sync();
  const int width = 2 * nqk + nv;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / width;
    const int c = static_cast<int>(i - t * width);
    const int at = c < nqk ? q_off + c : (c < 2 * nqk ? k_off + c - nqk : v_off + c - 2 * nqk);
    const float z = ld(proj + t * stride + at);
    float* dst = c < nqk ? qn + t * nqk + c : (c < 2 * nqk ? kn + t * nqk + c - nqk : vn + t * nv + c - 2 * nqk);
    *dst = act == 1 ? z * lr_sigmoid(z) : z;
  }
}

// The same, 16 bytes of the projection a thread: sections and sizes in whole vectors.
template <typename T>
__global__ void __launch_bounds__(256) act_split_vec_kernel(const T* __restrict__ proj, long long stride, int q_off, int k_off, int v_off,
                                                            int nqk, int nv, int act, float* __restrict__ qn, float* __restrict__ kn,
                                                            float* __restrict__ vn, long long total) {
  pdl_sync();
  constexpr int V = Vec16<T>::N;
  const int pieces = (2 * nqk + nv) / V;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / pieces;
    const int c = static_cast<int>(i - t * pieces) * V;
    const int at = c < nqk ? q_off + c : (c < 2 * nqk ? k_off + c - nqk : v_off + c - 2 * nqk);
    float* dst = c < nqk ? qn + t * nqk + c : (c < 2 * nqk ? kn + t * nqk + c - nqk : vn + t * nv + c - 2 * nqk);
    Vec16<T> z;
    z.load(proj + t * stride + at);
#pragma unroll
    for (int e = 0; e < V; e += 4) {
      float o[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) o[k] = act == 1 ? z.v[e + k] * lr_sigmoid(z.v[e + k]) : z.v[e + k];
      store4(dst + e, o);
    }
  }
}

// One block per token: cos and sin of the token's angles into shared memory, then q and k heads with their first turn.rot
// dimensions rotated (k times k_scale) and v, as float rows. Heads' columns in pieces of four where everything is aligned.
template <typename T>
__global__ void __launch_bounds__(256) rope_split_kernel(const T* __restrict__ proj, long long stride, int q_off, int k_off, int v_off,
                                                         int heads, int dim, int nv, Rotation turn, const int* __restrict__ positions,
                                                         float k_scale, float* __restrict__ qn, float* __restrict__ kn,
                                                         float* __restrict__ vn, int wide) {
  pdl_sync();
  extern __shared__ float cs[];              // [rot / 2] cosines, [rot / 2] sines
  const long long t = blockIdx.x;
  const int half = turn.rot / 2, nqk = heads * dim;
  for (int i = threadIdx.x; i < half; i += blockDim.x) turn.angle(positions[t], i, cs[i], cs[half + i]);
  __syncthreads();
  const T* row = proj + t * stride;
  float* qd = qn + t * nqk;
  float* kd = kn + t * nqk;
  if (wide) {                                // dim, nv and (halves) rot / 2 or (neighbours) rot in pieces of four
    const int per = dim / 4, items = 2 * heads * per;
    for (int it = threadIdx.x; it < items; it += blockDim.x) {
      const bool is_k = it >= heads * per;
      const int in = is_k ? it - heads * per : it, h = in / per, d = (in % per) * 4;
      const T* src = row + (is_k ? k_off : q_off) + h * dim;
      float* dst = (is_k ? kd : qd) + h * dim;
      const float c = is_k ? k_scale : 1.0f;
      float u[4];
      load4(src + d, u);
      if (d >= turn.rot) {
#pragma unroll
        for (int e = 0; e < 4; ++e) u[e] *= c;
        store4(dst + d, u);
      } else if (turn.neighbours) {
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const float cc = cs[(d + e) / 2], ss = cs[half + (d + e) / 2], a = u[e], b = u[e + 1];
          u[e] = c * (a * cc - b * ss);
          u[e + 1] = c * (b * cc + a * ss);
        }
        store4(dst + d, u);
      } else if (d < half) {                 // this thread makes both members of its four pairs
        float v[4], a[4], b[4];
        load4(src + d + half, v);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float cc = cs[d + e], ss = cs[half + d + e];
          a[e] = c * (u[e] * cc - v[e] * ss);
          b[e] = c * (v[e] * cc + u[e] * ss);
        }
        store4(dst + d, a);
        store4(dst + d + half, b);
      }
    }
    for (int d = threadIdx.x * 4; d < nv; d += blockDim.x * 4) {
      float u[4];
      load4(row + v_off + d, u);
      store4(vn + t * nv + d, u);
    }
    return;
  }
  const int rest = dim - turn.rot, per = half + rest;      // pairs, then the dimensions that pass
  for (int it = threadIdx.x; it < 2 * heads * per; it += blockDim.x) {
    const bool is_k = it >= heads * per;
    const int in = is_k ? it - heads * per : it, h = in / per, i = in % per;
    const T* src = row + (is_k ? k_off : q_off) + h * dim;
    float* dst = (is_k ? kd : qd) + h * dim;
    const float c = is_k ? k_scale : 1.0f;
    if (i < half) {
      const int j1 = turn.first(i), j2 = turn.second(i);
      const float a = ld(src + j1), b = ld(src + j2), cc = cs[i], ss = cs[half + i];
      dst[j1] = c * (a * cc - b * ss);
      dst[j2] = c * (b * cc + a * ss);
    } else {
      const int d = turn.rot + i - half;
      dst[d] = c * ld(src + d);
    }
  }
  for (int d = threadIdx.x; d < nv; d += blockDim.x) vn[t * nv + d] = ld(row + v_off + d);
}

struct SsdShape {
  int heads, groups, state, vdim, taps;
};

template <typename T>
__global__ void __launch_bounds__(128) ssd_prep_kernel(const T* __restrict__ proj, long long stride, int c_off, int b_off,
                                                       int x_off, int dt_off, const float* __restrict__ conv_w,
                                                       const float* __restrict__ conv_b, const float* __restrict__ state,
                                                       long long state_stride, long long conv_state_off,
                                                       const int* __restrict__ seq_of_row,
                                                       const int* __restrict__ query_start,
                                                       const int* __restrict__ state_slots, SsdShape sh,
                                                       const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                                                       float* __restrict__ cn, float* __restrict__ bn,
                                                       float* __restrict__ xn, float* __restrict__ dt,
                                                       float* __restrict__ decay) {
  pdl_sync();
  const int t = blockIdx.x, unit = blockIdx.y;
  const int G = sh.groups, H = sh.heads, N = sh.state, vdim = sh.vdim, taps = sh.taps;
  const int ngn = G * N, nv = H * vdim, C = 2 * ngn + nv;
  const T* row = proj + static_cast<long long>(t) * stride;
  if (unit == 2 * G + H) {
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
      const float step = lr_softplus(ld(row + dt_off + h) + dt_bias[h]);
      dt[static_cast<long long>(t) * H + h] = step;
      decay[static_cast<long long>(t) * H + h] = expf(-expf(a_log[h]) * step);
    }
    return;
  }
  const int s = seq_of_row[t];
  const int j = t - query_start[s];          // tokens of this sequence ahead of this one in the step
  const int slot = state_slots[s];
  const float* tail = slot >= 0 ? state + slot * state_stride + conv_state_off : nullptr;
  const bool is_x = unit >= 2 * G;
  const int width = is_x ? vdim : N;
  const int c0 = is_x ? 2 * ngn + (unit - 2 * G) * vdim : unit * N;      // the unit's first channel of all C
  float* dst = is_x ? xn + static_cast<long long>(t) * nv + (unit - 2 * G) * vdim
                    : (unit < G ? cn + static_cast<long long>(t) * ngn + unit * N
                                : bn + static_cast<long long>(t) * ngn + (unit - G) * N);
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    const int c = c0 + d;
    const int col = c < ngn ? c_off + c : (c < 2 * ngn ? b_off + (c - ngn) : x_off + (c - 2 * ngn));
    float y = conv_b ? conv_b[c] : 0.0f;
    for (int i = 0; i < taps; ++i) {
      const int back = taps - 1 - i;         // this tap's input is `back` tokens ahead of the current one
      float in;
      if (back <= j) in = ld(row - static_cast<long long>(back) * stride + col);
      else in = tail ? tail[static_cast<long long>(j + i) * C + c] : 0.0f;
      y = fmaf(conv_w[c * taps + i], in, y);
    }
    dst[d] = y * lr_sigmoid(y);
  }
}

// out[t, h] = (o[t, h] / rms(o[t, h])) * w * act(gate[t, h]) (w null: no weight); act 0: sigmoid, 1: silu. The gate has the
// storage type.
template <typename T>
__global__ void __launch_bounds__(128) head_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate,
                                                             long long gate_stride, const float* __restrict__ w, float eps,
                                                             T* __restrict__ out, int heads, int vdim, int act,
                                                             long long items) {
  pdl_sync();
  const int lane = threadIdx.x & 31;
  const long long item = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= items) return;
  const long long t = item / heads;
  const int h = static_cast<int>(item % heads);
  const float* x = o + item * vdim;
  float ss = 0.0f;
  for (int d = lane; d < vdim; d += 32) ss += x[d] * x[d];
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / static_cast<float>(vdim) + eps);
  for (int d = lane; d < vdim; d += 32) {
    const float g = ld(gate + t * gate_stride + h * vdim + d);
    const float a = act == 1 ? g * lr_sigmoid(g) : lr_sigmoid(g);
    st(out + item * vdim + d, (w != nullptr ? (x[d] * inv) * w[d] : x[d] * inv) * a);
  }
}

// The same for long heads (or one norm over a whole row): one block per (token, head).
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_block_kernel(const float* __restrict__ o, const T* __restrict__ gate,
                                                                   long long gate_stride, const float* __restrict__ w, float eps,
                                                                   T* __restrict__ out, int heads, int vdim, int act) {
  pdl_sync();
  __shared__ float scratch[33];
  const long long item = blockIdx.x, t = item / heads;
  const int h = static_cast<int>(item % heads);
  const float* x = o + item * vdim;
  float ss = 0.0f;
  for (int d = threadIdx.x; d < vdim; d += blockDim.x) ss += x[d] * x[d];
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(vdim) + eps);
  for (int d = threadIdx.x; d < vdim; d += blockDim.x) {
    const float g = ld(gate + t * gate_stride + h * vdim + d);
    const float a = act == 1 ? g * lr_sigmoid(g) : lr_sigmoid(g);
    st(out + item * vdim + d, (w != nullptr ? (x[d] * inv) * w[d] : x[d] * inv) * a);
  }
}

// Four columns a thread, the row in registers between its sum and its use (vdim a multiple of four, at most 4 NV threads).
template <typename T, int NV>
__global__ void __launch_bounds__(1024) head_norm_gate_vec4_kernel(const float* __restrict__ o, const T* __restrict__ gate,
                                                                   long long gate_stride, const float* __restrict__ w, float eps,
                                                                   T* __restrict__ out, int heads, int vdim, int act) {
  pdl_sync();
  __shared__ float scratch[33];
  const long long item = blockIdx.x, t = item / heads;
  const int h = static_cast<int>(item % heads);
  float x[NV][4], gv[NV][4], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (threadIdx.x + i * blockDim.x) * 4;
    if (d < vdim) {
      load4(o + item * vdim + d, x[i]);
      load4(gate + t * gate_stride + static_cast<long long>(h) * vdim + d, gv[i]);
#pragma unroll
      for (int e = 0; e < 4; ++e) ss = fmaf(x[i][e], x[i][e], ss);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(vdim) + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (threadIdx.x + i * blockDim.x) * 4;
    if (d < vdim) {
      float ww[4] = {1.0f, 1.0f, 1.0f, 1.0f}, r[4];
      if (w != nullptr) load4(w + d, ww);
#pragma unroll
      for (int e = 0; e < 4; ++e) r[e] = ((x[i][e] * inv) * ww[e]) * (act == 1 ? gv[i][e] * lr_sigmoid(gv[i][e]) : lr_sigmoid(gv[i][e]));
      store4(out + item * vdim + d, r);
    }
  }
}

// y = (o + skip[h] x) * silu(z), each of `parts` equal parts of the row divided by its own root mean square, times w.
template <typename T>
__global__ void __launch_bounds__(256) ssd_out_kernel(const float* __restrict__ o, const float* __restrict__ xn,
                                                      const T* __restrict__ z, long long z_stride,
                                                      const float* __restrict__ skip, const float* __restrict__ w, float eps,
                                                      T* __restrict__ out, int inner, int vdim, int parts) {
  pdl_sync();
  __shared__ float scratch[33];
  const long long t = blockIdx.x;
  const int part = blockIdx.y, size = inner / parts, c0 = part * size;
  float ss = 0.0f;
  for (int d = threadIdx.x; d < size; d += blockDim.x) {
    const int c = c0 + d;
    const float g = ld(z + t * z_stride + c);
    const float y = fmaf(skip[c / vdim], xn[t * inner + c], o[t * inner + c]) * (g * lr_sigmoid(g));
    ss += y * y;
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss / static_cast<float>(size) + eps);
  for (int d = threadIdx.x; d < size; d += blockDim.x) {
    const int c = c0 + d;
    const float g = ld(z + t * z_stride + c);
    const float y = fmaf(skip[c / vdim], xn[t * inner + c], o[t * inner + c]) * (g * lr_sigmoid(g));
    st(out + t * inner + c, (y * inv) * w[c]);
  }
}

}  // namespace tie

using namespace tie;

#define TIE_BY_DTYPE(dtype, CALL)                        \
  do {                                                   \
    if (dtype == TIE_F32) {                              \
      using T = float;                                   \
      CALL;                                              \
    } else if (dtype == TIE_BF16) {                      \
      using T = __nv_bfloat16;                           \
      CALL;                                              \
    } else {                                             \
      set_error("unknown dtype code %d", dtype);         \
      return kBadArgument;                               \
    }                                                    \
  } while (0)

TIE_API int tie_gla_prep(int dtype, const void* proj, long long stride, int q_off, int k_off, int v_off, int tokens, int heads,
                         int dim, int vdim, float q_scale, float tau, const float* z_bias, float* qn, float* kn, float* vn,
                         float* decay, long long decay_stride, cudaStream_t s) {
  TIE_REQUIRE(heads > 0 && dim > 0 && vdim > 0 && tau > 0.0f, "gla_prep: bad sizes heads=%d dim=%d vdim=%d tau=%g", heads, dim,
              vdim, static_cast<double>(tau));
  if (tokens <= 0) return kOk;
  TIE_BY_DTYPE(dtype, TIE_LAUNCH((gla_prep_kernel<T>), tokens, 256, 0, s, static_cast<const T*>(proj), stride, q_off, k_off, v_off,
                                 heads * dim, heads * vdim, q_scale, 1.0f / tau, z_bias, qn, kn, vn, decay, decay_stride));
  TIE_RETURN_LAUNCH("gla_prep");
}

TIE_API int tie_act_split(int dtype, const void* proj, long long stride, int q_off, int k_off, int v_off, int tokens, int nqk, int nv,
                          int act, float* qn, float* kn, float* vn, cudaStream_t s) {
  TIE_REQUIRE(nqk > 0 && nv > 0 && (act == 0 || act == 1), "act_split: bad sizes nqk=%d nv=%d act=%d", nqk, nv, act);
  if (tokens <= 0) return kOk;
  const int vec = dtype == TIE_F32 ? 4 : 8;
  auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const bool wide = on16(proj) && on16(qn) && on16(kn) && on16(vn) && stride % vec == 0 && q_off % vec == 0 && k_off % vec == 0 &&
                    v_off % vec == 0 && nqk % vec == 0 && nv % vec == 0;
  const long long total = static_cast<long long>(tokens) * (2 * nqk + nv) / (wide ? vec : 1);
  const int blocks = static_cast<int>(min(static_cast<long long>(148 * 8), (total + 255) / 256));
  if (wide) {
    TIE_BY_DTYPE(dtype, TIE_LAUNCH((act_split_vec_kernel<T>), blocks, 256, 0, s, static_cast<const T*>(proj), stride, q_off, k_off, v_off,
                                   nqk, nv, act, qn, kn, vn, total));
  } else {
    TIE_BY_DTYPE(dtype, TIE_LAUNCH((act_split_kernel<T>), blocks, 256, 0, s, static_cast<const T*>(proj), stride, q_off, k_off, v_off, nqk,
                                   nv, act, qn, kn, vn, total));
  }
  TIE_RETURN_LAUNCH("act_split");
}

TIE_API int tie_rope_split(int dtype, const void* proj, long long stride, int q_off, int k_off, int v_off, int tokens, int heads, int dim,
                           int nv, const float* inv_freq, const double* turns, int rot, int neighbours, const int* positions,
                           float k_scale, float* qn, float* kn, float* vn, cudaStream_t s) {
  TIE_REQUIRE(heads > 0 && dim > 0 && nv > 0 && rot >= 0 && rot % 2 == 0 && rot <= dim, "rope_split: bad sizes heads=%d dim=%d rot=%d nv=%d",
              heads, dim, rot, nv);
  TIE_REQUIRE(rot == 0 || ((inv_freq == nullptr) != (turns == nullptr) && positions != nullptr), "rope_split: a rotation takes one table of frequencies");
  TIE_REQUIRE(rot <= 8192, "rope_split: %d rotated dimensions", rot);
  if (tokens <= 0) return kOk;
  auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const bool wide = on16(proj) && on16(qn) && on16(kn) && on16(vn) && stride % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 &&
                    dim % 4 == 0 && nv % 4 == 0 && (neighbours ? rot % 4 == 0 : rot % 8 == 0);
  const Rotation turn{inv_freq, turns, rot, neighbours};
  TIE_BY_DTYPE(dtype, TIE_LAUNCH((rope_split_kernel<T>), tokens, 256, rot * sizeof(float), s, static_cast<const T*>(proj), stride, q_off, k_off,
                                 v_off, heads, dim, nv, turn, positions, k_scale, qn, kn, vn, wide ? 1 : 0));
  TIE_RETURN_LAUNCH("rope_split");
}

TIE_API int tie_ssd_prep(int dtype, const void* proj, long long stride, int c_off, int b_off, int x_off, int dt_off,
                         const float* conv_w, const float* conv_b, const float* state, long long state_stride,
                         long long conv_state_off, const int* seq_of_row, const int* query_start, const int* state_slots,
                         int tokens, int heads, int groups, int state_size, int vdim, int taps, const float* dt_bias,
                         const float* a_log, float* cn, float* bn, float* xn, float* dt, float* decay, cudaStream_t s) {
  TIE_REQUIRE(heads > 0 && groups > 0 && heads % groups == 0 && state_size > 0 && vdim > 0 && taps >= 1 && taps <= 16,
              "ssd_prep: bad shape heads=%d groups=%d state=%d vdim=%d taps=%d (1 to 16)", heads, groups, state_size, vdim, taps);
  if (tokens <= 0) return kOk;
  const int units = 2 * groups + heads + 1;
  TIE_REQUIRE(units <= 65535, "ssd_prep: %d heads exceed the grid", heads);
  const SsdShape sh{heads, groups, state_size, vdim, taps};
  TIE_BY_DTYPE(dtype, TIE_LAUNCH((ssd_prep_kernel<T>), dim3(tokens, units), 128, 0, s, static_cast<const T*>(proj), stride, c_off,
                                 b_off, x_off, dt_off, conv_w, conv_b, state, state_stride, conv_state_off, seq_of_row,
                                 query_start, state_slots, sh, dt_bias, a_log, cn, bn, xn, dt, decay));
  TIE_RETURN_LAUNCH("ssd_prep");
}

TIE_API int tie_head_norm_gate(int dtype, const float* o, const void* gate, long long gate_stride, const float* w, float eps,
                               void* out, int tokens, int heads, int vdim, int act, cudaStream_t s) {
  TIE_REQUIRE(tokens >= 0 && heads > 0 && vdim > 0 && (act == 0 || act == 1), "head_norm_gate: bad sizes tokens=%d heads=%d vdim=%d act=%d",
              tokens, heads, vdim, act);
  const long long items = static_cast<long long>(tokens) * heads;
  if (items == 0) return kOk;
  auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (vdim >= 512 && vdim % 4 == 0 && vdim <= 8192 && gate_stride % 4 == 0 && items <= 0x7fffffffLL && on16(o) && on16(w) && on16(out) &&
      reinterpret_cast<uintptr_t>(gate) % 16 == 0) {
    const int pieces = vdim / 4;
    int threads = items <= 512 ? 1024 : 256;
    while (threads < 1024 && pieces > 2 * threads) threads *= 2;
    while (threads > 32 && threads / 2 >= pieces) threads /= 2;
    TIE_BY_DTYPE(dtype, TIE_LAUNCH((head_norm_gate_vec4_kernel<T, 2>), static_cast<int>(items), threads, 0, s, o, static_cast<const T*>(gate),
                                   gate_stride, w, eps, static_cast<T*>(out), heads, vdim, act));
    TIE_RETURN_LAUNCH("head_norm_gate");
  }
  if (vdim >= 512 && items <= 0x7fffffffLL) {
    TIE_BY_DTYPE(dtype, TIE_LAUNCH((head_norm_gate_block_kernel<T>), static_cast<int>(items), 256, 0, s, o, static_cast<const T*>(gate),
                                   gate_stride, w, eps, static_cast<T*>(out), heads, vdim, act));
    TIE_RETURN_LAUNCH("head_norm_gate");
  }
  TIE_BY_DTYPE(dtype, TIE_LAUNCH((head_norm_gate_kernel<T>), ceil_div(items, 4), 128, 0, s, o, static_cast<const T*>(gate),
                                 gate_stride, w, eps, static_cast<T*>(out), heads, vdim, act, items));
  TIE_RETURN_LAUNCH("head_norm_gate");
}

TIE_API int tie_ssd_out(int dtype, const float* o, const float* xn, const void* z, long long z_stride, const float* skip,
                        const float* w, float eps, void* out, int tokens, int heads, int vdim, int parts, cudaStream_t s) {
  TIE_REQUIRE(heads > 0 && vdim > 0 && parts > 0 && (heads * vdim) % parts == 0 && parts <= 65535,
              "ssd_out: %d heads of %d do not split into %d equal parts", heads, vdim, parts);
  if (tokens <= 0) return kOk;
  TIE_BY_DTYPE(dtype, TIE_LAUNCH((ssd_out_kernel<T>), dim3(tokens, parts), 256, 0, s, o, xn, static_cast<const T*>(z), z_stride,
                                 skip, w, eps, static_cast<T*>(out), heads * vdim, vdim, parts));
  TIE_RETURN_LAUNCH("ssd_out");
}
