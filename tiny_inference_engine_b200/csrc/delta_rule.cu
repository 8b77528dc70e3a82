// The gated delta rule with one decay per key channel, as a recurrence over the tokens of each sequence.
//
// Per value head, a float matrix S (key channels x value channels) is carried from token to token:
//
//     S <- diag(decay_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
//
// (the read-out sees the token's own write). q_t and k_t are unit vectors per head (q also scaled), made from
// projections that pass a short causal convolution over time and SiLU; decay_t = exp(-rate_h softplus(a_t + bias))
// per key channel. Columns of S do not depend on one another, so the work is cut by (sequence, head, columns).
//
// Three kernels, all of them float inside:
//   delta_prep   one block per (token, head of q, k or v): convolution (its first taps - 1 inputs come from the
//                sequence's state slot or from the rows ahead of it in the step) + SiLU, unit norm of q and k per
//                head; further blocks turn the raw decay projection into decays (in place) and take beta's sigmoid.
//   delta_rule   one block per (sequence, head, 16 columns): the recurrence over the sequence's tokens of the
//                step, state read from and written back to the slot in row pieces through shared memory. Eight
//                lanes share a column; a chunk of tokens is staged in shared memory at a time. The blocks of a
//                sequence also move the convolution's last inputs into the slot, a slice of the channels each.
//   delta_out    one warp per (token, head): o / rms(o) * w * sigmoid(gate).
//
// A state slot is one float row: S of every head [heads, dim, vdim], then the convolution's last taps - 1
// inputs [taps - 1, channels] (oldest first), channels = q, k, v one after the other.
#include <math.h>

#include "common.cuh"

namespace tie {

struct DeltaShape {
  int heads, kv_heads, dim, vdim, taps;
  int channels() const { return 2 * kv_heads * dim + heads * vdim; }
};

__device__ __forceinline__ float sigmoidf_(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplusf_(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

// proj row: q at q_off [kv_heads * dim], k at k_off, v at v_off [heads * vdim], beta at b_off [heads].
// One block per (token, unit). Units: the q heads, the k heads, the v heads (convolution + SiLU over the unit's
// channels; q and k also their unit norm), then one unit per head that turns the raw decay projection into decays
// in place, and a last one for beta.
template <typename T>
__global__ void __launch_bounds__(128) delta_prep_kernel(const T* __restrict__ proj, long long stride, int q_off, int k_off,
                                                         int v_off, int b_off, const float* __restrict__ conv_w,
                                                         const float* __restrict__ state, long long state_stride,
                                                         long long conv_state_off, const int* __restrict__ seq_of_row,
                                                         const int* __restrict__ query_start,
                                                         const int* __restrict__ state_slots, DeltaShape sh, float unit_eps,
                                                         float q_scale, float* __restrict__ qn, float* __restrict__ kn,
                                                         float* __restrict__ vn, float* __restrict__ beta,
                                                         float* __restrict__ decay, long long decay_stride,
                                                         const float* __restrict__ dt_bias, const float* __restrict__ a_log) {
  pdl_sync();
  __shared__ float scratch[33];
  const int t = blockIdx.x, unit = blockIdx.y;
  const int G = sh.kv_heads, H = sh.heads, dim = sh.dim, vdim = sh.vdim, taps = sh.taps;
  const int nqk = G * dim, nv = H * vdim, C = 2 * nqk + nv;
  const T* row = proj + static_cast<long long>(t) * stride;
  if (unit == 2 * G + 2 * H) {
    for (int h = threadIdx.x; h < H; h += blockDim.x) beta[static_cast<long long>(t) * H + h] = sigmoidf_(ld(row + b_off + h));
    return;
  }
  if (unit >= 2 * G + H) {            // decay = exp(-rate * softplus(raw + bias)), in place
    const int h = unit - (2 * G + H);
    const float rate = expf(a_log[h]);
    float* a = decay + static_cast<long long>(t) * decay_stride + h * dim;
    for (int d = threadIdx.x; d < dim; d += blockDim.x) a[d] = expf(-rate * softplusf_(a[d] + dt_bias[h * dim + d]));
    return;
  }
  const int s = seq_of_row[t];
  const int j = t - query_start[s];          // tokens of this sequence ahead of this one in the step
  const int slot = state_slots[s];
  const float* tail = slot >= 0 ? state + slot * state_stride + conv_state_off : nullptr;
  const bool is_v = unit >= 2 * G;
  const int width = is_v ? vdim : dim;
  const int c0 = is_v ? 2 * nqk + (unit - 2 * G) * vdim : unit * dim;      // the unit's first channel of all C
  float* dst = is_v ? vn + static_cast<long long>(t) * nv + (unit - 2 * G) * vdim
                    : (unit < G ? qn + static_cast<long long>(t) * nqk + unit * dim
                                : kn + static_cast<long long>(t) * nqk + (unit - G) * dim);
  float vals[2] = {0.0f, 0.0f};              // dim <= 256: at most two channels of a q or k head per thread
  float ss = 0.0f;
  for (int d = threadIdx.x, n = 0; d < width; d += blockDim.x, ++n) {
    const int c = c0 + d;
    const int col = c < nqk ? q_off + c : (c < 2 * nqk ? k_off + (c - nqk) : v_off + (c - 2 * nqk));
    float y = 0.0f;
    for (int i = 0; i < taps; ++i) {
      const int back = taps - 1 - i;         // this tap's input is `back` tokens ahead of the current one
      float in;
      if (back <= j) in = ld(row - static_cast<long long>(back) * stride + col);
      else in = tail ? tail[static_cast<long long>(j + i) * C + c] : 0.0f;
      y = fmaf(conv_w[c * taps + i], in, y);
    }
    y = y * sigmoidf_(y);
    if (is_v) {
      dst[d] = y;
    } else {
      if (n < 2) vals[n] = y;
      ss += y * y;
    }
  }
  if (is_v) return;
  ss = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss + unit_eps);
  for (int d = threadIdx.x, n = 0; d < width && n < 2; d += blockDim.x, ++n) dst[d] = unit < G ? (vals[n] * inv) * q_scale : vals[n] * inv;
}

// The same with a warp a unit, four channels a lane and four taps: sizes and sections in whole pieces of four.
template <typename T>
__global__ void __launch_bounds__(128) delta_prep_warp_kernel(const T* __restrict__ proj, long long stride, int q_off, int k_off,
                                                              int v_off, int b_off, const float* __restrict__ conv_w,
                                                              const float* __restrict__ state, long long state_stride,
                                                              long long conv_state_off, const int* __restrict__ seq_of_row,
                                                              const int* __restrict__ query_start,
                                                              const int* __restrict__ state_slots, DeltaShape sh, float unit_eps,
                                                              float q_scale, float* __restrict__ qn, float* __restrict__ kn,
                                                              float* __restrict__ vn, float* __restrict__ beta,
                                                              float* __restrict__ decay, long long decay_stride,
                                                              const float* __restrict__ dt_bias, const float* __restrict__ a_log) {
  pdl_sync();
  const int t = blockIdx.x, unit = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int G = sh.kv_heads, H = sh.heads, dim = sh.dim, vdim = sh.vdim;
  const int nqk = G * dim, nv = H * vdim, C = 2 * nqk + nv;
  if (unit > 2 * G + 2 * H) return;
  const T* row = proj + static_cast<long long>(t) * stride;
  if (unit == 2 * G + 2 * H) {
    for (int h = lane; h < H; h += 32) beta[static_cast<long long>(t) * H + h] = sigmoidf_(ld(row + b_off + h));
    return;
  }
  if (unit >= 2 * G + H) {
    const int h = unit - (2 * G + H);
    const float rate = expf(a_log[h]);
    float* a = decay + static_cast<long long>(t) * decay_stride + h * dim;
    for (int d = lane * 4; d < dim; d += 128) {
      float z[4], b[4];
      load4(a + d, z);
      load4(dt_bias + h * dim + d, b);
#pragma unroll
      for (int e = 0; e < 4; ++e) z[e] = expf(-rate * softplusf_(z[e] + b[e]));
      store4(a + d, z);
    }
    return;
  }
  const int s = seq_of_row[t];
  const int j = t - query_start[s];
  const int slot = state_slots[s];
  const float* tail = slot >= 0 ? state + slot * state_stride + conv_state_off : nullptr;
  const bool is_v = unit >= 2 * G;
  const int width = is_v ? vdim : dim;
  const int c0 = is_v ? 2 * nqk + (unit - 2 * G) * vdim : unit * dim;
  const int col0 = is_v ? v_off + (unit - 2 * G) * vdim : (unit < G ? q_off + unit * dim : k_off + (unit - G) * dim);
  float* dst = is_v ? vn + static_cast<long long>(t) * nv + (unit - 2 * G) * vdim
                    : (unit < G ? qn + static_cast<long long>(t) * nqk + unit * dim
                                : kn + static_cast<long long>(t) * nqk + (unit - G) * dim);
  float kept[2][4], ss = 0.0f;               // dim <= 256: at most two pieces of a q or k head a lane
#pragma unroll 2
  for (int n = 0; n * 128 < width; ++n) {
    const int d = n * 128 + lane * 4;
    float y[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (d < width) {
      float in[4][4], w[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int back = 3 - i;
        load4(conv_w + (c0 + d + i) * 4, w[i]);      // w[e]: the taps of channel d + e
        if (back <= j) {
          load4(row - static_cast<long long>(back) * stride + col0 + d, in[i]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) in[i][e] = tail ? tail[static_cast<long long>(j + i) * C + c0 + d + e] : 0.0f;
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
#pragma unroll
        for (int i = 0; i < 4; ++i) y[e] = fmaf(w[e][i], in[i][e], y[e]);
        y[e] = y[e] * sigmoidf_(y[e]);
        ss = fmaf(y[e], y[e], ss);
      }
      if (is_v) store4(dst + d, y);
    }
    if (n < 2) {
#pragma unroll
      for (int e = 0; e < 4; ++e) kept[n & 1][e] = y[e];
    }
  }
  if (is_v) return;
  ss = warp_sum(ss);
  const float inv = (1.0f / sqrtf(ss + unit_eps)) * (unit < G ? q_scale : 1.0f);
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int d = n * 128 + lane * 4;
    if (d < width) {
#pragma unroll
      for (int e = 0; e < 4; ++e) kept[n][e] *= inv;
      store4(dst + d, kept[n]);
    }
  }
}

__device__ __forceinline__ void async_copy4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}
__device__ __forceinline__ void async_copy16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}
__device__ __forceinline__ void async_copies_done() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory"); }

constexpr int kDeltaCols = 16;       // columns of S that a block holds
constexpr int kDeltaPad = kDeltaCols + 1;
constexpr int kDeltaBatch = 4;       // tokens whose read-outs are summed over the lanes together

// The key channel that register r of lane `lane` (of the LANES that share a column) holds: four channels in a row, then the
// next four 4 LANES channels on, so that a lane reads its k, q and decay entries 16 bytes at a time and the lanes of a column
// read one piece of memory (the columns of a warp the same one).
template <int LANES>
__device__ __forceinline__ int delta_row(int r, int lane) { return (r >> 2) * (4 * LANES) + lane * 4 + (r & 3); }

// A token's rows as a lane holds them.
template <int R, bool ONE_DECAY>
struct DeltaToken {
  float k[R], q[R], g[ONE_DECAY ? 1 : R], v, beta, kq;
};

// What the recurrence does with a token (u is what it writes along its key):
//   kDeltaRule   S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   kDeltaPlain  S <- diag(g) S + k u^T, u = beta v;  o = S^T q
//   kDeltaBonus  o = S^T q + (sum_c bonus[h, c] k_c q_c) u, u = beta v: the token reads the state as the token before left it
//                and sees its own write through a weight per key channel;  then S <- diag(g) S + k u^T
enum DeltaMode { kDeltaRule, kDeltaPlain, kDeltaBonus };

// One block per (sequence, head, 16 columns of S). A column's key channels are spread over LANES (8 or 16) lanes, R a lane. What bounds
// the kernel is the chain from token to token: in the delta rule a product over the lane's channels, the exchanges and the
// update; without the correction the update alone. So everything else is kept off that chain and off the shared-memory pipe:
// a column has few lanes (fewer exchanges, and the columns of a warp read the same k, q and g), the
// read-outs of four tokens are summed over the lanes together (each exchange halves the tokens that a lane still holds), and
// k . q of a token is formed once a chunk, for all columns. In the delta rule the read-out of the updated state is
// (gS)^T q + (k . q) u, so it does not wait for the update.
// FULL: the head has exactly LANES * R key channels and its rows come in whole 16-byte pieces, and what the decays are
// (PER_HEAD: one a token and head) is known too: no tests inside the walk.
template <typename T, int R, int LANES, DeltaMode MODE, bool FULL, bool PER_HEAD>
__global__ void __launch_bounds__(kDeltaCols * LANES) delta_rule_kernel(
    const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ vn, const float* __restrict__ beta,
    const float* __restrict__ decay, long long decay_stride, float* __restrict__ state, long long state_stride,
    long long conv_state_off, const T* __restrict__ proj, long long proj_stride, int q_off, int k_off, int v_off,
    const int* __restrict__ query_start, const int* __restrict__ state_slots, DeltaShape sh, int chunk,
    float* __restrict__ out, int decay_per_head_, const float* __restrict__ bonus = nullptr) {
  const bool decay_per_head = FULL ? PER_HEAD : decay_per_head_ != 0;
  // A block is one long chain of dependent steps, and there are few blocks (sequences x heads x column tiles). Started early
  // (programmatic dependent launch), beside a kernel that still fills the GPU, the blocks were placed on the few SMs that had
  // room first and shared them. So for steps with portions the launcher starts this kernel only when the kernels ahead have
  // drained (launch_kernel_alone), and the kernel behind is let in when the walk over the tokens is done.
  pdl_wait();
  constexpr int kDeltaThreads = kDeltaCols * LANES;
  extern __shared__ float smem[];
  const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kDeltaCols;
  const int slot = state_slots[s];
  if (slot < 0) return;                       // a sequence that pads a captured batch
  const int t0 = query_start[s], n = query_start[s + 1] - t0;
  const int dim = FULL ? LANES * R : sh.dim, vdim = sh.vdim, nqk = sh.kv_heads * dim, nv = sh.heads * vdim;
  const int g = h / (sh.heads / sh.kv_heads);
  const int lane8 = threadIdx.x % LANES, cidx = threadIdx.x / LANES, col = col0 + cidx;
  const bool live = col < vdim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* S = state + slot * state_stride + static_cast<long long>(h) * dim * vdim;
  float* stage = smem;                        // the block's 16 columns of S on their way in and out, rows of kDeltaPad
  const bool quads = vdim % 4 == 0 && (reinterpret_cast<uintptr_t>(S) & 15) == 0;
  if (quads) {
#pragma unroll 4
    for (int i = threadIdx.x; i < dim * (kDeltaCols / 4); i += kDeltaThreads) {
      const int r = i / (kDeltaCols / 4), c = (i % (kDeltaCols / 4)) * 4;
      float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      if (col0 + c < vdim) load4(S + static_cast<long long>(r) * vdim + col0 + c, v);
#pragma unroll
      for (int e = 0; e < 4; ++e) stage[r * kDeltaPad + c + e] = v[e];
    }
  } else {
    for (int i = threadIdx.x; i < dim * kDeltaCols; i += kDeltaThreads) {
      const int r = i / kDeltaCols, c = i % kDeltaCols;
      stage[r * kDeltaPad + c] = col0 + c < vdim ? S[static_cast<long long>(r) * vdim + col0 + c] : 0.0f;
    }
  }
  // Chunks of tokens come through two buffers in turn: while one is worked on, asynchronous copies fill the other.
  // A buffer: k [chunk][dim], q [chunk][dim], decays [chunk][dim] (or [chunk]), v [chunk][kDeltaCols], beta [chunk].
  float* const buffers = smem + ((dim * kDeltaPad + 3) & ~3);
  const int g_ld = decay_per_head ? 1 : dim;
  const int buf_floats = (chunk * (2 * dim + g_ld + kDeltaCols + 1) + 3) & ~3;      // a buffer starts on a 16-byte boundary
  float* const kq = buffers + 2 * buf_floats;                                       // [chunk]: k . q of the chunk's tokens
  const bool vec4 = FULL || dim % 4 == 0;
  const bool wide = vec4 && nqk % 4 == 0 && ((reinterpret_cast<uintptr_t>(kn) | reinterpret_cast<uintptr_t>(qn)) & 15) == 0 &&
                    (decay_per_head || (decay_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(decay) & 15) == 0));
  auto fetch = [&](int c0, float* base) {
    const int cn = min(chunk, n - c0);
    float* kb = base;
    float* qb = kb + chunk * dim;
    float* gb = qb + chunk * dim;
    float* bb = gb + chunk * g_ld + chunk * kDeltaCols;
    if (wide) {
      const int pieces = dim / 4;
      for (int i = threadIdx.x; i < cn * pieces; i += kDeltaThreads) {
        const int tc = i / pieces, d = (i % pieces) * 4;
        const long long t = t0 + c0 + tc;
        async_copy16(kb + tc * dim + d, kn + t * nqk + g * dim + d);
        async_copy16(qb + tc * dim + d, qn + t * nqk + g * dim + d);
        if (!decay_per_head) async_copy16(gb + tc * dim + d, decay + t * decay_stride + h * dim + d);
      }
    } else {
      for (int i = threadIdx.x; i < cn * dim; i += kDeltaThreads) {
        const int tc = i / dim, d = i % dim;
        const long long t = t0 + c0 + tc;
        async_copy4(kb + i, kn + t * nqk + g * dim + d);
        async_copy4(qb + i, qn + t * nqk + g * dim + d);
        if (!decay_per_head) async_copy4(gb + i, decay + t * decay_stride + h * dim + d);
      }
    }
    float* vb = gb + chunk * g_ld;
    for (int i = threadIdx.x; i < cn * kDeltaCols; i += kDeltaThreads) {
      const int tc = i / kDeltaCols, c = col0 + i % kDeltaCols;
      if (c < vdim) async_copy4(vb + i, vn + (t0 + c0 + tc) * static_cast<long long>(nv) + h * vdim + c);
      else vb[i] = 0.0f;
    }
    for (int i = threadIdx.x; i < cn; i += kDeltaThreads) {
      if (decay_per_head) async_copy4(gb + i, decay + (t0 + c0 + i) * decay_stride + h);
      if (beta) async_copy4(bb + i, beta + (t0 + c0 + i) * static_cast<long long>(sh.heads) + h);
      else bb[i] = 1.0f;
    }
  };
  fetch(0, buffers);
  __syncthreads();
  float sreg[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int rowi = delta_row<LANES>(r, lane8);
    sreg[r] = FULL || rowi < dim ? stage[rowi * kDeltaPad + cidx] : 0.0f;
  }
  int turn = 0;
  for (int c0 = 0; c0 < n; c0 += chunk, turn ^= 1) {
    const int cn = min(chunk, n - c0);
    const float* kb = buffers + turn * buf_floats;
    const float* qb = kb + chunk * dim;
    const float* gb = qb + chunk * dim;
    const float* vb = gb + chunk * g_ld;
    const float* bb = vb + chunk * kDeltaCols;
    async_copies_done();
    __syncthreads();                          // this chunk is there, and everyone is through with the other buffer
    if (c0 + chunk < n) fetch(c0 + chunk, buffers + (turn ^ 1) * buf_floats);
    if (MODE != kDeltaPlain) {
      for (int tc = warp; tc < cn; tc += kDeltaThreads / 32) {
        float dot = 0.0f;
        for (int d = lane; d < dim; d += 32)
          dot = fmaf(MODE == kDeltaBonus ? kb[tc * dim + d] * bonus[h * dim + d] : kb[tc * dim + d], qb[tc * dim + d], dot);
        dot = warp_sum(dot);
        if (lane == 0) kq[tc] = dot;
      }
      __syncthreads();
    }
    // What a lane needs of a token. The next token's is fetched from shared memory ahead of this token's exchanges: the chain
    // from token to token then waits for no load.
    auto fetch_token = [&](int tc, DeltaToken<R, FULL && PER_HEAD>& x) {
      const float* kt = kb + tc * dim;
      const float* qt = qb + tc * dim;
      const float* gt = gb + tc * g_ld;
      x.v = vb[tc * kDeltaCols + cidx], x.beta = bb[tc];
      if (MODE != kDeltaPlain) x.kq = kq[tc];
      const float g1 = decay_per_head ? gt[0] : 1.0f;
      if (FULL && PER_HEAD) x.g[0] = g1;
#pragma unroll
      for (int q4 = 0; q4 < R / 4; ++q4) {
        const int r0 = delta_row<LANES>(4 * q4, lane8);
        float kk[4] = {0.0f, 0.0f, 0.0f, 0.0f}, qq[4] = {0.0f, 0.0f, 0.0f, 0.0f}, gg[4] = {g1, g1, g1, g1};
        if (vec4) {                              // the lane's four channels are one 16-byte piece
          if (FULL || r0 < dim) {
            load4(kt + r0, kk);
            load4(qt + r0, qq);
            if (!decay_per_head) load4(gt + r0, gg);
          }
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            if (r0 + e < dim) {
              kk[e] = kt[r0 + e];
              qq[e] = qt[r0 + e];
              if (!decay_per_head) gg[e] = gt[r0 + e];
            }
          }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          x.k[4 * q4 + e] = kk[e], x.q[4 * q4 + e] = qq[e];
          if (!(FULL && PER_HEAD)) x.g[4 * q4 + e] = gg[e];
        }
      }
    };
    DeltaToken<R, FULL && PER_HEAD> ahead;
    fetch_token(0, ahead);
    // One token: this lane's share of the read-out.
    auto step = [&](int tc) -> float {
      const DeltaToken<R, FULL && PER_HEAD> x = ahead;
      fetch_token(min(tc + 1, cn - 1), ahead);
      float y0 = 0.0f, y1 = 0.0f, d0 = 0.0f, d1 = 0.0f;
      float u = x.beta * x.v;
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const float before = sreg[r], kept = before * x.g[FULL && PER_HEAD ? 0 : r];
        if (MODE == kDeltaRule) {
          sreg[r] = kept;
          if (r & 1) d1 = fmaf(x.k[r], kept, d1), y1 = fmaf(x.q[r], kept, y1);
          else d0 = fmaf(x.k[r], kept, d0), y0 = fmaf(x.q[r], kept, y0);
        } else {
          sreg[r] = fmaf(x.k[r], u, kept);
          const float seen = MODE == kDeltaBonus ? before : sreg[r];
          if (r & 1) y1 = fmaf(x.q[r], seen, y1);
          else y0 = fmaf(x.q[r], seen, y0);
        }
      }
      float y = y0 + y1;
      if (MODE == kDeltaRule) {
        float d = d0 + d1;
#pragma unroll
        for (int o = 1; o < LANES; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
        u = x.beta * (x.v - d);
#pragma unroll
        for (int r = 0; r < R; ++r) sreg[r] = fmaf(x.k[r], u, sreg[r]);
      }
      if (MODE != kDeltaPlain && lane8 == 0) y = fmaf(x.kq, u, y);
      return y;
    };
    // Four tokens' shares to sums: lane l of a column ends up with the token l & 3.
    auto finish = [&](int tb, float (&y)[kDeltaBatch]) {
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const bool up = lane8 & 2;
        const float give = up ? y[q] : y[q + 2], keep = up ? y[q + 2] : y[q];
        y[q] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
      }
      const bool up = lane8 & 1;
      const float give = up ? y[0] : y[1], keep = up ? y[1] : y[0];
      float sum = keep + __shfl_xor_sync(0xffffffffu, give, 1);
#pragma unroll
      for (int o = 4; o < LANES; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (live && lane8 < kDeltaBatch && tb + lane8 < cn) out[(t0 + c0 + tb + lane8) * static_cast<long long>(nv) + h * vdim + col] = sum;
    };
    int tb = 0;
    for (; tb + kDeltaBatch <= cn; tb += kDeltaBatch) {
      float y[kDeltaBatch];
#pragma unroll
      for (int q = 0; q < kDeltaBatch; ++q) y[q] = step(tb + q);
      finish(tb, y);
    }
    if (tb < cn) {
      float y[kDeltaBatch] = {0.0f, 0.0f, 0.0f, 0.0f};
      for (int q = 0; tb + q < cn; ++q) {
        const float v = step(tb + q);
        if (q == 0) y[0] = v;
        else if (q == 1) y[1] = v;
        else y[2] = v;
      }
      finish(tb, y);
    }
  }
  pdl_launch_dependents();
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int rowi = delta_row<LANES>(r, lane8);
    if (rowi < dim) stage[rowi * kDeltaPad + cidx] = sreg[r];
  }
  __syncthreads();
  if (quads) {
#pragma unroll 4
    for (int i = threadIdx.x; i < dim * (kDeltaCols / 4); i += kDeltaThreads) {
      const int r = i / (kDeltaCols / 4), c = (i % (kDeltaCols / 4)) * 4;
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = stage[r * kDeltaPad + c + e];
      if (col0 + c < vdim) store4(S + static_cast<long long>(r) * vdim + col0 + c, v);
    }
  } else {
    for (int i = threadIdx.x; i < dim * kDeltaCols; i += kDeltaThreads) {
      const int r = i / kDeltaCols, c = i % kDeltaCols;
      if (col0 + c < vdim) S[static_cast<long long>(r) * vdim + col0 + c] = stage[r * kDeltaPad + c];
    }
  }
  // The convolution's last taps - 1 inputs after this step: from the step's rows where it brought enough, else
  // what the slot held moves up. Every block of the sequence takes a slice of the channels.
  if (sh.taps > 1) {
    const int C = 2 * nqk + nv, keep = sh.taps - 1;
    const int blocks = gridDim.y * gridDim.z, mine = blockIdx.y * gridDim.z + blockIdx.z;
    const int per = (C + blocks - 1) / blocks;
    const int c_end = min(C, (mine + 1) * per);
    float* tail = state + slot * state_stride + conv_state_off;
    for (int c = mine * per + threadIdx.x; c < c_end; c += blockDim.x) {
      const int pc = c < nqk ? q_off + c : (c < 2 * nqk ? k_off + (c - nqk) : v_off + (c - 2 * nqk));
      for (int i = 0; i < keep; ++i) {
        const int from = n - keep + i;        // offset in the step of the token that lands at place i
        tail[static_cast<long long>(i) * C + c] = from >= 0 ? ld(proj + (t0 + from) * proj_stride + pc)
                                                            : tail[static_cast<long long>(n + i) * C + c];
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) delta_out_kernel(const float* __restrict__ o, const float* __restrict__ gate,
                                                        long long gate_stride, const float* __restrict__ w, float eps,
                                                        T* __restrict__ out, int heads, int vdim, long long items) {
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
  for (int d = lane; d < vdim; d += 32)
    st(out + item * vdim + d, ((x[d] * inv) * w[d]) * sigmoidf_(gate[t * gate_stride + h * vdim + d]));
}

}  // namespace tie

using namespace tie;

static int check_delta(const DeltaShape& sh) {
  TIE_REQUIRE(sh.heads > 0 && sh.kv_heads > 0 && sh.heads % sh.kv_heads == 0 && sh.dim > 0 && sh.dim <= 256 && sh.vdim > 0 &&
                  sh.taps >= 1 && sh.taps <= 16,
              "delta rule: bad shape heads=%d/%d dim=%d (1 to 256) vdim=%d taps=%d (1 to 16)", sh.heads, sh.kv_heads, sh.dim,
              sh.vdim, sh.taps);
  return kOk;
}

TIE_API int tie_delta_prep(int dtype, const void* proj, long long stride, int q_off, int k_off, int v_off, int b_off,
                           const float* conv_w, const float* state, long long state_stride, long long conv_state_off,
                           const int* seq_of_row, const int* query_start, const int* state_slots, int tokens, int heads,
                           int kv_heads, int dim, int vdim, int taps, float unit_eps, float q_scale, float* qn, float* kn,
                           float* vn, float* beta, float* decay, long long decay_stride, const float* dt_bias,
                           const float* a_log, cudaStream_t s) {
  const DeltaShape sh{heads, kv_heads, dim, vdim, taps};
  if (const int st_ = check_delta(sh)) return st_;
  if (tokens <= 0) return kOk;
  const int units = 2 * kv_heads + 2 * heads + 1;
  TIE_REQUIRE(units <= 65535, "delta_prep: %d heads exceed the grid", heads);
  const dim3 grid(tokens, units);
  auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (taps == 4 && dim % 4 == 0 && vdim % 4 == 0 && stride % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 &&
      decay_stride % 4 == 0 && on16(proj) && on16(conv_w) && on16(qn) && on16(kn) && on16(vn) && on16(decay) && on16(dt_bias) &&
      (dtype == TIE_F32 || dtype == TIE_BF16)) {
    const dim3 warps(tokens, ceil_div(units, 4));
    if (dtype == TIE_F32)
      TIE_LAUNCH((delta_prep_warp_kernel<float>), warps, 128, 0, s, static_cast<const float*>(proj), stride, q_off, k_off, v_off, b_off,
                 conv_w, state, state_stride, conv_state_off, seq_of_row, query_start, state_slots, sh, unit_eps, q_scale, qn, kn, vn,
                 beta, decay, decay_stride, dt_bias, a_log);
    else
      TIE_LAUNCH((delta_prep_warp_kernel<__nv_bfloat16>), warps, 128, 0, s, static_cast<const __nv_bfloat16*>(proj), stride, q_off, k_off,
                 v_off, b_off, conv_w, state, state_stride, conv_state_off, seq_of_row, query_start, state_slots, sh, unit_eps, q_scale,
                 qn, kn, vn, beta, decay, decay_stride, dt_bias, a_log);
    TIE_RETURN_LAUNCH("delta_prep");
  }
  if (dtype == TIE_F32) {
    TIE_LAUNCH((delta_prep_kernel<float>), grid, 128, 0, s, static_cast<const float*>(proj), stride, q_off, k_off, v_off, b_off,
               conv_w, state, state_stride, conv_state_off, seq_of_row, query_start, state_slots, sh, unit_eps, q_scale, qn, kn,
               vn, beta, decay, decay_stride, dt_bias, a_log);
  } else if (dtype == TIE_BF16) {
    TIE_LAUNCH((delta_prep_kernel<__nv_bfloat16>), grid, 128, 0, s, static_cast<const __nv_bfloat16*>(proj), stride, q_off,
               k_off, v_off, b_off, conv_w, state, state_stride, conv_state_off, seq_of_row, query_start, state_slots, sh,
               unit_eps, q_scale, qn, kn, vn, beta, decay, decay_stride, dt_bias, a_log);
  } else {
    set_error("unknown dtype code %d", dtype);
    return kBadArgument;
  }
  TIE_RETURN_LAUNCH("delta_prep");
}

template <typename T>
static int launch_delta_rule(const float* qn, const float* kn, const float* vn, const float* beta, const float* decay,
                             long long decay_stride, float* state, long long state_stride, long long conv_state_off,
                             const void* proj, long long proj_stride, int q_off, int k_off, int v_off,
                             const int* query_start, const int* state_slots, int seqs, const DeltaShape& sh, float* out,
                             int plain, int decay_per_head, int single, cudaStream_t s, const float* bonus = nullptr) {
  const dim3 grid(seqs, sh.heads, ceil_div(sh.vdim, kDeltaCols));
  const int per_token = 2 * sh.dim + (decay_per_head ? 1 : sh.dim) + kDeltaCols + 1;
  int chunk = kDeltaBatch;                     // `single`: one token a sequence, small buffers, many blocks an SM
  if (!single) {
    chunk = (60 * 1024 / static_cast<int>(sizeof(float))) / (2 * per_token) / kDeltaBatch * kDeltaBatch;      // two buffers
    chunk = chunk > 32 ? 32 : (chunk < kDeltaBatch ? kDeltaBatch : chunk);
  }
  const int floats = ((sh.dim * kDeltaPad + 3) & ~3) + 2 * ((chunk * per_token + 3) & ~3) + chunk;
  const size_t smem = static_cast<size_t>(floats) * sizeof(float);
  const T* p = static_cast<const T*>(proj);
  int failed = 0;
  const int threads = kDeltaCols * (sh.dim <= 32 ? 8 : 16);
  auto run = [&](auto kernel) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess) {
      failed = 1;
      return;
    }
    if (single)
      TIE_LAUNCH(kernel, grid, threads, smem, s, qn, kn, vn, beta, decay, decay_stride, state, state_stride, conv_state_off, p,
                 proj_stride, q_off, k_off, v_off, query_start, state_slots, sh, chunk, out, decay_per_head, bonus);
    else
      launch_kernel_alone(kernel, grid, dim3(threads), smem, s, qn, kn, vn, beta, decay, decay_stride, state, state_stride,
                          conv_state_off, p, proj_stride, q_off, k_off, v_off, query_start, state_slots, sh, chunk, out, decay_per_head,
                          bonus);
  };
#define TIE_DELTA_CASE(R, LANES)                                                                    \
  do {                                                                                       \
    const bool full = sh.dim == LANES * R;                                             \
    if (bonus != nullptr) {                                                                  \
      if (full) run(delta_rule_kernel<T, R, LANES, kDeltaBonus, true, false>);                      \
      else run(delta_rule_kernel<T, R, LANES, kDeltaBonus, false, false>);                          \
    } else if (plain) {                                                                      \
      if (full && decay_per_head) run(delta_rule_kernel<T, R, LANES, kDeltaPlain, true, true>);     \
      else if (full) run(delta_rule_kernel<T, R, LANES, kDeltaPlain, true, false>);                 \
      else run(delta_rule_kernel<T, R, LANES, kDeltaPlain, false, false>);                          \
    } else {                                                                                 \
      if (full && !decay_per_head) run(delta_rule_kernel<T, R, LANES, kDeltaRule, true, false>);    \
      else run(delta_rule_kernel<T, R, LANES, kDeltaRule, false, false>);                           \
    }                                                                                        \
  } while (0)
  if (sh.dim <= 32) TIE_DELTA_CASE(4, 8);
  else if (sh.dim <= 64) TIE_DELTA_CASE(4, 16);
  else if (sh.dim <= 128) TIE_DELTA_CASE(8, 16);
  else TIE_DELTA_CASE(16, 16);
#undef TIE_DELTA_CASE
  if (failed) {
    set_error("delta_rule: cannot reserve %zu bytes of shared memory", smem);
    return kCudaError;
  }
  TIE_RETURN_LAUNCH("delta_rule");
}

// single != 0: every sequence brings one token.
TIE_API int tie_delta_rule(int dtype, const float* qn, const float* kn, const float* vn, const float* beta,
                           const float* decay, long long decay_stride, float* state, long long state_stride,
                           long long conv_state_off, const void* proj, long long proj_stride, int q_off, int k_off,
                           int v_off, const int* query_start, const int* state_slots, int seqs, int heads, int kv_heads,
                           int dim, int vdim, int taps, float* out, int plain, int decay_per_head, int single, cudaStream_t s) {
  const DeltaShape sh{heads, kv_heads, dim, vdim, taps};
  if (const int st_ = check_delta(sh)) return st_;
  if (seqs <= 0) return kOk;
  TIE_REQUIRE(beta != nullptr || plain, "delta_rule: the delta rule needs beta");
  TIE_REQUIRE(seqs <= 65535 * 32 && heads <= 65535, "delta_rule: %d sequences x %d heads exceed the grid", seqs, heads);
  if (dtype == TIE_F32)
    return launch_delta_rule<float>(qn, kn, vn, beta, decay, decay_stride, state, state_stride, conv_state_off, proj, proj_stride,
                                    q_off, k_off, v_off, query_start, state_slots, seqs, sh, out, plain, decay_per_head, single, s);
  if (dtype == TIE_BF16)
    return launch_delta_rule<__nv_bfloat16>(qn, kn, vn, beta, decay, decay_stride, state, state_stride, conv_state_off, proj,
                                            proj_stride, q_off, k_off, v_off, query_start, state_slots, seqs, sh, out, plain, decay_per_head, single, s);
  set_error("unknown dtype code %d", dtype);
  return kBadArgument;
}

TIE_API int tie_delta_out(int dtype, const float* o, const float* gate, long long gate_stride, const float* w, float eps,
                          void* out, int tokens, int heads, int vdim, cudaStream_t s) {
  TIE_REQUIRE(tokens >= 0 && heads > 0 && vdim > 0, "delta_out: bad sizes tokens=%d heads=%d vdim=%d", tokens, heads, vdim);
  const long long items = static_cast<long long>(tokens) * heads;
  if (items == 0) return kOk;
  if (dtype == TIE_F32) {
    TIE_LAUNCH((delta_out_kernel<float>), ceil_div(items, 4), 128, 0, s, o, gate, gate_stride, w, eps, static_cast<float*>(out), heads,
               vdim, items);
  } else if (dtype == TIE_BF16) {
    TIE_LAUNCH((delta_out_kernel<__nv_bfloat16>), ceil_div(items, 4), 128, 0, s, o, gate, gate_stride, w, eps,
               static_cast<__nv_bfloat16*>(out), heads, vdim, items);
  } else {
    set_error("unknown dtype code %d", dtype);
    return kBadArgument;
  }
  TIE_RETURN_LAUNCH("delta_out");
}

// The plain recurrence read before it is written, with a weight per head and key channel on the token's own write
// (`bonus`, float [heads * dim]; `single` as above): o_t = (S + diag(bonus) k_t u_t^T)^T q_t, then S <- diag(decay_t) S + k_t u_t^T.
TIE_API int tie_delta_rule_bonus(int dtype, const float* qn, const float* kn, const float* vn, const float* beta,
                                 const float* decay, long long decay_stride, float* state, long long state_stride,
                                 long long conv_state_off, const void* proj, long long proj_stride, int q_off, int k_off,
                                 int v_off, const int* query_start, const int* state_slots, int seqs, int heads,
                                 int kv_heads, int dim, int vdim, int taps, float* out, const float* bonus, int single, cudaStream_t s) {
  const DeltaShape sh{heads, kv_heads, dim, vdim, taps};
  if (const int st_ = check_delta(sh)) return st_;
  if (seqs <= 0) return kOk;
  TIE_REQUIRE(bonus != nullptr && heads == kv_heads, "delta_rule_bonus: a weight per head and key channel, and a key head per head");
  TIE_REQUIRE(seqs <= 65535 * 32 && heads <= 65535, "delta_rule: %d sequences x %d heads exceed the grid", seqs, heads);
  if (dtype == TIE_F32)
    return launch_delta_rule<float>(qn, kn, vn, beta, decay, decay_stride, state, state_stride, conv_state_off, proj, proj_stride,
                                    q_off, k_off, v_off, query_start, state_slots, seqs, sh, out, 1, 0, single, s, bonus);
  if (dtype == TIE_BF16)
    return launch_delta_rule<__nv_bfloat16>(qn, kn, vn, beta, decay, decay_stride, state, state_stride, conv_state_off, proj,
                                            proj_stride, q_off, k_off, v_off, query_start, state_slots, seqs, sh, out, 1, 0, single, s, bonus);
  set_error("unknown dtype code %d", dtype);
  return kBadArgument;
}
