// A recurrence with a diagonal state per channel whose step size depends on the token:
//
//     dt = softplus(raw + bias)                                   one per channel
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n
//     y_c = sum_n S[c, n] C_n + D_c x_c;   out_c = y_c * silu(z_c)
//
// S [channels, states] is float, lives in the request's slot and is carried from token to token. Channels do not depend on
// one another, so the work is cut by (sequence, 16 channels). LANES lanes of a warp share a channel, R neighbouring states
// each. Chunks of tokens come through two buffers in turn, filled by asynchronous copies while the other is worked on; a
// chunk's step sizes are formed once per channel, not once per lane. The lanes' partial read-outs of eight tokens are summed
// together: each exchange halves the tokens a lane still holds, so eight tokens cost seven exchanges (and log2(LANES / 8)
// more), not eight times log2(LANES).
#include <math.h>

#include <type_traits>

#include "common.cuh"

namespace tie {

constexpr int kScanChannels = 16;

template <typename T>
struct ScanArgs {
  const T* x;               // [rows, inner]: behind the convolution
  const T* z;               // the gate's columns
  const T* low;             // B at column b_off, C at column c_off
  const float* raw;         // [rows, inner]: the step sizes' projection
  const float *bias, *a2, *skip;     // [inner], [inner, states]: A * log2(e), [inner]
  float* state;
  T* out;                   // [rows, inner]
  long long x_stride, z_stride, low_stride, state_stride;
  const int* query_start;
  const int* state_slots;
  int b_off, c_off, inner, states, chunk;
  int wide;                 // rows and sections in whole 16-byte pieces: asynchronous copies of 16 bytes
};

__device__ __forceinline__ float ex2(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}
// 2^v for v <= 0 to half a unit in the last place and without a bias: a slow channel multiplies thousands of decays that are
// all close to one, and an approximation that errs to one side there shows in the float32 path. 2^v = 2^n e^(f ln 2) with n
// the nearest integer; |f ln 2| <= 0.347, where the exponential series to the seventh power leaves 5e-9.
__device__ __forceinline__ float ex2_precise(float v) {
  const float n = rintf(v), r = (v - n) * 0.69314718055994531f;
  float p = 1.0f / 5040.0f;
  p = fmaf(p, r, 1.0f / 720.0f);
  p = fmaf(p, r, 1.0f / 120.0f);
  p = fmaf(p, r, 1.0f / 24.0f);
  p = fmaf(p, r, 1.0f / 6.0f);
  p = fmaf(p, r, 0.5f);
  p = fmaf(p, r, 1.0f);
  p = fmaf(p, r, 1.0f);
  return v < -125.0f ? 0.0f : p * __int_as_float((static_cast<int>(n) + 127) << 23);
}
template <typename T>
__device__ __forceinline__ float decay_ex2(float v) {
  if constexpr (sizeof(T) == 4) return ex2_precise(v);
  else return ex2(v);
}
__device__ __forceinline__ void scan_copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}

// Sizes in bytes of what a chunk needs (all multiples of 16).
template <typename T>
struct ScanLayout {
  int n8, np, raw_x, raw_z, raw_dt, raw_bc, raw_bytes, steps, b, c, y, total;
  __host__ __device__ ScanLayout(int chunk, int states, int padded) {
    n8 = (states + 7) / 8 * 8, np = padded;
    raw_x = 0;
    raw_z = raw_x + chunk * kScanChannels * static_cast<int>(sizeof(T));
    raw_dt = raw_z + chunk * kScanChannels * static_cast<int>(sizeof(T));
    raw_bc = raw_dt + chunk * kScanChannels * 4;
    raw_bytes = raw_bc + 2 * chunk * n8 * static_cast<int>(sizeof(T));
    steps = 2 * raw_bytes;                                   // float2 (dt, dt x) per token and channel
    b = steps + chunk * kScanChannels * 8;
    c = b + chunk * np * 4;
    y = c + chunk * np * 4;
    total = y + chunk * kScanChannels * 4;
  }
};

template <typename T, int LANES, int R>
__global__ void __launch_bounds__(LANES * kScanChannels) selective_scan_kernel(ScanArgs<T> a) {
  extern __shared__ __align__(16) uint8_t scan_smem[];
  constexpr int THREADS = LANES * kScanChannels;
  const int s = blockIdx.y, c0 = blockIdx.x * kScanChannels;
  const int lane = threadIdx.x % LANES, ch = threadIdx.x / LANES, c = c0 + ch;
  const bool live = c < a.inner;
  float sr[R], ar[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {                // a weight: no kernel ahead writes it
    const int k = lane * R + r;
    ar[r] = live && k < a.states ? a.a2[static_cast<long long>(c) * a.states + k] : 0.0f;
  }
  pdl_wait();
  const int slot = a.state_slots[s];
  if (slot < 0) return;                        // a sequence that pads a captured batch
  const int t0 = a.query_start[s], n = a.query_start[s + 1] - t0;
  const ScanLayout<T> L(a.chunk, a.states, LANES * R);
  float* S = a.state + slot * a.state_stride + static_cast<long long>(c) * a.states;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int k = lane * R + r;
    sr[r] = live && k < a.states ? S[k] : 0.0f;
  }
  constexpr int V = Vec16<T>::N;
  auto fetch = [&](int k0, uint8_t* base) {
    const int cn = min(a.chunk, n - k0);
    T* xb = reinterpret_cast<T*>(base + L.raw_x);
    T* zb = reinterpret_cast<T*>(base + L.raw_z);
    float* db = reinterpret_cast<float*>(base + L.raw_dt);
    T* bb = reinterpret_cast<T*>(base + L.raw_bc);
    T* cb = bb + a.chunk * L.n8;
    if (a.wide) {
      constexpr int XP = kScanChannels / V, DP = kScanChannels / 4;
      for (int i = threadIdx.x; i < cn * XP; i += THREADS) {
        const int tc = i / XP, p = (i % XP) * V;
        const long long t = t0 + k0 + tc;
        if (c0 + p < a.inner) {
          scan_copy16(xb + tc * kScanChannels + p, a.x + t * a.x_stride + c0 + p);
          scan_copy16(zb + tc * kScanChannels + p, a.z + t * a.z_stride + c0 + p);
        }
      }
      for (int i = threadIdx.x; i < cn * DP; i += THREADS) {
        const int tc = i / DP, p = (i % DP) * 4;
        if (c0 + p < a.inner) scan_copy16(db + tc * kScanChannels + p, a.raw + (t0 + k0 + tc) * static_cast<long long>(a.inner) + c0 + p);
      }
      const int BP = L.n8 / V;
      for (int i = threadIdx.x; i < cn * BP; i += THREADS) {
        const int tc = i / BP, p = (i % BP) * V;
        const T* row = a.low + (t0 + k0 + tc) * a.low_stride;
        scan_copy16(bb + tc * L.n8 + p, row + a.b_off + p);
        scan_copy16(cb + tc * L.n8 + p, row + a.c_off + p);
      }
    } else {
      for (int i = threadIdx.x; i < cn * kScanChannels; i += THREADS) {
        const int tc = i / kScanChannels, p = i % kScanChannels;
        const long long t = t0 + k0 + tc;
        if (c0 + p < a.inner) {
          xb[i] = a.x[t * a.x_stride + c0 + p];
          zb[i] = a.z[t * a.z_stride + c0 + p];
          db[i] = a.raw[t * a.inner + c0 + p];
        }
      }
      for (int i = threadIdx.x; i < cn * a.states; i += THREADS) {
        const int tc = i / a.states, p = i % a.states;
        const T* row = a.low + (t0 + k0 + tc) * a.low_stride;
        bb[tc * L.n8 + p] = row[a.b_off + p];
        cb[tc * L.n8 + p] = row[a.c_off + p];
      }
    }
  };
  float2* steps = reinterpret_cast<float2*>(scan_smem + L.steps);
  float* bs = reinterpret_cast<float*>(scan_smem + L.b);
  float* cs = reinterpret_cast<float*>(scan_smem + L.c);
  float* ys = reinterpret_cast<float*>(scan_smem + L.y);
  fetch(0, scan_smem);
  int turn = 0;
  for (int k0 = 0; k0 < n; k0 += a.chunk, turn ^= 1) {
    const int cn = min(a.chunk, n - k0);
    const uint8_t* base = scan_smem + turn * L.raw_bytes;
    const T* xb = reinterpret_cast<const T*>(base + L.raw_x);
    const T* zb = reinterpret_cast<const T*>(base + L.raw_z);
    const float* db = reinterpret_cast<const float*>(base + L.raw_dt);
    const T* bb = reinterpret_cast<const T*>(base + L.raw_bc);
    const T* cb = bb + a.chunk * L.n8;
    asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
    __syncthreads();                           // this chunk is there, and everyone is through with the other buffer
    if (k0 + a.chunk < n) fetch(k0 + a.chunk, scan_smem + (turn ^ 1) * L.raw_bytes);
    for (int i = threadIdx.x; i < cn * kScanChannels; i += THREADS) {
      const int p = i % kScanChannels;
      float dt = 0.0f, x = 0.0f;
      if (c0 + p < a.inner) {
        const float v = db[i] + a.bias[c0 + p];
        dt = v > 20.0f ? v : log1pf(expf(v));
        x = ld(xb + i);
      }
      steps[i] = make_float2(dt, dt * x);
    }
    for (int i = threadIdx.x; i < cn * L.np; i += THREADS) {
      const int tc = i / L.np, p = i % L.np;
      bs[i] = p < a.states ? ld(bb + tc * L.n8 + p) : 0.0f;
      cs[i] = p < a.states ? ld(cb + tc * L.n8 + p) : 0.0f;
    }
    __syncthreads();
    // One token: this lane's share of the read-out.
    auto step = [&](int tc) -> float {
      const float2 d = steps[tc * kScanChannels + ch];
      const float* bt = bs + tc * L.np + lane * R;
      const float* ct = cs + tc * L.np + lane * R;
      float y = 0.0f;
#pragma unroll
      for (int r = 0; r < R; ++r) {
        sr[r] = fmaf(decay_ex2<T>(d.x * ar[r]), sr[r], d.y * bt[r]);
        y = fmaf(sr[r], ct[r], y);
      }
      return y;
    };
    for (int tb = 0; tb < cn; tb += 8) {
      float y[8];
      if (tb + 8 <= cn) {                      // no test between the tokens: their loads and exponentials overlap
#pragma unroll
        for (int q = 0; q < 8; ++q) y[q] = step(tb + q);
      } else {
#pragma unroll
        for (int q = 0; q < 8; ++q) {
          y[q] = 0.0f;
          if (tb + q < cn) y[q] = step(tb + q);
        }
      }
      // sums over the lanes: after the exchange over 4, 2, 1 lanes a lane holds one token (the one of its three low bits)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const bool up = lane & 4;
        const float give = up ? y[q] : y[q + 4], keep = up ? y[q + 4] : y[q];
        y[q] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
      }
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const bool up = lane & 2;
        const float give = up ? y[q] : y[q + 2], keep = up ? y[q + 2] : y[q];
        y[q] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
      }
      {
        const bool up = lane & 1;
        const float give = up ? y[0] : y[1], keep = up ? y[1] : y[0];
        y[0] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
      }
#pragma unroll
      for (int o = 8; o < LANES; o <<= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
      if (lane < 8 && tb + lane < cn) ys[(tb + lane) * kScanChannels + ch] = y[0];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < cn * kScanChannels; i += THREADS) {
      const int tc = i / kScanChannels, p = i % kScanChannels;
      if (c0 + p >= a.inner) continue;
      const float z = ld(zb + i);
      st(a.out + (t0 + k0 + tc) * static_cast<long long>(a.inner) + c0 + p,
         fmaf(a.skip[c0 + p], ld(xb + i), ys[i]) * (z / (1.0f + expf(-z))));
    }
  }
  pdl_launch_dependents();
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int k = lane * R + r;
    if (live && k < a.states) S[k] = sr[r];
  }
}

template <typename T, int LANES, int R>
static int launch_scan(ScanArgs<T> a, int seqs, int alone, cudaStream_t s) {
  a.chunk = alone ? 32 : 8;                    // single rows: small buffers, many blocks an SM
  while (a.chunk > 8 && ScanLayout<T>(a.chunk, a.states, LANES * R).total > 48 * 1024) a.chunk -= 8;
  const size_t smem = ScanLayout<T>(a.chunk, a.states, LANES * R).total;
  auto kernel = selective_scan_kernel<T, LANES, R>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess) {
    set_error("selective_scan: cannot reserve %zu bytes of shared memory", smem);
    return kCudaError;
  }
  const dim3 grid(ceil_div(a.inner, kScanChannels), seqs);
  if (alone) launch_kernel_alone(kernel, grid, dim3(LANES * kScanChannels), smem, s, a);
  else TIE_LAUNCH(kernel, grid, LANES * kScanChannels, smem, s, a);
  TIE_RETURN_LAUNCH("selective_scan");
}

template <typename T>
static int scan_of(const ScanArgs<T>& a, int seqs, int alone, cudaStream_t s) {
  if (!alone && a.states <= 16 && a.states > 8) return launch_scan<T, 8, 2>(a, seqs, alone, s);      // single rows: fewer, wider lanes
  if (a.states <= 8) return launch_scan<T, 8, 1>(a, seqs, alone, s);
  if (a.states <= 16) return launch_scan<T, 16, 1>(a, seqs, alone, s);
  if (a.states <= 32) return launch_scan<T, 16, 2>(a, seqs, alone, s);
  if (a.states <= 64) return launch_scan<T, 16, 4>(a, seqs, alone, s);
  if (a.states <= 128) return launch_scan<T, 32, 4>(a, seqs, alone, s);
  return launch_scan<T, 32, 8>(a, seqs, alone, s);
}

}  // namespace tie

using namespace tie;

// One recurrence over each sequence's rows of the step. x, z, low and out in the storage type; `alone`: start the blocks when
// the kernels ahead have drained (for steps with long portions).
TIE_API int tie_selective_scan(int dtype, const void* x, long long x_stride, const void* z, long long z_stride, const void* low,
                               long long low_stride, int b_off, int c_off, const float* raw, const float* bias, const float* a2,
                               const float* skip, float* state, long long state_stride, const int* query_start,
                               const int* state_slots, int seqs, int inner, int states, void* out, int alone, cudaStream_t s) {
  TIE_REQUIRE(inner > 0 && states > 0 && states <= 256 && b_off >= 0 && c_off >= b_off + states && low_stride >= c_off + states,
              "selective_scan: bad sizes inner=%d states=%d (1 to 256)", inner, states);
  if (seqs <= 0) return kOk;
  TIE_REQUIRE(seqs <= 65535, "selective_scan: %d sequences exceed the grid", seqs);
  auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int n8 = (states + 7) / 8 * 8;
  auto args = [&](auto* typed) {
    using T = std::remove_pointer_t<decltype(typed)>;
    constexpr int V = Vec16<T>::N;
    const int wide = on16(x) && on16(z) && on16(low) && on16(raw) && x_stride % V == 0 && z_stride % V == 0 && low_stride % V == 0 &&
                     b_off % V == 0 && c_off % V == 0 && inner % 8 == 0 && c_off >= b_off + n8 && low_stride >= c_off + n8;
    return ScanArgs<T>{static_cast<const T*>(x), static_cast<const T*>(z), static_cast<const T*>(low), raw, bias, a2, skip, state,
                       static_cast<T*>(out), x_stride, z_stride, low_stride, state_stride, query_start, state_slots, b_off, c_off, inner,
                       states, 0, wide};
  };
  if (dtype == TIE_F32) return scan_of<float>(args(static_cast<float*>(nullptr)), seqs, alone, s);
  if (dtype == TIE_BF16) return scan_of<__nv_bfloat16>(args(static_cast<__nv_bfloat16*>(nullptr)), seqs, alone, s);
  set_error("unknown dtype code %d", dtype);
  return kBadArgument;
}
