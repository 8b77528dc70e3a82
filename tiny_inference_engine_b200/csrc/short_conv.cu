// Short causal convolutions over time, one per channel, ahead of a mixer:
//
//     y_t = post + sum_j w[j] u_(t - taps + 1 + j),   u = a projection's column + pre,   zeros ahead of the sequence
//
// The last taps - 1 inputs u of every request (the tail) are part of its state: float [taps - 1, channels], oldest first,
// in its slot's row. A thread owns a few channels and walks down a tile of the step's rows with the inputs above it in
// registers; where a sequence starts, or the tile, the window comes from the rows above or from the tail.
//
//   short_conv_act    out = act(y), act the SiLU or none.
//   conv_rope_append  the channels are the q heads, then the k heads of an attention whose values are its keys: y of a k
//                     head goes into the value plane as it is; y of both, the first `rot` dimensions of each head turned in
//                     neighbouring pairs (2i, 2i+1) by position * f_i, into the key plane (k) and into `q_out` (q). The
//                     angle is formed in double precision as a fraction of a turn.
//   conv_tail         the tail after the step, for sequences whose rows lie in more than one tile. A sequence inside one
//                     tile leaves its tail in the two kernels above: the thread that reads a channel's old tail is the one
//                     that writes the new one.
#include <math.h>

#include <type_traits>

#include "common.cuh"

namespace tie {

struct ConvArgs {
  const void* proj;         // rows of `stride` elements; channel c is column col0 + c
  long long stride;
  int col0, channels, taps, rows, tile;
  const float* w;           // [taps, channels]: a tap of every channel side by side
  const float* pre;         // [channels] or null: added to every input (a projection's bias)
  const float* post;        // [channels] or null: added to y
  float* state;             // [slots, ...] rows of state_stride floats; the tail starts at tail_off
  long long state_stride, tail_off;
  const int* seq_of_row;
  const int* query_start;
  const int* state_slots;
};

constexpr int kConvThreads = 128;
constexpr int kConvMaxTile = 8;

// V channels of a row. VEC: four in one read; else the first n of them one by one.
template <typename T, int V, bool VEC>
__device__ __forceinline__ void conv_load(const T* p, int n, float (&v)[V]) {
  if constexpr (VEC) {
    static_assert(V == 4, "rows come four channels at a time");
    load4(p, v);
  } else {
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = e < n ? ld(p + e) : 0.0f;
  }
}

// Rows row0 .. row1-1 of channels c .. c+n-1 (n <= V); emit(row, y) for each. TAPS >= a.taps: the window's length here.
template <typename T, int V, int TAPS, bool VEC, typename Emit>
__device__ __forceinline__ void conv_walk(const ConvArgs& a, int c, int n, int row0, int row1, Emit emit) {
  float w[TAPS][V], win[TAPS][V], pre[V], post[V];      // tap i weighs the input TAPS - 1 - i rows above
#pragma unroll
  for (int i = 0; i < TAPS; ++i) {
    const int j = i - (TAPS - a.taps);
#pragma unroll
    for (int e = 0; e < V; ++e) w[i][e] = j >= 0 && e < n ? a.w[static_cast<long long>(j) * a.channels + c + e] : 0.0f;
  }
#pragma unroll
  for (int e = 0; e < V; ++e) {
    pre[e] = a.pre != nullptr && e < n ? a.pre[c + e] : 0.0f;
    post[e] = a.post != nullptr && e < n ? a.post[c + e] : 0.0f;
  }
  const T* col = static_cast<const T*>(a.proj) + a.col0 + c;
  // the tile's rows and their sequences, all asked for at once
  float rows[kConvMaxTile][V];
  int seqs[kConvMaxTile];
#pragma unroll
  for (int i = 0; i < kConvMaxTile; ++i) {
    if (row0 + i < row1) {
      seqs[i] = a.seq_of_row[row0 + i];
      conv_load<T, V, VEC>(col + static_cast<long long>(row0 + i) * a.stride, n, rows[i]);
    }
  }
  int seq = -1, last = -1;
  bool keeps = false;
  float* tail = nullptr;
#pragma unroll
  for (int i8 = 0; i8 < kConvMaxTile; ++i8) {
    const int t = row0 + i8;
    if (t >= row1) break;
    const int s = seqs[i8];
    if (s != seq) {
      seq = s;
      const int q0 = a.query_start[s], q1 = a.query_start[s + 1], slot = a.state_slots[s], j = t - q0;
      last = q1 - 1;
      tail = slot >= 0 && a.taps > 1 ? a.state + slot * a.state_stride + a.tail_off + c : nullptr;
      keeps = tail != nullptr && q0 / a.tile == last / a.tile;
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i) {
        const int back = TAPS - 1 - i;
#pragma unroll
        for (int e = 0; e < V; ++e) win[i][e] = 0.0f;
        if (back > a.taps - 1) continue;
        if (back <= j) {
          conv_load<T, V, VEC>(col + static_cast<long long>(t - back) * a.stride, n, win[i]);
#pragma unroll
          for (int e = 0; e < V; ++e) win[i][e] += pre[e];
        } else if (tail != nullptr) {
          const float* from = tail + static_cast<long long>(j + a.taps - 1 - back) * a.channels;
#pragma unroll
          for (int e = 0; e < V; ++e)
            if (e < n) win[i][e] = from[e];
        }
      }
    }
    float y[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      win[TAPS - 1][e] = rows[i8][e] + pre[e];
      y[e] = post[e];
#pragma unroll
      for (int i = 0; i < TAPS; ++i) y[e] = fmaf(w[i][e], win[i][e], y[e]);
    }
    emit(t, y);
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
#pragma unroll
      for (int e = 0; e < V; ++e) win[i][e] = win[i + 1][e];
    }
    if (keeps && t == last) {
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i) {
        const int at = i - (TAPS - a.taps);
        if (at < 0) continue;
#pragma unroll
        for (int e = 0; e < V; ++e)
          if (e < n) tail[static_cast<long long>(at) * a.channels + e] = win[i][e];
      }
    }
  }
}

template <typename T, int V, int TAPS, bool VEC>
__global__ void __launch_bounds__(kConvThreads) short_conv_act_kernel(ConvArgs a, int silu, T* __restrict__ out, long long out_stride) {
  pdl_sync();
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * V;
  if (c >= a.channels) return;
  const int n = min(V, a.channels - c), row0 = blockIdx.y * a.tile;
  conv_walk<T, V, TAPS, VEC>(a, c, n, row0, min(a.rows, row0 + a.tile), [&](int t, float (&y)[V]) {
    if (silu) {
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = y[e] / (1.0f + expf(-y[e]));
    }
    T* o = out + t * out_stride + c;
    if constexpr (VEC) {
      store4(o, y);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e)
        if (e < n) st(o + e, y[e]);
    }
  });
}

struct ConvRopeArgs {
  const int* positions;
  const double* turns;      // [rot / 2]: turns a position, f_i / (2 pi); null without rotation
  int rot;
  const int* slots;         // cache slot of every row; negative: nothing is written
  void *k_cache, *v_cache;  // [pages, kv_heads, page, dim]
  void* q_out;              // [rows, q_heads * dim]
  int q_heads, kv_heads, dim, page_size, k_col;     // k heads start at channel k_col
};

template <typename T, int V, int TAPS, bool VEC>
__global__ void __launch_bounds__(kConvThreads) conv_rope_append_kernel(ConvArgs a, ConvRopeArgs r) {
  pdl_sync();
  const int per_head = (r.dim + V - 1) / V;
  const int item = blockIdx.x * kConvThreads + threadIdx.x;
  if (item >= (r.q_heads + r.kv_heads) * per_head) return;
  const int head = item / per_head, d0 = (item % per_head) * V;
  const bool is_q = head < r.q_heads;
  const int kvh = head - r.q_heads;
  const int c = (is_q ? head * r.dim : r.k_col + kvh * r.dim) + d0;
  const int n = min(V, r.dim - d0), row0 = blockIdx.y * a.tile;
  auto put = [&](T* o, const float (&y)[V]) {
    if constexpr (VEC) {
      store4(o, y);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e)
        if (e < n) st(o + e, y[e]);
    }
  };
  conv_walk<T, V, TAPS, VEC>(a, c, n, row0, min(a.rows, row0 + a.tile), [&](int t, float (&y)[V]) {
    long long at = 0;
    int slot = -1;
    if (!is_q) {
      slot = r.slots[t];
      if (slot >= 0) {
        at = ((static_cast<long long>(slot / r.page_size) * r.kv_heads + kvh) * r.page_size + slot % r.page_size) * r.dim + d0;
        put(static_cast<T*>(r.v_cache) + at, y);
      }
    }
    if (d0 < r.rot) {
      const double pos = static_cast<double>(r.positions[t]);
#pragma unroll
      for (int e = 0; e + 1 < V; e += 2) {
        if (d0 + e + 1 < r.rot) {
          double turn = pos * r.turns[(d0 + e) >> 1];
          turn -= rint(turn);
          float sn, cs;
          sincospif(static_cast<float>(2.0 * turn), &sn, &cs);
          const float u = y[e], v = y[e + 1];
          y[e] = fmaf(u, cs, -(v * sn));
          y[e + 1] = fmaf(v, cs, u * sn);
        }
      }
    }
    if (is_q) put(static_cast<T*>(r.q_out) + static_cast<long long>(t) * r.q_heads * r.dim + head * r.dim + d0, y);
    else if (slot >= 0) put(static_cast<T*>(r.k_cache) + at, y);
  });
}

template <typename T>
__global__ void __launch_bounds__(256) conv_tail_kernel(ConvArgs a) {
  pdl_sync();
  const int s = blockIdx.y, slot = a.state_slots[s];
  const int q0 = a.query_start[s], q1 = a.query_start[s + 1], n = q1 - q0, keep = a.taps - 1;
  if (slot < 0 || n <= 0 || q0 / a.tile == (q1 - 1) / a.tile) return;
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= a.channels) return;
  float* tail = a.state + slot * a.state_stride + a.tail_off + c;
  const T* col = static_cast<const T*>(a.proj) + a.col0 + c;
  const float pre = a.pre != nullptr ? a.pre[c] : 0.0f;
  for (int i = 0; i < keep; ++i) {
    const int from = n - keep + i;        // offset in the step of the token that lands at place i
    tail[static_cast<long long>(i) * a.channels] = from >= 0 ? ld(col + static_cast<long long>(q0 + from) * a.stride) + pre
                                                             : tail[static_cast<long long>(n + i) * a.channels];
  }
}

}  // namespace tie

using namespace tie;

static int check_conv(const ConvArgs& a, const char* what) {
  TIE_REQUIRE(a.channels > 0 && a.taps >= 1 && a.taps <= 16 && a.rows >= 0 && a.tile >= 1 && a.tile <= kConvMaxTile && a.w != nullptr,
              "%s: bad sizes channels=%d taps=%d (1 to 16) rows=%d tile=%d (1 to 8)", what, a.channels, a.taps, a.rows, a.tile);
  TIE_REQUIRE(a.taps == 1 || a.state != nullptr, "%s: a convolution of %d taps needs a state", what, a.taps);
  TIE_REQUIRE(ceil_div(a.rows, a.tile) <= 65535, "%s: %d rows in tiles of %d exceed the grid", what, a.rows, a.tile);
  return kOk;
}

template <typename T>
static bool conv_vec(const ConvArgs& a) {
  constexpr int V = 4;
  return a.taps <= 4 && a.stride % V == 0 && a.col0 % V == 0 && reinterpret_cast<uintptr_t>(a.proj) % 16 == 0;
}

TIE_API int tie_short_conv_act(int dtype, const void* proj, long long stride, int col0, int channels, int taps, int rows, int tile,
                               const float* w, const float* pre, const float* post, float* state, long long state_stride,
                               long long tail_off, const int* seq_of_row, const int* query_start, const int* state_slots, int silu,
                               void* out, long long out_stride, cudaStream_t s) {
  const ConvArgs a{proj, stride, col0, channels, taps, rows, tile, w, pre, post, state, state_stride, tail_off, seq_of_row, query_start, state_slots};
  if (const int st_ = check_conv(a, "short_conv_act")) return st_;
  if (rows == 0) return kOk;
  auto run = [&](auto* typed) {
    using T = std::remove_pointer_t<decltype(typed)>;
    constexpr int V = 4;
    if (conv_vec<T>(a) && channels % V == 0 && out_stride % V == 0 && reinterpret_cast<uintptr_t>(out) % 16 == 0)
      TIE_LAUNCH((short_conv_act_kernel<T, V, 4, true>), dim3(ceil_div(channels / V, kConvThreads), ceil_div(rows, tile)), kConvThreads, 0, s,
                 a, silu, static_cast<T*>(out), out_stride);
    else
      TIE_LAUNCH((short_conv_act_kernel<T, 2, 16, false>), dim3(ceil_div((channels + 1) / 2, kConvThreads), ceil_div(rows, tile)),
                 kConvThreads, 0, s, a, silu, static_cast<T*>(out), out_stride);
  };
  if (dtype == TIE_F32) run(static_cast<float*>(nullptr));
  else if (dtype == TIE_BF16) run(static_cast<__nv_bfloat16*>(nullptr));
  else {
    set_error("unknown dtype code %d", dtype);
    return kBadArgument;
  }
  TIE_RETURN_LAUNCH("short_conv_act");
}

TIE_API int tie_conv_rope_append(int dtype, const void* proj, long long stride, int col0, int channels, int taps, int rows, int tile,
                                 const float* w, const float* pre, float* state, long long state_stride, long long tail_off,
                                 const int* seq_of_row, const int* query_start, const int* state_slots, const int* positions,
                                 const double* turns, int rot, const int* slots, void* k_cache, void* v_cache, void* q_out, int q_heads,
                                 int kv_heads, int dim, int page_size, int k_col, cudaStream_t s) {
  const ConvArgs a{proj, stride, col0, channels, taps, rows, tile, w, pre, nullptr, state, state_stride, tail_off, seq_of_row, query_start, state_slots};
  if (const int st_ = check_conv(a, "conv_rope_append")) return st_;
  TIE_REQUIRE(q_heads > 0 && kv_heads > 0 && dim > 0 && page_size > 0 && k_col >= q_heads * dim && channels >= k_col + kv_heads * dim &&
                  rot >= 0 && rot % 2 == 0 && rot <= dim && (rot == 0 || turns != nullptr),
              "conv_rope_append: bad geometry q_heads=%d kv_heads=%d dim=%d rot=%d k_col=%d channels=%d", q_heads, kv_heads, dim, rot, k_col,
              channels);
  if (rows == 0) return kOk;
  const ConvRopeArgs r{positions, turns, rot, slots, k_cache, v_cache, q_out, q_heads, kv_heads, dim, page_size, k_col};
  auto run = [&](auto* typed) {
    using T = std::remove_pointer_t<decltype(typed)>;
    constexpr int V = 4;
    auto on16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    if (conv_vec<T>(a) && dim % V == 0 && k_col % V == 0 && on16(k_cache) && on16(v_cache) && on16(q_out))
      TIE_LAUNCH((conv_rope_append_kernel<T, V, 4, true>), dim3(ceil_div((q_heads + kv_heads) * (dim / V), kConvThreads), ceil_div(rows, tile)),
                 kConvThreads, 0, s, a, r);
    else
      TIE_LAUNCH((conv_rope_append_kernel<T, 2, 16, false>),
                 dim3(ceil_div((q_heads + kv_heads) * ((dim + 1) / 2), kConvThreads), ceil_div(rows, tile)), kConvThreads, 0, s, a, r);
  };
  if (dtype == TIE_F32) run(static_cast<float*>(nullptr));
  else if (dtype == TIE_BF16) run(static_cast<__nv_bfloat16*>(nullptr));
  else {
    set_error("unknown dtype code %d", dtype);
    return kBadArgument;
  }
  TIE_RETURN_LAUNCH("conv_rope_append");
}

// For the first `seqs` sequences of the step.
TIE_API int tie_conv_tail(int dtype, const void* proj, long long stride, int col0, int channels, int taps, int tile, const float* pre,
                          float* state, long long state_stride, long long tail_off, const int* query_start, const int* state_slots,
                          int seqs, cudaStream_t s) {
  const ConvArgs a{proj, stride, col0, channels, taps, 0, tile, state, pre, nullptr, state, state_stride, tail_off, nullptr,
                   query_start, state_slots};
  if (const int st_ = check_conv(a, "conv_tail")) return st_;
  if (seqs <= 0 || taps <= 1) return kOk;
  TIE_REQUIRE(seqs <= 65535, "conv_tail: %d sequences exceed the grid", seqs);
  const dim3 grid(ceil_div(channels, 256), seqs);
  if (dtype == TIE_F32) {
    TIE_LAUNCH((conv_tail_kernel<float>), grid, 256, 0, s, a);
  } else if (dtype == TIE_BF16) {
    TIE_LAUNCH((conv_tail_kernel<__nv_bfloat16>), grid, 256, 0, s, a);
  } else {
    set_error("unknown dtype code %d", dtype);
    return kBadArgument;
  }
  TIE_RETURN_LAUNCH("conv_tail");
}
