// Sublayer outputs on their way into the residual stream: a term is a tensor in the storage type or the float partial
// sums of a split product (added in split order), times a factor.
#pragma once

#include "common.cuh"

namespace tie {

struct Term {
  const void* tensor;       // [T, D] in the compute type, or null
  const float* partial;     // [splits, T, D] float, or null
  long long stride;         // T * D
  int splits;
  float scale;
};

template <typename T>
__device__ __forceinline__ float term_at(const Term& term, long long at) {
  float v = 0.0f;
  if (term.tensor != nullptr) v = ld(static_cast<const T*>(term.tensor) + at);
  else if (term.partial != nullptr) {
    for (int z = 0; z < term.splits; ++z) v += term.partial[z * term.stride + at];
  } else return 0.0f;
  return term.scale * v;
}

// Four columns at a time (every pointer on a 16-byte boundary; the terms' rows likewise).
template <typename T>
__device__ __forceinline__ void term_add4(const Term& term, long long at, float (&v)[4]) {
  if (term.tensor != nullptr) {
    float d[4];
    load4(static_cast<const T*>(term.tensor) + at, d);
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = fmaf(term.scale, d[e], v[e]);
  } else if (term.partial != nullptr) {
    float sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    for (int z = 0; z < term.splits; ++z) {
      float d[4];
      load4(term.partial + z * term.stride + at, d);
#pragma unroll
      for (int e = 0; e < 4; ++e) sum[e] += d[e];
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = fmaf(term.scale, sum[e], v[e]);
  }
}

// Up to four of them, added in order.
constexpr int kMaxTerms = 4;
struct Terms {
  Term t[kMaxTerms];
  int n;
};

inline bool terms_on16(const Terms& terms) {
  for (int i = 0; i < terms.n; ++i) {
    const Term& t = terms.t[i];
    if (reinterpret_cast<uintptr_t>(t.tensor) % 16 || reinterpret_cast<uintptr_t>(t.partial) % 16 || t.stride % 4) return false;
  }
  return true;
}

}  // namespace tie
