// Rotary positions, for kernels that prepare queries and keys: which dimensions of a rotated part form a pair, and the cosine and
// sine of a pair's angle at a position.
#pragma once

#include "common.cuh"

namespace tie {

struct Rotation {
  const float* inv_freq;    // [rot / 2]: angle = float(position) * inv_freq[i], a float product; or
  const double* turns;      // [rot / 2]: position * turns[i] full turns, formed and reduced in double (far positions lose nothing)
  int rot;                  // dimensions that are rotated (0: none)
  int neighbours;           // pairs (2i, 2i + 1); otherwise (i, i + rot / 2)

  __device__ __forceinline__ bool on() const { return inv_freq != nullptr || turns != nullptr; }
  __device__ __forceinline__ int first(int i) const { return neighbours ? 2 * i : i; }
  __device__ __forceinline__ int second(int i) const { return neighbours ? 2 * i + 1 : i + rot / 2; }
  __device__ __forceinline__ void angle(int position, int i, float& c, float& s) const {
    if (turns != nullptr) {
      double turn = static_cast<double>(position) * turns[i];
      turn -= rint(turn);
      sincospif(static_cast<float>(2.0 * turn), &s, &c);
    } else {
      const float a = static_cast<float>(position) * inv_freq[i];
      c = cosf(a), s = sinf(a);
    }
  }
};

}  // namespace tie
