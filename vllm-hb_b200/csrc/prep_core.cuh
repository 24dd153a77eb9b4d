// Pieces of the kernels that turn projection rows into queries and cache entries.
#pragma once

#include "common.h"

namespace hb {

constexpr int kPrepThreads = 256;

// Elements in runs of V (1: any sizes; 8 bf16 or 4 fp32 numbers: 16-byte accesses).
template <typename T, int V>
struct Run {
  static __device__ __forceinline__ void load(float (&f)[V], const T* p) {
    if constexpr (V == 1) {
      f[0] = to_f32<T>(*p);
    } else {
      Vec16<T> v;
      v.load(p);
      v.unpack(f);
    }
  }
  static __device__ __forceinline__ void store(T* p, const float (&f)[V]) {
    if constexpr (V == 1) {
      *p = from_f32<T>(f[0]);
    } else {
      Vec16<T> v;
      v.pack(f);
      v.store(p);
    }
  }
};

// Where element d of kv head g of a row's key (value) lies in its pool.
__device__ __forceinline__ int64_t pool_at(int64_t slot, int G, int g, int width, int d) {
  return ((slot / HB_BLOCK_SIZE * G + g) * HB_BLOCK_SIZE + slot % HB_BLOCK_SIZE) * width + d;
}

// cs[i], cs[P + i] = gain * cos, sin of pos * frequency[i]: the angle less its whole turns in fp64, so
// that far positions keep the accuracy of near ones.
__device__ __forceinline__ void angles_of(float* cs, const double* frequency, int P, int pos, float gain) {
  const double turn = 6.283185307179586;
  for (int i = threadIdx.x; i < P; i += blockDim.x) {
    const double angle = (double)pos * frequency[i];
    float s, c;
    sincosf((float)(angle - turn * rint(angle * (1.0 / turn))), &s, &c);
    cs[i] = gain * c;
    cs[P + i] = gain * s;
  }
}

}  // namespace hb
