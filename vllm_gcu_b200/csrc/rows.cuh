// Rows of 16-bit or fp32 elements as fp32 vectors.
#pragma once
#include "common.cuh"

namespace b200 {

template <int V>
__device__ __forceinline__ void ldv(const float* p, float (&f)[V]) {
  if constexpr (V >= 4) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 u = *reinterpret_cast<const float4*>(p + i);
      f[i] = u.x; f[i + 1] = u.y; f[i + 2] = u.z; f[i + 3] = u.w;
    }
  } else {
    f[0] = p[0];
  }
}
template <int V>
__device__ __forceinline__ void ldv(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V == 8) {
    vec8_load<__nv_bfloat16>(p, f);
  } else if constexpr (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
    f[0] = __bfloat162float(p[0]);
  }
}
template <int V>
__device__ __forceinline__ void stv(float* p, const float (&f)[V]) {
  if constexpr (V >= 4) {
#pragma unroll
    for (int i = 0; i < V; i += 4)
      *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
  } else {
    p[0] = f[0];
  }
}
template <int V>
__device__ __forceinline__ void stv(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V == 8) {
    vec8_store<__nv_bfloat16>(p, f);
  } else if constexpr (V == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  } else {
    p[0] = __float2bfloat16(f[0]);
  }
}

// Threads for a row of H elements, V per thread, at most `most`.
static inline int row_threads(int H, int V, int most) {
  int n = (H / V + 31) / 32 * 32;
  return n < 32 ? 32 : (n > most ? most : n);
}

static inline bool aligned(const void* p, int bytes) {
  return (reinterpret_cast<uintptr_t>(p) % bytes) == 0;
}

}  // namespace b200
