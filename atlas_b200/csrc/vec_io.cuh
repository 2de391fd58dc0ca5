// Loads and stores of V consecutive elements as fp32, for kernels that exist for bf16 and fp32 activations.
#pragma once
#include "common.cuh"

namespace atlas {

ATLAS_DEVICE float to_f32(float v) { return v; }
ATLAS_DEVICE float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> ATLAS_DEVICE T from_f32(float v);
template <> ATLAS_DEVICE float from_f32<float>(float v) { return v; }
template <> ATLAS_DEVICE __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

template <int V>
ATLAS_DEVICE void load_vec(const float* p, float (&f)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 r = *reinterpret_cast<const float4*>(p + i);
      f[i] = r.x; f[i + 1] = r.y; f[i + 2] = r.z; f[i + 3] = r.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = p[i];
  }
}
template <int V>
ATLAS_DEVICE void load_vec(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V % 8 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 8) {
      const uint4 r = *reinterpret_cast<const uint4*>(p + i);
      const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[j]));
        f[i + 2 * j] = a.x; f[i + 2 * j + 1] = a.y;
      }
    }
  } else if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const uint2 r = *reinterpret_cast<const uint2*>(p + i);
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
      f[i] = a.x; f[i + 1] = a.y; f[i + 2] = b.x; f[i + 3] = b.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int V>
ATLAS_DEVICE void store_vec(float* p, const float (&f)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = f[i];
  }
}
template <int V>
ATLAS_DEVICE void store_vec(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V % 8 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 8)
      *reinterpret_cast<uint4*>(p + i) = make_uint4(pack_bf16x2(f[i], f[i + 1]), pack_bf16x2(f[i + 2], f[i + 3]),
                                                    pack_bf16x2(f[i + 4], f[i + 5]), pack_bf16x2(f[i + 6], f[i + 7]));
  } else if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4)
      *reinterpret_cast<uint2*>(p + i) = make_uint2(pack_bf16x2(f[i], f[i + 1]), pack_bf16x2(f[i + 2], f[i + 3]));
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16_rn(f[i]);
  }
}

// sigmoid(v) for results that leave in T: the fast exponential and division where they are rounded to bf16
template <typename T> ATLAS_DEVICE float sigmoid_for(float v) { return 1.f / (1.f + expf(-v)); }
template <> ATLAS_DEVICE float sigmoid_for<__nv_bfloat16>(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }

// rows of stride `ld` at `p` can be read V elements at a time (a null pointer can)
template <typename T, int V>
inline bool vec_ok(const void* p, long long ld) {
  const size_t unit = V * sizeof(T) > 16 ? 16 : V * sizeof(T);
  return p == nullptr || ((reinterpret_cast<uintptr_t>(p) % unit) == 0 && (ld * (long long)sizeof(T)) % (long long)unit == 0);
}

}  // namespace atlas
