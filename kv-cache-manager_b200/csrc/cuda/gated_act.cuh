// Activations of gated feed-forwards: what becomes of the gate's and the up projection's value of one element.
//   kGatedSilu    : silu(g) * u                (silu is rounded to the storage type before the product)
//   kGatedClamped : g' = min(g, limit), u' = clamp(u, -limit, limit);  g' * sigmoid(alpha g') * (u' + 1)
// The values arrive as the product would store them; the arithmetic is float.
// And of ungated ones, of one value z:
//   kUnaryReluSq   : max(z, 0)^2
//   kUnaryGeluTanh : 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), evaluated as z / (1 + exp(-2 sqrt(2/pi) (z + 0.044715 z^3)))
#pragma once
#include "common.cuh"

namespace kvcm {

enum GatedKind { kGatedNone = 0, kGatedSilu = 1, kGatedClamped = 2 };

enum UnaryKind { kUnaryNone = 0, kUnaryReluSq = 1, kUnaryGeluTanh = 2 };

struct GatedAct {
  float limit, alpha;                                          // kGatedClamped
  int unary;                                                   // ungated products: UnaryKind of what is stored
};

__device__ __forceinline__ float unary_act(int kind, float z) {
  if (kind == kUnaryReluSq) {
    const float r = fmaxf(z, 0.f);
    return r * r;
  }
  if (kind == kUnaryGeluTanh) return z / (1.f + expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z)));
  return z;
}
// The same where the result is rounded to bfloat16: CUDA's fast exponential and division (a few units in float's last place;
// a denominator beyond 2^126 gives zero, which is the limit).  Every kernel that stores bfloat16 takes this one.
__device__ __forceinline__ float unary_act_16(int kind, float z) {
  if (kind == kUnaryGeluTanh) return __fdividef(z, 1.f + __expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z)));
  return unary_act(kind, z);
}

template <int KIND, typename T>
__device__ __forceinline__ float gated_act(float g, float u, const GatedAct& a) {
  if constexpr (KIND == kGatedClamped) {
    const float gc = fminf(g, a.limit), uc = fminf(fmaxf(u, -a.limit), a.limit);
    return gc / (1.f + expf(-a.alpha * gc)) * (uc + 1.f);
  } else {
    return Store<T>::round(g / (1.f + expf(-g))) * u;
  }
}

}  // namespace kvcm
