// Activations of gated feed-forwards: what becomes of the gate's and the up projection's value of one element.
//   kGatedSilu    : silu(g) * u                (silu is rounded to the storage type before the product)
//   kGatedClamped : g' = min(g, limit), u' = clamp(u, -limit, limit);  g' * sigmoid(alpha g') * (u' + 1)
// The values arrive as the product would store them; the arithmetic is float.
#pragma once
#include "common.cuh"

namespace kvcm {

enum GatedKind { kGatedNone = 0, kGatedSilu = 1, kGatedClamped = 2 };

struct GatedAct {
  float limit, alpha;                                          // kGatedClamped
};

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
