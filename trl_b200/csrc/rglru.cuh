// Parameters of the real-gated linear recurrent unit shared by rglru.cu and rglru_tcgen05.cu.
#pragma once

namespace trlb {

struct RgLru {
  int C, slots;
  const float* lam;        // [C]
  const float* gate_bias;  // [2, C]: of r, of i
  const float* y_bias;     // [C]
  float* state;            // [slots, C] fp32, or null
  float decay;             // log a = -decay r softplus(lam)
};

__device__ __forceinline__ float rg_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

}  // namespace trlb
