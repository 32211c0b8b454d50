// Device helpers shared by the kernels of the layered decoders (mixers.cu, grouped_attn.cu, rglru*.cu, mixer_attn_*.cu,
// grouped_decode_*.cu, latent_decode_*.cu, mlstm_chunk_*.cu).
#pragma once
#include "common.cuh"

namespace trlb {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// Four consecutive elements (16-byte aligned fp32, 8-byte aligned bf16).
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

__device__ __forceinline__ float gelu_erf_f(float v) { return 0.5f * v * (1.f + erff(v * 0.70710678118654752f)); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
// 0.5 z (1 + tanh(w)) with w = sqrt(2 / pi) (z + 0.044715 z^3), as z sigmoid(2 w)
__device__ __forceinline__ float gelu_tanh_f(float z) { return z * sigmoid_f(1.5957691216057308f * (z + 0.044715f * z * z * z)); }

// The same on the exp2 / reciprocal approximations (relative error of a few 2^-23), for results that are rounded to bf16 or
// multiplied into fp32 sums of bf16 products.
__device__ __forceinline__ float fast_sigmoid(float z) {
  return __fdividef(1.f, 1.f + fast_exp2(fminf(-1.4426950408889634f * z, 125.f)));
}
__device__ __forceinline__ float fast_gelu_tanh(float z) {
  return z * fast_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z));
}
template <typename T>
__device__ __forceinline__ float sigmoid_t(float z) { return sizeof(T) == 2 ? fast_sigmoid(z) : sigmoid_f(z); }
template <typename T>
__device__ __forceinline__ float gelu_tanh_t(float z) { return sizeof(T) == 2 ? fast_gelu_tanh(z) : gelu_tanh_f(z); }

// tanh for capping attention scores in fp32.  Far from zero: 1 - 2 / (exp(2 x) + 1).  Near zero (|x| <= CAP_SERIES) the Taylor
// series through x^11, relative error below 2e-8, which costs no special-function work.
constexpr float CAP_SERIES = 0.35f;
__device__ __forceinline__ float tanh_exp(float x) {
  const float e = fast_exp2(fminf(2.8853900817779268f * x, 126.f));
  return fmaf(-2.f, __fdividef(1.f, e + 1.f), 1.f);
}
__device__ __forceinline__ float tanh_series(float x) {
  const float y = x * x;
  float p = fmaf(y, -1382.f / 155925.f, 62.f / 2835.f);
  p = fmaf(y, p, -17.f / 315.f);
  p = fmaf(y, p, 2.f / 15.f);
  p = fmaf(y, p, -1.f / 3.f);
  return fmaf(x * y, p, x);
}
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// A shared-memory matrix descriptor moved on by a multiple of 16 bytes (the address field cannot overflow inside 228 KB).  The
// thread that issues MMAs runs alone, so what it computes per MMA is paid in full: descriptors are built once.
__device__ __forceinline__ uint64_t desc_at(uint64_t desc, uint32_t bytes) { return desc + (bytes >> 4); }

// Sums `a` and `b` over the block (at most 32 warps); `red` is 64 floats of shared memory.  All threads get the result.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();
  if (lane == 0) { red[wid] = a; red[32 + wid] = b; }
  __syncthreads();
  a = b = 0.f;
  for (int w = 0; w < nw; ++w) { a += red[w]; b += red[32 + w]; }
  return make_float2(a, b);
}

}  // namespace trlb
