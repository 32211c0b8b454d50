// Real-gated linear recurrent unit of the layered decoders (Griffin's recurrent block): short causal convolution, recurrence
// over prompts and one decode step, for every size and dtype.  bf16 models whose blocks fit the tensor-core kernels run
// rglru_tcgen05.cu instead of the scan and the step here.
//
//     u_t = conv(x)_t,   log a_t = -decay r_t softplus(lam),   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,   out_t = S_t gelu(y_t)
//
// T is the model dtype; states, gates and decays are fp32.  Compiled without fast-math (csrc/build.py: EXACT_MATH).
#include <type_traits>

#include "mixers.cuh"
#include "rglru.cuh"

namespace trlb {

// u[t, c] = bias[c] + sum_j w[c, taps - 1 - j] (x[t - j, c] + xb[c]), taps before the start of a sequence left out.
// One thread per channel group of VEC and CONV_TOK tokens.
constexpr int CONV_TOK = 16;
template <typename T, int VEC, int TAPS>  // TAPS 0: any number, inputs read again for every tap
__global__ void __launch_bounds__(128)
conv_prompt_kernel(const T* __restrict__ x, long long ld, const float* __restrict__ xb, const float* __restrict__ w,
                   const float* __restrict__ bias, const int* __restrict__ positions, int n_tok, int C, int taps, T* __restrict__ u) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC;
  if (c >= C) return;
  const int t0 = blockIdx.y * CONV_TOK, t1 = min(n_tok, t0 + CONV_TOK);
  auto load = [&](int t, float (&d)[VEC]) {
    const T* p = x + (size_t)t * ld + c;
    if (VEC == 4) {
      const float4 v = load4(p);
      d[0] = v.x; d[1 % VEC] = v.y; d[2 % VEC] = v.z; d[3 % VEC] = v.w;
    } else {
      d[0] = to_f(p[0]);
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) d[i] += xb[c + i];
  };
  auto store = [&](int t, const float (&o)[VEC]) {
    if (VEC == 4) store4(u + (size_t)t * C + c, make_float4(o[0], o[1 % VEC], o[2 % VEC], o[3 % VEC]));
    else u[(size_t)t * C + c] = from_f<T>(o[0]);
  };
  float b[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) b[i] = bias[c + i];
  if constexpr (TAPS > 0) {
    float wt[TAPS][VEC], h[TAPS][VEC];  // h[j]: input of j tokens ago
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < VEC; ++i) { wt[j][i] = w[(size_t)(c + i) * TAPS + TAPS - 1 - j]; h[j][i] = 0.f; }
#pragma unroll
    for (int j = 1; j < TAPS; ++j)
      if (t0 - j >= 0) load(t0 - j, h[j - 1]);
    for (int t = t0; t < t1; ++t) {
      const int pos = positions[t];
#pragma unroll
      for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
        for (int i = 0; i < VEC; ++i) h[j][i] = h[j - 1][i];
      load(t, h[0]);
      float o[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = b[i];
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
        if (pos >= j) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) o[i] += wt[j][i] * h[j][i];
        }
      store(t, o);
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      const int pos = positions[t];
      float o[VEC], d[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = b[i];
      for (int j = 0; j < taps && j <= pos; ++j) {
        load(t - j, d);
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[i] += w[(size_t)(c + i) * taps + taps - 1 - j] * d[i];
      }
      store(t, o);
    }
  }
}

// The last taps - 1 inputs of every sequence, oldest first, zeros where it is shorter: state [slots, taps - 1, C].
template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const T* __restrict__ x, long long ld, const float* __restrict__ xb, const int* __restrict__ cu,
                  const int* __restrict__ seq_slot, int C, int keep, int slots, float* __restrict__ state) {
  const int seq = blockIdx.y, slot = seq_slot[seq], c = blockIdx.x * 256 + threadIdx.x;
  if (c >= C || slot < 0 || slot >= slots) return;
  const int beg = cu[seq], end = cu[seq + 1];
  for (int j = 0; j < keep; ++j) {
    const int t = end - keep + j;
    state[((size_t)slot * keep + j) * C + c] = t >= beg ? to_f(x[(size_t)t * ld + c]) + xb[c] : 0.f;
  }
}

// One token per slot: x is the slot's share of the input sums (cleared), the kept inputs move up by one.  One thread per slot
// and VEC channels.
template <typename T, int VEC>
__global__ void __launch_bounds__(128)
conv_step_kernel(float* __restrict__ x, long long ld, const float* __restrict__ xb, const float* __restrict__ w,
                 const float* __restrict__ bias, const int* __restrict__ seq_lens, int C, int taps, float* __restrict__ state,
                 T* __restrict__ u) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * VEC;
  if (c >= C) return;
  float* st = state + (size_t)b * (taps - 1) * C + c;
  float* xr = x + (size_t)b * ld + c;
  const float* wc = w + (size_t)c * taps;
  auto get = [](const float* p, float (&v)[VEC]) {
    if (VEC == 4) {
      const float4 t = load4(p);
      v[0] = t.x; v[1 % VEC] = t.y; v[2 % VEC] = t.z; v[3 % VEC] = t.w;
    } else {
      v[0] = *p;
    }
  };
  auto put = [](auto* p, const float (&v)[VEC]) {
    if (VEC == 4) store4(p, make_float4(v[0], v[1 % VEC], v[2 % VEC], v[3 % VEC]));
    else *p = from_f<typename std::remove_reference<decltype(*p)>::type>(v[0]);
  };
  float in[VEC], o[VEC], h[VEC], t[VEC];
  get(xr, in);
  get(xb + c, t);
  get(bias + c, o);
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    in[i] += t[i];
    t[i] = 0.f;
  }
  put(xr, t);
  if (seq_lens[b] < 0) {
    put(u + (size_t)b * C + c, t);
    return;
  }
#pragma unroll 3
  for (int j = 0; j < taps - 1; ++j) {
    get(st + (size_t)j * C, h);
#pragma unroll
    for (int i = 0; i < VEC; ++i) o[i] += wc[(size_t)i * taps + j] * h[i];
    if (j > 0) put(st + (size_t)(j - 1) * C, h);
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) o[i] += wc[(size_t)i * taps + taps - 1] * in[i];
  if (taps > 1) put(st + (size_t)(taps - 2) * C, in);
  put(u + (size_t)b * C + c, o);
}

// Recurrence over packed prompts: one thread per (sequence, channel).  z [T, 2, C] fp32: logits of r and i without their biases.
template <typename T>
__global__ void __launch_bounds__(64)
rglru_scan_kernel(const RgLru p, const float* __restrict__ z, const T* __restrict__ u, const T* __restrict__ y, long long y_ld,
                  const int* __restrict__ cu, const int* __restrict__ seq_slot, T* __restrict__ out) {
  const int seq = blockIdx.y, c = blockIdx.x * 64 + threadIdx.x;
  if (c >= p.C) return;
  const float sp = rg_softplus(p.lam[c]), br = p.gate_bias[c], bi = p.gate_bias[p.C + c], by = p.y_bias[c];
  float S = 0.f;
  for (int t = cu[seq]; t < cu[seq + 1]; ++t) {
    const float r = sigmoid_f(z[(size_t)t * 2 * p.C + c] + br), i = sigmoid_f(z[(size_t)t * 2 * p.C + p.C + c] + bi);
    const float la = -p.decay * r * sp;
    S = expf(la) * S + sqrtf(-expm1f(2.f * la)) * i * to_f(u[(size_t)t * p.C + c]);
    out[(size_t)t * p.C + c] = from_f<T>(S * gelu_tanh_f(to_f(y[(size_t)t * y_ld + c]) + by));
  }
  if (seq_slot != nullptr) {
    const int slot = seq_slot[seq];
    if (slot >= 0 && slot < p.slots) p.state[(size_t)slot * p.C + c] = S;
  }
}

// One token per slot: z [B, 2, C]; y: the slot's share of the input sums (cleared).
template <typename T>
__global__ void __launch_bounds__(128)
rglru_step_kernel(const RgLru p, const float* __restrict__ z, const T* __restrict__ u, float* __restrict__ y, long long y_ld,
                  const int* __restrict__ seq_lens, T* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
  if (c >= p.C) return;
  const float yv = y[(size_t)b * y_ld + c] + p.y_bias[c];
  y[(size_t)b * y_ld + c] = 0.f;
  float o = 0.f;
  if (seq_lens[b] >= 0) {
    const float r = sigmoid_f(z[(size_t)b * 2 * p.C + c] + p.gate_bias[c]);
    const float i = sigmoid_f(z[(size_t)b * 2 * p.C + p.C + c] + p.gate_bias[p.C + c]);
    const float la = -p.decay * r * rg_softplus(p.lam[c]);
    float* S = p.state + (size_t)b * p.C + c;
    o = expf(la) * *S + sqrtf(-expm1f(2.f * la)) * i * to_f(u[(size_t)b * p.C + c]);
    *S = o;
    o *= gelu_tanh_f(yv);
  }
  out[(size_t)b * p.C + c] = from_f<T>(o);
}

}  // namespace trlb

using namespace trlb;
using bf16 = __nv_bfloat16;
#define PDL trlb_host::pdl_enabled()

// x [n_tok rows of ld] -> u [n_tok, C]; w [C, taps] fp32.  state (null: not kept) [slots, taps - 1, C] of seq_slot[seq].
TRLB_API int trlb_conv_prompt(const void* x, long long ld, const float* xb, const float* w, const float* bias, const int* positions,
                              int n_tok, int C, int taps, const int* cu, int n_seq, const int* seq_slot, int slots, float* state,
                              void* u, int is_bf16, cudaStream_t st) {
  if (n_tok <= 0 || C <= 0) return 0;
  if (taps < 1) return -260;
  const bool v4 = C % 4 == 0 && ld % 4 == 0 && (reinterpret_cast<uintptr_t>(x) & (is_bf16 ? 7 : 15)) == 0;
  const int chunks = (n_tok + CONV_TOK - 1) / CONV_TOK;
  if (chunks > 65535) return -260;
  const dim3 grid((C / (v4 ? 4 : 1) + 127) / 128, chunks);
#define GO(TT, VV, NN) conv_prompt_kernel<TT, VV, NN><<<grid, 128, 0, st>>>((const TT*)x, ld, xb, w, bias, positions, n_tok, C, taps, (TT*)u)
#define PICK(TT, VV) do { if (taps == 4) GO(TT, VV, 4); else GO(TT, VV, 0); } while (0)
  if (is_bf16) { if (v4) PICK(bf16, 4); else PICK(bf16, 1); }
  else { if (v4) PICK(float, 4); else PICK(float, 1); }
#undef PICK
#undef GO
  if (state != nullptr && taps > 1 && n_seq > 0) {
    const dim3 g2((C + 255) / 256, n_seq);
    if (is_bf16) conv_state_kernel<bf16><<<g2, 256, 0, st>>>((const bf16*)x, ld, xb, cu, seq_slot, C, taps - 1, slots, state);
    else conv_state_kernel<float><<<g2, 256, 0, st>>>((const float*)x, ld, xb, cu, seq_slot, C, taps - 1, slots, state);
  }
  return (int)cudaGetLastError();
}

TRLB_API int trlb_conv_step(float* x, long long ld, const float* xb, const float* w, const float* bias, const int* seq_lens, int B,
                            int C, int taps, float* state, void* u, int is_bf16, cudaStream_t st) {
  if (B <= 0 || C <= 0) return 0;
  if (taps < 1) return -261;
  const bool v4 = C % 4 == 0 && ld % 4 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0;
  const dim3 grid((C / (v4 ? 4 : 1) + 127) / 128, B), blk(128);
#define GO(TT, VV) (int)trlb_host::launch_kernel(conv_step_kernel<TT, VV>, grid, blk, 0, st, PDL, x, ld, xb, w, bias, seq_lens, C, taps, state, (TT*)u)
  if (is_bf16) return v4 ? GO(bf16, 4) : GO(bf16, 1);
  return v4 ? GO(float, 4) : GO(float, 1);
#undef GO
}

TRLB_API int trlb_rglru_scan(const float* z, const void* u, const void* y, long long y_ld, const float* lam, const float* gate_bias,
                             const float* y_bias, const int* cu, int n_seq, const int* seq_slot, int slots, float* state, float decay, int C,
                             void* out, int is_bf16, cudaStream_t st) {
  if (n_seq <= 0 || C <= 0) return 0;
  const RgLru p = {C, slots, lam, gate_bias, y_bias, state, decay};
  const dim3 grid((C + 63) / 64, n_seq);
  const int* where = state != nullptr ? seq_slot : nullptr;
  if (is_bf16) rglru_scan_kernel<bf16><<<grid, 64, 0, st>>>(p, z, (const bf16*)u, (const bf16*)y, y_ld, cu, where, (bf16*)out);
  else rglru_scan_kernel<float><<<grid, 64, 0, st>>>(p, z, (const float*)u, (const float*)y, y_ld, cu, where, (float*)out);
  return (int)cudaGetLastError();
}

TRLB_API int trlb_rglru_step(const float* z, const void* u, float* y, long long y_ld, const float* lam, const float* gate_bias,
                             const float* y_bias, const int* seq_lens, int B, float* state, float decay, int C, void* out, int is_bf16,
                             cudaStream_t st) {
  if (B <= 0 || C <= 0) return 0;
  const RgLru p = {C, B, lam, gate_bias, y_bias, state, decay};
  const dim3 grid((C + 127) / 128, B), blk(128);
  if (is_bf16) return (int)trlb_host::launch_kernel(rglru_step_kernel<bf16>, grid, blk, 0, st, PDL, p, z, (const bf16*)u, y, y_ld, seq_lens, (bf16*)out);
  return (int)trlb_host::launch_kernel(rglru_step_kernel<float>, grid, blk, 0, st, PDL, p, z, (const float*)u, y, y_ld, seq_lens, (float*)out);
}
