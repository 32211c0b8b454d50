// HGRN2 of the layered decoders: linear attention whose forget gate per head and channel also decides what is written,
//
//     f = low + (1 - low) sigmoid(z + bias),   S = diag(f) S + (1 - f) v^T,   o = S^T silu(q),
//
// computed with k = 1 - f = (1 - low) sigmoid(-z - bias), which keeps its precision where f is close to one: S += k (v - S).  Here
// token by token for every size and dtype, the decode step, and the norm per head behind it (prompts on the tensor cores:
// hgrn2_chunk_tcgen05.cu).
//
// T is the model dtype (bf16 or fp32); gates, states, outputs and norms are fp32 in both.  Compiled without fast-math
// (csrc/build.py: EXACT_MATH).  State of a slot and head: S [dim, vdim].  In decode seq_lens[slot] is the position of the slot's
// new token, negative: idle.
#include "mixers.cuh"

namespace trlb {

__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }
__device__ __forceinline__ float write_f(float z, float low) { return (1.f - low) * sigmoid_f(-z); }

// ------------------------------------------------------------------------------------------------------------
// Prompts: grid (sequence, head, 32-column tile of vdim), 256 threads.  A thread holds NR rows of one column of S in registers;
// eight neighbouring lanes share a column.  Tokens are staged sixteen at a time.
// ------------------------------------------------------------------------------------------------------------
struct Hgrn2 {
  long long y_ld, z_ld;
  int heads, dim, vdim, v_off;
  const float* bias;   // [heads dim]
  const float* low;    // [heads dim]
  const int* cu;
  const int* seq_slot; // [n_seq] or null
  float* S;            // [slots, heads, dim, vdim]
  int slots;
};

constexpr int HG_STAGE = 16;

template <typename T, int NR>
__global__ void __launch_bounds__(256)
hgrn2_prompt_kernel(const Hgrn2 p, const T* __restrict__ y, const float* __restrict__ z, float* __restrict__ out) {
  constexpr int ROW = 8 * (NR + 4);  // a lane's rows start on another bank than its neighbours'
  extern __shared__ float sm[];
  float* qs = sm;                        // [HG_STAGE][ROW]
  float* ks = qs + HG_STAGE * ROW;       // [HG_STAGE][ROW]
  float* vs = ks + HG_STAGE * ROW;       // [HG_STAGE][32]
  const int seq = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * 32, tid = threadIdx.x, dg = tid & 7, ec = tid >> 3, e = e0 + ec;
  const int t0 = p.cu[seq], len = p.cu[seq + 1] - t0;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = 0.f;
  for (int i = tid; i < 2 * HG_STAGE * ROW; i += 256) sm[i] = 0.f;  // rows past dim write and read nothing
  for (int base = 0; base < len; base += HG_STAGE) {
    const int n = min(HG_STAGE, len - base);
    __syncthreads();
    for (int i = tid; i < n * p.dim; i += 256) {
      const int t = i / p.dim, d = i % p.dim, at = t * ROW + (d / NR) * (NR + 4) + d % NR, hd = h * p.dim + d;
      const size_t row = (size_t)(t0 + base + t);
      qs[at] = silu_f(to_f(y[row * p.y_ld + hd]));
      ks[at] = write_f(z[row * p.z_ld + hd] + p.bias[hd], p.low[hd]);
    }
    for (int i = tid; i < n * 32; i += 256) {
      const int t = i >> 5, c = e0 + (i & 31);
      vs[i] = c < p.vdim ? to_f(y[(size_t)(t0 + base + t) * p.y_ld + p.v_off + (size_t)h * p.vdim + c]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float v = vs[t * 32 + ec];
      const float* k = ks + t * ROW + dg * (NR + 4);
      const float* q = qs + t * ROW + dg * (NR + 4);
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < NR; i += 4) {
        const float4 a = load4(k + i), b = load4(q + i);
        S[i] = fmaf(a.x, v - S[i], S[i]);
        S[i + 1] = fmaf(a.y, v - S[i + 1], S[i + 1]);
        S[i + 2] = fmaf(a.z, v - S[i + 2], S[i + 2]);
        S[i + 3] = fmaf(a.w, v - S[i + 3], S[i + 3]);
        acc[0] = fmaf(S[i], b.x, acc[0]);
        acc[1] = fmaf(S[i + 1], b.y, acc[1]);
        acc[2] = fmaf(S[i + 2], b.z, acc[2]);
        acc[3] = fmaf(S[i + 3], b.w, acc[3]);
      }
      float o = (acc[0] + acc[1]) + (acc[2] + acc[3]);
#pragma unroll
      for (int x = 1; x < 8; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
      if (dg == 0 && e < p.vdim) out[((size_t)(t0 + base + t) * p.heads + h) * p.vdim + e] = o;
    }
  }
  if (p.seq_slot == nullptr || e >= p.vdim) return;
  const int slot = p.seq_slot[seq];
  if (slot < 0 || slot >= p.slots) return;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = dg * NR + i;
    if (d < p.dim) p.S[(((size_t)slot * p.heads + h) * p.dim + d) * p.vdim + e] = S[i];
  }
}

// y[t, h vdim + e] = o / rms(o of the head) * w[e] * scale.  One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
head_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, float eps, int heads, int vdim, long long n, float scale,
                 T* __restrict__ y, long long y_ld) {
  const int lane = threadIdx.x & 31;
  for (long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5); i < n; i += (long long)gridDim.x * 8) {
    const float* r = o + i * vdim;
    T* dst = y + (i / heads) * y_ld + (i % heads) * vdim;
    float ss = 0.f;
    const bool v4 = ((vdim | (int)(y_ld & 3)) & 3) == 0 && (reinterpret_cast<uintptr_t>(y) & (4 * sizeof(T) - 1)) == 0;
    if (v4 && vdim <= 128) {
      const bool on = 4 * lane < vdim;
      const float4 a = on ? load4(r + 4 * lane) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss = warp_sum(a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w);
      const float f = scale / sqrtf(ss / (float)vdim + eps);
      if (on) {
        const float4 g = load4(w + 4 * lane);
        store4(dst + 4 * lane, make_float4(a.x * f * g.x, a.y * f * g.y, a.z * f * g.z, a.w * f * g.w));
      }
    } else {
      for (int e = lane; e < vdim; e += 32) ss += r[e] * r[e];
      const float f = scale / sqrtf(warp_sum(ss) / (float)vdim + eps);
      for (int e = lane; e < vdim; e += 32) dst[e] = from_f<T>(r[e] * f * w[e]);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// One token per slot: grid (head, slot), 256 threads = 256 / groups row groups x `groups` column groups of VEC columns.  sums: fp32
// rows [q | v | z] of the input projection, zeroed behind the read; y: normed outputs, times scale.
// ------------------------------------------------------------------------------------------------------------
struct Hgrn2Step {
  float* sums;
  long long ld;
  int heads, dim, vdim, groups_log2;
  const float* bias;
  const float* low;
  const float* norm;   // [vdim]
  float eps, scale;
  const int* seq_lens;
  float* S;
  long long y_ld;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
hgrn2_step_kernel(const Hgrn2Step p, T* __restrict__ y) {
  extern __shared__ float sm[];  // q [dim], k [dim], v [vdim], partial sums [row groups][vdim]
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, cgs = 1 << p.groups_log2, cg = tid & (cgs - 1), rg = tid >> p.groups_log2;
  const int rgs = 256 >> p.groups_log2;
  const bool live = p.seq_lens[b] >= 0;
  constexpr int ROWS = 8;  // of S that a thread has under way at a time
  float* S = p.S + ((size_t)b * p.heads + h) * p.dim * p.vdim;
  float4 t[ROWS];
  auto fetch = [&](int e, int d0) {
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
      const int d = d0 + j * rgs;
      if (d >= p.dim) continue;
      if (VEC == 4) t[j] = load4(S + (size_t)d * p.vdim + e);
      else t[j].x = S[(size_t)d * p.vdim + e];
    }
  };
  if (live && cg * VEC < p.vdim) fetch(cg * VEC, rg);  // while the sums are read
  float* qs = sm;
  float* ks = qs + p.dim;
  float* vs = ks + p.dim;
  float* part = vs + p.vdim;
  float* q = p.sums + (size_t)b * p.ld + (size_t)h * p.dim;
  float* v = p.sums + (size_t)b * p.ld + (size_t)p.heads * p.dim + (size_t)h * p.vdim;
  float* z = p.sums + (size_t)b * p.ld + (size_t)p.heads * (p.dim + p.vdim) + (size_t)h * p.dim;
  for (int d = tid; d < p.dim; d += 256) {
    qs[d] = silu_f(q[d]);
    ks[d] = write_f(z[d] + p.bias[h * p.dim + d], p.low[h * p.dim + d]);
    q[d] = 0.f;
    z[d] = 0.f;
  }
  for (int e = tid; e < p.vdim; e += 256) {
    vs[e] = v[e];
    v[e] = 0.f;
  }
  if (!live) return;  // uniform
  __syncthreads();
  for (int e = cg * VEC; e < p.vdim; e += cgs * VEC) {
    float o[VEC], w[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      o[i] = 0.f;
      w[i] = vs[e + i];
    }
    for (int d0 = rg; d0 < p.dim; d0 += ROWS * rgs) {
      if (d0 != rg || e != cg * VEC) fetch(e, d0);
#pragma unroll
      for (int j = 0; j < ROWS; ++j) {
        const int d = d0 + j * rgs;
        if (d >= p.dim) continue;
        float s[4] = {t[j].x, t[j].y, t[j].z, t[j].w};
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          s[i] = fmaf(ks[d], w[i] - s[i], s[i]);
          o[i] = fmaf(s[i], qs[d], o[i]);
        }
        if (VEC == 4) store4(S + (size_t)d * p.vdim + e, make_float4(s[0], s[1], s[2], s[3]));
        else S[(size_t)d * p.vdim + e] = s[0];
      }
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) part[(size_t)rg * p.vdim + e + i] = o[i];
  }
  __syncthreads();
  float ss = 0.f;
  for (int e = tid; e < p.vdim; e += 256) {
    float o = 0.f;
    for (int r = 0; r < rgs; ++r) o += part[(size_t)r * p.vdim + e];
    vs[e] = o;
    ss += o * o;
  }
  const float f = p.scale / sqrtf(block_sum2(ss, 0.f, red).x / (float)p.vdim + p.eps);
  for (int e = tid; e < p.vdim; e += 256) y[(size_t)b * p.y_ld + (size_t)h * p.vdim + e] = from_f<T>(vs[e] * f * p.norm[e]);
}

}  // namespace trlb

using namespace trlb;

namespace {

template <typename K>
bool allow_smem(K kern, size_t bytes) {
  if (bytes <= 48 * 1024) return true;
  if (bytes > 227 * 1024) return false;
  return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) == cudaSuccess;
}

using bf16 = __nv_bfloat16;

template <typename T, int NR>
int hgrn2_prompt(const Hgrn2& p, const void* y, const float* z, float* out, int n_seq, cudaStream_t st) {
  const size_t smem = (size_t)HG_STAGE * (2 * 8 * (NR + 4) + 32) * 4;
  if (!allow_smem(hgrn2_prompt_kernel<T, NR>, smem)) return -301;
  const dim3 grid(n_seq, p.heads, (p.vdim + 31) / 32);
  hgrn2_prompt_kernel<T, NR><<<grid, 256, smem, st>>>(p, (const T*)y, z, out);
  return (int)cudaGetLastError();
}

template <typename T>
int hgrn2_prompt_any(const Hgrn2& p, const void* y, const float* z, float* out, int n_seq, cudaStream_t st) {
  if (p.dim <= 32) return hgrn2_prompt<T, 4>(p, y, z, out, n_seq, st);
  if (p.dim <= 64) return hgrn2_prompt<T, 8>(p, y, z, out, n_seq, st);
  if (p.dim <= 128) return hgrn2_prompt<T, 16>(p, y, z, out, n_seq, st);
  if (p.dim <= 256) return hgrn2_prompt<T, 32>(p, y, z, out, n_seq, st);
  return hgrn2_prompt<T, 64>(p, y, z, out, n_seq, st);
}

}  // namespace

// y [T rows of y_ld]: q at 0, v at v_off (elements), model dtype; z [T rows of z_ld] fp32 gate logits without bias.  Sequences by cu
// [n_seq + 1]; seq_slot null: no state is kept.  out [T, heads, vdim] fp32.  dim <= 512.
TRLB_API int trlb_hgrn2_prompt(const void* y, long long y_ld, int v_off, const float* z, long long z_ld, const float* bias, const float* low,
                               const int* cu, int n_seq, const int* seq_slot, float* S, int slots, int heads, int dim, int vdim,
                               float* out, int is_bf16, cudaStream_t st) {
  if (n_seq <= 0) return 0;
  if (heads <= 0 || dim <= 0 || dim > 512 || vdim <= 0 || (seq_slot != nullptr && S == nullptr)) return -300;
  const Hgrn2 p = {y_ld, z_ld, heads, dim, vdim, v_off, bias, low, cu, seq_slot, S, slots};
  return is_bf16 ? hgrn2_prompt_any<bf16>(p, y, z, out, n_seq, st) : hgrn2_prompt_any<float>(p, y, z, out, n_seq, st);
}

// o [rows, heads, vdim] fp32 -> y [rows of y_ld] in the model dtype; w [vdim]
TRLB_API int trlb_head_norm(const float* o, const float* w, float eps, int rows, int heads, int vdim, float scale, void* y, long long y_ld,
                            int is_bf16, cudaStream_t st) {
  if (rows <= 0) return 0;
  const long long n = (long long)rows * heads, want = (n + 7) / 8, cap = (long long)trlb_host::sm_count() * 32;
  const int grid = (int)(want < cap ? want : cap);
  if (is_bf16) head_norm_kernel<bf16><<<grid, 256, 0, st>>>(o, w, eps, heads, vdim, n, scale, (bf16*)y, y_ld);
  else head_norm_kernel<float><<<grid, 256, 0, st>>>(o, w, eps, heads, vdim, n, scale, (float*)y, y_ld);
  return (int)cudaGetLastError();
}

// sums [B rows of ld] fp32: q | v | z (zeroed); S [>= B slots, heads, dim, vdim]; y [B rows of y_ld] in the model dtype
TRLB_API int trlb_hgrn2_step(float* sums, long long ld, const float* bias, const float* low, const float* norm, float eps, float scale,
                             const int* seq_lens, int B, float* S, int heads, int dim, int vdim, void* y, long long y_ld, int is_bf16,
                             cudaStream_t st) {
  if (B <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0) return -302;
  const bool v4 = vdim % 4 == 0;
  int lg = 0;
  while ((v4 ? 4 : 1) << lg < vdim && lg < 6) ++lg;
  const Hgrn2Step p = {sums, ld, heads, dim, vdim, lg, bias, low, norm, eps, scale, seq_lens, S, y_ld};
  const size_t smem = (size_t)(2 * dim + vdim + (256 >> lg) * vdim) * 4;
  const dim3 grid(heads, B), blk(256);
#define GO(TT, VV) (allow_smem(hgrn2_step_kernel<TT, VV>, smem) ? (int)trlb_host::launch_kernel(hgrn2_step_kernel<TT, VV>, grid, blk, smem, st, trlb_host::pdl_enabled(), p, (TT*)y) : -303)
  if (is_bf16) return v4 ? GO(bf16, 4) : GO(bf16, 1);
  return v4 ? GO(float, 4) : GO(float, 1);
#undef GO
}
