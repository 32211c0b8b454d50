// Mixture of experts of the layered decoders around the grouped GEMM (grouped_gemm_tcgen05.cu): router choice, gathering of
// the tokens' rows by expert, weighted sum of the experts' rows into fp32, and the experts' products on the CUDA cores for
// fp32 models and for sizes the tensor-core kernel does not take.
//
// T is the model dtype (bf16 or fp32); logits, scores, weights and the sum are fp32.  Where a row of an expert stands among
// that expert's rows is decided by atomics; its values do not depend on it and the sum over a token's choices runs in the order
// of the choices.  Compiled without fast-math (csrc/build.py: EXACT_MATH).
#include "mixers.cuh"

namespace trlb {

constexpr int MR_MAX_E = 1024;

// ------------------------------------------------------------------------------------------------------------
// Router: scores sigmoid(z), or softmax(z); the `top` experts of the largest score + correction (ties: the lower index) with their
// bare scores as weights (renorm: over their sum), times gain.  One warp per token.  rank: place among the expert's rows.  ONE: a single block
// stores its counts; else counts are zeros before the launch and blocks of `span` tokens add theirs.  Negative positions mark idle rows,
// which choose nothing (expert -1).  clear: z is zeroed.
// ------------------------------------------------------------------------------------------------------------
struct MoeRoute {
  float* z;  // [T, E]
  const float* correction;  // [E] or null
  const int* positions;     // [T] or null
  int T, E, top, renorm, softmax, clear, span;
  float gain;
  int* choice;   // [T, top]
  int* rank;     // [T, top]
  float* weight; // [T, top]
  int* counts;   // [E]
};

template <bool ONE, int NI>  // NI: experts a lane
__global__ void __launch_bounds__(1024)
moe_route_kernel(const MoeRoute p) {
  __shared__ int cnt[32 * NI];   // tokens of this block per expert
  __shared__ int base[ONE ? 1 : 32 * NI];
  pdl_launch_dependents();
  pdl_wait();
  for (int e = threadIdx.x; e < p.E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  const int lane = threadIdx.x & 31, per = blockDim.x >> 5, t_end = min(p.T, (int)(blockIdx.x + 1) * p.span);
  for (int t = blockIdx.x * p.span + (threadIdx.x >> 5); t < t_end; t += per) {
    float* z = p.z + (size_t)t * p.E;
    const bool idle = p.positions != nullptr && p.positions[t] < 0;
    float w[NI], sc[NI];   // scores of experts lane, lane + 32, ...: bare and as they are chosen by
#pragma unroll
    for (int i = 0; i < NI; ++i) w[i] = lane + 32 * i < p.E ? z[lane + 32 * i] : -INFINITY;
    if (p.softmax) {
      float top = -INFINITY, sum = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) top = fmaxf(top, w[i]);
      top = warp_max(top);
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        w[i] = lane + 32 * i < p.E ? expf(w[i] - top) : 0.f;
        sum += w[i];
      }
      sum = warp_sum(sum);
#pragma unroll
      for (int i = 0; i < NI; ++i) w[i] /= sum;
    } else {
#pragma unroll
      for (int i = 0; i < NI; ++i) w[i] = sigmoid_f(w[i]);
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = lane + 32 * i;
      sc[i] = -INFINITY;
      if (e < p.E) {
        sc[i] = w[i] + (p.correction != nullptr ? p.correction[e] : 0.f);
        if (!(sc[i] > -INFINITY)) sc[i] = -3e38f;  // a NaN still has its place in the order
      }
    }
    float total = 0.f;
    for (int j = 0; j < p.top; ++j) {
      float best = -INFINITY, own = 0.f;
      int at = p.E;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        if (sc[i] > best) { best = sc[i]; at = lane + 32 * i; own = w[i]; }
      }
      const int mine = at;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int oa = __shfl_xor_sync(0xffffffffu, at, o);
        if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
      }
      if (mine == at) {  // one lane
        const size_t o = (size_t)t * p.top + j;
        p.choice[o] = idle ? -1 : at;
        p.weight[o] = own * p.gain;
        if (!idle) p.rank[o] = atomicAdd(&cnt[at], 1);
      }
      total += __shfl_sync(0xffffffffu, own, at & 31);
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        if (at == lane + 32 * i) sc[i] = -INFINITY;
      }
    }
    __syncwarp();
    if (p.renorm)
      for (int j = lane; j < p.top; j += 32) p.weight[(size_t)t * p.top + j] /= total + 1e-20f;
    if (p.clear)
      for (int e = lane; e < p.E; e += 32) z[e] = 0.f;
  }
  __syncthreads();
  if (ONE) {
    for (int e = threadIdx.x; e < p.E; e += blockDim.x) p.counts[e] = cnt[e];
  } else {  // the block's rows of an expert follow those of the blocks that counted before it
    for (int e = threadIdx.x; e < p.E; e += blockDim.x) base[e] = cnt[e] > 0 ? atomicAdd(&p.counts[e], cnt[e]) : 0;
    __syncthreads();
    for (long long i = (long long)blockIdx.x * p.span * p.top + threadIdx.x; i < (long long)t_end * p.top; i += blockDim.x) {
      const int e = p.choice[i];
      if (e >= 0) p.rank[i] += base[e];
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// Rows of h, one copy per choice, sorted by expert; row[t, j] = where choice j of token t stands (-1: idle), offsets [E + 1].
// ------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
moe_gather_kernel(const T* __restrict__ h, const int* __restrict__ choice, const int* __restrict__ rank, const int* __restrict__ counts,
                  int n_tok, int E, int top, int H, T* __restrict__ x, int* __restrict__ row, int* __restrict__ offsets) {
  __shared__ int off[MR_MAX_E + 1];
  __shared__ int part[9];
  pdl_launch_dependents();
  pdl_wait();
  // exclusive prefix of the counts: each thread sums a run of them, the runs' sums are scanned by warp and block
  const int run = (E + 255) / 256, e0 = threadIdx.x * run, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  int mine = 0;
  for (int e = e0; e < min(E, e0 + run); ++e) mine += counts[e];
  int inc = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += v;
  }
  if (lane == 31) part[wid] = inc;
  __syncthreads();
  int before = inc - mine;
  for (int w = 0; w < wid; ++w) before += part[w];
  for (int e = e0; e < min(E, e0 + run); ++e) {
    off[e] = before;
    before += counts[e];
    if (e == E - 1) off[E] = before;
  }
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e <= E; e += 256) offsets[e] = off[e];
  const bool vec = (H * sizeof(T)) % 16 == 0;
  const int n16 = (int)(H * sizeof(T) / 16);
  for (long long i = blockIdx.x; i < (long long)n_tok * top; i += gridDim.x) {
    const int e = choice[i], t = (int)(i / top);
    const int r = e < 0 ? -1 : off[e] + rank[i];
    if (threadIdx.x == 0) row[i] = r;
    if (r < 0) continue;
    const T* s = h + (size_t)t * H;
    T* d = x + (size_t)r * H;
    if (vec) {
      for (int v = threadIdx.x; v < n16; v += 256) reinterpret_cast<uint4*>(d)[v] = reinterpret_cast<const uint4*>(s)[v];
    } else {
      for (int v = threadIdx.x; v < H; v += 256) d[v] = s[v];
    }
  }
}

// out[t] = sum over the choices of weight * y[row]; fp32, stored or (add) added to.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
moe_sum_kernel(const T* __restrict__ y, const int* __restrict__ row, const float* __restrict__ weight, int top, int H,
               float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  for (int j = VEC * threadIdx.x; j < H; j += VEC * blockDim.x) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c = 0; c < top; ++c) {
      const int r = row[(size_t)t * top + c];
      if (r < 0) continue;
      const float w = weight[(size_t)t * top + c];
      if (VEC == 4) {
        const float4 v = load4(y + (size_t)r * H + j);
        a = make_float4(fmaf(w, v.x, a.x), fmaf(w, v.y, a.y), fmaf(w, v.z, a.z), fmaf(w, v.w, a.w));
      } else {
        a.x = fmaf(w, to_f(y[(size_t)r * H + j]), a.x);
      }
    }
    if (VEC == 4) store4(out + (size_t)t * H + j, a);
    else out[(size_t)t * H + j] = a.x;
  }
}

// ------------------------------------------------------------------------------------------------------------
// C[r, :] = A[r, :] W[e]^T for the rows r of expert e, any size: 64 x 64 tiles, 4 x 4 sums a thread.  grid: (N tiles, experts,
// row slices); a block walks every gridDim.z-th row tile of its expert.
// ------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
moe_rows_gemm_kernel(const T* __restrict__ A, const T* __restrict__ W, const int* __restrict__ offsets, T* __restrict__ C, int N, int K) {
  __shared__ float as[16][65], ws[16][65];
  const int e = blockIdx.y, n0 = blockIdx.x * 64, r_end = offsets[e + 1];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* w = W + (size_t)e * N * K;
  for (int r0 = offsets[e] + 64 * blockIdx.z; r0 < r_end; r0 += 64 * gridDim.z) {
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += 16) {
      for (int i = threadIdx.x; i < 64 * 16; i += 256) {
        const int r = i >> 4, k = i & 15;
        const bool kin = k0 + k < K;
        as[k][r] = kin && r0 + r < r_end ? to_f(A[(size_t)(r0 + r) * K + k0 + k]) : 0.f;
        ws[k][r] = kin && n0 + r < N ? to_f(w[(size_t)(n0 + r) * K + k0 + k]) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < 16; ++k) {
        float a[4], b[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) { a[i] = as[k][ty * 4 + i]; b[i] = ws[k][tx + 16 * i]; }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + ty * 4 + i;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + tx + 16 * j;
        if (r < r_end && n < N) C[(size_t)r * N + n] = from_f<T>(acc[i][j]);
      }
    }
  }
}

}  // namespace trlb

using namespace trlb;

#define PDL trlb_host::pdl_enabled()
using bf16 = __nv_bfloat16;

// z [T, E] fp32 logits (zeroed with clear); correction, positions may be null.  choice, rank, weight [T, top]; counts [E]: zeros
// when T > 128 (they are added to), else any.
TRLB_API int trlb_moe_route(float* z, const float* correction, const int* positions, int T, int E, int top, int renorm, int softmax,
                            float gain, int clear, int* choice, int* rank, float* weight, int* counts, cudaStream_t st) {
  if (T <= 0) return 0;
  if (E <= 0 || E > MR_MAX_E || top <= 0 || top > E) return -290;
  const MoeRoute p = {z, correction, positions, T, E, top, renorm, softmax, clear, T <= 128 ? T : 32, gain, choice, rank, weight, counts};
  const dim3 grid(T <= 128 ? 1 : (T + 31) / 32), blk(T > 128 ? (E <= 256 ? 512 : 256) : T >= 32 ? 1024 : T * 32);
#define GO(ONE, NI) (int)trlb_host::launch_kernel(moe_route_kernel<ONE, NI>, grid, blk, 0, st, PDL, p)
#define PICK(NI) (T <= 128 ? GO(true, NI) : GO(false, NI))
  return E <= 32 ? PICK(1) : E <= 64 ? PICK(2) : E <= 128 ? PICK(4) : E <= 256 ? PICK(8) : PICK(32);
#undef PICK
#undef GO
}

// h [T, H], x [T top, H] in the model dtype; row [T, top], offsets [E + 1]
TRLB_API int trlb_moe_gather(const void* h, const int* choice, const int* rank, const int* counts, int T, int E, int top, int H, void* x,
                             int* row, int* offsets, int is_bf16, cudaStream_t st) {
  if (T <= 0) return 0;
  if (E <= 0 || E > MR_MAX_E || top <= 0) return -291;
  const long long n = (long long)T * top, cap = (long long)trlb_host::sm_count() * 8;
  const dim3 grid((unsigned)(n < cap ? n : cap)), blk(256);
  if (is_bf16) return (int)trlb_host::launch_kernel(moe_gather_kernel<bf16>, grid, blk, 0, st, PDL, (const bf16*)h, choice, rank, counts, T, E, top, H, (bf16*)x, row, offsets);
  return (int)trlb_host::launch_kernel(moe_gather_kernel<float>, grid, blk, 0, st, PDL, (const float*)h, choice, rank, counts, T, E, top, H, (float*)x, row, offsets);
}

// y [rows, H] in the model dtype, out [T, H] fp32
TRLB_API int trlb_moe_sum(const void* y, const int* row, const float* weight, int T, int top, int H, float* out, int is_bf16, cudaStream_t st) {
  if (T <= 0) return 0;
  const bool v4 = H % 4 == 0;
  const dim3 blk(H >= 1024 ? 256 : 64);
#define GO(TT, VV) (int)trlb_host::launch_kernel(moe_sum_kernel<TT, VV>, dim3(T), blk, 0, st, PDL, (const TT*)y, row, weight, top, H, out)
  if (is_bf16) return v4 ? GO(bf16, 4) : GO(bf16, 1);
  return v4 ? GO(float, 4) : GO(float, 1);
#undef GO
}

// A [rows, K], W [E, N, K], C [rows, N] in the model dtype; rows of expert e: offsets[e] .. offsets[e + 1]
TRLB_API int trlb_moe_rows_gemm(const void* A, const void* W, const int* offsets, void* C, long long rows, int E, int N, int K, int is_bf16,
                                cudaStream_t st) {
  if (rows <= 0 || E <= 0) return 0;
  if (E > 65535) return -292;
  const long long tiles = (rows + 63) / 64;
  const dim3 grid((N + 63) / 64, E, (unsigned)(tiles < 8 ? tiles : 8));
  if (is_bf16) moe_rows_gemm_kernel<bf16><<<grid, 256, 0, st>>>((const bf16*)A, (const bf16*)W, offsets, (bf16*)C, N, K);
  else moe_rows_gemm_kernel<float><<<grid, 256, 0, st>>>((const float*)A, (const float*)W, offsets, (float*)C, N, K);
  return (int)cudaGetLastError();
}
