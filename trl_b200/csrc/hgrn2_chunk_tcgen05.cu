// HGRN2 over packed prompts in chunks of 128 tokens, on the 5th-generation tensor cores (bf16 q and v, fp32 gate logits, decays and
// states; token by token: hgrn2.cu).
//
// With f = 1 - k the forget gates (k = (1 - low) sigmoid(-z - bias)), S the state in front of a chunk and every product of gates per
// channel,
//
//     o_t = sum_{j <= t} (q_t . (k_j prod_{j < i <= t} f_i)) v_j  +  S^T (q_t prod_{i <= t} f_i)
//     S'  = diag(prod f) S + sum_j (k_j prod_{j < i} f_i) v_j^T
//
//   hgrn2_state_kernel   one CTA per (sequence, head, 128 columns of v) walks the chunks: the state is an accumulator in TMEM that is
//                        multiplied by the chunk's decay and takes in one 128 x 128 x 128 product;
//   hgrn2_output_kernel  one CTA per (chunk, head, 128 columns of v).
//
// A gate product between two tokens is the quotient of two prefix products, but a prefix over many tokens under- or overflows.  So the
// 128 x 128 scores of a chunk are taken apart by where query and key part: a pair that lies on both sides of the middle of a block of
// 128, 64, 32 or 16 tokens (levels of 64, 32, 16 and 8) has the product from the key to the middle times that from the middle to the
// query, both at most one.  On a level every token is a query or a key, so that level is one 128 x 64 product of scaled queries and
// keys.  Pairs inside a block of 8 are scaled about its middle: at most four factors, with gates held above 2^-24 (what lies below is
// lost in fp32 beside one), stay in range both ways.
//
// fp32 precision through bf16 operands: scaled queries and keys, scores and states enter the products as two bf16 each (value and
// remainder; the product of two remainders is left out).
#include "mixers.cuh"

namespace trlb {

constexpr int HC_L = 128;
constexpr uint32_t HC_BOX = 128 * 64 * 2;  // 128 rows of 64 elements, 128-byte swizzle

struct Hgrn2Chunk {
  const int* cu;
  int n_seq, heads, dim, vdim;
  const float* bias;       // [heads dim]
  const float* low;
  __nv_bfloat16* s_hi;     // [chunks, heads, dim, vdim] state in front of a chunk, value and remainder; the first chunk of a
  __nv_bfloat16* s_lo;     // sequence has none
  float* S;                // [slots, heads, dim, vdim] or null
  const int* seq_slot;
  int slots;
  const float* norm;       // [vdim]: the normed output goes to y_out; null: the output goes to out
  float eps, scale;
  __nv_bfloat16* y_out;    // [T rows of out_ld], heads x vdim
  long long out_ld;
  float* out;              // [T, heads, vdim]
  int* status;
};

__device__ __forceinline__ int hc_chunks(int len) { return (len + HC_L - 1) / HC_L; }

// exp bounded so that a product of two stays finite
__device__ __forceinline__ float hc_exp(float x) { return fast_exp2(fminf(1.4426950408889634f * x, 60.f)); }

// Eight values as bf16 and remainders to shared memory, 16 bytes each.
__device__ __forceinline__ void hc_put8(uint32_t hi, uint32_t lo, const float (&v)[8]) {
  uint32_t a[4], b[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    a[i] = pack_bf16(v[2 * i], v[2 * i + 1]);
    const float2 f = unpack_bf16(a[i]);
    b[i] = pack_bf16(v[2 * i] - f.x, v[2 * i + 1] - f.y);
  }
  asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(hi), "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]) : "memory");
  asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(lo), "r"(b[0]), "r"(b[1]), "r"(b[2]), "r"(b[3]) : "memory");
}

// The value, unknown to the compiler: it must not keep partial products of one step in registers for another.
__device__ __forceinline__ float hc_afresh(float w) {
  asm volatile("" : "+f"(w));
  return w;
}

template <int N>
struct HcInt {
  static constexpr int value = N;
};

// Barrier of the threads that compute; all of them get to every one, also after a wait that ran out.
template <int THREADS>
__device__ __forceinline__ void hc_sync() { asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory"); }

// Gate logits of channel d at token t of a tile that came as four boxes of 32 channels (rows of 128 bytes, swizzled).
__device__ __forceinline__ float hc_logit(uint32_t boxes, int d, int t) {
  const uint32_t w = (uint32_t)d & 31;
  float v;
  asm volatile("ld.shared.f32 %0, [%1];"
               : "=f"(v)
               : "r"(boxes + (uint32_t)(d >> 5) * HC_BOX + (w & 3) * 4 + (((w >> 2) ^ ((uint32_t)t & 7)) << 4) + (uint32_t)t * 128)
               : "memory");
  return v;
}
// The same of queries, two boxes of 64 channels.
__device__ __forceinline__ float hc_query(uint32_t boxes, int d, int t) {
  const uint32_t w = (uint32_t)d & 63;
  uint16_t v;
  asm volatile("ld.shared.u16 %0, [%1];"
               : "=h"(v)
               : "r"(boxes + (uint32_t)(d >> 6) * HC_BOX + (w & 7) * 2 + (((w >> 3) ^ ((uint32_t)t & 7)) << 4) + (uint32_t)t * 128)
               : "memory");
  return __uint_as_float((uint32_t)v << 16);
}

// ------------------------------------------------------------------------------------------------------------
// State pass.  Warps 0-15: thread (channel, quarter of the tokens) forms the scaled keys, warp (32 rows of S, 32 columns) scales the
// state; warp 16: TMA; warp 17: MMA.  The gate logits of the next chunk arrive while the products of this one run.  The state in front
// of a chunk goes out through the place of the keys, whole lines at a time.
// ------------------------------------------------------------------------------------------------------------
constexpr int HC_WORK = 512, HS_THREADS = HC_WORK + 64;
constexpr size_t HS_SMEM = 12 * (size_t)HC_BOX + 1024 + 4096 + 256;

__global__ void __launch_bounds__(HS_THREADS, 1)
hgrn2_state_kernel(const __grid_constant__ CUtensorMap tm_z, const __grid_constant__ CUtensorMap tm_v, const Hgrn2Chunk p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* z_s = smem;                 // four boxes of 32 channels, rows are tokens
  uint8_t* k_s = smem + 4 * HC_BOX;    // keys: two boxes of 64 tokens, rows are channels; then their remainders
  uint8_t* v_s = smem + 8 * HC_BOX;    // two buffers of two boxes of 64 columns, rows are tokens
  float* prod = reinterpret_cast<float*>(smem + 12 * HC_BOX);  // [2][4][128] product of the gates of a quarter
  uint64_t* bars = reinterpret_cast<uint64_t*>(prod + 1024);
  uint64_t* z_full = bars;
  uint64_t* z_free = bars + 1;
  uint64_t* v_full = bars + 2;   // [2]
  uint64_t* v_free = bars + 4;   // [2]
  uint64_t* ready = bars + 6;
  uint64_t* acc_full = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seq = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * 128;
  int chunk0 = 0;
  for (int s = 0; s < seq; ++s) chunk0 += hc_chunks(p.cu[s + 1] - p.cu[s]);
  const int beg = p.cu[seq], len = p.cu[seq + 1] - beg, nc = hc_chunks(len);
  const int cols = min(128, (p.vdim - e0 + 15) & ~15);

  if (tid == 0) {
    mbar_init(z_full, 1);
    mbar_init(z_free, HC_WORK);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&v_full[i], 1);
      mbar_init(&v_free[i], 1);
    }
    mbar_init(ready, HC_WORK);
    mbar_init(acc_full, 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_z);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 17) {
    tmem_alloc(tmem_slot, 128);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 16) {
    if (lane == 0) {
      for (int c = 0; c < nc; ++c) {
        const int b = c & 1;
        if (c > 0 && !mbar_wait(z_free, (uint32_t)((c - 1) & 1), abort_flag, p.status, 2000)) break;
        mbar_expect_tx(z_full, 4 * HC_BOX);
        for (int i = 0; i < 4; ++i) tma_load_3d(z_s + i * HC_BOX, &tm_z, z_full, 64 * i, h, beg + c * HC_L);
        if (c > 1 && !mbar_wait(&v_free[b], (uint32_t)(((c >> 1) - 1) & 1), abort_flag, p.status, 2001)) break;
        mbar_expect_tx(&v_full[b], 2 * HC_BOX);
        for (int i = 0; i < 2; ++i) tma_load_3d(v_s + (2 * b + i) * HC_BOX, &tm_v, &v_full[b], e0 + 64 * i, h, beg + c * HC_L);
      }
    }
    __syncwarp();
  } else if (warp == 17) {
    if (lane == 0) {
      const uint32_t idesc = umma_idesc_bf16_major(128, cols, false, true);
      const uint64_t ka = umma_desc_kmajor_sw128(smem_u32(k_s)), vb = umma_desc_mnmajor_sw128(smem_u32(v_s), HC_BOX);
      for (int c = 0; c < nc; ++c) {
        const int b = c & 1;
        if (!mbar_wait(&v_full[b], (uint32_t)((c >> 1) & 1), abort_flag, p.status, 2010)) break;
        if (!mbar_wait(ready, (uint32_t)(c & 1), abort_flag, p.status, 2011)) break;
        tc_fence_after();
        const uint64_t vd = desc_at(vb, (uint32_t)b * 2 * HC_BOX);
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int kk = 0; kk < HC_L / 16; ++kk)
            umma_bf16_ss(tmem_base, desc_at(ka, (2 * half + (kk >> 2)) * HC_BOX) + 2 * (kk & 3), desc_at(vd, kk * 2048), idesc,
                         c > 0 || (half | kk) != 0);
        umma_commit(&v_free[b]);
        umma_commit(acc_full);
      }
    }
    __syncwarp();
  } else {
    const int d = tid & 127, qt = tid >> 7, x0 = 32 * qt;  // also: this warp's columns of S
    const bool on = d < p.dim;
    const int hd = h * p.dim + (on ? d : 0);
    const float bias = p.bias[hd], room = 1.f - p.low[hd];
    const uint32_t t_row = tmem_base + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)x0;
    // eight tokens of this channel's keys, or eight columns of this row of the state: numbers 0 .. 3 of this quarter
    const uint32_t keys = smem_u32(k_s) + (uint32_t)(qt >> 1) * HC_BOX + (uint32_t)d * 128;
    auto eight = [&](int g) { return keys + ((((uint32_t)(qt & 1) * 4 + g) ^ ((uint32_t)d & 7)) << 4); };
    const int per_row = min(16, (p.vdim - e0) >> 3);  // pieces of eight columns
    bool ok = true;
    for (int c = 0; c < nc; ++c) {
      const int n = on ? len - c * HC_L - 32 * qt : 0;  // tokens here
      float k[32], all = 1.f;
      ok = ok && __all_sync(0xffffffffu, mbar_wait(z_full, (uint32_t)(c & 1), abort_flag, p.status, 2020));
#pragma unroll
      for (int i = 0; i < 32; ++i) k[i] = hc_logit(smem_u32(z_s), d, 32 * qt + i);
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        k[i] = i < n ? __fdividef(room, 1.f + hc_exp(k[i] + bias)) : 0.f;
        all = fmaf(-k[i], all, all);
      }
      mbar_arrive(z_free);
      float* pr = prod + (c & 1) * 512 + d;
      pr[128 * qt] = all;
      hc_sync<HC_WORK>();
      float w = 1.f;  // the gates of the quarters behind this one
      for (int i = 3; i > qt; --i) w *= pr[128 * i];
      const float decay = (pr[0] * pr[128]) * (pr[256] * pr[384]);
      // the products of the chunk before have read the keys and left the state
      if (c > 0) ok = ok && __all_sync(0xffffffffu, mbar_wait(acc_full, (uint32_t)((c - 1) & 1), abort_flag, p.status, 2021));
      if (c > 0) {
        if (ok && x0 < cols) {
          tc_fence_after();
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            float s[16];
            tmem_ld_32x16(t_row + 16 * y, s);
            tmem_ld_wait();
            uint32_t u[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) u[i] = __float_as_uint(s[i] * decay);
            tmem_st_32x16(t_row + 16 * y, u);
#pragma unroll
            for (int g = 0; g < 2; ++g) {
              const float v[8] = {s[8 * g], s[8 * g + 1], s[8 * g + 2], s[8 * g + 3], s[8 * g + 4], s[8 * g + 5], s[8 * g + 6], s[8 * g + 7]};
              hc_put8(eight(2 * y + g), eight(2 * y + g) + 2 * HC_BOX, v);
            }
          }
          tmem_st_wait();
        }
        hc_sync<HC_WORK>();
        const size_t base = ((size_t)(chunk0 + c) * p.heads + h) * p.dim * p.vdim + e0;
        const int g = tid & 15;
        for (int r = g < per_row ? tid >> 4 : p.dim; r < p.dim; r += HC_WORK / 16) {
          const uint8_t* src = k_s + (size_t)(g >> 3) * HC_BOX + (size_t)r * 128 + (((g & 7) ^ (r & 7)) << 4);
          const size_t at = base + (size_t)r * p.vdim + 8 * g;
          *reinterpret_cast<uint4*>(p.s_hi + at) = *reinterpret_cast<const uint4*>(src);
          *reinterpret_cast<uint4*>(p.s_lo + at) = *reinterpret_cast<const uint4*>(src + 2 * HC_BOX);
        }
        hc_sync<HC_WORK>();  // the keys may take the place
      }
      if (!ok) continue;
#pragma unroll
      for (int g = 3; g >= 0; --g) {
        float v[8];
#pragma unroll
        for (int i = 7; i >= 0; --i) {
          v[i] = k[8 * g + i] * w;
          w = fmaf(-k[8 * g + i], w, w);
        }
        hc_put8(eight(g), eight(g) + 2 * HC_BOX, v);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(ready);
    }
    if (nc > 0) {
      ok = ok && __all_sync(0xffffffffu, mbar_wait(acc_full, (uint32_t)((nc - 1) & 1), abort_flag, p.status, 2030));
      const int slot = p.seq_slot != nullptr ? p.seq_slot[seq] : -1;
      if (ok && slot >= 0 && slot < p.slots && x0 < cols) {
        tc_fence_after();
        float* dst = p.S + (((size_t)slot * p.heads + h) * p.dim + d) * p.vdim + e0 + x0;
#pragma unroll 1
        for (int x = 0; x < 32; x += 16) {
          float s[16];
          tmem_ld_32x16(t_row + x, s);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; i += 4)
            if (on && e0 + x0 + x + i < p.vdim) store4(dst + x + i, make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]));
        }
        tc_fence_before();
      }
    }
  }
  __syncthreads();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 17) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 128);
  }
}

// ------------------------------------------------------------------------------------------------------------
// Output pass.  Warps 0-7: thread (channel, half of the tokens) holds its keys and queries in registers and writes them, scaled,
// level by level (rows of the operands are channels: eight tokens are one 16-byte store); later warp (32 queries, 64 keys) turns the
// levels' products into scores, and (32 queries, 64 columns) norms the output.  Warp 8: TMA; warp 9: MMA.  Every barrier is used once.
//
// Gate logits and queries come to slot 1 and go to registers.  Steps: 0 blocks of 8, 1 - 4 levels of 64, 32, 16, 8, 5 queries against
// the state.  Two slots of shared memory (queries 64 KB, keys 32 KB, value and remainder each) and 32 KB more for the keys 64 .. 127 of
// step 0, where v goes later; the state goes where keys were.
// TMEM: levels [0, 256), blocks of 8 [256, 384), output [384, 512); the scores replace the levels of 64 and 32.
// ------------------------------------------------------------------------------------------------------------
constexpr int HO_WORK = 256, HO_THREADS = HO_WORK + 64;
constexpr uint32_t HO_SLOT = 6 * HC_BOX;
constexpr size_t HO_SMEM = 2 * (size_t)HO_SLOT + 2 * HC_BOX + 1024 + 1024 + 256;

__global__ void __launch_bounds__(HO_THREADS, 1)
hgrn2_output_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_z, const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_sh, const __grid_constant__ CUtensorMap tm_sl,
                    const Hgrn2Chunk p) {
  int seq = -1, c = (int)blockIdx.x;
  for (int s = 0; s < p.n_seq; ++s) {
    const int n = hc_chunks(p.cu[s + 1] - p.cu[s]);
    if (c < n) { seq = s; break; }
    c -= n;
  }
  if (seq < 0) return;  // uniform: before any barrier or TMEM use
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  // a slot: queries [2 groups of 64 tokens] value, remainder, keys [64 tokens] value, remainder
  uint8_t* x_s = smem + 2 * HO_SLOT;
  float* prod = reinterpret_cast<float*>(x_s + 2 * HC_BOX);  // [128] product of the gates of the first half
  float* norm = prod + 128;                                  // [128] weights of the norm
  uint64_t* bars = reinterpret_cast<uint64_t*>(norm + 128);
  uint64_t* full = bars;        // [6] operands of a step written
  uint64_t* done = bars + 6;    // [5] its products done
  uint64_t* v_full = bars + 11;
  uint64_t* s_full = bars + 12;
  uint64_t* p_full = bars + 13;
  uint64_t* o_full = bars + 14;
  uint64_t* in_full = bars + 15;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, e0 = blockIdx.z * 128, chunk = (int)blockIdx.x;  // chunks are numbered in the order of this search
  const int beg = p.cu[seq], len = p.cu[seq + 1] - beg, row0 = beg + c * HC_L;
  const int cols = min(128, (p.vdim - e0 + 15) & ~15), ksteps = (p.dim + 15) >> 4;
  const bool carried = c > 0;

  if (tid == 0) {
    for (int i = 0; i < 6; ++i) mbar_init(&full[i], HO_WORK);
    for (int i = 0; i < 5; ++i) mbar_init(&done[i], 1);
    mbar_init(v_full, 1);
    mbar_init(s_full, 1);
    mbar_init(p_full, HO_WORK);
    mbar_init(o_full, 1);
    mbar_init(in_full, 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_z);
    tma_prefetch_desc(&tm_v);
    tma_prefetch_desc(&tm_sh);
    tma_prefetch_desc(&tm_sl);
  }
  if (warp == 9) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  // state: values where the keys of step 3 were, remainders where those of step 4 were
  uint8_t* s_hi_s = smem + HO_SLOT + 4 * HC_BOX;
  uint8_t* s_lo_s = smem + 4 * HC_BOX;

  if (warp == 8) {
    if (lane == 0) {
      mbar_expect_tx(in_full, 6 * HC_BOX);
      for (int i = 0; i < 4; ++i) tma_load_3d(smem + HO_SLOT + i * HC_BOX, &tm_z, in_full, 64 * i, h, row0);
      for (int i = 0; i < 2; ++i) tma_load_3d(smem + HO_SLOT + (4 + i) * HC_BOX, &tm_q, in_full, 64 * i, h, row0);
      if (mbar_wait(&done[0], 0, abort_flag, p.status, 2100)) {
        mbar_expect_tx(v_full, 2 * HC_BOX);
        for (int i = 0; i < 2; ++i) tma_load_3d(x_s + i * HC_BOX, &tm_v, v_full, e0 + 64 * i, h, row0);
      }
      if (carried && mbar_wait(&done[3], 0, abort_flag, p.status, 2101)) {
        mbar_expect_tx(s_full, 4 * HC_BOX);
        for (int i = 0; i < 2; ++i) tma_load_3d(s_hi_s + i * HC_BOX, &tm_sh, s_full, e0 + 64 * i, 0, chunk * p.heads + h);
        if (mbar_wait(&done[4], 0, abort_flag, p.status, 2102))
          for (int i = 0; i < 2; ++i) tma_load_3d(s_lo_s + i * HC_BOX, &tm_sl, s_full, e0 + 64 * i, 0, chunk * p.heads + h);
      }
    }
    __syncwarp();
  } else if (warp == 9) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16_major(128, 64, true, true), idesc_0 = umma_idesc_bf16_major(128, 128, true, true);
      const uint32_t idesc_x = umma_idesc_bf16_major(128, cols, true, true), idesc_o = umma_idesc_bf16_major(128, cols, false, true);
      const uint64_t base = umma_desc_mnmajor_sw128(smem_u32(smem), HC_BOX);
      // step 0 reads keys from two places, 64 tokens each
      const uint64_t base0 = umma_desc_mnmajor_sw128(smem_u32(smem), 2 * HO_SLOT - 4 * HC_BOX);
      // value x value, value x remainder, remainder x value
      auto products = [&](uint32_t tmem_d, uint32_t slot, uint64_t keys, uint32_t idesc) {
#pragma unroll 1
        for (int part = 0; part < 3; ++part) {
          const uint64_t da = desc_at(base, slot + (part == 2 ? 2 * HC_BOX : 0)), db = desc_at(keys, slot + 4 * HC_BOX + (part == 1 ? HC_BOX : 0));
#pragma unroll 1
          for (int kk = 0; kk < ksteps; ++kk) umma_bf16_ss(tmem_d, desc_at(da, kk * 2048), desc_at(db, kk * 2048), idesc, (part | kk) != 0);
        }
      };
      bool ok = true;
      for (int s = 0; s < 5 && ok; ++s) {
        ok = mbar_wait(&full[s], 0, abort_flag, p.status, 2110 + s);
        if (!ok) break;
        tc_fence_after();
        const uint32_t slot = (s & 1) * HO_SLOT;
        if (s == 0) products(tmem_base + 256, slot, base0, idesc_0);
        else products(tmem_base + 64 * (s - 1), slot, base, idesc_s);
        umma_commit(&done[s]);
      }
      if (ok && carried) {
        ok = mbar_wait(&full[5], 0, abort_flag, p.status, 2116) && mbar_wait(s_full, 0, abort_flag, p.status, 2117);
        if (ok) {
          tc_fence_after();
          // the remainders of the state lie in slot 0, its values in slot 1
          const uint32_t s_hi = HO_SLOT + 4 * HC_BOX, s_lo = 4 * HC_BOX;
#pragma unroll 1
          for (int part = 0; part < 3; ++part) {
            const uint64_t da = desc_at(base, HO_SLOT + (part == 2 ? 2 * HC_BOX : 0)), db = desc_at(base, part == 1 ? s_lo : s_hi);
#pragma unroll 1
            for (int kk = 0; kk < ksteps; ++kk) umma_bf16_ss(tmem_base + 384, desc_at(da, kk * 2048), desc_at(db, kk * 2048), idesc_x, (part | kk) != 0);
          }
        }
      }
      if (ok) ok = mbar_wait(p_full, 0, abort_flag, p.status, 2118) && mbar_wait(v_full, 0, abort_flag, p.status, 2119);
      if (ok) {
        tc_fence_after();
        const uint64_t db = desc_at(base, 2 * HO_SLOT);
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int kk = 0; kk < HC_L / 16; ++kk)
            umma_bf16_ts(tmem_base + 384, tmem_base + (uint32_t)(half * 64 + kk * 8), desc_at(db, kk * 2048), idesc_o, carried || (half | kk) != 0);
        umma_commit(o_full);
      }
    }
    __syncwarp();
  } else {
    const int d = tid & 127, half = tid >> 7;
    float k[64], q[64];
    bool ok = __all_sync(0xffffffffu, mbar_wait(in_full, 0, abort_flag, p.status, 2131));
    {
      const bool on = d < p.dim;
      const int hd = h * p.dim + (on ? d : 0), n = on ? len - c * HC_L - 64 * half : 0;  // tokens here
      const float bias = p.bias[hd], room = 1.f - p.low[hd];
      float all = 1.f;
#pragma unroll
      for (int i = 0; i < 64; ++i) {  // silu(q) and (1 - low) sigmoid(-z - bias) with one division
        const float z = hc_logit(smem_u32(smem) + HO_SLOT, d, 64 * half + i), x = hc_query(smem_u32(smem) + HO_SLOT + 4 * HC_BOX, d, 64 * half + i);
        const float a = 1.f + hc_exp(-x), b = 1.f + hc_exp(z + bias), r = __fdividef(1.f, a * b);
        q[i] = i < n ? x * (r * b) : 0.f;
        k[i] = i < n ? room * (r * a) : 0.f;
        all = fmaf(-k[i], all, all);
      }
      if (half == 0) prod[d] = all;
      else if (p.norm != nullptr && d < p.vdim) norm[d] = p.norm[d];
    }
    hc_sync<HO_WORK>();  // slot 1 is free
    const uint32_t sw = (uint32_t)(d & 7), row = smem_u32(smem) + (uint32_t)d * 128;
    auto chunk16 = [&](uint32_t g) { return row + ((g ^ sw) << 4); };  // eight tokens, number g of a group of 64
    const uint32_t mine = (uint32_t)half * HC_BOX;  // this half's group of queries
    // queries i0 .. i0 + n - 1 of this half times the gates from i0 on (and w)
    auto queries = [&](uint32_t slot, auto i0c, auto nc, float w) {
      constexpr int i0 = decltype(i0c)::value, n = decltype(nc)::value;
      w = hc_afresh(w);
#pragma unroll
      for (int g = 0; g < n / 8; ++g) {
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          w = fmaf(-k[i0 + 8 * g + i], w, w);
          v[i] = q[i0 + 8 * g + i] * w;
        }
        const uint32_t at = chunk16((uint32_t)(i0 / 8 + g)) + mine + slot;
        hc_put8(at, at + 2 * HC_BOX, v);
      }
    };
    // keys i0 .. i0 + n - 1 times the gates behind them up to i0 + n - 1; g0: where they begin among the 64 of the level
    auto keys = [&](uint32_t slot, auto i0c, auto nc, int g0) {
      constexpr int i0 = decltype(i0c)::value, n = decltype(nc)::value;
      float w = hc_afresh(1.f);
#pragma unroll
      for (int g = n / 8 - 1; g >= 0; --g) {
        float v[8];
#pragma unroll
        for (int i = 7; i >= 0; --i) {
          v[i] = k[i0 + 8 * g + i] * w;
          w = fmaf(-k[i0 + 8 * g + i], w, w);
        }
        const uint32_t at = chunk16((uint32_t)(g0 + g)) + slot + 4 * HC_BOX;
        hc_put8(at, at + HC_BOX, v);
      }
    };
    constexpr uint32_t slot0 = 0, slot1 = HO_SLOT;
    auto filled = [&](int s) {
      fence_proxy_async_smem();
      mbar_arrive(&full[s]);
    };
    auto emptied = [&](int s) { return __all_sync(0xffffffffu, mbar_wait(&done[s], 0, abort_flag, p.status, 2120 + s)); };

    // step 0: about the middle of every block of 8 (behind its fourth token)
    {
      const uint32_t b = half == 0 ? slot0 + 4 * HC_BOX : 2 * HO_SLOT;
#pragma unroll
      for (int g = 0; g < 8; ++g) {
        auto gate = [&](int i) { return fmaxf(1.f - hc_afresh(k[8 * g + i]), 5.9604644775390625e-8f); };
        const uint32_t at = chunk16((uint32_t)g);
        // products of the gates from the middle to the ends of the block, and their inverses
        const float low = gate(1) * gate(2) * gate(3), high = gate(4) * gate(5) * gate(6) * gate(7);
        float v[8], w = __fdividef(1.f, low);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          v[i] = q[8 * g + i] * w;
          if (i < 3) w *= gate(i + 1);
        }
        w = 1.f;
#pragma unroll
        for (int i = 4; i < 8; ++i) {
          w *= gate(i);
          v[i] = q[8 * g + i] * w;
        }
        hc_put8(at + mine + slot0, at + mine + slot0 + 2 * HC_BOX, v);
        w = hc_afresh(__fdividef(1.f, high));
#pragma unroll
        for (int i = 7; i >= 4; --i) {
          v[i] = k[8 * g + i] * w;
          w *= gate(i);
        }
        w = hc_afresh(1.f);
#pragma unroll
        for (int i = 3; i >= 0; --i) {
          v[i] = k[8 * g + i] * w;
          w *= gate(i);
        }
        hc_put8(at + b, at + b + HC_BOX, v);
      }
    }
    filled(0);
    // step 1: the halves are keys or queries as a whole
    if (half == 0) keys(slot1, HcInt<0>{}, HcInt<64>{}, 0);
    else queries(slot1, HcInt<0>{}, HcInt<64>{}, 1.f);
    filled(1);
    ok = ok && emptied(0);
    if (ok) {
      keys(slot0, HcInt<0>{}, HcInt<32>{}, 4 * half);
      queries(slot0, HcInt<32>{}, HcInt<32>{}, 1.f);
      filled(2);
      ok = emptied(1);
    }
    if (ok) {
      keys(slot1, HcInt<0>{}, HcInt<16>{}, 4 * half);
      queries(slot1, HcInt<16>{}, HcInt<16>{}, 1.f);
      keys(slot1, HcInt<32>{}, HcInt<16>{}, 4 * half + 2);
      queries(slot1, HcInt<48>{}, HcInt<16>{}, 1.f);
      filled(3);
      ok = emptied(2);
    }
    if (ok) {
      keys(slot0, HcInt<0>{}, HcInt<8>{}, 4 * half);
      queries(slot0, HcInt<8>{}, HcInt<8>{}, 1.f);
      keys(slot0, HcInt<16>{}, HcInt<8>{}, 4 * half + 1);
      queries(slot0, HcInt<24>{}, HcInt<8>{}, 1.f);
      keys(slot0, HcInt<32>{}, HcInt<8>{}, 4 * half + 2);
      queries(slot0, HcInt<40>{}, HcInt<8>{}, 1.f);
      keys(slot0, HcInt<48>{}, HcInt<8>{}, 4 * half + 3);
      queries(slot0, HcInt<56>{}, HcInt<8>{}, 1.f);
      filled(4);
      ok = emptied(3);
    }
    if (ok && carried) {
      queries(slot1, HcInt<0>{}, HcInt<64>{}, half == 0 ? 1.f : prod[d]);
      filled(5);
    }
    if (ok) ok = emptied(4);
    // scores: warp (queries 32 rq .., keys 64 kh ..)
    const int rq = warp & 3, kh = warp >> 2;
    const uint32_t t_lane = tmem_base + ((uint32_t)(rq * 32) << 16);
    uint32_t a[2][16], b[2][16];
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int kq = 2 * kh + j;
        float v[32];
        if (kq < rq) {
          tmem_ld_32x32(t_lane + (uint32_t)(rq >= 2 && kq < 2 ? 32 * kq : 64 + 32 * (rq >> 1)), v);
          tmem_ld_wait();
        } else if (kq == rq) {
          float l16[16], l8[16];
          tmem_ld_32x32(t_lane + 256 + 32 * rq, v);
          tmem_ld_32x16(t_lane + 128 + 16 * rq, l16);
          tmem_ld_32x16(t_lane + 192 + 16 * rq, l8);
          tmem_ld_wait();
#pragma unroll
          for (int x = 0; x < 32; ++x) {
            float s = v[x];  // same block of 8
            if ((lane >> 3) != (x >> 3) && (x & 15) < 8) s = l8[8 * (x >> 4) + (x & 7)];
            if (x < 16 && lane >= 16) s = l16[x & 15];
            v[x] = x <= lane ? s : 0.f;
          }
        } else {
#pragma unroll
          for (int x = 0; x < 32; ++x) v[x] = 0.f;
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          a[j][i] = pack_bf16(v[2 * i], v[2 * i + 1]);
          const float2 f = unpack_bf16(a[j][i]);
          b[j][i] = pack_bf16(v[2 * i] - f.x, v[2 * i + 1] - f.y);
        }
      }
      tc_fence_before();
    }
    hc_sync<HO_WORK>();  // every warp has read what the scores replace
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        tmem_st_32x16(t_lane + 16 * (2 * kh + j), a[j]);
        tmem_st_32x16(t_lane + 64 + 16 * (2 * kh + j), b[j]);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(p_full);
      ok = __all_sync(0xffffffffu, mbar_wait(o_full, 0, abort_flag, p.status, 2130));
    }
    {
      tc_fence_after();
      const int t = c * HC_L + 32 * rq + lane, x0 = 64 * kh;  // this warp's columns
      const bool row_ok = ok && t < len;
      float o[2][32], ss = 0.f;
      if (ok && x0 < cols) {
        tmem_ld_32x32(t_lane + 384 + x0, o[0]);
        tmem_ld_32x32(t_lane + 416 + x0, o[1]);
        tmem_ld_wait();
      }
      if (p.norm != nullptr) {
        float* red = reinterpret_cast<float*>(smem);  // [2][128]: nothing reads the operands any more
        if (ok && x0 < cols) {
#pragma unroll
          for (int x = 0; x < 64; ++x) ss += x0 + x < p.vdim ? o[x >> 5][x & 31] * o[x >> 5][x & 31] : 0.f;
        }
        red[kh * 128 + 32 * rq + lane] = ss;
        hc_sync<HO_WORK>();
        const float* r = red + 32 * rq + lane;
        const float f = p.scale / sqrtf((r[0] + r[128]) / (float)p.vdim + p.eps);
        uint8_t* rows = smem + HC_BOX;  // two boxes of 64 columns, rows are tokens
#pragma unroll
        for (int x = 0; x < 64; x += 8) {
          if (x0 + x < p.vdim) {
            const float* u = &o[x >> 5][x & 31];
            const float4 g = load4(norm + x0 + x), g2 = load4(norm + x0 + x + 4);
            *reinterpret_cast<uint4*>(rows + (size_t)kh * HC_BOX + (size_t)(32 * rq + lane) * 128 + (((x >> 3) ^ (lane & 7)) << 4)) =
                make_uint4(pack_bf16(u[0] * f * g.x, u[1] * f * g.y), pack_bf16(u[2] * f * g.z, u[3] * f * g.w),
                           pack_bf16(u[4] * f * g2.x, u[5] * f * g2.y), pack_bf16(u[6] * f * g2.z, u[7] * f * g2.w));
          }
        }
        hc_sync<HO_WORK>();
        const int g = tid & 15, n = ok && g < (p.vdim >> 3) ? min(HC_L, len - c * HC_L) : 0;  // pieces of eight columns
        for (int r = tid >> 4; r < n; r += HO_WORK / 16) {
          *reinterpret_cast<uint4*>(p.y_out + (size_t)(row0 + r) * p.out_ld + (size_t)h * p.vdim + 8 * g) =
              *reinterpret_cast<const uint4*>(rows + (size_t)(g >> 3) * HC_BOX + (size_t)r * 128 + (((g & 7) ^ (r & 7)) << 4));
        }
      } else if (row_ok) {
        float* dst = p.out + ((size_t)(beg + t) * p.heads + h) * p.vdim + e0 + x0;
#pragma unroll
        for (int x = 0; x < 64; x += 4) {
          const float* u = &o[x >> 5][x & 31];
          if (e0 + x0 + x < p.vdim) store4(dst + x, make_float4(u[0], u[1], u[2], u[3]));
        }
      }
      tc_fence_before();
    }
  }
  __syncthreads();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

}  // namespace trlb

using namespace trlb;

// 1 when trlb_hgrn2_chunk takes these sizes.
TRLB_API int trlb_hgrn2_chunk_ok(int heads, int dim, int vdim) { return heads > 0 && dim > 0 && dim <= 128 && dim % 8 == 0 && vdim > 0 && vdim % 8 == 0; }

// Chunks (upper bound) of T packed tokens in n_seq sequences: the leading size of s_hi, s_lo [chunks, heads, dim, vdim] bf16.
TRLB_API int trlb_hgrn2_chunks(int T, int n_seq) { return (T + HC_L - 1) / HC_L + n_seq; }

// y [T rows of y_ld] bf16 on 16 bytes: q at 0, v at v_off (elements, a multiple of 8); z [T rows of z_ld] fp32 on 16 bytes, gate logits without
// bias.  S [slots, heads, dim, vdim] of seq_slot gets the final states (null: none).  norm [vdim] (vdim <= 128): y_out [T rows of out_ld on 16
// bytes] = outputs over their rms per head times norm and scale, bf16; else out [T, heads, vdim] fp32.
TRLB_API int trlb_hgrn2_chunk(const void* y, long long y_ld, int v_off, const float* z, long long z_ld, const float* bias, const float* low,
                              const int* cu, int n_seq, int T, const int* seq_slot, float* S, int slots, int heads, int dim, int vdim,
                              const float* norm, float eps, float scale, void* y_out, long long out_ld, float* out, void* s_hi, void* s_lo,
                              int* status, cudaStream_t st) {
  if (T <= 0 || n_seq <= 0) return 0;
  const auto off16 = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) != 0; };
  if (!trlb_hgrn2_chunk_ok(heads, dim, vdim) || (y_ld % 8) || (v_off % 8) || (z_ld % 4) || off16(y) || off16(z)) return -310;
  if (norm != nullptr ? vdim > 128 || y_out == nullptr || (out_ld % 8) || off16(y_out) || off16(norm) : out == nullptr) return -310;
  if (seq_slot != nullptr && S == nullptr) return -310;
  const int chunks = trlb_hgrn2_chunks(T, n_seq);
  const __nv_bfloat16* x = (const __nv_bfloat16*)y;
  CUtensorMap tq, tz, tv, tsh, tsl;
  using trlb_host::make_tmap_3d_bf16;
  if (make_tmap_3d_bf16(&tq, x, dim, heads, T, dim, (uint64_t)y_ld, 64, 1, 128)) return -315;
  // fp32 rows as twice as many 16-bit elements: they are only copied
  if (make_tmap_3d_bf16(&tz, z, 2 * dim, heads, T, 2 * dim, (uint64_t)z_ld * 2, 64, 1, 128)) return -316;
  if (make_tmap_3d_bf16(&tv, x + v_off, vdim, heads, T, vdim, (uint64_t)y_ld, 64, 1, 128)) return -311;
  if (make_tmap_3d_bf16(&tsh, s_hi, vdim, dim, (uint64_t)chunks * heads, vdim, (uint64_t)dim * vdim, 64, 128, 1)) return -312;
  if (make_tmap_3d_bf16(&tsl, s_lo, vdim, dim, (uint64_t)chunks * heads, vdim, (uint64_t)dim * vdim, 64, 128, 1)) return -313;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(hgrn2_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)HS_SMEM) != cudaSuccess ||
        cudaFuncSetAttribute(hgrn2_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)HO_SMEM) != cudaSuccess)
      return -314;
    attr_set = true;
  }
  Hgrn2Chunk p = {};
  p.cu = cu; p.n_seq = n_seq; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.bias = bias; p.low = low;
  p.s_hi = (__nv_bfloat16*)s_hi; p.s_lo = (__nv_bfloat16*)s_lo; p.S = S; p.seq_slot = seq_slot; p.slots = slots;
  p.norm = norm; p.eps = eps; p.scale = scale; p.y_out = (__nv_bfloat16*)y_out; p.out_ld = out_ld; p.out = out; p.status = status;
  const int tiles = (vdim + 127) / 128;
  hgrn2_state_kernel<<<dim3(n_seq, heads, tiles), HS_THREADS, HS_SMEM, st>>>(tz, tv, p);
  hgrn2_output_kernel<<<dim3(chunks, heads, tiles), HO_THREADS, HO_SMEM, st>>>(tq, tz, tv, tsh, tsl, p);
  return (int)cudaGetLastError();
}
