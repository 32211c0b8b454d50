// Real-gated linear recurrent unit on the 5th-generation tensor cores (bf16 models): the block-diagonal gate products, the
// recurrence and the multiplication by the GELU branch in one kernel, for prompts and for one decode step.
//
// The weights are the M operand: D[channel, token] = W_b[channel, :] u_t, one product for each of the two gates, so that an
// epilogue thread owns a channel and its tokens lie along the columns it reads: the recurrence runs in registers and no
// gate, decay or state crosses memory.
//
// Prompt: one CTA per (128 channels of a block, sequence) walks the sequence in 64-token tiles.  Both weight slices stay in
// shared memory; u tiles come through a TMA ring; the products are double-buffered in TMEM.  Four groups of 128 epilogue
// threads take 16 tokens each: a group forms its decays and inputs, runs its 16 tokens from a zero state and keeps the
// running product of the decays; (product, end) of the four groups meet in shared memory, and every thread folds them into
// the carried state (one barrier per tile).  S_t = local_t + product_t * S_in.
//
// Decode: one CTA per (128 channels, 16 slots); columns are slots, states are read and written in place.  The weights are
// requested before the wait on the previous kernel.
//
// sqrt(1 - a^2) = sqrt(-expm1(2 log a)): by its series where log a is small, by 1 - a^2 elsewhere.
#include "mixers.cuh"
#include "rglru.cuh"

namespace trlb {

constexpr int RG_N = 64, RG_GROUPS = 4, RG_PER = RG_N / RG_GROUPS;
constexpr int RG_EPI = 128 * RG_GROUPS, RG_THREADS = RG_EPI + 64;
constexpr uint32_t RG_WBOX = 128 * 64 * 2;  // 128 channels x 64 inputs
constexpr int RG_MAX_STAGES = 4;

struct RgTc {
  RgLru p;
  int blocks, wb, kb, tiles_per_block, stages;
  const int* cu;          // prompt
  const int* seq_slot;    // prompt, or null
  const int* seq_lens;    // decode
  int B;                  // decode
  const __nv_bfloat16* y; // prompt: [T rows of y_ld]
  float* y_sums;          // decode: [B rows of y_ld], cleared
  long long y_ld;
  __nv_bfloat16* out;     // [T or B, C]
  int* status;
};

__device__ __forceinline__ bool rg_vote(bool pred, int id, int count) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 q, %1, 0;\n\t"
      "bar.red.and.pred p, %2, %3, q;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(out)
      : "r"((uint32_t)pred), "r"(id), "r"(count)
      : "memory");
  return out != 0;
}

// decay a and weight of the input sqrt(1 - a^2) * i
__device__ __forceinline__ void rg_gates(float zr, float zi, float neg_sp, float& a, float& w) {
  const float la = neg_sp * fast_sigmoid(zr);
  a = fast_exp2(1.4426950408889634f * la);
  const float x = 2.f * la;  // 1 - a^2 = -x - x^2/2 - ... for small |x|
  float s = fmaf(x, 1.f / 5040.f, 1.f / 720.f);
  s = fmaf(x, s, 1.f / 120.f);
  s = fmaf(x, s, 1.f / 24.f);
  s = fmaf(x, s, 1.f / 6.f);
  s = fmaf(x, s, 0.5f);
  s = fmaf(x, s, 1.f);
  const float v = fmaxf(x > -0.25f ? -x * s : fmaf(-a, a, 1.f), 1e-37f);
  w = v * rsqrtf(v) * fast_sigmoid(zi);
}

__global__ void __launch_bounds__(RG_THREADS, 1)
rglru_prompt_tc_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_u, const RgTc q) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t u_bytes = (uint32_t)q.kb * RG_N * 128;
  uint8_t* w_s = smem;                                        // [2][kb] boxes
  uint8_t* u_s = w_s + (size_t)2 * q.kb * RG_WBOX;            // [stages][kb] boxes of 64 tokens
  float2* pl = reinterpret_cast<float2*>(u_s + (size_t)q.stages * u_bytes);  // [2][RG_GROUPS][128]
  uint64_t* bars = reinterpret_cast<uint64_t*>(pl + 2 * RG_GROUPS * 128);
  uint64_t* w_full = bars;
  uint64_t* u_full = bars + 1;                  // [RG_MAX_STAGES]
  uint64_t* u_empty = u_full + RG_MAX_STAGES;   // [RG_MAX_STAGES]
  uint64_t* t_full = u_empty + RG_MAX_STAGES;   // [2]
  uint64_t* t_empty = t_full + 2;               // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(t_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.y, blk = (int)blockIdx.x / q.tiles_per_block, c0 = ((int)blockIdx.x % q.tiles_per_block) * 128;
  const int beg = q.cu[seq], len = q.cu[seq + 1] - beg;
  const int n_t = (len + RG_N - 1) / RG_N;

  if (threadIdx.x == 0) {
    mbar_init(w_full, 1);
    for (int s = 0; s < RG_MAX_STAGES; ++s) {
      mbar_init(&u_full[s], 1);
      mbar_init(&u_empty[s], 1 + RG_EPI / 32);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&t_full[s], 1);
      mbar_init(&t_empty[s], RG_EPI / 32);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_u);
  }
  if (warp == RG_EPI / 32) {
    tmem_alloc(tmem_slot, 4 * RG_N);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == RG_EPI / 32 + 1) {
    // ---------------- TMA producer ----------------
    if (lane == 0 && n_t > 0) {
      mbar_expect_tx(w_full, (uint32_t)(2 * q.kb) * RG_WBOX);
      for (int g = 0; g < 2; ++g)
        for (int i = 0; i < q.kb; ++i)
          tma_load_3d(w_s + (size_t)(g * q.kb + i) * RG_WBOX, &tm_w, w_full, 64 * i, c0, g * q.blocks + blk);
      for (int j = 0; j < n_t; ++j) {
        const int s = j % q.stages;
        if (!mbar_wait(&u_empty[s], (uint32_t)(((j / q.stages) & 1) ^ 1), abort_flag, q.status, 1700 + s)) break;
        mbar_expect_tx(&u_full[s], u_bytes);
        for (int i = 0; i < q.kb; ++i)
          tma_load_3d(u_s + (size_t)s * u_bytes + (size_t)i * RG_N * 128, &tm_u, &u_full[s], 64 * i, blk, beg + j * RG_N);
      }
    }
    __syncwarp();
  } else if (warp == RG_EPI / 32) {
    // ---------------- MMA issuer ----------------
    if (lane == 0 && n_t > 0) {
      constexpr uint32_t idesc = umma_idesc_bf16(128, RG_N);
      const uint64_t w_d = umma_desc_kmajor_sw128(smem_u32(w_s)), u_d = umma_desc_kmajor_sw128(smem_u32(u_s));
      bool ok = mbar_wait(w_full, 0, abort_flag, q.status, 1710);
      for (int j = 0; j < n_t && ok; ++j) {
        const int s = j % q.stages, a = j & 1;
        if (!mbar_wait(&t_empty[a], (uint32_t)(((j >> 1) & 1) ^ 1), abort_flag, q.status, 1711 + a)) break;
        if (!mbar_wait(&u_full[s], (uint32_t)((j / q.stages) & 1), abort_flag, q.status, 1720 + s)) break;
        tc_fence_after();
        for (int g = 0; g < 2; ++g) {
          const uint32_t d = tmem_base + (uint32_t)(a * 2 + g) * RG_N;
          for (int i = 0; i < q.kb; ++i) {
            const uint64_t da = desc_at(w_d, (uint32_t)(g * q.kb + i) * RG_WBOX);
            const uint64_t db = desc_at(u_d, (uint32_t)s * u_bytes + (uint32_t)i * RG_N * 128);
            const int steps = min(4, (q.wb - 64 * i + 15) >> 4);
            for (int kk = 0; kk < steps; ++kk) umma_bf16_ss(d, da + 2 * kk, db + 2 * kk, idesc, (i | kk) != 0);
          }
        }
        umma_commit(&t_full[a]);
        umma_commit(&u_empty[s]);
      }
    }
    __syncwarp();
  } else {
    // ---------------- gates and recurrence: one thread per (channel, 16 tokens of a tile) ----------------
    const int g = warp >> 2, r = (warp & 3) * 32 + lane;
    const int cb = c0 + r;                      // channel inside the block
    const bool ch_ok = cb < q.wb;
    const int c = blk * q.wb + (ch_ok ? cb : 0);
    const float neg_sp = -q.p.decay * rg_softplus(q.p.lam[c]), br = q.p.gate_bias[c], bi = q.p.gate_bias[q.p.C + c], by = q.p.y_bias[c];
    const uint32_t t_row = tmem_base + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)(g * RG_PER);
    const uint32_t u_col = (uint32_t)(cb >> 6) * RG_N * 128 + (uint32_t)(cb & 7) * 2;
    const uint32_t u_chunk = (uint32_t)(cb & 63) >> 3;
    float carry = 0.f;
    bool ok = true;
    for (int j = 0; j < n_t; ++j) {
      const int s = j % q.stages, a = j & 1;
      const int first = j * RG_N + g * RG_PER, n_ok = max(0, min(RG_PER, len - first));
      const size_t row = (size_t)(beg + first);
      uint16_t yv[RG_PER];
#pragma unroll
      for (int i = 0; i < RG_PER; ++i)
        yv[i] = (i < n_ok && ch_ok) ? *reinterpret_cast<const uint16_t*>(q.y + (row + i) * q.y_ld + c) : (uint16_t)0;
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&t_full[a], (uint32_t)((j >> 1) & 1), abort_flag, q.status, 1730 + a));
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&u_full[s], (uint32_t)((j / q.stages) & 1), abort_flag, q.status, 1740 + s));
      float x[RG_PER], P[RG_PER];
      if (ok) {
        tc_fence_after();
        tmem_ld_32x16(t_row + (uint32_t)(a * 2) * RG_N, x);
        tmem_ld_32x16(t_row + (uint32_t)(a * 2 + 1) * RG_N, P);
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&t_empty[a]);
        float h = 0.f, prod = 1.f;
        const uint8_t* ut = u_s + (size_t)s * u_bytes + u_col;
#pragma unroll
        for (int i = 0; i < RG_PER; ++i) {
          const int n = g * RG_PER + i;
          float ac, w;
          rg_gates(x[i] + br, P[i] + bi, neg_sp, ac, w);
          const float uv = ch_ok ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(ut + n * 128 + ((u_chunk ^ (uint32_t)(n & 7)) << 4))) : 0.f;
          if (i < n_ok) {
            h = fmaf(ac, h, w * uv);
            prod *= ac;
          }
          x[i] = h;
          P[i] = prod;
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(&u_empty[s]);
        pl[((j & 1) * RG_GROUPS + g) * 128 + r] = make_float2(prod, h);
      }
      ok = rg_vote(ok, 1, RG_EPI);  // the four groups' (product, end) are in shared memory
      if (!ok) break;
      float h_in = 0.f, h = carry;
#pragma unroll
      for (int k = 0; k < RG_GROUPS; ++k) {
        if (k == g) h_in = h;
        const float2 e = pl[((j & 1) * RG_GROUPS + k) * 128 + r];
        h = fmaf(e.x, h, e.y);
      }
      carry = h;
      if (ch_ok) {
#pragma unroll
        for (int i = 0; i < RG_PER; ++i) {
          if (i < n_ok) {
            const float y = __bfloat162float(__ushort_as_bfloat16(yv[i])) + by;
            q.out[(row + i) * q.p.C + c] = __float2bfloat16(fmaf(P[i], h_in, x[i]) * fast_gelu_tanh(y));
          }
        }
      }
    }
    if (ok && g == 0 && ch_ok && q.seq_slot != nullptr && q.p.state != nullptr) {
      const int slot = q.seq_slot[seq];
      if (slot >= 0 && slot < q.p.slots) q.p.state[(size_t)slot * q.p.C + c] = carry;
    }
  }
  __syncthreads();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == RG_EPI / 32) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 4 * RG_N);
  }
}

constexpr int RG_SLOTS = 16;
__global__ void __launch_bounds__(192)
rglru_step_tc_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_u, const RgTc q) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* w_s = smem;                                   // [2][kb] boxes
  uint8_t* u_s = w_s + (size_t)2 * q.kb * RG_WBOX;       // [kb] boxes of 16 slots
  uint64_t* bars = reinterpret_cast<uint64_t*>(u_s + (size_t)q.kb * RG_SLOTS * 128);
  uint64_t* full = bars;
  uint64_t* done = bars + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blk = (int)blockIdx.x / q.tiles_per_block, c0 = ((int)blockIdx.x % q.tiles_per_block) * 128, b0 = (int)blockIdx.y * RG_SLOTS;
  if (threadIdx.x == 0) {
    mbar_init(full, 1);
    mbar_init(done, 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_u);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 32);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(full, (uint32_t)q.kb * (2 * RG_WBOX + RG_SLOTS * 128));
      for (int g = 0; g < 2; ++g)
        for (int i = 0; i < q.kb; ++i)
          tma_load_3d(w_s + (size_t)(g * q.kb + i) * RG_WBOX, &tm_w, full, 64 * i, c0, g * q.blocks + blk);
      pdl_wait();
      for (int i = 0; i < q.kb; ++i) tma_load_3d(u_s + (size_t)i * RG_SLOTS * 128, &tm_u, full, 64 * i, blk, b0);
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc_bf16(128, RG_SLOTS);
      if (mbar_wait(full, 0, abort_flag, q.status, 1760)) {
        tc_fence_after();
        const uint64_t w_d = umma_desc_kmajor_sw128(smem_u32(w_s)), u_d = umma_desc_kmajor_sw128(smem_u32(u_s));
        for (int g = 0; g < 2; ++g)
          for (int i = 0; i < q.kb; ++i) {
            const uint64_t da = desc_at(w_d, (uint32_t)(g * q.kb + i) * RG_WBOX), db = desc_at(u_d, (uint32_t)i * RG_SLOTS * 128);
            const int steps = min(4, (q.wb - 64 * i + 15) >> 4);
            for (int kk = 0; kk < steps; ++kk) umma_bf16_ss(tmem_base + g * RG_SLOTS, da + 2 * kk, db + 2 * kk, idesc, (i | kk) != 0);
          }
        umma_commit(done);
      }
    }
    __syncwarp();
  } else {
    const int r = (warp & 3) * 32 + lane, cb = c0 + r;
    const bool ch_ok = cb < q.wb;
    const int c = blk * q.wb + (ch_ok ? cb : 0);
    const float neg_sp = -q.p.decay * rg_softplus(q.p.lam[c]), br = q.p.gate_bias[c], bi = q.p.gate_bias[q.p.C + c], by = q.p.y_bias[c];
    pdl_wait();
    float y[RG_SLOTS], S[RG_SLOTS];
    uint32_t live = 0;
#pragma unroll
    for (int i = 0; i < RG_SLOTS; ++i) {
      const int b = b0 + i;
      const bool in = b < q.B && ch_ok;
      const bool on = in && q.seq_lens[b] >= 0;
      live |= (uint32_t)on << i;
      S[i] = on ? q.p.state[(size_t)b * q.p.C + c] : 0.f;
      y[i] = in ? q.y_sums[(size_t)b * q.y_ld + c] : 0.f;
      if (in) q.y_sums[(size_t)b * q.y_ld + c] = 0.f;
    }
    bool ok = __all_sync(0xffffffffu, mbar_wait(done, 0, abort_flag, q.status, 1770));
    ok = ok && __all_sync(0xffffffffu, mbar_wait(full, 0, abort_flag, q.status, 1771));
    if (ok) {
      tc_fence_after();
      float zr[RG_SLOTS], zi[RG_SLOTS];
      const uint32_t t_row = tmem_base + ((uint32_t)((warp & 3) * 32) << 16);
      tmem_ld_32x16(t_row, zr);
      tmem_ld_32x16(t_row + RG_SLOTS, zi);
      tmem_ld_wait();
      tc_fence_before();
      const uint8_t* ut = u_s + (size_t)(cb >> 6) * RG_SLOTS * 128 + (cb & 7) * 2;
      const uint32_t u_chunk = (uint32_t)(cb & 63) >> 3;
      if (ch_ok) {
#pragma unroll
        for (int i = 0; i < RG_SLOTS; ++i) {
          const int b = b0 + i;
          if (b < q.B) {
            float o = 0.f;
            if ((live >> i) & 1) {
              float ac, w;
              rg_gates(zr[i] + br, zi[i] + bi, neg_sp, ac, w);
              const float uv = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(ut + i * 128 + ((u_chunk ^ (uint32_t)(i & 7)) << 4)));
              const float h = fmaf(ac, S[i], w * uv);
              q.p.state[(size_t)b * q.p.C + c] = h;
              o = h * fast_gelu_tanh(y[i] + by);
            }
            q.out[(size_t)b * q.p.C + c] = __float2bfloat16(o);
          }
        }
      }
    }
  }
  __syncthreads();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 32);
  }
}

}  // namespace trlb

using namespace trlb;

namespace {

size_t rg_prompt_smem(int kb, int stages) {
  return (size_t)2 * kb * RG_WBOX + (size_t)stages * kb * RG_N * 128 + 2 * RG_GROUPS * 128 * 8 + 1024 + 256;
}
int rg_stages(int kb) {
  for (int s = RG_MAX_STAGES; s > 0; --s)
    if (rg_prompt_smem(kb, s) <= 227 * 1024) return s;
  return 0;
}
size_t rg_step_smem(int kb) { return (size_t)kb * (2 * RG_WBOX + RG_SLOTS * 128) + 1024 + 128; }

int rg_setup(RgTc& q, CUtensorMap& tw, CUtensorMap& tu, const void* w, const void* u, int C, int blocks, int rows, int box_rows) {
  q.blocks = blocks;
  q.wb = C / blocks;
  q.kb = (q.wb + 63) / 64;
  q.tiles_per_block = (q.wb + 127) / 128;
  using trlb_host::make_tmap_3d_bf16;
  if (make_tmap_3d_bf16(&tw, w, q.wb, q.wb, 2 * blocks, q.wb, (uint64_t)q.wb * q.wb, 64, 128, 1)) return -271;
  if (make_tmap_3d_bf16(&tu, u, q.wb, blocks, rows, q.wb, C, 64, 1, box_rows)) return -272;
  return 0;
}

}  // namespace

// 1 when the two kernels here take C channels in `blocks` blocks.
TRLB_API int trlb_rglru_tc_ok(int C, int blocks) {
  if (blocks <= 0 || C <= 0 || C % blocks) return 0;
  const int wb = C / blocks, kb = (wb + 63) / 64;
  return wb % 8 == 0 && rg_stages(kb) > 0 && rg_step_smem(kb) <= 227 * 1024;
}

// u [T, C], y [T rows of y_ld], w [2, blocks, C / blocks (out), C / blocks (in)], all bf16; sequences by cu [n_seq + 1];
// state (may be null) [slots, C] of seq_slot[seq]; out [T, C].
TRLB_API int trlb_rglru_prompt_tc(const void* u, const void* y, long long y_ld, const void* w, const float* lam,
                                  const float* gate_bias, const float* y_bias, const int* cu, int n_seq, int T,
                                  const int* seq_slot, int slots, float* state, float decay, int C, int blocks, void* out, int* status,
                                  cudaStream_t st) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (!trlb_rglru_tc_ok(C, blocks) || n_seq > 65535) return -270;
  RgTc q = {};
  CUtensorMap tw, tu;
  const int rc = rg_setup(q, tw, tu, w, u, C, blocks, T, RG_N);
  if (rc) return rc;
  q.p = {C, slots, lam, gate_bias, y_bias, state, decay};
  q.stages = rg_stages(q.kb);
  q.cu = cu; q.seq_slot = state != nullptr ? seq_slot : nullptr;
  q.y = (const __nv_bfloat16*)y; q.y_ld = y_ld; q.out = (__nv_bfloat16*)out; q.status = status;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(rglru_prompt_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -273;
    attr_set = true;
  }
  rglru_prompt_tc_kernel<<<dim3(blocks * q.tiles_per_block, n_seq), RG_THREADS, rg_prompt_smem(q.kb, q.stages), st>>>(tw, tu, q);
  return (int)cudaGetLastError();
}

// One token per slot: u [B, C] bf16, y_sums [B rows of y_ld] fp32 (cleared), state [B, C].
TRLB_API int trlb_rglru_step_tc(const void* u, float* y_sums, long long y_ld, const void* w, const float* lam,
                                const float* gate_bias, const float* y_bias, const int* seq_lens, int B, float* state, float decay,
                                int C, int blocks, void* out, int* status, cudaStream_t st) {
  if (B <= 0) return 0;
  if (!trlb_rglru_tc_ok(C, blocks)) return -270;
  RgTc q = {};
  CUtensorMap tw, tu;
  const int rc = rg_setup(q, tw, tu, w, u, C, blocks, B, RG_SLOTS);
  if (rc) return rc;
  q.p = {C, B, lam, gate_bias, y_bias, state, decay};
  q.seq_lens = seq_lens; q.B = B; q.y_sums = y_sums; q.y_ld = y_ld; q.out = (__nv_bfloat16*)out; q.status = status;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(rglru_step_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -274;
    attr_set = true;
  }
  return (int)trlb_host::launch_kernel(rglru_step_tc_kernel, dim3(blocks * q.tiles_per_block, (B + RG_SLOTS - 1) / RG_SLOTS), dim3(192),
                                       rg_step_smem(q.kb), st, trlb_host::pdl_enabled(), tw, tu, q);
}
