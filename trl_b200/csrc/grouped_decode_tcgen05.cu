// Decode attention of grouped-query mixers over the paged cache on the 5th-generation tensor cores (bf16).
//
// Cache: K [blocks, block_size, kv_heads, dim], V [blocks, block_size, kv_heads, vdim], both as the layer writes them.  Work
// item = (split of the pages, kv head and up to 8 of its query heads, slot).  Per 128-token tile:
//
//     S^T [128 tok, 16]   = K_tile [128 tok, dim] Q^T         both K-major straight from their TMA tiles
//     O^T [128 dims, 16]  = V_tile^T [dims, 128 tok] P^T      V read MN-major: nothing is transposed in memory
//
// Columns 0-7 are the query heads.  Probabilities keep 32-bit precision: P enters as two bf16, the value in columns 0-7 and
// its remainder in columns 8-15 of the same product (which has 16 columns anyway), and the two results are added.  A
// persistent CTA per SM: warp 0 = TMA producer over a ring of K + V tiles, warp 1 = MMA issuer (S^T double-buffered in TMEM),
// warps 2-5 = softmax (one thread per token) and output accumulation (one thread per value dimension, SLABS of 128; HEADS bounds
// the query heads of an item).  P and O^T have two buffers each: the output of a tile is collected after the probabilities of
// the next one have been handed over, so that product and softmax overlap.
// Scores may be capped (cap tanh(s / cap)); the softmax denominator may contain exp(sink[head]); the result may be multiplied by
// the sigmoid of per-element gate logits or by a factor per head.  With a window only its pages and those of the first `keep`
// tokens, which stay visible, are read: the pages of a slot are a list, kept ones first, that is cut into tiles.  Or tiles of means of
// the blocks of `pool` tokens before the window come first: the slot has its rows of them beside the pages (grouped_attn.cu).
// Splits leave fp32 partial sums that grouped_combine_kernel merges.
#include "mixers.cuh"

namespace trlb {

constexpr int GT_THREADS = 192;
constexpr int GT_MAX_STAGES = 4;
constexpr uint32_t GT_BOX = 128 * 64 * 2;  // 128 tokens x 64 dims
constexpr uint32_t GT_P_BYTES = 4096;      // 2 halves x [16 rows x 64 tok]; two such buffers

struct GroupedDecodeTc {
  const __nv_bfloat16* q;     // [B, heads, dim]
  const __nv_bfloat16* gate;  // [B, heads, vdim] logits, or null
  __nv_bfloat16* out;         // [B, heads, vdim]
  const int* seq_lens;
  const int* block_table;
  int max_blocks, block_size, B, heads, kv_heads, group, chunks, dim, vdim, nk, nv, stages, splits;
  float scale_log2;           // capped: 1
  float cap_in, cap_out;      // scale / cap (0: no cap), cap log2(e)
  float* part_o;              // [B, heads, splits, vdim]
  float2* part_ml;            // [B, heads, splits] (maximum in log2 units, sum)
  int* status;
  int window, keep;           // window 0: unlimited
  const float* sink;          // [heads] or null
  const float* head_gate;     // [B, heads] or null
  int pool, pool_rows;        // 0: no blocks; rows of means per slot
  long long out_ld;
  float out_scale;
};

__device__ __forceinline__ bool gt_vote(bool pred) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 q, %1, 0;\n\t"
      "bar.red.and.pred p, 1, 128, q;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(out)
      : "r"((uint32_t)pred)
      : "memory");
  return out != 0;
}

// What sums of weight L below a maximum m (log2 units) are multiplied by: the sink joins the denominator.
__device__ __forceinline__ float gt_factor(float m, float L, const float* sink, const float* head_gate, int h, size_t bh) {
  float f;
  if (sink != nullptr) {
    const float sk = sink[h] * 1.4426950408889634f, mt = fmaxf(m, sk), wm = fast_exp2(m - mt);
    f = wm / (L * wm + fast_exp2(sk - mt));
  } else {
    f = L > 0.f ? 1.f / L : 0.f;
  }
  return head_gate != nullptr ? f * head_gate[bh] : f;
}

struct GtItem {
  int b, kvh, h0, nh, sp, len, t0, t1;  // t0 .. t1: tiles of the slot's list of pages
  int lo, kp;                           // first page of the window, kept pages before it
  int nb, pt;                           // blocks before the window, tiles of their means (tiles 0 .. pt - 1)
  __device__ __forceinline__ int page(int i) const { return i < kp ? i : lo + i - kp; }
};

__device__ __forceinline__ GtItem gt_item(const GroupedDecodeTc& p, int item) {
  GtItem it;
  const int per = p.B * p.kv_heads * p.chunks;
  it.sp = item / per;
  const int rem = item % per, kc = rem / p.B;
  it.b = rem % p.B;
  it.kvh = kc / p.chunks;
  const int g0 = (kc % p.chunks) * 8;
  it.h0 = it.kvh * p.group + g0;
  it.nh = min(8, p.group - g0);
  const int sl = p.seq_lens[it.b];
  it.len = (sl < 0 || sl >= p.max_blocks * p.block_size) ? 0 : sl + 1;  // the new token is in the cache already
  const int bs = p.block_size;
  it.lo = p.window > 0 ? max(0, it.len - p.window) / bs : 0;
  it.kp = min((p.keep + bs - 1) / bs, it.lo);
  it.nb = p.pool > 0 ? min(max(0, it.len - p.window) / p.pool, p.pool_rows) : 0;
  it.pt = (it.nb + 127) >> 7;
  const int n_t = it.pt + (((it.kp + (it.len + bs - 1) / bs - it.lo) * bs + 127) >> 7);
  it.t0 = n_t * it.sp / p.splits;
  it.t1 = n_t * (it.sp + 1) / p.splits;
  return it;
}

// The first item with tiles from `item` on that this CTA takes (all roles skip the others alike: a role that has nothing to
// wait for in an item could otherwise overtake the rest by more than the barriers' two phases).
__device__ __forceinline__ int gt_next(const GroupedDecodeTc& p, int item, int n_items, GtItem& it) {
  for (; item < n_items; item += gridDim.x) {
    it = gt_item(p, item);
    if (it.t1 > it.t0) break;
  }
  return item;
}

// Maxima over the warp of N values a lane; lane i's result is that of value gt_slot<N>(i).  Each step halves the values a lane
// holds: N - 1 + log2(32 / N) shuffles.
template <int N>
__device__ __forceinline__ int gt_slot(int lane) {
  return N == 8 ? lane >> 2 & 7 : N == 4 ? lane >> 3 & 3 : N == 2 ? lane >> 4 & 1 : 0;
}
template <int N>
__device__ __forceinline__ float gt_warp_max(const float (&s)[N], int lane) {
  float v[N];
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = s[i];
  int o = 16;
#pragma unroll
  for (int n = N / 2; n > 0; n >>= 1, o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float mine = up ? v[i + n] : v[i], other = up ? v[i] : v[i + n];
      v[i] = fmaxf(mine, __shfl_xor_sync(0xffffffffu, other, o));
    }
  }
  for (; o > 0; o >>= 1) v[0] = fmaxf(v[0], __shfl_xor_sync(0xffffffffu, v[0], o));
  return v[0];
}

template <int SLABS, int HEADS>
__global__ void __launch_bounds__(GT_THREADS, 1)
grouped_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                         const __grid_constant__ CUtensorMap tm_pk, const __grid_constant__ CUtensorMap tm_pv, const GroupedDecodeTc p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  // a slab of O^T reads two boxes of V: the second one may exist only as space
  const uint32_t k_bytes = (uint32_t)p.nk * GT_BOX, stage_bytes = k_bytes + 2 * SLABS * GT_BOX, q_bytes = (uint32_t)p.nk * 2048;
  uint8_t* q_s = smem + (size_t)p.stages * stage_bytes;  // two buffers
  uint8_t* p_s = q_s + 2 * q_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_s + 2 * GT_P_BYTES);
  uint64_t* full_bar = bars;                        // [GT_MAX_STAGES]
  uint64_t* empty_bar = full_bar + GT_MAX_STAGES;   // [GT_MAX_STAGES]
  uint64_t* sfull_bar = empty_bar + GT_MAX_STAGES;  // [2]
  uint64_t* pfull_bar = sfull_bar + 2;              // [2]
  uint64_t* ofull_bar = pfull_bar + 2;              // [2]
  uint64_t* qfull_bar = ofull_bar + 2;              // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(qfull_bar + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* red_m = reinterpret_cast<float*>(tmem_slot + 4);  // [2][4][8]
  float* red_l = red_m + 64;                               // [4][8]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_items = p.B * p.kv_heads * p.chunks * p.splits;

  if (threadIdx.x == 0) {
    for (int s = 0; s < GT_MAX_STAGES; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&sfull_bar[s], 1);
      mbar_init(&qfull_bar[s], 128);
      mbar_init(&pfull_bar[s], 128);
      mbar_init(&ofull_bar[s], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 32 + 32 * SLABS <= 64 ? 64 : 128);  // S^T: 0, 16; O^T: 32 + 16 (SLABS buffer + slab)
    tmem_relinquish();
    tc_fence_before();
  }
  for (int i = threadIdx.x; i < (int)(2 * GT_P_BYTES / 16); i += GT_THREADS)  // rows of heads past HEADS stay zero
    reinterpret_cast<uint4*>(p_s)[i] = make_uint4(0, 0, 0, 0);
  fence_proxy_async_smem();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const int ppt = 128 / p.block_size;
  pdl_launch_dependents();
  pdl_wait();

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      int m = 0;
      bool ok = true;
      GtItem it;
      for (int item = gt_next(p, blockIdx.x, n_items, it); item < n_items && ok; item = gt_next(p, item + gridDim.x, n_items, it)) {
        const int last_page = (it.len - 1) / p.block_size;
        const int* bt = p.block_table + (size_t)it.b * p.max_blocks;
        for (int t = it.t0; t < it.t1; ++t, ++m) {
          const int stage = m % p.stages;
          if (!mbar_wait(&empty_bar[stage], (uint32_t)(((m / p.stages) & 1) ^ 1), abort_flag, p.status, 1800 + stage)) {
            ok = false;
            break;
          }
          uint8_t* st = smem + (size_t)stage * stage_bytes;
          mbar_expect_tx(&full_bar[stage], (uint32_t)(p.nk + p.nv) * GT_BOX);
          if (t < it.pt) {
            const int row = it.b * p.pool_rows + t * 128;  // rows past the slot's blocks: their scores are masked
            for (int i = 0; i < p.nk; ++i) tma_load_3d(st + i * GT_BOX, &tm_pk, &full_bar[stage], 64 * i, it.kvh, row);
            for (int i = 0; i < p.nv; ++i) tma_load_3d(st + k_bytes + i * GT_BOX, &tm_pv, &full_bar[stage], 64 * i, it.kvh, row);
            continue;
          }
          for (int g = 0; g < ppt; ++g) {
            // pages past the sequence's last one: that one again, its scores are masked
            const int row = bt[min(it.page((t - it.pt) * ppt + g), last_page)] * p.block_size;
            uint8_t* dst = st + g * p.block_size * 128;
            for (int i = 0; i < p.nk; ++i) tma_load_3d(dst + i * GT_BOX, &tm_k, &full_bar[stage], 64 * i, it.kvh, row);
            for (int i = 0; i < p.nv; ++i) tma_load_3d(dst + k_bytes + i * GT_BOX, &tm_v, &full_bar[stage], 64 * i, it.kvh, row);
          }
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(128, 16), idesc_o = umma_idesc_bf16_major(128, 16, true, false);
      const uint64_t k_d = umma_desc_kmajor_sw128(smem_u32(smem)), q_d = umma_desc_kmajor_sw128(smem_u32(q_s));
      const uint64_t v_d = umma_desc_mnmajor_sw128(smem_u32(smem) + k_bytes, GT_BOX), p_d = umma_desc_kmajor_sw128(smem_u32(p_s));
      int m = 0, j = 0;
      bool ok = true;
      auto mma1 = [&](int mm, int jj) -> bool {
        const int stage = mm % p.stages;
        if (!mbar_wait(&full_bar[stage], (uint32_t)((mm / p.stages) & 1), abort_flag, p.status, 1810 + stage)) return false;
        tc_fence_after();
        const uint32_t ts = tmem_base + (uint32_t)(mm & 1) * 16;
        for (int i = 0; i < p.nk; ++i) {
          const uint64_t da = desc_at(k_d, (uint32_t)stage * stage_bytes + (uint32_t)i * GT_BOX);
          const uint64_t db = desc_at(q_d, (uint32_t)(jj & 1) * q_bytes + (uint32_t)i * 2048);
          const int steps = min(4, (p.dim - 64 * i + 15) >> 4);
          for (int kk = 0; kk < steps; ++kk) umma_bf16_ss(ts, da + 2 * kk, db + 2 * kk, idesc_s, (i | kk) != 0);
        }
        umma_commit(&sfull_bar[mm & 1]);
        return true;
      };
      GtItem it;
      for (int item = gt_next(p, blockIdx.x, n_items, it); item < n_items && ok; item = gt_next(p, item + gridDim.x, n_items, it), ++j) {
        if (!mbar_wait(&qfull_bar[j & 1], (uint32_t)((j >> 1) & 1), abort_flag, p.status, 1820)) { ok = false; break; }
        const int n = it.t1 - it.t0;
        tc_fence_after();
        if (!mma1(m, j)) { ok = false; break; }
        for (int i = 0; i < n; ++i) {
          // with one stage the next K tile arrives only after this tile's products
          if (p.stages > 1 && i + 1 < n && !mma1(m + i + 1, j)) { ok = false; break; }
          const int mm = m + i, stage = mm % p.stages;
          if (!mbar_wait(&pfull_bar[mm & 1], (uint32_t)((mm >> 1) & 1), abort_flag, p.status, 1830)) { ok = false; break; }
          tc_fence_after();
#pragma unroll
          for (int s = 0; s < SLABS; ++s) {
            const uint64_t dv = desc_at(v_d, (uint32_t)stage * stage_bytes + (uint32_t)(2 * s) * GT_BOX);
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
              umma_bf16_ss(tmem_base + 32 + 16 * ((mm & 1) * SLABS + s), desc_at(dv, kk * 2048),
                           desc_at(p_d, (mm & 1) * GT_P_BYTES + (kk >> 2) * 2048) + 2 * (kk & 3), idesc_o, kk != 0);
          }
          umma_commit(&ofull_bar[mm & 1]);
          umma_commit(&empty_bar[stage]);
          if (p.stages == 1 && i + 1 < n && !mma1(m + i + 1, j)) { ok = false; break; }
        }
        m += n;
      }
    }
    __syncwarp();
  } else {
    // ---------------- softmax + output accumulation (128 threads) ----------------
    const int quarter = warp & 3, row = quarter * 32 + lane, ts = threadIdx.x - 64;
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    bool good = true;
    int m_cnt = 0, j = 0;

    auto write_q = [&](const GtItem& it, int buf) {
      uint8_t* dst = q_s + (size_t)buf * q_bytes;
      for (int ch = ts; ch < p.nk * 128; ch += 128) {  // 16 rows x 8 chunks of 8 dims per box
        const int box = ch >> 7, r = (ch >> 3) & 15, c8 = ch & 7, d = box * 64 + c8 * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < it.nh && d < p.dim) v = *reinterpret_cast<const uint4*>(p.q + ((size_t)it.b * p.heads + it.h0 + r) * p.dim + d);
        *reinterpret_cast<uint4*>(dst + box * 2048 + (r >> 3) * 1024 + (r & 7) * 128 + ((c8 ^ (r & 7)) << 4)) = v;
      }
      fence_proxy_async_smem();
      mbar_arrive(&qfull_bar[buf]);
    };

    if (p.splits == 1) {  // idle slots: their rows are read as operands later
      for (int item = blockIdx.x; item < n_items; item += gridDim.x) {
        const GtItem it = gt_item(p, item);
        if (it.t1 > it.t0) continue;
        for (int i = ts; i < it.nh * p.vdim; i += 128) p.out[(size_t)it.b * p.out_ld + (size_t)it.h0 * p.vdim + i] = __float2bfloat16(0.f);
      }
    } else {
      for (int item = blockIdx.x; item < n_items; item += gridDim.x) {
        const GtItem it = gt_item(p, item);
        if (it.t1 > it.t0 || ts >= it.nh) continue;
        p.part_ml[((size_t)it.b * p.heads + it.h0 + ts) * p.splits + it.sp] = make_float2(-INFINITY, 0.f);
      }
    }
    GtItem it, nxt;
    int item = gt_next(p, blockIdx.x, n_items, it);
    if (item < n_items) write_q(it, 0);
    for (int next; item < n_items && good; item = next, it = nxt, ++j) {
      next = gt_next(p, item + gridDim.x, n_items, nxt);
      if (next < n_items) write_q(nxt, (j + 1) & 1);
      float mrun[HEADS], lsum[HEADS], alpha[HEADS], acc[SLABS][HEADS];
#pragma unroll
      for (int g = 0; g < HEADS; ++g) {
        mrun[g] = -INFINITY;
        lsum[g] = 0.f;
        alpha[g] = 0.f;
#pragma unroll
        for (int s = 0; s < SLABS; ++s) acc[s][g] = 0.f;
      }
      // the output of tile m, whose probabilities were formed when alpha was what it is
      auto collect = [&](int m) -> bool {
        if (!__all_sync(0xffffffffu, mbar_wait(&ofull_bar[m & 1], (uint32_t)((m >> 1) & 1), abort_flag, p.status, 1850))) return false;
        tc_fence_after();
#pragma unroll
        for (int sl = 0; sl < SLABS; ++sl) {
          float o[16];
          tmem_ld_32x16(tmem_base + lane_off + 32 + 16 * ((m & 1) * SLABS + sl), o);
          tmem_ld_wait();
#pragma unroll
          for (int g = 0; g < HEADS; ++g) acc[sl][g] = fmaf(acc[sl][g], alpha[g], o[g] + o[8 + g]);
        }
        tc_fence_before();
        return true;
      };
      for (int t = it.t0; t < it.t1; ++t, ++m_cnt) {
        float s[HEADS];
        float* rm = red_m + (m_cnt & 1) * 32;
        good = good && __all_sync(0xffffffffu, mbar_wait(&sfull_bar[m_cnt & 1], (uint32_t)((m_cnt >> 1) & 1), abort_flag, p.status, 1840));
        if (good) {
          float all[8];
          tc_fence_after();
          tmem_ld_32x8(tmem_base + lane_off + (uint32_t)(m_cnt & 1) * 16, all);
          tmem_ld_wait();
#pragma unroll
          for (int g = 0; g < HEADS; ++g) s[g] = all[g];
          if (p.cap_in > 0.f) {
            float top = 0.f;
#pragma unroll
            for (int g = 0; g < HEADS; ++g) {
              s[g] *= p.cap_in;
              top = fmaxf(top, fabsf(s[g]));
            }
            const bool far = __any_sync(0xffffffffu, top > CAP_SERIES);
#pragma unroll
            for (int g = 0; g < HEADS; ++g) s[g] = p.cap_out * (far ? tanh_exp(s[g]) : tanh_series(s[g]));
          }
          const int tok = it.page((t - it.pt) * ppt + row / p.block_size) * p.block_size + row % p.block_size;
          const bool valid = t < it.pt ? t * 128 + row < it.nb : tok < it.len && (p.window == 0 || tok >= it.len - p.window || tok < p.keep);
#pragma unroll
          for (int g = 0; g < HEADS; ++g) s[g] = valid ? s[g] * p.scale_log2 : -INFINITY;
          const float wm = gt_warp_max<HEADS>(s, lane);
          if ((lane & (32 / HEADS - 1)) == 0) rm[quarter * 8 + gt_slot<HEADS>(lane)] = wm;
        }
        good = gt_vote(good);
        if (!good) break;
        float next[HEADS];
        uint8_t* prow = p_s + (m_cnt & 1) * GT_P_BYTES + (row >> 6) * 2048;  // the [16 x 64 tok] half of this token
        const int c = row & 63;
#pragma unroll
        for (int g = 0; g < HEADS; ++g) {
          const float mn = fmaxf(mrun[g], fmaxf(fmaxf(rm[g], rm[8 + g]), fmaxf(rm[16 + g], rm[24 + g])));
          next[g] = (mrun[g] == -INFINITY) ? 0.f : fast_exp2(mrun[g] - mn);
          const float pv = (s[g] == -INFINITY || g >= it.nh) ? 0.f : fast_exp2(s[g] - mn);
          mrun[g] = mn;
          lsum[g] = lsum[g] * next[g] + pv;
          const __nv_bfloat16 hi = __float2bfloat16(pv);
          uint8_t* at = prow + g * 128 + ((((c >> 3) ^ g) & 7) << 4) + (c & 7) * 2;
          *reinterpret_cast<__nv_bfloat16*>(at) = hi;
          *reinterpret_cast<__nv_bfloat16*>(at + 1024) = __float2bfloat16(pv - __bfloat162float(hi));  // row 8 + g
        }
        fence_proxy_async_smem();
        tc_fence_before();
        mbar_arrive(&pfull_bar[m_cnt & 1]);
        if (t > it.t0) good = collect(m_cnt - 1);
#pragma unroll
        for (int g = 0; g < HEADS; ++g) alpha[g] = next[g];
      }
      if (good) good = collect(m_cnt - 1);
#pragma unroll
      for (int g = 0; g < HEADS; ++g) {
        const float ws = warp_sum(lsum[g]);
        if (lane == 0) red_l[quarter * 8 + g] = ws;
      }
      good = gt_vote(good);  // every softmax thread gets here, also after a failed wait: the vote keeps them together
      if (!good) break;
#pragma unroll
      for (int g = 0; g < HEADS; ++g) {
        if (g >= it.nh) break;
        const size_t bh = (size_t)it.b * p.heads + it.h0 + g;
        const float L = red_l[g] + red_l[8 + g] + red_l[16 + g] + red_l[24 + g];
        const float f = p.splits == 1 ? gt_factor(mrun[g], L, p.sink, p.head_gate, it.h0 + g, bh) : 0.f;
#pragma unroll
        for (int sl = 0; sl < SLABS; ++sl) {
          const int d = sl * 128 + row;
          if (d >= p.vdim) continue;
          if (p.splits == 1) {
            float o = acc[sl][g] * f * p.out_scale;
            if (p.gate != nullptr) o *= fast_sigmoid(__bfloat162float(p.gate[bh * p.vdim + d]));
            p.out[(size_t)it.b * p.out_ld + (size_t)(it.h0 + g) * p.vdim + d] = __float2bfloat16(o);
          } else {
            p.part_o[(bh * p.splits + it.sp) * p.vdim + d] = acc[sl][g];
          }
        }
        if (p.splits > 1 && ts == g) p.part_ml[bh * p.splits + it.sp] = make_float2(mrun[g], L);
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
    tmem_dealloc(tmem_base, 32 + 32 * SLABS <= 64 ? 64 : 128);
  }
}

// One block per (head, slot).
__global__ void __launch_bounds__(128)
grouped_combine_kernel(const float* __restrict__ part_o, const float2* __restrict__ part_ml, const __nv_bfloat16* __restrict__ gate,
                       const int* __restrict__ seq_lens, const float* __restrict__ sink, const float* __restrict__ head_gate, int heads,
                       int vdim, int splits, long long out_ld, float out_scale, __nv_bfloat16* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  if (seq_lens[b] < 0) return;
  const size_t bh = (size_t)b * heads + h;
  float m = -INFINITY, den = 0.f;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, part_ml[bh * splits + s].x);
  for (int s = 0; s < splits; ++s) {
    const float2 ml = part_ml[bh * splits + s];
    if (ml.y > 0.f) den += ml.y * fast_exp2(ml.x - m);
  }
  const float f = gt_factor(m, den, sink, head_gate, h, bh) * out_scale;
  for (int d = threadIdx.x; d < vdim; d += 128) {
    float o = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float2 ml = part_ml[bh * splits + s];
      if (ml.y > 0.f) o = fmaf(part_o[(bh * splits + s) * vdim + d], fast_exp2(ml.x - m), o);
    }
    o *= f;
    if (gate != nullptr) o *= fast_sigmoid(__bfloat162float(gate[bh * vdim + d]));
    out[(size_t)b * out_ld + (size_t)h * vdim + d] = __float2bfloat16(o);
  }
}

}  // namespace trlb

using namespace trlb;

namespace {

size_t gt_smem(int nk, int slabs, int stages) {
  return (size_t)stages * (nk + 2 * slabs) * GT_BOX + 2 * (size_t)nk * 2048 + 2 * GT_P_BYTES + 1024 + 1024;
}
int gt_stages(int nk, int slabs) {
  for (int s = GT_MAX_STAGES; s > 0; --s)
    if (gt_smem(nk, slabs, s) <= 227 * 1024) return s;
  return 0;
}

}  // namespace

// 1 when trlb_grouped_decode_tc takes these sizes.
TRLB_API int trlb_grouped_decode_tc_ok(int heads, int kv_heads, int dim, int vdim, int block_size) {
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || dim % 8 || vdim % 8 || vdim > 256) return 0;
  if (block_size < 8 || block_size > 128 || 128 % block_size) return 0;
  return gt_stages((dim + 63) / 64, (vdim + 127) / 128) > 0;
}

// Work items of one split (splits are chosen so that every SM gets one).
TRLB_API int trlb_grouped_decode_tc_items(int B, int heads, int kv_heads) { return B * kv_heads * ((heads / kv_heads + 7) / 8); }

// q [B, heads, dim], caches [num_blocks, block_size, kv_heads, dim / vdim], gate logits [B, heads, vdim] or null; one new token per
// slot, in the cache already.  window <= 0: unlimited, else the first `keep` tokens stay visible; cap <= 0: none; sink [heads] and
// head_gate [B, heads] may be null.  pool > 0 (with a window): means pool_k, pool_v [pool_slots, pool_rows, kv_heads, dim / vdim].  out [B
// rows of out_ld], times out_scale.  splits > 1: part_o [B, heads, splits, vdim], part_ml [B, heads, splits, 2] fp32.
TRLB_API int trlb_grouped_decode_tc(const void* q, const void* k_cache, const void* v_cache, const void* gate, void* out,
                                    int num_blocks, int B, int heads, int kv_heads, int dim, int vdim, int window, int keep,
                                    float scale, float cap, const float* sink, const float* head_gate, const int* seq_lens, const int* block_table, int max_blocks, int block_size, int splits,
                                    float* part_o, float* part_ml, int pool, int pool_rows, int pool_slots, const void* pool_k,
                                    const void* pool_v, long long out_ld, float out_scale, int* status, cudaStream_t st) {
  if (B <= 0) return 0;
  if (pool > 0 && (pool_k == nullptr || pool_v == nullptr || pool_rows <= 0 || pool_slots < B || keep > 0)) return -280;
  if (!(scale > 0.f) || splits < 1 || !trlb_grouped_decode_tc_ok(heads, kv_heads, dim, vdim, block_size)) return -280;
  if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return -280;
  GroupedDecodeTc p = {};
  p.q = (const __nv_bfloat16*)q; p.gate = (const __nv_bfloat16*)gate; p.out = (__nv_bfloat16*)out;
  p.seq_lens = seq_lens; p.block_table = block_table; p.max_blocks = max_blocks; p.block_size = block_size;
  p.B = B; p.heads = heads; p.kv_heads = kv_heads; p.group = heads / kv_heads; p.chunks = (p.group + 7) / 8;
  p.dim = dim; p.vdim = vdim; p.nk = (dim + 63) / 64; p.nv = (vdim + 63) / 64; p.splits = splits;
  const int slabs = (vdim + 127) / 128;
  p.stages = gt_stages(p.nk, slabs);
  p.scale_log2 = cap > 0.f ? 1.f : scale * 1.4426950408889634f;
  p.cap_in = cap > 0.f ? scale / cap : 0.f;
  p.cap_out = cap * 1.4426950408889634f;
  p.window = window > 0 ? window : 0; p.keep = window > 0 && keep > 0 ? keep : 0; p.sink = sink; p.head_gate = head_gate;
  p.part_o = part_o; p.part_ml = (float2*)part_ml; p.status = status;
  p.pool = window > 0 && pool > 0 ? pool : 0; p.pool_rows = pool_rows; p.out_ld = out_ld; p.out_scale = out_scale;
  CUtensorMap tk, tv, tpk, tpv;
  using trlb_host::make_tmap_3d_bf16;
  const uint64_t rows = (uint64_t)num_blocks * block_size;
  if (make_tmap_3d_bf16(&tk, k_cache, dim, kv_heads, rows, dim, (uint64_t)kv_heads * dim, 64, 1, block_size)) return -281;
  if (make_tmap_3d_bf16(&tv, v_cache, vdim, kv_heads, rows, vdim, (uint64_t)kv_heads * vdim, 64, 1, block_size)) return -282;
  tpk = tk;
  tpv = tv;
  if (p.pool > 0) {
    const uint64_t means = (uint64_t)pool_slots * pool_rows;
    if (make_tmap_3d_bf16(&tpk, pool_k, dim, kv_heads, means, dim, (uint64_t)kv_heads * dim, 64, 1, 128)) return -284;
    if (make_tmap_3d_bf16(&tpv, pool_v, vdim, kv_heads, means, vdim, (uint64_t)kv_heads * vdim, 64, 1, 128)) return -285;
  }
  using Kern = void (*)(const CUtensorMap, const CUtensorMap, const CUtensorMap, const CUtensorMap, const GroupedDecodeTc);
  static const Kern kerns[2][4] = {{grouped_decode_tc_kernel<1, 1>, grouped_decode_tc_kernel<1, 2>, grouped_decode_tc_kernel<1, 4>, grouped_decode_tc_kernel<1, 8>},
                                   {grouped_decode_tc_kernel<2, 1>, grouped_decode_tc_kernel<2, 2>, grouped_decode_tc_kernel<2, 4>, grouped_decode_tc_kernel<2, 8>}};
  static bool attr_set = false;
  if (!attr_set) {
    for (int i = 0; i < 8; ++i)
      if (cudaFuncSetAttribute(kerns[i >> 2][i & 3], cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -283;
    attr_set = true;
  }
  const int items = trlb_grouped_decode_tc_items(B, heads, kv_heads) * splits;
  const dim3 grid(items < trlb_host::sm_count() ? items : trlb_host::sm_count()), blk(GT_THREADS);
  const size_t smem = gt_smem(p.nk, slabs, p.stages);
  const bool pdl = trlb_host::pdl_enabled();
  const Kern kern = kerns[slabs - 1][p.group > 4 ? 3 : p.group > 2 ? 2 : p.group > 1 ? 1 : 0];
  const int rc = (int)trlb_host::launch_kernel(kern, grid, blk, smem, st, pdl, tk, tv, tpk, tpv, p);
  if (rc || splits == 1) return rc;
  return (int)trlb_host::launch_kernel(grouped_combine_kernel, dim3(heads, B), dim3(128), 0, st, pdl, (const float*)part_o,
                                       (const float2*)part_ml, p.gate, seq_lens, sink, head_gate, heads, vdim, splits, out_ld, out_scale, p.out);
}
