// Decode attention of the latent-attention mixer on the 5th-generation tensor cores (bf16 cache, paged).
//
// In absorbed form all heads of a slot attend to ONE row per token, [latent | rotated key], which is also the value (its
// latent part).  The operands are swapped so that the tokens and the latent dimensions fill the 128 rows of an MMA and
// the heads (32 per CTA) are its columns:
//
//     S^T [128 tokens x heads]      = C [tokens x row]  Q^T            both K-major, straight from their TMA tiles
//     O^T [128 dims x heads] (+)=     C^T [dims x tokens] P^T          the same tile of C read MN-major
//
// so a cached row crosses HBM once, serves both products from shared memory, and no row of the tensor core is padding
// when there are few heads.  One CTA per (slot, head group, split of the visible pages), 192 threads: TMA warp, MMA warp,
// and one softmax thread per token of the 128-token tile.  Per-head maxima are formed with a shuffle reduce-scatter and
// exchanged between the four warps; the reference maximum of a head moves (and O^T is rescaled) only when it is exceeded
// by 2^8.  Probabilities keep 32-bit precision: they go to shared memory as two bf16 (value and remainder) that are
// separate columns of the second product, so the tile of C is read once for both.  A tile's 64-column boxes are released slab by slab as O^T consumes them, so the next tile streams
// in behind it.  Splits leave fp32 partial sums; latent_combine_kernel merges them with the softmax sink.
#include "mixers.cuh"

namespace trlb {

constexpr int LD_TOK = 128;
constexpr uint32_t LD_BOX = LD_TOK * 64 * 2;
constexpr int LD_MAX_BOX = 12;

struct LatentDecodeTc {
  int heads, kv_rank, boxes, slabs, lat_w, window, max_blocks, block_size, splits;
  float scale_log2;
  const int* seq_lens;
  const int* block_table;
  float* part_o;   // [B, heads, splits, kv_rank]
  float2* part_ml; // [B, heads, splits] (reference maximum in log2 units, sum)
  int* status;
};

// x[i] over 32 lanes -> lane l holds OP over all lanes of x[l]
template <bool MAX>
__device__ __forceinline__ float reduce_scatter32(float (&x)[32], int lane) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const bool up = (lane & o) != 0;
      const float keep = up ? x[i + o] : x[i], send = up ? x[i] : x[i + o];
      const float got = __shfl_xor_sync(0xffffffffu, send, o);
      x[i] = MAX ? fmaxf(keep, got) : keep + got;
    }
  }
  return x[0];
}

__global__ void __launch_bounds__(192, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_c,
                        const LatentDecodeTc p) {
  constexpr int HG = 32;  // heads per CTA
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* c_s = smem;                                            // [boxes] 128 tokens x 64 columns
  uint8_t* q_s = c_s + (size_t)p.boxes * LD_BOX;                  // [boxes] HG heads x 64 columns
  uint8_t* p_s = q_s + (size_t)p.boxes * HG * 128;                // 128 tokens x (32 values | 32 remainders)
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_s + LD_BOX);
  uint64_t* full = bars;                   // [LD_MAX_BOX]
  uint64_t* empty = full + LD_MAX_BOX;     // [LD_MAX_BOX]
  uint64_t* q_full = empty + LD_MAX_BOX;
  uint64_t* s_full = q_full + 1;
  uint64_t* p_full = s_full + 1;
  uint64_t* o_full = p_full + 1;
  uint64_t* red_full = o_full + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(red_full + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* red = reinterpret_cast<float*>(bars + 40);  // [2][4][HG]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h0 = (int)blockIdx.x * HG, split = blockIdx.y;

  if (threadIdx.x == 0) {
    for (int s = 0; s < LD_MAX_BOX; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(q_full, 1);
    mbar_init(s_full, 1);
    mbar_init(p_full, 128);
    mbar_init(o_full, 1);
    mbar_init(red_full, 128);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_c);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  pdl_wait();

  const int pos = p.seq_lens[b];
  const bool live = pos >= 0 && pos < p.max_blocks * p.block_size;
  const int first = (live && p.window > 0) ? max(0, pos - p.window + 1) : 0;
  const int page0 = first / p.block_size, ppt = LD_TOK / p.block_size;
  const int tiles = live ? (pos / p.block_size - page0) / ppt + 1 : 0;
  const int t_beg = tiles * split / p.splits, n_t = tiles * (split + 1) / p.splits - t_beg;

  if (warp == 0) {
    if (lane == 0 && n_t > 0) {
      const int* bt = p.block_table + (size_t)b * p.max_blocks;
      mbar_expect_tx(q_full, (uint32_t)(p.boxes * HG * 128));
      for (int i = 0; i < p.boxes; ++i) tma_load_3d(q_s + (size_t)i * HG * 128, &tm_q, q_full, 64 * i, h0, b);
      bool ok = true;
      for (int j = 0; j < n_t && ok; ++j) {
        // first cache row of page g of the tile (pages past the sequence's last one are masked: any page will do)
        auto row_of = [&](int g) { return bt[min(page0 + (t_beg + j) * ppt + g, pos / p.block_size)] * p.block_size; };
        const int row0 = row_of(0), row1 = row_of(ppt > 1 ? 1 : 0);
        for (int i = 0; i < p.boxes; ++i) {
          if (!mbar_wait(&empty[i], (uint32_t)((j & 1) ^ 1), abort_flag, p.status, 1500 + i)) { ok = false; break; }
          mbar_expect_tx(&full[i], LD_BOX);
          uint8_t* dst = c_s + (size_t)i * LD_BOX;
          tma_load_2d(dst, &tm_c, &full[i], 64 * i, row0);
          if (ppt > 1) tma_load_2d(dst + p.block_size * 128, &tm_c, &full[i], 64 * i, row1);
          for (int g = 2; g < ppt; ++g)  // pages shorter than 64 tokens
            tma_load_2d(dst + g * p.block_size * 128, &tm_c, &full[i], 64 * i, row_of(g));
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0 && n_t > 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16_major(128, HG, false, false);
      constexpr uint32_t idesc_o = umma_idesc_bf16_major(128, 2 * HG, true, true);
      const uint64_t c_k = umma_desc_kmajor_sw128(smem_u32(c_s)), q_k = umma_desc_kmajor_sw128(smem_u32(q_s));
      const uint64_t c_mn = umma_desc_mnmajor_sw128(smem_u32(c_s), LD_BOX), p_mn = umma_desc_mnmajor_sw128(smem_u32(p_s), LD_BOX);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status, 1520);
      for (int j = 0; j < n_t && ok; ++j) {
        uint64_t da = c_k, db = q_k;
        for (int i = 0; i < p.boxes && ok; ++i) {
          ok = mbar_wait(&full[i], (uint32_t)(j & 1), abort_flag, p.status, 1530 + i);
          if (!ok) break;
          tc_fence_after();
          const int steps = min(4, (p.lat_w - 64 * i + 15) >> 4);  // none for a box that only completes a slab
          // each step has an accumulator of its own (with so few columns the latency of one would show)
          if (steps == 4) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) umma_bf16_ss(tmem_base + kk * HG, da + 2 * kk, db + 2 * kk, idesc_s, i);
          } else {
            for (int kk = 0; kk < steps; ++kk) umma_bf16_ss(tmem_base + kk * HG, da + 2 * kk, db + 2 * kk, idesc_s, i);
          }
          da += LD_BOX >> 4;
          db += (HG * 128) >> 4;
          if (i >= 2 * p.slabs) umma_commit(&empty[i]);
        }
        if (!ok) break;
        umma_commit(s_full);
        if (!mbar_wait(p_full, (uint32_t)(j & 1), abort_flag, p.status, 1550)) break;
        tc_fence_after();
        for (int s = 0; s < p.slabs; ++s) {
          const uint64_t ds = desc_at(c_mn, (uint32_t)(2 * s) * LD_BOX);
#pragma unroll
          for (int kk = 0; kk < LD_TOK / 16; ++kk)
            umma_bf16_ss(tmem_base + 4 * HG + (uint32_t)(s * 2 * HG), desc_at(ds, kk * 2048), desc_at(p_mn, kk * 2048), idesc_o, (j | kk) != 0);
          umma_commit(&empty[2 * s]);
          umma_commit(&empty[2 * s + 1]);
        }
        umma_commit(o_full);
      }
    }
    __syncwarp();
  } else if (n_t > 0) {
    const int w4 = warp & 3, r = w4 * 32 + lane;
    const uint32_t ts = tmem_base + ((uint32_t)(w4 * 32) << 16), to = ts + 4 * HG;
    float m_ref = -INFINITY, l[HG];  // the reference maximum of head `lane`; per-head sums over this thread's tokens
#pragma unroll
    for (int i = 0; i < HG; ++i) l[i] = 0.f;
    bool ok = true;
    for (int j = 0; j < n_t && ok; ++j) {
      const int tok = (page0 + (t_beg + j) * ppt) * p.block_size + r;
      const bool seen = tok >= first && tok <= pos;
      // a complete S^T(j) also means that the products of the tile before it are done (same issuing thread)
      ok = __all_sync(0xffffffffu, mbar_wait(s_full, (uint32_t)(j & 1), abort_flag, p.status, 1560));
      if (!ok) break;
      tc_fence_after();
      float v[32], x[32];
      tmem_ld_32x32(ts, v);
      tmem_ld_wait();
      const int parts = min(4, (p.lat_w + 15) >> 4);  // partial sums of S^T that hold something
      for (int c = 1; c < parts; ++c) {
        tmem_ld_32x32(ts + (uint32_t)(c * HG), x);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) v[i] += x[i];
      }
#pragma unroll
      for (int i = 0; i < 32; ++i) x[i] = v[i] = seen ? v[i] * p.scale_log2 : -INFINITY;
      float* mine = red + (j & 1) * 4 * HG;
      mine[w4 * HG + lane] = reduce_scatter32<true>(x, lane);
      mbar_arrive(red_full);
      ok = __all_sync(0xffffffffu, mbar_wait(red_full, (uint32_t)(j & 1), abort_flag, p.status, 1570));
      if (!ok) break;
      const float mt = fmaxf(fmaxf(mine[lane], mine[HG + lane]), fmaxf(mine[2 * HG + lane], mine[3 * HG + lane]));
      float alpha = 1.f;
      bool moved = false;
      if (m_ref == -INFINITY) {
        m_ref = mt;
      } else if (mt > m_ref + 8.f) {
        alpha = exp2f(m_ref - mt);
        m_ref = mt;
        moved = true;
      }
      const float neg_m = m_ref == -INFINITY ? 0.f : -m_ref;
      if (__any_sync(0xffffffffu, moved)) {  // the same in all four warps
#pragma unroll
        for (int i = 0; i < HG; ++i) l[i] *= __shfl_sync(0xffffffffu, alpha, i);
        if (j > 0) {
#pragma unroll 1
          for (int y = 0; y < p.slabs * 2 * HG; y += 16) {
            float o[16];
            tmem_ld_32x16(to + (uint32_t)y, o);
            tmem_ld_wait();
            uint32_t w[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) w[i] = __float_as_uint(o[i] * __shfl_sync(0xffffffffu, alpha, (y & 31) + i));
            tmem_st_32x16(to + (uint32_t)y, w);
          }
          tmem_st_wait();
        }
      }
      // token r's weights: one 128-byte row of the P tile
#pragma unroll
      for (int c8 = 0; c8 < HG / 8; ++c8) {
        uint32_t a[4], bb[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int i = c8 * 8 + 2 * q;
          const float p0 = exp2f(v[i] + __shfl_sync(0xffffffffu, neg_m, i));
          const float p1 = exp2f(v[i + 1] + __shfl_sync(0xffffffffu, neg_m, i + 1));
          l[i] += p0;
          l[i + 1] += p1;
          a[q] = pack_bf16(p0, p1);
          const float2 back = unpack_bf16(a[q]);
          bb[q] = pack_bf16(p0 - back.x, p1 - back.y);
        }
        uint8_t* row = p_s + (size_t)r * 128;
        *reinterpret_cast<uint4*>(row + ((c8 ^ (r & 7)) << 4)) = make_uint4(a[0], a[1], a[2], a[3]);
        *reinterpret_cast<uint4*>(row + (((c8 + 4) ^ (r & 7)) << 4)) = make_uint4(bb[0], bb[1], bb[2], bb[3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(p_full);
    }
    if (ok) {
      // sums over the tokens; then O^T
      float* mine = red + (n_t & 1) * 4 * HG;
      mine[w4 * HG + lane] = reduce_scatter32<false>(l, lane);
      mbar_arrive(red_full);
      ok = __all_sync(0xffffffffu, mbar_wait(red_full, (uint32_t)(n_t & 1), abort_flag, p.status, 1580));
      if (ok) ok = __all_sync(0xffffffffu, mbar_wait(o_full, (uint32_t)((n_t - 1) & 1), abort_flag, p.status, 1590));
      if (ok) {
        tc_fence_after();
        const size_t bh0 = (size_t)b * p.heads + h0;
        if (w4 == 0 && h0 + lane < p.heads)
          p.part_ml[(bh0 + lane) * p.splits + split] =
              make_float2(m_ref, mine[lane] + mine[HG + lane] + mine[2 * HG + lane] + mine[3 * HG + lane]);
        const int nh = min(HG, p.heads - h0);
        for (int s = 0; s < p.slabs; ++s) {
          const int d = s * 128 + r;
          float o[32], e[32];
          tmem_ld_32x32(to + (uint32_t)(s * 2 * HG), o);
          tmem_ld_32x32(to + (uint32_t)(s * 2 * HG + HG), e);
          tmem_ld_wait();
          if (d < p.kv_rank) {
            float* dst = p.part_o + (bh0 * p.splits + split) * p.kv_rank + d;
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (i < nh) dst[(size_t)i * p.splits * p.kv_rank] = o[i] + e[i];
          }
        }
        tc_fence_before();
      }
    }
  } else if (live && threadIdx.x - 64 < HG) {
    const int h = h0 + (int)threadIdx.x - 64;
    if (h < p.heads) p.part_ml[((size_t)b * p.heads + h) * p.splits + split] = make_float2(-INFINITY, 0.f);
  }
  __syncthreads();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

// o_lat[b, h] = (sum over splits) / (sum of exponentials + exp(sink), no such term when sink is null).  One block per (head, slot).
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float2* __restrict__ part_ml, const float* __restrict__ sink,
                      const int* __restrict__ seq_lens, int heads, int kv_rank, int splits, __nv_bfloat16* __restrict__ o_lat) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  if (seq_lens[b] < 0) return;
  const size_t bh = (size_t)b * heads + h;
  const float sk = sink != nullptr ? sink[h] * 1.4426950408889634f : -INFINITY;
  float m = sk;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, part_ml[bh * splits + s].x);
  float den = exp2f(sk - m);
  for (int s = 0; s < splits; ++s) {
    const float2 ml = part_ml[bh * splits + s];
    den += ml.y * exp2f(ml.x - m);
  }
  const float inv = 1.f / den;
  for (int d = threadIdx.x * 4; d < kv_rank; d += 512) {  // kv_rank is a multiple of 8
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < splits; ++s) {
      const float2 ml = part_ml[bh * splits + s];
      if (ml.y > 0.f) {
        const float w = exp2f(ml.x - m) * inv;
        const float4 x = *reinterpret_cast<const float4*>(part_o + (bh * splits + s) * kv_rank + d);
        v.x = fmaf(x.x, w, v.x); v.y = fmaf(x.y, w, v.y); v.z = fmaf(x.z, w, v.z); v.w = fmaf(x.w, w, v.w);
      }
    }
    *reinterpret_cast<uint2*>(o_lat + bh * kv_rank + d) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
  }
}

// Query of a decode step: fp32 sums -> bf16 [B, heads, dim + rot] (only the unrotated part is used further) and the
// rotated part in its place in the latent-row layout.  The sums are cleared.
__global__ void __launch_bounds__(128)
latent_query_kernel(float* __restrict__ qacc, long long ld, __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ q_lat,
                    int heads, int dim, int rot, int kr_off, int lat_w, const int* __restrict__ positions,
                    const float2* __restrict__ table, int table_len) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  float* src = qacc + (size_t)b * ld + (size_t)h * (dim + rot);
  const size_t bh = (size_t)b * heads + h;
  const int pos = positions[b];
  for (int d = threadIdx.x; d < dim; d += 128) {
    q[bh * (dim + rot) + d] = __float2bfloat16(src[d]);
    src[d] = 0.f;
  }
  for (int i = threadIdx.x; i < rot / 2; i += 128) {
    const float u = __bfloat162float(__float2bfloat16(src[dim + 2 * i])), v = __bfloat162float(__float2bfloat16(src[dim + 2 * i + 1]));
    src[dim + 2 * i] = 0.f;
    src[dim + 2 * i + 1] = 0.f;
    if (pos < 0 || pos >= table_len) continue;
    const float2 cs = table[(size_t)pos * (rot / 2) + i];
    __nv_bfloat16* dst = q_lat + bh * lat_w + kr_off + 2 * i;
    dst[0] = __float2bfloat16(u * cs.x - v * cs.y);
    dst[1] = __float2bfloat16(v * cs.x + u * cs.y);
  }
}

// ------------------------------------------------------------------------------------------------------------
// Per-head product of a decode batch:  Y[b, h, m] = scale[b, h] * sum_k X[b, h, k] W_h[m, k]
// W_h is [M, K] with K contiguous, or (W_MN) [K, M] with M contiguous.  One CTA per (head, 128 rows of W_h, 128 slots): the
// weights are the M operand, the slots the columns.  Weight tiles are requested before the wait on the previous kernel.
constexpr int HG_STAGES = 4;
struct HeadGemm {
  int B, M, K, n_cols;
  long long y_b, y_h;    // strides of Y in elements
  const float* scale;    // [B, heads] or null
  int heads;
  __nv_bfloat16* Y;
  int* status;
};

template <bool W_MN>
__global__ void __launch_bounds__(192)
head_gemm_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const HeadGemm p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t x_bytes = (uint32_t)p.n_cols * 128, stage = LD_BOX + x_bytes;
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + (size_t)HG_STAGES * stage);
  uint64_t* empty = full + HG_STAGES;
  uint64_t* done = empty + HG_STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, m0 = (int)blockIdx.y * 128, b0 = (int)blockIdx.z * 128;
  const int kb = (p.K + 63) / 64;
  if (threadIdx.x == 0) {
    for (int s = 0; s < HG_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(done, 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_x);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 128);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  if (warp == 0) {
    if (lane == 0) {
      auto load_w = [&](int k) {
        uint8_t* st = smem + (size_t)(k % HG_STAGES) * stage;
        uint64_t* bar = &full[k % HG_STAGES];
        mbar_expect_tx(bar, stage);
        if (W_MN) {  // 64 rows of K, two boxes of 64 columns of M
          tma_load_3d(st, &tm_w, bar, m0, 64 * k, h);
          tma_load_3d(st + 8192, &tm_w, bar, m0 + 64, 64 * k, h);
        } else {
          tma_load_3d(st, &tm_w, bar, 64 * k, m0, h);
        }
      };
      const int ahead = min(kb, HG_STAGES);
      for (int k = 0; k < ahead; ++k) load_w(k);
      pdl_wait();
      for (int k = 0; k < kb; ++k) {
        const int s = k % HG_STAGES;
        if (k >= ahead) {
          if (!mbar_wait(&empty[s], (uint32_t)(((k / HG_STAGES) & 1) ^ 1), abort_flag, p.status, 1600 + s)) break;
          load_w(k);
        }
        tma_load_3d(smem + (size_t)s * stage + LD_BOX, &tm_x, &full[s], 64 * k, h, b0);
      }
    } else {
      pdl_wait();
    }
    __syncwarp();
  } else if (warp == 1) {
    pdl_wait();
    if (lane == 0) {
      const uint32_t idesc = umma_idesc_bf16_major(128, p.n_cols, W_MN, false);
      for (int k = 0; k < kb; ++k) {
        const int s = k % HG_STAGES;
        if (!mbar_wait(&full[s], (uint32_t)((k / HG_STAGES) & 1), abort_flag, p.status, 1610 + s)) break;
        tc_fence_after();
        const uint32_t st = smem_u32(smem + (size_t)s * stage);
        const int steps = min(4, (p.K - 64 * k + 15) >> 4);
        for (int kk = 0; kk < steps; ++kk) {
          const uint64_t da = W_MN ? umma_desc_mnmajor_sw128(st + (uint32_t)kk * 2048, 8192) : umma_desc_kmajor_sw128(st) + 2 * kk;
          umma_bf16_ss(tmem_base, da, umma_desc_kmajor_sw128(st + LD_BOX) + 2 * kk, idesc, (k | kk) != 0);
        }
        umma_commit(&empty[s]);
      }
      umma_commit(done);
    }
    __syncwarp();
  } else {
    pdl_wait();
    const int r = (warp & 3) * 32 + lane, m = m0 + r;
    float sc[4];  // the scale of slot b0 + 32 i + lane
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int b = b0 + 32 * i + lane;
      sc[i] = (p.scale != nullptr && b < p.B) ? p.scale[(size_t)b * p.heads + h] : 1.f;
    }
    if (__all_sync(0xffffffffu, mbar_wait(done, 0, abort_flag, p.status, 1620))) {
      tc_fence_after();
#pragma unroll
      for (int x = 0; x < 128; x += 16) {
        if (x < p.n_cols) {
          float o[16];
          tmem_ld_32x16(tmem_base + ((uint32_t)((warp & 3) * 32) << 16) + x, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const float y = o[i] * __shfl_sync(0xffffffffu, sc[x / 32], (x & 31) + i);
            const int b = b0 + x + i;
            if (m < p.M && b < p.B) p.Y[b * p.y_b + h * p.y_h + m] = __float2bfloat16(y);
          }
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
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 128);
  }
}

}  // namespace trlb

using namespace trlb;

namespace {

int ld_slabs(int kv_rank) { return (kv_rank + 127) / 128; }
int ld_boxes(int kv_rank, int lat_w) { return max((lat_w + 63) / 64, 2 * ld_slabs(kv_rank)); }
size_t ld_smem(int boxes) { return (size_t)boxes * (LD_BOX + 32 * 128) + LD_BOX + 1024 + 320 + 2 * 4 * 32 * 4; }

}  // namespace

// 1 when trlb_latent_decode_tc (and with it trlb_head_gemm for the absorption and expansion) takes these sizes.
TRLB_API int trlb_latent_decode_tc_ok(int heads, int dim, int rot, int vdim, int kv_rank, int lat_w, int block_size) {
  const int boxes = ld_boxes(kv_rank, lat_w);
  if (heads <= 0 || dim % 8 || rot % 8 || vdim <= 0 || kv_rank % 8 || lat_w % 8 || boxes > LD_MAX_BOX) return 0;
  if (block_size < 8 || block_size > 128 || 128 % block_size) return 0;
  return 4 * 32 + ld_slabs(kv_rank) * 64 <= 512 && ld_smem(boxes) <= 227 * 1024;
}

// q_lat [B, heads, lat_w], cache [num_blocks, block_size, lat_w] bf16 (lat_w as in csrc/mixers.cu), one new token per slot at
// seq_lens[slot]; part_o [B, heads, splits, kv_rank] and part_ml [B, heads, splits, 2] fp32 scratch; o_lat [B, heads, kv_rank].
TRLB_API int trlb_latent_decode_tc(const void* q_lat, const void* cache, int num_blocks, int B, int heads, int kv_rank, int lat_w,
                                   int window, float scale, const int* seq_lens, const int* block_table, int max_blocks,
                                   int block_size, const float* sink, int splits, float* part_o, float* part_ml, void* o_lat,
                                   int* status, cudaStream_t st) {
  if (B <= 0) return 0;
  const int boxes = ld_boxes(kv_rank, lat_w);
  if (!(scale > 0.f) || splits < 1 || !trlb_latent_decode_tc_ok(heads, 8, 8, 8, kv_rank, lat_w, block_size)) return -230;
  CUtensorMap tq, tc;
  if (trlb_host::make_tmap_3d_bf16(&tq, q_lat, lat_w, heads, B, lat_w, (uint64_t)heads * lat_w, 64, 32, 1)) return -231;
  if (trlb_host::make_tmap_2d_bf16(&tc, cache, (uint64_t)num_blocks * block_size, lat_w, lat_w, block_size, 64)) return -232;
  LatentDecodeTc p = {heads, kv_rank, boxes, ld_slabs(kv_rank), lat_w, window, max_blocks, block_size, splits,
                      scale * 1.4426950408889634f, seq_lens, block_table, part_o, (float2*)part_ml, status};
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(latent_decode_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess)
      return -233;
    attr_set = true;
  }
  const bool pdl = trlb_host::pdl_enabled();
  const int rc = (int)trlb_host::launch_kernel(latent_decode_tc_kernel, dim3((heads + 31) / 32, splits, B), dim3(192), ld_smem(boxes),
                                               st, pdl, tq, tc, p);
  if (rc) return rc;
  return (int)trlb_host::launch_kernel(latent_combine_kernel, dim3(heads, B), dim3(128), 0, st, pdl, (const float*)part_o,
                                       (const float2*)part_ml, sink, seq_lens, heads, kv_rank, splits, (__nv_bfloat16*)o_lat);
}

TRLB_API int trlb_latent_query(float* qacc, long long ld, void* q, void* q_lat, int B, int heads, int dim, int rot, int kr_off,
                               int lat_w, const int* positions, const float* table, int table_len, cudaStream_t st) {
  if (B <= 0) return 0;
  return (int)trlb_host::launch_kernel(latent_query_kernel, dim3(heads, B), dim3(128), 0, st, trlb_host::pdl_enabled(), qacc, ld,
                                       (__nv_bfloat16*)q, (__nv_bfloat16*)q_lat, heads, dim, rot, kr_off, lat_w, positions,
                                       (const float2*)table, table_len);
}

// Y[b, h, m] (element strides y_b, y_h) = scale[b, h] * sum_k X[b, h, k] W[h][m, k].  X: strides x_b, x_h; W: w_mn = 0: [heads, M,
// K], w_mn = 1: [heads, K, M]; all strides multiples of 8, pointers 16-byte aligned.  scale [B, heads] or null.
TRLB_API int trlb_head_gemm(const void* X, long long x_b, long long x_h, const void* W, int w_mn, void* Y, long long y_b,
                            long long y_h, const float* scale, int B, int heads, int M, int K, int* status, cudaStream_t st) {
  if (B <= 0 || heads <= 0) return 0;
  if ((x_b % 8) || (x_h % 8) || (w_mn ? M % 8 : K % 8)) return -240;
  const int n_cols = B >= 128 ? 128 : (B + 15) & ~15;
  CUtensorMap tw, tx;
  using trlb_host::make_tmap_3d_bf16;
  if (w_mn) {
    if (make_tmap_3d_bf16(&tw, W, M, K, heads, M, (uint64_t)M * K, 64, 64, 1)) return -241;
  } else if (make_tmap_3d_bf16(&tw, W, K, M, heads, K, (uint64_t)M * K, 64, 128, 1)) {
    return -241;
  }
  if (make_tmap_3d_bf16(&tx, X, K, heads, B, (uint64_t)x_h, (uint64_t)x_b, 64, 1, n_cols)) return -242;
  HeadGemm p = {B, M, K, n_cols, y_b, y_h, scale, heads, (__nv_bfloat16*)Y, status};
  const size_t smem = (size_t)HG_STAGES * (LD_BOX + n_cols * 128) + 1024 + 256;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(head_gemm_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(head_gemm_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess)
      return -243;
    attr_set = true;
  }
  const dim3 grid(heads, (M + 127) / 128, (B + 127) / 128), blk(192);
  if (w_mn) return (int)trlb_host::launch_kernel(head_gemm_kernel<true>, grid, blk, smem, st, trlb_host::pdl_enabled(), tw, tx, p);
  return (int)trlb_host::launch_kernel(head_gemm_kernel<false>, grid, blk, smem, st, trlb_host::pdl_enabled(), tw, tx, p);
}
