// mLSTM over packed prompts in chunks of 128 tokens, on the 5th-generation tensor cores (bf16 q, k, v; fp32 gates,
// weights, states).
//
// With b_t the running sum of the log forget gates inside a chunk, g_j = i_j - b_j, m_t the running maximum and
// (S, n, m_in) the state in front of the chunk,
//
//     o_t = [ sum_{j <= t} e^(b_t + g_j - m_t) (q_t . k_j) v_j  +  e^(b_t + m_in - m_t) S^T q_t ] / max(|n_t . q_t|, e^-m_t)
//     S' = e^(b_L + m_in - m_L) S + sum_j e^(b_L + g_j - m_L) k_j v_j^T            (L: last token of the chunk)
//
// which is the token-by-token recurrence regrouped.  Three kernels:
//
//   mlstm_scan_kernel    b, g and m of every token (one block per sequence and head; a warp scans a chunk, the chunks'
//                        maxima are chained);
//   mlstm_state_kernel   one CTA per (sequence, head, 128 x 64 tile of S): walks the chunks, the increment of each is one
//                        128 x 64 x 128 product (both operands MN-major straight from their TMA tiles, v scaled by its
//                        token's weight in place) and the tile itself stays in fp32 registers;
//   mlstm_output_kernel  one CTA per (chunk, head, 128 columns of v): Q K^T, weights, Q S and P V, all in TMEM.
//
// fp32 precision through bf16 operands: scaled v, the weighted scores P and the states S enter the products as two bf16
// each (value and remainder).
#include "mixers.cuh"

namespace trlb {

constexpr int ML_L = 128;
constexpr float ML_LOG2E = 1.4426950408889634f;
constexpr uint32_t ML_BOX = 128 * 64 * 2;

struct MlstmChunk {
  const int* cu;
  int n_seq, T, heads, dim, vdim;
  const float* b;     // [heads, T]
  const float* g;     // [heads, T]
  const float* m;     // [heads, T]
  float* n_in;        // [chunks, heads, dim]
  __nv_bfloat16* s_hi;  // [chunks, heads, dim, vdim] state in front of a chunk, leading part and remainder; the first
  __nv_bfloat16* s_lo;  // chunk of a sequence has none
  float* S;           // slot states (see mixers.cu) or null
  float* n;
  float* mm;
  const int* seq_slot;
  int slots;
  float qscale;
  float* out;         // [T, heads, vdim]
  int* status;
};

__device__ __forceinline__ int ml_chunks(int len) { return (len + ML_L - 1) / ML_L; }

// ------------------------------------------------------------------------------------------------------------
// ig, fg [T, heads] -> b, g, m [heads, T]
__global__ void __launch_bounds__(256)
mlstm_scan_kernel(const float* __restrict__ ig, const float* __restrict__ fg, const int* __restrict__ cu, int T, int heads,
                  float* __restrict__ b, float* __restrict__ g, float* __restrict__ m) {
  __shared__ float tot[8], top[8], m_in[9];
  const int seq = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = cu[seq], len = cu[seq + 1] - t0;
  if (threadIdx.x == 0) m_in[0] = 0.f;
  for (int base = 0; base < len; base += 8 * ML_L) {
    const int c0 = base + warp * ML_L + lane * 4;  // four consecutive tokens per lane
    float f[4], bb[4], gg[4], run = 0.f, mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[i] = c0 + i < len ? fg[(size_t)(t0 + c0 + i) * heads + h] : 0.f;
      run += f[i];
    }
    float pre = run;  // inclusive scan over the lanes
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, pre, o);
      if (lane >= o) pre += x;
    }
    float acc = __shfl_up_sync(0xffffffffu, pre, 1);
    if (lane == 0) acc = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      acc += f[i];
      bb[i] = acc;
      gg[i] = c0 + i < len ? ig[(size_t)(t0 + c0 + i) * heads + h] - acc : -INFINITY;
      mx = fmaxf(mx, gg[i]);
    }
    float pm = mx;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, pm, o);
      if (lane >= o) pm = fmaxf(pm, x);
    }
    float before = __shfl_up_sync(0xffffffffu, pm, 1);
    if (lane == 0) before = -INFINITY;
    if (lane == 31) { tot[warp] = bb[3]; top[warp] = pm; }
    __syncthreads();
    if (threadIdx.x == 0)
      for (int w = 0; w < 8; ++w) m_in[w + 1] = tot[w] + fmaxf(m_in[w], top[w]);
    __syncthreads();
    float best = fmaxf(before, m_in[warp]);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      best = fmaxf(best, gg[i]);
      if (c0 + i < len) {
        const size_t at = (size_t)h * T + t0 + c0 + i;
        b[at] = bb[i];
        g[at] = gg[i];
        m[at] = bb[i] + best;
      }
    }
    __syncthreads();
    if (threadIdx.x == 0) m_in[0] = m_in[8];
  }
}

// ------------------------------------------------------------------------------------------------------------
// State pass.  Warp 0: TMA; warp 1: MMA; warps 2-5: thread r scales token r of a chunk's v, and owns row r (of the
// CTA's 128 rows of S) in registers.
constexpr int MS_STAGES = 1;  // 64 KB: two CTAs per SM hide each other's loads; the work per chunk is in the row threads
constexpr uint32_t MS_STAGE_BYTES = 4 * ML_BOX;  // k (two boxes), v scaled in place, v remainder
constexpr size_t MS_SMEM = MS_STAGES * (size_t)MS_STAGE_BYTES + 1024 + 2048;

__global__ void __launch_bounds__(192, 2)
mlstm_state_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v, const MlstmChunk p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + MS_STAGES * MS_STAGE_BYTES);
  uint64_t* full = bars;                  // [MS_STAGES] TMA landed
  uint64_t* ready = full + MS_STAGES;     // [MS_STAGES] v scaled
  uint64_t* empty = ready + MS_STAGES;    // [MS_STAGES] stage free again: product done and (for n) k read
  uint64_t* acc_full = empty + MS_STAGES; // [2]
  uint64_t* acc_empty = acc_full + 2;     // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* u_s = reinterpret_cast<float*>(bars + 32);  // [2][128] token weights of two chunks

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.x, h = blockIdx.y;
  const int e_tiles = (p.vdim + 63) / 64;
  const int d0 = (int)(blockIdx.z / e_tiles) * 128, e0 = (int)(blockIdx.z % e_tiles) * 64;
  int chunk0 = 0;
  for (int s = 0; s < seq; ++s) chunk0 += ml_chunks(p.cu[s + 1] - p.cu[s]);
  const int beg = p.cu[seq], len = p.cu[seq + 1] - beg;
  const int nc = ml_chunks(len);
  const bool with_n = e0 == 0;

  if (threadIdx.x == 0) {
    for (int s = 0; s < MS_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&ready[s], 128);
      mbar_init(&empty[s], with_n ? 129 : 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&acc_full[s], 1);
      mbar_init(&acc_empty[s], 128);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 128);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      for (int c = 0; c < nc; ++c) {
        const int s = c % MS_STAGES;
        if (!mbar_wait(&empty[s], (uint32_t)(((c / MS_STAGES) & 1) ^ 1), abort_flag, p.status, 1300 + s)) break;
        uint8_t* st = smem + (size_t)s * MS_STAGE_BYTES;
        mbar_expect_tx(&full[s], 3 * ML_BOX);
        tma_load_3d(st, &tm_k, &full[s], d0, h, beg + c * ML_L);
        tma_load_3d(st + ML_BOX, &tm_k, &full[s], d0 + 64, h, beg + c * ML_L);
        tma_load_3d(st + 2 * ML_BOX, &tm_v, &full[s], e0, h, beg + c * ML_L);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc_bf16_major(128, 64, true, true);
      for (int c = 0; c < nc; ++c) {
        const int s = c % MS_STAGES, a = c & 1;
        if (!mbar_wait(&acc_empty[a], (uint32_t)(((c >> 1) & 1) ^ 1), abort_flag, p.status, 1310 + a)) break;
        if (!mbar_wait(&ready[s], (uint32_t)((c / MS_STAGES) & 1), abort_flag, p.status, 1320 + s)) break;
        tc_fence_after();
        const uint64_t st = umma_desc_mnmajor_sw128(smem_u32(smem + (size_t)s * MS_STAGE_BYTES), ML_BOX);
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int kk = 0; kk < ML_L / 16; ++kk)
            umma_bf16_ss(tmem_base + (uint32_t)a * 64, desc_at(st, kk * 2048), desc_at(st, (2 + half) * ML_BOX + kk * 2048), idesc,
                         (half | kk) != 0);
        umma_commit(&acc_full[a]);
        umma_commit(&empty[s]);
      }
    }
    __syncwarp();
  } else {
    const int r = (warp & 3) * 32 + lane;
    const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
    const int d = d0 + r;
    float st[64];
#pragma unroll
    for (int i = 0; i < 64; ++i) st[i] = 0.f;
    float n_run = 0.f, m_prev = 0.f;
    float keep_prev = 0.f;
    const float* bh = p.b + (size_t)h * p.T + beg;
    const float* gh = p.g + (size_t)h * p.T + beg;
    const float* mh = p.m + (size_t)h * p.T + beg;
    bool ok = true;
    // one iteration past the end: the increment of chunk c - 1 is taken in while that of chunk c is being formed
    for (int c = 0; c <= nc && ok; ++c) {
      float keep = 0.f;
      if (c < nc) {
        const int s = c % MS_STAGES;
        const int last = min(len, (c + 1) * ML_L) - 1;
        const int t = c * ML_L + r;
        const float bl = bh[last], ml = mh[last];
        keep = expf(bl + m_prev - ml);
        m_prev = ml;
        const float u = t < len ? expf(bl + gh[t] - ml) : 0.f;
        u_s[(c & 1) * 128 + r] = u;
        ok = __all_sync(0xffffffffu, mbar_wait(&full[s], (uint32_t)((c / MS_STAGES) & 1), abort_flag, p.status, 1330 + s));
        if (!ok) break;
        uint8_t* hi = smem + (size_t)s * MS_STAGE_BYTES + 2 * ML_BOX + (size_t)r * 128;
        uint8_t* lo = hi + ML_BOX;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int at = ((i + r) & 7) * 16;  // token r's row is 128 contiguous bytes; the swizzle only permutes inside it
          const uint4 x = *reinterpret_cast<const uint4*>(hi + at);
          const uint32_t w[4] = {x.x, x.y, x.z, x.w};
          uint32_t a[4], b2[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const float2 f = unpack_bf16(w[q]);
            a[q] = pack_bf16(f.x * u, f.y * u);
            const float2 back = unpack_bf16(a[q]);
            b2[q] = pack_bf16(f.x * u - back.x, f.y * u - back.y);
          }
          *reinterpret_cast<uint4*>(hi + at) = make_uint4(a[0], a[1], a[2], a[3]);
          *reinterpret_cast<uint4*>(lo + at) = make_uint4(b2[0], b2[1], b2[2], b2[3]);
        }
        fence_proxy_async_smem();
        mbar_arrive(&ready[s]);
      }
      if (c > 0) {
        const int a = (c - 1) & 1;
        ok = __all_sync(0xffffffffu, mbar_wait(&acc_full[a], (uint32_t)(((c - 1) >> 1) & 1), abort_flag, p.status, 1340 + a));
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int x = 0; x < 64; x += 32) {
          float v[32];
          tmem_ld_32x32(tmem_base + lane_off + (uint32_t)(a * 64 + x), v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) st[x + i] = fmaf(st[x + i], keep_prev, v[i]);
        }
        tc_fence_before();
        mbar_arrive(&acc_empty[a]);
        if (c < nc && d < p.dim) {
          const size_t row = (((size_t)(chunk0 + c) * p.heads + h) * p.dim + d) * p.vdim + e0;
#pragma unroll
          for (int x = 0; x < 64; x += 8) {
            if (e0 + x < p.vdim) {
              uint32_t a4[4], b4[4];
#pragma unroll
              for (int q = 0; q < 4; ++q) {
                a4[q] = pack_bf16(st[x + 2 * q], st[x + 2 * q + 1]);
                const float2 back = unpack_bf16(a4[q]);
                b4[q] = pack_bf16(st[x + 2 * q] - back.x, st[x + 2 * q + 1] - back.y);
              }
              *reinterpret_cast<uint4*>(p.s_hi + row + x) = make_uint4(a4[0], a4[1], a4[2], a4[3]);
              *reinterpret_cast<uint4*>(p.s_lo + row + x) = make_uint4(b4[0], b4[1], b4[2], b4[3]);
            }
          }
        }
      }
      if (c < nc && with_n) {
        // n: row r's column of k against the weights of all 128 tokens
        const int s = c % MS_STAGES;
        ok = __all_sync(0xffffffffu, mbar_wait(&ready[s], (uint32_t)((c / MS_STAGES) & 1), abort_flag, p.status, 1350 + s));
        if (!ok) break;
        if (c > 0 && d < p.dim) p.n_in[((size_t)(chunk0 + c) * p.heads + h) * p.dim + d] = n_run;
        const uint8_t* kb = smem + (size_t)s * MS_STAGE_BYTES + (size_t)(r >> 6) * ML_BOX;
        const int cc = r & 63;
        float add = 0.f;
#pragma unroll 8
        for (int j = 0; j < 128; ++j) {
          const uint32_t off = (uint32_t)j * 128 + (uint32_t)((((cc >> 3) ^ (j & 7)) << 4) | ((cc & 7) * 2));
          add = fmaf(u_s[(c & 1) * 128 + j], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(kb + off)), add);
        }
        n_run = fmaf(n_run, keep, add);
        mbar_arrive(&empty[s]);
      }
      keep_prev = keep;
    }
    if (ok && p.seq_slot != nullptr && d < p.dim) {
      const int slot = p.seq_slot[seq];
      if (slot >= 0 && slot < p.slots) {
        const int par = len & 1;
        float* dst = p.S + (((size_t)slot * p.heads + h) * p.dim + d) * p.vdim + e0;
#pragma unroll
        for (int x = 0; x < 64; x += 4)
          if (e0 + x < p.vdim) *reinterpret_cast<float4*>(dst + x) = make_float4(st[x], st[x + 1], st[x + 2], st[x + 3]);
        if (with_n) {
          p.n[(((size_t)par * p.slots + slot) * p.heads + h) * p.dim + d] = n_run;
          if (d == 0) p.mm[((size_t)par * p.slots + slot) * p.heads + h] = m_prev;
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
    tmem_dealloc(tmem_base, 128);
  }
}

// ------------------------------------------------------------------------------------------------------------
// Output pass.  Warp 0: TMA; warp 1: MMA; warps 2-5: one thread per token of the chunk.  Q stays in shared memory; K
// boxes, 64-row pieces of S (leading part, remainder) and finally the halves of V travel through one ring of 16 KB boxes.
// TMEM: scores / weights [0, 128), output [128, 256): two CTAs fit an SM when the ring is short enough.
constexpr int MO_MAX_STAGES = 6;

__global__ void __launch_bounds__(192, 2)
mlstm_output_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                    const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_sh,
                    const __grid_constant__ CUtensorMap tm_sl, const MlstmChunk p, const int stages) {
  int seq = -1, c = (int)blockIdx.x;
  for (int s = 0; s < p.n_seq; ++s) {
    const int n = ml_chunks(p.cu[s + 1] - p.cu[s]);
    if (c < n) { seq = s; break; }
    c -= n;
  }
  if (seq < 0) return;  // uniform: before any barrier or TMEM use
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nd = (p.dim + 63) / 64;
  uint8_t* q_s = smem;
  uint8_t* ring = q_s + (size_t)nd * ML_BOX;
  uint64_t* bars = reinterpret_cast<uint64_t*>(ring + (size_t)stages * ML_BOX);
  uint64_t* q_full = bars;
  uint64_t* full = bars + 1;                  // [MO_MAX_STAGES]
  uint64_t* empty = full + MO_MAX_STAGES;     // [MO_MAX_STAGES]
  uint64_t* s_full = empty + MO_MAX_STAGES;   // scores done
  uint64_t* x_full = s_full + 1;           // Q S done
  uint64_t* p_full = x_full + 1;           // weights in TMEM, output rescaled
  uint64_t* o_full = p_full + 1;
  uint64_t* g_full = o_full + 1;           // key weights in shared memory
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(g_full + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* g_s = reinterpret_cast<float*>(bars + 32);  // [128] g_j log2(e)
  float* n_s = g_s + 128;                            // [dim] n in front of the chunk

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, e0 = (int)blockIdx.z * 128;
  const int beg = p.cu[seq], len = p.cu[seq + 1] - beg;
  const int row0 = beg + c * ML_L;                  // first token of the chunk in the packed stream
  const int chunk = (int)blockIdx.x;                // chunks are numbered in the order of this search
  const int n_cols = min(128, (p.vdim - e0 + 15) & ~15);
  const bool carried = c > 0;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < MO_MAX_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(s_full, 1);
    mbar_init(x_full, 1);
    mbar_init(p_full, 128);
    mbar_init(o_full, 1);
    mbar_init(g_full, 128);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const int nv = (n_cols + 63) / 64, n_state = carried ? 2 * nd : 0;
  const int n_items = nd + n_state + nv;  // K boxes, state pieces, halves of V

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, (uint32_t)nd * ML_BOX);
      for (int i = 0; i < nd; ++i) tma_load_3d(q_s + (size_t)i * ML_BOX, &tm_q, q_full, 64 * i, h, row0);
      for (int it = 0; it < n_items; ++it) {
        const int s = it % stages;
        if (!mbar_wait(&empty[s], (uint32_t)(((it / stages) & 1) ^ 1), abort_flag, p.status, 1400 + s)) break;
        uint8_t* st = ring + (size_t)s * ML_BOX;
        mbar_expect_tx(&full[s], ML_BOX);
        if (it < nd) {
          tma_load_3d(st, &tm_k, &full[s], 64 * it, h, row0);
        } else if (it < nd + n_state) {
          // rows 64 i .. of S as two 64-column boxes of 8 KB
          const CUtensorMap* tm = ((it - nd) & 1) ? &tm_sl : &tm_sh;
          const int d = 64 * ((it - nd) >> 1), z = chunk * p.heads + h;
          tma_load_3d(st, tm, &full[s], e0, d, z);
          tma_load_3d(st + 8192, tm, &full[s], e0 + 64, d, z);
        } else {
          tma_load_3d(st, &tm_v, &full[s], e0 + 64 * (it - nd - n_state), h, row0);
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16_major(128, 128, false, false);
      const uint32_t idesc_o = umma_idesc_bf16_major(128, n_cols, false, true);
      const uint64_t q_k = umma_desc_kmajor_sw128(smem_u32(q_s)), r_k = umma_desc_kmajor_sw128(smem_u32(ring));
      const uint64_t r_s = umma_desc_mnmajor_sw128(smem_u32(ring), 8192), r_v = umma_desc_mnmajor_sw128(smem_u32(ring), ML_BOX);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status, 1410);
      for (int it = 0; it < n_items && ok; ++it) {
        const int s = it % stages;
        if (it == nd + n_state) ok = mbar_wait(p_full, 0, abort_flag, p.status, 1412);
        if (ok) ok = mbar_wait(&full[s], (uint32_t)((it / stages) & 1), abort_flag, p.status, 1420 + s);
        if (!ok) break;
        tc_fence_after();
        const uint32_t st = (uint32_t)s * ML_BOX;
        if (it < nd) {
          const int steps = min(4, (p.dim - 64 * it + 15) >> 4);
          const uint64_t da = desc_at(q_k, (uint32_t)it * ML_BOX), db = desc_at(r_k, st);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            if (kk < steps) umma_bf16_ss(tmem_base, da + 2 * kk, db + 2 * kk, idesc_s, (it | kk) != 0);
          if (it == nd - 1) umma_commit(s_full);
        } else if (it < nd + n_state) {
          const int i = (it - nd) >> 1;
          const int steps = min(4, (p.dim - 64 * i + 15) >> 4);
          const uint64_t da = desc_at(q_k, (uint32_t)i * ML_BOX), db = desc_at(r_s, st);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            if (kk < steps) umma_bf16_ss(tmem_base + 128, da + 2 * kk, desc_at(db, kk * 2048), idesc_o, (it > nd) || kk != 0);
          if (it == nd + n_state - 1) umma_commit(x_full);
        } else {
          const int i = it - nd - n_state;
          const uint32_t idesc_v = umma_idesc_bf16_major(128, min(64, n_cols - 64 * i), false, true);
          const uint64_t db = desc_at(r_v, st);
#pragma unroll
          for (int half = 0; half < 2; ++half)
#pragma unroll
            for (int kk = 0; kk < ML_L / 16; ++kk)
              umma_bf16_ts(tmem_base + 128 + 64 * i, tmem_base + (uint32_t)(half * 64 + kk * 8),
                           desc_at(db, kk * 2048), idesc_v, carried || (half | kk) != 0);
          if (it == n_items - 1) umma_commit(o_full);
        }
        umma_commit(&empty[s]);
      }
    }
    __syncwarp();
  } else {
    const int r = (warp & 3) * 32 + lane;
    const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
    const int t = c * ML_L + r;  // position in the sequence
    const bool row_ok = t < len;
    const size_t at = (size_t)h * p.T + beg;
    g_s[r] = row_ok ? p.g[at + t] * ML_LOG2E : -INFINITY;
    if (carried)
      for (int d = r; d < p.dim; d += 128) n_s[d] = p.n_in[((size_t)chunk * p.heads + h) * p.dim + d];
    mbar_arrive(g_full);
    const float bt = row_ok ? p.b[at + t] : 0.f, mt = row_ok ? p.m[at + t] : 0.f;
    const float m_in = carried ? p.m[at + c * ML_L - 1] : 0.f;
    const float carry = (carried && row_ok) ? expf(bt + m_in - mt) * p.qscale : 0.f;  // weight of the state, with q's scale
    const float c2 = (bt - mt) * ML_LOG2E;
    float nq = 0.f;
    bool ok = __all_sync(0xffffffffu, mbar_wait(q_full, 0, abort_flag, p.status, 1430));
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(g_full, 0, abort_flag, p.status, 1432));
    if (ok && carried) {
      for (int d = 0; d < p.dim; d += 8) {
        const int box = d >> 6, cc = (d & 63) >> 3;
        const uint4 x = *reinterpret_cast<const uint4*>(q_s + (size_t)box * ML_BOX + (size_t)r * 128 + ((cc ^ (r & 7)) << 4));
        const float4 n0 = *reinterpret_cast<const float4*>(n_s + d), n1 = *reinterpret_cast<const float4*>(n_s + d + 4);
        const float2 a = unpack_bf16(x.x), b = unpack_bf16(x.y), e = unpack_bf16(x.z), f = unpack_bf16(x.w);
        nq += a.x * n0.x + a.y * n0.y + b.x * n0.z + b.y * n0.w + e.x * n1.x + e.y * n1.y + f.x * n1.z + f.y * n1.w;
      }
      nq *= carry;
    }
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(s_full, 0, abort_flag, p.status, 1434));
    if (ok) {
      tc_fence_after();
      const uint32_t ts = tmem_base + lane_off, to = ts + 128;
      // the last 64 keys first: their packed weights wait in registers until the first 64 scores have been read too
      uint32_t late[2][32];
#pragma unroll
      for (int y = 0; y < 4; ++y) {
        const int x = y ^ 2;  // 2, 3, 0, 1
        float v[32];
        tmem_ld_32x32(ts + 32 * x, v);
        tmem_ld_wait();
        uint32_t a[16], b[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float w[2];
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            const int j = 32 * x + 2 * i + k;
            w[k] = (row_ok && j <= r) ? fast_exp2(c2 + g_s[j]) * p.qscale * v[2 * i + k] : 0.f;
            nq += w[k];
          }
          a[i] = pack_bf16(w[0], w[1]);
          const float2 back = unpack_bf16(a[i]);
          b[i] = pack_bf16(w[0] - back.x, w[1] - back.y);
        }
        if (y < 2) {
#pragma unroll
          for (int i = 0; i < 16; ++i) { late[y][i] = a[i]; late[y][16 + i] = b[i]; }
        } else {
          // columns [64, 128) have been read, and of [0, 64) those up to here
          tmem_st_32x16(ts + 16 * x, a);
          tmem_st_32x16(ts + 64 + 16 * x, b);
        }
      }
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        uint32_t a[16], b[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) { a[i] = late[y][i]; b[i] = late[y][16 + i]; }
        tmem_st_32x16(ts + 32 + 16 * y, a);
        tmem_st_32x16(ts + 96 + 16 * y, b);
      }
      if (carried) {
        ok = __all_sync(0xffffffffu, mbar_wait(x_full, 0, abort_flag, p.status, 1436));
        if (ok) {
          tc_fence_after();
#pragma unroll 1
          for (int x = 0; x < n_cols; x += 16) {
            float o[16];
            tmem_ld_32x16(to + x, o);
            tmem_ld_wait();
            uint32_t w[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) w[i] = __float_as_uint(o[i] * carry);
            tmem_st_32x16(to + x, w);
          }
        }
      }
      tmem_st_wait();
      tc_fence_before();
      if (ok) mbar_arrive(p_full);
    }
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(o_full, 0, abort_flag, p.status, 1438));
    if (ok) {
      tc_fence_after();
      const float inv = row_ok ? 1.f / (fmaxf(fabsf(nq), expf(-mt)) + 1e-6f) : 0.f;
      float* dst = p.out + ((size_t)(row0 + r) * p.heads + h) * p.vdim + e0;
#pragma unroll 1
      for (int x = 0; x < n_cols; x += 16) {
        float o[16];
        tmem_ld_32x16(tmem_base + lane_off + 128 + x, o);
        tmem_ld_wait();
        if (row_ok) {
#pragma unroll
          for (int i = 0; i < 16; i += 4)
            if (e0 + x + i < p.vdim)
              *reinterpret_cast<float4*>(dst + x + i) = make_float4(o[i] * inv, o[i + 1] * inv, o[i + 2] * inv, o[i + 3] * inv);
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
    tmem_dealloc(tmem_base, 256);
  }
}

}  // namespace trlb

using namespace trlb;

namespace {

size_t mo_smem(int dim, int stages) {
  return ((size_t)((dim + 63) / 64) + stages) * ML_BOX + 1024 + 256 + 512 + (size_t)dim * 4;
}

// Ring length: what lets two CTAs share an SM if that is at least two boxes, else what one CTA can have.
int mo_stages(int dim) {
  for (int limit : {113 * 1024, 227 * 1024})
    for (int n = MO_MAX_STAGES; n >= 2; --n)
      if (mo_smem(dim, n) <= (size_t)limit) return n;
  return 0;
}

}  // namespace

// 1 when trlb_mlstm_chunk takes these sizes.
TRLB_API int trlb_mlstm_chunk_ok(int heads, int dim, int vdim) {
  return heads > 0 && dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && mo_stages(dim) > 0;
}

// Chunks (upper bound) of T packed tokens in n_seq sequences: the leading size of s_hi, s_lo [chunks, heads, dim, vdim] bf16
// and n_in [chunks, heads, dim] fp32.
TRLB_API int trlb_mlstm_chunks(int T, int n_seq) { return (T + ML_L - 1) / ML_L + n_seq; }

// qkv [T, ld] bf16: q at 0, k at k_off, v at v_off (elements, multiples of 8).  ig, fg [T, heads] log gates; b, g, m [heads, T]
// scratch.  S, n, m_st: slot states (csrc/mixers.cu) or null.  out [T, heads, vdim] fp32.
TRLB_API int trlb_mlstm_chunk(const void* qkv, long long ld, int k_off, int v_off, const float* ig, const float* fg,
                              const int* cu, int n_seq, int T, const int* seq_slot, float* S, float* n, float* m_st, int slots,
                              int heads, int dim, int vdim, float qscale, float* b, float* g, float* m, float* n_in,
                              void* s_hi, void* s_lo, float* out, int* status, cudaStream_t st) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (!trlb_mlstm_chunk_ok(heads, dim, vdim) || (ld % 8) || (k_off % 8) || (v_off % 8)) return -220;
  const int chunks = trlb_mlstm_chunks(T, n_seq);
  const __nv_bfloat16* x = (const __nv_bfloat16*)qkv;
  CUtensorMap tq, tk, tv, tsh, tsl;
  using trlb_host::make_tmap_3d_bf16;
  if (make_tmap_3d_bf16(&tq, x, dim, heads, T, dim, (uint64_t)ld, 64, 1, 128)) return -221;
  if (make_tmap_3d_bf16(&tk, x + k_off, dim, heads, T, dim, (uint64_t)ld, 64, 1, 128)) return -222;
  if (make_tmap_3d_bf16(&tv, x + v_off, vdim, heads, T, vdim, (uint64_t)ld, 64, 1, 128)) return -223;
  if (make_tmap_3d_bf16(&tsh, s_hi, vdim, dim, (uint64_t)chunks * heads, vdim, (uint64_t)dim * vdim, 64, 64, 1)) return -224;
  if (make_tmap_3d_bf16(&tsl, s_lo, vdim, dim, (uint64_t)chunks * heads, vdim, (uint64_t)dim * vdim, 64, 64, 1)) return -225;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(mlstm_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MS_SMEM) != cudaSuccess ||
        cudaFuncSetAttribute(mlstm_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess)
      return -226;
    attr_set = true;
  }
  MlstmChunk p = {};
  p.cu = cu; p.n_seq = n_seq; p.T = T; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.b = b; p.g = g; p.m = m; p.n_in = n_in; p.s_hi = (__nv_bfloat16*)s_hi; p.s_lo = (__nv_bfloat16*)s_lo;
  p.S = S; p.n = n; p.mm = m_st; p.seq_slot = S ? seq_slot : nullptr; p.slots = slots;
  p.qscale = qscale; p.out = out; p.status = status;
  mlstm_scan_kernel<<<dim3(n_seq, heads), 256, 0, st>>>(ig, fg, cu, T, heads, b, g, m);
  const int tiles = ((dim + 127) / 128) * ((vdim + 63) / 64);
  mlstm_state_kernel<<<dim3(n_seq, heads, tiles), 192, MS_SMEM, st>>>(tk, tv, p);
  mlstm_output_kernel<<<dim3(chunks, heads, (vdim + 127) / 128), 192, mo_smem(dim, mo_stages(dim)), st>>>(tq, tk, tv, tsh, tsl, p,
                                                                                                                  mo_stages(dim));
  return (int)cudaGetLastError();
}
