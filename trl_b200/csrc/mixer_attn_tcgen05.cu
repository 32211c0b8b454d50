// Prompt attention of the layered decoders' mixers on the 5th-generation tensor cores (bf16, packed sequences).
//
// The structure is that of fa_varlen_tcgen05.cu (one CTA per 128-query tile and head; TMA warp, MMA warp, one softmax
// thread per query row; S double-buffered in TMEM, O accumulated in TMEM and rescaled only when a row's reference
// maximum moves by more than 2^8).  What differs:
//
//   * a query / key vector may have two parts that live in different tensors: `dim` elements per head and `rot` rotated
//     elements (in q behind the first part; keys in rows of their own, ONE for all heads).  Each part is loaded as
//     64-column TMA boxes, zero-filled past its end, so nothing is concatenated or expanded in memory; Q.K^T runs over
//     the 16-column steps that hold data.  rot = 0: no such part;
//   * groups of heads / kv_heads query heads read one key / value head;
//   * sizes are launch parameters: dim, rot, vdim any multiples of 8 (vdim <= 256) that leave room for one stage;
//   * probabilities keep 32-bit precision into P.V: each is split into two bf16 (value and remainder) that replace the scores
//     in TMEM, 32 keys at a time (16 columns of values, 16 of remainders), and P.V accumulates both products;
//   * scores may be capped, cap tanh(s / cap) (CAP): an odd polynomial (the Taylor series of tanh, its length by the largest
//     score of the tile) near zero, where scores of normed queries and keys lie, so that the special-function units are left
//     to the exponentials; exp2 and a division further out;
//   * NB = 1 when two CTAs fit an SM (vdim <= 128, at most 6 boxes of Q, K and V together): one S buffer of 128 columns and O
//     in 256 columns of TMEM; the softmax of one CTA runs beside the products of the other.  NB = 2 otherwise: one CTA, S
//     double-buffered;
//   * the softmax denominator may contain exp(sink[head]);
//   * the output may be multiplied by a gate: one fp32 factor per token and head, or the sigmoid of bf16 logits per
//     element;
//   * keys are those of the same sequence, with a window those at distance < window and the first `keep` of the sequence: the
//     tiles of a CTA are those that hold kept keys, then those of the window; the last kept tile is only as wide (in steps of
//     32 keys) as the kept keys reach;
//   * in place of kept keys there may be means of blocks of `pool` keys and values (tensors of their own, grouped_attn.cu), seen by
//     the queries whose window begins behind the block: tiles of these means come first.
#include "mixers.cuh"

namespace trlb {

constexpr int LA_BM = 128, LA_BN = 128;
constexpr int LA_THREADS = 192;
constexpr uint32_t LA_BOX = 128 * 64 * 2;  // one TMA box: 128 rows x 64 bf16, 128-byte swizzle

enum { GATE_NONE = 0, GATE_HEAD = 1, GATE_LOGITS = 2 };

struct MixerAttnTc {
  const int* cu;
  int n_seq, heads, group, dim, rot, vdim, window, keep, pool;
  int nn, nr, nv;      // boxes of the unrotated part, the rotated part and the value
  int k_stages, v_stages;
  float scale_log2;    // CAP: 1 (capped scores are in log2 units already)
  float cap_in, cap_out;  // CAP: scale / cap, cap log2(e)
  float poly[6];          // CAP: cap_out tanh(cap_in v) = v (poly[0] + poly[1] v^2 + ...)
  float near7, near11;    // CAP: |v| up to which the polynomial through v^7, v^11 serves
  const float* sink;   // [heads] or null
  int gate_mode;
  const void* gate;    // GATE_HEAD: fp32 [T, heads]; GATE_LOGITS: bf16 [T, gate_ld >= heads vdim]
  long long gate_ld;
  __nv_bfloat16* out;  // [T rows of out_ld], heads x vdim
  long long out_ld;
  float out_scale;
  int* status;
};

__device__ __forceinline__ bool la_find_tile(const int* cu, int n_seq, int slot, int& seq, int& tile) {
  for (int s = 0; s < n_seq; ++s) {
    const int nt = (cu[s + 1] - cu[s] + LA_BM - 1) / LA_BM;
    if (slot < nt) { seq = s; tile = nt - 1 - slot; return true; }
    slot -= nt;
  }
  return false;
}

// cap_out tanh(cap_in v); LEVEL 0, 1: the polynomial through v^7, v^11, 2: any v
template <int LEVEL>
__device__ __forceinline__ float la_capped(const MixerAttnTc& p, float v) {
  if (LEVEL == 2) return p.cap_out * tanh_exp(p.cap_in * v);
  const float z = v * v;
  float t = p.poly[3];
  if (LEVEL == 1) t = fmaf(z, fmaf(z, p.poly[5], p.poly[4]), t);
  t = fmaf(z, t, p.poly[2]);
  t = fmaf(z, t, p.poly[1]);
  return v * fmaf(z, t, p.poly[0]);
}

// Bits of the 32 scores from column c on that a row sees: first .. last, and the columns before `kept`.
__device__ __forceinline__ uint32_t la_visible(int c, int first, int last, int kept) {
  const int n = min(last - c, 31), k = min(kept - 1 - c, n), f = max(first - c, 0);
  uint32_t m = n >= f ? (0xffffffffu >> (31 - n)) & (0xffffffffu << f) : 0u;
  if (k >= 0) m |= 0xffffffffu >> (31 - k);
  return m;
}

// First pass over a row of scores: the largest visible one and (SPAN) the largest magnitude of any.  Loops over 32 scores stay
// rolled and tiles without masked keys have code of their own: instruction fetch and count are what limits these passes.
template <bool SPAN, bool FULL>
__device__ __forceinline__ float2 la_row_max(uint32_t ts, int width, int first, int last, int kept) {
  float mx[2] = {-INFINITY, -INFINITY}, mn[2] = {INFINITY, INFINITY};
#pragma unroll 1
  for (int c = 0; c < (FULL ? LA_BN : width); c += 32) {
    float v[32];
    tmem_ld_32x32(ts + c, v);
    const uint32_t seen = FULL ? 0u : la_visible(c, first, last, kept);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      if (SPAN) mn[i & 1] = fminf(mn[i & 1], FULL ? v[i] : -fabsf(v[i]));
      mx[i & 1] = fmaxf(mx[i & 1], FULL || (seen >> i & 1u) ? v[i] : -INFINITY);
    }
  }
  const float m = fmaxf(mx[0], mx[1]);
  return make_float2(m, SPAN ? fmaxf(m, -fminf(mn[0], mn[1])) : 0.f);
}

// Second pass: probabilities, as value and remainder, in place.  LEVEL -1: no cap.  Returns their sum.
template <int LEVEL, bool FULL>
__device__ __forceinline__ float la_probs(const MixerAttnTc& p, uint32_t ts, int width, float neg_m, int first, int last, int kept) {
  float sum[2] = {0.f, 0.f};
#pragma unroll 1
  for (int c = 0; c < (FULL ? LA_BN : width); c += 32) {
    float v[32];
    tmem_ld_32x32(ts + c, v);
    const uint32_t seen = FULL ? 0u : la_visible(c, first, last, kept);
    tmem_ld_wait();
    uint32_t a[16], b[16];
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      if (LEVEL < 0) v[i] = fast_exp2(fmaf(v[i], p.scale_log2, neg_m));
      else v[i] = fast_exp2(la_capped<LEVEL < 0 ? 0 : LEVEL>(p, v[i]) + neg_m);
      if (!FULL) v[i] = seen >> i & 1u ? v[i] : 0.f;
      sum[i & 1] += v[i];
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      a[i] = pack_bf16(v[2 * i], v[2 * i + 1]);
      const float2 f = unpack_bf16(a[i]);
      b[i] = pack_bf16(v[2 * i] - f.x, v[2 * i + 1] - f.y);
    }
    tmem_st_32x16(ts + c, a);
    tmem_st_32x16(ts + c + 16, b);
  }
  tmem_st_wait();
  return sum[0] + sum[1];
}

template <bool CAP, int NB>
__global__ void __launch_bounds__(LA_THREADS, 3 - NB)
mixer_attn_tc_kernel(const __grid_constant__ CUtensorMap tm_qn, const __grid_constant__ CUtensorMap tm_qr,
                      const __grid_constant__ CUtensorMap tm_kn, const __grid_constant__ CUtensorMap tm_kr,
                      const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_pk,
                      const __grid_constant__ CUtensorMap tm_pv, const MixerAttnTc p) {
  int seq, tile;
  if (!la_find_tile(p.cu, p.n_seq, (int)blockIdx.x, seq, tile)) return;  // uniform: before any barrier or TMEM use
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t k_bytes = (uint32_t)(p.nn + p.nr) * LA_BOX, v_bytes = (uint32_t)p.nv * LA_BOX;
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + k_bytes;
  uint8_t* v_s = k_s + (size_t)p.k_stages * k_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + (size_t)p.v_stages * v_bytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;        // [<= 3]
  uint64_t* k_empty = bars + 4;
  uint64_t* v_full = bars + 7;
  uint64_t* v_empty = bars + 10;
  uint64_t* s_full = bars + 13;       // [2]
  uint64_t* p_full = bars + 15;       // [2]
  uint64_t* o_full = bars + 17;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 18);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, hk = h / p.group;
  const int beg = p.cu[seq], len = p.cu[seq + 1] - beg;
  const int q_first = tile * LA_BM;
  const int q_last = min(len, q_first + LA_BM) - 1;
  const int hi = q_last / LA_BN;
  const int lo = p.window > 0 ? max(0, q_first - p.window + 1) / LA_BN : 0;
  // keys before the window (of the last query, which sees most of them) and their tiles
  const int before = p.pool > 0 ? max(0, q_last - p.window + 1) / p.pool : p.keep;
  const int kt = p.pool > 0 ? (before + LA_BN - 1) / LA_BN : min((p.keep + LA_BN - 1) / LA_BN, lo);
  const int n_kv = kt + hi - lo + 1;  // >= 1: a token sees itself
  auto tile_at = [&](int j) { return j < kt ? j : lo + j - kt; };
  auto width_at = [&](int j) { return j < kt ? min(LA_BN, (before - j * LA_BN + 31) & ~31) : LA_BN; };
  const int pool_row = p.pool > 0 ? beg / p.pool : 0;  // where the sequence's blocks begin

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < 3; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&s_full[s], 1);
      mbar_init(&p_full[s], 128);
    }
    mbar_init(o_full, 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_qn);
    tma_prefetch_desc(&tm_kn);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, NB * 256);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      mbar_expect_tx(q_full, k_bytes);
      for (int i = 0; i < p.nn; ++i) tma_load_3d(q_s + i * LA_BOX, &tm_qn, q_full, 64 * i, h, beg + q_first);
      for (int i = 0; i < p.nr; ++i) tma_load_3d(q_s + (p.nn + i) * LA_BOX, &tm_qr, q_full, 64 * i, h, beg + q_first);
      auto load_k = [&](int j) {
        const int s = j % p.k_stages;
        if (!mbar_wait(&k_empty[s], (uint32_t)(((j / p.k_stages) & 1) ^ 1), abort_flag, p.status, 1200 + s)) return false;
        uint8_t* ks = k_s + (size_t)s * k_bytes;
        const bool mean = p.pool > 0 && j < kt;
        const int row = (mean ? pool_row : beg) + tile_at(j) * LA_BN;
        mbar_expect_tx(&k_full[s], k_bytes);
        for (int i = 0; i < p.nn; ++i) tma_load_3d(ks + i * LA_BOX, mean ? &tm_pk : &tm_kn, &k_full[s], 64 * i, hk, row);
        for (int i = 0; i < p.nr; ++i) tma_load_2d(ks + (p.nn + i) * LA_BOX, &tm_kr, &k_full[s], 64 * i, row);
        return true;
      };
      bool ok = load_k(0);
      for (int j = 0; j < n_kv && ok; ++j) {
        if (NB == 2 && j + 1 < n_kv) ok = load_k(j + 1);
        if (!ok) break;
        const int s = j % p.v_stages;
        if (!mbar_wait(&v_empty[s], (uint32_t)(((j / p.v_stages) & 1) ^ 1), abort_flag, p.status, 1205 + s)) break;
        uint8_t* vs = v_s + (size_t)s * v_bytes;
        mbar_expect_tx(&v_full[s], v_bytes);
        const bool mean = p.pool > 0 && j < kt;
        const int row = (mean ? pool_row : beg) + tile_at(j) * LA_BN;
        for (int i = 0; i < p.nv; ++i) tma_load_3d(vs + i * LA_BOX, mean ? &tm_pv : &tm_v, &v_full[s], 64 * i, hk, row);
        if (NB == 1 && j + 1 < n_kv) ok = load_k(j + 1);  // one stage: free only after S(j)
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      const uint32_t idesc_o = umma_idesc_bf16_major(LA_BM, (p.vdim + 15) & ~15, false, true);  // V is MN-major
      const uint64_t q_d = umma_desc_kmajor_sw128(smem_u32(q_s)), k_d = umma_desc_kmajor_sw128(smem_u32(k_s));
      const uint64_t v_d = umma_desc_mnmajor_sw128(smem_u32(v_s), LA_BOX);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status, 1210);
      auto issue_s = [&](int j) {
        const int s = j % NB, kst = j % p.k_stages;
        // buffer s is free: its P.V product (tile j - NB) was issued before this call
        if (!mbar_wait(&k_full[kst], (uint32_t)((j / p.k_stages) & 1), abort_flag, p.status, 1220 + kst)) return false;
        tc_fence_after();
        const uint64_t k_t = desc_at(k_d, (uint32_t)kst * k_bytes);
        const uint32_t idesc_s = umma_idesc_bf16_major(LA_BM, width_at(j), false, false);
        uint32_t acc = 0;
        for (int i = 0; i < p.nn + p.nr; ++i) {
          const int left = i < p.nn ? p.dim - 64 * i : p.rot - 64 * (i - p.nn);
          const int steps = min(4, (left + 15) >> 4);
          const uint64_t da = desc_at(q_d, (uint32_t)i * LA_BOX), db = desc_at(k_t, (uint32_t)i * LA_BOX);
          for (int kk = 0; kk < steps; ++kk) {
            umma_bf16_ss(tmem_base + (uint32_t)s * LA_BN, da + 2 * kk, db + 2 * kk, idesc_s, acc);
            acc = 1;
          }
        }
        umma_commit(&s_full[s]);
        umma_commit(&k_empty[kst]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; j < n_kv && ok; ++j) {
        if (NB == 2 && j + 1 < n_kv) ok = issue_s(j + 1);
        if (!ok) break;
        const int sb = j % NB, s = j % p.v_stages;
        if (!mbar_wait(&p_full[sb], (uint32_t)((j / NB) & 1), abort_flag, p.status, 1240 + sb)) break;
        if (!mbar_wait(&v_full[s], (uint32_t)((j / p.v_stages) & 1), abort_flag, p.status, 1250 + s)) break;
        tc_fence_after();
        const uint64_t v_t = desc_at(v_d, (uint32_t)s * v_bytes);
        const int steps = width_at(j) / 16;
        // 32 keys are 16 columns of values and 16 of remainders, 16 keys an MMA step
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int kk = 0; kk < LA_BN / 16; ++kk)
            if (kk < steps) umma_bf16_ts(tmem_base + NB * 128, tmem_base + (uint32_t)(sb * LA_BN + (kk >> 1) * 32 + half * 16 + (kk & 1) * 8),
                         desc_at(v_t, kk * 2048), idesc_o, (j | half | kk) != 0);
        umma_commit(o_full);
        umma_commit(&v_empty[s]);
        if (NB == 1 && j + 1 < n_kv) ok = issue_s(j + 1);  // takes the place of the probabilities just consumed
      }
    }
    __syncwarp();
  } else {
    // ---------------- softmax: one thread per query row ----------------
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    const int q_pos = q_first + r;
    const bool row_ok = q_pos < len;
    const int k_max = row_ok ? q_pos : -1;
    const int k_min = p.window > 0 ? max(0, q_pos - p.window + 1) : 0;
    const uint32_t to = tmem_base + lane_off + NB * 128;
    float m_ref = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv && ok; ++j) {
      const int s = j % NB;
      const int key0 = tile_at(j) * LA_BN, width = width_at(j);
      const bool mean = p.pool > 0 && j < kt;
      const bool full = mean ? q_first + LA_BM <= len && key0 + LA_BN <= max(0, q_first - p.window + 1) / p.pool
                             : width == LA_BN && q_first + LA_BM <= len && key0 + LA_BN - 1 <= q_first &&
                        (p.window <= 0 || key0 >= q_first + LA_BM - p.window || key0 + LA_BN <= p.keep);
      ok = __all_sync(0xffffffffu, mbar_wait(&s_full[s], (uint32_t)((j / NB) & 1), abort_flag, p.status, 1270 + s));
      if (!ok) break;
      tc_fence_after();
      const uint32_t ts = tmem_base + lane_off + (uint32_t)s * LA_BN;
      const int first = (mean ? 0 : k_min) - key0, last = (mean ? (row_ok ? k_min / p.pool : 0) - 1 : k_max) - key0, kept = p.keep - key0;
      const float2 top = full ? la_row_max<CAP, true>(ts, width, first, last, kept) : la_row_max<CAP, false>(ts, width, first, last, kept);
      const float mx = top.x;
      int level = -1;
      float m_tile = mx * p.scale_log2;
      if (CAP) {
        level = !__any_sync(0xffffffffu, top.y > p.near7) ? 0 : !__any_sync(0xffffffffu, top.y > p.near11) ? 1 : 2;
        m_tile = mx == -INFINITY ? mx : level == 0 ? la_capped<0>(p, mx) : level == 1 ? la_capped<1>(p, mx) : la_capped<2>(p, mx);
      }
      float alpha = 1.f;
      bool moved = false;
      if (m_ref == -INFINITY) {
        m_ref = m_tile;  // nothing seen so far: the row of O is zero (or meaningless only through zero weights)
      } else if (m_tile > m_ref + 8.f) {
        alpha = fast_exp2(m_ref - m_tile);
        m_ref = m_tile;
        moved = true;
      }
      if (j > 0 && __any_sync(0xffffffffu, moved)) {
        ok = __all_sync(0xffffffffu, mbar_wait(o_full, (uint32_t)((j - 1) & 1), abort_flag, p.status, 1290));
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < p.vdim; c += 16) {
          float o[16];
          tmem_ld_32x16(to + c, o);
          tmem_ld_wait();
          uint32_t w[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) w[i] = __float_as_uint(o[i] * alpha);
          tmem_st_32x16(to + c, w);
        }
      }
      l_run *= alpha;
      const float neg_m = m_ref == -INFINITY ? 0.f : -m_ref;
      float sum;
      if (!CAP) sum = full ? la_probs<-1, true>(p, ts, width, neg_m, first, last, kept) : la_probs<-1, false>(p, ts, width, neg_m, first, last, kept);
      else if (level == 0) sum = full ? la_probs<0, true>(p, ts, width, neg_m, first, last, kept) : la_probs<0, false>(p, ts, width, neg_m, first, last, kept);
      else if (level == 1) sum = la_probs<1, false>(p, ts, width, neg_m, first, last, kept);
      else sum = la_probs<2, false>(p, ts, width, neg_m, first, last, kept);
      // P.V(last) completes phase `last` of o_full, and may do so before this thread looks: phase last - 1 has to be seen
      // first.  (With one S buffer the last S was issued after P.V(last - 1), so s_full has shown it.)
      if (NB == 2 && j > 0 && j == n_kv - 1)
        ok = __all_sync(0xffffffffu, mbar_wait(o_full, (uint32_t)((j - 1) & 1), abort_flag, p.status, 1294));
      tc_fence_before();
      mbar_arrive(&p_full[s]);
      l_run += sum;
    }
    if (ok) {
      const int last = n_kv - 1;
      ok = __all_sync(0xffffffffu, mbar_wait(o_full, (uint32_t)(last & 1), abort_flag, p.status, 1295));
      if (ok) {
        tc_fence_after();
        float f = 0.f;
        __nv_bfloat16* dst = nullptr;
        const __nv_bfloat16* gl = nullptr;
        if (row_ok) {
          const size_t t = (size_t)(beg + q_pos), th = t * p.heads + h;
          const float sk = p.sink != nullptr ? p.sink[h] * 1.4426950408889634f : -INFINITY, mt = fmaxf(m_ref, sk);
          const float wm = fast_exp2(m_ref - mt);
          f = p.out_scale * wm / (l_run * wm + fast_exp2(sk - mt));
          if (p.gate_mode == GATE_HEAD) f *= reinterpret_cast<const float*>(p.gate)[th];
          if (p.gate_mode == GATE_LOGITS) gl = reinterpret_cast<const __nv_bfloat16*>(p.gate) + t * p.gate_ld + (size_t)h * p.vdim;
          dst = p.out + t * p.out_ld + (size_t)h * p.vdim;
        }
#pragma unroll 1
        for (int c = 0; c < p.vdim; c += 32) {
          uint4 g[4];
          if (gl != nullptr) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
              if (c + 8 * i < p.vdim) g[i] = *reinterpret_cast<const uint4*>(gl + c + 8 * i);
          }
          float o[2][16];
          tmem_ld_32x16(to + c, o[0]);
          tmem_ld_32x16(to + (c + 16 < p.vdim ? c + 16 : c), o[1]);
          tmem_ld_wait();
          if (row_ok) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              if (c + 8 * i >= p.vdim) break;
              float* x = &o[i >> 1][8 * (i & 1)];
#pragma unroll
              for (int q = 0; q < 8; ++q) x[q] *= f;
              if (gl != nullptr) {
                const uint32_t w[4] = {g[i].x, g[i].y, g[i].z, g[i].w};
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                  const float2 z = unpack_bf16(w[q]);
                  x[2 * q] *= fast_sigmoid(z.x);
                  x[2 * q + 1] *= fast_sigmoid(z.y);
                }
              }
              *reinterpret_cast<uint4*>(dst + c + 8 * i) =
                  make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
            }
          }
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
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, NB * 256);
  }
}

}  // namespace trlb

using namespace trlb;

namespace {

size_t la_smem(int nk, int nv, int ks, int vs) { return (size_t)(nk + ks * nk + vs * nv) * LA_BOX + 1024 + 256; }

// Deepest rings that fit shared memory; false: not even one stage each.
bool la_stages(int nk, int nv, int& ks, int& vs) {
  constexpr int opt[6][2] = {{3, 3}, {3, 2}, {2, 2}, {2, 1}, {1, 1}, {0, 0}};
  for (int i = 0; opt[i][0]; ++i)
    if (la_smem(nk, nv, opt[i][0], opt[i][1]) <= 227 * 1024) { ks = opt[i][0]; vs = opt[i][1]; return true; }
  return false;
}

int la_boxes(int n) { return (n + 63) / 64; }

// Two CTAs per SM: 227 KB of shared memory in halves, each with the kilobyte the system takes.
bool la_pair(int nk, int nv, int vdim) { return vdim <= 128 && la_smem(nk, nv, 1, 1) <= 112 * 1024; }

}  // namespace

// 1 when trlb_mixer_attn_tc takes these sizes.
TRLB_API int trlb_mixer_attn_tc_ok(int heads, int kv_heads, int dim, int rot, int vdim) {
  int ks, vs;
  return dim > 0 && rot >= 0 && vdim > 0 && dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && vdim <= 256 && heads > 0 &&
         kv_heads > 0 && heads % kv_heads == 0 && la_stages(la_boxes(dim) + la_boxes(rot), la_boxes(vdim), ks, vs);
}

// q [T rows of q_ld]: heads x (dim + rot), rotated part last; k, v [T rows of k_ld / v_ld]: kv_heads x dim / vdim; krot [T rows
// of krot_ld]: the shared rotated keys (rot > 0).  All bf16, rows on 16 bytes.  window <= 0: unlimited, else the first `keep` keys stay
// visible; cap <= 0: none; scale > 0;
// pool > 0 (with a window, without rot and keep): pk, pv [T / pool + 1, kv_heads, dim / vdim], means as trlb_pool_blocks leaves them;
// out [T rows of out_ld on 16 bytes], times out_scale; sink may be null; gate by gate_mode (0 none, 1 fp32 [T, heads], 2 bf16 logits [T rows of gate_ld]).
TRLB_API int trlb_mixer_attn_tc(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld,
                                const void* krot, long long krot_ld, const int* cu, int n_seq, int T, int heads, int kv_heads,
                                int dim, int rot, int vdim, int window, int keep, float scale, float cap, const float* sink,
                                int gate_mode, const void* gate, long long gate_ld, int pool, const void* pk, const void* pv, void* out,
                                long long out_ld, float out_scale, int* status, cudaStream_t st) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (!trlb_mixer_attn_tc_ok(heads, kv_heads, dim, rot, vdim) || (q_ld % 8) || (k_ld % 8) || (v_ld % 8) || !(scale > 0.f)) return -210;
  if (rot > 0 && (krot_ld % 8)) return -210;
  if ((out_ld % 8) || (reinterpret_cast<uintptr_t>(out) & 15) || (pool > 0 && (pk == nullptr || pv == nullptr || keep > 0 || rot > 0))) return -210;
  if (gate_mode == GATE_LOGITS && ((gate_ld % 8) || (reinterpret_cast<uintptr_t>(gate) & 15))) return -210;
  MixerAttnTc p = {};
  p.cu = cu; p.n_seq = n_seq; p.heads = heads; p.group = heads / kv_heads; p.dim = dim; p.rot = rot; p.vdim = vdim; p.window = window; p.keep = window > 0 && keep > 0 ? keep : 0;
  p.pool = window > 0 && pool > 0 ? pool : 0;
  p.nn = la_boxes(dim); p.nr = la_boxes(rot); p.nv = la_boxes(vdim);
  const bool pair = la_pair(p.nn + p.nr, p.nv, vdim);
  if (pair) p.k_stages = p.v_stages = 1;
  else la_stages(p.nn + p.nr, p.nv, p.k_stages, p.v_stages);
  p.scale_log2 = cap > 0.f ? 1.f : scale * 1.4426950408889634f;
  p.cap_in = cap > 0.f ? scale / cap : 0.f;
  p.cap_out = cap * 1.4426950408889634f;
  if (cap > 0.f) {
    const double t[6] = {1.0, -1.0 / 3, 2.0 / 15, -17.0 / 315, 62.0 / 2835, -1382.0 / 155925}, in = (double)scale / cap;
    double f = (double)cap * 1.4426950408889634 * in;
    for (int i = 0; i < 6; ++i, f *= in * in) p.poly[i] = (float)(t[i] * f);
    p.near7 = (float)(0.12 / in);   // the first term left out is below 1e-9 of tanh
    p.near11 = (float)(0.35 / in);  // below 2e-8
  }
  p.sink = sink; p.gate_mode = gate_mode; p.gate = gate; p.gate_ld = gate_ld; p.out = (__nv_bfloat16*)out; p.out_ld = out_ld; p.out_scale = out_scale; p.status = status;
  const __nv_bfloat16* qb = (const __nv_bfloat16*)q;
  const int dq = dim + rot;
  CUtensorMap tqn, tqr, tkn, tkr, tv, tpk, tpv;
  using trlb_host::make_tmap_3d_bf16;
  if (make_tmap_3d_bf16(&tqn, qb, dim, heads, T, dq, (uint64_t)q_ld, 64, 1, 128)) return -211;
  if (make_tmap_3d_bf16(&tkn, k, dim, kv_heads, T, dim, (uint64_t)k_ld, 64, 1, 128)) return -213;
  if (make_tmap_3d_bf16(&tv, v, vdim, kv_heads, T, vdim, (uint64_t)v_ld, 64, 1, 128)) return -215;
  tqr = tqn;
  tkr = tkn;
  tpk = tkn;
  tpv = tv;
  if (p.pool > 0) {
    const uint64_t rows = (uint64_t)(T / pool + 1);
    if (make_tmap_3d_bf16(&tpk, pk, dim, kv_heads, rows, dim, (uint64_t)kv_heads * dim, 64, 1, 128)) return -217;
    if (make_tmap_3d_bf16(&tpv, pv, vdim, kv_heads, rows, vdim, (uint64_t)kv_heads * vdim, 64, 1, 128)) return -218;
  }
  if (rot > 0) {
    if (make_tmap_3d_bf16(&tqr, qb + dim, rot, heads, T, dq, (uint64_t)q_ld, 64, 1, 128)) return -212;
    if (trlb_host::make_tmap_2d_bf16(&tkr, krot, T, rot, (uint64_t)krot_ld, 128, 64)) return -214;
  }
  using Kern = void (*)(const CUtensorMap, const CUtensorMap, const CUtensorMap, const CUtensorMap, const CUtensorMap, const CUtensorMap,
                        const CUtensorMap, const MixerAttnTc);
  static const Kern kerns[4] = {mixer_attn_tc_kernel<false, 1>, mixer_attn_tc_kernel<true, 1>, mixer_attn_tc_kernel<false, 2>,
                                mixer_attn_tc_kernel<true, 2>};
  static bool attr_set = false;
  if (!attr_set) {
    for (Kern k : kerns)
      if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -216;
    attr_set = true;
  }
  const dim3 grid((T + LA_BM - 1) / LA_BM + n_seq, heads);
  const size_t smem = la_smem(p.nn + p.nr, p.nv, p.k_stages, p.v_stages);
  kerns[(pair ? 0 : 2) + (cap > 0.f)]<<<grid, LA_THREADS, smem, st>>>(tqn, tqr, tkn, tkr, tv, tpk, tpv, p);
  return (int)cudaGetLastError();
}
