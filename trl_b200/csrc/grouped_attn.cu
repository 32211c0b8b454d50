// Grouped-query attention of the layered decoders: preparation of queries, keys and values, and attention on the CUDA
// cores for every size and dtype (tcgen05 forms: mixer_attn_tcgen05.cu for prompts, grouped_decode_tcgen05.cu for decode).
//
// T is the model dtype (bf16 or fp32); norms, scores, softmax and its sums are fp32 in both.  Compiled without fast-math
// (csrc/build.py: EXACT_MATH).  In decode kernels seq_lens[slot] is the position of the slot's new token, negative: idle.
#include "mixers.cuh"

namespace trlb {

// ------------------------------------------------------------------------------------------------------------
// From the projections of a layer's input, rows [q | k | v | g] (no k and v in a layer that reads another one's cache, no v
// where the projected keys are the values, g per element, per head or absent): queries and keys divided (or not) by their rms, of a
// head or (WHOLE) of all heads, times a weight; queries times the temperature of their position and a factor per head; both
// rotated; keys and values to the paged cache.  With pools (decode) the token that completes a block of `pool` leaves the means
// of the block's keys and values, as the cache holds them, in the slot's rows of means.  S is the dtype of the rows: T (prompt: v and g per element stay where they are, q is replaced in
// place, k too unless k_out is given) or fp32 sums (decode: q and the gate logits go to buffers, everything read is zeroed).
// Gates per head leave as sigmoids.  One warp per (row, head of q / k / v / g or all gates of heads); WHOLE: one block per row.
// ------------------------------------------------------------------------------------------------------------
enum { GATES_NONE = 0, GATES_HEAD = 1, GATES_ELEMENT = 2 };

struct AttnPrep {
  long long ld;
  int rows, heads, kv_heads, dim, vdim, has_kv, has_v, gates;
  float eps;
  const int* positions;   // [rows]
  const int* tok_slot;    // [rows] or null (slot = row)
  const float* temp;      // [temp_len] factor of the query by position, or null
  int temp_len;
  const float* q_w;       // norm weights, [dim] or (WHOLE) [heads dim] / [kv_heads dim]; null: none
  const float* k_w;
  int rot, halves;        // rotated elements of a head; pairs (i, i + rot / 2) instead of (2 i, 2 i + 1)
  const float2* table;    // [table_len, rot / 2] (cos, sin) with the rotation's magnitude folded in
  int table_len;
  float* head_gate;       // [rows, heads]
  const int* block_table;  // null: no cache
  int max_blocks, block_size;
  int unit;                // 0: queries and keys are not normed
  const float* q_head;     // [heads] or null
  int pool, pool_rows;     // 0: no pools; rows of means per slot
  void* pool_k;            // [slots, pool_rows, kv_heads, dim] of T
  void* pool_v;            // [slots, pool_rows, kv_heads, vdim] of T
};

// Row of the cache that holds the token at `pos` of a slot.
__device__ __forceinline__ long long cache_row(const AttnPrep& p, int slot, int pos) {
  return (long long)p.block_table[(size_t)slot * p.max_blocks + pos / p.block_size] * p.block_size + pos % p.block_size;
}
// Whether the token at `pos` completes a block whose means have a row.
__device__ __forceinline__ bool completes(const AttnPrep& p, int pos) {
  return p.pool > 0 && (pos + 1) % p.pool == 0 && pos / p.pool < p.pool_rows;
}

template <typename T, typename S, bool WHOLE>
__global__ void __launch_bounds__(WHOLE ? 512 : 256)
attn_prep_kernel(const AttnPrep p, S* __restrict__ src, T* __restrict__ q_out, T* __restrict__ k_out, T* __restrict__ g_out,
                 T* __restrict__ k_cache, T* __restrict__ v_cache) {
  constexpr bool SUMS = !(sizeof(T) == 2 && sizeof(S) == 2);  // fp32 models: q_out tells (null: in place)
  __shared__ float red[WHOLE ? 64 : 1];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const bool in_place = !SUMS || q_out == nullptr;
  const int kv = p.has_kv ? p.kv_heads : 0, vv = p.has_v ? kv : 0;
  const int ge = p.gates == GATES_ELEMENT && !in_place ? p.heads : 0;
  const int units = p.heads + kv + vv + ge + (p.gates == GATES_HEAD ? 1 : 0);
  const int q_n = p.heads * p.dim, k_n = kv * p.dim, v_n = vv * p.vdim;
  int row, u, u_end, u_step;
  float sq = 0.f, sk = 0.f;  // WHOLE: 1 / rms of all queries, of all keys
  if (WHOLE) {
    row = blockIdx.x;
    u = threadIdx.x >> 5;
    u_end = units;
    u_step = blockDim.x >> 5;
    const S* r = src + (size_t)row * p.ld;
    const bool v4 = ((q_n | k_n | (int)p.ld) & 3) == 0 && (reinterpret_cast<uintptr_t>(src) & (4 * sizeof(S) - 1)) == 0;
    if (v4) {
      for (int j = 4 * threadIdx.x; j < q_n + k_n; j += 4 * blockDim.x) {
        const float4 v = load4(r + j);
        const float ss = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        if (j < q_n) sq += ss; else sk += ss;
      }
    } else {
      for (int j = threadIdx.x; j < q_n + k_n; j += blockDim.x) {
        const float v = to_f(r[j]);
        if (j < q_n) sq += v * v; else sk += v * v;
      }
    }
    const float2 s = block_sum2(sq, sk, red);  // a barrier: the row is replaced below
    sq = 1.f / sqrtf(s.x / (float)q_n + p.eps);
    sk = k_n > 0 ? 1.f / sqrtf(s.y / (float)k_n + p.eps) : 0.f;
  } else {
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (item >= (long long)p.rows * units) return;
    row = (int)(item / units);
    u = (int)(item % units);
    u_end = u + 1;
    u_step = 1;
  }
  const int pos = p.positions[row];
  S* r = src + (size_t)row * p.ld;
  long long at = -1;   // token's row in the cache
  const int slot = p.tok_slot ? p.tok_slot[row] : row;
  if (pos >= 0 && p.block_table != nullptr && slot >= 0 && pos / p.block_size < p.max_blocks) at = cache_row(p, slot, pos);
  const float2* cs = p.rot > 0 && pos >= 0 && pos < p.table_len ? p.table + (size_t)pos * (p.rot / 2) : nullptr;
  for (; u < u_end; u += u_step) {
    if (p.gates == GATES_HEAD && u == units - 1) {
      S* g = r + q_n + k_n + v_n;
      for (int h = lane; h < p.heads; h += 32) {
        p.head_gate[(size_t)row * p.heads + h] = sigmoid_f(to_f(g[h]));
        if (!in_place) g[h] = from_f<S>(0.f);
      }
      continue;
    }
    S* x;
    int n;
    bool normed = false;
    float mul = 1.f, s = 1.f;
    const float* w = nullptr;
    T* dst = nullptr;    // besides the cache
    T* paged = nullptr;
    T* raw = nullptr;    // cache row that gets the elements as they are
    bool put = false;    // back into the row
    if (u < p.heads) {
      x = r + (size_t)u * p.dim;
      n = p.dim;
      normed = true;
      w = p.q_w == nullptr ? nullptr : WHOLE ? p.q_w + (size_t)u * p.dim : p.q_w;
      s = sq;
      if (p.temp != nullptr && pos >= 0 && pos < p.temp_len) mul = p.temp[pos];
      if (p.q_head != nullptr) mul *= p.q_head[u];
      if (!in_place) dst = q_out + ((size_t)row * p.heads + u) * p.dim;
      put = in_place;
    } else if (u < p.heads + kv) {
      const int h = u - p.heads;
      x = r + q_n + (size_t)h * p.dim;
      n = p.dim;
      normed = true;
      w = p.k_w == nullptr ? nullptr : WHOLE ? p.k_w + (size_t)h * p.dim : p.k_w;
      s = sk;
      if (k_out != nullptr) dst = k_out + ((size_t)row * kv + h) * p.dim;
      if (at >= 0) {
        paged = k_cache + (size_t)(at * kv + h) * p.dim;
        if (vv == 0) raw = v_cache + (size_t)(at * kv + h) * p.dim;
      }
      put = in_place && k_out == nullptr;
    } else if (u < p.heads + kv + vv) {
      const int h = u - p.heads - kv;
      x = r + q_n + k_n + (size_t)h * p.vdim;
      n = p.vdim;
      if (at >= 0) paged = v_cache + (size_t)(at * kv + h) * p.vdim;
    } else {
      const int h = u - p.heads - kv - vv;
      x = r + q_n + k_n + v_n + (size_t)h * p.vdim;
      n = p.vdim;
      dst = g_out + ((size_t)row * p.heads + h) * p.vdim;
    }
    const int rot = normed ? p.rot : 0;
    const bool vec = ((n | (int)p.ld | (int)(x - r)) & 3) == 0 && (reinterpret_cast<uintptr_t>(src) & (4 * sizeof(S) - 1)) == 0 &&
                     (rot & (p.halves ? 7 : 3)) == 0;
    if (!p.unit) {
      s = 1.f;
    } else if (normed && !WHOLE) {
      float ss = 0.f;
      if (vec) {
        for (int j = 4 * lane; j < n; j += 128) {
          const float4 v = load4(x + j);
          ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
      } else {
        for (int j = lane; j < n; j += 32) ss += to_f(x[j]) * to_f(x[j]);
      }
      s = 1.f / sqrtf(warp_sum(ss) / (float)n + p.eps);
    }
    if (normed) s *= mul; else s = 1.f;
    if (vec) {
      auto get = [&](int j) {
        float4 v = load4(x + j);
        if (raw) store4(raw + j, v);
        v = make_float4(v.x * s, v.y * s, v.z * s, v.w * s);
        if (w != nullptr) {
          const float4 g = load4(w + j);
          v = make_float4(v.x * g.x, v.y * g.y, v.z * g.z, v.w * g.w);
        }
        return v;
      };
      auto set = [&](int j, float4 v) {
        if (dst) store4(dst + j, v);
        if (paged) store4(paged + j, v);
        if (!in_place) store4(x + j, make_float4(0.f, 0.f, 0.f, 0.f));
        else if (put) store4(x + j, v);
      };
      if (rot > 0 && p.halves) {
        const int half = rot / 2;
        for (int i = 4 * lane; i < half; i += 128) {
          const float4 a = get(i), b = get(i + half);
          float2 c[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) c[k] = cs != nullptr ? cs[i + k] : make_float2(1.f, 0.f);
          set(i, make_float4(a.x * c[0].x - b.x * c[0].y, a.y * c[1].x - b.y * c[1].y, a.z * c[2].x - b.z * c[2].y, a.w * c[3].x - b.w * c[3].y));
          set(i + half, make_float4(b.x * c[0].x + a.x * c[0].y, b.y * c[1].x + a.y * c[1].y, b.z * c[2].x + a.z * c[2].y, b.w * c[3].x + a.w * c[3].y));
        }
        for (int j = rot + 4 * lane; j < n; j += 128) set(j, get(j));
      } else {
        for (int j = 4 * lane; j < n; j += 128) {
          float4 v = get(j);
          if (j < rot && cs != nullptr) {
            const float2 c0 = cs[j / 2], c1 = cs[j / 2 + 1];
            v = make_float4(v.x * c0.x - v.y * c0.y, v.y * c0.x + v.x * c0.y, v.z * c1.x - v.w * c1.y, v.w * c1.x + v.z * c1.y);
          }
          set(j, v);
        }
      }
    } else {
      auto get = [&](int j) {
        const float v = to_f(x[j]);
        if (raw) raw[j] = from_f<T>(v);
        return w != nullptr ? v * s * w[j] : v * s;
      };
      auto set = [&](int j, float v) {
        if (dst) dst[j] = from_f<T>(v);
        if (paged) paged[j] = from_f<T>(v);
        if (!in_place) x[j] = from_f<S>(0.f);
        else if (put) x[j] = from_f<S>(v);
      };
      for (int i = lane; i < rot / 2; i += 32) {
        const int ia = p.halves ? i : 2 * i, ib = p.halves ? i + rot / 2 : 2 * i + 1;
        const float a = get(ia), b = get(ib);
        const float2 c = cs != nullptr ? cs[i] : make_float2(1.f, 0.f);
        set(ia, a * c.x - b * c.y);
        set(ib, b * c.x + a * c.y);
      }
      for (int j = rot + lane; j < n; j += 32) set(j, get(j));
    }
    if (paged != nullptr && completes(p, pos)) {
      // the block's rows, this one included, as the cache holds them
      const int h = normed ? u - p.heads : u - p.heads - kv;
      const T* cache = normed ? k_cache : v_cache;
      T* mean = reinterpret_cast<T*>(normed ? p.pool_k : p.pool_v) + (((size_t)slot * p.pool_rows + pos / p.pool) * kv + h) * n;
      __syncwarp();
      for (int j = lane; j < n; j += 32) {
        float sum = 0.f;
        for (int t = pos - p.pool + 1; t <= pos; ++t) sum += to_f(cache[(size_t)(cache_row(p, slot, t) * kv + h) * n + j]);
        mean[j] = from_f<T>(sum / (float)p.pool);
      }
    }
  }
}

// The same for sizes in multiples of 8 with heads of at most 256 elements: one block per row, 2^lanes_log2 threads with 8 elements
// each per head, so that a row is read once into registers (also for norms over all heads) and moves in 16-byte pieces.  A block
// takes its row in at most ROUNDS rounds.

__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = load4(p), b = load4(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = unpack_bf16(w[i]);
    v[2 * i] = f.x;
    v[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  store4(p, make_float4(v[0], v[1], v[2], v[3]));
  store4(p + 4, make_float4(v[4], v[5], v[6], v[7]));
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}

template <typename T, typename S, bool WHOLE, int ROUNDS>
__global__ void __launch_bounds__(512)
attn_prep_rows_kernel(const AttnPrep p, int lanes_log2, S* __restrict__ src, T* __restrict__ q_out, T* __restrict__ k_out,
                      T* __restrict__ g_out, T* __restrict__ k_cache, T* __restrict__ v_cache) {
  constexpr bool SUMS = !(sizeof(T) == 2 && sizeof(S) == 2);
  __shared__ float red[WHOLE ? 64 : 1];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, lanes = 1 << lanes_log2, c = threadIdx.x & (lanes - 1), j0 = 8 * c;
  const bool in_place = !SUMS || q_out == nullptr;
  const int kv = p.has_kv ? p.kv_heads : 0, vv = p.has_v ? kv : 0, ge = p.gates == GATES_ELEMENT && !in_place ? p.heads : 0;
  const int units = p.heads + kv + vv + ge;
  const int q_n = p.heads * p.dim, k_n = kv * p.dim, v_n = vv * p.vdim;
  S* r = src + (size_t)row * p.ld;
  const int per_round = blockDim.x >> lanes_log2, u0 = threadIdx.x >> lanes_log2;
  // where head u starts in the row
  auto place = [&](int u) {
    if (u < p.heads + kv) return u * p.dim;
    return q_n + k_n + (u - p.heads - kv) * p.vdim;
  };
  float x[ROUNDS][8];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < ROUNDS; ++i) {
    const int u = u0 + i * per_round;
    const bool on = u < units && j0 < (u < p.heads + kv ? p.dim : p.vdim);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[i][e] = 0.f;
    if (on) load8(r + place(u) + j0, x[i]);
    if (WHOLE && on && u < p.heads + kv) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[i][e] * x[i][e];
      if (u < p.heads) sq += ss; else sk += ss;
    }
  }
  if (WHOLE) {
    const float2 s = block_sum2(sq, sk, red);
    sq = 1.f / sqrtf(s.x / (float)q_n + p.eps);
    sk = k_n > 0 ? 1.f / sqrtf(s.y / (float)k_n + p.eps) : 0.f;
  }
  const int pos = p.positions[row];
  long long at = -1;
  const int slot = p.tok_slot ? p.tok_slot[row] : row;
  if (pos >= 0 && p.block_table != nullptr && slot >= 0 && pos / p.block_size < p.max_blocks) at = cache_row(p, slot, pos);
  // this thread's angles are the same in every head
  const bool turns = j0 < p.rot && pos >= 0 && pos < p.table_len;
  const int half = p.rot / 2, shift = half / 8;  // halves: the partner is `shift` threads away
  const bool upper = j0 >= half;
  const int partner = (threadIdx.x & 31) + (j0 >= p.rot ? 0 : upper ? -shift : shift);
  float2 cs[8];
  if (turns) {
    const float2* t = p.table + (size_t)pos * half + (p.halves ? (upper ? j0 - half : j0) : j0 / 2);
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (e < 4 || p.halves) cs[e] = t[e];
  }
#pragma unroll
  for (int i = 0; i < ROUNDS; ++i) {
    if (i * per_round >= units) break;  // uniform
    const int u = u0 + i * per_round;
    const bool normed = u < p.heads + kv, is_q = u < p.heads;
    const bool on = u < units && j0 < (normed ? p.dim : p.vdim);
    T* dst = nullptr;
    T* paged = nullptr;
    bool put = false;
    if (on) {
      if (is_q) {
        if (!in_place) dst = q_out + ((size_t)row * p.heads + u) * p.dim;
        put = in_place;
      } else if (normed) {
        const int h = u - p.heads;
        if (k_out != nullptr) dst = k_out + ((size_t)row * kv + h) * p.dim;
        put = in_place && k_out == nullptr;
        if (at >= 0) {
          paged = k_cache + (size_t)(at * kv + h) * p.dim;
          if (vv == 0) store8(v_cache + (size_t)(at * kv + h) * p.dim + j0, x[i]);
        }
      } else if (u < p.heads + kv + vv) {
        if (at >= 0) paged = v_cache + (size_t)(at * kv + u - p.heads - kv) * p.vdim;
      } else {
        dst = g_out + ((size_t)row * p.heads + u - p.heads - kv - vv) * p.vdim;
      }
    }
    float s = WHOLE && p.unit ? (is_q ? sq : sk) : 1.f;
    if (!WHOLE && p.unit) {  // uniform
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[i][e] * x[i][e];
      for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      s = 1.f / sqrtf(ss / (float)p.dim + p.eps);
    }
    if (normed) {
      if (is_q && p.temp != nullptr && pos >= 0 && pos < p.temp_len) s *= p.temp[pos];
      if (is_q && p.q_head != nullptr) s *= p.q_head[u];
      const float* w = is_q ? p.q_w : p.k_w;
      if (on && w != nullptr) {
        float g[8];
        load8(w + (WHOLE ? (size_t)(is_q ? u : u - p.heads) * p.dim : 0) + j0, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[i][e] *= s * g[e];
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) x[i][e] *= s;
      }
    }
    if (p.rot > 0 && p.halves) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {  // every lane takes part
        const float other = __shfl_sync(0xffffffffu, x[i][e], partner);
        if (turns && normed) x[i][e] = x[i][e] * cs[e].x + (upper ? other : -other) * cs[e].y;
      }
    } else if (turns && normed) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float a = x[i][2 * e], b = x[i][2 * e + 1];
        x[i][2 * e] = a * cs[e].x - b * cs[e].y;
        x[i][2 * e + 1] = b * cs[e].x + a * cs[e].y;
      }
    }
    if (on) {
      if (dst) store8(dst + j0, x[i]);
      if (paged) store8(paged + j0, x[i]);
      if (paged && completes(p, pos)) {
        const int h = normed ? u - p.heads : u - p.heads - kv, n = normed ? p.dim : p.vdim;
        const T* cache = (normed ? k_cache : v_cache) + (size_t)h * n + j0;
        float mean[8], v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) mean[e] = to_f(from_f<T>(x[i][e]));
        for (int t = pos - p.pool + 1; t < pos; ++t) {
          load8(cache + (size_t)(cache_row(p, slot, t) * kv) * n, v);
#pragma unroll
          for (int e = 0; e < 8; ++e) mean[e] += v[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) mean[e] /= (float)p.pool;
        store8(reinterpret_cast<T*>(normed ? p.pool_k : p.pool_v) + (((size_t)slot * p.pool_rows + pos / p.pool) * kv + h) * n + j0, mean);
      }
      if (!in_place) {
        const float zero[8] = {};
        store8(r + place(u) + j0, zero);
      } else if (put) {
        store8(r + place(u) + j0, x[i]);
      }
    }
  }
  if (p.gates == GATES_HEAD) {
    S* g = r + q_n + k_n + v_n;
    for (int h = threadIdx.x; h < p.heads; h += blockDim.x) {
      p.head_gate[(size_t)row * p.heads + h] = sigmoid_f(to_f(g[h]));
      if (!in_place) g[h] = from_f<S>(0.f);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// Means of blocks of P rows of packed keys and values (fp32 sums).  The blocks of the sequence that starts at token a are rows
// a / P + block of pk and pv (no two sequences meet there); rows of no block are zeros.  With slots also to the slots' rows.
// grid: (rows, slices of the columns).
// ------------------------------------------------------------------------------------------------------------
struct PoolBlocks {
  const int* cu;
  int n_seq, P, k_n, v_n;
  long long k_ld, v_ld;
  const int* seq_slot;   // [n_seq] or null
  int slots, slot_rows;
};

template <typename T>
__global__ void __launch_bounds__(128)
pool_blocks_kernel(const PoolBlocks p, const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ pk, T* __restrict__ pv,
                   T* __restrict__ slot_k, T* __restrict__ slot_v) {
  const int r = blockIdx.x;
  int seq = -1, beg = 0, b = 0;
  for (int s = 0; s < p.n_seq; ++s) {
    beg = p.cu[s];
    b = r - beg / p.P;
    if (b >= 0 && b < (p.cu[s + 1] - beg) / p.P) { seq = s; break; }
  }
  const int slot = seq >= 0 && p.seq_slot != nullptr && b < p.slot_rows ? p.seq_slot[seq] : -1;
  const bool kept = slot >= 0 && slot < p.slots;
  const size_t t0 = (size_t)beg + (size_t)b * p.P;
  const int n = p.k_n + p.v_n;
  const bool v4 = ((p.k_n | p.v_n | (int)(p.k_ld & 3) | (int)(p.v_ld & 3)) & 3) == 0 &&
                  ((reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & (4 * sizeof(T) - 1)) == 0;
  const float inv = 1.f / (float)p.P;
  const int vec = v4 ? 4 : 1;
  for (int c = vec * (blockIdx.y * blockDim.x + threadIdx.x); c < n; c += vec * gridDim.y * blockDim.x) {
    const bool key = c < p.k_n;
    const int j = key ? c : c - p.k_n, m = key ? p.k_n : p.v_n;
    const T* src = (key ? k : v) + t0 * (key ? p.k_ld : p.v_ld) + j;
    const long long ld = key ? p.k_ld : p.v_ld;
    T* dst = (key ? pk : pv) + (size_t)r * m + j;
    T* held = kept ? (key ? slot_k : slot_v) + ((size_t)slot * p.slot_rows + b) * m + j : nullptr;
    if (v4) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (seq >= 0) {
#pragma unroll 8
        for (int t = 0; t < p.P; ++t) {
          const float4 x = load4(src + (size_t)t * ld);
          a = make_float4(a.x + x.x, a.y + x.y, a.z + x.z, a.w + x.w);
        }
        a = make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv);
      }
      store4(dst, a);
      if (held) store4(held, a);
    } else {
      float a = 0.f;
      if (seq >= 0)
        for (int t = 0; t < p.P; ++t) a += to_f(src[(size_t)t * ld]);
      *dst = from_f<T>(a * inv);
      if (held) *held = from_f<T>(a * inv);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// Prompt attention, any size: one warp per (token, head).  Keys of token t are rows t - min(pos, window - 1) .. t of the
// packed stream (pos counts from the token's own sequence start), so no sequence table is needed.  Keys may have a second
// part of `rot` elements shared by the heads; scores may be capped; sink and gate may be null.  With a window the first `keep`
// keys of the sequence stay visible, or the means of the blocks before it (rows of pk, pv as pool_blocks_kernel leaves them): the
// keys of a token are a list of those before the window, then the window.
// ------------------------------------------------------------------------------------------------------------
struct MixerAttn {
  int T, heads, group, dim, rot, vdim, window, keep;
  long long q_ld, k_ld, v_ld, kr_ld, gate_ld;
  float scale, cap;
  const int* positions;
  const float* sink;       // [heads] or null
  int gate_mode;           // 0 none, 1 fp32 [T, heads], 2 logits of T [T rows of gate_ld]
  const float* head_gate;
  int pool;                // 0: no blocks
  long long out_ld;
  float out_scale;
};

__device__ __forceinline__ float capped(float s, float cap) { return cap > 0.f ? cap * tanhf(s / cap) : s; }

template <typename T>
__global__ void __launch_bounds__(128)
mixer_attn_kernel(const MixerAttn p, const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                  const T* __restrict__ krot, const T* __restrict__ gate, const T* __restrict__ pk, const T* __restrict__ pv,
                  T* __restrict__ out) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * 4 + warp;
  if (item >= (long long)p.T * p.heads) return;
  const int t = (int)(item / p.heads), h = (int)(item % p.heads), hk = h / p.group;
  const int dq = p.dim + p.rot;
  float* qs = sm + (size_t)warp * (dq + p.vdim);
  float* os = qs + dq;
  for (int d = lane; d < dq; d += 32) qs[d] = to_f(q[(size_t)t * p.q_ld + (size_t)h * dq + d]);
  for (int e = lane; e < p.vdim; e += 32) os[e] = 0.f;
  __syncwarp();
  const int pos = p.positions[t];
  const int start = t - pos, lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, kept = p.pool > 0 ? lo / p.pool : min(p.keep, lo);
  const int pool0 = p.pool > 0 ? start / p.pool : 0, k_n = p.heads / p.group * p.dim, v_n = p.heads / p.group * p.vdim;
  const int n_keys = kept + pos - lo + 1;
  auto key_row = [&](int i) { return start + (i < kept ? i : lo + i - kept); };
  float m = -INFINITY, l = 0.f;
  for (int base = 0; base < n_keys; base += 32) {
    const int key = key_row(base + lane);
    float s = -INFINITY;
    if (base + lane < n_keys) {
      const T* kn = (p.pool > 0 && base + lane < kept ? pk + (size_t)(pool0 + base + lane) * k_n : k + (size_t)key * p.k_ld) + (size_t)hk * p.dim;
      float acc = 0.f;
      for (int d = 0; d < p.dim; ++d) acc += qs[d] * to_f(kn[d]);
      if (p.rot > 0) {
        const T* kr = krot + (size_t)key * p.kr_ld;
        for (int d = 0; d < p.rot; ++d) acc += qs[p.dim + d] * to_f(kr[d]);
      }
      s = capped(acc * p.scale, p.cap);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float corr = m == -INFINITY ? 0.f : expf(m - mn);
    const float pr = base + lane < n_keys ? expf(s - mn) : 0.f;
    l = l * corr + warp_sum(pr);
    m = mn;
    const int nk = min(32, n_keys - base);
    const int e_end = (p.vdim + 31) & ~31;
    for (int e = lane; e < e_end; e += 32) {
      float acc = e < p.vdim ? os[e] * corr : 0.f;
      for (int j = 0; j < nk; ++j) {
        const float w = __shfl_sync(0xffffffffu, pr, j);
        const T* vr = p.pool > 0 && base + j < kept ? pv + (size_t)(pool0 + base + j) * v_n : v + (size_t)key_row(base + j) * p.v_ld;
        if (e < p.vdim) acc += w * to_f(vr[(size_t)hk * p.vdim + e]);
      }
      if (e < p.vdim) os[e] = acc;
    }
    __syncwarp();
  }
  const float sk = p.sink != nullptr ? p.sink[h] : -INFINITY, mt = fmaxf(m, sk);
  float f = p.out_scale * expf(m - mt) / (l * expf(m - mt) + expf(sk - mt));
  if (p.gate_mode == 1) f *= p.head_gate[(size_t)t * p.heads + h];
  for (int e = lane; e < p.vdim; e += 32) {
    float o = os[e] * f;
    if (p.gate_mode == 2) o *= sigmoid_f(to_f(gate[(size_t)t * p.gate_ld + (size_t)h * p.vdim + e]));
    out[(size_t)t * p.out_ld + (size_t)h * p.vdim + e] = from_f<T>(o);
  }
}

// ------------------------------------------------------------------------------------------------------------
// Decode attention over the paged cache, any size with dim, vdim <= 1024: one block per (slot, head), the four warps take
// keys in turn, lanes own dimensions.
// ------------------------------------------------------------------------------------------------------------
struct GroupedDecode {
  int B, heads, kv_heads, dim, vdim, max_blocks, block_size, window, keep;
  float scale, cap;
  const int* seq_lens;
  const int* block_table;
  const float* sink;       // [heads] or null
  const float* head_gate;  // [B, heads] or null
  int pool, pool_rows;     // 0: no blocks
  const void* pool_k;      // rows of means, see AttnPrep
  const void* pool_v;
  long long out_ld;
  float out_scale;
};

constexpr int GD_MAX_REG = 32;
template <typename T>
__global__ void __launch_bounds__(128)
grouped_decode_kernel(const GroupedDecode p, const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                      const T* __restrict__ gate, T* __restrict__ out) {
  extern __shared__ float sm[];  // [dim] query, [4][vdim] partial outputs, [8] max / sum
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, h = blockIdx.x, hk = h / (p.heads / p.kv_heads), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.seq_lens[b];
  if (pos < 0 || pos >= p.max_blocks * p.block_size) return;
  float* qs = sm;
  float* po = sm + p.dim;
  float* ml = po + 4 * p.vdim;
  for (int d = threadIdx.x; d < p.dim; d += 128) qs[d] = to_f(q[((size_t)b * p.heads + h) * p.dim + d]);
  __syncthreads();
  const int* bt = p.block_table + (size_t)b * p.max_blocks;
  float m = -INFINITY, l = 0.f, acc[GD_MAX_REG];
#pragma unroll
  for (int i = 0; i < GD_MAX_REG; ++i) acc[i] = 0.f;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int kept = p.pool > 0 ? min(lo / p.pool, p.pool_rows) : min(p.keep, lo), n_keys = kept + pos - lo + 1;
  for (int i = warp; i < n_keys; i += 4) {
    const bool mean = p.pool > 0 && i < kept;
    const int j = i < kept ? i : lo + i - kept;
    const size_t row = mean ? ((size_t)b * p.pool_rows + i) * p.kv_heads + hk
                            : ((size_t)bt[j / p.block_size] * p.block_size + j % p.block_size) * p.kv_heads + hk;
    const T* kr = (mean ? reinterpret_cast<const T*>(p.pool_k) : k_cache) + row * p.dim;
    const T* vr = (mean ? reinterpret_cast<const T*>(p.pool_v) : v_cache) + row * p.vdim;
    float s = 0.f;
    for (int d = lane; d < p.dim; d += 32) s += to_f(kr[d]) * qs[d];
    s = capped(warp_sum(s) * p.scale, p.cap);
    const float mn = fmaxf(m, s), corr = m == -INFINITY ? 0.f : expf(m - mn), w = expf(s - mn);
    l = l * corr + w;
    m = mn;
#pragma unroll
    for (int i = 0; i < GD_MAX_REG; ++i) {
      const int e = lane + 32 * i;
      if (e < p.vdim) acc[i] = acc[i] * corr + w * to_f(vr[e]);
    }
  }
#pragma unroll
  for (int i = 0; i < GD_MAX_REG; ++i) {
    const int e = lane + 32 * i;
    if (e < p.vdim) po[(size_t)warp * p.vdim + e] = acc[i];
  }
  if (lane == 0) { ml[warp] = m; ml[4 + warp] = l; }
  __syncthreads();
  float mt = ml[0], den = 0.f, f[4];  // warp 0 always has a key
  for (int w = 1; w < 4; ++w) mt = fmaxf(mt, ml[w]);
  if (p.sink != nullptr) {
    mt = fmaxf(mt, p.sink[h]);
    den = expf(p.sink[h] - mt);
  }
  for (int w = 0; w < 4; ++w) {
    f[w] = ml[w] == -INFINITY ? 0.f : expf(ml[w] - mt);
    den += f[w] * ml[4 + w];
  }
  for (int e = threadIdx.x; e < p.vdim; e += 128) {
    float o = 0.f;
    for (int w = 0; w < 4; ++w) o += f[w] * po[(size_t)w * p.vdim + e];
    o *= p.out_scale / den;
    if (p.head_gate != nullptr) o *= p.head_gate[(size_t)b * p.heads + h];
    const size_t i = ((size_t)b * p.heads + h) * p.vdim + e;
    if (gate != nullptr) o *= sigmoid_f(to_f(gate[i]));
    out[(size_t)b * p.out_ld + (size_t)h * p.vdim + e] = from_f<T>(o);
  }
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

}  // namespace

#define PDL trlb_host::pdl_enabled()

// rows [q | k | v | g] of ld elements; src_f32: fp32 sums (decode: q_out and, for gates per element, g_out given), else the model
// dtype.  temp, q_w, k_w, tok_slot, k_out, block_table may be null; gates: 0 none, 1 per head (to head_gate), 2 per element; rot 0:
// no rotation; unit: norms, whole: over all heads; q_head [heads] (factors of the queries) may be null; pool > 0 (decode): means of
// complete blocks to pool_k, pool_v [slots, pool_rows, kv_heads, dim / vdim].  Without has_v the keys as projected are the values (prompt: k_out is then required).
TRLB_API int trlb_attn_prep(void* src, int src_f32, long long ld, int rows, int heads, int kv_heads, int dim, int vdim, int has_kv,
                            int has_v, int gates, float eps, const int* positions, const int* tok_slot, const float* temp,
                            int temp_len, int whole, const float* q_w, const float* k_w, int rot, int halves, const float* table,
                            int table_len, void* q_out, void* k_out, void* g_out, float* head_gate, void* k_cache, void* v_cache,
                            const int* block_table, int max_blocks, int block_size, int unit, const float* q_head, int pool, int pool_rows, void* pool_k,
                            void* pool_v, int is_bf16, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (pool > 0 && (k_cache == nullptr || pool_k == nullptr || pool_v == nullptr || !has_v)) return -250;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || (is_bf16 && src_f32 && q_out == nullptr)) return -250;
  if (has_kv && !has_v && (dim != vdim || (q_out == nullptr && k_out == nullptr))) return -250;
  if (rot < 0 || rot > dim || (rot & 1) || (rot > 0 && table == nullptr)) return -250;
  if ((gates == GATES_HEAD && head_gate == nullptr) || (gates == GATES_ELEMENT && q_out != nullptr && g_out == nullptr)) return -250;
  if (k_cache != nullptr && (v_cache == nullptr || block_table == nullptr || block_size <= 0)) return -250;
  AttnPrep p = {ld, rows, heads, kv_heads, dim, vdim, has_kv, has_kv && has_v, gates, eps, positions, tok_slot, temp, temp_len, q_w,
                k_w, rot, halves, (const float2*)table, table_len, head_gate, k_cache ? block_table : nullptr, max_blocks, block_size,
                unit, q_head, pool, pool_rows, pool_k, pool_v};
  const int row_units = heads + (has_kv ? kv_heads * (has_v ? 2 : 1) : 0) + (gates == GATES_ELEMENT && q_out != nullptr ? heads : 0);
  const int widest = dim > vdim ? dim : vdim;
  int lanes_log2 = 0;
  while ((8 << lanes_log2) < widest) ++lanes_log2;
  const int threads = row_units << lanes_log2;  // of one round
  const auto aligned = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (((dim | vdim | (int)(ld & 7)) & 7) == 0 && widest <= 256 && threads <= 2048 && rot % (halves ? 16 : 8) == 0 && aligned(src) &&
      aligned(q_out) && aligned(k_out) && aligned(g_out) && aligned(k_cache) && aligned(v_cache) && aligned(q_w) && aligned(k_w) && aligned(pool_k) && aligned(pool_v)) {
    const int rounds = threads <= 256 ? 1 : threads <= 1024 ? 2 : 4;
    const dim3 block(((threads + rounds - 1) / rounds + 31) / 32 * 32);
#define GO(TT, SS, WW, RR) (int)trlb_host::launch_kernel(attn_prep_rows_kernel<TT, SS, WW, RR>, dim3(rows), block, 0, st, PDL, p, lanes_log2, (SS*)src, \
                                                         (TT*)q_out, (TT*)k_out, (TT*)g_out, (TT*)k_cache, (TT*)v_cache)
#define PICK(TT, SS, WW) (rounds == 1 ? GO(TT, SS, WW, 1) : rounds == 2 ? GO(TT, SS, WW, 2) : GO(TT, SS, WW, 4))
    if (is_bf16) return src_f32 ? (whole ? PICK(bf16, float, true) : PICK(bf16, float, false)) : (whole ? PICK(bf16, bf16, true) : PICK(bf16, bf16, false));
    return whole ? PICK(float, float, true) : PICK(float, float, false);
#undef PICK
#undef GO
  }
  const int units = row_units + (gates == GATES_HEAD ? 1 : 0);
  const dim3 grid(whole ? (unsigned)rows : (unsigned)(((long long)rows * units + 7) / 8));
  const dim3 blk(!whole ? 256 : units >= 16 ? 512 : units >= 8 ? 256 : 128);
#define GO(TT, SS, WW) (int)trlb_host::launch_kernel(attn_prep_kernel<TT, SS, WW>, grid, blk, 0, st, PDL, p, (SS*)src, (TT*)q_out, (TT*)k_out, \
                                                     (TT*)g_out, (TT*)k_cache, (TT*)v_cache)
  if (is_bf16) return src_f32 ? (whole ? GO(bf16, float, true) : GO(bf16, float, false)) : (whole ? GO(bf16, bf16, true) : GO(bf16, bf16, false));
  return whole ? GO(float, float, true) : GO(float, float, false);
#undef GO
}

// k, v [T rows of k_ld / v_ld]: k_n / v_n columns; pk, pv [T / P + 1, k_n / v_n]; with seq_slot [n_seq]: also to slot_k, slot_v
// [slots, slot_rows, k_n / v_n].
TRLB_API int trlb_pool_blocks(const void* k, long long k_ld, int k_n, const void* v, long long v_ld, int v_n, const int* cu, int n_seq, int T,
                              int P, void* pk, void* pv, const int* seq_slot, int slots, int slot_rows, void* slot_k, void* slot_v,
                              int is_bf16, cudaStream_t st) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (P <= 0 || (seq_slot != nullptr && (slot_k == nullptr || slot_v == nullptr))) return -254;
  const PoolBlocks p = {cu, n_seq, P, k_n, v_n, k_ld, v_ld, seq_slot, slots, slot_rows};
  const dim3 rows(T / P + 1, (k_n + v_n + 511) / 512);
  if (is_bf16) pool_blocks_kernel<bf16><<<rows, 128, 0, st>>>(p, (const bf16*)k, (const bf16*)v, (bf16*)pk, (bf16*)pv, (bf16*)slot_k, (bf16*)slot_v);
  else pool_blocks_kernel<float><<<rows, 128, 0, st>>>(p, (const float*)k, (const float*)v, (float*)pk, (float*)pv, (float*)slot_k, (float*)slot_v);
  return (int)cudaGetLastError();
}

// Arguments as trlb_mixer_attn_tc (mixer_attn_tcgen05.cu), in either dtype and any size; positions instead of sequence starts.
TRLB_API int trlb_mixer_attn(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld,
                             const void* krot, long long krot_ld, const int* positions, int T, int heads, int kv_heads, int dim,
                             int rot, int vdim, int window, int keep, float scale, float cap, const float* sink, int gate_mode,
                             const void* gate, long long gate_ld, int pool, const void* pk, const void* pv, void* out, long long out_ld,
                             float out_scale, int is_bf16, cudaStream_t st) {
  if (T <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || (pool > 0 && (pk == nullptr || pv == nullptr))) return -251;
  MixerAttn p = {T, heads, heads / kv_heads, dim, rot, vdim, window, keep, q_ld, k_ld, v_ld, krot_ld, gate_ld, scale, cap, positions,
                 sink, gate_mode, gate_mode == 1 ? (const float*)gate : nullptr, window > 0 ? pool : 0, out_ld, out_scale};
  const int grid = (int)(((long long)T * heads + 3) / 4);
  const size_t smem = (size_t)4 * (dim + rot + vdim) * 4;
  if (is_bf16) {
    if (!allow_smem(mixer_attn_kernel<bf16>, smem)) return -252;
    mixer_attn_kernel<bf16><<<grid, 128, smem, st>>>(p, (const bf16*)q, (const bf16*)k, (const bf16*)v, (const bf16*)krot,
                                                     gate_mode == 2 ? (const bf16*)gate : nullptr, (const bf16*)pk, (const bf16*)pv, (bf16*)out);
  } else {
    if (!allow_smem(mixer_attn_kernel<float>, smem)) return -252;
    mixer_attn_kernel<float><<<grid, 128, smem, st>>>(p, (const float*)q, (const float*)k, (const float*)v, (const float*)krot,
                                                      gate_mode == 2 ? (const float*)gate : nullptr, (const float*)pk, (const float*)pv, (float*)out);
  }
  return (int)cudaGetLastError();
}

// q [B, heads, dim], k_cache [blocks, block_size, kv_heads, dim], v_cache [.., vdim], gate logits [B, heads, vdim] or null,
// head_gate (factors) [B, heads] or null, sink [heads] or null.  window <= 0: unlimited, else the first `keep` keys stay visible, or
// (pool > 0) the means of the blocks before it.
TRLB_API int trlb_grouped_decode(const void* q, const void* k_cache, const void* v_cache, const void* gate, const float* head_gate,
                                 const float* sink, void* out, int B, int heads, int kv_heads, int dim, int vdim, int window,
                                 int keep, float scale, float cap, const int* seq_lens,
                                 const int* block_table, int max_blocks, int block_size, int pool, int pool_rows, const void* pool_k,
                                 const void* pool_v, long long out_ld, float out_scale, int is_bf16, cudaStream_t st) {
  if (B <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || (pool > 0 && (pool_k == nullptr || pool_v == nullptr)) || vdim > 32 * GD_MAX_REG) return -253;
  GroupedDecode p = {B, heads, kv_heads, dim, vdim, max_blocks, block_size, window, keep, scale, cap, seq_lens, block_table, sink, head_gate,
                     window > 0 ? pool : 0, pool_rows, pool_k, pool_v, out_ld, out_scale};
  const size_t smem = (size_t)(dim + 4 * vdim + 8) * 4;
  if (smem > 48 * 1024) return -253;
  const dim3 grid(heads, B), blk(128);
#define GO(TT) (int)trlb_host::launch_kernel(grouped_decode_kernel<TT>, grid, blk, smem, st, PDL, p, (const TT*)q, (const TT*)k_cache, (const TT*)v_cache, (const TT*)gate, (TT*)out)
  return is_bf16 ? GO(bf16) : GO(float);
#undef GO
}
