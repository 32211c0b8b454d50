// Element-wise, cache and recurrence kernels of the layered decoders (models/layered.py): embedding scale, Dynamic-Tanh and
// RMS norms fused with the residual addition, clamped gated linear unit, per-token side inputs, latent-attention
// preparation / absorption, mLSTM gates, steps and outputs.  Grouped-query attention is in grouped_attn.cu, the real-gated
// linear recurrent unit in rglru.cu.
//
// T is the model dtype (bf16 or fp32).  The residual stream, norm statistics, gates, attention scores and recurrent
// states are fp32 in both.  This file is compiled without fast-math (csrc/build.py: EXACT_MATH).
//
// Decode kernels work on one row per sequence slot; seq_lens[slot] is the position of the slot's new token and a
// negative value marks an idle slot.  fp32 sums of the stream-K decode GEMM are cleared by their last reader
// (`clear`), so no memset runs between two steps.
#include "mixers.cuh"

namespace trlb {

// ------------------------------------------------------------------------------------------------------------
// embedding and norm
// ------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
embed_scaled_kernel(const long long* __restrict__ ids, const T* __restrict__ emb, float* __restrict__ x, int H, int V,
                    float scale) {
  pdl_launch_dependents();
  pdl_wait();
  const long long id = ids[blockIdx.x];
  if ((H & 3) == 0 && id >= 0 && id < V) {
    for (int j = 4 * threadIdx.x; j < H; j += 4 * blockDim.x) {
      const float4 e = load4(emb + (size_t)id * H + j);
      store4(x + (size_t)blockIdx.x * H + j, make_float4(e.x * scale, e.y * scale, e.z * scale, e.w * scale));
    }
    return;
  }
  for (int j = threadIdx.x; j < H; j += blockDim.x)
    x[(size_t)blockIdx.x * H + j] = (id >= 0 && id < V) ? to_f(emb[(size_t)id * H + j]) * scale : 0.f;
}

// The same over its root mean square, times shift + w; copy (may be null) gets the row too.
template <typename T>
__global__ void __launch_bounds__(256)
embed_normed_kernel(const long long* __restrict__ ids, const T* __restrict__ emb, const float* __restrict__ w, float* __restrict__ x,
                    float* __restrict__ copy, int H, int V, float scale, float eps, float shift) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const long long id = ids[blockIdx.x];
  const bool ok = id >= 0 && id < V, v4 = (H & 3) == 0;
  const T* e = emb + (size_t)(ok ? id : 0) * H;
  const size_t row = (size_t)blockIdx.x * H;
  float s = 0.f;
  if (v4) {
    for (int j = 4 * threadIdx.x; j < H; j += 4 * blockDim.x) {
      const float4 v = load4(e + j);
      s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int j = threadIdx.x; j < H; j += blockDim.x) s += to_f(e[j]) * to_f(e[j]);
  }
  const float ss = block_sum2(s, 0.f, red).x;
  const float r = ok ? scale / sqrtf(ss * (scale * scale) / (float)H + eps) : 0.f;
  if (v4) {
    for (int j = 4 * threadIdx.x; j < H; j += 4 * blockDim.x) {
      const float4 v = load4(e + j), g = load4(w + j);
      const float4 o = make_float4(v.x * r * (shift + g.x), v.y * r * (shift + g.y), v.z * r * (shift + g.z), v.w * r * (shift + g.w));
      store4(x + row + j, o);
      if (copy != nullptr) store4(copy + row + j, o);
    }
  } else {
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
      const float o = to_f(e[j]) * r * (shift + w[j]);
      x[row + j] = o;
      if (copy != nullptr) copy[row + j] = o;
    }
  }
}

// The same (without the norm) plus a row of a table of token pairs: row (previous * mul_prev + current * mul_cur) mod buckets, or the last row,
// number `buckets`, at a sequence's first token.  Prompt rows (prev_state is written by a sequence's last row, tok_slot gives
// the slots; both may be null) take the previous token from ids; decode rows (one per slot, positions negative: idle) from
// prev_state, which moves on.
struct PairEmbed {
  const long long* ids;
  const int* positions;
  const int* tok_slot;
  long long* prev_state;
  long long mul_prev, mul_cur, buckets;
  int T, H, V, decode;
  float scale;
};

template <typename T>
__global__ void __launch_bounds__(256)
embed_pairs_kernel(const PairEmbed p, const T* __restrict__ emb, const T* __restrict__ pairs, float* __restrict__ x) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, pos = p.positions[r];
  const long long id = p.ids[r];
  const bool ok = id >= 0 && id < p.V;
  long long prev = -1;
  if (pos > 0) prev = p.decode ? p.prev_state[r] : p.ids[r - 1];
  long long row = p.buckets;
  if (prev >= 0) {
    row = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
    if (row < 0) row += p.buckets;
  }
  const T* e = emb + (size_t)(ok ? id : 0) * p.H;
  const T* g = pairs + (size_t)row * p.H;
  float* o = x + (size_t)r * p.H;
  if ((p.H & 3) == 0) {
    for (int j = 4 * threadIdx.x; j < p.H; j += 4 * blockDim.x) {
      const float4 a = ok ? load4(e + j) : make_float4(0.f, 0.f, 0.f, 0.f), b = load4(g + j);
      store4(o + j, make_float4(a.x * p.scale + b.x, a.y * p.scale + b.y, a.z * p.scale + b.z, a.w * p.scale + b.w));
    }
  } else {
    for (int j = threadIdx.x; j < p.H; j += blockDim.x) o[j] = (ok ? to_f(e[j]) * p.scale : 0.f) + to_f(g[j]);
  }
  if (p.prev_state == nullptr || pos < 0) return;
  if (p.decode) {
    __syncthreads();  // everyone has read the old one
    if (threadIdx.x == 0) p.prev_state[r] = id;
  } else if (threadIdx.x == 0 && (r + 1 == p.T || p.positions[r + 1] == 0)) {
    p.prev_state[p.tok_slot[r]] = id;
  }
}

// x (+= delta) ; out = tanh(alpha x) w + b.  VEC elements per thread along H (H % VEC == 0).
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
dynamic_tanh_kernel(float* __restrict__ x, float* __restrict__ delta, const float* __restrict__ alpha_p,
                    const float* __restrict__ w, const float* __restrict__ b, T* __restrict__ out, long long n_vec,
                    int H, int clear) {
  pdl_launch_dependents();
  pdl_wait();
  const float alpha = *alpha_p;
  for (long long v = blockIdx.x * (long long)blockDim.x + threadIdx.x; v < n_vec; v += (long long)gridDim.x * blockDim.x) {
    const long long e = v * VEC;
    const int j = (int)(e % H);
    float a[VEC];
    if (VEC == 4) {
      const float4 t = *reinterpret_cast<const float4*>(x + e);
      a[0] = t.x; a[1 % VEC] = t.y; a[2 % VEC] = t.z; a[3 % VEC] = t.w;
    } else {
      a[0] = x[e];
    }
    if (delta != nullptr) {
      if (VEC == 4) {
        const float4 d = *reinterpret_cast<const float4*>(delta + e);
        a[0] += d.x; a[1 % VEC] += d.y; a[2 % VEC] += d.z; a[3 % VEC] += d.w;
        *reinterpret_cast<float4*>(x + e) = make_float4(a[0], a[1 % VEC], a[2 % VEC], a[3 % VEC]);
        if (clear) *reinterpret_cast<float4*>(delta + e) = make_float4(0.f, 0.f, 0.f, 0.f);
      } else {
        a[0] += delta[e];
        x[e] = a[0];
        if (clear) delta[e] = 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) out[e + i] = from_f<T>(tanhf(alpha * a[i]) * w[j + i] + b[j + i]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
gelu_erf_kernel(const T* __restrict__ z, T* __restrict__ out, long long n) {
  const long long stride = (long long)gridDim.x * blockDim.x, first = blockIdx.x * (long long)blockDim.x + threadIdx.x;
#pragma unroll 2
  for (long long i = first; i < n / 4; i += stride) {
    const float4 v = load4(z + 4 * i);
    store4(out + 4 * i, make_float4(gelu_erf_f(v.x), gelu_erf_f(v.y), gelu_erf_f(v.z), gelu_erf_f(v.w)));
  }
  for (long long i = n / 4 * 4 + first; i < n; i += stride) out[i] = from_f<T>(gelu_erf_f(to_f(z[i])));
}

// ------------------------------------------------------------------------------------------------------------
// RMS norms around the residual stream, in one pass over a row:
//     x += mult d                     or, with `post`,   x += mult d / rms(d) * (shift + post) * post_scale
//     out = x / rms(x) * (shift + w) * gain              or, without `w`,   out = x
// where d is delta, plus delta2, or plus the sum over the choices c of weight[c] * y[row[c]] (the experts' rows of this token; a
// negative row: nothing).  x also gets anchor and bump, when given; out2 is the norm with w2 instead of w.
// (no post_scale: 1).  `clear` zeroes delta behind itself.  One block per row; NV float4 of the row live in each thread's registers.
// ------------------------------------------------------------------------------------------------------------
struct RmsResidual {
  float* x;
  float* delta;        // null: nothing is added
  const float* post;   // null: delta is added as it is
  const float* w;      // null: the sum itself is the output
  int H, clear;
  float eps;
  const float* post_scale;  // null: 1
  float shift, gain, mult;
  const float* delta2;      // [T, H] or null
  const void* y;            // [rows, H] in the dtype of the output, or null
  const int* row;           // [T, top]
  const float* weight;      // [T, top]
  int top;
  const float* anchor;      // [T, H] or null
  const float* bump;        // [H] or null
  const float* w2;          // null: one output
  void* out2;
};

__device__ __forceinline__ float4 rms_weight4(const float* w, const float* scale, float shift, float gain, int j) {
  float4 g = load4(w + j);
  g = make_float4((shift + g.x) * gain, (shift + g.y) * gain, (shift + g.z) * gain, (shift + g.w) * gain);
  if (scale != nullptr) {
    const float4 c = load4(scale + j);
    g = make_float4(g.x * c.x, g.y * c.y, g.z * c.z, g.w * c.w);
  }
  return g;
}
__device__ __forceinline__ float4 fma4(float s, float4 a, float4 b) {
  return make_float4(fmaf(s, a.x, b.x), fmaf(s, a.y, b.y), fmaf(s, a.z, b.z), fmaf(s, a.w, b.w));
}

template <typename T, int NV>
__global__ void __launch_bounds__(256)
rms_residual_kernel(const RmsResidual p, T* __restrict__ out) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = (size_t)blockIdx.x * p.H;
  const int n4 = p.H / 4, nt = blockDim.x;
  float4 a[NV], d[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * nt;
    a[i] = j < n4 ? load4(p.x + row + 4 * j) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (p.delta != nullptr) {
    float sd = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int j = threadIdx.x + i * nt;
      d[i] = j < n4 ? load4(p.delta + row + 4 * j) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.delta2 != nullptr && j < n4) d[i] = fma4(1.f, load4(p.delta2 + row + 4 * j), d[i]);
    }
    if (p.y != nullptr) {
      for (int c = 0; c < p.top; ++c) {
        const int at = p.row[(size_t)blockIdx.x * p.top + c];
        if (at < 0) continue;
        const float wt = p.weight[(size_t)blockIdx.x * p.top + c];
        const T* y = reinterpret_cast<const T*>(p.y) + (size_t)at * p.H;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int j = threadIdx.x + i * nt;
          if (j < n4) d[i] = fma4(wt, load4(y + 4 * j), d[i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) sd += d[i].x * d[i].x + d[i].y * d[i].y + d[i].z * d[i].z + d[i].w * d[i].w;
    float r = 1.f;
    if (p.post != nullptr) r = 1.f / sqrtf(block_sum2(sd, 0.f, red).x / (float)p.H + p.eps);
    r *= p.mult;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int j = threadIdx.x + i * nt;
      if (j < n4) {
        const float4 g = p.post != nullptr ? rms_weight4(p.post, p.post_scale, p.shift, 1.f, 4 * j) : make_float4(1.f, 1.f, 1.f, 1.f);
        a[i].x += d[i].x * r * g.x; a[i].y += d[i].y * r * g.y; a[i].z += d[i].z * r * g.z; a[i].w += d[i].w * r * g.w;
        if (p.clear) store4(p.delta + row + 4 * j, make_float4(0.f, 0.f, 0.f, 0.f));
      }
    }
  }
  if (p.delta != nullptr || p.anchor != nullptr || p.bump != nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int j = threadIdx.x + i * nt;
      if (j < n4) {
        if (p.anchor != nullptr) a[i] = fma4(1.f, load4(p.anchor + row + 4 * j), a[i]);
        if (p.bump != nullptr) a[i] = fma4(1.f, load4(p.bump + 4 * j), a[i]);
        store4(p.x + row + 4 * j, a[i]);
      }
    }
  }
  float r = 1.f;
  if (p.w != nullptr) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += a[i].x * a[i].x + a[i].y * a[i].y + a[i].z * a[i].z + a[i].w * a[i].w;
    r = 1.f / sqrtf(block_sum2(s, 0.f, red).x / (float)p.H + p.eps);
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * nt;
    if (j < n4) {
      const float4 g = p.w != nullptr ? rms_weight4(p.w, nullptr, p.shift, p.gain, 4 * j) : make_float4(1.f, 1.f, 1.f, 1.f);
      store4(out + row + 4 * j, make_float4(a[i].x * r * g.x, a[i].y * r * g.y, a[i].z * r * g.z, a[i].w * r * g.w));
      if (p.w2 != nullptr) {
        const float4 h = rms_weight4(p.w2, nullptr, p.shift, p.gain, 4 * j);
        store4(reinterpret_cast<T*>(p.out2) + row + 4 * j, make_float4(a[i].x * r * h.x, a[i].y * r * h.y, a[i].z * r * h.z, a[i].w * r * h.w));
      }
    }
  }
}

// The same for any row length.
template <typename T>
__global__ void __launch_bounds__(256)
rms_residual_any_kernel(const RmsResidual p, T* __restrict__ out) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = (size_t)blockIdx.x * p.H;
  float* x = p.x + row;
  float* d = p.delta == nullptr ? nullptr : p.delta + row;
  auto added = [&](int j) {
    float v = d[j];
    if (p.delta2 != nullptr) v += p.delta2[row + j];
    if (p.y != nullptr) {
      for (int c = 0; c < p.top; ++c) {
        const int at = p.row[(size_t)blockIdx.x * p.top + c];
        if (at >= 0) v = fmaf(p.weight[(size_t)blockIdx.x * p.top + c], to_f(reinterpret_cast<const T*>(p.y)[(size_t)at * p.H + j]), v);
      }
    }
    return v;
  };
  float r = 1.f, s = 0.f;
  if (d != nullptr && p.post != nullptr) {
    for (int j = threadIdx.x; j < p.H; j += 256) {
      const float v = added(j);
      s += v * v;
    }
    r = 1.f / sqrtf(block_sum2(s, 0.f, red).x / (float)p.H + p.eps);
  }
  r *= p.mult;
  s = 0.f;
  for (int j = threadIdx.x; j < p.H; j += 256) {
    float a = x[j];
    if (d != nullptr) {
      const float v = added(j) * r;
      a += p.post != nullptr ? v * (p.shift + p.post[j]) * (p.post_scale != nullptr ? p.post_scale[j] : 1.f) : v;
      if (p.clear) d[j] = 0.f;
    }
    if (p.anchor != nullptr) a += p.anchor[row + j];
    if (p.bump != nullptr) a += p.bump[j];
    x[j] = a;
    s += a * a;
  }
  float rx = 1.f;
  if (p.w != nullptr) rx = 1.f / sqrtf(block_sum2(s, 0.f, red).x / (float)p.H + p.eps);
  for (int j = threadIdx.x; j < p.H; j += 256) {
    out[row + j] = from_f<T>(p.w != nullptr ? x[j] * rx * (p.shift + p.w[j]) * p.gain : x[j]);
    if (p.w2 != nullptr) reinterpret_cast<T*>(p.out2)[row + j] = from_f<T>(x[j] * rx * (p.shift + p.w2[j]) * p.gain);
  }
}

// Gated linear units, z [rows, 2 n] = gate | up.  GELU: gelu_tanh(gate) up.  Else clamped: g sigmoid(alpha g) (u + shift), g =
// min(gate, limit), u = up clamped to [-limit, limit].
template <typename T, int VEC, bool GELU>
__global__ void __launch_bounds__(256)
glu_kernel(const T* __restrict__ z, T* __restrict__ out, long long total, int n, float limit, float alpha, float shift) {
  const int per = n / VEC;
  for (long long v = blockIdx.x * (long long)blockDim.x + threadIdx.x; v < total; v += (long long)gridDim.x * blockDim.x) {
    const long long row = v / per;
    const int j = (int)(v % per) * VEC;
    const T* zr = z + row * 2 * n + j;
    auto act = [&](float g, float u) {
      if (GELU) return gelu_tanh_t<T>(g) * u;
      g = fminf(g, limit);
      u = fminf(fmaxf(u, -limit), limit);
      return g * sigmoid_t<T>(alpha * g) * (u + shift);
    };
    if (VEC == 4) {
      const float4 g = load4(zr), u = load4(zr + n);
      store4(out + row * n + j, make_float4(act(g.x, u.x), act(g.y, u.y), act(g.z, u.z), act(g.w, u.w)));
    } else {
      out[row * n + j] = from_f<T>(act(to_f(zr[0]), to_f(zr[n])));
    }
  }
}

// Side input of a layer: out[row] = gelu_tanh(z[row]) * table[ids[row], off : off + n].  Z: dtype of z; `clear` zeroes it.
template <typename T, typename Z, int VEC>
__global__ void __launch_bounds__(256)
side_gate_kernel(Z* __restrict__ z, const long long* __restrict__ ids, const T* __restrict__ table, long long table_ld, int off,
                 int n, long long total, int V, int clear, T* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = n / VEC;
  for (long long v = blockIdx.x * (long long)blockDim.x + threadIdx.x; v < total; v += (long long)gridDim.x * blockDim.x) {
    const long long row = v / per, id = ids[row], at = v * VEC;
    const bool ok = id >= 0 && id < V;
    const T* e = table + (size_t)(ok ? id : 0) * table_ld + off + (int)(v % per) * VEC;
    if (VEC == 4) {
      const float4 a = load4(z + at), b = ok ? load4(e) : make_float4(0.f, 0.f, 0.f, 0.f);
      store4(out + at, make_float4(gelu_tanh_t<T>(a.x) * b.x, gelu_tanh_t<T>(a.y) * b.y, gelu_tanh_t<T>(a.z) * b.z, gelu_tanh_t<T>(a.w) * b.w));
      if (clear) store4(z + at, make_float4(0.f, 0.f, 0.f, 0.f));
    } else {
      out[at] = from_f<T>(gelu_tanh_t<T>(to_f(z[at])) * (ok ? to_f(*e) : 0.f));
      if (clear) z[at] = from_f<Z>(0.f);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// latent attention
// ------------------------------------------------------------------------------------------------------------
struct LatentPrep {
  float* acc;           // [rows, ld]: query latent | key/value latent | rotated key | gate logits
  long long ld;
  int q_rank, kv_rank, rot, heads, clear;
  const float* q_norm;
  const float* kv_norm;
  float eps;
  const int* positions;  // [rows] position of every row (prompt) or of every slot (decode); negative: idle
  const int* tok_slot;   // [rows] or null (slot = row)
  const float2* table;   // [table_len, rot / 2] (cos, sin) with the rotation's magnitude folded in; unused if rot == 0
  int table_len;
  float* gate;           // [rows, heads] sigmoid of the gate logits
  int kr_off, lat_w;     // a latent row: [kv_rank | pad to kr_off | rot | pad to lat_w]
  const int* block_table;  // null: no cache
  int max_blocks, block_size;
};

template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const LatentPrep p, T* __restrict__ cq, T* __restrict__ lat, T* __restrict__ cache) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  float* a = p.acc + (size_t)row * p.ld;
  const float* akv = a + p.q_rank;
  const float* ar = akv + p.kv_rank;
  const float* ag = ar + p.rot;
  float sq = 0.f, sk = 0.f;
  const bool vec = ((p.q_rank | p.kv_rank | (int)p.ld) & 3) == 0 && (reinterpret_cast<uintptr_t>(p.acc) & 15) == 0;
  if (vec) {
#pragma unroll 2
    for (int j = 4 * threadIdx.x; j < p.q_rank; j += 4 * blockDim.x) {
      const float4 v = load4(a + j);
      sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    for (int j = 4 * threadIdx.x; j < p.kv_rank; j += 4 * blockDim.x) {
      const float4 v = load4(akv + j);
      sk += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int j = threadIdx.x; j < p.q_rank; j += blockDim.x) sq += a[j] * a[j];
    for (int j = threadIdx.x; j < p.kv_rank; j += blockDim.x) sk += akv[j] * akv[j];
  }
  const float2 s = block_sum2(sq, sk, red);
  const float rq = p.q_rank > 0 ? 1.f / sqrtf(s.x / (float)p.q_rank + p.eps) : 0.f, rk = 1.f / sqrtf(s.y / (float)p.kv_rank + p.eps);
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  if (vec) {
#pragma unroll 2
    for (int j = 4 * threadIdx.x; j < p.q_rank; j += 4 * blockDim.x) {
      const float4 v = load4(a + j), w = load4(p.q_norm + j);
      store4(cq + (size_t)row * p.q_rank + j, make_float4(v.x * rq * w.x, v.y * rq * w.y, v.z * rq * w.z, v.w * rq * w.w));
      if (p.clear) store4(a + j, zero);
    }
  } else {
    for (int j = threadIdx.x; j < p.q_rank; j += blockDim.x) {
      cq[(size_t)row * p.q_rank + j] = from_f<T>(a[j] * rq * p.q_norm[j]);
      if (p.clear) a[j] = 0.f;
    }
  }
  for (int h = threadIdx.x; h < p.heads; h += blockDim.x) {
    p.gate[(size_t)row * p.heads + h] = sigmoid_f(ag[h]);
    if (p.clear) a[p.q_rank + p.kv_rank + p.rot + h] = 0.f;
  }
  const int pos = p.positions[row];
  const bool live = pos >= 0 && (p.rot == 0 || pos < p.table_len);
  T* dense = lat == nullptr ? nullptr : lat + (size_t)row * p.lat_w;
  T* paged = nullptr;
  if (live && p.block_table != nullptr) {
    const int slot = p.tok_slot ? p.tok_slot[row] : row;
    if (slot >= 0 && pos / p.block_size < p.max_blocks) {
      const int blk = p.block_table[(size_t)slot * p.max_blocks + pos / p.block_size];
      paged = cache + ((size_t)blk * p.block_size + pos % p.block_size) * p.lat_w;
    }
  }
  float* akw = a + p.q_rank;
  if (vec) {
    for (int j = 4 * threadIdx.x; j < p.kv_rank; j += 4 * blockDim.x) {
      const float4 v = load4(akv + j), w = load4(p.kv_norm + j);
      const float4 y = make_float4(v.x * rk * w.x, v.y * rk * w.y, v.z * rk * w.z, v.w * rk * w.w);
      if (dense) store4(dense + j, y);
      if (paged) store4(paged + j, y);
      if (p.clear) store4(akw + j, zero);
    }
  } else {
    for (int j = threadIdx.x; j < p.kv_rank; j += blockDim.x) {
      const T v = from_f<T>(akv[j] * rk * p.kv_norm[j]);
      if (dense) dense[j] = v;
      if (paged) paged[j] = v;
      if (p.clear) akw[j] = 0.f;
    }
  }
  for (int i = threadIdx.x; i < p.rot / 2; i += blockDim.x) {
    const float2 cs = live ? p.table[(size_t)pos * (p.rot / 2) + i] : make_float2(1.f, 0.f);
    const float u = ar[2 * i], v = ar[2 * i + 1];
    const T x0 = from_f<T>(u * cs.x - v * cs.y), x1 = from_f<T>(v * cs.x + u * cs.y);
    if (dense) { dense[p.kr_off + 2 * i] = x0; dense[p.kr_off + 2 * i + 1] = x1; }
    if (paged) { paged[p.kr_off + 2 * i] = x0; paged[p.kr_off + 2 * i + 1] = x1; }
    if (p.clear) {
      akw[p.kv_rank + 2 * i] = 0.f;
      akw[p.kv_rank + 2 * i + 1] = 0.f;
    }
  }
}

// q [rows, heads, dim + rot]: the rot part of every head turned in place.
template <typename T, int PAIRS>  // pairs per thread: 2 needs dim and rot to be multiples of 4
__global__ void __launch_bounds__(256)
rotate_q_kernel(T* __restrict__ q, int heads, int dim, int rot, const int* __restrict__ positions,
                const float2* __restrict__ table, int table_len, long long n) {
  const int half = rot / 2, groups = half / PAIRS;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const int f = (int)(i % groups) * PAIRS;
    const long long th = i / groups;
    const int pos = positions[th / heads];
    if (pos < 0 || pos >= table_len) continue;
    T* d = q + (size_t)th * (dim + rot) + dim + 2 * f;
    if (PAIRS == 2) {
      const float4 cs = *reinterpret_cast<const float4*>(table + (size_t)pos * half + f), v = load4(d);
      store4(d, make_float4(v.x * cs.x - v.y * cs.y, v.y * cs.x + v.x * cs.y, v.z * cs.z - v.w * cs.w, v.w * cs.z + v.z * cs.w));
      continue;
    }
    const float2 cs = table[(size_t)pos * half + f];
    const float u = to_f(d[0]), v = to_f(d[1]);
    d[0] = from_f<T>(u * cs.x - v * cs.y);
    d[1] = from_f<T>(v * cs.x + u * cs.y);
  }
}

// Decode, any size.  Absorption: q_lat[b, h] = [ W_uk[h]^T q_nope | rotated q_rot ] in the layout of a latent row.
template <typename T>
__global__ void __launch_bounds__(128)
latent_absorb_kernel(float* __restrict__ qacc, long long ld, const T* __restrict__ uk, T* __restrict__ q_lat, int heads,
                     int dim, int rot, int kv_rank, int kr_off, int lat_w, const int* __restrict__ positions,
                     const float2* __restrict__ table, int table_len, int clear) {
  extern __shared__ float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  float* q = qacc + (size_t)b * ld + (size_t)h * (dim + rot);
  for (int d = threadIdx.x; d < dim + rot; d += blockDim.x) {
    // the query has the precision of the model dtype, as in a prompt
    sm[d] = to_f(from_f<T>(q[d]));
    if (clear) q[d] = 0.f;
  }
  __syncthreads();
  const int pos = positions[b];
  if (pos < 0 || (rot > 0 && pos >= table_len)) return;
  T* dst = q_lat + ((size_t)b * heads + h) * lat_w;
  for (int r = threadIdx.x; r < lat_w; r += blockDim.x) {
    float v = 0.f;
    if (r < kv_rank) {
      const T* w = uk + (size_t)h * dim * kv_rank + r;
      for (int d = 0; d < dim; ++d) v += sm[d] * to_f(w[(size_t)d * kv_rank]);
    } else if (r >= kr_off && r < kr_off + rot) {
      const int i = (r - kr_off) >> 1;
      const float2 cs = table[(size_t)pos * (rot / 2) + i];
      const float a = sm[dim + 2 * i], c = sm[dim + 2 * i + 1];
      v = ((r - kr_off) & 1) ? c * cs.x + a * cs.y : a * cs.x - c * cs.y;
    }
    dst[r] = from_f<T>(v);
  }
}

struct LatentDecode {
  int B, heads, kv_rank, lat_w, window, max_blocks, block_size, splits;
  float scale;
  const int* seq_lens;
  const int* block_table;
  const float* sink;  // [heads] or null
};

// One block per (slot, head, split): the four warps take keys in turn, lanes own dimensions of the latent row.
constexpr int LD_MAX_REG = 32;  // lat_w <= 1024
template <typename T>
__global__ void __launch_bounds__(128)
latent_decode_kernel(const LatentDecode p, const T* __restrict__ q_lat, const T* __restrict__ cache, T* __restrict__ o_lat) {
  extern __shared__ float sm[];  // [lat_w] query, [4][kv_rank] partial outputs, [8] max / sum
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.seq_lens[b];
  if (pos < 0 || pos >= p.max_blocks * p.block_size) return;
  float* qs = sm;
  float* po = sm + p.lat_w;
  float* ml = po + 4 * p.kv_rank;
  for (int d = threadIdx.x; d < p.lat_w; d += 128) qs[d] = to_f(q_lat[((size_t)b * p.heads + h) * p.lat_w + d]);
  __syncthreads();
  const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int* bt = p.block_table + (size_t)b * p.max_blocks;
  float m = -INFINITY, l = 0.f, acc[LD_MAX_REG];
#pragma unroll
  for (int i = 0; i < LD_MAX_REG; ++i) acc[i] = 0.f;
  for (int j = first + warp; j <= pos; j += 4) {
    const T* row = cache + ((size_t)bt[j / p.block_size] * p.block_size + j % p.block_size) * p.lat_w;
    float c[LD_MAX_REG], s = 0.f;
#pragma unroll
    for (int i = 0; i < LD_MAX_REG; ++i) {
      const int d = lane + 32 * i;
      c[i] = d < p.lat_w ? to_f(row[d]) : 0.f;
      if (d < p.lat_w) s += c[i] * qs[d];
    }
    s = warp_sum(s) * p.scale;
    const float mn = fmaxf(m, s), corr = m == -INFINITY ? 0.f : expf(m - mn), w = expf(s - mn);
    l = l * corr + w;
    m = mn;
#pragma unroll
    for (int i = 0; i < LD_MAX_REG; ++i) acc[i] = acc[i] * corr + w * c[i];
  }
#pragma unroll
  for (int i = 0; i < LD_MAX_REG; ++i) {
    const int d = lane + 32 * i;
    if (d < p.kv_rank) po[(size_t)warp * p.kv_rank + d] = acc[i];
  }
  if (lane == 0) { ml[warp] = m; ml[4 + warp] = l; }
  __syncthreads();
  const float sk = p.sink != nullptr ? p.sink[h] : -INFINITY;
  float mt = sk;
  for (int w = 0; w < 4; ++w) mt = fmaxf(mt, ml[w]);
  float den = expf(sk - mt), f[4];
  for (int w = 0; w < 4; ++w) {
    f[w] = ml[w] == -INFINITY ? 0.f : expf(ml[w] - mt);
    den += f[w] * ml[4 + w];
  }
  for (int d = threadIdx.x; d < p.kv_rank; d += 128) {
    float v = 0.f;
    for (int w = 0; w < 4; ++w) v += f[w] * po[(size_t)w * p.kv_rank + d];
    o_lat[((size_t)b * p.heads + h) * p.kv_rank + d] = from_f<T>(v / den);
  }
}

// out[b, h, e] = gate[b, h] (1 without gates) * sum_r uv[h, e, r] o_lat[b, h, r]
template <typename T>
__global__ void __launch_bounds__(128)
latent_expand_kernel(const T* __restrict__ o_lat, const T* __restrict__ uv, const float* __restrict__ gate,
                     T* __restrict__ out, int heads, int vdim, int kv_rank, const int* __restrict__ positions) {
  extern __shared__ float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool live = positions[b] >= 0;
  for (int r = threadIdx.x; r < kv_rank; r += 128) sm[r] = live ? to_f(o_lat[((size_t)b * heads + h) * kv_rank + r]) : 0.f;
  __syncthreads();
  const float g = gate != nullptr ? gate[(size_t)b * heads + h] : 1.f;
  for (int e = warp; e < vdim; e += 4) {
    const T* w = uv + ((size_t)h * vdim + e) * kv_rank;
    float v = 0.f;
    for (int r = lane; r < kv_rank; r += 32) v += sm[r] * to_f(w[r]);
    v = warp_sum(v);
    if (lane == 0) out[((size_t)b * heads + h) * vdim + e] = from_f<T>(v * g);
  }
}

// ------------------------------------------------------------------------------------------------------------
// mLSTM.  State of a slot and head: S [dim, vdim], n [dim], m, all fp32.  n and m are kept twice, indexed by the parity
// of the number of tokens consumed, so that the blocks that share a head can all read the old values.
// ------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void mlstm_log_gates(float zi, float zf, float cap, float& ig, float& fg) {
  ig = cap * tanhf(zi / cap);
  fg = log_sigmoid_f(cap * tanhf(zf / cap));
}

// z [T, 2 heads] -> log input gates and log forget gates, both [T, heads]
__global__ void __launch_bounds__(256)
mlstm_gates_kernel(const float* __restrict__ z, const float* __restrict__ bias, float cap, int heads, long long n,
                   float* __restrict__ ig, float* __restrict__ fg) {
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / heads;
    const int h = (int)(i % heads);
    mlstm_log_gates(z[t * 2 * heads + h] + bias[h], z[t * 2 * heads + heads + h] + bias[heads + h], cap, ig[i], fg[i]);
  }
}

struct MlstmState {
  float* S;   // [slots, heads, dim, vdim]
  float* n;   // [2, slots, heads, dim]
  float* m;   // [2, slots, heads]
  int slots;
};

// Prompts token by token: grid (sequence, head, 32-column tile of vdim), 256 threads.  Every size and dtype.
template <typename T>
__global__ void __launch_bounds__(256)
mlstm_prompt_kernel(const T* __restrict__ qkv, long long ld, int k_off, int v_off, const float* __restrict__ ig,
                    const float* __restrict__ fg, const int* __restrict__ cu, const int* __restrict__ seq_slot, MlstmState st,
                    int heads, int dim, int vdim, float qscale, float* __restrict__ out) {
  extern __shared__ float sm[];
  __shared__ float red[64];
  float* S = sm;               // [dim][32]
  float* n = S + (size_t)dim * 32;
  float* qs = n + dim;
  float* ks = qs + dim;
  float* part = ks + dim;      // [8][32]
  const int seq = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * 32, tid = threadIdx.x;
  const int ec = tid & 31, g = tid >> 5, e = e0 + ec;
  for (int i = tid; i < dim * 32; i += 256) S[i] = 0.f;
  for (int i = tid; i < dim; i += 256) n[i] = 0.f;
  float m = 0.f;
  const int t0 = cu[seq], t1 = cu[seq + 1];
  for (int t = t0; t < t1; ++t) {
    __syncthreads();
    const T* row = qkv + (size_t)t * ld;
    for (int d = tid; d < dim; d += 256) {
      qs[d] = to_f(row[(size_t)h * dim + d]) * qscale;
      ks[d] = to_f(row[k_off + (size_t)h * dim + d]);
    }
    const float li = ig[(size_t)t * heads + h], lf = fg[(size_t)t * heads + h];
    const float mn = fmaxf(lf + m, li), keep = expf(lf + m - mn), wr = expf(li - mn);
    m = mn;
    const float v = e < vdim ? to_f(row[v_off + (size_t)h * vdim + e]) : 0.f;
    __syncthreads();
    float nq = 0.f;
    for (int d = tid; d < dim; d += 256) {
      const float nn = keep * n[d] + wr * ks[d];
      n[d] = nn;
      nq += nn * qs[d];
    }
    float acc = 0.f;
    for (int d = g; d < dim; d += 8) {
      const float s = keep * S[d * 32 + ec] + wr * ks[d] * v;
      S[d * 32 + ec] = s;
      acc += s * qs[d];
    }
    part[g * 32 + ec] = acc;
    nq = block_sum2(nq, 0.f, red).x;
    if (tid < 32 && e < vdim) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) o += part[w * 32 + tid];
      out[((size_t)t * heads + h) * vdim + e] = o / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
    }
  }
  __syncthreads();
  if (seq_slot == nullptr) return;
  const int slot = seq_slot[seq];
  if (slot < 0 || slot >= st.slots) return;
  const int par = (t1 - t0) & 1;
  for (int i = tid; i < dim * 32; i += 256) {
    const int d = i >> 5, c = e0 + (i & 31);
    if (c < vdim) st.S[(((size_t)slot * heads + h) * dim + d) * vdim + c] = S[i];
  }
  if (blockIdx.z == 0) {
    for (int d = tid; d < dim; d += 256) st.n[(((size_t)par * st.slots + slot) * heads + h) * dim + d] = n[d];
    if (tid == 0) st.m[((size_t)par * st.slots + slot) * heads + h] = m;
  }
}

// One token per slot: grid (head, slot, 16 * VEC-column tile of vdim), 256 threads = 16 column groups x 16 row groups.
// acc [rows, ld] fp32: q | k | v | output gate | input gate | forget gate.  It is read by several blocks, so the
// output kernel clears it.
template <int VEC>
__global__ void __launch_bounds__(256)
mlstm_step_kernel(const float* __restrict__ acc, long long ld, const float* __restrict__ gate_bias, float cap,
                  const int* __restrict__ seq_lens, MlstmState st, int heads, int dim, int vdim, float qscale,
                  float* __restrict__ out) {
  extern __shared__ float sm[];  // q [dim], k [dim], partial sums [16][16 VEC]
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, cg = tid & 15, rg = tid >> 4;
  const int pos = seq_lens[b];
  if (pos < 0) return;
  float* qs = sm;
  float* ks = sm + dim;
  float* part = ks + dim;
  const float* row = acc + (size_t)b * ld;
  const int qd = heads * dim, vd = heads * vdim;
  const int par = pos & 1;
  const size_t bh = (size_t)b * heads + h;
  const float* n_old = st.n + ((size_t)par * st.slots * heads + bh) * dim;
  float* n_new = st.n + ((size_t)(par ^ 1) * st.slots * heads + bh) * dim;
  const float m_old = st.m[(size_t)par * st.slots * heads + bh];
  float li, lf;
  const int gr = 2 * qd + 2 * vd;
  mlstm_log_gates(row[gr + h] + gate_bias[h], row[gr + heads + h] + gate_bias[heads + h], cap, li, lf);
  const float m = fmaxf(lf + m_old, li), keep = expf(lf + m_old - m), wr = expf(li - m);
  float nq = 0.f;
  for (int d = tid; d < dim; d += 256) {
    const float q = row[h * dim + d] * qscale, k = row[qd + h * dim + d];
    qs[d] = q;
    ks[d] = k * wr;
    const float nn = keep * n_old[d] + wr * k;
    if (blockIdx.z == 0) n_new[d] = nn;
    nq += nn * q;
  }
  if (blockIdx.z == 0 && tid == 0) st.m[(size_t)(par ^ 1) * st.slots * heads + bh] = m;
  nq = block_sum2(nq, 0.f, red).x;  // also orders the shared q and k
  const int e = blockIdx.z * 16 * VEC + cg * VEC;
  float o[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) o[i] = 0.f;
  if (e < vdim) {
    float v[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = row[2 * qd + h * vdim + e + i];
    float* S = st.S + bh * dim * vdim + e;
#pragma unroll 4
    for (int d = rg; d < dim; d += 16) {
      float s[VEC];
      if (VEC == 4) {
        const float4 t = *reinterpret_cast<const float4*>(S + (size_t)d * vdim);
        s[0] = t.x; s[1 % VEC] = t.y; s[2 % VEC] = t.z; s[3 % VEC] = t.w;
      } else {
        s[0] = S[(size_t)d * vdim];
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        s[i] = keep * s[i] + ks[d] * v[i];
        o[i] += s[i] * qs[d];
      }
      if (VEC == 4)
        *reinterpret_cast<float4*>(S + (size_t)d * vdim) = make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]);
      else
        S[(size_t)d * vdim] = s[0];
    }
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) part[rg * 16 * VEC + cg * VEC + i] = o[i];
  __syncthreads();
  const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
  for (int c = tid; c < 16 * VEC; c += 256) {
    const int ee = blockIdx.z * 16 * VEC + c;
    if (ee < vdim) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < 16; ++w) s += part[w * 16 * VEC + c];
      out[bh * vdim + ee] = s * inv;
    }
  }
}

// y = unit_rms(o per head) * norm * sigmoid(g).  G: dtype of the gate logits (g_ld elements between rows).  With
// `clear_row` the block also zeroes its share of the fp32 sums the step kernel has read.
template <typename T, typename G>
__global__ void __launch_bounds__(128)
mlstm_out_kernel(const float* __restrict__ o, const G* __restrict__ gl, long long g_ld, const float* __restrict__ norm,
                 float eps, int heads, int vdim, T* __restrict__ y, float* __restrict__ clear_row, long long clear_ld,
                 int clear_n) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x;
  const size_t row = blockIdx.y, base = (row * heads + h) * vdim;
  float ss = 0.f;
  const bool vec = ((vdim | (int)g_ld) & 3) == 0 && (reinterpret_cast<uintptr_t>(gl) & (4 * sizeof(G) - 1)) == 0;
  if (vec) {
    for (int e = 4 * threadIdx.x; e < vdim; e += 512) {
      const float4 v = load4(o + base + e);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int e = threadIdx.x; e < vdim; e += 128) ss += o[base + e] * o[base + e];
  }
  const float r = 1.f / sqrtf(block_sum2(ss, 0.f, red).x / (float)vdim + eps);
  if (vec) {
    for (int e = 4 * threadIdx.x; e < vdim; e += 512) {
      const float4 v = load4(o + base + e), w = load4(norm + h * vdim + e), g = load4(gl + row * g_ld + (size_t)h * vdim + e);
      store4(y + base + e, make_float4(v.x * r * w.x * sigmoid_f(g.x), v.y * r * w.y * sigmoid_f(g.y),
                                       v.z * r * w.z * sigmoid_f(g.z), v.w * r * w.w * sigmoid_f(g.w)));
    }
  } else for (int e = threadIdx.x; e < vdim; e += 128)
    y[base + e] = from_f<T>(o[base + e] * r * norm[h * vdim + e] * sigmoid_f(to_f(gl[row * g_ld + (size_t)h * vdim + e])));
  if (clear_row != nullptr) {
    // every head's gate logits belong to this block alone; the rest of the row (q, k, v, input and forget gates) has
    // been consumed by the step kernel.  clear_n = elements before / after the gates, dealt over the heads' blocks
    float* c = clear_row + row * clear_ld;
    __syncthreads();
    const int g0 = clear_n, vd = heads * vdim;
    for (int i = h * 128 + threadIdx.x; i < g0; i += heads * 128) c[i] = 0.f;
    for (int e = threadIdx.x; e < vdim; e += 128) c[g0 + h * vdim + e] = 0.f;
    for (int i = h * 128 + threadIdx.x; i < 2 * heads; i += heads * 128) c[g0 + vd + i] = 0.f;
  }
}

}  // namespace trlb

using namespace trlb;

namespace {

int grid_for(long long work, int per_block) {
  long long g = (work + per_block - 1) / per_block;
  const long long cap = (long long)trlb_host::sm_count() * 16;
  return (int)(g < 1 ? 1 : (g > cap ? cap : g));
}

// dynamic shared memory above the default limit has to be announced once per kernel
template <typename K>
bool allow_smem(K kern, size_t bytes) {
  if (bytes <= 48 * 1024) return true;
  if (bytes > 227 * 1024) return false;
  return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) == cudaSuccess;
}

using bf16 = __nv_bfloat16;

}  // namespace

#define PDL trlb_host::pdl_enabled()

TRLB_API int trlb_embed_scaled(const long long* ids, const void* emb, float* x, int T, int H, int V, float scale, int is_bf16,
                               cudaStream_t st) {
  if (T <= 0) return 0;
  if (is_bf16) return (int)trlb_host::launch_kernel(embed_scaled_kernel<bf16>, dim3(T), dim3(256), 0, st, PDL, ids, (const bf16*)emb, x, H, V, scale);
  return (int)trlb_host::launch_kernel(embed_scaled_kernel<float>, dim3(T), dim3(256), 0, st, PDL, ids, (const float*)emb, x, H, V, scale);
}

// copy may be null
TRLB_API int trlb_embed_normed(const long long* ids, const void* emb, const float* w, float* x, float* copy, int T, int H, int V, float scale,
                               float eps, float shift, int is_bf16, cudaStream_t st) {
  if (T <= 0) return 0;
  const dim3 blk(H >= 1024 ? 256 : 64);
  if (is_bf16) return (int)trlb_host::launch_kernel(embed_normed_kernel<bf16>, dim3(T), blk, 0, st, PDL, ids, (const bf16*)emb, w, x, copy, H, V, scale, eps, shift);
  return (int)trlb_host::launch_kernel(embed_normed_kernel<float>, dim3(T), blk, 0, st, PDL, ids, (const float*)emb, w, x, copy, H, V, scale, eps, shift);
}

// pairs [buckets + 1, H] in the dtype of emb; prev_state [slots] (decode: one row per slot) may be null, tok_slot in decode
TRLB_API int trlb_embed_pairs(const long long* ids, const void* emb, const void* pairs, float* x, int T, int H, int V, float scale,
                              long long mul_prev, long long mul_cur, long long buckets, const int* positions, const int* tok_slot,
                              long long* prev_state, int decode, int is_bf16, cudaStream_t st) {
  if (T <= 0) return 0;
  if (buckets <= 0 || positions == nullptr || (decode && prev_state == nullptr) || (!decode && prev_state != nullptr && tok_slot == nullptr))
    return -207;
  const PairEmbed p = {ids, positions, tok_slot, prev_state, mul_prev, mul_cur, buckets, T, H, V, decode, scale};
  const dim3 blk(H >= 1024 ? 256 : 64);
  if (is_bf16) return (int)trlb_host::launch_kernel(embed_pairs_kernel<bf16>, dim3(T), blk, 0, st, PDL, p, (const bf16*)emb, (const bf16*)pairs, x);
  return (int)trlb_host::launch_kernel(embed_pairs_kernel<float>, dim3(T), blk, 0, st, PDL, p, (const float*)emb, (const float*)pairs, x);
}

TRLB_API int trlb_dynamic_tanh(float* x, float* delta, const float* alpha, const float* w, const float* b, void* out, int T,
                               int H, int clear, int is_bf16, cudaStream_t st) {
  if (T <= 0) return 0;
  const bool v4 = (H % 4) == 0;
  const long long n = (long long)T * H / (v4 ? 4 : 1);
  const dim3 grid(grid_for(n, 256)), blk(256);
#define GO(TT, VV) (int)trlb_host::launch_kernel(dynamic_tanh_kernel<TT, VV>, grid, blk, 0, st, PDL, x, delta, alpha, w, b, (TT*)out, n, H, clear)
  if (is_bf16) return v4 ? GO(bf16, 4) : GO(bf16, 1);
  return v4 ? GO(float, 4) : GO(float, 1);
#undef GO
}

// post, post_scale, w, delta, delta2, y, anchor, bump, w2 may be null (see RmsResidual); H: row length
TRLB_API int trlb_rms_residual(float* x, float* delta, const float* post, const float* post_scale, const float* w, void* out, int T,
                               int H, float eps, float shift, float gain, float mult, int clear, const float* delta2, const void* y,
                               const int* row, const float* weight, int top, const float* anchor, const float* bump, const float* w2,
                               void* out2, int is_bf16, cudaStream_t st) {
  if (T <= 0) return 0;
  if ((delta == nullptr && (delta2 != nullptr || y != nullptr)) || (w2 != nullptr && (w == nullptr || out2 == nullptr))) return -208;
  const RmsResidual p = {x, delta, post, w, H, clear, eps, post_scale, shift, gain, mult, delta2, y, row, weight, top, anchor, bump, w2, out2};
  const int n4 = H / 4;
  const bool regs = H % 4 == 0 && n4 <= 256 * 8;
#define GO(TT, NN) (int)trlb_host::launch_kernel(rms_residual_kernel<TT, NN>, dim3(T), dim3(n4 >= 256 ? 256 : (n4 + 31) / 32 * 32), 0, st, PDL, p, (TT*)out)
#define PICK(TT) (n4 <= 256 ? GO(TT, 1) : n4 <= 512 ? GO(TT, 2) : n4 <= 1024 ? GO(TT, 4) : GO(TT, 8))
  if (regs) return is_bf16 ? PICK(bf16) : PICK(float);
#undef PICK
#undef GO
  if (is_bf16) return (int)trlb_host::launch_kernel(rms_residual_any_kernel<bf16>, dim3(T), dim3(256), 0, st, PDL, p, (bf16*)out);
  return (int)trlb_host::launch_kernel(rms_residual_any_kernel<float>, dim3(T), dim3(256), 0, st, PDL, p, (float*)out);
}

TRLB_API int trlb_clamped_glu(const void* z, void* out, int rows, int n, float limit, float alpha, float shift, int is_bf16,
                              cudaStream_t st) {
  if (rows <= 0 || n <= 0) return 0;
  const bool v4 = n % 4 == 0;
  const long long total = (long long)rows * n / (v4 ? 4 : 1);
#define GO(TT, VV) glu_kernel<TT, VV, false><<<grid_for(total, 256), 256, 0, st>>>((const TT*)z, (TT*)out, total, n, limit, alpha, shift)
  if (is_bf16) { if (v4) GO(bf16, 4); else GO(bf16, 1); }
  else { if (v4) GO(float, 4); else GO(float, 1); }
#undef GO
  return (int)cudaGetLastError();
}

// z [rows, 2 n] = gate | up -> gelu_tanh(gate) up
TRLB_API int trlb_gelu_glu(const void* z, void* out, int rows, int n, int is_bf16, cudaStream_t st) {
  if (rows <= 0 || n <= 0) return 0;
  const bool v4 = n % 4 == 0;
  const long long total = (long long)rows * n / (v4 ? 4 : 1);
#define GO(TT, VV) glu_kernel<TT, VV, true><<<grid_for(total, 256), 256, 0, st>>>((const TT*)z, (TT*)out, total, n, 0.f, 0.f, 0.f)
  if (is_bf16) { if (v4) GO(bf16, 4); else GO(bf16, 1); }
  else { if (v4) GO(float, 4); else GO(float, 1); }
#undef GO
  return (int)cudaGetLastError();
}

// z [rows, n] (fp32 if z_f32, else the dtype of the table), table [V, table_ld]
TRLB_API int trlb_side_gate(void* z, int z_f32, const long long* ids, const void* table, long long table_ld, int off, int rows,
                            int n, int V, int clear, void* out, int is_bf16, cudaStream_t st) {
  if (rows <= 0 || n <= 0) return 0;
  const bool v4 = ((n | off | (int)(table_ld & 3)) & 3) == 0 && (reinterpret_cast<uintptr_t>(table) & 15) == 0;
  const long long total = (long long)rows * n / (v4 ? 4 : 1);
#define GO(TT, ZZ, VV) (int)trlb_host::launch_kernel(side_gate_kernel<TT, ZZ, VV>, dim3(grid_for(total, 256)), dim3(256), 0, st, PDL, (ZZ*)z, ids, \
                                                     (const TT*)table, table_ld, off, n, total, V, clear, (TT*)out)
  if (is_bf16) return z_f32 ? (v4 ? GO(bf16, float, 4) : GO(bf16, float, 1)) : (v4 ? GO(bf16, bf16, 4) : GO(bf16, bf16, 1));
  return v4 ? GO(float, float, 4) : GO(float, float, 1);
#undef GO
}

TRLB_API int trlb_gelu_erf(const void* z, void* out, long long n, int is_bf16, cudaStream_t st) {
  if (n <= 0) return 0;
  if (is_bf16) gelu_erf_kernel<bf16><<<grid_for(n, 256), 256, 0, st>>>((const bf16*)z, (bf16*)out, n);
  else gelu_erf_kernel<float><<<grid_for(n, 256), 256, 0, st>>>((const float*)z, (float*)out, n);
  return (int)cudaGetLastError();
}

TRLB_API int trlb_latent_prep(float* acc, long long ld, int rows, int q_rank, int kv_rank, int rot, int heads, int clear,
                              const float* q_norm, const float* kv_norm, float eps, const int* positions,
                              const int* tok_slot, const float* table, int table_len, void* cq, void* lat, float* gate,
                              int kr_off, int lat_w, void* cache, const int* block_table, int max_blocks, int block_size,
                              int is_bf16, cudaStream_t st) {
  if (rows <= 0) return 0;
  if ((rot & 1) || kr_off < kv_rank || lat_w < kr_off + rot || (cache != nullptr && block_table == nullptr)) return -200;
  LatentPrep p = {acc, ld, q_rank, kv_rank, rot, heads, clear, q_norm, kv_norm, eps, positions, tok_slot,
                  (const float2*)table, table_len, gate, kr_off, lat_w, cache ? block_table : nullptr, max_blocks, block_size};
  const int widest = q_rank > kv_rank ? q_rank : kv_rank;
  const dim3 blk(widest > 512 ? 256 : widest > 256 ? 128 : 64);
  if (is_bf16)
    return (int)trlb_host::launch_kernel(latent_prep_kernel<bf16>, dim3(rows), blk, 0, st, PDL, p, (bf16*)cq, (bf16*)lat, (bf16*)cache);
  return (int)trlb_host::launch_kernel(latent_prep_kernel<float>, dim3(rows), blk, 0, st, PDL, p, (float*)cq, (float*)lat, (float*)cache);
}

TRLB_API int trlb_rotate_q(void* q, int rows, int heads, int dim, int rot, const int* positions, const float* table,
                           int table_len, int is_bf16, cudaStream_t st) {
  const bool two = dim % 4 == 0 && rot % 4 == 0;
  const long long n = (long long)rows * heads * (rot / 2) / (two ? 2 : 1);
  if (n <= 0) return 0;
#define GO(TT, PP) rotate_q_kernel<TT, PP><<<grid_for(n, 256), 256, 0, st>>>((TT*)q, heads, dim, rot, positions, (const float2*)table, table_len, n)
  if (is_bf16) { if (two) GO(bf16, 2); else GO(bf16, 1); }
  else { if (two) GO(float, 2); else GO(float, 1); }
#undef GO
  return (int)cudaGetLastError();
}

TRLB_API int trlb_latent_absorb(float* qacc, long long ld, const void* uk, void* q_lat, int B, int heads, int dim, int rot,
                                int kv_rank, int kr_off, int lat_w, const int* positions, const float* table,
                                int table_len, int clear, int is_bf16, cudaStream_t st) {
  if (B <= 0) return 0;
  const size_t smem = (size_t)(dim + rot) * 4;
  const dim3 grid(heads, B), blk(128);
  if (smem > 48 * 1024) return -202;
  if (is_bf16)
    return (int)trlb_host::launch_kernel(latent_absorb_kernel<bf16>, grid, blk, smem, st, PDL, qacc, ld, (const bf16*)uk, (bf16*)q_lat,
                                         heads, dim, rot, kv_rank, kr_off, lat_w, positions, (const float2*)table, table_len, clear);
  return (int)trlb_host::launch_kernel(latent_absorb_kernel<float>, grid, blk, smem, st, PDL, qacc, ld, (const float*)uk, (float*)q_lat,
                                       heads, dim, rot, kv_rank, kr_off, lat_w, positions, (const float2*)table, table_len, clear);
}

TRLB_API int trlb_latent_decode(const void* q_lat, const void* cache, void* o_lat, int B, int heads, int kv_rank, int lat_w,
                                int window, float scale, const int* seq_lens, const int* block_table, int max_blocks,
                                int block_size, const float* sink, int is_bf16, cudaStream_t st) {
  if (B <= 0) return 0;
  if (lat_w > 32 * LD_MAX_REG) return -203;
  LatentDecode p = {B, heads, kv_rank, lat_w, window, max_blocks, block_size, 1, scale, seq_lens, block_table, sink};
  const size_t smem = (size_t)(lat_w + 4 * kv_rank + 8) * 4;
  const dim3 grid(heads, B), blk(128);
  if (smem > 48 * 1024) return -203;
  if (is_bf16)
    return (int)trlb_host::launch_kernel(latent_decode_kernel<bf16>, grid, blk, smem, st, PDL, p, (const bf16*)q_lat, (const bf16*)cache, (bf16*)o_lat);
  return (int)trlb_host::launch_kernel(latent_decode_kernel<float>, grid, blk, smem, st, PDL, p, (const float*)q_lat, (const float*)cache, (float*)o_lat);
}

TRLB_API int trlb_latent_expand(const void* o_lat, const void* uv, const float* gate, void* out, int B, int heads, int vdim,
                                int kv_rank, const int* positions, int is_bf16, cudaStream_t st) {
  if (B <= 0) return 0;
  const size_t smem = (size_t)kv_rank * 4;
  const dim3 grid(heads, B), blk(128);
  if (smem > 48 * 1024) return -204;
  if (is_bf16)
    return (int)trlb_host::launch_kernel(latent_expand_kernel<bf16>, grid, blk, smem, st, PDL, (const bf16*)o_lat, (const bf16*)uv, gate, (bf16*)out, heads, vdim, kv_rank, positions);
  return (int)trlb_host::launch_kernel(latent_expand_kernel<float>, grid, blk, smem, st, PDL, (const float*)o_lat, (const float*)uv, gate, (float*)out, heads, vdim, kv_rank, positions);
}

TRLB_API int trlb_mlstm_gates(const float* z, const float* bias, float cap, int T, int heads, float* ig, float* fg, cudaStream_t st) {
  const long long n = (long long)T * heads;
  if (n <= 0) return 0;
  mlstm_gates_kernel<<<grid_for(n, 256), 256, 0, st>>>(z, bias, cap, heads, n, ig, fg);
  return (int)cudaGetLastError();
}

// qkv [T, ld]: q at 0, k at k_off, v at v_off (elements).  Sequences by cu [n_seq + 1]; seq_slot null: no state is kept.
TRLB_API int trlb_mlstm_prompt(const void* qkv, long long ld, int k_off, int v_off, const float* ig, const float* fg,
                               const int* cu, int n_seq, const int* seq_slot, float* S, float* n, float* m, int slots,
                               int heads, int dim, int vdim, float qscale, float* out, int is_bf16, cudaStream_t st) {
  if (n_seq <= 0) return 0;
  const size_t smem = (size_t)(dim * 32 + 3 * dim + 256) * 4;
  const dim3 grid(n_seq, heads, (vdim + 31) / 32);
  MlstmState s = {S, n, m, slots};
  if (is_bf16) {
    if (!allow_smem(mlstm_prompt_kernel<bf16>, smem)) return -205;
    mlstm_prompt_kernel<bf16><<<grid, 256, smem, st>>>((const bf16*)qkv, ld, k_off, v_off, ig, fg, cu, seq_slot, s, heads, dim, vdim, qscale, out);
  } else {
    if (!allow_smem(mlstm_prompt_kernel<float>, smem)) return -205;
    mlstm_prompt_kernel<float><<<grid, 256, smem, st>>>((const float*)qkv, ld, k_off, v_off, ig, fg, cu, seq_slot, s, heads, dim, vdim, qscale, out);
  }
  return (int)cudaGetLastError();
}

TRLB_API int trlb_mlstm_step(const float* acc, long long ld, const float* gate_bias, float cap, const int* seq_lens, float* S,
                             float* n, float* m, int slots, int B, int heads, int dim, int vdim, float qscale, float* out,
                             cudaStream_t st) {
  if (B <= 0) return 0;
  if (B > slots) return -206;
  MlstmState s = {S, n, m, slots};
  const bool v4 = (vdim % 4) == 0;
  const int tile = v4 ? 64 : 16;
  const dim3 grid(heads, B, (vdim + tile - 1) / tile), blk(256);
  const size_t smem = (size_t)(2 * dim + 16 * tile) * 4;
  if (smem > 48 * 1024) return -206;
  if (v4) return (int)trlb_host::launch_kernel(mlstm_step_kernel<4>, grid, blk, smem, st, PDL, acc, ld, gate_bias, cap, seq_lens, s, heads, dim, vdim, qscale, out);
  return (int)trlb_host::launch_kernel(mlstm_step_kernel<1>, grid, blk, smem, st, PDL, acc, ld, gate_bias, cap, seq_lens, s, heads, dim, vdim, qscale, out);
}

// g_bf16 / y_bf16: dtypes of the gate logits and of the output (bf16 else fp32).  clear_row (fp32 sums, gates at clear_n) may be null.
TRLB_API int trlb_mlstm_out(const float* o, const void* gl, long long g_ld, int g_bf16, const float* norm, float eps, int rows,
                            int heads, int vdim, void* y, int y_bf16, float* clear_row, long long clear_ld, int clear_n,
                            cudaStream_t st) {
  if (rows <= 0) return 0;
  const dim3 blk(128);
  // rows on y: prompts can be longer than 65535 tokens, so they are launched in slices
  for (int r0 = 0; r0 < rows; r0 += 32768) {
    const int nr = rows - r0 < 32768 ? rows - r0 : 32768;
    const dim3 grid(heads, nr);
    const size_t off = (size_t)r0 * heads * vdim;
    int rc;
#define GO(TT, GG) (int)trlb_host::launch_kernel(mlstm_out_kernel<TT, GG>, grid, blk, 0, st, PDL, o + off, (const GG*)gl + (size_t)r0 * g_ld, g_ld, \
                                                norm, eps, heads, vdim, (TT*)y + off, clear_row ? clear_row + (size_t)r0 * clear_ld : nullptr, clear_ld, clear_n)
    if (y_bf16) rc = g_bf16 ? GO(bf16, bf16) : GO(bf16, float);
    else rc = g_bf16 ? GO(float, bf16) : GO(float, float);
#undef GO
    if (rc) return rc;
  }
  return 0;
}
