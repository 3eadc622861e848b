// Token-wise kernels of the layer-by-layer designs: fp32 residual stream (embedding, norm), gated RMS norms of mixer outputs,
// per-head products, and the 32-bit forms of the matrix product, gated activation and greedy head.
#include "stream.cuh"

namespace lx {

// ------------------------------------------------------------------------------------------------
// Residual stream: x[t] = table[ids[t]] * mult (+ pos[positions[t]]) in fp32; `copy` takes x in the model's dtype.
// Pairs: the vector of (token before, token) is added too.  The token before a row is the row before it or, for a sequence's first row of
// the step, stands in the paged token ids, where every row leaves its own (a page's slot is written once per token, and read by the
// steps behind it only).
// ------------------------------------------------------------------------------------------------
struct EmbedPairs {
  const void* vectors;         // [buckets + 1, W], the last row for a sequence's first token; null: no pairs
  int* pages;                  // [blocks * page] token ids
  const int* slots;            // [T] slot of the row's token, < 0: none
  long long mul_prev, mul_cur;
  int buckets, page;
  StepRows rows;
};

// Token in front of row t, or -1.
LX_DEVICE int token_before(const EmbedPairs& e, const int* ids, int t) {
  int before;
  const int* bt;
  if (t < e.rows.nd) {
    before = e.rows.ctx_lens[t] - 1;
    bt = e.rows.dec_bt + (long long)t * e.rows.dec_max_blocks;
  } else {
    const int b = seq_of(e.rows, t - e.rows.nd), i = t - e.rows.nd - e.rows.cu_q[b];
    if (i > 0) return ids[t - 1];
    before = e.rows.cache_lens[b];
    bt = e.rows.bt + (long long)b * e.rows.max_blocks;
  }
  return before > 0 ? e.pages[(long long)bt[(before - 1) / e.page] * e.page + (before - 1) % e.page] : -1;
}

template <typename T>
__global__ void __launch_bounds__(128) embed_stream_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out,
                                                           int W, int V, float mult, const T* __restrict__ pos,
                                                           const int* __restrict__ positions, int P, T* __restrict__ copy,
                                                           const EmbedPairs pairs) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int id = min(max(ids[t], 0), V - 1);
  const int at = pos != nullptr ? min(max(positions[t], 0), P - 1) : 0;
  const T* pair = nullptr;
  if (pairs.vectors != nullptr) {
    const int prev = token_before(pairs, ids, t);
    const long long row = prev < 0 ? pairs.buckets : (min(prev, V - 1) * pairs.mul_prev + id * pairs.mul_cur) % pairs.buckets;
    pair = reinterpret_cast<const T*>(pairs.vectors) + row * W;
    if (threadIdx.x == 0 && pairs.slots[t] >= 0) pairs.pages[pairs.slots[t]] = id;
  }
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float f[8];
    load8(table + (long long)id * W + c, f);
#pragma unroll
    for (int q = 0; q < 8; ++q) f[q] *= mult;
    if (pos != nullptr) {
      float g[8];
      load8(pos + (long long)at * W + c, g);
#pragma unroll
      for (int q = 0; q < 8; ++q) f[q] += g[q];
    }
    if (pair != nullptr) {
      float g[8];
      load8(pair + c, g);
#pragma unroll
      for (int q = 0; q < 8; ++q) f[q] += g[q];
    }
    store8(out + (long long)t * W + c, f);
    if (copy != nullptr) store8(copy + (long long)t * W + c, f);
  }
}

// ------------------------------------------------------------------------------------------------
// residual += pending (fp32); out = residual / sqrt(sum / n + eps) * (w + w_offset).  One CTA per row.  PAIRS: what is added to a token is
// the weighted sum of the rows pos[t, 0 .. k) (-1: none) of pending (the outputs of its experts).  rows: only these rows, and the
// residual stays as it is.
// ------------------------------------------------------------------------------------------------
constexpr int kNsThreads = 256, kNsMaxVec = 8;      // 16384 columns at most

struct NormStreamParams {
  float* residual;
  const void* pending;         // [T or pairs, ldp] or null
  long long ldp;
  const float* w;
  void* out;
  const int* pos;              // [T, k]
  const float* weights;        // [T, k]
  const int* rows;             // or null
  int k, W;
  float inv_n, eps, w_offset;
};

template <typename T, bool PAIRS, int NV>
__global__ void __launch_bounds__(kNsThreads) norm_stream_kernel(const NormStreamParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[kNsThreads / 32];
  const int t = p.rows != nullptr ? p.rows[blockIdx.x] : (int)blockIdx.x;
  float* res = p.residual + (long long)t * p.W;
  const T* pending = reinterpret_cast<const T*>(p.pending);
  float v[NV][8];
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < NV; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
    if (c < p.W) {
      load8(res + c, v[it]);
      if (pending != nullptr) {
        if constexpr (PAIRS) {
          float sum[8];
#pragma unroll
          for (int q = 0; q < 8; ++q) sum[q] = 0.f;
          for (int j = 0; j < p.k; ++j) {
            const int row = p.pos[(long long)t * p.k + j];
            if (row < 0) continue;
            const float wj = p.weights[(long long)t * p.k + j];
            float f[8];
            load8(pending + (long long)row * p.ldp + c, f);
#pragma unroll
            for (int q = 0; q < 8; ++q) sum[q] = fmaf(wj, f[q], sum[q]);
          }
#pragma unroll
          for (int q = 0; q < 8; ++q) v[it][q] += sum[q];
        } else {
          float f[8];
          load8(pending + (long long)t * p.ldp + c, f);
#pragma unroll
          for (int q = 0; q < 8; ++q) v[it][q] += f[q];
        }
        if (p.rows == nullptr) store8(res + c, v[it]);
      }
#pragma unroll
      for (int q = 0; q < 8; ++q) ss += v[it][q] * v[it][q];
    }
  }
  const float r = rsqrtf(block_sum(ss, red) * p.inv_n + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + (long long)blockIdx.x * p.W;
#pragma unroll
  for (int it = 0; it < NV; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
    if (c < p.W) {
      float g[8];
      load8(p.w + c, g);
#pragma unroll
      for (int q = 0; q < 8; ++q) g[q] = v[it][q] * r * (g[q] + p.w_offset);
      store8(out + c, g);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// Norm of a sublayer's output, added to the stream: residual += mult * (norm(y) * w + b), copy = residual in the model's dtype.  One
// CTA per row.  Columns from n on are padding: they take no part in mean and variance, and w and b are zero there.  PAIRS: y of a
// token is the weighted sum of the rows pos[t, 0 .. k) (-1: none) of y (the outputs of its experts).  NEXT: y is multiplied by
// sigmoid(gate) first when there is one, and copy = norm(residual) * next_w, of `rows` only when given (the residual then stays as it is).
// ------------------------------------------------------------------------------------------------
struct NormAddParams {
  float* residual;
  const void* y;
  long long ldy;
  const float* w;
  const float* b;              // or null
  void* copy;                  // or null
  const int* pos;              // [T, k]
  const float* weights;        // [T, k]
  int k, W, n, layernorm;
  float inv_n, eps, mult;
  const void* gate;            // [T, ldg] or null
  long long ldg;
  const float* next_w;         // [W] (NEXT)
  const int* rows;             // or null
};

// In place on a row held as NV vectors of eight columns per thread: v <- norm(v) * w + b.
template <int NV>
LX_DEVICE void norm_row(float (&v)[NV][8], const float* __restrict__ w, const float* __restrict__ b, int W, int n, float inv_n, float eps,
                        int layernorm, float w_offset, float* red) {
  float mean = 0.f;
  if (layernorm) {
    float s = 0.f;
#pragma unroll
    for (int it = 0; it < NV; ++it)
#pragma unroll
      for (int q = 0; q < 8; ++q) s += v[it][q];                   // (padding holds zeros)
    mean = block_sum(s, red) * inv_n;
  }
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < NV; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      v[it][q] -= mean;
      if (c + q < n) ss += v[it][q] * v[it][q];
    }
  }
  const float r = rsqrtf(block_sum(ss, red) * inv_n + eps);
#pragma unroll
  for (int it = 0; it < NV; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
    if (c < W) {
      float g[8], h[8];
      load8(w + c, g);
#pragma unroll
      for (int q = 0; q < 8; ++q) h[q] = 0.f;
      if (b != nullptr) load8(b + c, h);
#pragma unroll
      for (int q = 0; q < 8; ++q) v[it][q] = v[it][q] * r * (g[q] + w_offset) + h[q];
    }
  }
}

template <typename T>
LX_DEVICE float gate_f(float z) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : sigmoid_f(z);
}

template <typename T, bool PAIRS, int NV, bool NEXT>
__global__ void __launch_bounds__(kNsThreads, NEXT && NV <= 2 ? 4 : 1) norm_add_kernel(const NormAddParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[kNsThreads / 32];
  const int t = NEXT && p.rows != nullptr ? p.rows[blockIdx.x] : (int)blockIdx.x;
  const T* y = reinterpret_cast<const T*>(p.y);
  float v[NV][8];
#pragma unroll
  for (int it = 0; it < NV; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
#pragma unroll
    for (int q = 0; q < 8; ++q) v[it][q] = 0.f;
    if (c >= p.W) continue;
    if constexpr (PAIRS) {
      for (int j = 0; j < p.k; ++j) {
        const int row = p.pos[(long long)t * p.k + j];
        if (row < 0) continue;
        const float wj = p.weights[(long long)t * p.k + j];
        float f[8];
        load8(y + (long long)row * p.ldy + c, f);
#pragma unroll
        for (int q = 0; q < 8; ++q) v[it][q] = fmaf(wj, f[q], v[it][q]);
      }
    } else {
      load8(y + (long long)t * p.ldy + c, v[it]);
    }
    if (NEXT && p.gate != nullptr) {
      float g[8];
      load8(reinterpret_cast<const T*>(p.gate) + (long long)t * p.ldg + c, g);
#pragma unroll
      for (int q = 0; q < 8; ++q) v[it][q] *= gate_f<T>(g[q]);
    }
  }
  float* res = p.residual + (long long)t * p.W;
  T* copy = reinterpret_cast<T*>(p.copy);
  if constexpr (NEXT) {
    constexpr bool EARLY = NV <= 2;            // the stream's row is on its way while the first norm is formed
    float x[EARLY ? NV : 1][8];
    if constexpr (EARLY) {
#pragma unroll
      for (int it = 0; it < NV; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < p.W) load8(res + c, x[it]);
      }
    }
    norm_row<NV>(v, p.w, nullptr, p.W, p.n, p.inv_n, p.eps, 0, 0.f, red);
#pragma unroll
    for (int it = 0; it < NV; ++it) {
      const int c = (threadIdx.x + it * blockDim.x) * 8;
      if (c < p.W) {
        float (&own)[8] = x[EARLY ? it : 0];
        if constexpr (!EARLY) load8(res + c, own);
#pragma unroll
        for (int q = 0; q < 8; ++q) v[it][q] = fmaf(p.mult, v[it][q], own[q]);
        if (p.rows == nullptr) store8(res + c, v[it]);
      }
    }
    norm_row<NV>(v, p.next_w, nullptr, p.W, p.n, p.inv_n, p.eps, 0, 0.f, red);
#pragma unroll
    for (int it = 0; it < NV; ++it) {
      const int c = (threadIdx.x + it * blockDim.x) * 8;
      if (c < p.W) store8(copy + (long long)blockIdx.x * p.W + c, v[it]);
    }
    return;
  }
  norm_row<NV>(v, p.w, p.b, p.W, p.n, p.inv_n, p.eps, p.layernorm, 0.f, red);
#pragma unroll
  for (int it = 0; it < NV; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
    if (c < p.W) {
      float x[8];
      load8(res + c, x);
#pragma unroll
      for (int q = 0; q < 8; ++q) x[q] = fmaf(p.mult, v[it][q], x[q]);
      store8(res + c, x);
      if (copy != nullptr) store8(copy + (long long)t * p.W + c, x);
    }
  }
}

// out[i] = norm(residual[rows[i]]) (rows null: every row)
template <typename T>
__global__ void __launch_bounds__(kNsThreads) norm_rows_kernel(const float* __restrict__ residual, const int* __restrict__ rows,
                                                               const float* __restrict__ w, const float* __restrict__ b, T* __restrict__ out,
                                                               int W, int n, float inv_n, float eps, float w_offset, int layernorm) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[kNsThreads / 32];
  const float* res = residual + (long long)(rows != nullptr ? rows[blockIdx.x] : (int)blockIdx.x) * W;
  float v[kNsMaxVec][8];
#pragma unroll
  for (int it = 0; it < kNsMaxVec; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
#pragma unroll
    for (int q = 0; q < 8; ++q) v[it][q] = 0.f;
    if (c < W) load8(res + c, v[it]);
  }
  norm_row<kNsMaxVec>(v, w, b, W, n, inv_n, eps, layernorm, w_offset, red);
#pragma unroll
  for (int it = 0; it < kNsMaxVec; ++it) {
    const int c = (threadIdx.x + it * blockDim.x) * 8;
    if (c < W) store8(out + (long long)blockIdx.x * W + c, v[it]);
  }
}

// ------------------------------------------------------------------------------------------------
// Gated RMS norm: every `group` columns of x (fp32) divided by their root mean square (over n columns), times weight, times
// sigmoid(gate) or silu(gate).  WARP: one warp per group (up to 512 columns), else one CTA per group.
// ------------------------------------------------------------------------------------------------
template <typename T, bool WARP>
__global__ void __launch_bounds__(256) norm_gate_kernel(const float* __restrict__ x, const float* __restrict__ w, const T* __restrict__ gate,
                                                        long long ldg, T* __restrict__ out, long long ldo, int groups, int group, float inv_n,
                                                        float eps, int silu) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const int t = blockIdx.x;
  const int lane = WARP ? (threadIdx.x & 31) : threadIdx.x;
  const int width = WARP ? 32 : blockDim.x;
  const int g = WARP ? blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.y;
  if (WARP && g >= groups) return;
  const long long base = (long long)t * groups * group + (long long)g * group;
  float ss = 0.f;
  for (int c = lane * 4; c < group; c += width * 4) {
    const float4 a = load4(x + base + c);
    ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
  }
  ss = WARP ? warp_sum(ss) : block_sum(ss, red);
  const float r = rsqrtf(ss * inv_n + eps);
  for (int c = lane * 4; c < group; c += width * 4) {
    float4 a = load4(x + base + c);
    const int col = g * group + c;
    const float4 ww = load4(w + col);
    const float4 z = load4(gate + (long long)t * ldg + col);
    if (silu) {
      a.x *= r * ww.x * silu_f(z.x); a.y *= r * ww.y * silu_f(z.y); a.z *= r * ww.z * silu_f(z.z); a.w *= r * ww.w * silu_f(z.w);
    } else {
      a.x *= r * ww.x * sigmoid_f(z.x); a.y *= r * ww.y * sigmoid_f(z.y); a.z *= r * ww.z * sigmoid_f(z.z); a.w *= r * ww.w * sigmoid_f(z.w);
    }
    store4(out + (long long)t * ldo + col, a);
  }
}

// ------------------------------------------------------------------------------------------------
// The gate first, then the norm: rows of H heads of vd columns (PP apart) of y (fp32) and z, u = y * silu(z) closed up to [H * vd], every
// `part` columns divided by their own root mean square, times w; zeros in the columns behind them up to ncols.  One CTA per (row, part).
// VEC: four columns per access; parts of up to kGnWarpPart columns then take a warp each.
// ------------------------------------------------------------------------------------------------
struct GateNormParams {
  const float* y;              // [T, H * PP]
  const void* z;               // [T, ldz]
  const float* w;              // [H * vd]
  void* out;                   // [T, ldo]
  long long ldz, ldo;
  int H, vd, PP, part, ncols;
  float eps;
};
constexpr int kGnThreads = 256, kGnVec = 8, kGnWarpPart = 32 * 4 * kGnVec;

template <typename T>
LX_DEVICE float gn_gate(float y, float z) {
  return sizeof(T) == 2 ? __fdividef(y * z, 1.f + __expf(-z)) : y * silu_f(z);
}

template <typename T, bool VEC, bool WARP>
__global__ void __launch_bounds__(kGnThreads) gate_norm_kernel(const GateNormParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[kGnThreads / 32];
  const int t = blockIdx.x, lane = WARP ? threadIdx.x & 31 : threadIdx.x;
  constexpr int width = WARP ? 32 : kGnThreads;
  const int first = (WARP ? blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.y) * p.part;
  const int inner = p.H * p.vd;
  const float* y = p.y + (long long)t * p.H * p.PP;
  const T* z = reinterpret_cast<const T*>(p.z) + (long long)t * p.ldz;
  T* out = reinterpret_cast<T*>(p.out) + (long long)t * p.ldo;
  if (blockIdx.y == 0)
    for (int c = inner + threadIdx.x; c < p.ncols; c += blockDim.x) put(out + c, 0.f);
  if (WARP && first >= inner) return;
  float ss = 0.f;
  if constexpr (VEC) {
    float4 v[kGnVec];                            // (part is at most kGnVec * 4 * width)
#pragma unroll
    for (int it = 0; it < kGnVec; ++it) {
      const int c = (lane + it * width) * 4;
      v[it] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < p.part) {
        const int col = first + c, at = p.vd == p.PP ? col : col / p.vd * p.PP + col % p.vd;
        const float4 a = load4(y + at), g = load4(z + at);
        v[it] = make_float4(gn_gate<T>(a.x, g.x), gn_gate<T>(a.y, g.y), gn_gate<T>(a.z, g.z), gn_gate<T>(a.w, g.w));
      }
      ss += v[it].x * v[it].x + v[it].y * v[it].y + v[it].z * v[it].z + v[it].w * v[it].w;
    }
    const float r = rsqrtf((WARP ? warp_sum(ss) : block_sum(ss, red)) / p.part + p.eps);
#pragma unroll
    for (int it = 0; it < kGnVec; ++it) {
      const int c = (lane + it * width) * 4;
      if (c < p.part) {
        const float4 w = load4(p.w + first + c);
        store4(out + first + c, make_float4(v[it].x * r * w.x, v[it].y * r * w.y, v[it].z * r * w.z, v[it].w * r * w.w));
      }
    }
  } else {
    auto value = [&](int col) {
      const int at = col / p.vd * p.PP + col % p.vd;
      return gn_gate<T>(y[at], to_f(z[at]));
    };
    for (int c = lane; c < p.part; c += width) {
      const float v = value(first + c);
      ss += v * v;
    }
    const float r = rsqrtf(block_sum(ss, red) / p.part + p.eps);
    for (int c = lane; c < p.part; c += width) put(out + first + c, value(first + c) * r * p.w[first + c]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) tanh_kernel(T* __restrict__ x, long long n8) {
  pdl_trigger();
  pdl_wait();
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n8; i += (long long)gridDim.x * blockDim.x) {
    float f[8];
    load8(x + i * 8, f);
#pragma unroll
    for (int q = 0; q < 8; ++q) f[q] = tanhf(f[q]);
    store8(x + i * 8, f);
  }
}

// out[t, i] = act(x[t, i]) (* x[t, I + i]) for fp32 rows
__global__ void __launch_bounds__(256) act_mul_f32_kernel(const float* __restrict__ x, float* __restrict__ out, int I, long long ldx,
                                                          long long ldo, long long total4, int act, int gated) {
  pdl_trigger();
  pdl_wait();
  const int per_row = I / 4;
  for (long long v = blockIdx.x * (long long)blockDim.x + threadIdx.x; v < total4; v += (long long)gridDim.x * blockDim.x) {
    const long long t = v / per_row;
    const int c = (int)(v % per_row) * 4;
    float4 a = load4(x + t * ldx + c);
    float* e = reinterpret_cast<float*>(&a);
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float z = e[q];
      if (act == 0) e[q] = silu_f(z);
      else if (act == 1) e[q] = 0.5f * z * (1.f + erff(z * 0.70710678118654752f));
      else if (act == 2) e[q] = 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
      else { const float r = fmaxf(z, 0.f); e[q] = act == 4 ? r * r : r; }
    }
    if (gated) {
      const float4 u = load4(x + t * ldx + I + c);
      a.x *= u.x; a.y *= u.y; a.z *= u.z; a.w *= u.w;
    }
    store4(out + t * ldo + c, a);
  }
}

// out[t, i] = g * sigmoid(alpha g) * (u + 1), g = min(x[t, i], limit), u = x[t, I + i] within +-limit.
template <typename T>
__global__ void __launch_bounds__(256) clamped_swiglu_kernel(const T* __restrict__ x, T* __restrict__ out, int I, long long ldx, long long ldo,
                                                             long long total, float alpha, float limit) {
  pdl_trigger();
  pdl_wait();
  const int per_row = I / 8;
  for (long long v = blockIdx.x * (long long)blockDim.x + threadIdx.x; v < total; v += (long long)gridDim.x * blockDim.x) {
    const long long t = v / per_row;
    const int c = (int)(v - t * per_row) * 8;
    float g[8], u[8];
    load8(x + t * ldx + c, g);
    load8(x + t * ldx + I + c, u);
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      const float a = fminf(g[q], limit), b = fminf(fmaxf(u[q], -limit), limit);
      g[q] = a * gate_f<T>(alpha * a) * (b + 1.f);
    }
    store8(out + t * ldo + c, g);
  }
}

// Greedy head over fp32 logits: arg-max (lowest index on ties) and its log-probability.
__global__ void __launch_bounds__(512) argmax_f32_kernel(const float* __restrict__ logits, long long ld, int V, int* __restrict__ ids,
                                                         float* __restrict__ lps, float softcap) {
  pdl_trigger();
  pdl_wait();
  const float* row = logits + (long long)blockIdx.x * ld;
  __shared__ float sm[16], red[16];
  __shared__ int si[16];
  float best = -INFINITY;
  int bi = 0x7fffffff;
  for (int i = threadIdx.x; i < V; i += blockDim.x) {
    float x = row[i];
    if (softcap > 0.f) x = softcap * tanhf(x / softcap);
    if (x > best) { best = x; bi = i; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ob = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
  }
  if ((threadIdx.x & 31) == 0) { sm[threadIdx.x >> 5] = best; si[threadIdx.x >> 5] = bi; }
  __syncthreads();
  best = sm[0]; bi = si[0];
  for (int i = 1; i < (int)(blockDim.x >> 5); ++i)
    if (sm[i] > best || (sm[i] == best && si[i] < bi)) { best = sm[i]; bi = si[i]; }
  float s = 0.f;
  for (int i = threadIdx.x; i < V; i += blockDim.x) {
    float x = row[i];
    if (softcap > 0.f) x = softcap * tanhf(x / softcap);
    s += expf(x - best);
  }
  s = block_sum(s, red);
  if (threadIdx.x == 0) {
    ids[blockIdx.x] = bi;
    if (lps) lps[blockIdx.x] = -logf(s);
  }
}

// ------------------------------------------------------------------------------------------------
// Batched product in true fp32: out[b][t, n] = sum_k x[b][t, k] * w[b][n, k] (* sigmoid(gate[t, b]), or of gate[t, b * N + n]).
// 64 x 64 tiles.
// ------------------------------------------------------------------------------------------------
struct BatchedGemmParams {
  const void* x; const void* w; void* out; const void* gate;
  long long ldx, sx, ldw, sw, ldo, so, ldg;
  int T, N, K;
  float out_scale;
  const float* bias;           // fp32 product: [N] or null
  int gate_wide;               // the gate has a column for every output column: b * N + n
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const BatchedGemmParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float xs[16][68], ws[16][68];
  const int b = blockIdx.z, t0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const float* x = reinterpret_cast<const float*>(p.x) + b * p.sx;
  const float* w = reinterpret_cast<const float*>(p.w) + b * p.sw;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int k = k0 + lk + q;
      xs[lk + q][lr] = (t0 + lr < p.T && k < p.K) ? x[(long long)(t0 + lr) * p.ldx + k] : 0.f;
      ws[lk + q][lr] = (n0 + lr < p.N && k < p.K) ? w[(long long)(n0 + lr) * p.ldw + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[4], c[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) { a[q] = xs[k][ty * 4 + q]; c[q] = ws[k][tx * 4 + q]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], c[j], acc[i][j]);
    }
    __syncthreads();
  }
  float* out = reinterpret_cast<float*>(p.out) + b * p.so;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + ty * 4 + i;
    if (t >= p.T) continue;
    const float* gate = p.gate ? reinterpret_cast<const float*>(p.gate) + (long long)t * p.ldg : nullptr;
    float s = gate && !p.gate_wide ? p.out_scale * sigmoid_f(gate[b]) : p.out_scale;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (gate && p.gate_wide && n < p.N) s = p.out_scale * sigmoid_f(gate[(long long)b * p.N + n]);
      if (n < p.N) out[(long long)t * p.ldo + n] = acc[i][j] * s + (p.bias != nullptr ? p.bias[n] : 0.f);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// The same product per head in bf16 on mma.sync (K and N of a head are small: the work is a batch of skinny products).  64 tokens x
// 64 columns per CTA of four warps, K in steps of 32 through a double-buffered shared-memory ring.
// ------------------------------------------------------------------------------------------------
LX_DEVICE void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
LX_DEVICE void ldsm4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}

constexpr int kGhK = 64, kGhLd = kGhK + 8;      // row pitch 144 bytes: eight rows of one ldmatrix hit different banks

__global__ void __launch_bounds__(128) gemm_heads_kernel(const BatchedGemmParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) __nv_bfloat16 xs[2][64 * kGhLd], ws[2][64 * kGhLd];
  const int b = blockIdx.z, t0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + b * p.sx;
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w) + b * p.sw;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  auto load = [&](int st, int k0) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = threadIdx.x + i * 128, r = c >> 3, k = k0 + (c & 7) * 8;
      const bool okx = t0 + r < p.T && k < p.K, okw = n0 + r < p.N && k < p.K;
      cp_async_16(&xs[st][r * kGhLd + (c & 7) * 8], okx ? x + (long long)(t0 + r) * p.ldx + k : x, okx);
      cp_async_16(&ws[st][r * kGhLd + (c & 7) * 8], okw ? w + (long long)(n0 + r) * p.ldw + k : w, okw);
    }
    cp_async_commit();
  };
  const int nk = (p.K + kGhK - 1) / kGhK;
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  load(0, 0);
  for (int s = 0; s < nk; ++s) {
    if (s + 1 < nk) load((s + 1) & 1, (s + 1) * kGhK); else cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t xa = smem_u32(xs[s & 1]) + ((warp * 16 + (lane & 15)) * kGhLd + (lane >> 4) * 8) * 2;
    const uint32_t wa = smem_u32(ws[s & 1]) + (((lane & 7) + (lane >> 4) * 8) * kGhLd + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int ks = 0; ks < kGhK / 16; ++ks) {
      uint32_t a[4];
      ldsm4(a[0], a[1], a[2], a[3], xa + ks * 32);
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        uint32_t b0, b1, b2, b3;
        ldsm4(b0, b1, b2, b3, wa + nt * 16 * kGhLd * 2 + ks * 32);
        mma16816(acc[2 * nt], a, b0, b1);
        mma16816(acc[2 * nt + 1], a, b2, b3);
      }
    }
    __syncthreads();
  }
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + b * p.so;
#pragma unroll
  for (int hr = 0; hr < 2; ++hr) {
    const int t = t0 + warp * 16 + (lane >> 2) + hr * 8;
    if (t >= p.T) continue;
    const __nv_bfloat16* gate = p.gate ? reinterpret_cast<const __nv_bfloat16*>(p.gate) + (long long)t * p.ldg : nullptr;
    float2 s = make_float2(1.f, 1.f);
    if (gate && !p.gate_wide) s.x = s.y = sigmoid_f(to_f(gate[b]));
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
      const int n = n0 + nt * 8 + (lane & 3) * 2;
      if (n >= p.N) continue;
      if (gate && p.gate_wide) {
        const float2 z = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(gate + (long long)b * p.N + n));
        s = make_float2(gate_f<__nv_bfloat16>(z.x), gate_f<__nv_bfloat16>(z.y));
      }
      *reinterpret_cast<uint32_t*>(out + (long long)t * p.ldo + n) = pack_bf16x2(acc[nt][2 * hr] * s.x, acc[nt][2 * hr + 1] * s.y);
    }
  }
}

}  // namespace lx

extern "C" {

int lx_embed_pairs_bytes() { return (int)sizeof(lx::EmbedPairs); }

// `f32` selects the element type of activations and weights everywhere below (0: bf16, 1: fp32).
int lx_embed_stream(const int* ids, const void* table, void* out, int T, int W, int V, float mult, const void* pos, const int* positions, int P,
                    void* copy, const void* pairs, int f32, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (W % 8 != 0 || V <= 0 || (pos != nullptr && P <= 0)) return -1;
  const EmbedPairs e = pairs != nullptr ? *reinterpret_cast<const EmbedPairs*>(pairs) : EmbedPairs{};
  if (e.vectors != nullptr && (e.buckets <= 0 || e.page <= 0 || e.mul_prev < 0 || e.mul_cur < 0 || e.slots == nullptr || e.pages == nullptr)) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  float* o = reinterpret_cast<float*>(out);
#define LX_ES(TY)                                                                                                                        \
  launch_pdl(embed_stream_kernel<TY>, dim3(T), dim3(128), 0, s, ids, reinterpret_cast<const TY*>(table), o, W, V, mult,                     \
             reinterpret_cast<const TY*>(pos), positions, P, reinterpret_cast<TY*>(copy), e)
  if (f32) LX_ES(float); else LX_ES(__nv_bfloat16);
#undef LX_ES
  return -(int)cudaGetLastError();
}

int lx_norm_add_bytes() { return (int)sizeof(lx::NormAddParams); }

// T: rows of y (with p.rows: of the result).
int lx_norm_add(const void* params, int T, int f32, void* stream) {
  using namespace lx;
  const NormAddParams& p = *reinterpret_cast<const NormAddParams*>(params);
  if (T <= 0) return 0;
  if (p.W % 8 != 0 || p.W > kNsThreads * kNsMaxVec * 8 || p.n <= 0 || p.n > p.W || p.ldy % 8 != 0 || p.ldy < p.W) return -1;
  if (p.next_w != nullptr && (p.b != nullptr || p.layernorm)) return -3;
  if (p.next_w != nullptr ? p.copy == nullptr || (p.gate != nullptr && p.ldg % 8 != 0) : p.gate != nullptr || p.rows != nullptr) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int threads = p.W / 8 >= kNsThreads ? kNsThreads : (p.W / 8 + 31) / 32 * 32;
  const int nv = (p.W / 8 + threads - 1) / threads;
#define LX_NA(TY, PR, NX)                                                                                   \
  if (nv <= 1) launch_pdl(norm_add_kernel<TY, PR, 1, NX>, dim3(T), dim3(threads), 0, s, p);                   \
  else if (nv <= 2) launch_pdl(norm_add_kernel<TY, PR, 2, NX>, dim3(T), dim3(threads), 0, s, p);              \
  else if (nv <= 4) launch_pdl(norm_add_kernel<TY, PR, 4, NX>, dim3(T), dim3(threads), 0, s, p);              \
  else launch_pdl(norm_add_kernel<TY, PR, kNsMaxVec, NX>, dim3(T), dim3(threads), 0, s, p);
#define LX_NAP(TY, NX)  \
  if (p.pos != nullptr) { LX_NA(TY, true, NX) } else { LX_NA(TY, false, NX) }
  if (f32) { if (p.next_w != nullptr) { LX_NAP(float, true) } else { LX_NAP(float, false) } }
  else { if (p.next_w != nullptr) { LX_NAP(__nv_bfloat16, true) } else { LX_NAP(__nv_bfloat16, false) } }
#undef LX_NAP
#undef LX_NA
  return -(int)cudaGetLastError();
}

int lx_norm_rows(const void* residual, const int* rows, const void* w, const void* b, void* out, int T, int W, int n, float eps, float w_offset,
                 int layernorm, int f32, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (W % 8 != 0 || W > kNsThreads * kNsMaxVec * 8 || n <= 0 || n > W) return -1;
  const int threads = W / 8 >= kNsThreads ? kNsThreads : (W / 8 + 31) / 32 * 32;
#define LX_NR(TY)                                                                                                                       \
  launch_pdl(norm_rows_kernel<TY>, dim3(T), dim3(threads), 0, reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<const float*>(residual), \
             rows, reinterpret_cast<const float*>(w), reinterpret_cast<const float*>(b), reinterpret_cast<TY*>(out), W, n, 1.f / n, eps, w_offset, \
             layernorm)
  if (f32) LX_NR(float); else LX_NR(__nv_bfloat16);
#undef LX_NR
  return -(int)cudaGetLastError();
}

int lx_norm_stream_bytes() { return (int)sizeof(lx::NormStreamParams); }

// T: rows of the result (p.rows null: of the residual too).
int lx_norm_stream(const void* params, int T, int f32, void* stream) {
  using namespace lx;
  const NormStreamParams& p = *reinterpret_cast<const NormStreamParams*>(params);
  if (T <= 0) return 0;
  if (p.W % 8 != 0 || p.W > kNsThreads * kNsMaxVec * 8 || p.ldp % 8 != 0) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int threads = p.W / 8 >= kNsThreads ? kNsThreads : (p.W / 8 + 31) / 32 * 32;
  const int nv = (p.W / 8 + threads - 1) / threads;
#define LX_NS(TY, PR)                                                                                   \
  if (nv <= 1) launch_pdl(norm_stream_kernel<TY, PR, 1>, dim3(T), dim3(threads), 0, s, p);                \
  else if (nv <= 2) launch_pdl(norm_stream_kernel<TY, PR, 2>, dim3(T), dim3(threads), 0, s, p);           \
  else if (nv <= 4) launch_pdl(norm_stream_kernel<TY, PR, 4>, dim3(T), dim3(threads), 0, s, p);           \
  else launch_pdl(norm_stream_kernel<TY, PR, kNsMaxVec>, dim3(T), dim3(threads), 0, s, p);
  if (f32) { if (p.pos != nullptr) { LX_NS(float, true) } else { LX_NS(float, false) } }
  else { if (p.pos != nullptr) { LX_NS(__nv_bfloat16, true) } else { LX_NS(__nv_bfloat16, false) } }
#undef LX_NS
  return -(int)cudaGetLastError();
}

int lx_gate_norm_bytes() { return (int)sizeof(lx::GateNormParams); }

int lx_gate_norm(const void* params, int T, int f32, void* stream) {
  using namespace lx;
  const GateNormParams& p = *reinterpret_cast<const GateNormParams*>(params);
  if (T <= 0) return 0;
  if (p.part <= 0 || p.vd <= 0 || p.vd > p.PP || p.H * p.vd % p.part != 0 || p.ncols < p.H * p.vd) return -1;
  const bool vec = p.vd % 4 == 0 && p.PP % 4 == 0 && p.part % 4 == 0 && p.ldz % 4 == 0 && p.ldo % 4 == 0 && p.part <= kGnVec * 4 * kGnThreads;
  const bool warp = vec && p.part <= kGnWarpPart;
  const int parts = p.H * p.vd / p.part, per = parts < 4 ? parts : 4;          // parts per CTA of warps
  const dim3 grid(T, warp ? (parts + per - 1) / per : parts), block(warp ? 32 * per : kGnThreads);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define LX_GN(TY)                                                                              \
  if (warp) launch_pdl(gate_norm_kernel<TY, true, true>, grid, block, 0, s, p);                  \
  else if (vec) launch_pdl(gate_norm_kernel<TY, true, false>, grid, block, 0, s, p);             \
  else launch_pdl(gate_norm_kernel<TY, false, false>, grid, block, 0, s, p);
  if (f32) { LX_GN(float) } else { LX_GN(__nv_bfloat16) }
#undef LX_GN
  return -(int)cudaGetLastError();
}

int lx_norm_gate(const void* x, const void* w, const void* gate, long long ldg, void* out, long long ldo, int T, int groups, int group, int n,
                 float eps, int silu, int f32, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (group % 4 != 0 || ldg % 4 != 0 || ldo % 4 != 0 || n <= 0) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool warp = group <= 512;
  const int wpb = groups < 8 ? groups : 8;
  const dim3 grid(T, warp ? (groups + wpb - 1) / wpb : groups), block(warp ? 32 * wpb : 256);
  const float* xp = reinterpret_cast<const float*>(x);
  const float* wp = reinterpret_cast<const float*>(w);
#define LX_NG(TY, WP)                                                                                                                  \
  launch_pdl(norm_gate_kernel<TY, WP>, grid, block, 0, s, xp, wp, reinterpret_cast<const TY*>(gate), ldg, reinterpret_cast<TY*>(out), ldo, \
             groups, group, 1.f / n, eps, silu)
  if (f32) { if (warp) LX_NG(float, true); else LX_NG(float, false); }
  else { if (warp) LX_NG(__nv_bfloat16, true); else LX_NG(__nv_bfloat16, false); }
#undef LX_NG
  return -(int)cudaGetLastError();
}

int lx_tanh(void* x, long long n, int f32, void* stream) {
  using namespace lx;
  if (n <= 0) return 0;
  if (n % 8 != 0) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const long long n8 = n / 8;
  const int grid = (int)((n8 + 255) / 256 < 148 * 8 ? (n8 + 255) / 256 : 148 * 8);
  if (f32) launch_pdl(tanh_kernel<float>, dim3(grid), dim3(256), 0, s, reinterpret_cast<float*>(x), n8);
  else launch_pdl(tanh_kernel<__nv_bfloat16>, dim3(grid), dim3(256), 0, s, reinterpret_cast<__nv_bfloat16*>(x), n8);
  return -(int)cudaGetLastError();
}

int lx_act_mul_f32(const void* x, void* out, int T, int I, long long ldx, long long ldo, int act, int gated, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (I % 4 != 0 || ldx % 4 != 0 || ldo % 4 != 0) return -1;
  const long long total = (long long)T * (I / 4);
  const int grid = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  launch_pdl(act_mul_f32_kernel, dim3(grid), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<const float*>(x),
             reinterpret_cast<float*>(out), I, ldx, ldo, total, act, gated);
  return -(int)cudaGetLastError();
}

int lx_clamped_swiglu(const void* x, void* out, int T, int I, long long ldx, long long ldo, float alpha, float limit, int f32, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (I % 8 != 0 || ldx % 8 != 0 || ldo % 8 != 0) return -1;
  const long long total = (long long)T * (I / 8);
  const int grid = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define LX_CS(TY) \
  launch_pdl(clamped_swiglu_kernel<TY>, dim3(grid), dim3(256), 0, s, reinterpret_cast<const TY*>(x), reinterpret_cast<TY*>(out), I, ldx, ldo, total, alpha, limit)
  if (f32) LX_CS(float); else LX_CS(__nv_bfloat16);
#undef LX_CS
  return -(int)cudaGetLastError();
}

int lx_argmax_f32(const void* logits, long long ld, int T, int V, int* ids, float* logprobs, float softcap, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  launch_pdl(argmax_f32_kernel, dim3(T), dim3(512), 0, reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<const float*>(logits), ld, V, ids,
             logprobs, softcap);
  return -(int)cudaGetLastError();
}

// out[b][t, n] = x[b][t, :] . w[b][n, :] over `batch` products with element strides sx / sw / so; gate [T, ldg]: column b, or
// (gate_wide) column b * N + n.  bias [N]: fp32 only.
int lx_gemm_batched(const void* x, long long ldx, long long sx, const void* w, long long ldw, long long sw, void* out, long long ldo,
                    long long so, const void* gate, long long ldg, int T, int N, int K, int batch, float out_scale, const float* bias, int gate_wide,
                    int f32, void* stream) {
  using namespace lx;
  if (T <= 0 || N <= 0 || batch <= 0) return 0;
  BatchedGemmParams p{x, w, out, gate, ldx, sx, ldw, sw, ldo, so, ldg, T, N, K, out_scale, bias, gate_wide};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((N + 63) / 64, (T + 63) / 64, batch);
  if (bias != nullptr && !f32) return -2;
  if (f32) {
    launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, s, p);
  } else {
    if (K % 8 != 0 || N % 2 != 0 || ldx % 8 != 0 || sx % 8 != 0 || ldw % 8 != 0 || sw % 8 != 0 || ldo % 2 != 0 || so % 2 != 0) return -1;
    if (gate_wide && ldg % 2 != 0) return -3;
    launch_pdl(gemm_heads_kernel, grid, dim3(128), 0, s, p);
  }
  return -(int)cudaGetLastError();
}

}  // extern "C"
