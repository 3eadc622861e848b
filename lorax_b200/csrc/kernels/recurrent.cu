// Linear recurrences with a matrix state per head and request, S [d, dv] in fp32:
//
//   linear attention  S <- decay_h S + k v^T,        o = S^T q            (q, k, v pass through silu; decay constant per head)
//   WKV               o = (S + diag(u) k v^T)^T r,   S <- diag(w) S + k v^T   (w = exp(-exp(z + w0)) per token and key channel)
//   SSD               S <- exp(A_h s) S + s k v^T,   o = S^T q + D_h v        (Mamba-2: s = softplus(z + w0) per token and head; q, k, v
//                     are C, B, x, and hpg heads share q and k)
//
// Decode rows take one step each: the state streams through once (read, update, write).  Prompt tokens are cut into segments.  A first
// pass computes every segment's own contribution to the state and its total decay, a second one carries the state over the segments of
// a sequence, a third one runs through the segments again from their true initial states and writes the outputs.  A sequence of a
// single segment needs the last pass only.  A sequence whose first token is at position 0 starts from zeros whatever its slot holds.
#include "stream.cuh"

namespace lx {

enum RecMode : int { kLinAttn = 0, kWkv = 1, kSsd = 2 };

struct RecParams {
  const void* q;            // [T, ldq] q (linear attention) or r (WKV), head h at column (h / hpg) * d
  const void* k;
  const void* v;            // head h at column h * dv
  const void* z;            // WKV: decay logits [T, ldz]; SSD: step sizes before the softplus, head h at column h
  long long ldq, ldk, ldv, ldz;
  const float* decay;       // linear attention: [H]
  const float* w0;          // WKV: [H * d]; SSD: [H]
  const float* u;           // WKV: [H * d]; SSD: A [H], negative
  const float* skip;        // SSD: D [H]
  float* state;             // [slots, H, d, dv]
  float* out;               // [T, H * dv]
  int H, d, dv, hpg;
  StepRows rows;
  // prefill segments
  const int* seg_seq;       // [nseg]
  const int* seg_q0;        // [nseg] first token of the segment within its sequence
  int nseg, seg_len;
  float* seg_state;         // [nseg, H, d, dv]: contribution of the segment, then the state in front of it
  float* seg_decay;         // product of the segment's decays: WKV [nseg, H, d], SSD [nseg, H]
};

// ------------------------------------------------------------------------------------------------
// Decode: one CTA per (row, head).  Thread = four columns x every RG-th row of the state.
// ------------------------------------------------------------------------------------------------
constexpr int kRecStepThreads = 256;

template <typename T, int MODE>
__global__ void __launch_bounds__(kRecStepThreads) rec_step_kernel(const RecParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  const int t = blockIdx.x, h = blockIdx.y, d = p.d, dv = p.dv;
  float* sq = sm;                 // [d]
  float* sk = sq + d;             // [d]
  float* sw = sk + d;             // [d]
  float* sv = sw + d;             // [dv]
  float* part = sv + dv;          // [row groups][dv]
  __shared__ float red[kRecStepThreads / 32];
  const int ctx = p.rows.ctx_lens[t];
  float* out = p.out + ((long long)t * p.H + h) * dv;
  if (ctx <= 0) {
    for (int c = threadIdx.x; c < dv; c += blockDim.x) out[c] = 0.f;
    return;
  }
  const int hk = MODE == kSsd ? h / p.hpg : h;
  const T* q = reinterpret_cast<const T*>(p.q) + (long long)t * p.ldq + hk * d;
  const T* k = reinterpret_cast<const T*>(p.k) + (long long)t * p.ldk + hk * d;
  const T* v = reinterpret_cast<const T*>(p.v) + (long long)t * p.ldv + h * dv;
  float bonus = 0.f, size = 1.f, lam = 1.f;
  if (MODE == kSsd) {
    size = softplus_f(to_f(reinterpret_cast<const T*>(p.z)[(long long)t * p.ldz + h]) + p.w0[h]);
    lam = expf(p.u[h] * size);
  }
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    float a = to_f(q[i]), b = to_f(k[i]);
    if (MODE == kLinAttn) {
      a = silu_f(a); b = silu_f(b);
      sw[i] = p.decay[h];
    } else if (MODE == kSsd) {
      b *= size;
      sw[i] = lam;
    } else {
      const T* z = reinterpret_cast<const T*>(p.z) + (long long)t * p.ldz + h * d;
      sw[i] = expf(-expf(to_f(z[i]) + p.w0[h * d + i]));
      bonus += a * p.u[h * d + i] * b;
    }
    sq[i] = a;
    sk[i] = b;
  }
  for (int c = threadIdx.x; c < dv; c += blockDim.x) sv[c] = MODE == kLinAttn ? silu_f(to_f(v[c])) : to_f(v[c]);
  if (MODE == kWkv) bonus = block_sum(bonus, red);
  __syncthreads();
  const int nc = dv / 4, rg_n = blockDim.x / nc;
  const int c4 = threadIdx.x % nc, rg = threadIdx.x / nc;
  const bool fresh = ctx == 1;
  float* S = p.state + ((long long)p.rows.dec_slots[t] * p.H + h) * d * dv;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (rg < rg_n) {
    const float4 vv = *reinterpret_cast<const float4*>(sv + c4 * 4);
    for (int i0 = rg; i0 < d; i0 += rg_n * 4) {
      float4 s[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = i0 + j * rg_n;
        s[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < d && !fresh) s[j] = *reinterpret_cast<const float4*>(S + (long long)i * dv + c4 * 4);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = i0 + j * rg_n;
        if (i < d) {
          const float a = sq[i], kk = sk[i], w = sw[i];
          if (MODE == kWkv) { o.x += a * s[j].x; o.y += a * s[j].y; o.z += a * s[j].z; o.w += a * s[j].w; }
          s[j].x = w * s[j].x + kk * vv.x; s[j].y = w * s[j].y + kk * vv.y;
          s[j].z = w * s[j].z + kk * vv.z; s[j].w = w * s[j].w + kk * vv.w;
          if (MODE != kWkv) { o.x += a * s[j].x; o.y += a * s[j].y; o.z += a * s[j].z; o.w += a * s[j].w; }
          *reinterpret_cast<float4*>(S + (long long)i * dv + c4 * 4) = s[j];
        }
      }
    }
    *reinterpret_cast<float4*>(part + rg * dv + c4 * 4) = o;
  }
  __syncthreads();
  for (int c = threadIdx.x; c < dv; c += blockDim.x) {
    float s = MODE == kWkv ? bonus * sv[c] : MODE == kSsd ? p.skip[h] * sv[c] : 0.f;
    for (int g = 0; g < rg_n; ++g) s += part[g * dv + c];
    out[c] = s;
  }
}

// ------------------------------------------------------------------------------------------------
// Prefill segments, token by token: one CTA per (segment, head, 64 columns).  A warp owns RPT rows of the state for all 64 columns
// (two per lane) in registers; q, k and the decays of a block of tokens are staged in shared memory and read as broadcasts.
// STATES: compute the segment's contribution to the state only (first pass); else outputs and, at the end of a sequence, its state.
// ------------------------------------------------------------------------------------------------
template <typename T, int MODE, int RPT, bool STATES>
__global__ void __launch_bounds__(256) rec_scan_kernel(const RecParams p, int tc) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  const int seg = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * 64, d = p.d, dv = p.dv;
  const int b = p.seg_seq[seg], q0 = p.seg_q0[seg];
  const int r0 = p.rows.cu_q[b], qlen = p.rows.cu_q[b + 1] - r0;
  const int n = min(p.seg_len, qlen - q0);
  const bool last = q0 + p.seg_len >= qlen;
  if (STATES && last) return;                      // nothing follows the last segment
  const int nw = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row0 = warp * RPT;
  const int ca = c0 + 2 * lane;                    // this thread's columns ca, ca + 1
  const bool live = ca < dv;
  float* sq = sm;                                  // [tc][d]
  float* sk = sq + tc * d;
  float* sw = sk + tc * d;                         // WKV only
  float* sv = sw + (MODE == kWkv ? tc * d : 0);    // [tc][64]
  float* part = sv + tc * 64;                      // [tc][warps][64]
  float* bonus = part + (STATES ? 0 : tc * nw * 64);   // [tc]; SSD: the tokens' decays
  float* ssize = bonus + tc;                       // SSD: the tokens' step sizes
  float lam = MODE == kLinAttn ? p.decay[h] : 0.f;
  const int hk = MODE == kSsd ? h / p.hpg : h;

  float2 S[RPT];
  // (a sequence of several segments reads its first state from the carry pass too: its last segment overwrites the slot meanwhile)
  const float* init = nullptr;
  if (!STATES) {
    if (qlen > p.seg_len) init = p.seg_state + ((long long)seg * p.H + h) * d * dv;
    else if (p.rows.cache_lens[b] > 0) init = p.state + ((long long)p.rows.slots[b] * p.H + h) * d * dv;
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    S[i] = make_float2(0.f, 0.f);
    if (init != nullptr && live && row0 + i < d) S[i] = *reinterpret_cast<const float2*>(init + (long long)(row0 + i) * dv + ca);
  }
  float dprod[2] = {1.f, 1.f};                     // decay products of channels threadIdx.x and threadIdx.x + blockDim.x
  const long long tok0 = (long long)p.rows.nd + r0 + q0;
  for (int t0 = 0; t0 < n; t0 += tc) {
    const int m = min(tc, n - t0);
    __syncthreads();
    if (MODE == kSsd) {
      if ((int)threadIdx.x < m) {
        const float z = to_f(reinterpret_cast<const T*>(p.z)[(tok0 + t0 + threadIdx.x) * p.ldz + h]);
        const float size = softplus_f(z + p.w0[h]);
        ssize[threadIdx.x] = size;
        bonus[threadIdx.x] = expf(p.u[h] * size);
      }
      __syncthreads();
    }
    for (int e = threadIdx.x * 4; e < m * d; e += blockDim.x * 4) {
      const int tt = e / d, i = e % d;
      const long long tok = tok0 + t0 + tt;
      float4 kk = load4(reinterpret_cast<const T*>(p.k) + tok * p.ldk + hk * d + i);
      float4 qq = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!STATES) qq = load4(reinterpret_cast<const T*>(p.q) + tok * p.ldq + hk * d + i);
      if (MODE == kSsd) {
        const float size = ssize[tt];
        kk = make_float4(kk.x * size, kk.y * size, kk.z * size, kk.w * size);
      } else if (MODE == kLinAttn) {
        kk = make_float4(silu_f(kk.x), silu_f(kk.y), silu_f(kk.z), silu_f(kk.w));
        if (!STATES) qq = make_float4(silu_f(qq.x), silu_f(qq.y), silu_f(qq.z), silu_f(qq.w));
      } else {
        const float4 z = load4(reinterpret_cast<const T*>(p.z) + tok * p.ldz + h * d + i);
        const float4 w0 = load4(p.w0 + h * d + i);
        *reinterpret_cast<float4*>(sw + e) =
            make_float4(expf(-expf(z.x + w0.x)), expf(-expf(z.y + w0.y)), expf(-expf(z.z + w0.z)), expf(-expf(z.w + w0.w)));
      }
      *reinterpret_cast<float4*>(sk + e) = kk;
      if (!STATES) *reinterpret_cast<float4*>(sq + e) = qq;
    }
    for (int e = threadIdx.x * 4; e < m * 64; e += blockDim.x * 4) {
      const int tt = e >> 6, c = c0 + (e & 63);
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < dv) v = load4(reinterpret_cast<const T*>(p.v) + (tok0 + t0 + tt) * p.ldv + h * dv + c);
      if (MODE == kLinAttn) v = make_float4(silu_f(v.x), silu_f(v.y), silu_f(v.z), silu_f(v.w));
      *reinterpret_cast<float4*>(sv + e) = v;
    }
    __syncthreads();
    if (MODE == kSsd) {
      if (STATES && threadIdx.x == 0)
        for (int tt = 0; tt < m; ++tt) dprod[0] *= bonus[tt];
    }
    if (MODE == kWkv) {
      if (STATES) {
        if (blockIdx.z == 0) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int i = threadIdx.x + j * blockDim.x;
            if (i < d)
              for (int tt = 0; tt < m; ++tt) dprod[j] *= sw[tt * d + i];
          }
        }
      } else {
        for (int tt = warp; tt < m; tt += nw) {
          float s = 0.f;
          for (int i = lane; i < d; i += 32) s += sq[tt * d + i] * p.u[h * d + i] * sk[tt * d + i];
          s = warp_sum(s);
          if (lane == 0) bonus[tt] = s;
        }
      }
    }
    for (int tt = 0; tt < m; ++tt) {
      const float2 v = *reinterpret_cast<const float2*>(sv + tt * 64 + 2 * lane);
      float ox = 0.f, oy = 0.f;
      if (MODE == kSsd) lam = bonus[tt];
#pragma unroll
      for (int i = 0; i < RPT; i += 4) {
        if (row0 + i < d) {
          const float4 k4 = *reinterpret_cast<const float4*>(sk + tt * d + row0 + i);
          float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f), w4 = make_float4(lam, lam, lam, lam);
          if (!STATES) q4 = *reinterpret_cast<const float4*>(sq + tt * d + row0 + i);
          if (MODE == kWkv) w4 = *reinterpret_cast<const float4*>(sw + tt * d + row0 + i);
          const float ka[4] = {k4.x, k4.y, k4.z, k4.w}, qa[4] = {q4.x, q4.y, q4.z, q4.w}, wa[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            if (MODE == kWkv && !STATES) { ox = fmaf(qa[j], S[i + j].x, ox); oy = fmaf(qa[j], S[i + j].y, oy); }
            S[i + j].x = fmaf(wa[j], S[i + j].x, ka[j] * v.x);
            S[i + j].y = fmaf(wa[j], S[i + j].y, ka[j] * v.y);
            if (MODE != kWkv && !STATES) { ox = fmaf(qa[j], S[i + j].x, ox); oy = fmaf(qa[j], S[i + j].y, oy); }
          }
        }
      }
      if (!STATES) *reinterpret_cast<float2*>(part + (tt * nw + warp) * 64 + 2 * lane) = make_float2(ox, oy);
    }
    if (!STATES) {
      __syncthreads();
      for (int e = threadIdx.x; e < m * 64; e += blockDim.x) {
        const int tt = e >> 6, c = e & 63;
        if (c0 + c < dv) {
          float s = MODE == kWkv ? bonus[tt] * sv[e] : MODE == kSsd ? p.skip[h] * sv[e] : 0.f;
          for (int g = 0; g < nw; ++g) s += part[(tt * nw + g) * 64 + c];
          p.out[(tok0 + t0 + tt) * (long long)p.H * dv + (long long)h * dv + c0 + c] = s;
        }
      }
    }
  }
  float* dst = nullptr;
  if (STATES) dst = p.seg_state + ((long long)seg * p.H + h) * d * dv;
  else if (last) dst = p.state + ((long long)p.rows.slots[b] * p.H + h) * d * dv;
  if (dst != nullptr && live) {
#pragma unroll
    for (int i = 0; i < RPT; ++i)
      if (row0 + i < d) *reinterpret_cast<float2*>(dst + (long long)(row0 + i) * dv + ca) = S[i];
  }
  if (STATES && MODE == kSsd && blockIdx.z == 0 && threadIdx.x == 0) p.seg_decay[(long long)seg * p.H + h] = dprod[0];
  if (STATES && MODE == kWkv && blockIdx.z == 0) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < d) p.seg_decay[((long long)seg * p.H + h) * d + i] = dprod[j];
    }
  }
}

// Second pass: the state in front of every segment of a sequence, from the segments' contributions (in place).
template <int MODE>
__global__ void __launch_bounds__(256) rec_carry_kernel(const RecParams p) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y;
  const int e = (blockIdx.z * blockDim.x + threadIdx.x) * 4;
  const int dd = p.d * p.dv;
  if (e >= dd) return;
  const int qlen = p.rows.cu_q[b + 1] - p.rows.cu_q[b];
  const int ns = (qlen + p.seg_len - 1) / p.seg_len;
  if (ns <= 1) return;
  int lo = 0, hi = p.nseg;                        // first segment of the sequence
  while (lo < hi) {
    const int mid = (lo + hi) >> 1;
    if (p.seg_seq[mid] < b) lo = mid + 1; else hi = mid;
  }
  const int row = e / p.dv;
  float4 run = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.rows.cache_lens[b] > 0) run = load4(p.state + ((long long)p.rows.slots[b] * p.H + h) * dd + e);
  const float lam = MODE == kLinAttn ? powf(p.decay[h], (float)p.seg_len) : 0.f;
  for (int j0 = 0; j0 < ns; j0 += 8) {            // eight segments' loads in flight: only the sums are a chain
    float4 own[8];
    float w[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const long long at = (long long)(lo + j0 + u) * p.H + h;
      own[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      w[u] = lam;
      if (j0 + u + 1 < ns) {
        own[u] = load4(p.seg_state + at * dd + e);
        if (MODE == kWkv) w[u] = p.seg_decay[at * p.d + row];
        if (MODE == kSsd) w[u] = p.seg_decay[at];
      }
    }
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      if (j0 + u >= ns) break;
      store4(p.seg_state + ((long long)(lo + j0 + u) * p.H + h) * dd + e, run);
      run.x = w[u] * run.x + own[u].x; run.y = w[u] * run.y + own[u].y;
      run.z = w[u] * run.z + own[u].z; run.w = w[u] * run.w + own[u].w;
    }
  }
}

enum RecPass : int { kRecStep = 1, kRecStates = 2, kRecCarry = 4, kRecOutputs = 8 };

template <typename T, int MODE>
static int rec_launch(const RecParams& p, int what, cudaStream_t s) {
  if ((what & kRecStep) && p.rows.nd > 0) {
    const int nc = p.dv / 4;
    const size_t smem = sizeof(float) * (3 * p.d + p.dv + (kRecStepThreads / nc) * p.dv);
    launch_pdl(rec_step_kernel<T, MODE>, dim3(p.rows.nd, p.H), dim3(kRecStepThreads), smem, s, p);
  }
  if ((what & ~kRecStep) && p.rows.B > 0 && p.nseg > 0) {
    const int rpt = p.d <= 128 ? 16 : 32;
    const int nw = (p.d + rpt - 1) / rpt;
    const int tc = p.d <= 128 ? 16 : 8;
    const size_t smem = sizeof(float) * ((MODE == kWkv ? 3 : 2) * tc * p.d + tc * 64 + tc * nw * 64 + 2 * tc);
    const dim3 grid(p.nseg, p.H, (p.dv + 63) / 64), block(32 * nw);
    if (what & kRecStates) {
      if (rpt == 16) {
        cudaFuncSetAttribute(rec_scan_kernel<T, MODE, 16, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_pdl(rec_scan_kernel<T, MODE, 16, true>, grid, block, smem, s, p, tc);
      } else {
        cudaFuncSetAttribute(rec_scan_kernel<T, MODE, 32, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_pdl(rec_scan_kernel<T, MODE, 32, true>, grid, block, smem, s, p, tc);
      }
    }
    if (what & kRecCarry)
      launch_pdl(rec_carry_kernel<MODE>, dim3(p.rows.B, p.H, (p.d * p.dv / 4 + 255) / 256), dim3(256), 0, s, p);
    if (!(what & kRecOutputs)) return -(int)cudaGetLastError();
    if (rpt == 16) {
      cudaFuncSetAttribute(rec_scan_kernel<T, MODE, 16, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      launch_pdl(rec_scan_kernel<T, MODE, 16, false>, grid, block, smem, s, p, tc);
    } else {
      cudaFuncSetAttribute(rec_scan_kernel<T, MODE, 32, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      launch_pdl(rec_scan_kernel<T, MODE, 32, false>, grid, block, smem, s, p, tc);
    }
  }
  return -(int)cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------
// Token shift: out[s][t] = h[t] + (h[t - 1] - h[t]) * mu[s].  In front of a sequence's first row stands the row its slot remembers
// (zeros at position 0).  Decode rows leave their own row in the slot here; prompt sequences do so in a second launch, after every
// row has read the old one.
// ------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) token_shift_kernel(const T* __restrict__ h, const float* __restrict__ mu, T* __restrict__ shift,
                                                          T* __restrict__ out, int n_mix, int W, int Trows, StepRows rows) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const T* prev = nullptr;
  T* keep = nullptr;
  if (t < rows.nd) {
    const int ctx = rows.ctx_lens[t];
    T* mine = shift + (long long)rows.dec_slots[t] * W;
    if (ctx > 1) prev = mine;
    if (ctx > 0) keep = mine;
  } else {
    const int b = seq_of(rows, t - rows.nd);
    if (t - rows.nd > rows.cu_q[b]) prev = h + (long long)(t - 1) * W;
    else if (rows.cache_lens[b] > 0) prev = shift + (long long)rows.slots[b] * W;
  }
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float x[8], y[8];
    load8(h + (long long)t * W + c, x);
#pragma unroll
    for (int q = 0; q < 8; ++q) y[q] = 0.f;
    if (prev != nullptr) load8(prev + c, y);
    if (keep != nullptr) store8(keep + c, x);
#pragma unroll
    for (int q = 0; q < 8; ++q) y[q] -= x[q];
    for (int s = 0; s < n_mix; ++s) {
      float g[8];
      load8(mu + (long long)s * W + c, g);
#pragma unroll
      for (int q = 0; q < 8; ++q) g[q] = fmaf(y[q], g[q], x[q]);
      store8(out + ((long long)s * Trows + t) * W + c, g);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) shift_store_kernel(const T* __restrict__ h, T* __restrict__ shift, int W, StepRows rows) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x;
  const int end = rows.cu_q[b + 1];
  if (end <= rows.cu_q[b]) return;
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float x[8];
    load8(h + (long long)(rows.nd + end - 1) * W + c, x);
    store8(shift + (long long)rows.slots[b] * W + c, x);
  }
}

}  // namespace lx

extern "C" {

// Description of a step's rows (StepRows, stream.cuh) and of a recurrence (RecParams above), passed by pointer from Python.
int lx_step_rows_bytes() { return (int)sizeof(lx::StepRows); }
int lx_rec_params_bytes() { return (int)sizeof(lx::RecParams); }

// mode 0: linear attention, 1: WKV, 2: SSD.  what: the passes to launch (1 decode rows, 2 the segments' contributions, 4 the carry over the
// segments, 8 outputs and final states); 2 and 4 are needed, with seg_state / seg_decay, when some sequence has more than one segment.
int lx_recurrence(const void* params, int mode, int what, int f32, void* stream) {
  using namespace lx;
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  if (p.d % 16 != 0 || p.dv % 16 != 0 || p.d > 256 || p.dv > 1024 || p.H <= 0) return -1;
  if (p.ldq % 4 != 0 || p.ldk % 4 != 0 || p.ldv % 4 != 0 || (mode == kWkv && p.ldz % 4 != 0)) return -2;
  if ((what & (kRecStates | kRecCarry)) && (p.seg_state == nullptr || (mode != kLinAttn && p.seg_decay == nullptr))) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (mode == kSsd) {
    if (p.hpg <= 0 || p.H % p.hpg != 0) return -4;
    return f32 ? rec_launch<float, kSsd>(p, what, s) : rec_launch<__nv_bfloat16, kSsd>(p, what, s);
  }
  if (f32) return mode == kLinAttn ? rec_launch<float, kLinAttn>(p, what, s) : rec_launch<float, kWkv>(p, what, s);
  return mode == kLinAttn ? rec_launch<__nv_bfloat16, kLinAttn>(p, what, s) : rec_launch<__nv_bfloat16, kWkv>(p, what, s);
}

int lx_token_shift(const void* h, const void* mu, void* shift, void* out, int n_mix, int W, int T, const void* rows_, int f32, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (W % 8 != 0) return -1;
  const StepRows& rows = *reinterpret_cast<const StepRows*>(rows_);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const float* m = reinterpret_cast<const float*>(mu);
  if (f32) {
    float* st = reinterpret_cast<float*>(shift);
    launch_pdl(token_shift_kernel<float>, dim3(T), dim3(256), 0, s, reinterpret_cast<const float*>(h), m, st, reinterpret_cast<float*>(out), n_mix, W, T, rows);
    if (rows.B > 0) launch_pdl(shift_store_kernel<float>, dim3(rows.B), dim3(256), 0, s, reinterpret_cast<const float*>(h), st, W, rows);
  } else {
    __nv_bfloat16* st = reinterpret_cast<__nv_bfloat16*>(shift);
    launch_pdl(token_shift_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, reinterpret_cast<const __nv_bfloat16*>(h), m, st,
               reinterpret_cast<__nv_bfloat16*>(out), n_mix, W, T, rows);
    if (rows.B > 0)
      launch_pdl(shift_store_kernel<__nv_bfloat16>, dim3(rows.B), dim3(256), 0, s, reinterpret_cast<const __nv_bfloat16*>(h), st, W, rows);
  }
  return -(int)cudaGetLastError();
}

}  // extern "C"
