// Linear attention over prompt segments in chunks of 64 tokens on the tensor cores (bf16 activations, fp32 state).
//
// One CTA of eight warps = one segment x one head x 64 value columns: four warps form the outputs of a chunk while the other four
// advance the state past it.  Within a chunk of tokens i, j with decay c:
//   o_i  = c^(i+1) q_i S + sum_{j <= i} c^(i-j) (q_i . k_j) v_j        S: the state in front of the chunk
//   S    = c^n S + sum_j c^(n-1-j) k_j v_j^T
// The state lives in fp32 accumulators.  Whatever is fp32 and enters a product (the state, the decayed weights, the decayed keys) is
// split into two bf16 terms, value and remainder, and multiplied as two operands; q, k and v arrive as bf16 with their silu applied
// (silu_cols_kernel: they are read by two passes and two column halves).
// STATES: the segment's own contribution to the state only (each group of four warps takes half of the columns).
//
// SSD (Mamba-2): q, k, v are C, B, x, which hpg heads share for C and B; a token has a step size s = softplus(z + w0) and the decay
// exp(A s).  With the running sum L of A s within a chunk, c^(i+1) becomes exp(L_i), c^(i-j) becomes exp(L_i - L_j) s_j, c^(n-1-j) becomes
// exp(L_(n-1) - L_j) s_j (no exponent is positive), and D x is added to the outputs.
#include "stream.cuh"

namespace lx {

struct LinTcParams {
  const __nv_bfloat16* q; const __nv_bfloat16* k; const __nv_bfloat16* v;
  long long ldq, ldk, ldv;
  const float* decay;
  float* state;            // [slots, H, d, dv]
  float* seg_state;        // [nseg, H, d, dv]
  float* out;              // [T, H * dv]
  int H, dv;
  StepRows rows;
  const int* seg_seq; const int* seg_q0;
  int seg_len, hpg;
  const __nv_bfloat16* z;  // SSD: [T, ldz], head h at column h
  long long ldz;
  const float* w0; const float* A; const float* skip;      // [H]
  float* seg_decay;        // [nseg, H]
};

constexpr int kLtC = 64;                        // tokens per chunk
constexpr int kLtV = 64;                        // value columns per CTA
constexpr int kLtVLd = kLtV + 8;
constexpr int kLtThreads = 256;

LX_DEVICE void lt_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
LX_DEVICE void lt_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LX_DEVICE void lt_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LX_DEVICE void lt_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 back = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - back.x, b - back.y);
}
// rows [0, n) of a [64, COLS] tile -> shared (row pitch COLS + 8), zeros behind
template <int COLS>
LX_DEVICE void lt_fetch(__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int n) {
#pragma unroll
  for (int i = 0; i < COLS / 32; ++i) {
    const int e = threadIdx.x + i * kLtThreads, r = e / (COLS / 8), c = e % (COLS / 8) * 8;
    cp_async_16(dst + r * (COLS + 8) + c, r < n ? src + r * ld + c : src, r < n);
  }
}

// rows [0, n) of a tile of COLS columns on their way to L2, for the chunk after this one
template <int COLS>
LX_DEVICE void lt_prefetch(const __nv_bfloat16* src, long long ld, int n) {
  constexpr int LINES = COLS / 64;
  for (int e = threadIdx.x; e < n * LINES; e += kLtThreads)
    asm volatile("prefetch.global.L2 [%0];" ::"l"(src + (e / LINES) * ld + (e % LINES) * 64));
}

// Barrier over the whole CTA from the two loops of the kernel (outputs, state), which pass it equally often.
LX_DEVICE void lt_sync() { asm volatile("bar.sync 0;" ::: "memory"); }

// silu in place over the columns [0, cols) of a row-strided matrix (the projections of prompt rows, read several times below)
__global__ void __launch_bounds__(256) silu_cols_kernel(__nv_bfloat16* __restrict__ x, long long ld, int cols, long long total) {
  pdl_trigger();
  pdl_wait();
  const int per_row = cols / 8;
  for (long long e = blockIdx.x * (long long)blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
    __nv_bfloat16* at = x + (e / per_row) * ld + (e % per_row) * 8;
    float f[8];
    load8(at, f);
#pragma unroll
    for (int q = 0; q < 8; ++q) f[q] = __fdividef(f[q], 1.f + __expf(-f[q]));
    store8(at, f);
  }
}

template <int D, bool STATES>
struct LtSmem {
  static constexpr int kQ = STATES ? 0 : kLtC * (D + 8) * 2;
  static constexpr int kK = kLtC * (D + 8) * 2;
  static constexpr int kV = kLtC * kLtVLd * 2;
  static constexpr int kS = STATES ? 0 : 2 * D * kLtVLd * 2;
  static constexpr int kTotal = kQ + kK + kV + kS + 2 * (kLtC + 1) * 4 + 16;
};

template <int D, bool STATES, bool SSD>
__global__ void __launch_bounds__(kLtThreads, 2) linear_attn_tc_kernel(const LinTcParams p) {
  pdl_trigger();
  pdl_wait();
  using M = LtSmem<D, STATES>;
  constexpr int LD = D + 8, MT = D / 64;         // 16-row tiles of the state per warp
  extern __shared__ __align__(16) uint8_t lt_sm[];
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(lt_sm);
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(lt_sm + M::kQ);
  __nv_bfloat16* sv = reinterpret_cast<__nv_bfloat16*>(lt_sm + M::kQ + M::kK);
  __nv_bfloat16* ss = reinterpret_cast<__nv_bfloat16*>(lt_sm + M::kQ + M::kK + M::kV);      // [2 terms][D][kLtVLd]
  float* pw = reinterpret_cast<float*>(lt_sm + M::kQ + M::kK + M::kV + M::kS);             // decay^e, e = 0 .. 64; SSD: L of the chunk
  float* sz = pw + kLtC + 1;                                                              // SSD: step sizes (zero behind the last token)
  const int seg = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kLtV;
  const int b = p.seg_seq[seg], q0 = p.seg_q0[seg];
  const int r0 = p.rows.cu_q[b], qlen = p.rows.cu_q[b + 1] - r0;
  const int n = min(p.seg_len, qlen - q0);
  const bool last = q0 + p.seg_len >= qlen;
  if (STATES && last) return;
  const int warp = (threadIdx.x >> 5) & 3, group = threadIdx.x >> 7, lane = threadIdx.x & 31;
  constexpr int NS = STATES ? 4 : 8;             // 8-wide column tiles of a state warp
  const int cs = STATES ? group * 32 : 0;        // its first column
  const int hk = SSD ? h / p.hpg : h;
  if (!SSD) {
    const float lam = p.decay[h];
    for (int e = threadIdx.x; e <= kLtC; e += kLtThreads) pw[e] = powf(lam, (float)e);
  }
  const long long tok0 = (long long)p.rows.nd + r0 + q0;

  // every thread: the chunk's rows on their way, and for SSD its decays
  auto fetch = [&](int t0, int m_tok) {
    lt_sync();
    if (!STATES) lt_fetch<D>(sq, p.q + (tok0 + t0) * p.ldq + hk * D, p.ldq, m_tok);
    lt_fetch<D>(sk, p.k + (tok0 + t0) * p.ldk + hk * D, p.ldk, m_tok);
    lt_fetch<kLtV>(sv, p.v + (tok0 + t0) * p.ldv + h * p.dv + c0, p.ldv, m_tok);
    cp_async_commit();
    if (t0 + kLtC < n) {
      const int ahead = min(kLtC, n - t0 - kLtC);
      const long long tok = tok0 + t0 + kLtC;
      if (!STATES) lt_prefetch<D>(p.q + tok * p.ldq + hk * D, p.ldq, ahead);
      lt_prefetch<D>(p.k + tok * p.ldk + hk * D, p.ldk, ahead);
      lt_prefetch<kLtV>(p.v + tok * p.ldv + h * p.dv + c0, p.ldv, ahead);
    }
    if (SSD && threadIdx.x < 32) {                 // the first warp, two tokens per lane
      float a[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int j = 2 * lane + u;
        const float size = j < m_tok ? softplus_f(__bfloat162float(p.z[(tok0 + t0 + j) * p.ldz + h]) + p.w0[h]) : 0.f;
        sz[j] = size;
        a[u] = p.A[h] * size;
      }
      float sum = a[0] + a[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      pw[2 * lane] = sum - a[1];
      pw[2 * lane + 1] = sum;
    }
  };
  auto ready = [&]() {
    cp_async_wait<0>();
    lt_sync();
  };

  if (!STATES && group == 0) {
    // ---- outputs
    const uint32_t q_a = smem_u32(sq) + ((warp * 16 + (lane & 15)) * LD + (lane >> 4) * 8) * 2;
    const uint32_t k_b = smem_u32(sk) + (((lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t v_b = smem_u32(sv) + (((lane & 7) + ((lane >> 3) & 1) * 8) * kLtVLd + (lane >> 4) * 8) * 2;
    const uint32_t s_b = smem_u32(ss) + (((lane & 7) + ((lane >> 3) & 1) * 8) * kLtVLd + (lane >> 4) * 8) * 2;
    const int i0 = warp * 16 + (lane >> 2), i1 = i0 + 8;
    const float skip = SSD ? p.skip[h] : 0.f;
    for (int t0 = 0; t0 < n; t0 += kLtC) {
      const int m_tok = min(kLtC, n - t0);
      fetch(t0, m_tok);
      ready();
      if (warp * 16 >= m_tok) continue;
      float o[8][4], s[8][4];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
        s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
      }
      // (keys behind the rows of this warp are multiplied too, which keeps the loop free of branches; their weights are zero)
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t a[4];
        lt_ldsm(a, q_a + ks * 32);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t kb[4], sb[4], sl[4];
          lt_ldsm(kb, k_b + n2 * 16 * LD * 2 + ks * 32);
          lt_ldsm_t(sb, s_b + ks * 16 * kLtVLd * 2 + n2 * 32);
          lt_ldsm_t(sl, s_b + (D + ks * 16) * kLtVLd * 2 + n2 * 32);
          lt_mma(s[2 * n2], a, kb[0], kb[1]);
          lt_mma(s[2 * n2 + 1], a, kb[2], kb[3]);
          lt_mma(o[2 * n2], a, sb[0], sb[1]);
          lt_mma(o[2 * n2 + 1], a, sb[2], sb[3]);
          lt_mma(o[2 * n2], a, sl[0], sl[1]);
          lt_mma(o[2 * n2 + 1], a, sl[2], sl[3]);
        }
      }
      const float f0 = SSD ? __expf(pw[i0]) : pw[i0 + 1], f1 = SSD ? __expf(pw[i1]) : pw[i1 + 1];
      // weight of key j for the query row i, j <= i
      auto weight = [&](int i, int j) { return SSD ? __expf(pw[i] - pw[j]) * sz[j] : pw[i - j]; };
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) { o[nt][0] *= f0; o[nt][1] *= f0; o[nt][2] *= f1; o[nt][3] *= f1; }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk > warp) continue;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int j = kk * 16 + u * 8 + (lane & 3) * 2;
          const float* x = s[2 * kk + u];
          lt_split(j <= i0 ? x[0] * weight(i0, j) : 0.f, j + 1 <= i0 ? x[1] * weight(i0, j + 1) : 0.f, ph[2 * u], pl[2 * u]);
          lt_split(j <= i1 ? x[2] * weight(i1, j) : 0.f, j + 1 <= i1 ? x[3] * weight(i1, j + 1) : 0.f, ph[2 * u + 1], pl[2 * u + 1]);
        }
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t vb[4];
          lt_ldsm_t(vb, v_b + kk * 16 * kLtVLd * 2 + n2 * 32);
          lt_mma(o[2 * n2], ph, vb[0], vb[1]);
          lt_mma(o[2 * n2 + 1], ph, vb[2], vb[3]);
          lt_mma(o[2 * n2], pl, vb[0], vb[1]);
          lt_mma(o[2 * n2 + 1], pl, vb[2], vb[3]);
        }
      }
      if constexpr (SSD) {
        const __nv_bfloat16* x0 = sv + i0 * kLtVLd + (lane & 3) * 2;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          const float2 a = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(x0 + nt * 8));
          const float2 b = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(x0 + 8 * kLtVLd + nt * 8));
          o[nt][0] = fmaf(skip, a.x, o[nt][0]); o[nt][1] = fmaf(skip, a.y, o[nt][1]);
          o[nt][2] = fmaf(skip, b.x, o[nt][2]); o[nt][3] = fmaf(skip, b.y, o[nt][3]);
        }
      }
      const long long ldo = (long long)p.H * p.dv;
      float* orow = p.out + (tok0 + t0 + i0) * ldo + (long long)h * p.dv + c0 + (lane & 3) * 2;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        if (i0 < m_tok) *reinterpret_cast<float2*>(orow + nt * 8) = make_float2(o[nt][0], o[nt][1]);
        if (i1 < m_tok) *reinterpret_cast<float2*>(orow + 8 * ldo + nt * 8) = make_float2(o[nt][2], o[nt][3]);
      }
    }
    return;
  }

  // ---- state: rows warp * D / 4 + m * 16 + lane / 4 (+ 8), columns c0 + cs + nt * 8 + 2 (lane % 4)
  float S[MT][NS][4];
  const float* init = nullptr;
  if (!STATES) {
    if (qlen > p.seg_len) init = p.seg_state + ((long long)seg * p.H + h) * D * p.dv;
    else if (p.rows.cache_lens[b] > 0) init = p.state + ((long long)p.rows.slots[b] * p.H + h) * D * p.dv;
  }
  const long long s_at = (long long)(warp * (D / 4) + (lane >> 2)) * p.dv + c0 + cs + (lane & 3) * 2;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nt = 0; nt < NS; ++nt)
#pragma unroll
      for (int hr = 0; hr < 2; ++hr) {
        float2 v = make_float2(0.f, 0.f);
        if (init != nullptr) v = *reinterpret_cast<const float2*>(init + s_at + (long long)(m * 16 + hr * 8) * p.dv + nt * 8);
        S[m][nt][2 * hr] = v.x;
        S[m][nt][2 * hr + 1] = v.y;
      }
  const uint32_t kt_a = smem_u32(sk) + (((lane & 7) + (lane >> 4) * 8) * LD + warp * (D / 4) + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t v_b = smem_u32(sv) + (((lane & 7) + ((lane >> 3) & 1) * 8) * kLtVLd + (lane >> 4) * 8) * 2;
  float total = 0.f;                             // SSD: sum of L over the chunks so far
  for (int t0 = 0; t0 < n; t0 += kLtC) {
    const int m_tok = min(kLtC, n - t0);
    fetch(t0, m_tok);
    if (!STATES) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int nt = 0; nt < NS; ++nt)
#pragma unroll
          for (int hr = 0; hr < 2; ++hr) {
            uint32_t hi, lo;
            lt_split(S[m][nt][2 * hr], S[m][nt][2 * hr + 1], hi, lo);
            __nv_bfloat16* d = ss + (warp * (D / 4) + m * 16 + (lane >> 2) + hr * 8) * kLtVLd + nt * 8 + (lane & 3) * 2;
            *reinterpret_cast<uint32_t*>(d) = hi;
            *reinterpret_cast<uint32_t*>(d + D * kLtVLd) = lo;
          }
    }
    ready();
    const float fs = SSD ? __expf(pw[kLtC - 1]) : pw[m_tok];
    if (SSD) total += pw[kLtC - 1];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NS; ++nt) { S[m][nt][0] *= fs; S[m][nt][1] *= fs; S[m][nt][2] *= fs; S[m][nt][3] *= fs; }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t kh[MT][4], kl[MT][4];
      const int j = kk * 16 + (lane & 3) * 2;
      // (rows behind the chunk's last token are zero: their factor only has to exist)
      auto factor = [&](int t) { return SSD ? __expf(pw[kLtC - 1] - pw[t]) * sz[t] : pw[max(m_tok - 1 - t, 0)]; };
      const float g0 = factor(j), g1 = factor(j + 1), g8 = factor(j + 8), g9 = factor(j + 9);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        uint32_t a[4];
        lt_ldsm_t(a, kt_a + kk * 16 * LD * 2 + m * 32);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 x = unpack_bf16x2(a[e]);
          lt_split(x.x * (e < 2 ? g0 : g8), x.y * (e < 2 ? g1 : g9), kh[m][e], kl[m][e]);
        }
      }
#pragma unroll
      for (int n2 = 0; n2 < NS / 2; ++n2) {
        uint32_t vb[4];
        lt_ldsm_t(vb, v_b + kk * 16 * kLtVLd * 2 + (cs + n2 * 16) * 2);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          lt_mma(S[m][2 * n2], kh[m], vb[0], vb[1]);
          lt_mma(S[m][2 * n2 + 1], kh[m], vb[2], vb[3]);
          lt_mma(S[m][2 * n2], kl[m], vb[0], vb[1]);
          lt_mma(S[m][2 * n2 + 1], kl[m], vb[2], vb[3]);
        }
      }
    }
  }
  if (SSD && STATES && blockIdx.z == 0 && threadIdx.x == 0) p.seg_decay[(long long)seg * p.H + h] = expf(total);
  float* dst = nullptr;
  if (STATES) dst = p.seg_state + ((long long)seg * p.H + h) * D * p.dv;
  else if (last) dst = p.state + ((long long)p.rows.slots[b] * p.H + h) * D * p.dv;
  if (dst != nullptr) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NS; ++nt)
#pragma unroll
        for (int hr = 0; hr < 2; ++hr)
          *reinterpret_cast<float2*>(dst + s_at + (long long)(m * 16 + hr * 8) * p.dv + nt * 8) = make_float2(S[m][nt][2 * hr], S[m][nt][2 * hr + 1]);
  }
}

template <int D, bool STATES, bool SSD>
static int lt_launch(const LinTcParams& p, int nseg, cudaStream_t s) {
  cudaFuncSetAttribute(linear_attn_tc_kernel<D, STATES, SSD>, cudaFuncAttributeMaxDynamicSharedMemorySize, LtSmem<D, STATES>::kTotal);
  launch_pdl(linear_attn_tc_kernel<D, STATES, SSD>, dim3(nseg, p.H, p.dv / kLtV), dim3(kLtThreads), (size_t)LtSmem<D, STATES>::kTotal, s, p);
  return -(int)cudaGetLastError();
}

}  // namespace lx

extern "C" {

int lx_linear_attn_tc_bytes() { return (int)sizeof(lx::LinTcParams); }
int lx_linear_attn_tc_supported(int d, int dv) { return ((d == 64 || d == 128) && dv % 64 == 0) ? 1 : 0; }

// silu in place over columns [0, cols) of T rows.
int lx_silu_cols(void* x, long long ld, int T, int cols, void* stream) {
  using namespace lx;
  if (T <= 0 || cols <= 0) return 0;
  if (cols % 8 != 0 || ld % 8 != 0) return -1;
  const long long total = (long long)T * (cols / 8);
  const int grid = (int)((total + 255) / 256 < 148 * 8 ? (total + 255) / 256 : 148 * 8);
  launch_pdl(silu_cols_kernel, dim3(grid), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<__nv_bfloat16*>(x), ld, cols, total);
  return -(int)cudaGetLastError();
}

// q, k, v with their silu applied (ssd: the inputs of the state space recurrence, and z, w0, A, skip, hpg).  One pass over the segments:
// states != 0 the segments' contributions, else outputs and final states (the carry pass in between is lx_recurrence's).
int lx_linear_attn_tc(const void* params, int d, int nseg, int states, int ssd, void* stream) {
  using namespace lx;
  if (nseg <= 0) return 0;
  const LinTcParams& p = *reinterpret_cast<const LinTcParams*>(params);
  if (!lx_linear_attn_tc_supported(d, p.dv) || p.ldq % 8 != 0 || p.ldk % 8 != 0 || p.ldv % 8 != 0) return -1;
  if (ssd && (p.hpg <= 0 || p.H % p.hpg != 0 || (states && p.seg_decay == nullptr))) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (ssd) {
    if (states) return d == 64 ? lt_launch<64, true, true>(p, nseg, s) : lt_launch<128, true, true>(p, nseg, s);
    return d == 64 ? lt_launch<64, false, true>(p, nseg, s) : lt_launch<128, false, true>(p, nseg, s);
  }
  if (states) return d == 64 ? lt_launch<64, true, false>(p, nseg, s) : lt_launch<128, true, false>(p, nseg, s);
  return d == 64 ? lt_launch<64, false, false>(p, nseg, s) : lt_launch<128, false, false>(p, nseg, s);
}

}  // extern "C"
