// WKV recurrence over prompt segments on the tensor cores, heads of 64 channels, bf16 activations, fp32 state.
//
// One CTA of eight warps = one segment x one head, walked in blocks of 32 tokens = two chunks of 16.  With w_t the decays of a chunk,
// P_t = prod_{s < t} w_s and Q_j = prod_{s > j} w_s (per key channel, within the chunk):
//   o_t = (r_t P_t) S + sum_{j < t} A_tj v_j + (r_t . u k_t) v_t,    A_tj = sum_c r_tc k_jc prod_{j < s < t} w_sc
//   S   = diag(P_16) S + sum_j (k_j Q_j) v_j^T
// All products of decays are running products of factors <= 1: nothing is divided or exponentiated, so decays of any strength are safe.
// A is formed in fp32 on the CUDA cores (lane = key j x eight channels, walking t); the other products run on the tensor cores with
// their fp32 operands split into two bf16 terms, value and remainder.
// STATES: the segment's own contribution to the state and its total decay only.
#include "stream.cuh"

namespace lx {

struct WkvTcParams {
  const __nv_bfloat16* r; const __nv_bfloat16* k; const __nv_bfloat16* v; const __nv_bfloat16* z;
  long long ldr, ldk, ldv, ldz;
  const float* w0; const float* u;         // [H * 64]
  float* state;                            // [slots, H, 64, 64]
  float* seg_state; float* seg_decay;      // [nseg, H, 64, 64], [nseg, H, 64]
  float* out;                              // [T, H * 64]
  int H;
  StepRows rows;
  const int* seg_seq; const int* seg_q0;
  int seg_len;
};

constexpr int kWkD = 64, kWkB = 32, kWkThreads = 256;
constexpr int kWkF = kWkD + 4;             // fp32 row pitch
constexpr int kWkH = kWkD + 8;             // bf16 row pitch (144 bytes: ldmatrix rows in different banks)
constexpr int kWkA = 24;                   // row pitch of the 16 x 16 weights

LX_DEVICE void wk_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
LX_DEVICE void wk_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LX_DEVICE void wk_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LX_DEVICE void wk_ldsm2_t(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
LX_DEVICE void wk_split1(float a, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(a);
  lo = __float2bfloat16(a - __bfloat162float(hi));
}

// two fp32 numbers in one 64-bit register: one instruction multiplies or accumulates both
LX_DEVICE unsigned long long wk_pair(float a, float b) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
LX_DEVICE float2 wk_unpair(unsigned long long v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
LX_DEVICE unsigned long long wk_mul2(unsigned long long a, unsigned long long b) {
  unsigned long long r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
LX_DEVICE unsigned long long wk_fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
LX_DEVICE void wk_load4(unsigned long long (&x)[4], const float* p) {
  const ulonglong2 a = reinterpret_cast<const ulonglong2*>(p)[0], b = reinterpret_cast<const ulonglong2*>(p)[1];
  x[0] = a.x; x[1] = a.y; x[2] = b.x; x[3] = b.y;
}

struct WkSmem {
  float w[kWkB * kWkF];
  float r[kWkB * kWkF];
  __nv_bfloat16 k[kWkB * kWkH];
  __nv_bfloat16 v[kWkB * kWkH];
  __nv_bfloat16 rp[2][kWkB * kWkH];        // r P, two terms
  __nv_bfloat16 kq[2][kWkB * kWkH];        // k Q
  __nv_bfloat16 s[2][kWkD * kWkH];         // the state in front of the chunk
  __nv_bfloat16 a[2][2][16 * kWkA];        // [chunk][term]: A with the bonus on its diagonal
  float part[2][4][16 * 17];               // [chunk][channel quarter]
  float tot[2][kWkD];                      // P_16 of each chunk
};

template <bool STATES>
__global__ void __launch_bounds__(kWkThreads, 2) wkv_tc_kernel(const WkvTcParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t wk_raw[];
  WkSmem& sm = *reinterpret_cast<WkSmem*>(wk_raw);
  const int seg = blockIdx.x, h = blockIdx.y;
  const int b = p.seg_seq[seg], q0 = p.seg_q0[seg];
  const int r0 = p.rows.cu_q[b], qlen = p.rows.cu_q[b + 1] - r0;
  const int n = min(p.seg_len, qlen - q0);
  const bool last = q0 + p.seg_len >= qlen;
  if (STATES && last) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  // this warp's part of the state: rows (warp & 3) * 16 + lane / 4 (+ 8), columns (warp >> 2) * 32 + nt * 8 + 2 (lane % 4)
  const int srow = (warp & 3) * 16 + (lane >> 2), scol = (warp >> 2) * 32 + (lane & 3) * 2;
  const float* init = nullptr;
  if (!STATES) {
    if (qlen > p.seg_len) init = p.seg_state + ((long long)seg * p.H + h) * kWkD * kWkD;
    else if (p.rows.cache_lens[b] > 0) init = p.state + ((long long)p.rows.slots[b] * p.H + h) * kWkD * kWkD;
  }
  float S[4][4];
#pragma unroll
  for (int nt = 0; nt < 4; ++nt)
#pragma unroll
    for (int hr = 0; hr < 2; ++hr) {
      float2 x = make_float2(0.f, 0.f);
      if (init != nullptr) x = *reinterpret_cast<const float2*>(init + (srow + hr * 8) * kWkD + scol + nt * 8);
      S[nt][2 * hr] = x.x;
      S[nt][2 * hr + 1] = x.y;
    }
  float dprod = 1.f;                       // channel tid of the segment's total decay (tid < 64)
  const int lt = tid >> 3, lc = (tid & 7) * 8;         // loading: token, first of eight channels
  float w0[8];
  load8(p.w0 + h * kWkD + lc, w0);
  // A: lane = key j x eight channels
  const int aj = lane & 15, ac = ((warp & 3) * 2 + (lane >> 4)) * 8, asub = warp >> 2;
  float u[8];
  if (!STATES) load8(p.u + h * kWkD + ac, u);
  const long long tok0 = (long long)p.rows.nd + r0 + q0;

  const uint4 zero4 = make_uint4(0, 0, 0, 0);
  uint4 gr = zero4, gk = zero4, gv = zero4, gz = zero4;
  auto fetch = [&](int t0) {
    const long long t = tok0 + t0 + lt;
    const bool ok = t0 + lt < n;
    const int c = h * kWkD + lc;
    gk = ok ? __ldg(reinterpret_cast<const uint4*>(p.k + t * p.ldk + c)) : zero4;
    gv = ok ? __ldg(reinterpret_cast<const uint4*>(p.v + t * p.ldv + c)) : zero4;
    gz = ok ? __ldg(reinterpret_cast<const uint4*>(p.z + t * p.ldz + c)) : zero4;
    if (!STATES) gr = ok ? __ldg(reinterpret_cast<const uint4*>(p.r + t * p.ldr + c)) : zero4;
  };
  fetch(0);

  for (int t0 = 0; t0 < n; t0 += kWkB) {
    __syncthreads();
    {
      const uint32_t zw[4] = {gz.x, gz.y, gz.z, gz.w}, rw[4] = {gr.x, gr.y, gr.z, gr.w};
      float wv[8], rv[8];
      const bool ok = t0 + lt < n;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 zz = unpack_bf16x2(zw[q]);
        wv[2 * q] = ok ? expf(-expf(zz.x + w0[2 * q])) : 1.f;
        wv[2 * q + 1] = ok ? expf(-expf(zz.y + w0[2 * q + 1])) : 1.f;
        const float2 rr = unpack_bf16x2(rw[q]);
        rv[2 * q] = rr.x;
        rv[2 * q + 1] = rr.y;
      }
      store8(sm.w + lt * kWkF + lc, wv);
      if (!STATES) store8(sm.r + lt * kWkF + lc, rv);
      *reinterpret_cast<uint4*>(sm.k + lt * kWkH + lc) = gk;
      *reinterpret_cast<uint4*>(sm.v + lt * kWkH + lc) = gv;
    }
    if (t0 + kWkB < n) fetch(t0 + kWkB);
    __syncthreads();
    // ---- running products: threads 0..127 forward (channel x chunk), 128..255 backward
    {
      const int c = tid & 63, sub = (tid >> 6) & 1;
      const float* wc = sm.w + sub * 16 * kWkF + c;
      if (tid < 128) {
        float P = 1.f;
#pragma unroll
        for (int t = 0; t < 16; ++t) {
          if (!STATES) {
            const int at = (sub * 16 + t) * kWkH + c;
            wk_split1(sm.r[(sub * 16 + t) * kWkF + c] * P, sm.rp[0][at], sm.rp[1][at]);
          }
          P *= wc[t * kWkF];
        }
        sm.tot[sub][c] = P;
      } else {
        float Q = 1.f;
#pragma unroll
        for (int t = 15; t >= 0; --t) {
          const int at = (sub * 16 + t) * kWkH + c;
          wk_split1(__bfloat162float(sm.k[at]) * Q, sm.kq[0][at], sm.kq[1][at]);
          Q *= wc[t * kWkF];
        }
      }
    }
    // ---- A: every lane carries k_j times the running decay through t = j + 1 .. 15
    if (!STATES) {
      float e[8];
      load8(sm.k + (asub * 16 + aj) * kWkH + ac, e);
      float diag = 0.f;
      {
        float rj[8];
        load8(sm.r + (asub * 16 + aj) * kWkF + ac, rj);
#pragma unroll
        for (int q = 0; q < 8; ++q) diag = fmaf(rj[q] * u[q], e[q], diag);
      }
      unsigned long long e2[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) e2[q] = wk_pair(e[2 * q], e[2 * q + 1]);
      float* dst = sm.part[asub][warp & 3];
      const float* rb = sm.r + asub * 16 * kWkF + ac;
      const float* wb = sm.w + asub * 16 * kWkF + ac;
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        unsigned long long x[4], wv[4];
        wk_load4(x, rb + t * kWkF);
        wk_load4(wv, wb + t * kWkF);
        unsigned long long s0 = wk_mul2(x[0], e2[0]), s1 = wk_mul2(x[1], e2[1]);
        s0 = wk_fma2(x[2], e2[2], s0);
        s1 = wk_fma2(x[3], e2[3], s1);
        if (t > aj) {
#pragma unroll
          for (int q = 0; q < 4; ++q) e2[q] = wk_mul2(e2[q], wv[q]);
        }
        const float2 f0 = wk_unpair(s0), f1 = wk_unpair(s1);
        float a = t > aj ? (f0.x + f0.y) + (f1.x + f1.y) : (t == aj ? diag : 0.f);
        a += __shfl_xor_sync(0xffffffffu, a, 16);
        if (lane < 16) dst[t * 17 + aj] = a;
      }
    }
    __syncthreads();
    if (!STATES) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int e = tid + i * 256, sub = e >> 8, t = (e >> 4) & 15, j = e & 15;
        float a = 0.f;
#pragma unroll
        for (int g = 0; g < 4; ++g) a += sm.part[sub][g][t * 17 + j];
        wk_split1(a, sm.a[sub][0][t * kWkA + j], sm.a[sub][1][t * kWkA + j]);
      }
    }
    if (tid < kWkD) dprod *= sm.tot[0][tid] * sm.tot[1][tid];
#pragma unroll
    for (int sub = 0; sub < 2; ++sub) {
      if (!STATES) {
        if (sub > 0) __syncthreads();                  // the state of the previous chunk has been read
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
          for (int hr = 0; hr < 2; ++hr) {
            const int at = (srow + hr * 8) * kWkH + scol + nt * 8;
            const uint32_t hi = pack_bf16x2(S[nt][2 * hr], S[nt][2 * hr + 1]);
            const float2 back = unpack_bf16x2(hi);
            *reinterpret_cast<uint32_t*>(sm.s[0] + at) = hi;
            *reinterpret_cast<uint32_t*>(sm.s[1] + at) = pack_bf16x2(S[nt][2 * hr] - back.x, S[nt][2 * hr + 1] - back.y);
          }
        __syncthreads();
        // outputs: 16 tokens x this warp's 8 columns
        float o[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        const uint32_t ra = smem_u32(sm.rp[0]) + ((sub * 16 + (lane & 15)) * kWkH + (lane >> 4) * 8) * 2;
        const uint32_t sa = smem_u32(sm.s[0]) + (lane * kWkH + warp * 8) * 2;
        constexpr uint32_t kRpTerm = kWkB * kWkH * 2, kSTerm = kWkD * kWkH * 2;
#pragma unroll
        for (int k2 = 0; k2 < 2; ++k2) {
          uint32_t sh[4], sl[4];
          wk_ldsm_t(sh, sa + k2 * 32 * kWkH * 2);
          wk_ldsm_t(sl, sa + kSTerm + k2 * 32 * kWkH * 2);
#pragma unroll
          for (int kk = 0; kk < 2; ++kk) {
            uint32_t ah[4], al[4];
            wk_ldsm(ah, ra + (k2 * 2 + kk) * 32);
            wk_ldsm(al, ra + kRpTerm + (k2 * 2 + kk) * 32);
            wk_mma(o[0], ah, sh[2 * kk], sh[2 * kk + 1]);
            wk_mma(o[1], al, sh[2 * kk], sh[2 * kk + 1]);
            wk_mma(o[1], ah, sl[2 * kk], sl[2 * kk + 1]);
          }
        }
        uint32_t ah[4], al[4], v0, v1;
        const uint32_t aa = smem_u32(sm.a[sub][0]) + ((lane & 15) * kWkA + (lane >> 4) * 8) * 2;
        wk_ldsm(ah, aa);
        wk_ldsm(al, aa + 16 * kWkA * 2);
        wk_ldsm2_t(v0, v1, smem_u32(sm.v) + ((sub * 16 + (lane & 15)) * kWkH + warp * 8) * 2);
        wk_mma(o[0], ah, v0, v1);
        wk_mma(o[1], al, v0, v1);
        const int tt = t0 + sub * 16 + (lane >> 2);
        float* op = p.out + (tok0 + tt) * (long long)p.H * kWkD + h * kWkD + warp * 8 + (lane & 3) * 2;
        if (tt < n) *reinterpret_cast<float2*>(op) = make_float2(o[0][0] + o[1][0], o[0][1] + o[1][1]);
        if (tt + 8 < n) *reinterpret_cast<float2*>(op + 8ll * p.H * kWkD) = make_float2(o[0][2] + o[1][2], o[0][3] + o[1][3]);
      }
      // state
      const float f0 = sm.tot[sub][srow], f1 = sm.tot[sub][srow + 8];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) { S[nt][0] *= f0; S[nt][1] *= f0; S[nt][2] *= f1; S[nt][3] *= f1; }
      uint32_t kh[4], kl[4];
      const uint32_t ka = smem_u32(sm.kq[0]) + ((sub * 16 + (lane & 7) + (lane >> 4) * 8) * kWkH + (warp & 3) * 16 + ((lane >> 3) & 1) * 8) * 2;
      wk_ldsm_t(kh, ka);
      wk_ldsm_t(kl, ka + kWkB * kWkH * 2);
      const uint32_t va = smem_u32(sm.v) + ((sub * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kWkH + (warp >> 2) * 32 + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        uint32_t vb[4];
        wk_ldsm_t(vb, va + n2 * 32);
        wk_mma(S[2 * n2], kh, vb[0], vb[1]);
        wk_mma(S[2 * n2 + 1], kh, vb[2], vb[3]);
        wk_mma(S[2 * n2], kl, vb[0], vb[1]);
        wk_mma(S[2 * n2 + 1], kl, vb[2], vb[3]);
      }
    }
  }
  float* dst = nullptr;
  if (STATES) dst = p.seg_state + ((long long)seg * p.H + h) * kWkD * kWkD;
  else if (last) dst = p.state + ((long long)p.rows.slots[b] * p.H + h) * kWkD * kWkD;
  if (dst != nullptr) {
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int hr = 0; hr < 2; ++hr)
        *reinterpret_cast<float2*>(dst + (srow + hr * 8) * kWkD + scol + nt * 8) = make_float2(S[nt][2 * hr], S[nt][2 * hr + 1]);
  }
  if (STATES && tid < kWkD) p.seg_decay[((long long)seg * p.H + h) * kWkD + tid] = dprod;
}

}  // namespace lx

extern "C" {

int lx_wkv_tc_bytes() { return (int)sizeof(lx::WkvTcParams); }
int lx_wkv_tc_supported(int d) { return d == lx::kWkD ? 1 : 0; }

// One pass over the segments: states != 0 the segments' contributions and total decays, else outputs and final states (the carry pass
// in between is lx_recurrence's).
int lx_wkv_tc(const void* params, int nseg, int states, void* stream) {
  using namespace lx;
  if (nseg <= 0) return 0;
  const WkvTcParams& p = *reinterpret_cast<const WkvTcParams*>(params);
  if (p.ldr % 8 != 0 || p.ldk % 8 != 0 || p.ldv % 8 != 0 || p.ldz % 8 != 0) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  cudaFuncSetAttribute(wkv_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(WkSmem));
  cudaFuncSetAttribute(wkv_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(WkSmem));
  if (states) launch_pdl(wkv_tc_kernel<true>, dim3(nseg, p.H), dim3(kWkThreads), sizeof(WkSmem), s, p);
  else launch_pdl(wkv_tc_kernel<false>, dim3(nseg, p.H), dim3(kWkThreads), sizeof(WkSmem), s, p);
  return -(int)cudaGetLastError();
}

}  // extern "C"
