// Kernels of attention over the paged KV cache; attention.cu and gqa.cu describe and instantiate them.
#pragma once

#include <cuda_fp8.h>

#include "attn_tail.cuh"

namespace lx {

constexpr int kPage = 32;
constexpr float kLog2e = 1.4426950408889634f;

LX_DEVICE void mma_bf16_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
LX_DEVICE void ldsm_x4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
LX_DEVICE void ldsm_x4_t(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}

// A [ROWS, D] bf16 plane in shared memory; 16-byte chunk c of row r lives at chunk (c ^ (r & 7)) so that
// ldmatrix (8 rows, same logical chunk) touches 8 different bank groups.
template <int D>
LX_DEVICE uint32_t swz(int r, int c) { return (uint32_t)((r * (D / 8) + (c ^ (r & 7))) * 16); }

// Copy ROWS x D bf16 (contiguous in global memory) into a swizzled plane with `NT` cooperating threads.
template <int D, int ROWS, int NT>
LX_DEVICE void load_plane(uint32_t smem_base, const __nv_bfloat16* g, int tid, bool valid) {
  constexpr int CPR = D / 8;
  constexpr int CHUNKS = ROWS * CPR;
#pragma unroll
  for (int c = tid; c < CHUNKS; c += NT) {
    const int r = c / CPR, cc = c % CPR;
    const uint32_t dst = smem_base + swz<D>(r, cc);
    const int sz = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(g + (long long)c * 8), "r"(sz) : "memory");
  }
}

// Copy ROWS x D e4m3 bytes (contiguous in global memory) into a linear staging area.
template <int D, int ROWS, int NT>
LX_DEVICE void load_plane8(uint32_t smem_base, const uint8_t* g, int tid, bool valid) {
  constexpr int CHUNKS = ROWS * D / 16;
#pragma unroll
  for (int c = tid; c < CHUNKS; c += NT) {
    const int sz = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_base + c * 16), "l"(g + (long long)c * 16), "r"(sz) : "memory");
  }
}
LX_DEVICE uint32_t e4m3x2_to_bf16x2(uint32_t two) {
  const __half2_raw h = __nv_cvt_fp8x2_to_halfraw2((__nv_fp8x2_storage_t)(two & 0xffffu), __NV_E4M3);
  const float2 f = __half22float2(*reinterpret_cast<const __half2*>(&h));
  return pack_bf16x2(f.x, f.y);
}
// Expand a staged e4m3 plane into a swizzled bf16 plane (every e4m3 value is exact in bf16).
template <int D, int ROWS, int NT>
LX_DEVICE void expand_plane8(uint32_t dst_plane, uint32_t src8, int tid) {
  constexpr int CHUNKS = ROWS * D / 16;
#pragma unroll
  for (int c = tid; c < CHUNKS; c += NT) {
    uint32_t w0, w1, w2, w3;
    asm volatile("ld.shared.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(w0), "=r"(w1), "=r"(w2), "=r"(w3) : "r"(src8 + c * 16));
    const int r = (c * 16) / D, cc = ((c * 16) % D) / 8;
    asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};" ::"r"(dst_plane + swz<D>(r, cc)), "r"(e4m3x2_to_bf16x2(w0)),
                 "r"(e4m3x2_to_bf16x2(w0 >> 16)), "r"(e4m3x2_to_bf16x2(w1)), "r"(e4m3x2_to_bf16x2(w1 >> 16)) : "memory");
    asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};" ::"r"(dst_plane + swz<D>(r, cc + 1)), "r"(e4m3x2_to_bf16x2(w2)),
                 "r"(e4m3x2_to_bf16x2(w2 >> 16)), "r"(e4m3x2_to_bf16x2(w3)), "r"(e4m3x2_to_bf16x2(w3 >> 16)) : "memory");
  }
}

// S[16, NKEYS] (+)= Q[16, D] K[NKEYS, D]^T for one warp.  qf holds the A fragments of Q.
template <int D, int NKEYS>
LX_DEVICE void qk_tile(float (&sacc)[NKEYS / 8][4], const uint32_t (&qf)[D / 16][4], uint32_t k_smem, int lane) {
#pragma unroll
  for (int nt = 0; nt < NKEYS / 8; ++nt) {
#pragma unroll
    for (int q = 0; q < 4; ++q) sacc[nt][q] = 0.f;
#pragma unroll
    for (int ks = 0; ks < D / 16; ks += 2) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4(b0, b1, b2, b3, k_smem + swz<D>(nt * 8 + (lane & 7), 2 * ks + (lane >> 3)));
      mma_bf16_16816(sacc[nt], qf[ks], b0, b1);
      mma_bf16_16816(sacc[nt], qf[ks + 1], b2, b3);
    }
  }
}

// O[16, D] += P[16, NKEYS] V[NKEYS, D].  WIDE: the fp32 weights P enter as two bf16 terms, value and remainder.
template <int D, int NKEYS, bool WIDE = false>
LX_DEVICE void pv_tile(float (&oacc)[D / 8][4], const float (&sacc)[NKEYS / 8][4], uint32_t v_smem, int lane) {
#pragma unroll
  for (int kk = 0; kk < NKEYS / 16; ++kk) {
    uint32_t pa[4];
    pa[0] = pack_bf16x2(sacc[2 * kk][0], sacc[2 * kk][1]);
    pa[1] = pack_bf16x2(sacc[2 * kk][2], sacc[2 * kk][3]);
    pa[2] = pack_bf16x2(sacc[2 * kk + 1][0], sacc[2 * kk + 1][1]);
    pa[3] = pack_bf16x2(sacc[2 * kk + 1][2], sacc[2 * kk + 1][3]);
    uint32_t pl[4];
    if constexpr (WIDE) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 hi = unpack_bf16x2(pa[q]);
        pl[q] = pack_bf16x2(sacc[2 * kk + (q >> 1)][2 * (q & 1)] - hi.x, sacc[2 * kk + (q >> 1)][2 * (q & 1) + 1] - hi.y);
      }
    }
#pragma unroll
    for (int nd = 0; nd < D / 8; nd += 2) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4_t(b0, b1, b2, b3, v_smem + swz<D>(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, nd + (lane >> 4)));
      mma_bf16_16816(oacc[nd], pa, b0, b1);
      mma_bf16_16816(oacc[nd + 1], pa, b2, b3);
      if constexpr (WIDE) {
        mma_bf16_16816(oacc[nd], pl, b0, b1);
        mma_bf16_16816(oacc[nd + 1], pl, b2, b3);
      }
    }
  }
}

// Online-softmax update for the two rows (lane/4 and lane/4 + 8) a thread owns.  `sacc` holds raw dot
// products on entry and probabilities on exit.  key0 = index of column 0; keys outside [lo, hi) are masked.
template <int D, int NKEYS>
LX_DEVICE void softmax_tile(float (&sacc)[NKEYS / 8][4], float (&oacc)[D / 8][4], float (&m)[2], float (&l)[2], int key0,
                            int lo0, int hi0, int lo1, int hi1, float scale, float softcap, int lane, float slope0 = 0.f,
                            float slope1 = 0.f) {
  float mx[2] = {-INFINITY, -INFINITY};
  const float cap_k = softcap > 0.f ? 2.f * kLog2e / softcap : 0.f;
#pragma unroll
  for (int nt = 0; nt < NKEYS / 8; ++nt) {
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int key = key0 + nt * 8 + 2 * (lane & 3) + (q & 1);
      const int r = q >> 1;
      float s = sacc[nt][q] * scale;
      if (softcap > 0.f) s = softcap_score(s, softcap, cap_k);
      // ALiBi: the bias -slope * (query position - key position) differs from slope * key position by a per-row constant,
      // which the softmax does not see
      s += (r == 0 ? slope0 : slope1) * (float)key;
      const bool ok = r == 0 ? (key >= lo0 && key < hi0) : (key >= lo1 && key < hi1);
      s = ok ? s : -INFINITY;
      sacc[nt][q] = s;
      mx[r] = fmaxf(mx[r], s);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
    mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
  }
  float corr[2], mnew[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    mnew[r] = fmaxf(m[r], mx[r]);
    corr[r] = (mnew[r] == -INFINITY) ? 1.f : exp2f((m[r] - mnew[r]) * kLog2e);
    m[r] = mnew[r];
    l[r] *= corr[r];
  }
#pragma unroll
  for (int nt = 0; nt < NKEYS / 8; ++nt) {
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int r = q >> 1;
      const float pz = (mnew[r] == -INFINITY) ? 0.f : exp2f((sacc[nt][q] - mnew[r]) * kLog2e);
      sacc[nt][q] = pz;
      l[r] += pz;
    }
  }
#pragma unroll
  for (int nd = 0; nd < D / 8; ++nd) {
    oacc[nd][0] *= corr[0]; oacc[nd][1] *= corr[0];
    oacc[nd][2] *= corr[1]; oacc[nd][3] *= corr[1];
  }
}

// ------------------------------------------------------------------------------------------------
// Decode
// ------------------------------------------------------------------------------------------------
struct DecodeParams {
  const __nv_bfloat16* q;     // [T, ldq], head h at column h * DK
  long long ldq;
  const __nv_bfloat16* kv;    // cache of this layer
  const int* block_tables;    // [T, max_blocks]
  int max_blocks;
  const int* ctx_lens;        // [T] number of keys visible to the token (includes itself); <= 0: skip row
  __nv_bfloat16* out;         // [T, ldo]
  long long ldo;
  float* part_o;              // split-KV partials [T, nh, nsplit, DV]
  float* part_lse;            // [T, nh, nsplit]
  int nh, nkv, group, gchunks;
  int window;                 // <= 0: none
  float scale, softcap;
  int nsplit;
  const float* alibi;         // [nh] ALiBi slopes, or null
  float v_scale;              // fp8 cache: multiplies the output (the K scale is folded into `scale` by the host)
  AttnTail tail;
};

// NW warps per CTA split the pages of a (row, KV head): four for long contexts; two, so that two CTAs fit an SM and one streams
// while the other starts or combines, for the short contexts of a large decode batch.
// DK, DV: widths of keys and values (a page of one head holds its key plane, then its value plane).
template <int DK, int DV, int STAGES, bool KV8, int NW, bool WIDE = false>
__global__ void __launch_bounds__(32 * NW) attn_decode_kernel(const DecodeParams p) {
  pdl_trigger();
  pdl_wait();      // every block waits, also those that return early below
  extern __shared__ __align__(1024) uint8_t dsm[];
  static_assert(!KV8 || DK == DV, "e4m3 pages hold keys and values of one width");
  constexpr int PLANE = kPage * DK * 2, VPLANE = kPage * DV * 2;
  constexpr int PLANE8 = kPage * DK;
  constexpr int STAGE = KV8 ? 2 * PLANE8 : PLANE + VPLANE;
  constexpr int WARP_BYTES = STAGES * STAGE + (KV8 ? 2 * PLANE : 0);     // fp8: staged bytes + one expanded K and V plane
  const int t = blockIdx.x;
  const int kvh = blockIdx.y / p.gchunks, gc = blockIdx.y % p.gchunks;
  const int split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ctx = p.ctx_lens[t];
  const int g0 = gc * 16;
  const int grows = min(16, p.group - g0);
  const int head0 = kvh * p.group + g0;

  int key_lo = 0;
  if (p.window > 0 && ctx > p.window) key_lo = ctx - p.window;
  const int page_lo = key_lo / kPage;
  const int page_hi = ctx > 0 ? (ctx + kPage - 1) / kPage : 0;
  const int npages = max(page_hi - page_lo, 0);
  const int per_split = (npages + p.nsplit - 1) / p.nsplit;
  const int pb = page_lo + split * per_split;
  const int pe = min(pb + per_split, page_hi);

  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float oacc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) { oacc[i][0] = oacc[i][1] = oacc[i][2] = oacc[i][3] = 0.f; }

  // Q fragments straight from global memory (row = head in group, zero beyond the group).
  uint32_t qf[DK / 16][4];
  {
    const int r0 = lane >> 2, r1 = r0 + 8;
    const __nv_bfloat16* q0 = p.q + (long long)t * p.ldq + (long long)(head0 + r0) * DK;
    const __nv_bfloat16* q1 = p.q + (long long)t * p.ldq + (long long)(head0 + r1) * DK;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      const int c = ks * 16 + 2 * (lane & 3);
      qf[ks][0] = r0 < grows ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
      qf[ks][1] = r1 < grows ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
      qf[ks][2] = r0 < grows ? *reinterpret_cast<const uint32_t*>(q0 + c + 8) : 0u;
      qf[ks][3] = r1 < grows ? *reinterpret_cast<const uint32_t*>(q1 + c + 8) : 0u;
    }
  }

  const uint32_t wbase = smem_u32(dsm) + warp * WARP_BYTES;
  const uint32_t wwork = wbase + STAGES * STAGE;
  const int* bt = p.block_tables + (long long)t * p.max_blocks;
  float slope0 = 0.f, slope1 = 0.f;
  if (p.alibi != nullptr) {
    const int r0 = lane >> 2, r1 = r0 + 8;
    slope0 = r0 < grows ? p.alibi[head0 + r0] : 0.f;
    slope1 = r1 < grows ? p.alibi[head0 + r1] : 0.f;
  }
  const int my_first = pb + warp;
  const int my_count = my_first < pe ? (pe - my_first + NW - 1) / NW : 0;

  auto issue = [&](int i) {
    if (i < my_count) {
      const int page = my_first + NW * i;
      const long long blk = bt[page];
      const uint32_t sb = wbase + (i % STAGES) * STAGE;
      if constexpr (KV8) {
        const uint8_t* src = reinterpret_cast<const uint8_t*>(p.kv) + ((blk * p.nkv + kvh) * 2) * (long long)(kPage * DK);
        load_plane8<DK, 2 * kPage, 32>(sb, src, lane, true);            // the K plane and the V plane are one contiguous run
      } else {
        const __nv_bfloat16* src = p.kv + (blk * p.nkv + kvh) * (long long)(kPage * (DK + DV));
        load_plane<DK, kPage, 32>(sb, src, lane, true);
        load_plane<DV, kPage, 32>(sb + PLANE, src + kPage * DK, lane, true);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) issue(s);

  for (int i = 0; i < my_count; ++i) {
    issue(i + STAGES - 1);
    cp_async_wait<STAGES - 1>();
    __syncwarp();
    uint32_t sb = wbase + (i % STAGES) * STAGE;
    if constexpr (KV8) {
      expand_plane8<DK, kPage, 32>(wwork, sb, lane);
      expand_plane8<DK, kPage, 32>(wwork + PLANE, sb + PLANE8, lane);
      __syncwarp();
      sb = wwork;
    }
    const int page = my_first + NW * i;
    float sacc[kPage / 8][4];
    qk_tile<DK, kPage>(sacc, qf, sb, lane);
    softmax_tile<DV, kPage>(sacc, oacc, m, l, page * kPage, key_lo, ctx, key_lo, ctx, p.scale, p.softcap, lane, slope0, slope1);
    pv_tile<DV, kPage, WIDE>(oacc, sacc, sb + PLANE, lane);
    __syncwarp();
  }
  cp_async_wait<0>();
  __syncthreads();

  // ---- combine the four warps through shared memory (pipeline buffers are free now)
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  float* so = reinterpret_cast<float*>(dsm);            // [NW][16][DV]
  float* sm = so + NW * 16 * DV;                          // [NW][16]
  float* sl = sm + NW * 16;                              // [NW][16]
  {
    const int r0 = lane >> 2, r1 = r0 + 8;
#pragma unroll
    for (int nd = 0; nd < DV / 8; ++nd) {
      const int c = nd * 8 + 2 * (lane & 3);
      *reinterpret_cast<float2*>(so + (warp * 16 + r0) * DV + c) = make_float2(oacc[nd][0], oacc[nd][1]);
      *reinterpret_cast<float2*>(so + (warp * 16 + r1) * DV + c) = make_float2(oacc[nd][2], oacc[nd][3]);
    }
    if ((lane & 3) == 0) {
      sm[warp * 16 + r0] = m[0]; sm[warp * 16 + r1] = m[1];
      sl[warp * 16 + r0] = l[0]; sl[warp * 16 + r1] = l[1];
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x * 2; idx < grows * DV; idx += 64 * NW) {
    const int g = idx / DV, d = idx % DV;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < NW; ++w) M = fmaxf(M, sm[w * 16 + g]);
    float2 num = make_float2(0.f, 0.f);
    float den = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) {
      const float mw = sm[w * 16 + g];
      const float wgt = (mw == -INFINITY) ? 0.f : exp2f((mw - M) * kLog2e);
      const float2 v = *reinterpret_cast<const float2*>(so + (w * 16 + g) * DV + d);
      num.x += wgt * v.x;
      num.y += wgt * v.y;
      den += wgt * sl[w * 16 + g];
    }
    const int head = head0 + g;
    if (p.nsplit == 1) {                         // (of several splits the tail joins where they are combined)
      const float f = (den > 0.f ? attn_denominator(p.tail, head, M * kLog2e, den) : 0.f) * (KV8 ? p.v_scale : 1.f);
      const float2 o = attn_turn_back(p.tail, make_float2(num.x * f, num.y * f), d, ctx - 1);
      const int col = head * DV + d;
      __nv_bfloat16* dst = p.out + (long long)t * p.ldo + col;
      dst[0] = __float2bfloat16(attn_tail(p.tail, o.x, t, col));
      dst[1] = __float2bfloat16(attn_tail(p.tail, o.y, t, col + 1));
    } else {
      const float f = (den > 0.f ? 1.f / den : 0.f) * (KV8 ? p.v_scale : 1.f);
      const long long pi = ((long long)t * p.nh + head) * p.nsplit + split;
      *reinterpret_cast<float2*>(p.part_o + pi * DV + d) = make_float2(num.x * f, num.y * f);
      if (d == 0) p.part_lse[pi] = den > 0.f ? M + __logf(den) : -INFINITY;
    }
  }
}

template <int D>
__global__ void __launch_bounds__(D) attn_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse,
                                                         __nv_bfloat16* __restrict__ out, long long ldo, int nh, int nsplit,
                                                         const AttnTail tail, const int* __restrict__ ctx_lens) {
  pdl_trigger();
  pdl_wait();      // every block waits, also those that return early below
  const int t = blockIdx.x, h = blockIdx.y, d = threadIdx.x;
  const long long base = ((long long)t * nh + h) * nsplit;
  float M = -INFINITY;
  for (int s = 0; s < nsplit; ++s) M = fmaxf(M, part_lse[base + s]);
  const bool any = M > -INFINITY;
  if (tail.sink != nullptr) M = fmaxf(M, tail.sink[h]);
  float num = 0.f, den = tail.sink != nullptr ? __expf(tail.sink[h] - M) : 0.f;
  for (int s = 0; s < nsplit; ++s) {
    const float ls = part_lse[base + s];
    const float w = (ls == -INFINITY) ? 0.f : __expf(ls - M);
    num += w * part_o[(base + s) * D + d];
    den += w;
  }
  float o = any ? num / den : 0.f;
  if (tail.turn != nullptr && any) {             // (the whole block takes this branch or none of it)
    const float other = __shfl_xor_sync(0xffffffffu, o, 1);
    const float2 both = attn_turn_back(tail, d & 1 ? make_float2(other, o) : make_float2(o, other), d & ~1, ctx_lens[t] - 1);
    o = d & 1 ? both.y : both.x;
  }
  out[(long long)t * ldo + (long long)h * D + d] = __float2bfloat16(any ? attn_tail(tail, o, t, h * D + d) : 0.f);
}

// ------------------------------------------------------------------------------------------------
// Prefill: 64 queries x 1 head per CTA (16 query rows per warp), 64-key tiles = two cache pages.
// ------------------------------------------------------------------------------------------------
struct PrefillParams {
  const __nv_bfloat16* q;     // [T, ldq]
  long long ldq;
  const __nv_bfloat16* kv;
  const int* block_tables;    // [B, max_blocks]
  int max_blocks;
  const int* cu_q;            // [B + 1] start of each sequence's chunk in the ragged token dimension
  const int* cache_lens;      // [B] keys already cached before this chunk
  const int* tile_seq;        // [num_tiles] sequence of each 64-query tile
  const int* tile_q0;         // [num_tiles] first query (within the chunk) of the tile
  __nv_bfloat16* out;
  long long ldo;
  int nh, nkv;
  int window;
  float scale, softcap;
  const float* alibi;         // [nh] ALiBi slopes, or null
  float v_scale;              // fp8 cache: multiplies the output
  AttnTail tail;
};

template <int DK, int DV, bool KV8, bool WIDE = false>
__global__ void __launch_bounds__(128) attn_prefill_kernel(const PrefillParams p) {
  pdl_trigger();
  pdl_wait();      // every block waits, also those that return early below
  extern __shared__ __align__(1024) uint8_t psm[];
  constexpr int KT = 64;                         // keys per tile
  static_assert(!KV8 || DK == DV, "e4m3 pages hold keys and values of one width");
  constexpr int PLANE = kPage * DK * 2, VPLANE = kPage * DV * 2;           // one page of K, of V
  constexpr int PLANE8 = kPage * DK;
  constexpr int STAGE = KV8 ? 4 * PLANE8 : 2 * (PLANE + VPLANE);        // K page0, K page1, V page0, V page1 (fp8: K0 V0 K1 V1 as bytes)
  const int tile = blockIdx.x, head = blockIdx.y;
  const int kvh = head / (p.nh / p.nkv);
  const int b = p.tile_seq[tile];
  const int q0 = p.tile_q0[tile];
  const int qlen = p.cu_q[b + 1] - p.cu_q[b];
  const int cache = p.cache_lens[b];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* bt = p.block_tables + (long long)b * p.max_blocks;

  // rows owned by this thread
  const int qr0 = q0 + warp * 16 + (lane >> 2), qr1 = qr0 + 8;
  const long long tok0 = (long long)p.cu_q[b] + qr0, tok1 = (long long)p.cu_q[b] + qr1;
  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks) {
    const int c = ks * 16 + 2 * (lane & 3);
    const __nv_bfloat16* a0 = p.q + tok0 * p.ldq + (long long)head * DK + c;
    const __nv_bfloat16* a1 = p.q + tok1 * p.ldq + (long long)head * DK + c;
    qf[ks][0] = qr0 < qlen ? *reinterpret_cast<const uint32_t*>(a0) : 0u;
    qf[ks][1] = qr1 < qlen ? *reinterpret_cast<const uint32_t*>(a1) : 0u;
    qf[ks][2] = qr0 < qlen ? *reinterpret_cast<const uint32_t*>(a0 + 8) : 0u;
    qf[ks][3] = qr1 < qlen ? *reinterpret_cast<const uint32_t*>(a1 + 8) : 0u;
  }
  // visible key range per row: [lo, hi) with hi = position + 1
  const int pos0 = cache + qr0, pos1 = cache + qr1;
  const int hi0 = qr0 < qlen ? pos0 + 1 : 0, hi1 = qr1 < qlen ? pos1 + 1 : 0;
  const int lo0 = (p.window > 0 && hi0 > p.window) ? hi0 - p.window : 0;
  const int lo1 = (p.window > 0 && hi1 > p.window) ? hi1 - p.window : 0;

  // key tiles needed by the CTA
  const int last_q = min(q0 + 63, qlen - 1);
  const int key_hi = cache + last_q + 1;
  int key_lo = 0;
  if (p.window > 0) key_lo = max(cache + q0 + 1 - p.window, 0);
  const int t_lo = key_lo / KT, t_hi = (key_hi + KT - 1) / KT;
  const int total_pages = (key_hi + kPage - 1) / kPage;

  const uint32_t base = smem_u32(psm);
  auto issue = [&](int kt) {
    if (kt < t_hi) {
      const uint32_t sb = base + (kt & 1) * STAGE;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int page = kt * 2 + h;
        const bool valid = page < total_pages;
        const long long blk = valid ? bt[page] : 0;
        if constexpr (KV8) {
          const uint8_t* src = reinterpret_cast<const uint8_t*>(p.kv) + ((blk * p.nkv + kvh) * 2) * (long long)(kPage * DK);
          load_plane8<DK, 2 * kPage, 128>(sb + h * 2 * PLANE8, src, threadIdx.x, valid);
        } else {
          const __nv_bfloat16* src = p.kv + (blk * p.nkv + kvh) * (long long)(kPage * (DK + DV));
          load_plane<DK, kPage, 128>(sb + h * PLANE, src, threadIdx.x, valid);
          load_plane<DV, kPage, 128>(sb + 2 * PLANE + h * VPLANE, src + kPage * DK, threadIdx.x, valid);
        }
      }
    }
    cp_async_commit();
  };
  const uint32_t work = base + 2 * STAGE;        // fp8: the expanded bf16 planes of the tile being multiplied

  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float oacc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) { oacc[i][0] = oacc[i][1] = oacc[i][2] = oacc[i][3] = 0.f; }
  const float slope = p.alibi != nullptr ? p.alibi[head] : 0.f;

  issue(t_lo);
  for (int kt = t_lo; kt < t_hi; ++kt) {
    issue(kt + 1);
    cp_async_wait<1>();
    __syncthreads();
    uint32_t sb = base + (kt & 1) * STAGE;
    if constexpr (KV8) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        expand_plane8<DK, kPage, 128>(work + h * PLANE, sb + h * 2 * PLANE8, threadIdx.x);
        expand_plane8<DK, kPage, 128>(work + (2 + h) * PLANE, sb + h * 2 * PLANE8 + PLANE8, threadIdx.x);
      }
      __syncthreads();
      sb = work;
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float sacc[kPage / 8][4];
      qk_tile<DK, kPage>(sacc, qf, sb + h * PLANE, lane);
      softmax_tile<DV, kPage>(sacc, oacc, m, l, kt * KT + h * kPage, lo0, hi0, lo1, hi1, p.scale, p.softcap, lane, slope, slope);
      pv_tile<DV, kPage, WIDE>(oacc, sacc, sb + 2 * PLANE + h * VPLANE, lane);
    }
    __syncthreads();
  }
  cp_async_wait<0>();

#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  const float vs = KV8 ? p.v_scale : 1.f;
  const float inv0 = l[0] > 0.f ? vs * attn_denominator(p.tail, head, m[0] * kLog2e, l[0]) : 0.f;
  const float inv1 = l[1] > 0.f ? vs * attn_denominator(p.tail, head, m[1] * kLog2e, l[1]) : 0.f;
#pragma unroll
  for (int nd = 0; nd < DV / 8; ++nd) {
    const int c = nd * 8 + 2 * (lane & 3), col = head * DV + c;
    if (qr0 < qlen) {
      const float2 o = attn_turn_back(p.tail, make_float2(oacc[nd][0] * inv0, oacc[nd][1] * inv0), c, pos0);
      *reinterpret_cast<uint32_t*>(p.out + tok0 * p.ldo + (long long)head * DV + c) = pack_bf16x2(attn_tail(p.tail, o.x, tok0, col), attn_tail(p.tail, o.y, tok0, col + 1));
    }
    if (qr1 < qlen) {
      const float2 o = attn_turn_back(p.tail, make_float2(oacc[nd][2] * inv1, oacc[nd][3] * inv1), c, pos1);
      *reinterpret_cast<uint32_t*>(p.out + tok1 * p.ldo + (long long)head * DV + c) = pack_bf16x2(attn_tail(p.tail, o.x, tok1, col), attn_tail(p.tail, o.y, tok1, col + 1));
    }
  }
}

// Opts a kernel into `smem` bytes of dynamic shared memory, once per device.
template <typename K>
inline int attn_opt_in(K kernel, int smem, bool (&configured)[64]) {
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return -(int)e;
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  return 0;
}

template <int DK, int DV, int STAGES, bool KV8, int NW, bool WIDE = false>
static int launch_decode_nw(const DecodeParams& p, int T, cudaStream_t s) {
  constexpr int SMEM = KV8 ? NW * (STAGES * 2 * kPage * DK + 2 * kPage * DK * 2) : NW * STAGES * kPage * (DK + DV) * 2;
  static_assert(SMEM >= (NW * 16 * DV + 2 * NW * 16) * 4, "combine buffer must fit in the pipeline buffers");
  static bool configured[64] = {false};          // the shared-memory opt-in is a per-device attribute
  if (int rc = attn_opt_in(attn_decode_kernel<DK, DV, STAGES, KV8, NW, WIDE>, SMEM, configured)) return rc;
  dim3 grid(T, p.nkv * p.gchunks, p.nsplit);
  launch_pdl(attn_decode_kernel<DK, DV, STAGES, KV8, NW, WIDE>, grid, dim3(32 * NW), (size_t)SMEM, s, p);
  if (p.nsplit > 1) {
    dim3 g2(T, p.nh);
    launch_pdl(attn_combine_kernel<DV>, g2, dim3(DV), 0, s, p.part_o, p.part_lse, p.out, p.ldo, p.nh, p.nsplit, p.tail, p.ctx_lens);
  }
  return -(int)cudaGetLastError();
}

template <int DK, int DV, bool KV8, bool WIDE = false>
static int launch_prefill(const PrefillParams& p, int num_tiles, cudaStream_t s) {
  constexpr int SMEM = KV8 ? 2 * 4 * kPage * DK + 4 * kPage * DK * 2 : 2 * 2 * kPage * (DK + DV) * 2;
  static bool configured[64] = {false};
  if (int rc = attn_opt_in(attn_prefill_kernel<DK, DV, KV8, WIDE>, SMEM, configured)) return rc;
  dim3 grid(num_tiles, p.nh);
  launch_pdl(attn_prefill_kernel<DK, DV, KV8, WIDE>, grid, dim3(128), (size_t)SMEM, s, p);
  return -(int)cudaGetLastError();
}

}  // namespace lx
