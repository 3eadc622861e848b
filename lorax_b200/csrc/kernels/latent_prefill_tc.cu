// Prompt attention of the latent mixer on the tensor cores (tcgen05): the latents of the sequences of a step are gathered from their
// pages (with a window: what a portion's first query sees), expanded to per-head keys and values by one GEMM, and attended to here as
// plain multi-head attention with a key part that all heads share.  (The absorbed form in latent_attn.cu reads the latents once per query row instead: right for single tokens, three to
// four times the products for a prompt.)
//
// One CTA = 128 queries of one sequence x one head.  Keys are walked in blocks of 64:
//   loader (warp 0, one lane)   Q, then K panels (per-head part from the expansion, shared part from the gathered rows) and V panels by
//                               TMA, K and V in separate two-stage rings: a K stage is free as soon as its scores are done
//   MMA    (warp 1, one lane)   S_j = Q K_j^T into TMEM (double buffered); O += P_j V_j, accumulated in TMEM over all blocks
//   softmax (warps 2..5)        one thread per query: 64 scores in registers, exp2 against a reference maximum.  The weights stay fp32:
//                               they are split into two bf16 terms (value + remainder) and multiplied as two operands.  O is rescaled in
//                               TMEM only when a row's maximum grew by more than 2^8 over its reference.
// The output gate, one number per head or per element, multiplies the result on its way out.  Every wait is bounded and reports through the status word.
#include "stream.cuh"

namespace lx {

constexpr int kLpQ = 128, kLpKeys = 64, kLpThreads = 192;
constexpr float kLpLog2e = 1.4426950408889634f;
constexpr float kLpSlack = 8.f;                    // log2 of how far a row's maximum may run ahead of its reference

struct LatentPrefillParams {
  const int* tile_seq; const int* tile_q0;         // 128-query tiles
  const int* cu_q; const int* cache_lens;
  const int* ctx_off;                              // [B + 1] first gathered row of every sequence
  const __nv_bfloat16* gate; long long ldg;        // [T, ldg]; column h, or (gate_wide) the output's column
  __nv_bfloat16* out; long long ldo;               // rows of the prompt tokens
  int kv_head;                                     // columns of one head in the expansion (key part, then value)
  int q_head;                                      // columns of one head in q
  float scale;
  int* status;
  int window, gate_wide;                           // window <= 0: none
};

LX_DEVICE float lp_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
LX_DEVICE void tmem_st_32x32b_x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
      "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]),
      "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}

// NK / NR: 64-wide panels of the per-head and of the shared key part; NV: 64-wide panels of the value.
template <int NK, int NR, int NV>
struct LpSmem {
  static constexpr int kQ = (NK + NR) * kLpQ * 128;
  static constexpr int kK = (NK + NR) * kLpKeys * 128;
  static constexpr int kV = NV * kLpKeys * 128;
  static constexpr int kP = kLpQ * 128;            // one bf16 term of the weights
  static constexpr int kTotal = kQ + 2 * kK + 2 * kV + 4 * kP + 512 + 1024;
};

template <int NK, int NR, int NV>
__global__ void __launch_bounds__(kLpThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv,
                      const __grid_constant__ CUtensorMap tmap_rot, const LatentPrefillParams p) {
  pdl_trigger();
  using S = LpSmem<NK, NR, NV>;
  constexpr int NP = NK + NR;
  extern __shared__ uint8_t lp_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lp_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sq = smem;
  uint8_t* sk = sq + S::kQ;
  uint8_t* sv = sk + 2 * S::kK;
  uint8_t* sp = sv + 2 * S::kV;                    // [2 buffers][value, remainder]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sp + 4 * S::kP);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;       // 2
  uint64_t* k_empty = bars + 3;      // 2
  uint64_t* v_full = bars + 5;       // 2
  uint64_t* v_empty = bars + 7;      // 2
  uint64_t* s_full = bars + 9;       // 2
  uint64_t* s_empty = bars + 11;     // 2 (128 arrivals)
  uint64_t* p_full = bars + 13;      // 2 (128 arrivals)
  uint64_t* pv_done = bars + 15;     // 2
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 18);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile = (int)gridDim.x - 1 - (int)blockIdx.x;      // later tiles of a sequence see more keys: start the long ones first
  const int h = blockIdx.y;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 128);
      mbar_init(&p_full[i], 128); mbar_init(&pv_done[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_kv);
    tma_prefetch_desc(&tmap_rot);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 256); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;           // columns [0, 128): scores (two buffers of 64), [128, 128 + 64 NV): O
  pdl_wait();

  const int b = p.tile_seq[tile];
  const int q0 = p.tile_q0[tile];
  const int tok0 = p.cu_q[b];
  const int qlen = p.cu_q[b + 1] - tok0;
  const int cache = p.window > 0 ? min(p.cache_lens[b], p.window - 1) : p.cache_lens[b];       // gathered rows in front of the portion
  const int key_hi = cache + min(q0 + kLpQ, qlen);             // keys of the tile, in gathered rows: [key_lo, key_hi)
  const int key_lo = p.window > 0 ? max(cache + q0 + 1 - p.window, 0) : 0;
  const int first = key_lo / kLpKeys;                          // (block 0 below holds the rows from first * kLpKeys on)
  const int row_base = p.ctx_off[b] + first * kLpKeys;
  const int nblk = (key_hi + kLpKeys - 1) / kLpKeys - first;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, (uint32_t)S::kQ);
      for (int i = 0; i < NP; ++i) tma_load_2d(sq + i * kLpQ * 128, &tmap_q, q_full, h * p.q_head + i * 64, tok0 + q0);
      for (int j = 0; j < nblk; ++j) {
        const int st = j & 1;
        const int row = row_base + j * kLpKeys;
        if (!mbar_wait(&k_empty[st], ((j >> 1) & 1) ^ 1, abort_flag)) { report_status(p.status, kTimeoutEmptyBarrier, tile); *abort_flag = 1; break; }
        mbar_expect_tx(&k_full[st], (uint32_t)S::kK);
        for (int i = 0; i < NK; ++i) tma_load_2d(sk + st * S::kK + i * kLpKeys * 128, &tmap_kv, &k_full[st], h * p.kv_head + i * 64, row);
        for (int i = 0; i < NR; ++i) tma_load_2d(sk + st * S::kK + (NK + i) * kLpKeys * 128, &tmap_rot, &k_full[st], i * 64, row);
        if (!mbar_wait(&v_empty[st], ((j >> 1) & 1) ^ 1, abort_flag)) { report_status(p.status, kTimeoutEmptyBarrier, tile); *abort_flag = 1; break; }
        mbar_expect_tx(&v_full[st], (uint32_t)S::kV);
        for (int i = 0; i < NV; ++i) tma_load_2d(sv + st * S::kV + i * kLpKeys * 128, &tmap_kv, &v_full[st], h * p.kv_head + NK * 64 + i * 64, row);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc(128, kLpKeys, kFmtBF16, kFmtBF16);
      const uint32_t idesc_pv = make_idesc(128, NV * 64, kFmtBF16, kFmtBF16, 0, 1);
      const uint32_t sq_a = smem_u32(sq);
      bool ok = mbar_wait(q_full, 0, abort_flag);
      if (!ok) { report_status(p.status, kTimeoutFullBarrier, tile); *abort_flag = 1; }
      auto scores = [&](int j) -> bool {
        const int st = j & 1;
        if (!mbar_wait(&k_full[st], (j >> 1) & 1, abort_flag) || !mbar_wait(&s_empty[st], ((j >> 1) & 1) ^ 1, abort_flag)) {
          report_status(p.status, kTimeoutFullBarrier, tile); *abort_flag = 1; return false;
        }
        tc_fence_after();
        const uint32_t sk_a = smem_u32(sk + st * S::kK);
#pragma unroll
        for (int ks = 0; ks < NP * 4; ++ks) {
          const uint64_t da = make_desc_k_sw128(sq_a + (uint32_t)((ks >> 2) * kLpQ * 128)) + (uint64_t)((ks & 3) * 2);
          const uint64_t db = make_desc_k_sw128(sk_a + (uint32_t)((ks >> 2) * kLpKeys * 128)) + (uint64_t)((ks & 3) * 2);
          umma_f16_ss(tmem_base + (uint32_t)(st * 64), da, db, idesc_s, ks > 0 ? 1u : 0u);
        }
        tc_commit(&s_full[st]);
        tc_commit(&k_empty[st]);
        return true;
      };
      if (ok) ok = scores(0);
      for (int j = 0; ok && j < nblk; ++j) {
        const int st = j & 1;
        if (j + 1 < nblk && !scores(j + 1)) { ok = false; break; }
        if (!mbar_wait(&v_full[st], (j >> 1) & 1, abort_flag) || !mbar_wait(&p_full[st], (j >> 1) & 1, abort_flag)) {
          report_status(p.status, kTimeoutTmemEmpty, tile); *abort_flag = 1; ok = false; break;
        }
        tc_fence_after();
        const uint32_t sv_a = smem_u32(sv + st * S::kV);
#pragma unroll
        for (int term = 0; term < 2; ++term) {
          const uint32_t sp_a = smem_u32(sp + (st * 2 + term) * S::kP);
#pragma unroll
          for (int ks = 0; ks < kLpKeys / 16; ++ks) {
            const uint64_t da = make_desc_k_sw128(sp_a) + (uint64_t)(ks * 2);
            const uint64_t db = make_desc_mn_sw128(sv_a + (uint32_t)(ks * 2048), kLpKeys * 128, 1024);
            umma_f16_ss(tmem_base + 128u, da, db, idesc_pv, (j > 0 || term > 0 || ks > 0) ? 1u : 0u);
          }
        }
        tc_commit(&v_empty[st]);
        tc_commit(&pv_done[st]);
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3;
    const int row = quad * 32 + lane;
    const int qi = q0 + row;
    const bool row_ok = qi < qlen;
    const int hi = row_ok ? cache + qi + 1 : 0;                // keys this row sees
    const int lo = p.window > 0 ? max(hi - p.window, 0) : 0;
    const int hi_min = (q0 + kLpQ <= qlen) ? cache + q0 + 1 : 0;
    const int lo_max = p.window > 0 ? max(key_hi - p.window, 0) : 0;
    const float scale_l2 = p.scale * kLpLog2e;
    const uint32_t trow = tmem_base + ((uint32_t)(quad * 32) << 16);
    float m = -INFINITY, l = 0.f;                              // reference maximum (log2 domain), sum against it
    bool alive = true;
    for (int j = 0; j < nblk; ++j) {
      const int st = j & 1;
      if (!mbar_wait(&s_full[st], (j >> 1) & 1, abort_flag)) { report_status(p.status, kTimeoutTmemFull, tile); *abort_flag = 1; alive = false; break; }
      tc_fence_after();
      uint32_t r0[32], r1[32];
      tmem_ld_32x32b_x32(trow + (uint32_t)(st * 64), r0);
      tmem_ld_32x32b_x32(trow + (uint32_t)(st * 64 + 32), r1);
      tc_wait_ld();
      tc_fence_before();
      mbar_arrive(&s_empty[st]);
      float s[64];
#pragma unroll
      for (int i = 0; i < 32; ++i) { s[i] = __uint_as_float(r0[i]); s[32 + i] = __uint_as_float(r1[i]); }
      const int kb0 = (first + j) * kLpKeys;
      if (kb0 + kLpKeys > hi_min || kb0 < lo_max) {
#pragma unroll
        for (int i = 0; i < 64; ++i) s[i] = kb0 + i < hi && kb0 + i >= lo ? s[i] : -INFINITY;
      }
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 64; i += 4) {
        mx[0] = fmaxf(mx[0], s[i]); mx[1] = fmaxf(mx[1], s[i + 1]); mx[2] = fmaxf(mx[2], s[i + 2]); mx[3] = fmaxf(mx[3], s[i + 3]);
      }
      const float raw = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
      // scale may be negative or zero: then the largest score is not at the largest product
      float bm = raw * scale_l2;
      if (!(scale_l2 > 0.f)) {
        bm = -INFINITY;
#pragma unroll
        for (int i = 0; i < 64; ++i) bm = fmaxf(bm, s[i] == -INFINITY ? -INFINITY : s[i] * scale_l2);
      }
      float alpha = 1.f;
      if (bm > m + kLpSlack || m == -INFINITY) {
        alpha = m == -INFINITY ? (bm == -INFINITY ? 1.f : 0.f) : lp_ex2(m - bm);
        m = fmaxf(m, bm);
      }
      l *= alpha;
      const bool any = __any_sync(0xffffffffu, alpha != 1.f);
      // this buffer of weights is free once the products of block j - 2 are done
      if (!mbar_wait(&pv_done[st], ((j >> 1) & 1) ^ 1, abort_flag)) { report_status(p.status, kTimeoutTmemEmpty, tile); *abort_flag = 1; alive = false; break; }
      const float neg_m = m == -INFINITY ? 0.f : -m;
      uint8_t* pr = sp + st * 2 * S::kP + row * 128;
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        uint32_t w_hi[4], w_lo[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int i = c * 8 + q * 2;
          const float e0 = s[i] == -INFINITY ? 0.f : lp_ex2(fmaf(s[i], scale_l2, neg_m));
          const float e1 = s[i + 1] == -INFINITY ? 0.f : lp_ex2(fmaf(s[i + 1], scale_l2, neg_m));
          sum += e0 + e1;
          w_hi[q] = pack_bf16x2(e0, e1);
          const float2 back = unpack_bf16x2(w_hi[q]);
          w_lo[q] = pack_bf16x2(e0 - back.x, e1 - back.y);
        }
        const int at = ((c ^ (row & 7)) << 4);
        *reinterpret_cast<uint4*>(pr + at) = make_uint4(w_hi[0], w_hi[1], w_hi[2], w_hi[3]);
        *reinterpret_cast<uint4*>(pr + S::kP + at) = make_uint4(w_lo[0], w_lo[1], w_lo[2], w_lo[3]);
      }
      l += sum;
      if (any && j > 0) {
        if (!mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1, abort_flag)) { report_status(p.status, kTimeoutTmemFull, tile); *abort_flag = 1; alive = false; break; }
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < NV * 64; c += 32) {
          uint32_t o[32];
          tmem_ld_32x32b_x32(trow + (uint32_t)(128 + c), o);
          tc_wait_ld();
#pragma unroll
          for (int q = 0; q < 32; ++q) o[q] = __float_as_uint(__uint_as_float(o[q]) * alpha);
          tmem_st_32x32b_x32(trow + (uint32_t)(128 + c), o);
        }
        tc_wait_st();
      }
      tc_fence_before();
      fence_proxy_async_smem();
      mbar_arrive(&p_full[st]);
    }
    if (alive) {
      const int last = nblk - 1;
      if (mbar_wait(&pv_done[last & 1], (last >> 1) & 1, abort_flag)) {
        tc_fence_after();
        const long long tok = (long long)tok0 + qi;
        float f = 0.f;
        if (row_ok) f = (l > 0.f ? 1.f / l : 0.f) * (p.gate && !p.gate_wide ? sigmoid_f(to_f(p.gate[tok * p.ldg + h])) : 1.f);
        const __nv_bfloat16* grow = p.gate && p.gate_wide && row_ok ? p.gate + tok * p.ldg + (long long)h * NV * 64 : nullptr;
        __nv_bfloat16* orow = p.out + tok * p.ldo + (long long)h * NV * 64;
#pragma unroll
        for (int c = 0; c < NV * 64; c += 32) {
          uint32_t o[32];
          tmem_ld_32x32b_x32(trow + (uint32_t)(128 + c), o);
          tc_wait_ld();
          if (grow != nullptr) {
#pragma unroll
            for (int q = 0; q < 32; q += 8) {
              float z[8];
              load8(grow + c + q, z);
#pragma unroll
              for (int u = 0; u < 8; ++u) o[q + u] = __float_as_uint(__fdividef(__uint_as_float(o[q + u]), 1.f + __expf(-z[u])));
            }
          }
          if (row_ok) {
#pragma unroll
            for (int q = 0; q < 32; q += 8)
              *reinterpret_cast<uint4*>(orow + c + q) =
                  make_uint4(pack_bf16x2(__uint_as_float(o[q]) * f, __uint_as_float(o[q + 1]) * f),
                             pack_bf16x2(__uint_as_float(o[q + 2]) * f, __uint_as_float(o[q + 3]) * f),
                             pack_bf16x2(__uint_as_float(o[q + 4]) * f, __uint_as_float(o[q + 5]) * f),
                             pack_bf16x2(__uint_as_float(o[q + 6]) * f, __uint_as_float(o[q + 7]) * f));
          }
        }
      } else {
        report_status(p.status, kTimeoutTmemFull, tile);
        *abort_flag = 1;
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, 256); }
}

// Rows of the sequences' pages, in order, as one contiguous matrix: latents [N, KR] and shared key parts [N, RR].  With a window a
// sequence's rows begin window - 1 in front of its portion.
__global__ void __launch_bounds__(128) latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ bt, int max_blocks,
                                                            const int* __restrict__ ctx_off, const int* __restrict__ cache_lens, int window,
                                                            int B, int page, int KR, int RR,
                                                            __nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ rot) {
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  int lo = 0, hi = B;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (ctx_off[mid] <= r) lo = mid; else hi = mid;
  }
  const int pos = r - ctx_off[lo] + (window > 0 ? max(cache_lens[lo] - (window - 1), 0) : 0);
  const __nv_bfloat16* src = cache + ((long long)bt[(long long)lo * max_blocks + pos / page] * page + pos % page) * (KR + RR);
  for (int c = threadIdx.x * 8; c < KR + RR; c += blockDim.x * 8) {
    const uint4 v = *reinterpret_cast<const uint4*>(src + c);
    if (c < KR) *reinterpret_cast<uint4*>(lat + (long long)r * KR + c) = v;
    else *reinterpret_cast<uint4*>(rot + (long long)r * RR + c - KR) = v;
  }
}

typedef CUresult (*LpEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                               const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static int lp_map(CUtensorMap* m, const void* ptr, long long cols, long long rows, long long ld, int box_rows) {
  static LpEncodeFn fn = nullptr;
  if (fn == nullptr) {
    void* sym = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) return -1;
    fn = reinterpret_cast<LpEncodeFn>(sym);
  }
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
  cuuint32_t box[2] = {64, (cuuint32_t)box_rows};
  cuuint32_t es[2] = {1, 1};
  return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -2;
}

template <int NK, int NR, int NV>
static int lp_launch(const CUtensorMap& tq, const CUtensorMap& tkv, const CUtensorMap& tr, const LatentPrefillParams& p, int tiles, int H,
                     cudaStream_t s) {
  using S = LpSmem<NK, NR, NV>;
  static_assert(S::kTotal <= 227 * 1024, "shared memory");
  cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<NK, NR, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::kTotal);
  if (e != cudaSuccess) return -(int)e;
  launch_pdl(latent_prefill_kernel<NK, NR, NV>, dim3(tiles, H), dim3(kLpThreads), (size_t)S::kTotal, s, tq, tkv, tr, p);
  return -(int)cudaGetLastError();
}

}  // namespace lx

extern "C" {

int lx_latent_gather(const void* cache, const int* bt, int max_blocks, const int* ctx_off, const int* cache_lens, int window, int B, int rows,
                     int page, int KR, int RR, void* lat, void* rot, void* stream) {
  using namespace lx;
  if (rows <= 0) return 0;
  if (KR % 8 != 0 || RR % 8 != 0) return -1;
  launch_pdl(latent_gather_kernel, dim3(rows), dim3(128), 0, reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<const __nv_bfloat16*>(cache), bt,
             max_blocks, ctx_off, cache_lens, window, B, page, KR, RR, reinterpret_cast<__nv_bfloat16*>(lat), reinterpret_cast<__nv_bfloat16*>(rot));
  return -(int)cudaGetLastError();
}

// 1: head sizes (per-head key part, shared key part, value) the kernel takes.  A shared part of less than 64 columns is a panel whose tail
// the tensor map fills with zeros on the keys' side (the queries' side reads the columns behind the head's, which then count nothing).
int lx_latent_prefill_supported(int dk, int rot, int dv) {
  return rot > 0 && rot <= 64 && rot % 16 == 0 && ((dk == 128 && dv == 128) || (dk == 64 && (dv == 64 || dv == 128))) ? 1 : 0;
}

// q [T, ldq]: head h at column h * (dk + rot), per-head part first.  kv [rows, H * (dk + dv)] the expansion, rot_keys [rows, rot].
int lx_latent_prefill(const void* q, long long ldq, int T, const void* kv, const void* rot_keys, int rows, const int* ctx_off, const int* cu_q,
                      const int* cache_lens, const int* tile_seq, const int* tile_q0, int tiles, const void* gate, long long ldg, void* out,
                      long long ldo, int H, int dk, int rot, int dv, float scale, int window, int gate_wide, int* status, void* stream) {
  using namespace lx;
  if (tiles <= 0) return 0;
  if (!lx_latent_prefill_supported(dk, rot, dv) || ldq % 8 != 0 || ldo % 8 != 0 || (gate_wide && ldg % 8 != 0)) return -1;
  CUtensorMap tq, tkv, tr;
  if (lp_map(&tq, q, (long long)H * (dk + rot), T, ldq, kLpQ) || lp_map(&tkv, kv, (long long)H * (dk + dv), rows, (long long)H * (dk + dv), kLpKeys) ||
      lp_map(&tr, rot_keys, rot, rows, rot, kLpKeys))
    return -2;
  LatentPrefillParams p{};
  p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.cu_q = cu_q; p.cache_lens = cache_lens; p.ctx_off = ctx_off;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate); p.ldg = ldg;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.window = window; p.gate_wide = gate_wide;
  p.kv_head = dk + dv; p.q_head = dk + rot; p.scale = scale; p.status = status;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (dk == 128) return lp_launch<2, 1, 2>(tq, tkv, tr, p, tiles, H, s);
  if (dv == 64) return lp_launch<1, 1, 1>(tq, tkv, tr, p, tiles, H, s);
  return lp_launch<1, 1, 2>(tq, tkv, tr, p, tiles, H, s);
}

}  // extern "C"
