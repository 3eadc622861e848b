// Absorbed latent attention for single query rows (decode rows, and portions too short to be worth an expansion): every cached row
// [latent | shared key part] is read once and serves as key and value of 16 or 32 heads at a time.
//
// One CTA of eight warps = one row x MT * 16 heads x one share of the keys, in tiles of 32 or 64 keys through a two-stage cp.async ring:
//   scores   four K slices x two key halves over the warps; the query fragments stay in registers, the slices' partial sums meet in
//            shared memory
//   softmax  fp32, eight or sixteen threads per head; the weights are split into two bf16 terms (value + remainder)
//   output   every warp owns an eighth of the latent columns of all heads, accumulated in registers
// Partial results of the key shares are combined by a second kernel.
#include "stream.cuh"

namespace lx {


struct LatentDecodeParams {
  const __nv_bfloat16* q_lat; long long ld_ql;    // [T, H * KR]
  const __nv_bfloat16* q; long long ldq;          // [T, H * head], shared-key part at rot_off
  int head, rot_off;
  const __nv_bfloat16* cache;                     // [blocks * page, R]
  __nv_bfloat16* out; long long ldo;              // [T, H * KR]
  StepRows rows;
  int H, R, page, nsplit;
  float scale;
  float* part_o;                                  // [T, H, nsplit, KR]
  float* part_ml;                                 // [T, H, nsplit, 2] maximum (log2 domain), sum
  int window;                                     // <= 0: none
};

LX_DEVICE void ld_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
LX_DEVICE void ld_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LX_DEVICE void ld_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LX_DEVICE float ld_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int MT, int KEYS, int WARPS>
struct LdSmem {
  static constexpr int kRows = MT * 16;
  static constexpr int kPartLd = KEYS + 4;
  static constexpr int kPLd = KEYS + 8;
  static constexpr int kPart = WARPS / 2 * kRows * kPartLd * 4;
  static constexpr int kP = 2 * kRows * kPLd * 2;
  static constexpr int kVec = 3 * kRows * 4;
  static int total(int R) { return 2 * KEYS * (R + 8) * 2 + kPart + kP + kVec; }
};

// KS: 16-wide K steps per slice; KR: latent columns; KEYS: keys per tile; WARPS: per CTA; OCC: CTAs per SM.
template <int MT, int KS, int KR, int KEYS, int WARPS, int OCC>
__global__ void __launch_bounds__(32 * WARPS, OCC) latent_decode_kernel(const LatentDecodeParams p) {
  pdl_trigger();
  pdl_wait();
  using S = LdSmem<MT, KEYS, WARPS>;
  constexpr int kLdThreads = 32 * WARPS, KG = WARPS / 2;      // K slices of the score products
  constexpr int NK2 = KEYS / 32;                   // 16-key steps of a warp's half of the tile
  constexpr int NT = KR / (8 * WARPS);                    // 8-wide column tiles per warp
  extern __shared__ __align__(16) uint8_t ld_sm[];
  const int pitch = (p.R + 8) * 2;                 // bytes; an odd multiple of 16: ldmatrix rows fall into different banks
  uint8_t* sk = ld_sm;
  float* part = reinterpret_cast<float*>(ld_sm + 2 * KEYS * pitch);
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(reinterpret_cast<uint8_t*>(part) + S::kPart);
  float* s_alpha = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(sp) + S::kP);
  float* s_m = s_alpha + S::kRows;
  float* s_l = s_m + S::kRows;
  const int t = blockIdx.x, h0 = blockIdx.y * S::kRows, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* bt;
  int keys;
  if (t < p.rows.nd) {
    keys = p.rows.ctx_lens[t];
    bt = p.rows.dec_bt + (long long)t * p.rows.dec_max_blocks;
  } else {
    const int b = seq_of(p.rows, t - p.rows.nd);
    keys = p.rows.cache_lens[b] + (t - p.rows.nd - p.rows.cu_q[b]) + 1;
    bt = p.rows.bt + (long long)b * p.rows.max_blocks;
  }
  keys = max(keys, 0);
  const int lo = p.window > 0 ? max(keys - p.window, 0) : 0;
  const int first = lo / KEYS, tiles = (keys + KEYS - 1) / KEYS;
  const int per = (tiles - first + p.nsplit - 1) / p.nsplit;
  const int t_lo = first + split * per, t_hi = min(t_lo + per, tiles);

  const int kg = warp % KG, kh = warp / KG;         // K slice, key half of the score products
  const int nk = p.R / 16;
  uint32_t qf[MT][KS][4];
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int s = 0; s < KS; ++s) {
      const int ks = kg * KS + s;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int hd = h0 + m * 16 + (lane >> 2) + (e & 1) * 8, c = ks * 16 + (lane & 3) * 2 + (e >> 1) * 8;
        uint32_t v = 0;
        if (hd < p.H && ks < nk)
          v = c < KR ? *reinterpret_cast<const uint32_t*>(p.q_lat + (long long)t * p.ld_ql + (long long)hd * KR + c)
                     : *reinterpret_cast<const uint32_t*>(p.q + (long long)t * p.ldq + (long long)hd * p.head + p.rot_off + c - KR);
        qf[m][s][e] = v;
      }
    }
  }
  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;

  auto load = [&](int tile, int st) {
    constexpr int TPK = kLdThreads / KEYS;          // threads per key
    const int r = threadIdx.x / TPK, key = tile * KEYS + r;
    const bool ok = key < keys;
    const __nv_bfloat16* src = p.cache;
    if (ok) src += ((long long)bt[key / p.page] * p.page + key % p.page) * p.R;
    uint8_t* dst = sk + (st * KEYS + r) * pitch;
    for (int c = threadIdx.x % TPK; c < p.R / 8; c += TPK) cp_async_16(dst + c * 16, ok ? src + c * 8 : src, ok);
    cp_async_commit();
  };

  constexpr int TPR = kLdThreads / S::kRows;       // softmax threads per head
  constexpr int KPT = KEYS / TPR;                  // keys of each
  static_assert(KPT % 2 == 0, "a softmax thread reads its keys' scores in pairs");
  const int srow = threadIdx.x / TPR, sk0 = (threadIdx.x % TPR) * KPT;
  const float scale_l2 = p.scale * 1.4426950408889634f;
  float mx = -INFINITY, sum = 0.f;                 // of head srow; sum: this thread's keys only

  if (t_lo < t_hi) load(t_lo, 0);
  for (int i = t_lo; i < t_hi; ++i) {
    const int st = (i - t_lo) & 1;
    cp_async_wait<0>();
    __syncthreads();
    if (i + 1 < t_hi) load(i + 1, st ^ 1);
    const uint32_t kb = smem_u32(sk) + (uint32_t)(st * KEYS * pitch);
    // ---- scores
    {
      float acc[MT][2 * NK2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2 * NK2; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
      const uint32_t a0 = kb + (uint32_t)((kh * (KEYS / 2) + (lane & 7) + (lane >> 4) * 8) * pitch + ((lane >> 3) & 1) * 16);
#pragma unroll
      for (int s = 0; s < KS; ++s) {
        const int ks = kg * KS + s;
        if (ks < nk) {
#pragma unroll
          for (int n2 = 0; n2 < NK2; ++n2) {
            uint32_t b[4];
            ld_ldsm(b, a0 + (uint32_t)(n2 * 16 * pitch + ks * 32));
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              ld_mma(acc[m][2 * n2], qf[m][s], b[0], b[1]);
              ld_mma(acc[m][2 * n2 + 1], qf[m][s], b[2], b[3]);
            }
          }
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2 * NK2; ++n) {
          float* d = part + (kg * S::kRows + m * 16 + (lane >> 2)) * S::kPartLd + kh * (KEYS / 2) + n * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(d) = make_float2(acc[m][n][0], acc[m][n][1]);
          *reinterpret_cast<float2*>(d + 8 * S::kPartLd) = make_float2(acc[m][n][2], acc[m][n][3]);
        }
    }
    __syncthreads();
    // ---- softmax
    {
      float s[KPT], bm = -INFINITY;
#pragma unroll
      for (int q = 0; q < KPT; q += 2) {
        float2 v = make_float2(0.f, 0.f);
#pragma unroll
        for (int g = 0; g < KG; ++g) {
          const float2 a = *reinterpret_cast<const float2*>(part + (g * S::kRows + srow) * S::kPartLd + sk0 + q);
          v.x += a.x; v.y += a.y;
        }
        s[q] = v.x; s[q + 1] = v.y;
      }
#pragma unroll
      for (int q = 0; q < KPT; ++q) {
        const int key = i * KEYS + sk0 + q;
        s[q] = (key >= lo && key < keys) ? s[q] * scale_l2 : -INFINITY;
        bm = fmaxf(bm, s[q]);
      }
#pragma unroll
      for (int w = TPR / 2; w > 0; w >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, w));
      const float mn = fmaxf(mx, bm);              // finite: every tile holds at least one visible key
      const float alpha = mx == -INFINITY ? 0.f : ld_ex2(mx - mn);
      mx = mn;
      sum *= alpha;
      __nv_bfloat16* ph = sp + srow * S::kPLd + sk0;
      __nv_bfloat16* pl = ph + S::kRows * S::kPLd;
#pragma unroll
      for (int q = 0; q < KPT; q += 2) {
        const float e0 = ld_ex2(s[q] - mn), e1 = ld_ex2(s[q + 1] - mn);
        sum += e0 + e1;
        const uint32_t hi = pack_bf16x2(e0, e1);
        const float2 back = unpack_bf16x2(hi);
        *reinterpret_cast<uint32_t*>(ph + q) = hi;
        *reinterpret_cast<uint32_t*>(pl + q) = pack_bf16x2(e0 - back.x, e1 - back.y);
      }
      if (threadIdx.x % TPR == 0) s_alpha[srow] = alpha;
    }
    __syncthreads();
    // ---- weighted latents
    {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float f0 = s_alpha[m * 16 + (lane >> 2)], f1 = s_alpha[m * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[m][n][0] *= f0; o[m][n][1] *= f0; o[m][n][2] *= f1; o[m][n][3] *= f1; }
      }
      const uint32_t pa = smem_u32(sp) + (uint32_t)(((lane & 15) * S::kPLd + (lane >> 4) * 8) * 2);
      const uint32_t vb = kb + (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (warp * (KR / WARPS) + (lane >> 4) * 8) * 2);
#pragma unroll
      for (int ks = 0; ks < KEYS / 16; ++ks) {
        uint32_t ah[MT][4], al[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          ld_ldsm(ah[m], pa + (uint32_t)((m * 16 * S::kPLd + ks * 16) * 2));
          ld_ldsm(al[m], pa + (uint32_t)(((S::kRows + m * 16) * S::kPLd + ks * 16) * 2));
        }
#pragma unroll
        for (int n2 = 0; n2 < NT / 2; ++n2) {
          uint32_t b[4];
          ld_ldsm_t(b, vb + (uint32_t)(ks * 16 * pitch + n2 * 32));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            ld_mma(o[m][2 * n2], ah[m], b[0], b[1]);
            ld_mma(o[m][2 * n2 + 1], ah[m], b[2], b[3]);
            ld_mma(o[m][2 * n2], al[m], b[0], b[1]);
            ld_mma(o[m][2 * n2 + 1], al[m], b[2], b[3]);
          }
        }
      }
    }
  }
#pragma unroll
  for (int w = TPR / 2; w > 0; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
  if (threadIdx.x % TPR == 0) { s_m[srow] = mx; s_l[srow] = sum; }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int hr = 0; hr < 2; ++hr) {
      const int r = m * 16 + (lane >> 2) + hr * 8, hd = h0 + r;
      if (hd >= p.H) continue;
      const float l = s_l[r], inv = l > 0.f ? 1.f / l : 0.f;
      const int c0 = warp * (KR / WARPS) + (lane & 3) * 2;
      if (p.nsplit == 1) {
        __nv_bfloat16* d = p.out + (long long)t * p.ldo + (long long)hd * KR + c0;
#pragma unroll
        for (int n = 0; n < NT; ++n)
          *reinterpret_cast<uint32_t*>(d + n * 8) = pack_bf16x2(o[m][n][2 * hr] * inv, o[m][n][2 * hr + 1] * inv);
      } else {
        const long long at = ((long long)t * p.H + hd) * p.nsplit + split;
#pragma unroll
        for (int n = 0; n < NT; ++n)
          *reinterpret_cast<float2*>(p.part_o + at * KR + c0 + n * 8) = make_float2(o[m][n][2 * hr], o[m][n][2 * hr + 1]);
        if (warp == 0 && (lane & 3) == 0) { p.part_ml[2 * at] = s_m[r]; p.part_ml[2 * at + 1] = l; }
      }
    }
}

// Shares of the keys -> one row: out = sum_s 2^(m_s - M) o_s / sum_s 2^(m_s - M) l_s.
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                             __nv_bfloat16* __restrict__ out, long long ldo, int H, int KR, int nsplit) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y;
  const long long base = ((long long)t * H + h) * nsplit;
  float M = -INFINITY, den = 0.f;
  for (int s = 0; s < nsplit; ++s)
    if (part_ml[2 * (base + s) + 1] > 0.f) M = fmaxf(M, part_ml[2 * (base + s)]);
  for (int s = 0; s < nsplit; ++s)
    if (part_ml[2 * (base + s) + 1] > 0.f) den += ld_ex2(part_ml[2 * (base + s)] - M) * part_ml[2 * (base + s) + 1];
  const float inv = den > 0.f ? 1.f / den : 0.f;
  for (int c = threadIdx.x * 4; c < KR; c += blockDim.x * 4) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < nsplit; ++s) {
      if (!(part_ml[2 * (base + s) + 1] > 0.f)) continue;
      const float w = ld_ex2(part_ml[2 * (base + s)] - M);
      const float4 v = load4(part_o + (base + s) * KR + c);
      a.x += w * v.x; a.y += w * v.y; a.z += w * v.z; a.w += w * v.w;
    }
    store4(out + (long long)t * ldo + (long long)h * KR + c, make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv));
  }
}

template <int MT, int KS, int KR, int KEYS, int WARPS, int OCC>
static int ld_launch(const LatentDecodeParams& p, int T, cudaStream_t s) {
  const int smem = LdSmem<MT, KEYS, WARPS>::total(p.R);
  if (smem > 227 * 1024) return -4;
  cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<MT, KS, KR, KEYS, WARPS, OCC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return -(int)e;
  const int groups = (p.H + MT * 16 - 1) / (MT * 16);
  launch_pdl(latent_decode_kernel<MT, KS, KR, KEYS, WARPS, OCC>, dim3(T, groups, p.nsplit), dim3(32 * WARPS), (size_t)smem, s, p);
  if (p.nsplit > 1)
    launch_pdl(latent_combine_kernel, dim3(T, p.H), dim3(128), 0, s, (const float*)p.part_o, (const float*)p.part_ml, p.out, p.ldo, p.H, KR, p.nsplit);
  return -(int)cudaGetLastError();
}

}  // namespace lx

extern "C" {

int lx_latent_decode_bytes() { return (int)sizeof(lx::LatentDecodeParams); }

// 1: latent and row widths the kernel takes (latent 128, 256 or 512 columns, shared key part of up to 64).
int lx_latent_decode_supported(int KR, int R) { return (R % 16 == 0 && R > KR && R - KR <= 64 && (KR == 128 || KR == 256 || KR == 512)) ? 1 : 0; }

int lx_latent_decode(const void* params, int KR, int T, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  const LatentDecodeParams& p = *reinterpret_cast<const LatentDecodeParams*>(params);
  if (!lx_latent_decode_supported(KR, p.R) || p.nsplit < 1 || (p.nsplit > 1 && (p.part_o == nullptr || p.part_ml == nullptr))) return -1;
  if (p.head % 2 != 0 || p.rot_off % 2 != 0 || p.ldq % 2 != 0 || p.ld_ql % 2 != 0 || p.ldo % 4 != 0) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  // up to 16 heads: 32-key tiles, two CTAs per SM hide each other's barriers; more: 32 heads share a 64-key tile
  const bool two = p.H > 16;
  if (KR == 512) return two ? ld_launch<2, 9, 512, 64, 8, 1>(p, T, s) : ld_launch<1, 9, 512, 32, 8, 2>(p, T, s);
  if (KR == 256) return two ? ld_launch<2, 5, 256, 64, 8, 1>(p, T, s) : ld_launch<1, 5, 256, 32, 8, 2>(p, T, s);
  return two ? ld_launch<2, 3, 128, 64, 8, 1>(p, T, s) : ld_launch<1, 3, 128, 32, 8, 2>(p, T, s);
}

}  // extern "C"
