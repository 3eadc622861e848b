// Mixture-of-experts feed-forward on the device: routing, dispatch, grouped expert GEMMs, combine.
//
//   router logits   logits[t, e] = x[t, :] . Wr[e, :]: bf16 products, fp32 sums (mma.sync; K over the warps of a CTA)
//   select          one warp per token.  softmax: top-k of the logits, the weights renormalised over the chosen (the reference's routing
//                   math, server/lorax_server/models/custom_modeling/flash_mixtral_modeling.py:449-459) or over all experts.  sigmoid: the
//                   choice goes by score + correction; the weights are the scores without the correction, normalised or not.  Both: the
//                   choice may be limited to the best groups of neighbouring experts (by the largest of a group or its two largest), and
//                   the weights are multiplied by a constant
//   place, gather   the rows routed to each expert this rank owns become one contiguous run seg[e] .. seg[e+1] of a sorted order, and
//                   xg[p, :] = x[token of sorted row p, :]
//   grouped GEMM    work items (expert, 128 features of its weight, token tile of its run) on tcgen05: weights on the UMMA M
//                   side through one tensor map over the experts' stacked matrices, tokens on N, accumulators in TMEM;
//                   a token tile that runs past its expert's rows computes a few columns nobody stores
//   combine         out[t, :] = sum_j w[t, j] * y[pos[t, j], :]
//
// Shared experts (every token, weight one or sigmoid(one more router row)) are further runs of the same grouped products; their input rows
// are the tokens themselves and stand in xg once.
//
// Only the k experts a token was routed to do work for it (the reference gets that from megablocks' block-sparse kernels,
// flash_mixtral_modeling.py:517-666, and falls back to a dense all-experts bmm under 256 tokens, :668-722).  Every count lives
// on the device, every launch has static shapes (k * tokens rows at most), so a decode step with experts is one CUDA graph.
// Under expert parallelism a rank owns experts [e0, e0 + e_local): rows routed elsewhere get pos = -1 and the per-rank outputs
// are summed by the all-reduce that follows.
#include "common.cuh"

namespace lx {

constexpr int kMoeMaxExperts = 256;      // routed experts
constexpr int kMoeMaxShared = 32;
constexpr int kMoeMaxRuns = kMoeMaxExperts + kMoeMaxShared;
constexpr int kMoeMaxK = 32;

// ------------------------------------------------------------------------------------------------ router logits
// 16 * MT tokens x 8 * NT experts per CTA.  A lane loads eight neighbouring elements of a row of x and of Wr (16 bytes) and feeds them
// to two MMAs as the k pairs the fragment layout asks of it: x and Wr see the same permutation of k, so the sum is the same.
constexpr int kRouterWarps = 8;

LX_DEVICE void moe_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int MT, int NT, int UNROLL>
__global__ void __launch_bounds__(32 * kRouterWarps) moe_router_logits_kernel(const __nv_bfloat16* __restrict__ x, long long ldx,
                                                                              const __nv_bfloat16* __restrict__ wr, long long ldw,
                                                                              float* __restrict__ logits, int T, int E, int H, int* counts,
                                                                              int ncounts) {
  pdl_wait();
  __shared__ float red[kRouterWarps][16][8 * NT + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane >> 2, c = lane & 3;
  const int t0 = blockIdx.x * 16 * MT, n0 = blockIdx.y * 8 * NT;
  if (blockIdx.x == 0 && blockIdx.y == 0)
    for (int i = threadIdx.x; i < ncounts; i += blockDim.x) counts[i] = 0;
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int k0 = warp * 32; k0 < H; k0 += kRouterWarps * 32 * UNROLL) {
    uint4 b[UNROLL][NT], xa[UNROLL][MT][2];
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
      const int k = k0 + u * kRouterWarps * 32 + c * 8;
      const bool ok = k < H;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int e = n0 + n * 8 + r;
        b[u][n] = (ok && e < E) ? __ldg(reinterpret_cast<const uint4*>(wr + (long long)e * ldw + k)) : zero;
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = t0 + m * 16 + h * 8 + r;
          xa[u][m][h] = (ok && t < T) ? *reinterpret_cast<const uint4*>(x + (long long)t * ldx + k) : zero;
        }
    }
#pragma unroll
    for (int u = 0; u < UNROLL; ++u)
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const uint4 &p = xa[u][m][0], &q = xa[u][m][1];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          moe_mma(acc[m][n], p.x, q.x, p.y, q.y, b[u][n].x, b[u][n].y);
          moe_mma(acc[m][n], p.z, q.z, p.w, q.w, b[u][n].z, b[u][n].w);
        }
      }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    if (m > 0) __syncthreads();
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      red[warp][r][n * 8 + 2 * c] = acc[m][n][0];
      red[warp][r][n * 8 + 2 * c + 1] = acc[m][n][1];
      red[warp][r + 8][n * 8 + 2 * c] = acc[m][n][2];
      red[warp][r + 8][n * 8 + 2 * c + 1] = acc[m][n][3];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 16 * 8 * NT; i += blockDim.x) {
      const int row = i / (8 * NT), col = i % (8 * NT), t = t0 + m * 16 + row;
      if (t >= T || n0 + col >= E) continue;
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < kRouterWarps; ++w) sum += red[w][row][col];
      logits[(long long)t * E + n0 + col] = sum;
    }
  }
}

// ------------------------------------------------------------------------------------------------ select
struct MoeSelectParams {
  const float* logits;     // [T, ldl]
  const float* correction; // [E] or null (sigmoid)
  int* topk_ids;           // [T, k]
  float* topk_w;           // [T, k + shared]
  int* rank;               // [T, k + shared]: place of the row within its expert's run (-1: not on this rank)
  int* counts;             // [e_local], zero on entry
  long long ldl;
  int T, E, k, e0, e_local;
  int sigmoid, groups, keep, shared, group_top, renorm;
  float scale;
  int shared_one;          // the shared experts' weight is one (else the sigmoid of router row E)
  const float* bias;       // [E], added to the logits, or null
};

// Largest value of the warp and its index; the lower index on ties.
LX_DEVICE void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
  }
}

constexpr int kSelWarps = 8;

// The order of rows inside a run depends on the order of the atomics; every row's result is independent of it and the combine sums
// a token's contributions in index order.  PER: experts per lane.
template <int PER>
__global__ void __launch_bounds__(32 * kSelWarps) moe_select_kernel(const MoeSelectParams p) {
  pdl_wait();
  __shared__ float choice_s[kSelWarps][32 * PER];
  __shared__ uint8_t kept_s[kSelWarps][32 * PER];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * kSelWarps + warp;
  if (t >= p.T) return;
  const float* row = p.logits + (long long)t * p.ldl;
  auto logit = [&](int e) { return p.bias != nullptr ? row[e] + p.bias[e] : row[e]; };
  float choice[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i;
    float v = -INFINITY;
    if (e < p.E) {
      v = logit(e);
      if (p.sigmoid) v = 1.f / (1.f + expf(-v)) + (p.correction != nullptr ? p.correction[e] : 0.f);
    }
    choice[i] = v;
  }
  if (p.groups > 0) {
    const int gs = p.E / p.groups;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (lane + 32 * i < p.E) choice_s[warp][lane + 32 * i] = choice[i];
    __syncwarp();
    float score[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int g = lane + 32 * i;
      score[i] = -INFINITY;
      if (g < p.groups) {
        kept_s[warp][g] = 0;
        float a = -INFINITY, b = -INFINITY;                        // the two largest
        for (int q = 0; q < gs; ++q) {
          const float v = choice_s[warp][g * gs + q];
          if (v > a) { b = a; a = v; } else if (v > b) { b = v; }
        }
        score[i] = gs > 1 && p.group_top > 1 ? a + b : a;
      }
    }
    __syncwarp();
    for (int j = 0; j < p.keep; ++j) {
      float bv = -INFINITY;
      int bi = 0x7fffffff;
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if (score[i] > bv) { bv = score[i]; bi = lane + 32 * i; }
      warp_argmax(bv, bi);
      if (bi >= p.groups) bi = j;                                  // (scores that are not numbers: any group)
      if (lane == (bi & 31)) {
        kept_s[warp][bi] = 1;
#pragma unroll
        for (int i = 0; i < PER; ++i)
          if (i == (bi >> 5)) score[i] = -INFINITY;
      }
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = lane + 32 * i;
      if (e < p.E && !kept_s[warp][e / gs]) choice[i] = -INFINITY;
    }
  }
  int id = 0;
  float top = 0.f;
  for (int j = 0; j < p.k; ++j) {
    float bv = -INFINITY;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (choice[i] > bv) { bv = choice[i]; bi = lane + 32 * i; }
    warp_argmax(bv, bi);
    if (bi >= p.E) bi = j;
    if (lane == (bi & 31)) {
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if (i == (bi >> 5)) choice[i] = -INFINITY;
    }
    if (lane == j) id = bi;
    if (j == 0) top = logit(bi);
  }
  float w = 0.f;
  if (lane < p.k) w = p.sigmoid ? 1.f / (1.f + expf(-logit(id))) : expf(logit(id) - top);
  float sum = 1.f;
  if (p.renorm) {
    sum = warp_sum(w) + (p.sigmoid ? 1e-20f : 0.f);
  } else if (!p.sigmoid) {                       // (the first chosen logit is the largest of all)
    float own = 0.f;
    for (int e = lane; e < p.E; e += 32) own += expf(logit(e) - top);
    sum = warp_sum(own);
  }
  const int kw = p.k + p.shared;
  if (lane < p.k) {
    const int le = id - p.e0;
    p.topk_ids[(long long)t * p.k + lane] = id;
    p.topk_w[(long long)t * kw + lane] = w / sum * p.scale;
    p.rank[(long long)t * kw + lane] = (le >= 0 && le < p.e_local) ? atomicAdd(&p.counts[le], 1) : -1;
  }
  if (p.shared > 0) {
    const float g = p.shared_one ? 1.f : 1.f / (1.f + expf(-row[p.E]));
    for (int j = lane; j < p.shared; j += 32) p.topk_w[(long long)t * kw + p.k + j] = g;
  }
}

// ------------------------------------------------------------------------------------------------ place, gather, combine
// Every CTA sums the counts up by itself; one warp per (token, 2 KB of its row) turns the ranks of the token's choices into sorted rows
// and writes its part of the row to each of them (and to the shared experts' rows, which are the tokens in order).
struct MoePlaceParams {
  const uint8_t* x;
  uint8_t* xg;
  long long ldx, ldg;      // bytes
  int row_bytes;
  const int* counts;
  const int* topk_ids;
  const int* rank;         // [T, k + shared] of lx_moe_select
  int* pos;                // [T, k + shared]: sorted row (or -1)
  int* seg;                // [e_local + shared + 1]
  int T, k, e0, e_local, shared, rows_cap;
};

__global__ void __launch_bounds__(256) moe_place_kernel(const MoePlaceParams p) {
  pdl_wait();
  __shared__ int start[kMoeMaxExperts + 1];
  __shared__ int wsum[8];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  {
    const int c = (int)threadIdx.x < p.e_local ? p.counts[threadIdx.x] : 0;
    int v = c;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += u;
    }
    if (lane == 31) wsum[warp] = v;
    __syncthreads();
    for (int i = 0; i < warp; ++i) v += wsum[i];
    if ((int)threadIdx.x < p.e_local) start[threadIdx.x + 1] = v;
    if (threadIdx.x == 0) start[0] = 0;
  }
  __syncthreads();
  const int total = start[p.e_local], kw = p.k + p.shared;
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e <= p.e_local; e += blockDim.x) p.seg[e] = start[e];
    for (int i = threadIdx.x; i < p.shared; i += blockDim.x) p.seg[p.e_local + 1 + i] = total + (i + 1) * p.T;
  }
  constexpr int kPart = 2048;
  const int parts = (p.row_bytes + kPart - 1) / kPart;
  for (long long it = (blockIdx.x * (long long)blockDim.x + threadIdx.x) >> 5; it < (long long)p.T * parts;
       it += ((long long)gridDim.x * blockDim.x) >> 5) {
    const int t = (int)(it / parts), part = (int)(it % parts);
    uint4 v[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int b = part * kPart + i * 512 + lane * 16;
      if (b < p.row_bytes) v[i] = *reinterpret_cast<const uint4*>(p.x + (long long)t * p.ldx + b);
    }
    int q = -1;
    if (lane < p.k) {
      const int rank = p.rank[(long long)t * kw + lane];
      if (rank >= 0) q = start[p.topk_ids[(long long)t * p.k + lane] - p.e0] + rank;
      if (part == 0) p.pos[(long long)t * kw + lane] = q;
    }
    if (part == 0)
      for (int i = lane; i < p.shared; i += 32) p.pos[(long long)t * kw + p.k + i] = total + i * p.T + t;
    const int rows = p.k + (p.shared > 0 ? 1 : 0);
    for (int j = 0; j < rows; ++j) {
      const int row = j < p.k ? __shfl_sync(0xffffffffu, q, j) : total + t;
      if (row < 0 || row >= p.rows_cap) continue;
      uint8_t* dst = p.xg + (long long)row * p.ldg;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int b = part * kPart + i * 512 + lane * 16;
        if (b < p.row_bytes) *reinterpret_cast<uint4*>(dst + b) = v[i];
      }
    }
  }
}

// out[t, :] = sum_j w[t, j] * y[pos[t, j], :] over the experts of the token that this rank owns (fp32 sum in index order).
__global__ void __launch_bounds__(256) moe_combine_kernel(const __nv_bfloat16* __restrict__ y, long long ldy, const int* __restrict__ pos,
                                                          const float* __restrict__ w, int k, __nv_bfloat16* __restrict__ out, long long ldo,
                                                          int T, int H) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  for (int t = (blockIdx.x * blockDim.x + threadIdx.x) >> 5; t < T; t += (gridDim.x * blockDim.x) >> 5) {
    for (int h = lane * 8; h < H; h += 256) {
      float acc[8];
#pragma unroll
      for (int q = 0; q < 8; ++q) acc[q] = 0.f;
      for (int j = 0; j < k; ++j) {
        const int q = pos[t * k + j];
        if (q < 0) continue;
        const float wj = w[t * k + j];
        const uint4 v = *reinterpret_cast<const uint4*>(y + (long long)q * ldy + h);
        const uint32_t vw[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float2 f = unpack_bf16x2(vw[u]);
          acc[2 * u] = fmaf(wj, f.x, acc[2 * u]);
          acc[2 * u + 1] = fmaf(wj, f.y, acc[2 * u + 1]);
        }
      }
      *reinterpret_cast<uint4*>(out + (long long)t * ldo + h) =
          make_uint4(pack_bf16x2(acc[0], acc[1]), pack_bf16x2(acc[2], acc[3]), pack_bf16x2(acc[4], acc[5]), pack_bf16x2(acc[6], acc[7]));
    }
  }
}

// ------------------------------------------------------------------------------------------------ grouped GEMM
constexpr int kMgBM = 128;
constexpr int kMgBK = 64;
constexpr int kMgThreads = 192;

// swiglu: the weight's rows are gate and up in turn, output column i is silu(row 2i) * row 2i + 1.
enum MoeAct : int { kMoeActNone = 0, kMoeActRelu2 = 1, kMoeActSwiglu = 2 };
LX_DEVICE float moe_act(float v, int act) {
  if (act == kMoeActRelu2) { v = fmaxf(v, 0.f); v *= v; }
  return v;
}

struct MoeGemmParams {
  int K, n_w, runs;               // runs: routed experts of this rank, then the shared ones
  const int* seg;                 // [runs + 1] rows of every run in the sorted order
  __nv_bfloat16* out;             // [rows, n_w], swiglu: [rows, n_w / 2]
  long long ldo;
  int bn;                         // token tile = UMMA N (multiple of 16, <= BN)
  int rows_cap;                   // rows the output holds
  int shared, tokens;             // the last `shared` runs all read the `tokens` input rows of the first of them (0: their own)
  int act;
  int* status;
};

constexpr int kMgTail = 1024 + (2 * (kMoeMaxRuns + 1) * 4 + 1023) / 1024 * 1024;      // barriers, then the run table

template <int BN, int STAGES>
struct MgSmem {
  static constexpr int kABytes = kMgBM * kMgBK * 2;
  static constexpr int kBBytes = BN * kMgBK * 2;
  static constexpr int kStage = kABytes + kBBytes;
  static constexpr int kTotal = STAGES * kStage + 1024 + kMgTail;
};

// Work item g -> (run, feature tile, token tile).  Token tiles of one (run, feature tile) are adjacent, so CTAs that run side by
// side read the same weight tile through L2 and it leaves HBM once.
struct MgIter {
  int runs, tiles_a, bn;
  const int* start;               // [runs + 1] first row of every run (shared memory)
  const int* cum;                 // [runs + 1] work items before it
  // one warp fills the two tables
  static LX_DEVICE void build(const int* seg, int runs, int rows_cap, int tiles_a, int bn, int* start, int* cum) {
    const int lane = threadIdx.x & 31;
    int base = 0;
    for (int e0 = 0; e0 < runs; e0 += 32) {
      const int e = e0 + lane;
      int a = 0, v = 0;
      if (e < runs) {
        a = min(seg[e], rows_cap);
        v = tiles_a * ((min(seg[e + 1], rows_cap) - a + bn - 1) / bn);
      }
      int s = v;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += u;
      }
      if (e < runs) { start[e] = a; cum[e] = base + s - v; }
      base += __shfl_sync(0xffffffffu, s, 31);
    }
    if (lane == 0) { start[runs] = min(seg[runs], rows_cap); cum[runs] = base; }
  }
  __device__ int total() const { return cum[runs]; }
  __device__ void decode(int g, int& e, int& ta, int& tb, int& row0, int& nrows) const {
    int lo = 0, hi = runs;                       // the last run with cum <= g (an empty run before it has the same cum)
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (cum[mid] <= g) lo = mid; else hi = mid;
    }
    e = lo;
    const int local = g - cum[e];
    const int cnt = start[e + 1] - start[e];
    const int nt = (cnt + bn - 1) / bn;
    ta = local / nt;
    tb = local - ta * nt;
    row0 = start[e] + tb * bn;
    nrows = min(bn, cnt - tb * bn);
  }
};

template <int BN, int STAGES>
__global__ void __launch_bounds__(kMgThreads, 1)
moe_grouped_gemm_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, const MoeGemmParams p) {
  using S = MgSmem<BN, STAGES>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* tiles = smem;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + STAGES * S::kStage);
  uint64_t* empty_bar = full_bar + STAGES;
  uint64_t* tmem_full = empty_bar + STAGES;
  uint64_t* tmem_empty = tmem_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tmem_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* start_s = reinterpret_cast<int*>(smem + STAGES * S::kStage + 1024);             // [runs + 1]
  int* cum_s = start_s + kMoeMaxRuns + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr uint32_t kTmemCols = (2 * BN < 32) ? 32 : 2 * BN;
  const int kblocks = (p.K + kMgBK - 1) / kMgBK;

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
    for (int s = 0; s < 2; ++s) { mbar_init(&tmem_full[s], 1); mbar_init(&tmem_empty[s], 4); }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmap_w);
    tma_prefetch_desc(&tmap_x);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, kTmemCols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_wait();
  if (warp == 0) MgIter::build(p.seg, p.runs, p.rows_cap, p.n_w / kMgBM, p.bn, start_s, cum_s);
  __syncthreads();
  const MgIter it{p.runs, p.n_w / kMgBM, p.bn, start_s, cum_s};
  const int shared0 = p.runs - p.shared;

  if (warp == 0) {
    if (lane == 0) {
      const uint64_t pol_w = policy_evict_first(), pol_x = policy_evict_last();
      int stage = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int g = (int)blockIdx.x; ok && g < it.total(); g += (int)gridDim.x) {
        int e, ta, tb, row0, nrows;
        it.decode(g, e, ta, tb, row0, nrows);
        const int xrow = row0 - (e > shared0 ? (e - shared0) * p.tokens : 0);
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&empty_bar[stage], phase ^ 1, abort_flag)) { report_status(p.status, kTimeoutEmptyBarrier, g); *abort_flag = 1; ok = false; break; }
          uint8_t* sa = tiles + stage * S::kStage;
          mbar_expect_tx(&full_bar[stage], (uint32_t)(S::kABytes + p.bn * kMgBK * 2));
          tma_load_2d_hint(sa, &tmap_w, &full_bar[stage], kb * kMgBK, e * p.n_w + ta * kMgBM, pol_w);
          tma_load_2d_hint(sa + S::kABytes, &tmap_x, &full_bar[stage], kb * kMgBK, xrow, pol_x);
          if (++stage == STAGES) { stage = 0; phase ^= 1; }
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = make_idesc(kMgBM, (uint32_t)p.bn, kFmtBF16, kFmtBF16);
      int stage = 0, acc = 0;
      uint32_t phase = 0, acc_phase[2] = {0, 0};
      bool ok = true;
      for (int g = (int)blockIdx.x; ok && g < it.total(); g += (int)gridDim.x) {
        if (!mbar_wait(&tmem_empty[acc], acc_phase[acc] ^ 1, abort_flag)) { report_status(p.status, kTimeoutTmemEmpty, g); *abort_flag = 1; break; }
        tc_fence_after();
        const uint32_t tmem_d = tmem_base + (uint32_t)(acc * BN);
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&full_bar[stage], phase, abort_flag)) { report_status(p.status, kTimeoutFullBarrier, g); *abort_flag = 1; ok = false; break; }
          tc_fence_after();
          const uint32_t sa = smem_u32(tiles + stage * S::kStage);
          const uint64_t da = make_desc_k_sw128(sa), db = make_desc_k_sw128(sa + S::kABytes);
#pragma unroll
          for (int k = 0; k < kMgBK / 16; ++k) umma_f16_ss(tmem_d, da + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc, (kb > 0 || k > 0) ? 1u : 0u);
          tc_commit(&empty_bar[stage]);
          if (++stage == STAGES) { stage = 0; phase ^= 1; }
        }
        if (!ok) break;
        tc_commit(&tmem_full[acc]);
        acc_phase[acc] ^= 1;
        acc ^= 1;
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3;
    int acc = 0;
    uint32_t acc_phase[2] = {0, 0};
    for (int g = (int)blockIdx.x; g < it.total(); g += (int)gridDim.x) {
      int e, ta, tb, row0, nrows;
      it.decode(g, e, ta, tb, row0, nrows);
      if (!mbar_wait(&tmem_full[acc], acc_phase[acc], abort_flag)) { report_status(p.status, kTimeoutTmemFull, g); *abort_flag = 1; break; }
      tc_fence_after();
      acc_phase[acc] ^= 1;
      const uint32_t taddr = tmem_base + ((uint32_t)(quad * 32) << 16) + (uint32_t)(acc * BN);
      const int i = ta * kMgBM + quad * 32 + lane;             // feature of this lane
      constexpr int CH = (BN >= 32) ? 32 : 16;
#pragma unroll 1
      for (int c = 0; c < p.bn; c += CH) {
        float v[CH];
        if constexpr (CH == 32) {
          uint32_t r[32];
          tmem_ld_32x32b_x32(taddr + c, r);
          tc_wait_ld();
#pragma unroll
          for (int q = 0; q < 32; ++q) v[q] = __uint_as_float(r[q]);
        } else {
          uint32_t r[16];
          tmem_ld_32x32b_x16(taddr + c, r);
          tc_wait_ld();
#pragma unroll
          for (int q = 0; q < 16; ++q) v[q] = __uint_as_float(r[q]);
        }
        if (p.act == kMoeActSwiglu) {
          // gate and up of a column sit in neighbouring lanes: each lane of the pair finishes half of the tokens
          const bool odd = lane & 1;
#pragma unroll
          for (int q = 0; q < CH / 2; ++q) {
            const float other = __shfl_xor_sync(0xffffffffu, odd ? v[q] : v[q + CH / 2], 1);
            const float g = odd ? other : v[q], up = odd ? v[q + CH / 2] : other;
            const int tok = c + q + (odd ? CH / 2 : 0);
            if (tok < nrows) p.out[(long long)(row0 + tok) * p.ldo + (i >> 1)] = __float2bfloat16(__fdividef(g, 1.f + __expf(-g)) * up);
          }
        } else if (i < p.n_w) {
#pragma unroll
          for (int q = 0; q < CH; ++q) {
            if (c + q < nrows) p.out[(long long)(row0 + c + q) * p.ldo + i] = __float2bfloat16(moe_act(v[q], p.act));
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tmem_empty[acc]);
      acc ^= 1;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, kTmemCols); }
}

// The same product in true fp32: 64 features x 64 rows of one run per CTA.
__global__ void __launch_bounds__(256) moe_grouped_gemm_f32_kernel(const float* __restrict__ x, long long ldx, const float* __restrict__ w,
                                                                   long long ldw, float* __restrict__ out, const MoeGemmParams p) {
  pdl_wait();
  __shared__ float xs[16][68], ws[16][68];
  __shared__ int tile_s[3];
  if (threadIdx.x == 0) {
    int left = blockIdx.y, e = 0;
    tile_s[0] = -1;
    for (; e < p.runs; ++e) {
      const int cnt = min(p.seg[e + 1], p.rows_cap) - min(p.seg[e], p.rows_cap), nt = (cnt + 63) / 64;
      if (left < nt) { tile_s[0] = e; tile_s[1] = min(p.seg[e], p.rows_cap) + left * 64; tile_s[2] = min(64, cnt - left * 64); break; }
      left -= nt;
    }
  }
  __syncthreads();
  const int e = tile_s[0], row0 = tile_s[1], nrows = tile_s[2], n0 = blockIdx.x * 64;
  if (e < 0) return;
  const int shared0 = p.runs - p.shared;
  const float* xr = x + (long long)(row0 - (e > shared0 ? (e - shared0) * p.tokens : 0)) * ldx;
  const float* we = w + (long long)e * p.n_w * ldw;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int k = k0 + lk + q;
      xs[lk + q][lr] = (lr < nrows && k < p.K) ? xr[(long long)lr * ldx + k] : 0.f;
      ws[lk + q][lr] = (n0 + lr < p.n_w && k < p.K) ? we[(long long)(n0 + lr) * ldw + k] : 0.f;
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
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= nrows) continue;
    if (p.act == kMoeActSwiglu) {
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        const int n = n0 + tx * 4 + j;
        if (n < p.n_w) out[(long long)(row0 + r) * p.ldo + (n >> 1)] = acc[i][j] / (1.f + expf(-acc[i][j])) * acc[i][j + 1];
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < p.n_w) out[(long long)(row0 + r) * p.ldo + n] = moe_act(acc[i][j], p.act);
    }
  }
}

int make_tmap_bf16_kmajor(CUtensorMap* out, const void* base, uint64_t rows, uint64_t K, uint64_t row_stride_elems, uint32_t box_rows);

template <int BN, int STAGES>
static int launch_moe_gemm(const CUtensorMap& tw, const CUtensorMap& tx, const MoeGemmParams& p, int grid, cudaStream_t stream) {
  using S = MgSmem<BN, STAGES>;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    cudaError_t e = cudaFuncSetAttribute(moe_grouped_gemm_kernel<BN, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::kTotal);
    if (e != cudaSuccess) return -(int)e;
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  launch_pdl(moe_grouped_gemm_kernel<BN, STAGES>, dim3(grid), dim3(kMgThreads), (size_t)S::kTotal, stream, tw, tx, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

}  // namespace lx

extern "C" {

// logits[T, E] (fp32) = x[T, H] @ wr[E, H]^T; also zeroes counts[0 .. ncounts) for lx_moe_select.
int lx_moe_router_logits(const void* x, long long ldx, const void* wr, long long ldw, float* logits, int T, int E, int H, int* counts,
                         int ncounts, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (H % 8 != 0 || ldx % 8 != 0 || ldw % 8 != 0) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const __nv_bfloat16* xp = reinterpret_cast<const __nv_bfloat16*>(x);
  const __nv_bfloat16* wp = reinterpret_cast<const __nv_bfloat16*>(wr);
#define LX_RL(MT, NT, UN)                                                                                                                    \
  launch_pdl(moe_router_logits_kernel<MT, NT, UN>, dim3((T + 16 * MT - 1) / (16 * MT), (E + 8 * NT - 1) / (8 * NT)), dim3(32 * kRouterWarps), 0, s, \
             xp, ldx, wp, ldw, logits, T, E, H, counts, ncounts)
  const int tiles = (E + 7) / 8;
  if (tiles == 1) { if (T >= 4096) LX_RL(2, 1, 4); else LX_RL(1, 1, 8); }
  else if (T <= 512) LX_RL(1, 2, 8);                               // few tokens: the experts' rows are spread over the CTAs
  else if (tiles == 2) LX_RL(2, 2, 4);
  else if (tiles == 3) LX_RL(2, 3, 4);
  else if (tiles <= 5) LX_RL(2, 5, 2);
  else if (tiles <= 8) LX_RL(2, 8, 2);
  else LX_RL(2, 9, 2);
#undef LX_RL
  return -(int)cudaGetLastError();
}

int lx_moe_select_bytes() { return (int)sizeof(lx::MoeSelectParams); }
int lx_moe_place_bytes() { return (int)sizeof(lx::MoePlaceParams); }

int lx_moe_select(const void* params, void* stream) {
  using namespace lx;
  const MoeSelectParams& p = *reinterpret_cast<const MoeSelectParams*>(params);
  if (p.T <= 0) return 0;
  if (p.E > kMoeMaxExperts || p.E < 1 || p.k > kMoeMaxK || p.k > p.E || p.k < 1 || p.e_local > kMoeMaxExperts || p.shared > kMoeMaxShared) return -1;
  if (p.ldl < p.E + (p.shared > 0 && !p.shared_one ? 1 : 0)) return -2;
  if (p.group_top < 1 || p.group_top > 2 || (!p.sigmoid && p.groups > 0 && p.group_top != 1)) return -4;
  if (p.groups > 0 && (p.E % p.groups != 0 || p.keep < 1 || p.keep > p.groups || p.keep * (p.E / p.groups) < p.k)) return -3;
  const dim3 grid((p.T + kSelWarps - 1) / kSelWarps), block(32 * kSelWarps);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (p.E <= 32) launch_pdl(moe_select_kernel<1>, grid, block, 0, s, p);
  else if (p.E <= 64) launch_pdl(moe_select_kernel<2>, grid, block, 0, s, p);
  else if (p.E <= 128) launch_pdl(moe_select_kernel<4>, grid, block, 0, s, p);
  else launch_pdl(moe_select_kernel<8>, grid, block, 0, s, p);
  return -(int)cudaGetLastError();
}

int lx_moe_place(const void* params, void* stream) {
  using namespace lx;
  const MoePlaceParams& p = *reinterpret_cast<const MoePlaceParams*>(params);
  if (p.T <= 0) return 0;
  if (p.row_bytes % 16 != 0 || p.ldx % 16 != 0 || p.ldg % 16 != 0 || p.e_local > kMoeMaxExperts || p.e_local < 1) return -1;
  const long long items = (long long)p.T * ((p.row_bytes + 2047) / 2048);
  const int blocks = (int)(items / 8 + 1 < 148 * 8 ? items / 8 + 1 : 148 * 8);
  launch_pdl(moe_place_kernel, dim3(blocks), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), p);
  return -(int)cudaGetLastError();
}

int lx_moe_combine(const void* y, long long ldy, const int* pos, const float* w, int k, void* out, long long ldo, int T, int H, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (H % 8 != 0 || ldy % 8 != 0 || ldo % 8 != 0) return -1;
  const int blocks = min((T * 32 + 255) / 256, 148 * 8);
  launch_pdl(moe_combine_kernel, dim3(blocks), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<const __nv_bfloat16*>(y), ldy,
             pos, w, k, reinterpret_cast<__nv_bfloat16*>(out), ldo, T, H);
  return -(int)cudaGetLastError();
}

// out[q, :] = act(xg[q, :] @ W_e(q)^T) for every sorted row q, e(q) the run that holds q.  w: the experts' matrices stacked
// [runs * n_w, K]; n_w must be a multiple of 128.  The last `shared` runs all read the `tokens` rows at the beginning of the first of
// them (0: every run has input rows of its own).  x_rows / rows_cap: rows of xg / of out.  avg_rows (rows per expert the caller
// expects) picks the token tile.
int lx_moe_grouped_gemm(const void* xg, long long ldx, const void* w, long long ldw, void* out, long long ldo, const int* seg, int runs, int x_rows,
                        int rows_cap, int n_w, int K, int avg_rows, int shared, int tokens, int act, int f32, int* status, int num_sms,
                        void* stream) {
  using namespace lx;
  if (rows_cap <= 0 || runs <= 0) return 0;
  if (n_w % kMgBM != 0 || K % 8 != 0 || ldx % 8 != 0 || ldw % 8 != 0 || runs > kMoeMaxRuns || shared < 0 || shared > runs) return -1;
  MoeGemmParams p{};
  p.K = K; p.n_w = n_w; p.runs = runs; p.seg = seg; p.shared = shared; p.tokens = shared > 0 ? tokens : 0; p.act = act;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.rows_cap = rows_cap; p.status = status;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (f32) {
    launch_pdl(moe_grouped_gemm_f32_kernel, dim3((n_w + 63) / 64, rows_cap / 64 + runs), dim3(256), 0, s, reinterpret_cast<const float*>(xg), ldx,
               reinterpret_cast<const float*>(w), ldw, reinterpret_cast<float*>(out), p);
    return -(int)cudaGetLastError();
  }
  // few rows per expert: a tile twice the average holds most runs whole (a second tile would read the weights again)
  int bn = ((avg_rows < 128 ? 2 * avg_rows : avg_rows) + 15) / 16 * 16;
  if (bn < 16) bn = 16;
  if (bn > 256) bn = 256;
  const int tbn = bn <= 16 ? 16 : bn <= 32 ? 32 : bn <= 64 ? 64 : bn <= 128 ? 128 : 256;
  p.bn = bn;
  CUtensorMap tw, tx;
  if (make_tmap_bf16_kmajor(&tw, w, (uint64_t)runs * n_w, K, ldw, kMgBM)) return -2;
  if (make_tmap_bf16_kmajor(&tx, xg, x_rows, K, ldx, bn)) return -3;
  switch (tbn) {
    case 16:  return launch_moe_gemm<16, 8>(tw, tx, p, num_sms, s);
    case 32:  return launch_moe_gemm<32, 8>(tw, tx, p, num_sms, s);
    case 64:  return launch_moe_gemm<64, 8>(tw, tx, p, num_sms, s);
    case 128: return launch_moe_gemm<128, 6>(tw, tx, p, num_sms, s);
    default:  return launch_moe_gemm<256, 4>(tw, tx, p, num_sms, s);
  }
}

}  // extern "C"
