// Grouped-query attention of the layer-by-layer designs: per-head norms of queries and keys fused with the cache write, and softmax
// attention with head counts, widths of keys and values, and a window that belong to the layer.
//
//   qk_norm_kvwrite   q and k divided by their root mean square per head (fp32), times a weight; where asked for, their first columns
//                     rotated, and the values by a table of their own (pairs of neighbours); k and v to the paged cache
//   bf16              the kernels of attention.cuh with the fp32 softmax weights carried into the value product as two bf16 terms
//                     (widths 64, 128, 256); prompts with keys and values of 128 run on attn_prefill_tc.cu
//   fp32              one warp per (token, head)
//
// Cache of a layer: [num_blocks, kv heads, page * (DK + DV)], a page of one head being its key plane, then its value plane.
#include "attention.cuh"
#include "stream.cuh"

namespace lx {

// ------------------------------------------------------------------------------------------------
// Eight columns per thread; the threads of one head are neighbours within a warp.  blockIdx.y = 0: q and k heads, 1: v heads.
// ------------------------------------------------------------------------------------------------
struct QkNormParams {
  void* qkv;                   // [T, ld]: q heads (DK wide), k heads (DK), v heads (DV)
  long long ld;
  void* cache;
  const int* slots;            // [T] token slot in the cache, < 0: none
  const float* q_norm;         // [DK]
  const float* k_norm;
  int T, H, G, DK, DV, page;
  float inv_n, eps;
  const int* positions;        // [T] (with a table)
  const float* cos_sin;        // [P, rot] cos, then sin; null: no rotation of q and k
  const float* v_cos_sin;      // [P, v_rot]; null: none of v
  int rot, v_rot, P;
};

// Columns [c, c + 8) of a head turned by row `pos` of the table.
LX_DEVICE void turn8(float (&f)[8], const float* __restrict__ table, int rot, int pos, int c) {
  const float* cs = table + (long long)pos * rot + (c >> 1);
  float co[4], si[4];
  if (rot % 8 == 0) {
    const float4 a = __ldg(reinterpret_cast<const float4*>(cs)), b = __ldg(reinterpret_cast<const float4*>(cs + (rot >> 1)));
    co[0] = a.x; co[1] = a.y; co[2] = a.z; co[3] = a.w;
    si[0] = b.x; si[1] = b.y; si[2] = b.z; si[3] = b.w;
  } else {
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const bool on = c + 2 * q < rot;
      co[q] = on ? __ldg(cs + q) : 1.f;
      si[q] = on ? __ldg(cs + (rot >> 1) + q) : 0.f;
    }
  }
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    const float u = f[2 * q], v = f[2 * q + 1];
    f[2 * q] = u * co[q] - v * si[q];
    f[2 * q + 1] = v * co[q] + u * si[q];
  }
}

template <typename T>
__global__ void __launch_bounds__(256) qk_norm_kvwrite_kernel(const QkNormParams p) {
  pdl_trigger();
  pdl_wait();
  const bool values = blockIdx.y == 1;
  const int width = values ? p.DV : p.DK, lanes = width / 8;                      // 8, 16 or 32 threads
  const unsigned heads = values ? p.G : p.H + p.G;
  const unsigned item = (blockIdx.x * blockDim.x + threadIdx.x) >> (31 - __clz(lanes));
  const int c = (int)(threadIdx.x & (lanes - 1)) * 8;
  const bool live = item < (unsigned)p.T * heads;
  const int t = live ? (int)(item / heads) : 0, h = live ? (int)(item - t * heads) : 0;
  T* src = reinterpret_cast<T*>(p.qkv) + t * p.ld + (values ? (long long)(p.H + p.G) * p.DK : 0) + (long long)h * width + c;
  float f[8];
  load8(src, f);
  if (!values) {
    float ss = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) ss += f[q] * f[q];
    for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float r = rsqrtf(ss * p.inv_n + p.eps);
    float g[8];
    load8((h < p.H ? p.q_norm : p.k_norm) + c, g);
#pragma unroll
    for (int q = 0; q < 8; ++q) f[q] *= r * g[q];
  }
  if (!live) return;
  const float* table = values ? p.v_cos_sin : p.cos_sin;
  const int rot = values ? p.v_rot : p.rot;
  if (table != nullptr && c < rot) turn8(f, table, rot, min(max(p.positions[t], 0), p.P - 1), c);
  if (!values && h < p.H) {
    store8(src, f);
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  const int g = values ? h : h - p.H;
  T* page = reinterpret_cast<T*>(p.cache) + ((long long)(slot / p.page) * p.G + g) * p.page * (p.DK + p.DV);
  store8(page + (values ? p.page * p.DK : 0) + (slot % p.page) * width + c, f);
}

// ------------------------------------------------------------------------------------------------
// fp32: one warp per (token, head).  Keys in chunks of 32, one per lane for the scores; the value product has the lanes side by side
// over the columns.
// ------------------------------------------------------------------------------------------------
constexpr int kGqaMaxWidth = 256, kGqaWarps = 4;

struct GqaF32Params {
  const float* q;
  long long ldq;
  const float* cache;
  float* out;
  long long ldo;
  StepRows rows;
  int T, H, G, DK, DV, page, window;
  float scale, softcap, out_scale;
  const float* sink;            // [H] or null
  const float* gate;            // [T, ldg] or null
  long long ldg;
  const float* turn;            // [turn_rows, turn_dims] or null
  int turn_dims, turn_rows;
};

__global__ void __launch_bounds__(32 * kGqaWarps) gqa_attn_f32_kernel(const GqaF32Params p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float qs[kGqaWarps][kGqaMaxWidth];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, h = blockIdx.y * kGqaWarps + warp;
  if (h >= p.H) return;
  int ctx;
  const int* bt;
  if (t < p.rows.nd) {
    ctx = p.rows.ctx_lens[t];
    bt = p.rows.dec_bt + (long long)t * p.rows.dec_max_blocks;
  } else {
    const int b = seq_of(p.rows, t - p.rows.nd);
    ctx = p.rows.cache_lens[b] + (t - p.rows.nd - p.rows.cu_q[b]) + 1;
    bt = p.rows.bt + (long long)b * p.rows.max_blocks;
  }
  for (int c = lane; c < p.DK; c += 32) qs[warp][c] = p.q[(long long)t * p.ldq + (long long)h * p.DK + c];
  __syncwarp();
  const int g = h / (p.H / p.G), lo = p.window > 0 ? max(ctx - p.window, 0) : 0;
  const long long page_elems = (long long)p.page * (p.DK + p.DV);
  float m = -INFINITY, l = 0.f, o[kGqaMaxWidth / 32];
#pragma unroll
  for (int i = 0; i < kGqaMaxWidth / 32; ++i) o[i] = 0.f;
  for (int k0 = lo; k0 < ctx; k0 += 32) {
    const int key = k0 + lane;
    const float* base = nullptr;
    float s = -INFINITY;
    if (key < ctx) {
      base = p.cache + ((long long)bt[key / p.page] * p.G + g) * page_elems;
      const float* kr = base + (key % p.page) * p.DK;
      float acc = 0.f;
      for (int c = 0; c < p.DK; c += 4) {
        const float4 a = load4(kr + c), b = load4(&qs[warp][c]);
        acc = fmaf(a.x, b.x, acc); acc = fmaf(a.y, b.y, acc); acc = fmaf(a.z, b.z, acc); acc = fmaf(a.w, b.w, acc);
      }
      s = acc * p.scale;
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      base += p.page * p.DK + (key % p.page) * p.DV;
    }
    const float mn = fmaxf(m, warp_max(s));
    const float corr = expf(m - mn), w = key < ctx ? expf(s - mn) : 0.f;
    m = mn;
    l = l * corr + warp_sum(w);
#pragma unroll
    for (int i = 0; i < kGqaMaxWidth / 32; ++i) o[i] *= corr;
    const int n = min(32, ctx - k0);
    for (int j = 0; j < n; ++j) {
      const float wj = __shfl_sync(0xffffffffu, w, j);
      const float* vr = reinterpret_cast<const float*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(base), j));
#pragma unroll
      for (int i = 0; i < kGqaMaxWidth / 32; ++i)
        if (i * 32 < p.DV) o[i] = fmaf(wj, vr[i * 32 + lane], o[i]);
    }
  }
  float inv = 0.f;
  if (l > 0.f) {
    const float sink = p.sink != nullptr ? p.sink[h] : -INFINITY, top = fmaxf(m, sink), keep = expf(m - top);
    inv = keep / (l * keep + expf(sink - top)) * p.out_scale;
  }
#pragma unroll
  for (int i = 0; i < kGqaMaxWidth / 32; ++i) {
    if (i * 32 >= p.DV) continue;
    const int col = h * p.DV + i * 32 + lane;
    float y = o[i] * inv;
    const float other = __shfl_xor_sync(0xffffffffu, y, 1);
    if (p.turn != nullptr && i * 32 + lane < p.turn_dims) {
      const float* cs = p.turn + (long long)min(max(ctx - 1, 0), p.turn_rows - 1) * p.turn_dims + ((i * 32 + lane) >> 1);
      const float c = cs[0], s = cs[p.turn_dims >> 1];
      y = lane & 1 ? y * c - other * s : y * c + other * s;
    }
    if (p.gate != nullptr) y *= sigmoid_f(p.gate[(long long)t * p.ldg + col]);
    p.out[(long long)t * p.ldo + col] = y;
  }
}

template <int DK, int DV>
static int gqa_decode(const DecodeParams& p, int T, cudaStream_t s) {
  constexpr int STAGES = DK + DV <= 128 ? 4 : 3;
  // four warps per CTA while the CTAs are few, two (more CTAs per SM) when they are many; wide heads have room for two only
  if constexpr (DK + DV <= 256) {
    if ((long long)T * p.nkv * p.gchunks * p.nsplit < 2 * 148) return launch_decode_nw<DK, DV, STAGES, false, 4, true>(p, T, s);
  }
  return launch_decode_nw<DK, DV, STAGES, false, 2, true>(p, T, s);
}

static bool gqa_width(int d) { return d == 64 || d == 128 || d == 256; }

}  // namespace lx

#define LX_GQA_DISPATCH(CALL)                                                                                              \
  switch (dk * 1024 + dv) {                                                                                                \
    case 64 * 1024 + 64: return CALL(64, 64);                                                                              \
    case 64 * 1024 + 128: return CALL(64, 128);                                                                            \
    case 64 * 1024 + 256: return CALL(64, 256);                                                                            \
    case 128 * 1024 + 64: return CALL(128, 64);                                                                            \
    case 128 * 1024 + 128: return CALL(128, 128);                                                                          \
    case 128 * 1024 + 256: return CALL(128, 256);                                                                          \
    case 256 * 1024 + 64: return CALL(256, 64);                                                                            \
    case 256 * 1024 + 128: return CALL(256, 128);                                                                          \
    case 256 * 1024 + 256: return CALL(256, 256);                                                                          \
    default: return -3;                                                                                                    \
  }

extern "C" {

int lx_gqa_page_size() { return lx::kPage; }
int lx_qk_norm_bytes() { return (int)sizeof(lx::QkNormParams); }
int lx_gqa_f32_bytes() { return (int)sizeof(lx::GqaF32Params); }

int lx_qk_norm_kvwrite(const void* params, int f32, void* stream) {
  using namespace lx;
  const QkNormParams& p = *reinterpret_cast<const QkNormParams*>(params);
  if (p.T <= 0) return 0;
  if (!gqa_width(p.DK) || !gqa_width(p.DV) || p.ld % 8 != 0) return -1;
  if ((p.cos_sin != nullptr || p.v_cos_sin != nullptr) && (p.positions == nullptr || p.P <= 0)) return -3;
  if ((p.cos_sin != nullptr && (p.rot % 2 != 0 || p.rot > p.DK)) || (p.v_cos_sin != nullptr && (p.v_rot % 2 != 0 || p.v_rot > p.DV))) return -4;
  const long long threads = (long long)p.T * ((p.H + p.G) * (p.DK / 8) > p.G * (p.DV / 8) ? (p.H + p.G) * (p.DK / 8) : p.G * (p.DV / 8));
  if (threads >= 1ll << 31) return -2;
  const dim3 grid((unsigned)((threads + 255) / 256), 2);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (f32) launch_pdl(qk_norm_kvwrite_kernel<float>, grid, dim3(256), 0, s, p);
  else launch_pdl(qk_norm_kvwrite_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, p);
  return -(int)cudaGetLastError();
}

// softcap > 0: scores become softcap * tanh(score / softcap).  sink [nh] (or null): a score that only the denominator contains.  The outputs'
// first turn_dims columns of a head are turned back by the token's row of turn [turn_rows, turn_dims] (or null); then they are multiplied
// by out_scale and by sigmoid(gate[t, column]) (gate [T, ldg] or null).
//
// Decode rows (bf16).  part_o / part_lse: T * nh * nsplit * dv and T * nh * nsplit floats, touched when nsplit > 1.
int lx_gqa_decode(const void* q, long long ldq, const void* cache, const int* block_tables, int max_blocks, const int* ctx_lens, void* out,
                  long long ldo, float* part_o, float* part_lse, int T, int nh, int nkv, int dk, int dv, int window, float scale, int nsplit,
                  float softcap, const float* sink, const void* gate, long long ldg, float out_scale, const float* turn, int turn_dims,
                  int turn_rows, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (nkv <= 0 || nh % nkv != 0 || ldq % 2 != 0 || turn_dims % 2 != 0 || turn_dims > dv) return -1;
  DecodeParams p{};
  p.q = reinterpret_cast<const __nv_bfloat16*>(q); p.ldq = ldq;
  p.kv = reinterpret_cast<const __nv_bfloat16*>(cache);
  p.block_tables = block_tables; p.max_blocks = max_blocks; p.ctx_lens = ctx_lens;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.part_o = part_o; p.part_lse = part_lse;
  p.nh = nh; p.nkv = nkv; p.group = nh / nkv; p.gchunks = (p.group + 15) / 16;
  p.window = window; p.scale = scale; p.softcap = softcap; p.v_scale = 1.f;
  p.tail = AttnTail{sink, reinterpret_cast<const __nv_bfloat16*>(gate), ldg, out_scale, turn, turn_dims, turn_rows};
  p.nsplit = nsplit < 1 ? 1 : nsplit;
  if (p.nsplit > 1 && (part_o == nullptr || part_lse == nullptr)) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define LX_CALL(DK, DV) gqa_decode<DK, DV>(p, T, s)
  LX_GQA_DISPATCH(LX_CALL)
#undef LX_CALL
}

// Prompt rows (bf16): 64-query tiles listed by tile_seq / tile_q0.
int lx_gqa_prefill(const void* q, long long ldq, const void* cache, const int* block_tables, int max_blocks, const int* cu_q,
                   const int* cache_lens, const int* tile_seq, const int* tile_q0, int num_tiles, void* out, long long ldo, int nh, int nkv,
                   int dk, int dv, int window, float scale, float softcap, const float* sink, const void* gate, long long ldg, float out_scale,
                   const float* turn, int turn_dims, int turn_rows, void* stream) {
  using namespace lx;
  if (num_tiles <= 0) return 0;
  if (nkv <= 0 || nh % nkv != 0 || ldq % 2 != 0 || ldo % 2 != 0 || turn_dims % 2 != 0 || turn_dims > dv) return -1;
  PrefillParams p{};
  p.q = reinterpret_cast<const __nv_bfloat16*>(q); p.ldq = ldq;
  p.kv = reinterpret_cast<const __nv_bfloat16*>(cache);
  p.block_tables = block_tables; p.max_blocks = max_blocks; p.cu_q = cu_q; p.cache_lens = cache_lens;
  p.tile_seq = tile_seq; p.tile_q0 = tile_q0;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.nh = nh; p.nkv = nkv; p.window = window; p.scale = scale; p.softcap = softcap; p.v_scale = 1.f;
  p.tail = AttnTail{sink, reinterpret_cast<const __nv_bfloat16*>(gate), ldg, out_scale, turn, turn_dims, turn_rows};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define LX_CALL(DK, DV) launch_prefill<DK, DV, false, true>(p, num_tiles, s)
  LX_GQA_DISPATCH(LX_CALL)
#undef LX_CALL
}

int lx_gqa_attn_f32(const void* params, void* stream) {
  using namespace lx;
  const GqaF32Params& p = *reinterpret_cast<const GqaF32Params*>(params);
  if (p.T <= 0) return 0;
  if (!gqa_width(p.DK) || !gqa_width(p.DV) || p.G <= 0 || p.H % p.G != 0 || p.turn_dims % 2 != 0 || p.turn_dims > p.DV) return -1;
  launch_pdl(gqa_attn_f32_kernel, dim3(p.T, (p.H + kGqaWarps - 1) / kGqaWarps), dim3(32 * kGqaWarps), 0, reinterpret_cast<cudaStream_t>(stream), p);
  return -(int)cudaGetLastError();
}

}  // extern "C"
