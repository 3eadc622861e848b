// Short causal convolutions over a step's rows, one weight per channel and tap, and what follows them:
//
//   causal_conv         y_t = act(sum_j w_j u_(t - taps + 1 + j) + b)                                (state space mixers)
//   conv_rope_kvwrite   rows [q | k | v]: the convolution when there is one, q and k rotated in interleaved pairs, q to a buffer, k and
//                       v to the paged cache                                                       (attention)
//
// The last taps - 1 rows of a request are its state, [slots, taps - 1, C].  Prompts: a CTA stages 64 tokens x 128 channels and the taps - 1
// rows in front of them (rows of the step, of the state, or zeros) in shared memory; a thread owns eight channels of eight tokens.  The
// CTA of a sequence's first tokens is the only one that reads its old state, and leaves the new one.  Decode rows: a thread owns eight
// channels of a row and of its state.
#include "stream.cuh"

namespace lx {

constexpr int kCvMaxTaps = 9;
constexpr int kCvTile = 64, kCvCols = 128, kCvRun = 8;               // prompt tokens and channels of a CTA, tokens of a thread
constexpr int kCvVecs = kCvCols / 8, kCvRows = 8;                    // threads across the channels; decode rows (or runs) of a CTA
constexpr int kCvThreads = kCvVecs * kCvRows;

struct ConvParams {
  const void* x;               // [T, ldx], channel c of the convolution at column c
  long long ldx;
  void* out;                   // [T, ldo]: all channels, or the q heads
  long long ldo;
  const float* w;              // [taps, C]
  const float* b;              // [C] or null
  void* state;                 // [slots, taps - 1, C]
  StepRows rows;
  const int* tile_seq;         // prompt tiles of kCvTile tokens
  const int* tile_q0;
  int C, taps, silu, dec_ctas;
  // attention
  void* cache;
  const int* slots;            // [T] token slot in the cache, < 0: none
  const int* positions;
  const float* cos_sin;        // [P, rot]
  int P, rot, H, G, DK, DV, page;
};

template <typename T>
LX_DEVICE float cv_silu(float z) {
  return sizeof(T) == 2 ? __fdividef(z, 1.f + __expf(-z)) : silu_f(z);
}

// Where eight finished channels go; what depends on the channel only is worked out once per thread.
template <typename T, bool ATTN>
struct CvSink {
  const ConvParams& p;
  int c, rot_at;               // channel; its column within the head when it is rotated (-1: not)
  bool to_out;
  long long plane;             // k, v: offset of the head's plane within a block
  int width, at;
  LX_DEVICE CvSink(const ConvParams& p, int c) : p(p), c(c), rot_at(-1), to_out(true), plane(0), width(0), at(0) {
    if (!ATTN) return;
    const int qk = (p.H + p.G) * p.DK, d = c % p.DK;
    if (c < qk && d < p.rot) rot_at = d;
    if (c < p.H * p.DK) return;
    to_out = false;
    const bool value = c >= qk;
    width = value ? p.DV : p.DK;
    const int in = value ? c - qk : c - p.H * p.DK;
    at = in % width;
    plane = (long long)(in / width) * p.page * (p.DK + p.DV) + (value ? p.page * p.DK : 0);
  }
  LX_DEVICE void operator()(int t, int pos, int slot, float (&u)[8]) const {
    if constexpr (!ATTN) {
      if (p.silu) {
#pragma unroll
        for (int q = 0; q < 8; ++q) u[q] = cv_silu<T>(u[q]);
      }
    } else {
      if (rot_at >= 0) {
        const float* cs = p.cos_sin + (long long)min(pos, p.P - 1) * p.rot + (rot_at >> 1);
        float co[4], si[4];
        if (p.rot % 8 == 0) {
          const float4 a = __ldg(reinterpret_cast<const float4*>(cs)), b = __ldg(reinterpret_cast<const float4*>(cs + (p.rot >> 1)));
          co[0] = a.x; co[1] = a.y; co[2] = a.z; co[3] = a.w;
          si[0] = b.x; si[1] = b.y; si[2] = b.z; si[3] = b.w;
        } else {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const bool on = rot_at + 2 * q < p.rot;
            co[q] = on ? __ldg(cs + q) : 1.f;
            si[q] = on ? __ldg(cs + (p.rot >> 1) + q) : 0.f;
          }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float a = u[2 * q], b = u[2 * q + 1];
          u[2 * q] = a * co[q] - b * si[q];
          u[2 * q + 1] = b * co[q] + a * si[q];
        }
      }
      if (!to_out) {
        if (slot < 0) return;
        const unsigned block = (unsigned)slot / (unsigned)p.page, off = slot - block * p.page;
        store8(reinterpret_cast<T*>(p.cache) + (long long)block * p.G * p.page * (p.DK + p.DV) + plane + off * width + at, u);
        return;
      }
    }
    store8(reinterpret_cast<T*>(p.out) + (long long)t * p.ldo + c, u);
  }
};

// TAPS 1 .. 4: the weights in registers; 0: any number up to kCvMaxTaps; -1: no convolution.
template <typename T, bool ATTN, int TAPS>
__global__ void __launch_bounds__(kCvThreads) conv_kernel(const ConvParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t cv_raw[];
  const int c0 = blockIdx.y * kCvCols, vec = threadIdx.x % kCvVecs, run = threadIdx.x / kCvVecs, c = c0 + vec * 8;
  const int keep = TAPS < 0 ? 0 : (TAPS > 0 ? TAPS : p.taps) - 1;
  const bool live = c < p.C;
  const T* x = reinterpret_cast<const T*>(p.x);
  T* state = reinterpret_cast<T*>(p.state);
  float w[TAPS > 0 ? TAPS : 1][8], bias[8];
#pragma unroll
  for (int q = 0; q < 8; ++q) bias[q] = 0.f;
  if (TAPS >= 0 && live && p.b != nullptr) load8(p.b + c, bias);
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
    if (live) load8(p.w + (long long)j * p.C + c, w[j]);
  const CvSink<T, ATTN> sink(p, min(c, p.C - 8));
  // taps j of y += w[j] * u
  auto tap = [&](float (&y)[8], int j, const float (&u)[8]) {
    float own[8];
    if constexpr (TAPS == 0) load8(p.w + (long long)j * p.C + c, own);
#pragma unroll
    for (int q = 0; q < 8; ++q) y[q] = fmaf(TAPS > 0 ? w[TAPS > 0 ? j : 0][q] : own[q], u[q], y[q]);
  };

  if ((int)blockIdx.x < p.dec_ctas) {
    const int t = blockIdx.x * kCvRows + run;
    if (t >= p.rows.nd || !live) return;
    const int ctx = p.rows.ctx_lens[t];
    if (ctx <= 0) return;
    float y[8], u[8];
    load8(x + (long long)t * p.ldx + c, u);
    if constexpr (TAPS < 0) {
#pragma unroll
      for (int q = 0; q < 8; ++q) y[q] = u[q];
    } else {
      T* mine = state + (long long)p.rows.dec_slots[t] * keep * p.C + c;
#pragma unroll
      for (int q = 0; q < 8; ++q) y[q] = bias[q];
      if constexpr (TAPS > 0) {
        float old[TAPS][8];
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) {
#pragma unroll
          for (int q = 0; q < 8; ++q) old[j][q] = 0.f;
          if (ctx > 1) load8(mine + (long long)j * p.C, old[j]);
        }
#pragma unroll
        for (int q = 0; q < 8; ++q) old[TAPS - 1][q] = u[q];
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) store8(mine + (long long)j * p.C, old[j + 1]);
#pragma unroll
        for (int j = 0; j < TAPS; ++j) tap(y, j, old[j]);
      } else {
        for (int j = 0; j < keep; ++j) {
          float old[8];
#pragma unroll
          for (int q = 0; q < 8; ++q) old[q] = 0.f;
          if (ctx > 1) load8(mine + (long long)j * p.C, old);
          tap(y, j, old);
          if (j > 0) store8(mine + (long long)(j - 1) * p.C, old);
        }
        if (keep > 0) store8(mine + (long long)(keep - 1) * p.C, u);
        tap(y, keep, u);
      }
    }
    sink(t, ATTN && sink.rot_at >= 0 ? p.positions[t] : 0, ATTN && !sink.to_out ? p.slots[t] : 0, y);
    return;
  }

  T* tile = reinterpret_cast<T*>(cv_raw);                              // [keep + kCvTile][kCvCols]
  __shared__ int slot_s[kCvTile];
  const int b = p.tile_seq[blockIdx.x - p.dec_ctas], q0 = p.tile_q0[blockIdx.x - p.dec_ctas];
  const int r0 = p.rows.cu_q[b], qlen = p.rows.cu_q[b + 1] - r0, before = p.rows.cache_lens[b];
  const int n = min(kCvTile, qlen - q0), first = p.rows.nd + r0;       // row of the sequence's first token
  T* kept = keep > 0 ? state + (long long)p.rows.slots[b] * keep * p.C : nullptr;
  constexpr int PER = 16 / sizeof(T), CH = kCvCols / PER;              // 16-byte pieces
  for (int e = threadIdx.x; e < (keep + n) * CH; e += kCvThreads) {
    const int r = e / CH, col = (e % CH) * PER, q = q0 + r - keep;     // token of the sequence
    const bool old = q < 0;
    const bool ok = c0 + col < p.C && (!old || before > 0);
    const T* src = old ? kept + (long long)(keep + q) * p.C + c0 + col : x + (long long)(first + q) * p.ldx + c0 + col;
    cp_async_16(tile + r * kCvCols + col, ok ? src : x, ok);
  }
  cp_async_commit();
  if (ATTN && (int)threadIdx.x < n) slot_s[threadIdx.x] = p.slots[first + q0 + threadIdx.x];
  cp_async_wait<0>();
  __syncthreads();
  if (!live) return;
  const T* mine = tile + vec * 8;
  if (keep > 0 && q0 == 0 && run == 0) {
    // the sequence's last rows; those in front of its first token of this step stand in the tile
    for (int j = 0; j < keep; ++j) {
      const int q = qlen - keep + j;
      float f[8];
      if (q < n) load8(mine + (keep + q) * kCvCols, f); else load8(x + (long long)(first + q) * p.ldx + c, f);
      store8(kept + (long long)j * p.C + c, f);
    }
  }
  const int i0 = run * kCvRun;
  if (i0 >= n) return;
  if constexpr (TAPS > 0) {
    float win[TAPS][8];
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) load8(mine + (i0 + j) * kCvCols, win[j]);
#pragma unroll
    for (int i = 0; i < kCvRun; ++i) {
      if (i0 + i < n) {
        load8(mine + (i0 + i + TAPS - 1) * kCvCols, win[(i + TAPS - 1) % TAPS]);
        float y[8];
#pragma unroll
        for (int q = 0; q < 8; ++q) y[q] = bias[q];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) tap(y, j, win[(i + j) % TAPS]);
        sink(first + q0 + i0 + i, before + q0 + i0 + i, ATTN ? slot_s[i0 + i] : 0, y);
      }
    }
  } else {
    for (int i = i0; i < min(i0 + kCvRun, n); ++i) {
      float y[8];
      if constexpr (TAPS < 0) {
        load8(mine + i * kCvCols, y);
      } else {
#pragma unroll
        for (int q = 0; q < 8; ++q) y[q] = bias[q];
        for (int j = 0; j <= keep; ++j) {
          float u[8];
          load8(mine + (i + j) * kCvCols, u);
          tap(y, j, u);
        }
      }
      sink(first + q0 + i, before + q0 + i, ATTN ? slot_s[i] : 0, y);
    }
  }
}

template <typename T, bool ATTN>
static int conv_launch(const ConvParams& p, int tiles, cudaStream_t s) {
  const dim3 grid(p.dec_ctas + tiles, (p.C + kCvCols - 1) / kCvCols), block(kCvThreads);
  const size_t smem = tiles > 0 ? (size_t)((p.taps > 0 ? p.taps - 1 : 0) + kCvTile) * kCvCols * sizeof(T) : 0;      // (at most 36 KB)
  switch (p.taps) {
    case 0:
      if constexpr (ATTN) launch_pdl(conv_kernel<T, ATTN, -1>, grid, block, smem, s, p);
      else return -4;
      break;
    case 1: launch_pdl(conv_kernel<T, ATTN, 1>, grid, block, smem, s, p); break;
    case 2: launch_pdl(conv_kernel<T, ATTN, 2>, grid, block, smem, s, p); break;
    case 3: launch_pdl(conv_kernel<T, ATTN, 3>, grid, block, smem, s, p); break;
    case 4: launch_pdl(conv_kernel<T, ATTN, 4>, grid, block, smem, s, p); break;
    default: launch_pdl(conv_kernel<T, ATTN, 0>, grid, block, smem, s, p); break;
  }
  return -(int)cudaGetLastError();
}

}  // namespace lx

extern "C" {

int lx_conv_bytes() { return (int)sizeof(lx::ConvParams); }

// attn 0: causal_conv, 1: conv_rope_kvwrite (taps 0: no convolution; `out` may then be `x` itself).  tiles: prompt tiles of 64 tokens.
int lx_conv(const void* params, int tiles, int attn, int f32, void* stream) {
  using namespace lx;
  ConvParams p = *reinterpret_cast<const ConvParams*>(params);
  p.dec_ctas = (p.rows.nd + kCvRows - 1) / kCvRows;
  if (p.dec_ctas + tiles <= 0 || p.C <= 0) return 0;
  if (p.C % 8 != 0 || p.ldx % 8 != 0 || p.ldo % 8 != 0 || p.taps < 0 || p.taps > kCvMaxTaps) return -1;
  if (p.taps > 1 && p.state == nullptr) return -2;
  if (attn && (p.DK % 8 != 0 || p.DV % 8 != 0 || p.rot % 2 != 0 || p.rot > p.DK || p.page <= 0 || (p.rot > 0 && (p.cos_sin == nullptr || p.P <= 0)) ||
               p.C != (p.H + p.G) * p.DK + p.G * p.DV))
    return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (f32) return attn ? conv_launch<float, true>(p, tiles, s) : conv_launch<float, false>(p, tiles, s);
  return attn ? conv_launch<__nv_bfloat16, true>(p, tiles, s) : conv_launch<__nv_bfloat16, false>(p, tiles, s);
}

}  // extern "C"
