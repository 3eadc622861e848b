// Short causal convolutions over a step's rows, one weight per channel and tap, and what follows them:
//
//   causal_conv         y_t = act(sum_j w_j u_(t - taps + 1 + j) + b)                                (state space mixers)
//   conv_rope_kvwrite   rows [q | k | v]: the convolution when there is one, q and k rotated in interleaved pairs, q to a buffer, k and
//                       v to the paged cache                                                       (attention)
//
// The last taps - 1 rows of a request are its state, [slots, taps - 1, C].  A thread owns eight channels of a decode row, or of a run of
// kCvRun consecutive prompt tokens whose window it slides through registers.  Whoever owns the first tokens of a sequence also reads its
// old state and leaves the new one, so nothing has to wait for another thread: all other runs start at least taps - 1 tokens later and
// see rows of the step only.
#include "stream.cuh"

namespace lx {

constexpr int kCvRun = 8, kCvMaxTaps = kCvRun + 1;
constexpr int kCvThreads = 256, kCvVecs = 32;      // 32 vectors of eight channels x 8 runs (or decode rows)
constexpr int kCvTile = 64;                        // prompt tokens per CTA

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

// Eight finished channels c .. c + 7 of row t (u: their values).
template <typename T, bool ATTN>
LX_DEVICE void cv_emit(const ConvParams& p, int t, int c, float (&u)[8]) {
  if constexpr (!ATTN) {
    if (p.silu) {
#pragma unroll
      for (int q = 0; q < 8; ++q) u[q] = silu_f(u[q]);
    }
    store8(reinterpret_cast<T*>(p.out) + (long long)t * p.ldo + c, u);
    return;
  }
  const int qk = (p.H + p.G) * p.DK;
  if (c < qk) {
    const int d = c % p.DK;
    if (d < p.rot) {
      const float* cs = p.cos_sin + (long long)min(p.positions[t], p.P - 1) * p.rot;
#pragma unroll
      for (int q = 0; q < 8; q += 2) {
        if (d + q < p.rot) {
          const float co = cs[(d + q) >> 1], si = cs[(p.rot + d + q) >> 1];
          const float a = u[q], b = u[q + 1];
          u[q] = a * co - b * si;
          u[q + 1] = b * co + a * si;
        }
      }
    }
    if (c < p.H * p.DK) {
      store8(reinterpret_cast<T*>(p.out) + (long long)t * p.ldo + c, u);
      return;
    }
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  const bool value = c >= qk;
  const int width = value ? p.DV : p.DK, at = value ? c - qk : c - p.H * p.DK;
  T* page = reinterpret_cast<T*>(p.cache) + ((long long)(slot / p.page) * p.G + at / width) * p.page * (p.DK + p.DV);
  store8(page + (value ? p.page * p.DK : 0) + (slot % p.page) * width + at % width, u);
}

// TAPS 1 .. 4: the window in registers; 0: any number up to kCvMaxTaps, rows read again per tap; -1: no convolution.
template <typename T, bool ATTN, int TAPS>
__global__ void __launch_bounds__(kCvThreads) conv_kernel(const ConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.y * kCvVecs + (threadIdx.x & (kCvVecs - 1))) * 8, run = threadIdx.x / kCvVecs;
  if (c >= p.C) return;
  int t0, n, keep_n = 0;                           // first row, rows; rows of the sequence (for its owner)
  const T* old = nullptr;                          // the sequence's state, when these are its first rows and it has one
  T* state = nullptr;                              // where its owner leaves the new one
  int lead = 0;                                    // rows of the step in front of t0 that belong to the sequence
  const int keep = TAPS < 0 ? 0 : (TAPS > 0 ? TAPS : p.taps) - 1;
  if ((int)blockIdx.x < p.dec_ctas) {
    t0 = blockIdx.x * (kCvThreads / kCvVecs) + run;
    if (t0 >= p.rows.nd) return;
    n = 1;
    const int ctx = p.rows.ctx_lens[t0];
    if (ctx <= 0) return;
    if (keep > 0) {
      state = reinterpret_cast<T*>(p.state) + (long long)p.rows.dec_slots[t0] * keep * p.C + c;
      keep_n = 1;
      if (ctx > 1) old = state;
    }
  } else {
    const int tile = blockIdx.x - p.dec_ctas, b = p.tile_seq[tile], q0 = p.tile_q0[tile] + run * kCvRun;
    const int r0 = p.rows.cu_q[b], qlen = p.rows.cu_q[b + 1] - r0;
    if (q0 >= qlen) return;
    t0 = p.rows.nd + r0 + q0;
    n = min(kCvRun, qlen - q0);
    lead = q0;
    if (keep > 0 && q0 == 0) {
      state = reinterpret_cast<T*>(p.state) + (long long)p.rows.slots[b] * keep * p.C + c;
      keep_n = qlen;
      if (p.rows.cache_lens[b] > 0) old = state;
    }
  }
  const T* x = reinterpret_cast<const T*>(p.x) + (long long)t0 * p.ldx + c;
  // row i of the run's input: a row of the step, of the state, or zeros
  auto fetch = [&](int i, float (&f)[8]) {
    if (i >= 0 || lead > 0) load8(x + (long long)i * p.ldx, f);
    else if (old != nullptr) load8(old + (long long)(keep + i) * p.C, f);
    else {
#pragma unroll
      for (int q = 0; q < 8; ++q) f[q] = 0.f;
    }
  };
  float bias[8];
#pragma unroll
  for (int q = 0; q < 8; ++q) bias[q] = 0.f;
  if (TAPS >= 0 && p.b != nullptr) load8(p.b + c, bias);
  if constexpr (TAPS > 0) {
    float w[TAPS][8], win[TAPS][8];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load8(p.w + (long long)j * p.C + c, w[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) fetch(j - (TAPS - 1), win[j + 1]);
#pragma unroll
    for (int i = 0; i < kCvRun; ++i) {
      if (i < n) {
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
          for (int q = 0; q < 8; ++q) win[j][q] = win[j + 1][q];
        load8(x + (long long)i * p.ldx, win[TAPS - 1]);
        float y[8];
#pragma unroll
        for (int q = 0; q < 8; ++q) y[q] = bias[q];
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
          for (int q = 0; q < 8; ++q) y[q] = fmaf(w[j][q], win[j][q], y[q]);
        cv_emit<T, ATTN>(p, t0 + i, c, y);
      }
    }
  } else {
    for (int i = 0; i < n; ++i) {
      float y[8];
#pragma unroll
      for (int q = 0; q < 8; ++q) y[q] = bias[q];
      if constexpr (TAPS == 0) {
        for (int j = 0; j <= keep; ++j) {
          float w[8], u[8];
          load8(p.w + (long long)j * p.C + c, w);
          fetch(i - keep + j, u);
#pragma unroll
          for (int q = 0; q < 8; ++q) y[q] = fmaf(w[q], u[q], y[q]);
        }
      } else {
        load8(x + (long long)i * p.ldx, y);
      }
      cv_emit<T, ATTN>(p, t0 + i, c, y);
    }
  }
  if (TAPS >= 0 && state != nullptr) {
    // rows keep_n - keep .. keep_n - 1 of the sequence; negative ones are in the old state, behind the places written before them
    for (int j = 0; j < keep; ++j) {
      float f[8];
      fetch(keep_n - keep + j, f);
      store8(state + (long long)j * p.C, f);
    }
  }
}

template <typename T, bool ATTN>
static int conv_launch(const ConvParams& p, int tiles, cudaStream_t s) {
  const dim3 grid(p.dec_ctas + tiles, (p.C / 8 + kCvVecs - 1) / kCvVecs), block(kCvThreads);
  switch (p.taps) {
    case 0:
      if constexpr (ATTN) launch_pdl(conv_kernel<T, ATTN, -1>, grid, block, 0, s, p);
      else return -4;
      break;
    case 1: launch_pdl(conv_kernel<T, ATTN, 1>, grid, block, 0, s, p); break;
    case 2: launch_pdl(conv_kernel<T, ATTN, 2>, grid, block, 0, s, p); break;
    case 3: launch_pdl(conv_kernel<T, ATTN, 3>, grid, block, 0, s, p); break;
    case 4: launch_pdl(conv_kernel<T, ATTN, 4>, grid, block, 0, s, p); break;
    default: launch_pdl(conv_kernel<T, ATTN, 0>, grid, block, 0, s, p); break;
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
  p.dec_ctas = (p.rows.nd + kCvThreads / kCvVecs - 1) / (kCvThreads / kCvVecs);
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
