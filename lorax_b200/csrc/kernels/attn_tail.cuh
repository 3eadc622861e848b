// What the attention kernels share around the softmax: capped scores, sinks, and the last step of an output element.
#pragma once

#include "common.cuh"

namespace lx {

// cap * tanh(s / cap) by tanh(x) = 1 - 2 / (exp(2x) + 1); k = 2 log2(e) / cap.  The absolute error is a few 2^-24 of the cap.
LX_DEVICE float softcap_score(float s, float cap, float k) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(s * k));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.f));
  return fmaf(-2.f * cap, r, cap);
}

// What may follow the softmax: a sink per head, a score that only the denominator contains; the first turn_dims columns of a head turned
// back by the token's position (pairs of neighbours); a factor; a gate, sigmoid(gate[t, column]).
struct AttnTail {
  const float* sink = nullptr;            // [nh]
  const __nv_bfloat16* gate = nullptr;    // [T, ldg]
  long long ldg = 0;
  float scale = 1.f;                      // of the output
  const float* turn = nullptr;            // [turn_rows, turn_dims] cos, then sin of every position's angles
  int turn_dims = 0, turn_rows = 0;
};

// 1 / denominator of a row whose weights were formed with the maximum m and sum to l > 0 (both in the log2 domain): the sink joins, and
// the maximum moves up to it when it is the larger one.
LX_DEVICE float attn_denominator(const AttnTail& tail, int head, float m, float l) {
  if (tail.sink == nullptr) return 1.f / l;
  const float sink = tail.sink[head] * 1.4426950408889634f, top = fmaxf(m, sink), keep = exp2f(m - top);
  return keep / (l * keep + exp2f(sink - top));
}

// Columns d (even) and d + 1 of a head, turned back by the angles of position pos.
LX_DEVICE float2 attn_turn_back(const AttnTail& tail, float2 o, int d, int pos) {
  if (tail.turn == nullptr || d >= tail.turn_dims) return o;
  const float* cs = tail.turn + (long long)min(pos, tail.turn_rows - 1) * tail.turn_dims + (d >> 1);
  const float c = __ldg(cs), s = __ldg(cs + (tail.turn_dims >> 1));
  return make_float2(o.x * c + o.y * s, o.y * c - o.x * s);
}

// The same for columns [d, d + 8), d a multiple of eight.
LX_DEVICE void attn_turn_back8(const AttnTail& tail, float (&v)[8], int d, int pos) {
  if (tail.turn_dims % 8 == 0) {
    if (d >= tail.turn_dims) return;
    const float* cs = tail.turn + (long long)min(pos, tail.turn_rows - 1) * tail.turn_dims + (d >> 1);
    const float4 c = __ldg(reinterpret_cast<const float4*>(cs)), s = __ldg(reinterpret_cast<const float4*>(cs + (tail.turn_dims >> 1)));
    const float co[4] = {c.x, c.y, c.z, c.w}, si[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float a = v[2 * u], b = v[2 * u + 1];
      v[2 * u] = a * co[u] + b * si[u];
      v[2 * u + 1] = b * co[u] - a * si[u];
    }
    return;
  }
#pragma unroll
  for (int u = 0; u < 8; u += 2) {
    const float2 o = attn_turn_back(tail, make_float2(v[u], v[u + 1]), d + u, pos);
    v[u] = o.x;
    v[u + 1] = o.y;
  }
}

// One finished output element.
LX_DEVICE float attn_tail(const AttnTail& tail, float o, long long t, int col) {
  o *= tail.scale;
  if (tail.gate != nullptr) o = __fdividef(o, 1.f + __expf(-__bfloat162float(tail.gate[t * tail.ldg + col])));
  return o;
}

}  // namespace lx
