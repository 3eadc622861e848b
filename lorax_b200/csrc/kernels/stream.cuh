// Element access shared by the kernels of the layer-by-layer designs, which exist for bf16 and for fp32 activations.
#pragma once

#include "common.cuh"

namespace lx {

// Eight consecutive elements (16-byte aligned rows for bf16, 32 for fp32) as fp32, and back.
LX_DEVICE void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    const float2 t = unpack_bf16x2(w[q]);
    f[2 * q] = t.x;
    f[2 * q + 1] = t.y;
  }
}
LX_DEVICE void load8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
LX_DEVICE void store8(__nv_bfloat16* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) =
      make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
}
LX_DEVICE void store8(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}
LX_DEVICE float4 load4(const __nv_bfloat16* p) {
  const uint2 a = *reinterpret_cast<const uint2*>(p);
  const float2 x = unpack_bf16x2(a.x), y = unpack_bf16x2(a.y);
  return make_float4(x.x, x.y, y.x, y.y);
}
LX_DEVICE float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
LX_DEVICE void store4(__nv_bfloat16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w)); }
LX_DEVICE void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
LX_DEVICE float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
LX_DEVICE float to_f(float v) { return v; }
LX_DEVICE void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
LX_DEVICE void put(float* p, float v) { *p = v; }

LX_DEVICE float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
LX_DEVICE float silu_f(float z) { return z / (1.f + expf(-z)); }
LX_DEVICE float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// Sum over the block, the same value in every thread; `red` holds one float per warp.
LX_DEVICE float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) s += red[i];
  return s;
}

// Rows of a step: [0, nd) are decode rows (one token each), the rows after them ragged prompt tokens.
struct StepRows {
  int nd;                      // decode rows
  const int* dec_slots;        // [nd] state slot
  const int* ctx_lens;         // [nd] tokens of the request including this one; <= 0: padding
  const int* dec_bt;           // [nd, max_blocks]
  int B;                       // prefill sequences
  const int* cu_q;             // [B + 1] relative to row nd
  const int* cache_lens;       // [B] tokens before the step
  const int* slots;            // [B] state slot
  const int* bt;               // [B, max_blocks]
  int max_blocks, dec_max_blocks;
};

// Sequence of prefill token t (row nd + t).
LX_DEVICE int seq_of(const StepRows& s, int t) {
  int lo = 0, hi = s.B;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (s.cu_q[mid] <= t) lo = mid; else hi = mid;
  }
  return lo;
}

}  // namespace lx
