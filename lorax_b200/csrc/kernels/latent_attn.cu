// Latent attention: per token one latent vector and one rotated key part, shared by all heads, live in the paged cache
// [blocks, page, R] with R = kv rank + rotated width.  A head's query is carried into the latent space (q_lat = W_uk^T q) so that
// scores and the weighted sum run on the cached rows themselves; W_uv is applied to the result.
#include "stream.cuh"

namespace lx {

// ------------------------------------------------------------------------------------------------
// Preparation of a token: RMS norm of the query down-projection (-> cq) or, without one, interleaved rotation of the queries in place; RMS
// norm of the key/value latent and interleaved rotation of the shared key part (-> cache row).  One CTA per token.
// ------------------------------------------------------------------------------------------------
struct LatentPrepParams {
  const void* dq; const void* dkv;      // [T, ld] rows of the fused projection; dq null (QR 0): no query latent
  long long ld_dq, ld_dkv;
  const float* dq_norm;                 // [QR] padded with zeros
  const float* dkv_norm;                // [KR]
  void* cq;                             // [T, QR]
  void* cache;                          // [blocks * page, R]
  const int* positions; const int* slots;
  const float* cos_sin;                 // [max_pos, rot]
  int QR, KR, R, q_rank, kv_rank, rot;
  float eps;
  void* q;                              // [T, ldq] or null: columns [off, off + rot) of every head are rotated
  long long ldq;
  int H, head, off;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[4];
  const int t = blockIdx.x;
  const T* dq = reinterpret_cast<const T*>(p.dq) + (long long)t * p.ld_dq;
  const T* dkv = reinterpret_cast<const T*>(p.dkv) + (long long)t * p.ld_dkv;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * 8; c < p.QR; c += blockDim.x * 8) {
    float f[8];
    load8(dq + c, f);
#pragma unroll
    for (int q = 0; q < 8; ++q) sq += f[q] * f[q];
  }
  for (int c = threadIdx.x * 8; c < p.KR; c += blockDim.x * 8) {
    float f[8];
    load8(dkv + c, f);
#pragma unroll
    for (int q = 0; q < 8; ++q) sk += f[q] * f[q];
  }
  const float* cs = p.cos_sin + (long long)p.positions[t] * p.rot;
  const int half = p.rot / 2;
  if (p.q != nullptr) {
    T* x = reinterpret_cast<T*>(p.q) + (long long)t * p.ldq + p.off;
    if (p.rot % 8 == 0) {
      const int per = p.rot / 8;
      for (int e = threadIdx.x; e < p.H * per; e += blockDim.x) {
        const int h = e / per, i = (e - h * per) * 4;
        const float4 c = __ldg(reinterpret_cast<const float4*>(cs + i)), s = __ldg(reinterpret_cast<const float4*>(cs + half + i));
        T* at = x + (long long)h * p.head + 2 * i;
        float f[8];
        load8(at, f);
        const float g[8] = {f[0] * c.x - f[1] * s.x, f[1] * c.x + f[0] * s.x, f[2] * c.y - f[3] * s.y, f[3] * c.y + f[2] * s.y,
                            f[4] * c.z - f[5] * s.z, f[5] * c.z + f[4] * s.z, f[6] * c.w - f[7] * s.w, f[7] * c.w + f[6] * s.w};
        store8(at, g);
      }
    } else {
      for (int e = threadIdx.x; e < p.H * half; e += blockDim.x) {
        const int h = e / half, i = e - h * half;
        T* at = x + (long long)h * p.head + 2 * i;
        const float u = to_f(at[0]), v = to_f(at[1]), c = cs[i], s = cs[half + i];
        put(at, u * c - v * s);
        put(at + 1, v * c + u * s);
      }
    }
  }
  const float rq = p.QR > 0 ? rsqrtf(block_sum(sq, red) / p.q_rank + p.eps) : 0.f;
  const float rk = rsqrtf(block_sum(sk, red) / p.kv_rank + p.eps);
  T* cq = reinterpret_cast<T*>(p.cq) + (long long)t * p.QR;
  for (int c = threadIdx.x * 8; c < p.QR; c += blockDim.x * 8) {
    float f[8], w[8];
    load8(dq + c, f);
    load8(p.dq_norm + c, w);
#pragma unroll
    for (int q = 0; q < 8; ++q) f[q] *= rq * w[q];
    store8(cq + c, f);
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  T* row = reinterpret_cast<T*>(p.cache) + (long long)slot * p.R;
  for (int c = threadIdx.x * 8; c < p.KR; c += blockDim.x * 8) {
    float f[8], w[8];
    load8(dkv + c, f);
    load8(p.dkv_norm + c, w);
#pragma unroll
    for (int q = 0; q < 8; ++q) f[q] *= rk * w[q];
    store8(row + c, f);
  }
  for (int i = threadIdx.x; i < (p.R - p.KR) / 2; i += blockDim.x) {
    float a = 0.f, b = 0.f;
    if (i < half) {
      const float u = to_f(dkv[p.KR + 2 * i]), v = to_f(dkv[p.KR + 2 * i + 1]);
      const float c = cs[i], s = cs[half + i];
      a = u * c - v * s;
      b = v * c + u * s;
    }
    put(row + p.KR + 2 * i, a);
    put(row + p.KR + 2 * i + 1, b);
  }
}

// Interleaved rotation of columns [off, off + rot) of every head of x [T, H * head], in place.
template <typename T>
__global__ void __launch_bounds__(256) rope_pairs_kernel(T* __restrict__ x, long long ldx, const int* __restrict__ positions,
                                                         const float* __restrict__ cos_sin, int H, int head, int off, int rot) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, half = rot / 2;
  const float* cs = cos_sin + (long long)positions[t] * rot;
  for (int e = threadIdx.x; e < H * half; e += blockDim.x) {
    const int h = e / half, i = e % half;
    T* q = x + (long long)t * ldx + (long long)h * head + off + 2 * i;
    const float u = to_f(q[0]), v = to_f(q[1]), c = cs[i], s = cs[half + i];
    put(q, u * c - v * s);
    put(q + 1, v * c + u * s);
  }
}

// ------------------------------------------------------------------------------------------------
// Attention over the cached rows, one CTA per (token, head): four warps walk the keys, a lane holds every 32nd group of eight channels
// of a row, scores are warp sums, the weighted latents stay in registers.  All in fp32; any sizes.
// ------------------------------------------------------------------------------------------------
struct LatentAttnParams {
  const void* q_lat; long long ld_ql;    // [T, H * KR]
  const void* q; long long ldq;          // [T, H * head], rotated part at rot_off
  int head, rot_off;
  const void* cache;                     // [blocks * page, R]
  void* out; long long ldo;              // [T, H * KR]
  StepRows rows;
  int H, KR, R, page;
  float scale;
  int window;                            // <= 0: none
};

constexpr int kLaMaxVec = 5;             // R <= 32 * 8 * 5

template <typename T>
__global__ void __launch_bounds__(128) latent_attn_kernel(const LatentAttnParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];          // [4 warps][KR] partial sums, then m and l of every warp
  const int t = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
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
  const T* ql = reinterpret_cast<const T*>(p.q_lat) + (long long)t * p.ld_ql + (long long)h * p.KR;
  const T* qr = reinterpret_cast<const T*>(p.q) + (long long)t * p.ldq + (long long)h * p.head + p.rot_off;
  const int nv = p.R / 8, nkv = p.KR / 8;
  float q[kLaMaxVec][8], acc[kLaMaxVec][8];
#pragma unroll
  for (int i = 0; i < kLaMaxVec; ++i) {
    const int v = lane + 32 * i;
#pragma unroll
    for (int e = 0; e < 8; ++e) { q[i][e] = 0.f; acc[i][e] = 0.f; }
    if (v < nkv) load8(ql + v * 8, q[i]);
    else if (v < nv) load8(qr + (v - nkv) * 8, q[i]);
#pragma unroll
    for (int e = 0; e < 8; ++e) q[i][e] *= p.scale;
  }
  float m = -INFINITY, l = 0.f;
  for (int j = (p.window > 0 ? max(keys - p.window, 0) : 0) + warp; j < keys; j += 4) {
    const T* row = reinterpret_cast<const T*>(p.cache) + ((long long)bt[j / p.page] * p.page + j % p.page) * p.R;
    float k[kLaMaxVec][8], s = 0.f;
#pragma unroll
    for (int i = 0; i < kLaMaxVec; ++i) {
      const int v = lane + 32 * i;
      if (v < nv) {
        load8(row + v * 8, k[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) s = fmaf(q[i][e], k[i][e], s);
      }
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s), c = expf(m - mn), w = expf(s - mn);
    m = mn;
    l = l * c + w;
#pragma unroll
    for (int i = 0; i < kLaMaxVec; ++i)
      if (lane + 32 * i < nkv)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[i][e] = acc[i][e] * c + w * k[i][e];
  }
  float* sml = sm + 4 * p.KR;
#pragma unroll
  for (int i = 0; i < kLaMaxVec; ++i)
    if (lane + 32 * i < nkv) store8(sm + warp * p.KR + (lane + 32 * i) * 8, acc[i]);
  if (lane == 0) { sml[warp] = m; sml[4 + warp] = l; }
  __syncthreads();
  float M = -INFINITY;
  for (int w = 0; w < 4; ++w) M = fmaxf(M, sml[w]);
  float den = 0.f, f[4];
  for (int w = 0; w < 4; ++w) {
    f[w] = sml[w] == -INFINITY ? 0.f : expf(sml[w] - M);
    den += f[w] * sml[4 + w];
  }
  const float inv = den > 0.f ? 1.f / den : 0.f;
  T* out = reinterpret_cast<T*>(p.out) + (long long)t * p.ldo + (long long)h * p.KR;
  for (int c = threadIdx.x; c < p.KR; c += blockDim.x) {
    float o = 0.f;
    for (int w = 0; w < 4; ++w) o += f[w] * sm[w * p.KR + c];
    put(out + c, o * inv);
  }
}

}  // namespace lx

extern "C" {

int lx_latent_prep_bytes() { return (int)sizeof(lx::LatentPrepParams); }
int lx_latent_attn_bytes() { return (int)sizeof(lx::LatentAttnParams); }

int lx_latent_prep(const void* params, int T, int f32, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  const LatentPrepParams& p = *reinterpret_cast<const LatentPrepParams*>(params);
  if (p.QR % 8 != 0 || p.KR % 8 != 0 || p.R % 8 != 0 || p.ld_dq % 8 != 0 || p.ld_dkv % 8 != 0 || p.rot % 2 != 0 || p.rot > p.R - p.KR) return -1;
  if (p.q != nullptr && (p.head % 8 != 0 || p.off % 8 != 0 || p.ldq % 8 != 0 || p.off + p.rot > p.head)) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (f32) launch_pdl(latent_prep_kernel<float>, dim3(T), dim3(128), 0, s, p);
  else launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, s, p);
  return -(int)cudaGetLastError();
}

int lx_rope_pairs(void* x, long long ldx, const int* positions, const float* cos_sin, int T, int H, int head, int off, int rot, int f32,
                  void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (rot % 2 != 0 || off + rot > head) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (f32) launch_pdl(rope_pairs_kernel<float>, dim3(T), dim3(256), 0, s, reinterpret_cast<float*>(x), ldx, positions, cos_sin, H, head, off, rot);
  else launch_pdl(rope_pairs_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, reinterpret_cast<__nv_bfloat16*>(x), ldx, positions, cos_sin, H, head, off, rot);
  return -(int)cudaGetLastError();
}

int lx_latent_attn(const void* params, int T, int f32, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  const LatentAttnParams& p = *reinterpret_cast<const LatentAttnParams*>(params);
  if (p.R % 8 != 0 || p.KR % 8 != 0 || p.R > kLaMaxVec * 256 || p.head % 8 != 0 || p.rot_off % 8 != 0 || p.ldq % 8 != 0 || p.ld_ql % 8 != 0) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const size_t smem = sizeof(float) * (4 * p.KR + 8);
  if (f32) launch_pdl(latent_attn_kernel<float>, dim3(T, p.H), dim3(128), smem, s, p);
  else launch_pdl(latent_attn_kernel<__nv_bfloat16>, dim3(T, p.H), dim3(128), smem, s, p);
  return -(int)cudaGetLastError();
}

}  // extern "C"
