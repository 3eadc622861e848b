// Attention over the paged KV cache.
//
// (attention.cuh holds the kernels)
//
//   attn_decode_kernel   one query token per row, GQA group packed into the MMA M dimension, keys split
//                        across the four warps of a CTA (each with a private cp.async pipeline) and
//                        optionally across CTAs (split-KV with a second combine pass).
//   attn_prefill_kernel  causal flash attention for ragged (padding-free) prompt chunks; K and V are read
//                        from the paged cache, so plain prefill, chunked prefill and prefill on top of a
//                        cached prefix are the same code path.
//
// Both honour a sliding window and logit soft-capping.  They stand in for the reference's third-party
// kernels: vLLM `paged_attention_v1/v2` (call site server/lorax_server/utils/paged_attention.py:127-178) and
// flash-attn `varlen_fwd` (utils/flash_attn.py:180-201).
//
// Cache layout (one tensor per layer): [num_blocks, kv_heads, 2, PAGE, D] -- for each (block, head) the K
// plane [PAGE, D] is followed by the V plane, so one page of one head is a single contiguous 2*PAGE*D run.
//
// fp8 cache (template flag KV8): pages hold e4m3 bytes in the same layout, written by `rope_kvwrite` as value / scale with one
// scale for K and one for V per layer (the reference's k_scale / v_scale, server/lorax_server/utils/paged_attention.py:23-47).
// A page arrives in shared memory as bytes (half the traffic of the bf16 cache, which is what bounds decode attention) and is
// expanded to a bf16 plane before the MMAs; the K scale is folded into the softmax scale and the V scale into the output.
#include "attention.cuh"

namespace lx {

template <int D, int STAGES, bool KV8>
static int launch_decode(const DecodeParams& p, int T, cudaStream_t s) {
  // Enough CTAs for several waves over the GPU: two warps per CTA, two CTAs per SM (their start-up and combine phases overlap the
  // other's streaming).  Few CTAs (small batches, split contexts): four warps each, so that one CTA keeps more pages in flight.
  static int force = -1;
  if (force < 0) {
    const char* e = getenv("LORAX_ATTN_DECODE_WARPS");
    force = e ? atoi(e) : 0;
  }
  const long long ctas = (long long)T * p.nkv * p.gchunks * p.nsplit;
  const bool two = force == 2 || (force != 4 && ctas >= 2 * 148);
  if (two) return launch_decode_nw<D, D, STAGES, KV8, 2>(p, T, s);
  return launch_decode_nw<D, D, STAGES, KV8, 4>(p, T, s);
}

}  // namespace lx

extern "C" {

int lx_attn_page_size() { return lx::kPage; }

// part_o / part_lse are only touched when nsplit > 1: sizes T*nh*nsplit*D and T*nh*nsplit floats.
int lx_attn_decode_alibi(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* ctx_lens,
                         void* out, long long ldo, float* part_o, float* part_lse, int T, int nh, int nkv, int d, int window, float scale,
                         float softcap, int nsplit, const float* alibi, void* stream);
int lx_attn_prefill_alibi(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* cu_q,
                          const int* cache_lens, const int* tile_seq, const int* tile_q0, int num_tiles, void* out, long long ldo, int nh,
                          int nkv, int d, int window, float scale, float softcap, const float* alibi, void* stream);

int lx_attn_decode(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* ctx_lens,
                   void* out, long long ldo, float* part_o, float* part_lse, int T, int nh, int nkv, int d, int window, float scale,
                   float softcap, int nsplit, void* stream) {
  return lx_attn_decode_alibi(q, ldq, kv, block_tables, max_blocks, ctx_lens, out, ldo, part_o, part_lse, T, nh, nkv, d, window, scale,
                              softcap, nsplit, nullptr, stream);
}

static int attn_decode_impl(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* ctx_lens,
                            void* out, long long ldo, float* part_o, float* part_lse, int T, int nh, int nkv, int d, int window, float scale,
                            float softcap, int nsplit, const float* alibi, bool kv8, float k_scale, float v_scale, void* stream) {
  using namespace lx;
  if (T <= 0) return 0;
  if (nh % nkv != 0) return -1;
  DecodeParams p{};
  p.q = reinterpret_cast<const __nv_bfloat16*>(q); p.ldq = ldq;
  p.kv = reinterpret_cast<const __nv_bfloat16*>(kv);
  p.block_tables = block_tables; p.max_blocks = max_blocks; p.ctx_lens = ctx_lens;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.part_o = part_o; p.part_lse = part_lse;
  p.nh = nh; p.nkv = nkv; p.group = nh / nkv; p.gchunks = (p.group + 15) / 16;
  p.window = window; p.scale = kv8 ? scale * k_scale : scale; p.softcap = softcap; p.alibi = alibi;
  p.v_scale = v_scale;
  p.nsplit = nsplit < 1 ? 1 : nsplit;
  if (p.nsplit > 1 && (part_o == nullptr || part_lse == nullptr)) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (kv8) {
    if (d == 128) return launch_decode<128, 3, true>(p, T, s);
    if (d == 64) return launch_decode<64, 4, true>(p, T, s);
    return -3;
  }
  if (d == 128) return launch_decode<128, 3, false>(p, T, s);
  if (d == 64) return launch_decode<64, 4, false>(p, T, s);
  return -3;
}

// `alibi`: [nh] fp32 slopes on the device (BLOOM, MPT), or null.
int lx_attn_decode_alibi(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* ctx_lens,
                         void* out, long long ldo, float* part_o, float* part_lse, int T, int nh, int nkv, int d, int window, float scale,
                         float softcap, int nsplit, const float* alibi, void* stream) {
  return attn_decode_impl(q, ldq, kv, block_tables, max_blocks, ctx_lens, out, ldo, part_o, part_lse, T, nh, nkv, d, window, scale, softcap,
                          nsplit, alibi, false, 1.f, 1.f, stream);
}

// The same over an e4m3 cache: stored value * k_scale (v_scale) is the key (value).
int lx_attn_decode_kv8(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* ctx_lens,
                       void* out, long long ldo, float* part_o, float* part_lse, int T, int nh, int nkv, int d, int window, float scale,
                       float softcap, int nsplit, const float* alibi, float k_scale, float v_scale, void* stream) {
  return attn_decode_impl(q, ldq, kv, block_tables, max_blocks, ctx_lens, out, ldo, part_o, part_lse, T, nh, nkv, d, window, scale, softcap,
                          nsplit, alibi, true, k_scale, v_scale, stream);
}

int lx_attn_prefill(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* cu_q,
                    const int* cache_lens, const int* tile_seq, const int* tile_q0, int num_tiles, void* out, long long ldo, int nh,
                    int nkv, int d, int window, float scale, float softcap, void* stream) {
  return lx_attn_prefill_alibi(q, ldq, kv, block_tables, max_blocks, cu_q, cache_lens, tile_seq, tile_q0, num_tiles, out, ldo, nh, nkv, d,
                               window, scale, softcap, nullptr, stream);
}

static int attn_prefill_impl(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* cu_q,
                             const int* cache_lens, const int* tile_seq, const int* tile_q0, int num_tiles, void* out, long long ldo, int nh,
                             int nkv, int d, int window, float scale, float softcap, const float* alibi, bool kv8, float k_scale,
                             float v_scale, void* stream) {
  using namespace lx;
  if (num_tiles <= 0) return 0;
  if (nh % nkv != 0) return -1;
  PrefillParams p{};
  p.q = reinterpret_cast<const __nv_bfloat16*>(q); p.ldq = ldq;
  p.kv = reinterpret_cast<const __nv_bfloat16*>(kv);
  p.block_tables = block_tables; p.max_blocks = max_blocks; p.cu_q = cu_q; p.cache_lens = cache_lens;
  p.tile_seq = tile_seq; p.tile_q0 = tile_q0;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.nh = nh; p.nkv = nkv; p.window = window; p.scale = kv8 ? scale * k_scale : scale; p.softcap = softcap; p.alibi = alibi;
  p.v_scale = v_scale;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (kv8) {
    if (d == 128) return launch_prefill<128, 128, true>(p, num_tiles, s);
    if (d == 64) return launch_prefill<64, 64, true>(p, num_tiles, s);
    return -3;
  }
  if (d == 128) return launch_prefill<128, 128, false>(p, num_tiles, s);
  if (d == 64) return launch_prefill<64, 64, false>(p, num_tiles, s);
  return -3;
}

int lx_attn_prefill_alibi(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* cu_q,
                          const int* cache_lens, const int* tile_seq, const int* tile_q0, int num_tiles, void* out, long long ldo, int nh,
                          int nkv, int d, int window, float scale, float softcap, const float* alibi, void* stream) {
  return attn_prefill_impl(q, ldq, kv, block_tables, max_blocks, cu_q, cache_lens, tile_seq, tile_q0, num_tiles, out, ldo, nh, nkv, d, window,
                           scale, softcap, alibi, false, 1.f, 1.f, stream);
}

int lx_attn_prefill_kv8(const void* q, long long ldq, const void* kv, const int* block_tables, int max_blocks, const int* cu_q,
                        const int* cache_lens, const int* tile_seq, const int* tile_q0, int num_tiles, void* out, long long ldo, int nh,
                        int nkv, int d, int window, float scale, float softcap, const float* alibi, float k_scale, float v_scale,
                        void* stream) {
  return attn_prefill_impl(q, ldq, kv, block_tables, max_blocks, cu_q, cache_lens, tile_seq, tile_q0, num_tiles, out, ldo, nh, nkv, d, window,
                           scale, softcap, alibi, true, k_scale, v_scale, stream);
}

}  // extern "C"
