// Chunked-prefill attention with sinks, sliding windows, separate key / value head sizes and any GQA group on the
// tcgen05 kernel (prefill_attention_umma.cuh with kExt).  Values wider than 128 dims take several passes of 128
// (each pass computes the scores again).
#include "prefill_attention_umma.cuh"

namespace mie {

// Defined in decode_attention.cu: cached 4-D tensor map over [pages, kv_heads, page, dim], box 16 tokens x 64 dims.
int page_tensor_map(const mie_view4_t& pages, int num_blocks, int kv_heads, int block_size, int dim, int dtype,
                    CUtensorMap* out);

namespace {

template <int KH, int VH>
int launch_sink_prefill(const CUtensorMap& kmap, const CUtensorMap& vmap, const UmmaPrefillParams& p, int q_tiles,
                        cudaStream_t stream) {
  using T = __nv_bfloat16;
  using Tile = PrefillTile<KH, VH>;
  static bool configured[64] = {false};
  int dev = 0;
  MIE_CUDA(cudaGetDevice(&dev));
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    MIE_CUDA(cudaFuncSetAttribute(prefill_umma_kernel<T, KH, VH, true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                  Tile::kSmemBytes));
    configured[dev] = true;
  }
  dim3 grid((unsigned)q_tiles, (unsigned)p.requests, (unsigned)(p.kv_heads * p.v_passes));
  prefill_umma_kernel<T, KH, VH, true><<<grid, kThreads, Tile::kSmemBytes, stream>>>(kmap, vmap, p, q_tiles);
  MIE_LAUNCH_CHECK("prefill_umma_kernel");
  return MIE_OK;
}

template <int KH>
int launch_sink_prefill_v(int vh, const CUtensorMap& kmap, const CUtensorMap& vmap, const UmmaPrefillParams& p,
                          int q_tiles, cudaStream_t stream) {
  return vh == 1 ? launch_sink_prefill<KH, 1>(kmap, vmap, p, q_tiles, stream)
                 : launch_sink_prefill<KH, 2>(kmap, vmap, p, q_tiles, stream);
}

int page_map(const mie_view4_t& pages, int num_blocks, int kv_heads, int block_size, int dim, int box_groups, bool slab,
             CUtensorMap* out) {
  return slab ? page_slab_map(pages, num_blocks, kv_heads, block_size, dim, box_groups, MIE_DTYPE_BF16, out)
              : page_tensor_map(pages, num_blocks, kv_heads, block_size, dim, MIE_DTYPE_BF16, out);
}

bool rows_aligned(const void* p, long long s0, long long s1) {
  return s0 % 8 == 0 && s1 % 8 == 0 && (reinterpret_cast<uintptr_t>(p) & 15) == 0;
}

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_sink_prefill_supported(int32_t q_heads, int32_t kv_heads, int32_t dim, int32_t value_dim,
                                          int32_t block_size, int32_t dtype, float scale) {
  return dtype == MIE_DTYPE_BF16 && kv_heads >= 1 && q_heads % kv_heads == 0 && q_heads / kv_heads <= kRows &&
         dim >= 8 && dim % 8 == 0 && dim <= 256 && value_dim >= 8 && value_dim % 8 == 0 && block_size >= kSub &&
         block_size % kSub == 0 && scale > 0.f;
}

extern "C" int mie_sink_prefill_attention(const void* query, int64_t q_token_stride, int64_t q_head_stride, void* out,
                                          int64_t o_token_stride, int64_t o_head_stride, mie_view4_t key_blocks,
                                          mie_view4_t value_blocks, mie_index_t block_tables, mie_index_t cu_seqlens,
                                          mie_index_t kv_lens, int32_t requests, int32_t max_query_len,
                                          int32_t q_heads, int32_t kv_heads, int32_t dim, int32_t value_dim,
                                          int32_t block_size, int32_t num_blocks, int32_t table_width, int32_t dtype,
                                          float scale, int64_t window, const float* sinks, int32_t* status,
                                          void* stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  MIE_CHECK_ARG(mie_sink_prefill_supported(q_heads, kv_heads, dim, value_dim, block_size, dtype, scale),
                "sink prefill attention takes bf16, key sizes that are multiples of 8 up to 256, value sizes that are "
                "multiples of 8, at most 128 query heads per KV head, pages of whole 16-token tiles and scale > 0");
  MIE_CHECK_ARG(query && out && key_blocks.ptr && value_blocks.ptr && block_tables.ptr && cu_seqlens.ptr && kv_lens.ptr,
                "null tensor pointer");
  MIE_CHECK_ARG(requests >= 0 && max_query_len >= 0 && num_blocks >= 1 && table_width >= 1 && window >= 0,
                "invalid sizes");
  MIE_CHECK_ARG(rows_aligned(query, q_token_stride, q_head_stride) && rows_aligned(out, o_token_stride, o_head_stride),
                "query / out rows must be 16-byte aligned");
  for (const mie_view4_t* v : {&key_blocks, &value_blocks}) {
    MIE_CHECK_ARG(v->stride[3] == 1 && (reinterpret_cast<uintptr_t>(v->ptr) & 15) == 0, "pages must be 16-byte aligned");
    for (int i = 0; i < 3; ++i)
      MIE_CHECK_ARG(v->stride[i] > 0 && v->stride[i] % 8 == 0, "page strides must be multiples of 16 bytes");
  }
  if (requests == 0 || max_query_len == 0) return MIE_OK;
  const int group = q_heads / kv_heads;
  const int kh = (dim + 63) / 64, vh = value_dim <= 64 ? 1 : 2;
  const bool k_slab = pages_fit_slab_map(key_blocks, block_size, dim);
  const bool v_slab = pages_fit_slab_map(value_blocks, block_size, value_dim);
  CUtensorMap kmap, vmap;
  if (int rc = page_map(key_blocks, num_blocks, kv_heads, block_size, dim, kh, k_slab, &kmap)) return rc;
  if (int rc = page_map(value_blocks, num_blocks, kv_heads, block_size, value_dim, vh, v_slab, &vmap)) return rc;
  UmmaPrefillParams p{(const char*)query, q_token_stride, q_head_stride, (char*)out, o_token_stride, o_head_stride,
                      IndexView(block_tables), IndexView(cu_seqlens), IndexView(kv_lens), requests, q_heads, kv_heads,
                      group, block_size, num_blocks, table_width, scale * 1.4426950408889634f, status, dim, value_dim,
                      (value_dim + vh * 64 - 1) / (vh * 64), k_slab ? 1 : 0, v_slab ? 1 : 0, window, sinks};
  const int tokens_per_tile = kRows / group;
  const int q_tiles = (max_query_len + tokens_per_tile - 1) / tokens_per_tile;
  switch (kh) {
    case 1: return launch_sink_prefill_v<1>(vh, kmap, vmap, p, q_tiles, stream);
    case 2: return launch_sink_prefill_v<2>(vh, kmap, vmap, p, q_tiles, stream);
    case 3: return launch_sink_prefill_v<3>(vh, kmap, vmap, p, q_tiles, stream);
    default: return launch_sink_prefill_v<4>(vh, kmap, vmap, p, q_tiles, stream);
  }
}
