// Host side of chunked-prefill attention on the 5th-generation tensor cores at head_dim 128; the kernel is in
// prefill_attention_umma.cuh.
#include <mutex>
#include <unordered_map>

#include "prefill_attention_umma.cuh"

namespace mie {
namespace {

struct TileMapKey {
  void* ptr;
  long long s0, s2;
  int num_blocks, kv_heads, block_size, dim, box_groups, dtype;
  bool operator==(const TileMapKey& o) const {
    return ptr == o.ptr && s0 == o.s0 && s2 == o.s2 && num_blocks == o.num_blocks && kv_heads == o.kv_heads &&
           block_size == o.block_size && dim == o.dim && box_groups == o.box_groups && dtype == o.dtype;
  }
};
struct TileMapKeyHash {
  size_t operator()(const TileMapKey& k) const {
    size_t h = reinterpret_cast<size_t>(k.ptr);
    h = h * 1000003u ^ (size_t)k.s0;
    h = h * 1000003u ^ (size_t)k.s2;
    h = h * 1000003u ^ (size_t)(k.num_blocks * 131 + k.kv_heads * 17 + k.block_size * 3 + k.dim * 7 + k.box_groups * 5 + k.dtype);
    return h;
  }
};

}  // namespace

// 5-D map over pages [page, head, token, dim] whose box is 16 whole tokens (4 KiB at dim 128):
//   d0 = 64 dims, d1 = token % 8, d2 = 64-dim group, d3 = (head, token / 8) merged, d4 = page.
// Merging head and token / 8 needs head stride == block_size * token stride; the caller checks that.
int page_slab_map(const mie_view4_t& pages, int num_blocks, int kv_heads, int block_size, int dim, int box_groups,
                  int dtype, CUtensorMap* out) {
  static std::mutex mu;
  static std::unordered_map<TileMapKey, CUtensorMap, TileMapKeyHash> cache;
  TileMapKey key{pages.ptr, pages.stride[0], pages.stride[2], num_blocks, kv_heads, block_size, dim, box_groups, dtype};
  {
    std::lock_guard<std::mutex> lock(mu);
    auto it = cache.find(key);
    if (it != cache.end()) {
      *out = it->second;
      return MIE_OK;
    }
  }
  const uint64_t tok = (uint64_t)pages.stride[2] * 2;  // bytes between tokens
  const uint64_t dims[5] = {64, 8, (uint64_t)dim / 64, (uint64_t)kv_heads * (block_size / 8), (uint64_t)num_blocks};
  const uint64_t strides[4] = {tok, 128, 8 * tok, (uint64_t)pages.stride[0] * 2};
  const uint32_t box[5] = {64, 8, (uint32_t)box_groups, kSub / 8, 1};
  const int rc = make_tensor_map(out, dtype == MIE_DTYPE_BF16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16
                                                              : CU_TENSOR_MAP_DATA_TYPE_FLOAT16,
                                 5, pages.ptr, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc != MIE_OK) return rc;
  std::lock_guard<std::mutex> lock(mu);
  if (cache.size() > 8192) cache.clear();
  cache.emplace(key, *out);
  return MIE_OK;
}

bool pages_fit_slab_map(const mie_view4_t& v, int block_size, int dim) {
  if (dim % 64 != 0 || block_size % kSub != 0 || v.stride[3] != 1 || v.stride[2] != dim) return false;
  if (v.stride[1] != (long long)block_size * v.stride[2]) return false;
  if (v.stride[0] <= 0 || (v.stride[0] * 2) % 16 != 0) return false;
  return (reinterpret_cast<uintptr_t>(v.ptr) & 15) == 0;
}

namespace {

constexpr int kDim = 128;
constexpr int kSmemBytes = PrefillTile<2, 2>::kSmemBytes;

template <typename T>
int launch_umma(const CUtensorMap& kmap, const CUtensorMap& vmap,
                const UmmaPrefillParams& p, int q_tiles, cudaStream_t stream) {
  static bool configured[64] = {false};
  int dev = 0;
  MIE_CUDA(cudaGetDevice(&dev));
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    MIE_CUDA(cudaFuncSetAttribute(prefill_umma_kernel<T, 2, 2, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemBytes));
    configured[dev] = true;
  }
  dim3 grid((unsigned)q_tiles, (unsigned)p.requests, (unsigned)p.kv_heads);
  prefill_umma_kernel<T, 2, 2, false><<<grid, kThreads, kSmemBytes, stream>>>(kmap, vmap, p, q_tiles);
  MIE_LAUNCH_CHECK("prefill_umma_kernel");
  return MIE_OK;
}

}  // namespace

// Returns MIE_ERR_UNSUPPORTED (without an error message) when the shape does not fit this kernel, so the
// caller can take the mma.sync kernel instead.
int prefill_attention_umma(const void* query, long long q_st, long long q_sh, long long total_tokens, void* out,
                           long long o_st, long long o_sh, const mie_view4_t& key_blocks,
                           const mie_view4_t& value_blocks, const mie_index_t& block_tables,
                           const mie_index_t& cu_seqlens, const mie_index_t& kv_lens, int requests, int max_query_len,
                           int q_heads, int kv_heads, int block_size, int num_blocks, int table_width, int dtype,
                           float scale, int* status, cudaStream_t stream) {
  const int group = q_heads / kv_heads;
  if (!(group == 1 || group == 2 || group == 4 || group == 8)) return MIE_ERR_UNSUPPORTED;
  if ((q_st * 2) % 16 || (q_sh * 2) % 16 || (reinterpret_cast<uintptr_t>(query) & 15)) return MIE_ERR_UNSUPPORTED;
  if ((o_st * 2) % 16 || (o_sh * 2) % 16 || (reinterpret_cast<uintptr_t>(out) & 15)) return MIE_ERR_UNSUPPORTED;
  if (total_tokens <= 0 || !(scale > 0.f)) return MIE_ERR_UNSUPPORTED;
  if (!pages_fit_slab_map(key_blocks, block_size, kDim) || !pages_fit_slab_map(value_blocks, block_size, kDim))
    return MIE_ERR_UNSUPPORTED;
  if ((long long)table_width * block_size / kSub + kKv / kSub > kMaxIds) return MIE_ERR_UNSUPPORTED;
  CUtensorMap kmap, vmap;
  if (int rc = page_slab_map(key_blocks, num_blocks, kv_heads, block_size, kDim, 2, dtype, &kmap)) return rc;
  if (int rc = page_slab_map(value_blocks, num_blocks, kv_heads, block_size, kDim, 2, dtype, &vmap)) return rc;
  UmmaPrefillParams p{(const char*)query, q_st, q_sh, (char*)out, o_st, o_sh, IndexView(block_tables), IndexView(cu_seqlens), IndexView(kv_lens),
                      requests, q_heads, kv_heads, group, block_size, num_blocks, table_width,
                      scale * 1.4426950408889634f, status, kDim, kDim, 1, 1, 1, 0, nullptr};
  const int tok_per_tile = kRows / group;
  const int q_tiles = (max_query_len + tok_per_tile - 1) / tok_per_tile;
  if (dtype == MIE_DTYPE_BF16) return launch_umma<__nv_bfloat16>(kmap, vmap, p, q_tiles, stream);
  return launch_umma<__half>(kmap, vmap, p, q_tiles, stream);
}

}  // namespace mie
