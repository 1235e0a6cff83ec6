// Ragged paged decode attention with sinks, sliding windows, separate key / value head sizes and any GQA group:
//
//   out = sum_j exp(s_j) v_j / (exp(sink_h) + sum_j exp(s_j)),   s_j = (q . k_j) * scale,
//
// over the last `window` cached keys (all of them without a window).  Same work plan, persistent warps and TMA
// rings as the plain kernel (decode_attention.cuh: decode_kernel with kExt); scores and weights stay fp32 (the
// weights enter P.V as a rounded bf16 part plus remainder).  The split-KV partials of a request are merged by one
// block per (request, query head).
#include "decode_attention.cuh"

namespace mie {
namespace {

constexpr int kMaxBoxes = 4;  // head sizes up to 256

template <int KH, int VH>
int launch_sink(const DecodeParams& p, const CUtensorMap& kmap, const CUtensorMap& vmap, cudaStream_t stream) {
  using Tile = DecodeTile<KH, VH>;
  using T = __nv_bfloat16;
  static bool configured[64] = {false};
  int dev = 0;
  MIE_CUDA(cudaGetDevice(&dev));
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    MIE_CUDA(cudaFuncSetAttribute(decode_kernel<T, KH, VH, true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                  (int)Tile::kSmem));
    configured[dev] = true;
  }
  MIE_CUDA(launch_chained(decode_kernel<T, KH, VH, true>, dim3(sm_count()), dim3(Tile::kWarps * 32), Tile::kSmem,
                          stream, kmap, vmap, p));
  MIE_LAUNCH_CHECK("decode_kernel");
  MIE_CUDA(launch_chained(merge_rows_kernel<T, VH>, dim3((unsigned)(p.batch * p.q_heads)), dim3(kMergeWarps * 32), 0,
                          stream, p));
  MIE_LAUNCH_CHECK("merge_rows_kernel");
  return MIE_OK;
}

template <int KH>
int launch_sink_v(int vh, const DecodeParams& p, const CUtensorMap& kmap, const CUtensorMap& vmap,
                  cudaStream_t stream) {
  switch (vh) {
    case 1: return launch_sink<KH, 1>(p, kmap, vmap, stream);
    case 2: return launch_sink<KH, 2>(p, kmap, vmap, stream);
    case 3: return launch_sink<KH, 3>(p, kmap, vmap, stream);
    default: return launch_sink<KH, 4>(p, kmap, vmap, stream);
  }
}

int boxes(int dim) { return (dim + 63) / 64; }
int item_heads_of(int q_heads, int kv_heads) { return kv_heads * ((q_heads / kv_heads + 7) / 8); }

bool pages_stream(const mie_view4_t& v, int block_size) {
  if (block_size % kTileTokens != 0 || v.stride[3] != 1 || (reinterpret_cast<uintptr_t>(v.ptr) & 15)) return false;
  for (int i = 0; i < 3; ++i)
    if (v.stride[i] <= 0 || v.stride[i] % 8 != 0) return false;
  return true;
}

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_sink_decode_supported(int32_t dim, int32_t value_dim, int32_t block_size, int32_t dtype) {
  return dtype == MIE_DTYPE_BF16 && dim >= 8 && value_dim >= 8 && dim % 8 == 0 && value_dim % 8 == 0 &&
         boxes(dim) <= kMaxBoxes && boxes(value_dim) <= kMaxBoxes && block_size >= kTileTokens &&
         block_size % kTileTokens == 0;
}

extern "C" int mie_sink_decode_attention(const void* query, int64_t q_row_stride, int64_t q_head_stride, void* out,
                                         int64_t o_row_stride, int64_t o_head_stride, mie_view4_t key_blocks,
                                         mie_view4_t value_blocks, mie_index_t block_tables,
                                         mie_index_t sequence_lengths, int32_t batch, int32_t q_heads,
                                         int32_t kv_heads, int32_t dim, int32_t value_dim, int32_t block_size,
                                         int32_t num_blocks, int32_t table_width, int32_t dtype, float scale,
                                         int64_t window, const float* sinks, int32_t split_policy, void* scratch,
                                         int64_t scratch_bytes, int32_t use_plan, int32_t plan_slot, int32_t* status,
                                         void* stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  MIE_CHECK_ARG(mie_sink_decode_supported(dim, value_dim, block_size, dtype),
                "sink decode attention takes bf16, head sizes that are multiples of 8 up to 256 and pages of whole "
                "16-token tiles (got %d, %d, page %d)", dim, value_dim, block_size);
  MIE_CHECK_ARG(batch >= 0 && q_heads >= 1 && kv_heads >= 1 && q_heads % kv_heads == 0,
                "query heads (%d) must be a positive multiple of KV heads (%d)", q_heads, kv_heads);
  MIE_CHECK_ARG(query && out && key_blocks.ptr && value_blocks.ptr && block_tables.ptr && sequence_lengths.ptr &&
                    scratch,
                "null pointer");
  MIE_CHECK_ARG(num_blocks >= 1 && table_width >= 1 && window >= 0 && split_policy >= 0, "invalid sizes");
  MIE_CHECK_ARG(plan_slot >= 0 && plan_slot < kCounters, "plan_slot must be in [0, %d)", kCounters);
  MIE_CHECK_ARG(pages_stream(key_blocks, block_size) && pages_stream(value_blocks, block_size),
                "pages must be 16-byte aligned rows with a contiguous last dimension");
  MIE_CHECK_ARG(q_row_stride % 2 == 0 && q_head_stride % 2 == 0 && o_row_stride % 2 == 0 && o_head_stride % 2 == 0 &&
                    (reinterpret_cast<uintptr_t>(query) & 3) == 0 && (reinterpret_cast<uintptr_t>(out) & 3) == 0,
                "query / out rows must be 4-byte aligned");
  MIE_CHECK_ARG((reinterpret_cast<uintptr_t>(scratch) & 255) == 0, "scratch must be 256-byte aligned");
  if (batch == 0) return MIE_OK;
  Scratch sc = carve(scratch, scratch_bytes, batch, q_heads, kv_heads, value_dim);
  MIE_CHECK_ARG(sc.cap > batch, "scratch of %lld bytes is too small for batch %d", (long long)scratch_bytes, batch);
  mie_view4_t q{const_cast<void*>(query), {q_row_stride, q_head_stride, 0, 1}};
  mie_view4_t o{out, {o_row_stride, o_head_stride, 0, 1}};
  const int item_heads = item_heads_of(q_heads, kv_heads);
  DecodeParams p{View4(q), View4(o), IndexView(block_tables), IndexView(sequence_lengths), IndexView(), sc, batch,
                 q_heads, kv_heads, q_heads / kv_heads, block_size, num_blocks, table_width,
                 scale * 1.4426950408889634f, plan_slot, status, nullptr, 0, nullptr, 0, 0, dim, value_dim, item_heads,
                 window, sinks};
  const int kh = boxes(dim), vh = boxes(value_dim);
  if (!use_plan) {
    const int warps = kh + vh <= 6 ? 8 : 6;
    plan_kernel<<<1, plan_threads(batch), 0, stream>>>(p.lengths, p.positions, batch,
                                                       (long long)table_width * block_size, item_heads, split_policy,
                                                       sm_count() * warps, 128, (long long)window, sc, status);
    MIE_LAUNCH_CHECK("plan_kernel");
  }
  CUtensorMap kmap, vmap;
  if (int rc = page_tensor_map(key_blocks, num_blocks, kv_heads, block_size, dim, dtype, &kmap)) return rc;
  if (int rc = page_tensor_map(value_blocks, num_blocks, kv_heads, block_size, value_dim, dtype, &vmap)) return rc;
  switch (kh) {
    case 1: return launch_sink_v<1>(vh, p, kmap, vmap, stream);
    case 2: return launch_sink_v<2>(vh, p, kmap, vmap, stream);
    case 3: return launch_sink_v<3>(vh, p, kmap, vmap, stream);
    default: return launch_sink_v<4>(vh, p, kmap, vmap, stream);
  }
}
