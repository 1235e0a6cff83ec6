// Paged causal attention row by row: one warp per (token, query head), any head sizes, any page size, bf16 or
// fp32 pages, everything between load and store in fp32.  It serves 32-bit models and shapes the tiled kernels
// do not take; decode rows and prompt rows are the same thing to it (a row is a token with a position and a
// block-table row, and it sees the cached keys up to its own position, or the last `window` of them).
//
// The warp walks its keys 32 at a time: lane j owns key j for Q.K (the query row sits in shared memory), the
// online softmax runs over the lanes, and for P.V the lanes own output dimensions and the 32 weights are passed
// round with shuffles.  A sink score starts the running maximum and contributes exp(sink) to the denominator.
#include "common.cuh"

namespace mie {
namespace {

constexpr int kRowWarps = 4;
constexpr int kDimsPerLane = 8;  // output dimensions one pass accumulates per lane; wider values take more passes

struct RowsParams {
  const void* q;
  long long q_st, q_sh;
  void* out;
  long long o_st, o_sh;
  const void* kb;
  const void* vb;
  long long kb_s[3], vb_s[3];
  IndexView positions, token_to_sequence, tables;
  const float* sinks;
  int tokens, q_heads, kv_heads, dim, vdim, page, num_pages, table_rows, table_width;
  long long window;
  float scale;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(kRowWarps * 32) attention_rows_kernel(RowsParams p) {
  extern __shared__ float rows_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* qs = rows_smem + (size_t)warp * p.dim;
  chain_wait();
  chain_release();
  const long long item = (long long)blockIdx.x * kRowWarps + warp;
  if (item >= (long long)p.tokens * p.q_heads) return;
  const long long t = item / p.q_heads;
  const int head = (int)(item % p.q_heads), kvh = head / (p.q_heads / p.kv_heads);
  T* orow = reinterpret_cast<T*>(p.out) + t * p.o_st + (long long)head * p.o_sh;
  const long long pos = p.positions.at(t);
  const long long seq = p.token_to_sequence.valid() ? p.token_to_sequence.at(t) : t;
  const bool bad_seq = seq < 0 || seq >= p.table_rows;
  const bool bad_pos = pos < 0 || pos >= (long long)p.table_width * p.page;
  if (bad_seq || bad_pos) {
    if (lane == 0) raise_status(p.status, bad_seq ? MIE_STATUS_BAD_SEQUENCE : MIE_STATUS_BAD_POSITION);
    for (int d = lane; d < p.vdim; d += 32) orow[d] = from_float<T>(0.f);
    return;
  }
  const T* qrow = reinterpret_cast<const T*>(p.q) + t * p.q_st + (long long)head * p.q_sh;
  for (int d = lane; d < p.dim; d += 32) qs[d] = to_float<T>(qrow[d]);
  __syncwarp();
  const long long begin = p.window > 0 && pos + 1 > p.window ? pos + 1 - p.window : 0;

  for (int d0 = 0; d0 < p.vdim; d0 += 32 * kDimsPerLane) {
    float m = -INFINITY, l = 0.f;
    if (p.sinks != nullptr) {
      m = p.sinks[head];
      l = 1.f;
    }
    float acc[kDimsPerLane];
#pragma unroll
    for (int i = 0; i < kDimsPerLane; ++i) acc[i] = 0.f;
    for (long long key0 = begin; key0 <= pos; key0 += 32) {
      const long long key = key0 + lane;
      float score = -INFINITY;
      long long vrow = 0;
      if (key <= pos) {
        long long page = p.tables.at(seq, key / p.page);
        if (page < 0 || page >= p.num_pages) {
          raise_status(p.status, MIE_STATUS_BAD_PAGE);
          page = 0;
        }
        const long long slot = key % p.page;
        const T* k = reinterpret_cast<const T*>(p.kb) + page * p.kb_s[0] + (long long)kvh * p.kb_s[1] + slot * p.kb_s[2];
        vrow = page * p.vb_s[0] + (long long)kvh * p.vb_s[1] + slot * p.vb_s[2];
        float dot = 0.f;
#pragma unroll 4
        for (int d = 0; d < p.dim; ++d) dot = fmaf(qs[d], to_float<T>(k[d]), dot);
        score = dot * p.scale;
      }
      const float m_new = fmaxf(m, warp_max(score));  // finite: the first key of a group is always visible
      const float alpha = expf(m - m_new);
      const float weight = key <= pos ? expf(score - m_new) : 0.f;
      l = l * alpha + warp_sum(weight);
      m = m_new;
#pragma unroll
      for (int i = 0; i < kDimsPerLane; ++i) acc[i] *= alpha;
      const int live = (int)(pos - key0 + 1 < 32 ? pos - key0 + 1 : 32);
      for (int j = 0; j < live; ++j) {
        const float w = __shfl_sync(0xffffffffu, weight, j);
        const T* v = reinterpret_cast<const T*>(p.vb) + __shfl_sync(0xffffffffu, vrow, j);
#pragma unroll
        for (int i = 0; i < kDimsPerLane; ++i) {
          const int d = d0 + 32 * i + lane;
          if (d < p.vdim) acc[i] = fmaf(w, to_float<T>(v[d]), acc[i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < kDimsPerLane; ++i) {
      const int d = d0 + 32 * i + lane;
      if (d < p.vdim) orow[d] = from_float<T>(acc[i] / l);
    }
  }
}

template <typename T>
int launch_rows(const RowsParams& p, cudaStream_t stream) {
  const long long items = (long long)p.tokens * p.q_heads;
  const size_t smem = (size_t)kRowWarps * p.dim * sizeof(float);
  MIE_CUDA(launch_chained(attention_rows_kernel<T>, dim3((unsigned)((items + kRowWarps - 1) / kRowWarps)),
                          dim3(kRowWarps * 32), smem, stream, p));
  MIE_LAUNCH_CHECK("attention_rows_kernel");
  return MIE_OK;
}

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_paged_attention_rows(const void* query, int64_t q_token_stride, int64_t q_head_stride, void* out,
                                        int64_t o_token_stride, int64_t o_head_stride, mie_view4_t key_blocks,
                                        mie_view4_t value_blocks, mie_index_t positions,
                                        mie_index_t token_to_sequence, mie_index_t block_tables, int32_t tokens,
                                        int32_t q_heads, int32_t kv_heads, int32_t dim, int32_t value_dim,
                                        int32_t block_size, int32_t num_blocks, int32_t table_rows,
                                        int32_t table_width, int32_t dtype, float scale, int64_t window,
                                        const float* sinks, int32_t* status, void* stream) {
  MIE_CHECK_ARG(dtype == MIE_DTYPE_BF16 || dtype == MIE_DTYPE_F32, "row attention takes bf16 or fp32");
  MIE_CHECK_ARG(query && out && key_blocks.ptr && value_blocks.ptr && positions.ptr && block_tables.ptr,
                "null tensor pointer");
  MIE_CHECK_ARG(tokens >= 0 && q_heads >= 1 && kv_heads >= 1 && q_heads % kv_heads == 0,
                "query heads (%d) must be a positive multiple of KV heads (%d)", q_heads, kv_heads);
  MIE_CHECK_ARG(dim >= 1 && dim <= 2048 && value_dim >= 1, "invalid head sizes (%d, %d)", dim, value_dim);
  MIE_CHECK_ARG(block_size >= 1 && num_blocks >= 1 && table_rows >= 1 && table_width >= 1, "invalid page geometry");
  MIE_CHECK_ARG(key_blocks.stride[3] == 1 && value_blocks.stride[3] == 1, "page rows must be contiguous");
  MIE_CHECK_ARG(window >= 0, "window must be >= 0 (0: none)");
  if (tokens == 0) return MIE_OK;
  RowsParams p;
  p.q = query;
  p.q_st = q_token_stride;
  p.q_sh = q_head_stride;
  p.out = out;
  p.o_st = o_token_stride;
  p.o_sh = o_head_stride;
  p.kb = key_blocks.ptr;
  p.vb = value_blocks.ptr;
  for (int i = 0; i < 3; ++i) {
    p.kb_s[i] = key_blocks.stride[i];
    p.vb_s[i] = value_blocks.stride[i];
  }
  p.positions = IndexView(positions);
  p.token_to_sequence = IndexView(token_to_sequence);
  p.tables = IndexView(block_tables);
  p.sinks = sinks;
  p.tokens = tokens;
  p.q_heads = q_heads;
  p.kv_heads = kv_heads;
  p.dim = dim;
  p.vdim = value_dim;
  p.page = block_size;
  p.num_pages = num_blocks;
  p.table_rows = table_rows;
  p.table_width = table_width;
  p.window = window;
  p.scale = scale;
  p.status = status;
  if (dtype == MIE_DTYPE_BF16) return launch_rows<__nv_bfloat16>(p, (cudaStream_t)stream);
  return launch_rows<float>(p, (cudaStream_t)stream);
}
