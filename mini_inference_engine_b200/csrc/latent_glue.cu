// What stands between the projections of latent attention and its attention kernels.  A layer caches one row per
// token, shared by all heads: [latent (rank) | rotated key part (rot_dim)].
//
//   latent_write_kernel   merged row [query latent | latent | key part] -> normed query latent; normed latent and
//                         rotated key part into the token's page slot
//   rotate_heads_kernel   rotation of the last rot_dim entries of every query head, in place or into other rows
//   latent_spans_kernel   which cached tokens the packed chunks of a step can see: a 16-token-aligned span of every
//                         request, laid end to end
//   latent_gather_kernel  those tokens' cached rows, contiguous, for the projection to per-head keys and values
#include "rows.cuh"

namespace mie {
namespace {

// Entries 2i and 2i + 1 turned by position * turns[i]; entries past the rotated ones pass.
template <typename T>
__device__ __forceinline__ void rotate_row(const T* src, T* dst, int rot_dim, int rotated, const float2* turns,
                                           float position, int lane, int lanes) {
  for (int i = lane; i < rotated / 2; i += lanes) {
    float sine, cosine;
    turn_sincos(position, turns[i], &sine, &cosine);
    const float u = to_float<T>(src[2 * i]), v = to_float<T>(src[2 * i + 1]);
    dst[2 * i] = from_float<T>(u * cosine - v * sine);
    dst[2 * i + 1] = from_float<T>(v * cosine + u * sine);
  }
  if (dst != src)
    for (int c = rotated + lane; c < rot_dim; c += lanes) dst[c] = src[c];
}

// One warp's RMS norm of a row.
template <typename T, int VEC>
__device__ __forceinline__ void warp_norm(const T* src, const T* weight, T* dst, int n, float eps, int lane) {
  float ss = 0.f;
  for (int c = lane * VEC; c < n; c += 32 * VEC) {
    float v[VEC];
    Vec<T, VEC>::load(src + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)n + eps);
  for (int c = lane * VEC; c < n; c += 32 * VEC) {
    float v[VEC], w[VEC];
    Vec<T, VEC>::load(src + c, v);
    Vec<T, VEC>::load(weight + c, w);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv * w[j];
    Vec<T, VEC>::store(dst + c, v);
  }
}

struct LatentWriteParams {
  const void* rows;  // [tokens][ld]: q_rank | rank | rot_dim (the last two only with pages)
  long long ld;
  int q_rank, rank, rot_dim, rotated;
  const void* q_weight;
  const void* weight;
  const float2* turns;
  void* q_out;
  long long ldq;
  void* pages;  // null: the layer caches nothing of its own
  long long page_stride, slot_stride;
  int tokens;
  float eps;
  Placement place;
};

template <typename T, int VEC>
__global__ void latent_write_kernel(LatentWriteParams p) {
  chain_wait();
  chain_release();
  const int lane = threadIdx.x & 31, parts = p.pages == nullptr ? 1 : 2;
  const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (item >= (long long)p.tokens * parts) return;
  const long long t = item / parts;
  const T* row = reinterpret_cast<const T*>(p.rows) + t * p.ld;
  if (item % parts == 0) {
    warp_norm<T, VEC>(row, reinterpret_cast<const T*>(p.q_weight), reinterpret_cast<T*>(p.q_out) + t * p.ldq, p.q_rank,
                      p.eps, lane);
    return;
  }
  const long long pos = p.place.positions.at(t);
  const long long page = p.place.page_of(p.place.sequence(t), pos, lane == 0);
  if (page < 0) return;
  T* slot = reinterpret_cast<T*>(p.pages) + page * p.page_stride + (pos % p.place.page) * p.slot_stride;
  warp_norm<T, VEC>(row + p.q_rank, reinterpret_cast<const T*>(p.weight), slot, p.rank, p.eps, lane);
  rotate_row<T>(row + p.q_rank + p.rank, slot + p.rank, p.rot_dim, p.rotated, p.turns, (float)pos, lane, 32);
}

// `lanes` lanes per token and group of heads; a lane turns one pair of every head of its group by the same angle.
constexpr int kRotateHeads = 8;

template <typename T>
__global__ void rotate_heads_kernel(const T* src, long long s_token, long long s_head, T* dst, long long d_token,
                                    long long d_head, IndexView positions, const float2* turns, int tokens, int heads,
                                    int rot_dim, int rotated, int lanes) {
  chain_wait();
  chain_release();
  const long long t = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / lanes;
  const int lane = threadIdx.x % lanes;
  if (t >= tokens) return;
  const float position = (float)positions.at(t);
  const int h0 = blockIdx.y * kRotateHeads;
  src += t * s_token + h0 * s_head;
  dst += t * d_token + h0 * d_head;
  heads = heads - h0 < kRotateHeads ? heads - h0 : kRotateHeads;
  for (int i = lane; i < rotated / 2; i += lanes) {
    float sine, cosine, u[kRotateHeads], v[kRotateHeads];  // all loads first: source and target may be the same rows
#pragma unroll
    for (int j = 0; j < kRotateHeads; ++j)
      if (j < heads) u[j] = to_float<T>(src[j * s_head + 2 * i]), v[j] = to_float<T>(src[j * s_head + 2 * i + 1]);
    turn_sincos(position, turns[i], &sine, &cosine);
#pragma unroll
    for (int j = 0; j < kRotateHeads; ++j)
      if (j < heads) {
        dst[j * d_head + 2 * i] = from_float<T>(u[j] * cosine - v[j] * sine);
        dst[j * d_head + 2 * i + 1] = from_float<T>(v[j] * cosine + u[j] * sine);
      }
  }
  if (dst != src)
    for (int j = 0; j < heads; ++j)
      for (int c = rotated + lane; c < rot_dim; c += lanes) dst[j * d_head + c] = src[j * s_head + c];
}

// spans: [requests] first row of a request's span in the gathered buffer, then [requests] its first token, then the
// total number of rows.  lens_out: kv length counted from the span's first token.  table_out: identity pages.
__global__ void latent_spans_kernel(IndexView cu_seqlens, IndexView kv_lens, int requests, long long window,
                                    int table_width, long long row_capacity, long long token_capacity, int* spans,
                                    int* lens_out, int* table_out, int* status) {
  chain_wait();
  chain_release();
  __shared__ int base_s;
  if (threadIdx.x == 0) base_s = 0;
  __syncthreads();
  for (int r = 0; r < requests; ++r) {
    const int base = base_s;
    __syncthreads();
    const long long q_len = cu_seqlens.at(r + 1) - cu_seqlens.at(r), kv_len = kv_lens.at(r);
    long long first = 0, rows = 0;
    bool good = q_len >= 0 && kv_len >= q_len && kv_len <= token_capacity;
    if (good && q_len > 0) {
      const long long start = kv_len - q_len;
      first = start + 1 > window ? (start + 1 - window) / 16 * 16 : 0;
      rows = (kv_len - first + 15) / 16 * 16;
      if (base + rows > row_capacity || rows > (long long)table_width * 16) good = false;
    }
    if (!good) {
      if (threadIdx.x == 0) raise_status(status, MIE_STATUS_BAD_LENGTH);
      first = rows = 0;
    }
    if (threadIdx.x == 0) {
      spans[r] = base;
      spans[requests + r] = (int)first;
      lens_out[r] = rows > 0 ? (int)(kv_len - first) : 0;
      base_s = base + (int)rows;
    }
    for (int i = threadIdx.x; i < table_width; i += blockDim.x)
      table_out[(long long)r * table_width + i] = i * 16 < rows ? base / 16 + i : -1;
    __syncthreads();
  }
  if (threadIdx.x == 0) spans[2 * requests] = base_s;
}

// One warp per gathered row: 16-byte copies, or element by element.
struct GatherParams {
  const char* pages;
  long long page_stride, slot_stride;  // bytes
  const int* spans;
  IndexView kv_lens, tables;
  char* out;
  int row_bytes, requests, page, num_pages, table_width;
  long long rows;
  int* status;
};

template <typename Unit>
__global__ void latent_gather_kernel(GatherParams p) {
  chain_wait();
  chain_release();
  const int lane = threadIdx.x & 31;
  const long long row = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (row >= p.rows || row >= p.spans[2 * p.requests]) return;
  int lo = 0, hi = p.requests - 1;  // last request whose span starts at or before this row
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (p.spans[mid] <= row) lo = mid;
    else hi = mid - 1;
  }
  const long long token = p.spans[p.requests + lo] + (row - p.spans[lo]);
  const int units = p.row_bytes / (int)sizeof(Unit);
  Unit* out = reinterpret_cast<Unit*>(p.out + row * p.row_bytes);
  const Unit* src = nullptr;
  if (token < p.kv_lens.at(lo) && token < (long long)p.table_width * p.page) {
    const long long id = p.tables.at(lo, token / p.page);
    if (id < 0 || id >= p.num_pages) {
      if (lane == 0) raise_status(p.status, MIE_STATUS_BAD_PAGE);
    } else {
      src = reinterpret_cast<const Unit*>(p.pages + id * p.page_stride + (token % p.page) * p.slot_stride);
    }
  }
  for (int i = lane; i < units; i += 32) {
    Unit v{};
    if (src != nullptr) v = src[i];
    out[i] = v;  // zero past the request's end
  }
}

template <typename T>
int launch_latent_write(const LatentWriteParams& p, bool vec, cudaStream_t stream) {
  const long long warps = (long long)p.tokens * (p.pages == nullptr ? 1 : 2);
  const dim3 grid((unsigned)((warps + 3) / 4)), block(128);
  MIE_CUDA(vec ? launch_chained(latent_write_kernel<T, 8>, grid, block, 0, stream, p)
               : launch_chained(latent_write_kernel<T, 1>, grid, block, 0, stream, p));
  MIE_LAUNCH_CHECK("latent_write_kernel");
  return MIE_OK;
}

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_latent_norm_write(const void* rows, int64_t ld, int32_t q_rank, int32_t rank, int32_t rot_dim,
                                     int32_t rotated, const void* q_weight, const void* weight, const float* turns,
                                     void* q_out, int64_t ldq, void* pages, int64_t page_stride, int64_t slot_stride,
                                     mie_index_t positions, mie_index_t token_to_sequence, mie_index_t block_tables,
                                     int32_t tokens, int32_t dtype, int32_t block_size, int32_t num_blocks,
                                     int32_t table_rows, int32_t table_width, float eps, int32_t* status,
                                     void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(rows && q_weight && q_out && positions.ptr, "null pointer");
  MIE_CHECK_ARG(tokens >= 0 && q_rank >= 1, "invalid sizes");
  MIE_CHECK_ARG(!pages || (weight && block_tables.ptr && rank >= 1 && rot_dim >= 0 && block_size >= 1 &&
                           num_blocks >= 1 && table_rows >= 1 && table_width >= 1),
                "writing the cache needs a norm weight, sizes and page geometry");
  MIE_CHECK_ARG(!pages || (rotated >= 0 && rotated % 2 == 0 && rotated <= rot_dim && (rotated == 0 || turns) &&
                           aligned(turns, 8)),
                "the rotated part must be an even number of entries of the key part, with its turns");
  if (tokens == 0) return MIE_OK;
  LatentWriteParams p;
  p.rows = rows;
  p.ld = ld;
  p.q_rank = q_rank;
  p.rank = rank;
  p.rot_dim = rot_dim;
  p.rotated = rotated;
  p.q_weight = q_weight;
  p.weight = weight;
  p.turns = reinterpret_cast<const float2*>(turns);
  p.q_out = q_out;
  p.ldq = ldq;
  p.pages = pages;
  p.page_stride = page_stride;
  p.slot_stride = slot_stride;
  p.tokens = tokens;
  p.eps = eps;
  p.place = placement(positions, token_to_sequence, block_tables, block_size, num_blocks, table_rows, table_width,
                      status);
  bool vec = q_rank % 8 == 0 && ld % 8 == 0 && ldq % 8 == 0 && aligned(rows, 16) && aligned(q_weight, 16) &&
             aligned(q_out, 16);
  if (pages)
    vec = vec && rank % 8 == 0 && page_stride % 8 == 0 && slot_stride % 8 == 0 && aligned(weight, 16) &&
          aligned(pages, 16);
  if (dtype == MIE_DTYPE_BF16) return launch_latent_write<__nv_bfloat16>(p, vec, (cudaStream_t)stream);
  return launch_latent_write<float>(p, vec, (cudaStream_t)stream);
}

extern "C" int mie_rotate_heads(const void* src, int64_t src_token_stride, int64_t src_head_stride, void* dst,
                                int64_t dst_token_stride, int64_t dst_head_stride, mie_index_t positions,
                                const float* turns, int32_t tokens, int32_t heads, int32_t rot_dim, int32_t rotated,
                                int32_t dtype, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(src && dst && positions.ptr, "null pointer");
  MIE_CHECK_ARG(tokens >= 0 && heads >= 1 && rot_dim >= 0, "invalid sizes");
  MIE_CHECK_ARG(rotated >= 0 && rotated % 2 == 0 && rotated <= rot_dim && (rotated == 0 || turns) && aligned(turns, 8),
                "the rotated part must be an even number of entries, with its turns");
  if (tokens == 0 || rot_dim == 0) return MIE_OK;
  int lanes = 1;
  while (lanes < 32 && lanes < (rot_dim + 1) / 2) lanes *= 2;
  const long long threads = (long long)tokens * lanes;
  const dim3 grid((unsigned)((threads + 127) / 128), (unsigned)((heads + kRotateHeads - 1) / kRotateHeads)), block(128);
  const float2* pairs = reinterpret_cast<const float2*>(turns);
  if (dtype == MIE_DTYPE_BF16)
    MIE_CUDA(launch_chained(rotate_heads_kernel<__nv_bfloat16>, grid, block, 0, (cudaStream_t)stream,
                            (const __nv_bfloat16*)src, (long long)src_token_stride, (long long)src_head_stride,
                            (__nv_bfloat16*)dst, (long long)dst_token_stride, (long long)dst_head_stride,
                            IndexView(positions), pairs, tokens, heads, rot_dim, rotated, lanes));
  else
    MIE_CUDA(launch_chained(rotate_heads_kernel<float>, grid, block, 0, (cudaStream_t)stream, (const float*)src,
                            (long long)src_token_stride, (long long)src_head_stride, (float*)dst,
                            (long long)dst_token_stride, (long long)dst_head_stride, IndexView(positions), pairs,
                            tokens, heads, rot_dim, rotated, lanes));
  MIE_LAUNCH_CHECK("rotate_heads_kernel");
  return MIE_OK;
}

extern "C" int mie_latent_spans(mie_index_t cu_seqlens, mie_index_t kv_lens, int32_t requests, int64_t window,
                                int32_t span_table_width, int64_t row_capacity, int64_t token_capacity, int32_t* spans,
                                int32_t* span_lens, int32_t* span_table, int32_t* status, void* stream) {
  MIE_CHECK_ARG(cu_seqlens.ptr && kv_lens.ptr && spans && span_lens && span_table, "null pointer");
  MIE_CHECK_ARG(requests >= 0 && window >= 1 && span_table_width >= 1 && row_capacity >= 0 &&
                    row_capacity < (1ll << 31),
                "invalid sizes");
  if (requests == 0) return MIE_OK;
  MIE_CUDA(launch_chained(latent_spans_kernel, dim3(1), dim3(128), 0, (cudaStream_t)stream, IndexView(cu_seqlens),
                          IndexView(kv_lens), requests, (long long)window, span_table_width, (long long)row_capacity,
                          (long long)token_capacity, spans, span_lens, span_table, status));
  MIE_LAUNCH_CHECK("latent_spans_kernel");
  return MIE_OK;
}

extern "C" int mie_latent_gather(const void* pages, int64_t page_stride, int64_t slot_stride, const int32_t* spans,
                                 mie_index_t kv_lens, mie_index_t block_tables, void* out, int64_t rows, int32_t cols,
                                 int32_t requests, int32_t dtype, int32_t block_size, int32_t num_blocks,
                                 int32_t table_width, int32_t* status, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(pages && spans && kv_lens.ptr && block_tables.ptr && out, "null pointer");
  MIE_CHECK_ARG(rows >= 0 && cols >= 1 && requests >= 1 && block_size >= 1 && num_blocks >= 1 && table_width >= 1,
                "invalid sizes");
  if (rows == 0) return MIE_OK;
  const int size = dtype == MIE_DTYPE_BF16 ? 2 : 4;
  const GatherParams p{(const char*)pages, page_stride * size, slot_stride * size, spans, IndexView(kv_lens),
                       IndexView(block_tables), (char*)out, cols * size, requests, block_size, num_blocks, table_width,
                       rows, status};
  const bool wide = p.row_bytes % 16 == 0 && p.page_stride % 16 == 0 && p.slot_stride % 16 == 0 && aligned(pages, 16) &&
                    aligned(out, 16);
  const dim3 grid((unsigned)((rows + 7) / 8)), block(256);
  if (wide)
    MIE_CUDA(launch_chained(latent_gather_kernel<uint4>, grid, block, 0, (cudaStream_t)stream, p));
  else if (size == 2)
    MIE_CUDA(launch_chained(latent_gather_kernel<uint16_t>, grid, block, 0, (cudaStream_t)stream, p));
  else
    MIE_CUDA(launch_chained(latent_gather_kernel<uint32_t>, grid, block, 0, (cudaStream_t)stream, p));
  MIE_LAUNCH_CHECK("latent_gather_kernel");
  return MIE_OK;
}
