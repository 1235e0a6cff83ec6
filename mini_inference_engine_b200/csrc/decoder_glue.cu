// Memory-bound glue for decoders with a 32-bit residual stream: token embedding with its additive parts, RMS
// norm of a scaled residual sum, the pass between the merged q/k/v projection and attention, and a clamped
// gated activation.  Every constant is a parameter.  Activations (GEMM operands and results) are bf16 or fp32
// (`dtype`), the residual stream, norms, angles and gates are fp32.
//
// Rows may have any width: a row whose width and strides allow it is read in 8- or 4-element vectors,
// otherwise element by element.
#include "rows.cuh"

namespace mie {
namespace {

// ---------------------------------------------------------------------------
// Embedding: x = table[id] * scale (+ bigram[row(previous id, id)]) (+ sinusoid(position)).
// One CTA per token.  A token's predecessor is the token before it in the flat stream when that belongs to
// the same sequence at the position before; otherwise it comes from the paged token history that every call
// also appends to.
// ---------------------------------------------------------------------------
struct EmbedParams {
  IndexView ids;
  const void* table;
  long long vocab;
  float scale;
  const void* bigram;         // [buckets + 1][width] or null; the last row is for a sequence's first token
  long long buckets, mul_prev, mul_cur;
  const float2* turns;        // [ceil(width / 2)] turns per position as a rounded fp32 part and its remainder, or null
  int* history;               // [num_pages][page] token ids, or null (needed by the bigram part)
  Placement place;
  float* out32;
  void* out;                  // activation copy, may be null
  int tokens, width;
};

template <typename T, int VEC>
__global__ void embed_kernel(EmbedParams p) {
  chain_wait();
  chain_release();
  const int t = blockIdx.x;
  const bool first_thread = threadIdx.x == 0;
  long long id = p.ids.at(t);
  if (id < 0 || id >= p.vocab) {
    if (first_thread) raise_status(p.place.status, MIE_STATUS_BAD_TOKEN);
    id = 0;
  }
  const long long pos = p.place.positions.at(t);
  const T* bigram_row = nullptr;
  if (p.history != nullptr) {
    const long long seq = p.place.sequence(t);
    if (p.bigram != nullptr) {
      long long row = p.buckets;
      if (pos > 0) {
        long long prev = -1;
        if (t > 0 && p.place.sequence(t - 1) == seq && p.place.positions.at(t - 1) == pos - 1) {
          prev = p.ids.at(t - 1);
        } else {
          const long long page = p.place.page_of(seq, pos - 1, first_thread);
          if (page >= 0) prev = p.history[page * p.place.page + (pos - 1) % p.place.page];
        }
        if (prev < 0 || prev >= p.vocab) {
          if (first_thread) raise_status(p.place.status, MIE_STATUS_BAD_TOKEN);
          prev = 0;
        }
        row = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
        if (row < 0) row += p.buckets;
      }
      bigram_row = reinterpret_cast<const T*>(p.bigram) + row * p.width;
    }
    if (first_thread) {
      const long long page = p.place.page_of(seq, pos, true);
      if (page >= 0) p.history[page * p.place.page + pos % p.place.page] = (int)id;
    }
  }
  const T* row = reinterpret_cast<const T*>(p.table) + id * p.width;
  float* out32 = p.out32 + (long long)t * p.width;
  T* out = p.out == nullptr ? nullptr : reinterpret_cast<T*>(p.out) + (long long)t * p.width;
  const float position = (float)pos;
  for (int c = threadIdx.x * VEC; c < p.width; c += blockDim.x * VEC) {
    float v[VEC];
    Vec<T, VEC>::load(row + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= p.scale;
    if (bigram_row != nullptr) {
      float b[VEC];
      Vec<T, VEC>::load(bigram_row + c, b);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] += b[j];
    }
    if (p.turns != nullptr) {
      if (VEC == 1) {
        float sine, cosine;
        turn_sincos(position, p.turns[c / 2], &sine, &cosine);
        v[0] += c % 2 == 0 ? sine : cosine;
      } else {
#pragma unroll
        for (int j = 0; j + 1 < VEC; j += 2) {
          float sine, cosine;
          turn_sincos(position, p.turns[(c + j) / 2], &sine, &cosine);
          v[j] += sine;
          v[j + 1] += cosine;
        }
      }
    }
    Vec<float, VEC>::store(out32 + c, v);
    if (out != nullptr) Vec<T, VEC>::store(out + c, v);
  }
}

// ---------------------------------------------------------------------------
// RMS norm of alpha * x + y: one CTA per row.  out = n * (offset + weight), n = s / sqrt(mean(s^2) + eps).
// ---------------------------------------------------------------------------
struct SumNormParams {
  const float* x;
  long long ldx;
  const void* y;  // may be null
  long long ldy;
  float alpha;
  const void* weight;
  float weight_offset;
  float* out32;  // may be null (may alias x)
  long long ld32;
  void* out;  // may be null
  long long ldo;
  int rows, cols;
  float eps;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(1024) sum_norm_kernel(SumNormParams p) {
  __shared__ float red[32];
  chain_wait();
  chain_release();
  const int row = blockIdx.x, tid = threadIdx.x;
  const float* x = p.x + (long long)row * p.ldx;
  const T* y = p.y == nullptr ? nullptr : reinterpret_cast<const T*>(p.y) + (long long)row * p.ldy;
  auto sum_at = [&](int c, float (&v)[VEC]) {
    Vec<float, VEC>::load(x + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= p.alpha;
    if (y != nullptr) {
      float r[VEC];
      Vec<T, VEC>::load(y + c, r);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] += r[j];
    }
  };
  const int step = blockDim.x * VEC;
  float kept[VEC];  // this thread's first group stays in registers; rows wider than one sweep are read again
  float ss = 0.f;
  for (int c = tid * VEC; c < p.cols; c += step) {
    float v[VEC];
    sum_at(c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      ss += v[j] * v[j];
      if (c < step) kept[j] = v[j];
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < (int)((blockDim.x + 31) >> 5); ++w) total += red[w];
  const float inv = 1.f / sqrtf(total / (float)p.cols + p.eps);
  for (int c = tid * VEC; c < p.cols; c += step) {
    float v[VEC], w[VEC];
    if (c < step) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = kept[j];
    } else {
      sum_at(c, v);
    }
    Vec<T, VEC>::load(reinterpret_cast<const T*>(p.weight) + c, w);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv * (p.weight_offset + w[j]);
    if (p.out32 != nullptr) Vec<float, VEC>::store(p.out32 + (long long)row * p.ld32 + c, v);
    if (p.out != nullptr) Vec<T, VEC>::store(reinterpret_cast<T*>(p.out) + (long long)row * p.ldo + c, v);
  }
}

// ---------------------------------------------------------------------------
// Between the merged projection and attention: LANES lanes per (token, head slot).
//   q: optional unit-RMS norm, optional position-dependent temperature, to q_out
//   k: optional unit-RMS norm, to its page
//   v: optional blend with another layer's values of the same token, to its page
// ---------------------------------------------------------------------------
struct QkvMixParams {
  const void* qkv;  // [tokens][ld]: q heads x dim | k heads x dim | v heads x vdim
  long long ld;
  const void* v_first;  // [tokens][ld_first]: v heads x vdim, or null
  long long ld_first;
  float lambda;
  int unit_norm;
  float eps;
  float temp_coef;
  long long temp_every;  // 0: no temperature
  void* q_out;           // [tokens][q_heads][dim]
  char* key_blocks;
  char* value_blocks;
  long long kb_s[3], vb_s[3];  // page, head, token strides (elements)
  int tokens, q_heads, kv_heads, dim, vdim;
  Placement place;
};

template <typename T, int VEC, int LANES>
__global__ void qkv_mix_kernel(QkvMixParams p) {
  chain_wait();
  chain_release();
  const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / LANES;
  const int lane = threadIdx.x % LANES;
  const int slots = p.q_heads + 2 * p.kv_heads;
  const bool live = item < (long long)p.tokens * slots;  // idle lanes stay for the shuffles of their warp
  const long long t = live ? item / slots : 0;
  const int h = live ? (int)(item % slots) : 0;
  const bool is_q = h < p.q_heads, is_v = h >= p.q_heads + p.kv_heads;
  const int kvh = is_v ? h - p.q_heads - p.kv_heads : h - p.q_heads;
  const int n = is_v ? p.vdim : p.dim;
  const long long offset = is_v ? (long long)(p.q_heads + p.kv_heads) * p.dim + (long long)kvh * p.vdim
                                : (long long)h * p.dim;
  const T* src = reinterpret_cast<const T*>(p.qkv) + t * p.ld + offset;
  const long long pos = p.place.positions.at(t);
  float factor = 1.f;
  if (p.unit_norm) {
    float ss = 0.f;
    if (!is_v) {
      for (int c = lane * VEC; c < n; c += LANES * VEC) {
        float v[VEC];
        Vec<T, VEC>::load(src + c, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
      }
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!is_v) factor = 1.f / sqrtf(ss / (float)n + p.eps);
  }
  if (!live) return;
  if (is_q && p.temp_every > 0) {
    const long long block = (pos + 1) / p.temp_every;
    factor *= 1.f + p.temp_coef * logf((float)(block + 1));
  }
  T* dst;
  if (is_q) {
    dst = reinterpret_cast<T*>(p.q_out) + (t * p.q_heads + h) * p.dim;
  } else {
    const long long page = p.place.page_of(p.place.sequence(t), pos, lane == 0);
    if (page < 0) return;
    const long long* st = is_v ? p.vb_s : p.kb_s;
    dst = reinterpret_cast<T*>(is_v ? p.value_blocks : p.key_blocks) + page * st[0] + (long long)kvh * st[1] +
          (pos % p.place.page) * st[2];
  }
  const T* first = is_v && p.v_first != nullptr
                       ? reinterpret_cast<const T*>(p.v_first) + t * p.ld_first + (long long)kvh * p.vdim
                       : nullptr;
  for (int c = lane * VEC; c < n; c += LANES * VEC) {
    float v[VEC];
    Vec<T, VEC>::load(src + c, v);
    if (first != nullptr) {
      float f[VEC];
      Vec<T, VEC>::load(first + c, f);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = (1.f - p.lambda) * v[j] + p.lambda * f[j];
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= factor;
    Vec<T, VEC>::store(dst + c, v);
  }
}

// ---------------------------------------------------------------------------
// Clamped gated activation: g = min(gate, limit), u = clamp(up, -limit, limit),
// out = g * sigmoid(slope * g) * (u + up_offset).
// ---------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void clamped_glu_kernel(const T* gate, const T* up, long long ld_in, T* out, long long ldo, int rows,
                                   int cols, float limit, float slope, float up_offset) {
  chain_wait();
  chain_release();
  const int per_row = cols / VEC;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)rows * per_row) return;
  const long long row = idx / per_row;
  const int c = (int)(idx % per_row) * VEC;
  float g[VEC], u[VEC];
  Vec<T, VEC>::load(gate + row * ld_in + c, g);
  Vec<T, VEC>::load(up + row * ld_in + c, u);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const float a = fminf(g[j], limit);
    const float b = fminf(fmaxf(u[j], -limit), limit);
    g[j] = a / (1.f + expf(-slope * a)) * (b + up_offset);
  }
  Vec<T, VEC>::store(out + row * ldo + c, g);
}

template <typename T>
int launch_sum_norm(const SumNormParams& p, bool vec, cudaStream_t stream) {
  const int groups = vec ? p.cols / 8 : p.cols;
  int threads = (groups + 31) / 32 * 32;
  if (threads > 1024) threads = 1024;
  if (vec)
    MIE_CUDA(launch_chained(sum_norm_kernel<T, 8>, dim3(p.rows), dim3(threads), 0, stream, p));
  else
    MIE_CUDA(launch_chained(sum_norm_kernel<T, 1>, dim3(p.rows), dim3(threads), 0, stream, p));
  MIE_LAUNCH_CHECK("sum_norm_kernel");
  return MIE_OK;
}

template <typename T>
int launch_qkv_mix(const QkvMixParams& p, int vec, cudaStream_t stream) {
  const long long slots = (long long)p.tokens * (p.q_heads + 2 * p.kv_heads);
  const int threads = 256, lanes = vec == 8 ? 16 : 32;
  const dim3 grid((unsigned)((slots * lanes + threads - 1) / threads)), block(threads);
  MIE_CUDA(vec == 8   ? launch_chained(qkv_mix_kernel<T, 8, 16>, grid, block, 0, stream, p)
           : vec == 4 ? launch_chained(qkv_mix_kernel<T, 4, 32>, grid, block, 0, stream, p)
                      : launch_chained(qkv_mix_kernel<T, 1, 32>, grid, block, 0, stream, p));
  MIE_LAUNCH_CHECK("qkv_mix_kernel");
  return MIE_OK;
}

template <typename T>
int launch_glu(const void* gate, const void* up, long long ld_in, void* out, long long ldo, int rows, int cols,
               float limit, float slope, float up_offset, bool vec, cudaStream_t stream) {
  const long long items = (long long)rows * (vec ? cols / 8 : cols);
  const int threads = 256;
  const dim3 grid((unsigned)((items + threads - 1) / threads));
  if (vec)
    MIE_CUDA(launch_chained(clamped_glu_kernel<T, 8>, grid, dim3(threads), 0, stream, (const T*)gate, (const T*)up,
                            ld_in, (T*)out, ldo, rows, cols, limit, slope, up_offset));
  else
    MIE_CUDA(launch_chained(clamped_glu_kernel<T, 1>, grid, dim3(threads), 0, stream, (const T*)gate, (const T*)up,
                            ld_in, (T*)out, ldo, rows, cols, limit, slope, up_offset));
  MIE_LAUNCH_CHECK("clamped_glu_kernel");
  return MIE_OK;
}

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_embed_tokens(mie_index_t ids, const void* table, int64_t vocab, float scale, const void* bigram,
                                int64_t buckets, int64_t mul_prev, int64_t mul_cur, const float* turns,
                                int32_t* history, mie_index_t positions, mie_index_t token_to_sequence,
                                mie_index_t block_tables, float* out32, void* out, int32_t tokens, int32_t width,
                                int32_t dtype, int32_t block_size, int32_t num_blocks, int32_t table_rows,
                                int32_t table_width, int32_t* status, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(ids.ptr && table && positions.ptr && out32, "null pointer");
  MIE_CHECK_ARG(tokens >= 0 && width >= 1 && vocab >= 1, "invalid sizes");
  MIE_CHECK_ARG(!bigram || (history && buckets >= 1), "the bigram part needs a bucket count and the token history");
  MIE_CHECK_ARG(!history || (block_tables.ptr && block_size >= 1 && num_blocks >= 1 && table_rows >= 1 &&
                             table_width >= 1),
                "the token history needs page geometry");
  if (tokens == 0) return MIE_OK;
  EmbedParams p;
  p.ids = IndexView(ids);
  p.table = table;
  p.vocab = vocab;
  p.scale = scale;
  p.bigram = bigram;
  p.buckets = buckets;
  p.mul_prev = mul_prev;
  p.mul_cur = mul_cur;
  p.turns = reinterpret_cast<const float2*>(turns);
  p.history = history;
  p.place = placement(positions, token_to_sequence, block_tables, block_size, num_blocks, table_rows, table_width,
                      status);
  p.out32 = out32;
  p.out = out;
  p.tokens = tokens;
  p.width = width;
  MIE_CHECK_ARG(aligned(turns, 8), "the turns must be 8-byte aligned pairs");
  const bool vec = width % 8 == 0 && aligned(table, 16) && aligned(bigram, 16) && aligned(out32, 16) && aligned(out, 16);
  int threads = ((vec ? width / 8 : width) + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  const dim3 grid(tokens), block(threads);
  if (dtype == MIE_DTYPE_BF16)
    MIE_CUDA(vec ? launch_chained(embed_kernel<__nv_bfloat16, 8>, grid, block, 0, (cudaStream_t)stream, p)
                 : launch_chained(embed_kernel<__nv_bfloat16, 1>, grid, block, 0, (cudaStream_t)stream, p));
  else
    MIE_CUDA(vec ? launch_chained(embed_kernel<float, 8>, grid, block, 0, (cudaStream_t)stream, p)
                 : launch_chained(embed_kernel<float, 1>, grid, block, 0, (cudaStream_t)stream, p));
  MIE_LAUNCH_CHECK("embed_kernel");
  return MIE_OK;
}

extern "C" int mie_sum_rms_norm(const float* x, int64_t ldx, const void* y, int64_t ldy, float alpha,
                                const void* weight, float weight_offset, float* out32, int64_t ld32, void* out,
                                int64_t ldo, int32_t rows, int32_t cols, int32_t dtype, float eps, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(x && weight && (out32 || out), "null pointer");
  MIE_CHECK_ARG(rows >= 0 && cols >= 1, "invalid sizes");
  if (rows == 0) return MIE_OK;
  SumNormParams p{x, ldx, y, ldy, alpha, weight, weight_offset, out32, ld32, out, ldo, rows, cols, eps};
  const bool vec = cols % 8 == 0 && ldx % 4 == 0 && ldy % 8 == 0 && ld32 % 4 == 0 && ldo % 8 == 0 && aligned(x, 16) &&
                   aligned(y, 16) && aligned(weight, 16) && aligned(out32, 16) && aligned(out, 16);
  if (dtype == MIE_DTYPE_BF16) return launch_sum_norm<__nv_bfloat16>(p, vec, (cudaStream_t)stream);
  return launch_sum_norm<float>(p, vec, (cudaStream_t)stream);
}

extern "C" int mie_qkv_norm_mix_write(const void* qkv, int64_t ld, const void* v_first, int64_t ld_first,
                                      float lambda, int32_t unit_norm, float eps, float temp_coef, int64_t temp_every,
                                      mie_index_t positions, mie_index_t token_to_sequence, mie_index_t block_tables,
                                      void* q_out, mie_view4_t key_blocks, mie_view4_t value_blocks, int32_t tokens,
                                      int32_t q_heads, int32_t kv_heads, int32_t dim, int32_t value_dim,
                                      int32_t dtype, int32_t block_size, int32_t num_blocks, int32_t table_rows,
                                      int32_t table_width, int32_t* status, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(qkv && q_out && key_blocks.ptr && value_blocks.ptr && positions.ptr && block_tables.ptr,
                "null pointer");
  MIE_CHECK_ARG(tokens >= 0 && q_heads >= 1 && kv_heads >= 1 && dim >= 1 && value_dim >= 1, "invalid sizes");
  MIE_CHECK_ARG(temp_every >= 0 && block_size >= 1 && num_blocks >= 1 && table_rows >= 1 && table_width >= 1,
                "invalid page geometry or temperature period");
  MIE_CHECK_ARG(key_blocks.stride[3] == 1 && value_blocks.stride[3] == 1, "page rows must be contiguous");
  if (tokens == 0) return MIE_OK;
  QkvMixParams p;
  p.qkv = qkv;
  p.ld = ld;
  p.v_first = v_first;
  p.ld_first = ld_first;
  p.lambda = lambda;
  p.unit_norm = unit_norm;
  p.eps = eps;
  p.temp_coef = temp_coef;
  p.temp_every = temp_every;
  p.q_out = q_out;
  p.key_blocks = (char*)key_blocks.ptr;
  p.value_blocks = (char*)value_blocks.ptr;
  // Widest vector that every row, stride and address allows.
  auto fits = [&](int v) {
    const int bytes = v * (dtype == MIE_DTYPE_BF16 ? 2 : 4) < 16 ? 8 : 16;
    bool ok = dim % v == 0 && value_dim % v == 0 && ld % v == 0 && ld_first % v == 0 && aligned(qkv, bytes) &&
              aligned(v_first, bytes) && aligned(q_out, bytes) && aligned(key_blocks.ptr, bytes) &&
              aligned(value_blocks.ptr, bytes);
    for (int i = 0; i < 3; ++i) ok = ok && key_blocks.stride[i] % v == 0 && value_blocks.stride[i] % v == 0;
    return ok;
  };
  for (int i = 0; i < 3; ++i) {
    p.kb_s[i] = key_blocks.stride[i];
    p.vb_s[i] = value_blocks.stride[i];
  }
  const int vec = fits(8) ? 8 : fits(4) ? 4 : 1;
  p.tokens = tokens;
  p.q_heads = q_heads;
  p.kv_heads = kv_heads;
  p.dim = dim;
  p.vdim = value_dim;
  p.place = placement(positions, token_to_sequence, block_tables, block_size, num_blocks, table_rows, table_width,
                      status);
  if (dtype == MIE_DTYPE_BF16) return launch_qkv_mix<__nv_bfloat16>(p, vec, (cudaStream_t)stream);
  return launch_qkv_mix<float>(p, vec, (cudaStream_t)stream);
}

extern "C" int mie_clamped_glu(const void* gate, const void* up, int64_t ld_in, void* out, int64_t ldo, int32_t rows,
                               int32_t cols, int32_t dtype, float limit, float slope, float up_offset, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(gate && up && out, "null pointer");
  MIE_CHECK_ARG(rows >= 0 && cols >= 1, "invalid sizes");
  if (rows == 0) return MIE_OK;
  const bool vec = cols % 8 == 0 && ld_in % 8 == 0 && ldo % 8 == 0 && aligned(gate, 16) && aligned(up, 16) &&
                   aligned(out, 16);
  if (dtype == MIE_DTYPE_BF16)
    return launch_glu<__nv_bfloat16>(gate, up, ld_in, out, ldo, rows, cols, limit, slope, up_offset, vec,
                                     (cudaStream_t)stream);
  return launch_glu<float>(gate, up, ld_in, out, ldo, rows, cols, limit, slope, up_offset, vec, (cudaStream_t)stream);
}
