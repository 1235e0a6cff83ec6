// Row kernels around the sublayers of a decoder that norms a sublayer's input and its output: the fused
// "norm the result, add it to the residual stream, norm the stream for the next sublayer", a tanh-gelu with an
// optional per-token table factor, a gated norm, and a soft cap of logits.  Residual stream, norms, gates and
// logits are fp32, the other rows bf16 or fp32 (`dtype`).
#include "rows.cuh"

namespace mie {
namespace {

// ---------------------------------------------------------------------------
// x += alpha * rms_norm(y) * y_weight; then out = rms_norm(x) * next_weight, or out = x without a next weight.
// One CTA per row; x is updated in place.
// ---------------------------------------------------------------------------
struct ResidualParams {
  float* x;
  long long ldx;
  const void* y;
  long long ldy;
  const void* y_weight;
  float alpha;
  const void* next_weight;  // may be null
  void* out;                // may be null
  long long ldo;
  int cols;
  float eps;
};

// A thread's first kKept groups of VEC entries, one block width apart, stay in registers with their operands, which
// are all fetched before the first reduction; wider rows are read again.
constexpr int kKept = 2;

template <typename T, int VEC>
__global__ void __launch_bounds__(512) residual_norm_kernel(ResidualParams p) {
  __shared__ float red[2][32];
  chain_wait();
  chain_release();
  const int tid = threadIdx.x, step = blockDim.x * VEC;
  float* x = p.x + (long long)blockIdx.x * p.ldx;
  const T* y = reinterpret_cast<const T*>(p.y) + (long long)blockIdx.x * p.ldy;
  const T* yw = reinterpret_cast<const T*>(p.y_weight);
  const T* nw = p.out == nullptr ? nullptr : reinterpret_cast<const T*>(p.next_weight);
  float sums[kKept][VEC], ys[kKept][VEC], yws[kKept][VEC];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kKept; ++k) {
    const int c = (k * blockDim.x + tid) * VEC;
    if (c < p.cols) {
      Vec<T, VEC>::load(y + c, ys[k]);
      Vec<float, VEC>::load(x + c, sums[k]);
      Vec<T, VEC>::load(yw + c, yws[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < kKept; ++k)
    if ((k * (int)blockDim.x + tid) * VEC < p.cols)
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss += ys[k][j] * ys[k][j];
  for (int c = (kKept * blockDim.x + tid) * VEC; c < p.cols; c += step) {
    float v[VEC];
    Vec<T, VEC>::load(y + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
  }
  const float inv_y = p.alpha / sqrtf(block_sum(ss, red[0]) / (float)p.cols + p.eps);
  ss = 0.f;
#pragma unroll
  for (int k = 0; k < kKept; ++k) {
    const int c = (k * blockDim.x + tid) * VEC;
    if (c < p.cols) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        sums[k][j] += ys[k][j] * inv_y * yws[k][j];
        ss += sums[k][j] * sums[k][j];
      }
      Vec<float, VEC>::store(x + c, sums[k]);
    }
  }
  for (int c = (kKept * blockDim.x + tid) * VEC; c < p.cols; c += step) {
    float v[VEC], w[VEC], r[VEC];
    Vec<T, VEC>::load(y + c, v);
    Vec<T, VEC>::load(yw + c, w);
    Vec<float, VEC>::load(x + c, r);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      r[j] += v[j] * inv_y * w[j];
      ss += r[j] * r[j];
    }
    Vec<float, VEC>::store(x + c, r);
  }
  if (p.out == nullptr) return;
  const float inv_x = nw == nullptr ? 1.f : 1.f / sqrtf(block_sum(ss, red[1]) / (float)p.cols + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + (long long)blockIdx.x * p.ldo;
  auto emit = [&](int c, float (&v)[VEC]) {
    if (nw != nullptr) {
      float w[VEC];
      Vec<T, VEC>::load(nw + c, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv_x * w[j];
    }
    Vec<T, VEC>::store(out + c, v);
  };
#pragma unroll
  for (int k = 0; k < kKept; ++k) {
    const int c = (k * blockDim.x + tid) * VEC;
    if (c < p.cols) emit(c, sums[k]);
  }
  for (int c = (kKept * blockDim.x + tid) * VEC; c < p.cols; c += step) {
    float v[VEC];
    Vec<float, VEC>::load(x + c, v);
    emit(c, v);
  }
}

// ---------------------------------------------------------------------------
// out = gelu(in) (* table[ids[row]][c]), gelu(z) = z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))).
// ---------------------------------------------------------------------------
struct GeluParams {
  const void* in;
  long long ld_in;
  IndexView ids;  // with the table
  const void* table;
  long long ld_table, vocab;
  void* out;
  long long ldo;
  int rows, cols;
  int* status;
};

__device__ __forceinline__ float gelu_tanh(float z) {
  const float inner = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return 0.5f * z * (1.f + tanhf(inner));
}

template <typename T, int VEC>
__global__ void gelu_kernel(GeluParams p) {
  chain_wait();
  chain_release();
  const int per_row = p.cols / VEC;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)p.rows * per_row) return;
  const long long row = idx / per_row;
  const int c = (int)(idx % per_row) * VEC;
  float v[VEC];
  Vec<T, VEC>::load(reinterpret_cast<const T*>(p.in) + row * p.ld_in + c, v);
#pragma unroll
  for (int j = 0; j < VEC; ++j) v[j] = gelu_tanh(v[j]);
  if (p.table != nullptr) {
    long long id = p.ids.at(row);
    if (id < 0 || id >= p.vocab) {
      if (c == 0) raise_status(p.status, MIE_STATUS_BAD_TOKEN);
      id = 0;
    }
    float e[VEC];
    Vec<T, VEC>::load(reinterpret_cast<const T*>(p.table) + id * p.ld_table + c, e);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= e[j];
  }
  Vec<T, VEC>::store(reinterpret_cast<T*>(p.out) + row * p.ldo + c, v);
}

// ---------------------------------------------------------------------------
// out = rms_norm(x) * weight * sigmoid(gate).  One CTA per row.
// ---------------------------------------------------------------------------
struct GatedNormParams {
  const void* x;
  long long ldx;
  const void* gate;
  long long ldg;
  const void* weight;
  void* out;
  long long ldo;
  int cols;
  float eps;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(512) gated_norm_kernel(GatedNormParams p) {
  __shared__ float red[32];
  chain_wait();
  chain_release();
  const int tid = threadIdx.x, step = blockDim.x * VEC;
  const T* x = reinterpret_cast<const T*>(p.x) + (long long)blockIdx.x * p.ldx;
  const T* gate = reinterpret_cast<const T*>(p.gate) + (long long)blockIdx.x * p.ldg;
  T* out = reinterpret_cast<T*>(p.out) + (long long)blockIdx.x * p.ldo;
  const T* weight = reinterpret_cast<const T*>(p.weight);
  float xs[kKept][VEC], ws[kKept][VEC], gs[kKept][VEC];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kKept; ++k) {
    const int c = (k * blockDim.x + tid) * VEC;
    if (c < p.cols) {
      Vec<T, VEC>::load(x + c, xs[k]);
      Vec<T, VEC>::load(weight + c, ws[k]);
      Vec<T, VEC>::load(gate + c, gs[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < kKept; ++k)
    if ((k * (int)blockDim.x + tid) * VEC < p.cols)
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss += xs[k][j] * xs[k][j];
  for (int c = (kKept * blockDim.x + tid) * VEC; c < p.cols; c += step) {
    float v[VEC];
    Vec<T, VEC>::load(x + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.cols + p.eps);
  auto emit = [&](int c, float (&v)[VEC], const float (&w)[VEC], const float (&g)[VEC]) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = __fdividef(v[j] * inv * w[j], 1.f + expf(-g[j]));
    Vec<T, VEC>::store(out + c, v);
  };
#pragma unroll
  for (int k = 0; k < kKept; ++k) {
    const int c = (k * blockDim.x + tid) * VEC;
    if (c < p.cols) emit(c, xs[k], ws[k], gs[k]);
  }
  for (int c = (kKept * blockDim.x + tid) * VEC; c < p.cols; c += step) {
    float v[VEC], w[VEC], g[VEC];
    Vec<T, VEC>::load(x + c, v);
    Vec<T, VEC>::load(weight + c, w);
    Vec<T, VEC>::load(gate + c, g);
    emit(c, v, w, g);
  }
}

// logits <- cap * tanh(logits / cap), in place.
__global__ void softcap_kernel(float* logits, long long count, float cap) {
  chain_wait();
  chain_release();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < count) logits[i] = cap * tanhf(logits[i] / cap);
}

int row_threads(int cols, bool vec) {
  const int groups = vec ? cols / 8 : cols;
  const int threads = ((groups + kKept - 1) / kKept + 31) / 32 * 32;
  return threads > 512 ? 512 : threads;
}

// One CTA per row, in the vector width the rows allow.
#define MIE_LAUNCH_ROWS(kernel, dtype, rows, cols, vec, params)                                                     \
  do {                                                                                                              \
    const dim3 grid__((unsigned)(rows)), block__((unsigned)row_threads(cols, vec));                                 \
    if ((dtype) == MIE_DTYPE_BF16)                                                                                  \
      MIE_CUDA(vec ? launch_chained(kernel<__nv_bfloat16, 8>, grid__, block__, 0, (cudaStream_t)stream, params)     \
                   : launch_chained(kernel<__nv_bfloat16, 1>, grid__, block__, 0, (cudaStream_t)stream, params));   \
    else                                                                                                            \
      MIE_CUDA(vec ? launch_chained(kernel<float, 8>, grid__, block__, 0, (cudaStream_t)stream, params)             \
                   : launch_chained(kernel<float, 1>, grid__, block__, 0, (cudaStream_t)stream, params));           \
    MIE_LAUNCH_CHECK(#kernel);                                                                                      \
  } while (0)

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_residual_norm(float* x, int64_t ldx, const void* y, int64_t ldy, const void* y_weight, float alpha,
                                 const void* next_weight, void* out, int64_t ldo, int32_t rows, int32_t cols,
                                 int32_t dtype, float eps, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(x && y && y_weight, "null pointer");
  MIE_CHECK_ARG(!next_weight || out, "a next norm needs an output");
  MIE_CHECK_ARG(rows >= 0 && cols >= 1, "invalid sizes");
  if (rows == 0) return MIE_OK;
  const ResidualParams p{x, ldx, y, ldy, y_weight, alpha, next_weight, out, ldo, cols, eps};
  const bool vec = cols % 8 == 0 && ldx % 4 == 0 && ldy % 8 == 0 && ldo % 8 == 0 && aligned(x, 16) && aligned(y, 16) &&
                   aligned(y_weight, 16) && aligned(next_weight, 16) && aligned(out, 16);
  MIE_LAUNCH_ROWS(residual_norm_kernel, dtype, rows, cols, vec, p);
  return MIE_OK;
}

extern "C" int mie_gelu(const void* in, int64_t ld_in, mie_index_t ids, const void* table, int64_t ld_table,
                        int64_t vocab, void* out, int64_t ldo, int32_t rows, int32_t cols, int32_t dtype,
                        int32_t* status, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(in && out, "null pointer");
  MIE_CHECK_ARG(!table || (ids.ptr && vocab >= 1), "a table factor needs token ids and the table's size");
  MIE_CHECK_ARG(rows >= 0 && cols >= 1, "invalid sizes");
  if (rows == 0) return MIE_OK;
  const GeluParams p{in, ld_in, IndexView(ids), table, ld_table, vocab, out, ldo, rows, cols, status};
  const bool vec = cols % 8 == 0 && ld_in % 8 == 0 && ldo % 8 == 0 && aligned(in, 16) && aligned(out, 16) &&
                   (!table || (ld_table % 8 == 0 && aligned(table, 16)));
  const long long items = (long long)rows * (vec ? cols / 8 : cols);
  const dim3 grid((unsigned)((items + 255) / 256)), block(256);
  if (dtype == MIE_DTYPE_BF16)
    MIE_CUDA(vec ? launch_chained(gelu_kernel<__nv_bfloat16, 8>, grid, block, 0, (cudaStream_t)stream, p)
                 : launch_chained(gelu_kernel<__nv_bfloat16, 1>, grid, block, 0, (cudaStream_t)stream, p));
  else
    MIE_CUDA(vec ? launch_chained(gelu_kernel<float, 8>, grid, block, 0, (cudaStream_t)stream, p)
                 : launch_chained(gelu_kernel<float, 1>, grid, block, 0, (cudaStream_t)stream, p));
  MIE_LAUNCH_CHECK("gelu_kernel");
  return MIE_OK;
}

extern "C" int mie_gated_norm(const void* x, int64_t ldx, const void* gate, int64_t ldg, const void* weight, void* out,
                              int64_t ldo, int32_t rows, int32_t cols, int32_t dtype, float eps, void* stream) {
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(x && gate && weight && out, "null pointer");
  MIE_CHECK_ARG(rows >= 0 && cols >= 1, "invalid sizes");
  if (rows == 0) return MIE_OK;
  const GatedNormParams p{x, ldx, gate, ldg, weight, out, ldo, cols, eps};
  const bool vec = cols % 8 == 0 && ldx % 8 == 0 && ldg % 8 == 0 && ldo % 8 == 0 && aligned(x, 16) &&
                   aligned(gate, 16) && aligned(weight, 16) && aligned(out, 16);
  MIE_LAUNCH_ROWS(gated_norm_kernel, dtype, rows, cols, vec, p);
  return MIE_OK;
}

extern "C" int mie_softcap(float* logits, int64_t count, float cap, void* stream) {
  MIE_CHECK_ARG(logits && count >= 0 && cap > 0.f, "soft cap needs logits and a positive cap");
  if (count == 0) return MIE_OK;
  MIE_CUDA(launch_chained(softcap_kernel, dim3((unsigned)((count + 255) / 256)), dim3(256), 0, (cudaStream_t)stream,
                          logits, (long long)count, cap));
  MIE_LAUNCH_CHECK("softcap_kernel");
  return MIE_OK;
}
