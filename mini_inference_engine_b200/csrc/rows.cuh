// What the row kernels of decoders with a 32-bit residual stream share: vector access to bf16 or fp32 activations,
// the place of a token in the paged cache, rotation angles, block-wide sums.
#pragma once

#include "common.cuh"

namespace mie {
namespace {

// VEC consecutive activations <-> fp32.
template <typename T, int VEC>
struct Vec;
template <typename T>
struct Vec<T, 1> {
  __device__ __forceinline__ static void load(const T* p, float (&v)[1]) { v[0] = to_float<T>(*p); }
  __device__ __forceinline__ static void store(T* p, const float (&v)[1]) { *p = from_float<T>(v[0]); }
};
template <int VEC>
struct Vec<float, VEC> {
  __device__ __forceinline__ static void load(const float* p, float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) {
      const float4 f = *reinterpret_cast<const float4*>(p + i);
      v[i] = f.x, v[i + 1] = f.y, v[i + 2] = f.z, v[i + 3] = f.w;
    }
  }
  __device__ __forceinline__ static void store(float* p, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  }
};
template <>
struct Vec<float, 1> {
  __device__ __forceinline__ static void load(const float* p, float (&v)[1]) { v[0] = *p; }
  __device__ __forceinline__ static void store(float* p, const float (&v)[1]) { *p = v[0]; }
};
template <int VEC>
struct Vec<__nv_bfloat16, VEC> {
  static_assert(VEC == 4 || VEC == 8, "vector width");
  __device__ __forceinline__ static void load(const __nv_bfloat16* p, float (&v)[VEC]) {
    uint32_t raw[VEC / 2];
    if (VEC == 8) {
      const uint4 r = *reinterpret_cast<const uint4*>(p);
      raw[0] = r.x, raw[1] = r.y, raw[VEC / 2 - 2] = r.z, raw[VEC / 2 - 1] = r.w;
    } else {
      const uint2 r = *reinterpret_cast<const uint2*>(p);
      raw[0] = r.x, raw[1] = r.y;
    }
#pragma unroll
    for (int i = 0; i < VEC / 2; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[i]));
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  }
  __device__ __forceinline__ static void store(__nv_bfloat16* p, const float (&v)[VEC]) {
    uint32_t raw[VEC / 2];
#pragma unroll
    for (int i = 0; i < VEC / 2; ++i) {
      const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
      raw[i] = *reinterpret_cast<const uint32_t*>(&b);
    }
    if (VEC == 8)
      *reinterpret_cast<uint4*>(p) = make_uint4(raw[0], raw[1], raw[VEC / 2 - 2], raw[VEC / 2 - 1]);
    else
      *reinterpret_cast<uint2*>(p) = make_uint2(raw[0], raw[1]);
  }
};
template <>
struct Vec<__nv_bfloat16, 1> {
  __device__ __forceinline__ static void load(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
  __device__ __forceinline__ static void store(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
};

// Where a token's cached row lives: page id and slot, or a status bit.
struct Placement {
  IndexView positions, token_to_sequence, tables;
  int page, num_pages, table_rows, table_width;
  int* status;
  __device__ __forceinline__ long long sequence(long long t) const {
    return token_to_sequence.valid() ? token_to_sequence.at(t) : t;
  }
  __device__ __forceinline__ long long page_of(long long seq, long long pos, bool report) const {
    if (seq < 0 || seq >= table_rows) {
      if (report) raise_status(status, MIE_STATUS_BAD_SEQUENCE);
      return -1;
    }
    if (pos < 0 || pos >= (long long)table_width * page) {
      if (report) raise_status(status, MIE_STATUS_BAD_POSITION);
      return -1;
    }
    const long long id = tables.at(seq, pos / page);
    if (id < 0 || id >= num_pages) {
      if (report) raise_status(status, MIE_STATUS_BAD_PAGE);
      return -1;
    }
    return id;
  }
};

// sin and cos of position * turns * 2 pi: the whole turns of the product are taken off with its rounding error kept,
// so that a far position has a full fp32 angle.
__device__ __forceinline__ void turn_sincos(float position, float2 turns, float* sine, float* cosine) {
  const float product = position * turns.x;
  const float error = fmaf(position, turns.x, -product);
  const float rest = (product - rintf(product)) + fmaf(position, turns.y, error);
  sincospif(2.f * rest, sine, cosine);
}

// Sum over the block; `red` holds one float per warp and may be reused after the next block-wide barrier.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < (int)((blockDim.x + 31) >> 5); ++w) total += red[w];
  return total;
}

inline bool aligned(const void* p, int bytes) { return p == nullptr || reinterpret_cast<uintptr_t>(p) % bytes == 0; }

inline Placement placement(const mie_index_t& positions, const mie_index_t& token_to_sequence, const mie_index_t& tables,
                    int page, int num_pages, int table_rows, int table_width, int* status) {
  Placement out;
  out.positions = IndexView(positions);
  out.token_to_sequence = IndexView(token_to_sequence);
  out.tables = IndexView(tables);
  out.page = page;
  out.num_pages = num_pages;
  out.table_rows = table_rows;
  out.table_width = table_width;
  out.status = status;
  return out;
}

}  // namespace
}  // namespace mie

#define MIE_CHECK_ACT_DTYPE(dtype) \
  MIE_CHECK_ARG((dtype) == MIE_DTYPE_BF16 || (dtype) == MIE_DTYPE_F32, "activations are bf16 or fp32")
