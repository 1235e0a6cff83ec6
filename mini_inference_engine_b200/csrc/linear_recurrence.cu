// Recurrent mixers whose state lives in a slot per request (fp32), bf16 or fp32 activations:
//
//   decayed outer products   S <- decay_h S + k v^T,  o = S^T q per head, q / k / v through silu
//   gated average            S <- (1 - z) S + z c element by element, z = sigmoid(a + bias),
//                            c = u + 1/2 (u >= 0) or sigmoid(u), output S silu(g)
//
// A slot is a row of one state buffer (slot_stride floats); a layer's part of it starts at the pointer it passes.
// A sequence whose first token of the call has position 0 starts from zero, whatever the slot holds, so slots are
// handed over without clearing.  Every kernel reads a request's state, advances it by the tokens of the call and
// writes it back.
//
// Packed chunks are cut into segments.  With several segments to a request three launches run: what every segment
// adds from a zero state, a carry pass over the segments of each request, and the segments with their true initial
// state; with one segment to a request only the last of them.
#include "rows.cuh"

namespace mie {
namespace {

// 2^x and 1 / x on the special-function unit (about 22 bits).
__device__ __forceinline__ float exp2_unit(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float reciprocal_unit(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// 1 + e^-v, the denominator of sigmoid(v); v bounded from below so that a product of two stays finite.
__device__ __forceinline__ float sigmoid_denominator(float v) {
  return 1.f + exp2_unit(fminf(v * -1.4426950408889634f, 60.f));
}
__device__ __forceinline__ float silu(float v) { return v * reciprocal_unit(1.f + exp2_unit(v * -1.4426950408889634f)); }

struct Slots {
  float* state;
  long long stride;
  IndexView slots;
  int count;
  int* status;
  __device__ __forceinline__ float* at(long long row) const {
    const long long slot = slots.at(row);
    if (slot < 0 || slot >= count) {
      raise_status(status, MIE_STATUS_BAD_SLOT);
      return nullptr;
    }
    return state + slot * stride;
  }
};

// Segment `index` of packed chunks cut into pieces of `length` tokens.
struct Segment {
  int request, index, first_of_request;  // segment number inside the request; number of the request's first segment
  long long begin, end;                  // tokens
  bool last;
};
struct Segments {
  IndexView cu_seqlens;
  int requests, length;
  __device__ __forceinline__ bool find(int number, Segment* out) const {
    int first = 0;
    for (int r = 0; r < requests; ++r) {
      const long long begin = cu_seqlens.at(r), end = cu_seqlens.at(r + 1);
      const int pieces = end > begin ? (int)((end - begin + length - 1) / length) : 0;
      if (number < first + pieces) {
        out->request = r;
        out->index = number - first;
        out->first_of_request = first;
        out->begin = begin + (long long)out->index * length;
        out->end = out->begin + length < end ? out->begin + length : end;
        out->last = out->index == pieces - 1;
        return true;
      }
      first += pieces;
    }
    return false;
  }
};

// ---------------------------------------------------------------------------
// Decayed outer products
// ---------------------------------------------------------------------------
struct OuterParams {
  const void* rows;  // [tokens][ld]: q heads x dim | k heads x dim | v heads x vdim
  long long ld;
  const float* decay;  // [heads]
  void* out;           // [tokens][ldo], heads x vdim
  long long ldo;
  Slots slots;
  IndexView positions;  // by token
  int tokens, heads, dim, vdim;
  Segments seg;
  float* carry;  // [segments][heads][dim][vdim], null: every request is one segment
};

constexpr int kOuterWarps = 8;

// One token per row: the warps share the state's rows (key dims), a lane owns VEC of its columns (value dims).
template <typename T, int VEC>
__global__ void __launch_bounds__(kOuterWarps * 32) outer_decode_kernel(OuterParams p) {
  extern __shared__ float outer_smem[];
  chain_wait();
  chain_release();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = blockIdx.x / p.heads, h = blockIdx.x % p.heads;
  const int col = (blockIdx.y * 32 + lane) * VEC;
  float* qs = outer_smem;
  float* ks = qs + p.dim;
  float* red = ks + p.dim;  // [warps][32 * VEC]
  const T* src = reinterpret_cast<const T*>(p.rows) + (long long)row * p.ld;
  for (int i = threadIdx.x; i < p.dim; i += blockDim.x) {
    qs[i] = silu(to_float<T>(src[h * p.dim + i]));
    ks[i] = silu(to_float<T>(src[(p.heads + h) * p.dim + i]));
  }
  __syncthreads();
  float* slot = p.slots.at(row);
  const bool live = col < p.vdim && slot != nullptr;
  float o[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) o[j] = 0.f;
  if (live) {
    const bool fresh = p.positions.at(row) == 0;
    const float decay = p.decay[h];
    float v[VEC];
    Vec<T, VEC>::load(src + 2 * p.heads * p.dim + h * p.vdim + col, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = silu(v[j]);
    float* state = slot + (long long)h * p.dim * p.vdim + col;
#pragma unroll 4
    for (int i = warp; i < p.dim; i += kOuterWarps) {
      float s[VEC];
      if (fresh) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) s[j] = 0.f;
      } else {
        Vec<float, VEC>::load(state + (long long)i * p.vdim, s);
      }
      const float k = ks[i], q = qs[i];
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        s[j] = decay * s[j] + k * v[j];
        o[j] += s[j] * q;
      }
      Vec<float, VEC>::store(state + (long long)i * p.vdim, s);
    }
  }
#pragma unroll
  for (int j = 0; j < VEC; ++j) red[(warp * 32 + lane) * VEC + j] = o[j];
  __syncthreads();
  if (warp == 0 && col < p.vdim) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      float sum = 0.f;
      for (int w = 0; w < kOuterWarps; ++w) sum += red[(w * 32 + lane) * VEC + j];
      o[j] = sum;
    }
    Vec<T, VEC>::store(reinterpret_cast<T*>(p.out) + (long long)row * p.ldo + h * p.vdim + col, o);
  }
}

// Any sizes, token after token: one CTA per (request, head, 32 value dims), the state tile in shared memory.
template <typename T>
__global__ void __launch_bounds__(kOuterWarps * 32) outer_rows_kernel(OuterParams p) {
  extern __shared__ float outer_smem[];
  chain_wait();
  chain_release();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.x / p.heads, h = blockIdx.x % p.heads, col = blockIdx.y * 32 + lane;
  const long long begin = p.seg.cu_seqlens.at(r), end = p.seg.cu_seqlens.at(r + 1);
  if (end <= begin) return;
  float* slot = p.slots.at(r);
  if (slot == nullptr) return;
  float* qs = outer_smem;
  float* ks = qs + p.dim;
  float* red = ks + p.dim;                // [warps][32]
  float* tile = red + kOuterWarps * 32;   // [dim][32]
  const bool live = col < p.vdim, fresh = p.positions.at(begin) == 0;
  float* state = slot + (long long)h * p.dim * p.vdim + col;
  for (int i = warp; i < p.dim; i += kOuterWarps)
    tile[i * 32 + lane] = live && !fresh ? state[(long long)i * p.vdim] : 0.f;
  const float decay = p.decay[h];
  for (long long t = begin; t < end; ++t) {
    const T* src = reinterpret_cast<const T*>(p.rows) + t * p.ld;
    for (int i = threadIdx.x; i < p.dim; i += blockDim.x) {
      qs[i] = silu(to_float<T>(src[h * p.dim + i]));
      ks[i] = silu(to_float<T>(src[(p.heads + h) * p.dim + i]));
    }
    const float v = live ? silu(to_float<T>(src[2 * p.heads * p.dim + h * p.vdim + col])) : 0.f;
    __syncthreads();
    float o = 0.f;
    for (int i = warp; i < p.dim; i += kOuterWarps) {
      const float s = decay * tile[i * 32 + lane] + ks[i] * v;
      tile[i * 32 + lane] = s;
      o += s * qs[i];
    }
    red[warp * 32 + lane] = o;
    __syncthreads();
    if (warp == 0 && live) {
      float sum = 0.f;
      for (int w = 0; w < kOuterWarps; ++w) sum += red[w * 32 + lane];
      reinterpret_cast<T*>(p.out)[t * p.ldo + h * p.vdim + col] = from_float<T>(sum);
    }
  }
  if (live)
    for (int i = warp; i < p.dim; i += kOuterWarps) state[(long long)i * p.vdim] = tile[i * 32 + lane];
}

// The chunked form on tensor cores (bf16): one CTA per (segment, head, 64 * VD value dims) walks its segment 64 tokens
// at a time with the state in registers.  With q, k, v of 64 tokens and the state S before them,
//
//   o_i  = decay^(i+1) S^T q_i + sum_(j <= i) A_ij v_j,   A_ij = decay^(i-j) (q_i . k_j)
//   S   <- decay^n S + sum_j k_j (decay^(n-1-j) v_j)^T
//
// q, k, v are the bf16 activations; S, A and the decayed v enter products as a rounded part plus its remainder (two
// MMAs), sums are fp32.  The rows of the next tile are copied to a staging area while this one is computed; a thread
// converts (silu) the 16-byte units it copied itself.  8 * VD warps: a warp computes 16 x (32 / VD) of A, 32 tokens x
// 16 value dims of o, and 16 key dims x (KD * 32) value dims of the state.
constexpr int kOuterTokens = 64;

template <int KD, int VD>  // 64-dim groups of a key row, of a CTA's value row
struct OuterTile {
  static constexpr int kThreads = 256 * VD;
  static constexpr int kRow = 8192;  // 64 rows x 64 bf16, 128-byte rows, 16-byte units XOR-swizzled by row
  static constexpr int kOffQ = 0;
  static constexpr int kOffK = kOffQ + KD * kRow;
  static constexpr int kOffV = kOffK + KD * kRow;
  static constexpr int kOffW = kOffV + VD * kRow;           // decayed v: rounded part, remainder
  static constexpr int kOffS = kOffW + 2 * VD * kRow;       // state: rounded part, remainder; [key dim][value dim]
  static constexpr int kOffA = kOffS + 2 * KD * VD * kRow;  // A: rounded part, remainder
  static constexpr int kOffStage = kOffA + 2 * kRow;        // one 16-byte unit per thread and pass
  static constexpr int kKeyPasses = kOuterTokens * KD * 8 / kThreads;
  static constexpr int kValuePasses = kOuterTokens * VD * 8 / kThreads;
  static constexpr int kOffPow = kOffStage + (2 * kKeyPasses + kValuePasses) * kThreads * 16;
  static constexpr int kSmem = kOffPow + 80 * 4;
};

__device__ __forceinline__ uint32_t swizzled(int row, int unit) { return row * 128 + ((unit ^ (row & 7)) << 4); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) { return Mma16816<__nv_bfloat16>::pack(lo, hi); }

// 16 bytes global -> shared, or zeros.
__device__ __forceinline__ void copy_async16(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

template <int KD, int VD, bool kEmit>
__global__ void __launch_bounds__(256 * VD, KD + VD == 2 ? 2 : 1) outer_chunk_kernel(OuterParams p) {
  using Tile = OuterTile<KD, VD>;
  using T = __nv_bfloat16;
  using Mma = Mma16816<T>;
  constexpr int kThreads = Tile::kThreads, kRow = Tile::kRow;
  extern __shared__ __align__(1024) uint8_t chunk_smem[];
  float* powers = reinterpret_cast<float*>(chunk_smem + Tile::kOffPow);
  const uint32_t base = smem_u32(chunk_smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, col0 = blockIdx.z * VD * 64;
  chain_wait();
  chain_release();
  Segment seg;
  if (!p.seg.find(blockIdx.x, &seg)) return;
  if (!kEmit && seg.last) return;  // nobody needs what the last segment adds
  float* slot = p.slots.at(seg.request);
  if (slot == nullptr) return;
  const float decay = p.decay[h];
  if (tid <= kOuterTokens) powers[tid] = powf(decay, (float)tid);

  // Staging: passes of q, k, v units in turn, a thread's own unit of a pass at its own place.
  auto stage = [&](long long tok0) {
    const T* rows = reinterpret_cast<const T*>(p.rows);
    uint32_t dst = base + Tile::kOffStage + tid * 16;
#pragma unroll
    for (int which = 0; which < 2; ++which)
#pragma unroll
      for (int pass = 0; pass < Tile::kKeyPasses; ++pass, dst += kThreads * 16) {
        if (!kEmit && which == 0) continue;
        const int i = pass * kThreads + tid, r = i / (KD * 8), unit = i % (KD * 8);
        const bool live = tok0 + r < seg.end && unit * 8 < p.dim;
        copy_async16(dst, rows + (live ? (tok0 + r) * p.ld + (which * p.heads + h) * p.dim + unit * 8 : 0), live);
      }
#pragma unroll
    for (int pass = 0; pass < Tile::kValuePasses; ++pass, dst += kThreads * 16) {
      const int i = pass * kThreads + tid, r = i / (VD * 8), unit = i % (VD * 8);
      const bool live = tok0 + r < seg.end && col0 + unit * 8 < p.vdim;
      copy_async16(dst, rows + (live ? (tok0 + r) * p.ld + 2 * p.heads * p.dim + h * p.vdim + col0 + unit * 8 : 0), live);
    }
    copy_async_commit();
  };
  stage(seg.begin);

  // State tile of this warp: key dims s_row + {g, g + 8}, value dims s_col + nt * 8 + {2 t4, 2 t4 + 1}.
  constexpr int kStateTiles = KD * 4;
  float s[kStateTiles][4];
  const int s_row = warp % (KD * 4) * 16, s_col = warp / (KD * 4) * (KD * 32);
  const long long head_state = (long long)h * p.dim * p.vdim;
  const long long carry_at = ((long long)blockIdx.x * p.heads + h) * p.dim * p.vdim;
  const float* init = nullptr;
  if (kEmit) {
    if (p.carry != nullptr)
      init = p.carry + carry_at;
    else if (p.positions.at(p.seg.cu_seqlens.at(seg.request)) != 0)
      init = slot + head_state;
  }
  auto each_pair = [&](auto&& visit) {  // two neighbouring columns of a state row
#pragma unroll
    for (int nt = 0; nt < kStateTiles; ++nt)
#pragma unroll
      for (int half = 0; half < 2; ++half)
        visit(s_row + g + half * 8, s_col + nt * 8 + 2 * t4, s[nt][2 * half], s[nt][2 * half + 1]);
  };
  each_pair([&](int d, int c, float& a, float& b) {
    a = b = 0.f;
    if (init != nullptr && d < p.dim && col0 + c < p.vdim) {
      const float2 v = *reinterpret_cast<const float2*>(init + (long long)d * p.vdim + col0 + c);
      a = v.x;
      b = v.y;
    }
  });

  // ldmatrix lane geometry: plain B operand ([n][k] rows), transposed B operand ([k][n] rows), A operand, transposed A.
  const int b_row = (lane & 7) + ((lane >> 4) & 1) * 8, b_sel = (lane >> 3) & 1;
  const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_sel = (lane >> 4) & 1;
  const int at_row = b_row, at_sel = b_sel;
  const int a_row = v_row, a_sel = v_sel;

  for (long long tok0 = seg.begin; tok0 < seg.end; tok0 += kOuterTokens) {
    const int n = (int)(seg.end - tok0 < kOuterTokens ? seg.end - tok0 : kOuterTokens);
    copy_async_wait();
    __syncthreads();  // the previous tile has been read (first pass: the powers are there)
    const uint8_t* staged = chunk_smem + Tile::kOffStage + tid * 16;
    auto unpack = [&](float (&v)[8]) {
      Vec<T, 8>::load(reinterpret_cast<const T*>(staged), v);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = silu(v[j]);
      staged += kThreads * 16;
    };
    // q and k through silu; rows past the segment and dims past the head are zero.
#pragma unroll
    for (int which = 0; which < 2; ++which) {
      if (!kEmit && which == 0) {
        staged += Tile::kKeyPasses * kThreads * 16;
        continue;
      }
#pragma unroll
      for (int pass = 0; pass < Tile::kKeyPasses; ++pass) {
        const int i = pass * kThreads + tid, r = i / (KD * 8), unit = i % (KD * 8);
        float v[8];
        unpack(v);
        *reinterpret_cast<uint4*>(chunk_smem + (which == 0 ? Tile::kOffQ : Tile::kOffK) + (unit >> 3) * kRow +
                                  swizzled(r, unit & 7)) =
            make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
      }
    }
#pragma unroll
    for (int pass = 0; pass < Tile::kValuePasses; ++pass) {
      const int i = pass * kThreads + tid, r = i / (VD * 8), unit = i % (VD * 8);
      float v[8];
      unpack(v);
      const float weight = r < n ? powers[n - 1 - r] : 0.f;
      uint32_t whole[4], high[4], low[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        whole[j] = pack_bf16(v[2 * j], v[2 * j + 1]);
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&whole[j]));
        const float wa = b.x * weight, wb = b.y * weight;
        high[j] = pack_bf16(wa, wb);
        const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high[j]));
        low[j] = pack_bf16(wa - k.x, wb - k.y);
      }
      const uint32_t off = (unit >> 3) * kRow + swizzled(r, unit & 7);
      if (kEmit) *reinterpret_cast<uint4*>(chunk_smem + Tile::kOffV + off) = make_uint4(whole[0], whole[1], whole[2], whole[3]);
      *reinterpret_cast<uint4*>(chunk_smem + Tile::kOffW + off) = make_uint4(high[0], high[1], high[2], high[3]);
      *reinterpret_cast<uint4*>(chunk_smem + Tile::kOffW + VD * kRow + off) = make_uint4(low[0], low[1], low[2], low[3]);
    }
    if (tok0 + kOuterTokens < seg.end) stage(tok0 + kOuterTokens);
    if (kEmit) {
      each_pair([&](int d, int c, float& a, float& b) {
        const uint32_t off = ((d >> 6) * VD + (c >> 6)) * kRow + swizzled(d & 63, (c & 63) >> 3) + (c & 7) * 2;
        const uint32_t high = pack_bf16(a, b);
        const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high));
        *reinterpret_cast<uint32_t*>(chunk_smem + Tile::kOffS + off) = high;
        *reinterpret_cast<uint32_t*>(chunk_smem + Tile::kOffS + KD * VD * kRow + off) = pack_bf16(a - k.x, b - k.y);
      });
    }
    __syncthreads();

    float o[2][2][4];  // tokens o_tok + mt * 16 + {g, g + 8}, value dims o_col + nt * 8 + ...
    const int o_tok = (warp & 1) * 32, o_col = (warp >> 1) * 16;
    const uint32_t o_group = (o_col >> 6) * kRow;
    const int o_unit = (o_col & 63) >> 3;
    if (kEmit) {
      // A: tokens 16 (warp & 3) ..., keys from block j_blk on; blocks above the diagonal are never read.
      constexpr int kBlocks = 2 / VD;
      const int i_blk = warp & 3, j_blk = (warp >> 2) * kBlocks;
      if (j_blk <= i_blk) {
        float a[2 * kBlocks][4];
#pragma unroll
        for (int i = 0; i < 2 * kBlocks; ++i) a[i][0] = a[i][1] = a[i][2] = a[i][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < KD * 4; ++ks) {
          const uint32_t group = (ks >> 2) * kRow;
          uint32_t q[4], r[4];
          ldmatrix_x4(q[0], q[1], q[2], q[3],
                      base + Tile::kOffQ + group + swizzled(i_blk * 16 + a_row, (ks & 3) * 2 + a_sel));
#pragma unroll
          for (int np = 0; np < kBlocks; ++np) {
            if (np > 0 && j_blk + np > i_blk) break;
            ldmatrix_x4(r[0], r[1], r[2], r[3],
                        base + Tile::kOffK + group + swizzled((j_blk + np) * 16 + b_row, (ks & 3) * 2 + b_sel));
            Mma::run(a[2 * np], q[0], q[1], q[2], q[3], r[0], r[1]);
            Mma::run(a[2 * np + 1], q[0], q[1], q[2], q[3], r[2], r[3]);
          }
        }
        const int i0 = i_blk * 16 + g;
#pragma unroll
        for (int nt = 0; nt < 2 * kBlocks; ++nt) {
          const int j = j_blk * 16 + nt * 8 + 2 * t4;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int i = i0 + e * 8;
            const float x = i >= j ? a[nt][2 * e] * powers[i - j] : 0.f;
            const float y = i >= j + 1 ? a[nt][2 * e + 1] * powers[i - j - 1] : 0.f;
            const uint32_t off = Tile::kOffA + swizzled(i, j >> 3) + (j & 7) * 2, high = pack_bf16(x, y);
            const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high));
            *reinterpret_cast<uint32_t*>(chunk_smem + off) = high;
            *reinterpret_cast<uint32_t*>(chunk_smem + off + kRow) = pack_bf16(x - k.x, y - k.y);
          }
        }
      }
      // S^T q.
#pragma unroll
      for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) o[mt][nt][0] = o[mt][nt][1] = o[mt][nt][2] = o[mt][nt][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KD * 4; ++ks) {
        uint32_t q[2][4];
#pragma unroll
        for (int mt = 0; mt < 2; ++mt)
          ldmatrix_x4(q[mt][0], q[mt][1], q[mt][2], q[mt][3],
                      base + Tile::kOffQ + (ks >> 2) * kRow + swizzled(o_tok + mt * 16 + a_row, (ks & 3) * 2 + a_sel));
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          uint32_t r[4];
          ldmatrix_x4_trans(r[0], r[1], r[2], r[3],
                            base + Tile::kOffS + (part * KD + (ks >> 2)) * VD * kRow + o_group +
                                swizzled((ks & 3) * 16 + v_row, o_unit + v_sel));
#pragma unroll
          for (int mt = 0; mt < 2; ++mt) {
            Mma::run(o[mt][0], q[mt][0], q[mt][1], q[mt][2], q[mt][3], r[0], r[1]);
            Mma::run(o[mt][1], q[mt][0], q[mt][1], q[mt][2], q[mt][3], r[2], r[3]);
          }
        }
      }
#pragma unroll
      for (int mt = 0; mt < 2; ++mt) {
        const float d0 = powers[o_tok + mt * 16 + g + 1], d1 = powers[o_tok + mt * 16 + g + 9];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) o[mt][nt][0] *= d0, o[mt][nt][1] *= d0, o[mt][nt][2] *= d1, o[mt][nt][3] *= d1;
      }
    }

    // State after the tile.
    const float whole = powers[n];
    each_pair([&](int, int, float& a, float& b) {
      a *= whole;
      b *= whole;
    });
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {  // k and v past the segment are zero
      uint32_t ka[4];
      const int unit = (s_row >> 3) + at_sel;  // 16-byte unit of the key row
      ldmatrix_x4_trans(ka[0], ka[1], ka[2], ka[3],
                        base + Tile::kOffK + (unit >> 3) * kRow + swizzled(kt * 16 + at_row, unit & 7));
#pragma unroll
      for (int np = 0; np < kStateTiles / 2; ++np)
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          const int c = s_col + np * 16;
          uint32_t r[4];
          ldmatrix_x4_trans(r[0], r[1], r[2], r[3],
                            base + Tile::kOffW + (part * VD + (c >> 6)) * kRow +
                                swizzled(kt * 16 + v_row, ((c & 63) >> 3) + v_sel));
          Mma::run(s[2 * np], ka[0], ka[1], ka[2], ka[3], r[0], r[1]);
          Mma::run(s[2 * np + 1], ka[0], ka[1], ka[2], ka[3], r[2], r[3]);
        }
    }

    if (kEmit) {
      __syncthreads();  // A is complete
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt * 16 > o_tok + 16) break;
        uint32_t r[4];
        ldmatrix_x4_trans(r[0], r[1], r[2], r[3], base + Tile::kOffV + o_group + swizzled(kt * 16 + v_row, o_unit + v_sel));
#pragma unroll
        for (int mt = 0; mt < 2; ++mt) {
          if (kt * 16 > o_tok + mt * 16) continue;  // above the diagonal
#pragma unroll
          for (int part = 0; part < 2; ++part) {
            uint32_t a[4];
            ldmatrix_x4(a[0], a[1], a[2], a[3],
                        base + Tile::kOffA + part * kRow + swizzled(o_tok + mt * 16 + a_row, kt * 2 + a_sel));
            Mma::run(o[mt][0], a[0], a[1], a[2], a[3], r[0], r[1]);
            Mma::run(o[mt][1], a[0], a[1], a[2], a[3], r[2], r[3]);
          }
        }
      }
      T* out = reinterpret_cast<T*>(p.out) + tok0 * p.ldo + h * p.vdim + col0;
#pragma unroll
      for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const int c = o_col + nt * 8 + 2 * t4;
          if (col0 + c >= p.vdim) continue;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int i = o_tok + mt * 16 + g + e * 8;
            if (i < n)
              *reinterpret_cast<uint32_t*>(out + (long long)i * p.ldo + c) = pack_bf16(o[mt][nt][2 * e], o[mt][nt][2 * e + 1]);
          }
        }
    }
  }

  float* dst = kEmit ? (seg.last ? slot + head_state : nullptr) : p.carry + carry_at;
  if (dst == nullptr) return;
  each_pair([&](int d, int c, float& a, float& b) {
    if (d < p.dim && col0 + c < p.vdim)
      *reinterpret_cast<float2*>(dst + (long long)d * p.vdim + col0 + c) = make_float2(a, b);
  });
}

constexpr int kCarryBatch = 8;  // segments whose loads are in flight together

// carry[segment] <- state before the segment, from what the segments before it added.
__global__ void outer_carry_kernel(OuterParams p) {
  chain_wait();
  chain_release();
  const int r = blockIdx.x / p.heads, h = blockIdx.x % p.heads;
  const int e = blockIdx.y * blockDim.x + threadIdx.x, size = p.dim * p.vdim;
  if (e >= size) return;
  int first = 0;
  for (int i = 0; i < r; ++i) {
    const long long len = p.seg.cu_seqlens.at(i + 1) - p.seg.cu_seqlens.at(i);
    if (len > 0) first += (int)((len + p.seg.length - 1) / p.seg.length);
  }
  const long long begin = p.seg.cu_seqlens.at(r), len = p.seg.cu_seqlens.at(r + 1) - begin;
  if (len <= 0) return;
  const int pieces = (int)((len + p.seg.length - 1) / p.seg.length);
  const float* slot = p.slots.at(r);
  if (slot == nullptr) return;
  float state = p.positions.at(begin) == 0 ? 0.f : slot[(long long)h * size + e];
  const float decay = powf(p.decay[h], (float)p.seg.length);
  const long long stride = (long long)p.heads * size;
  float* at = p.carry + (long long)first * stride + (long long)h * size + e;
  for (int i0 = 0; i0 < pieces; i0 += kCarryBatch, at += kCarryBatch * stride) {
    float added[kCarryBatch];
#pragma unroll
    for (int i = 0; i < kCarryBatch; ++i) added[i] = i0 + i + 1 < pieces ? at[i * stride] : 0.f;
#pragma unroll
    for (int i = 0; i < kCarryBatch; ++i) {
      if (i0 + i >= pieces) break;
      at[i * stride] = state;
      state = decay * state + added[i];
    }
  }
}

// ---------------------------------------------------------------------------
// Gated average
// ---------------------------------------------------------------------------
struct AverageParams {
  const void* rows;  // [tokens][ld]: z | u | g, width each
  long long ld;
  const void* z_bias;
  const void* u_bias;
  void* out;  // [tokens][ldo]
  long long ldo;
  Slots slots;
  IndexView positions;
  int tokens, width;
  Segments seg;
  float* carry;  // [segments][2][width], null: every request is one segment
};

// keep = 1 - z, add = z * candidate.  The two sigmoids share one reciprocal.
__device__ __forceinline__ void average_gates(float a, float u, float* keep, float* add) {
  const float da = sigmoid_denominator(a), du = sigmoid_denominator(u);
  const float inv = reciprocal_unit(da * du);
  const float gate = inv * du;
  *keep = 1.f - gate;
  *add = gate * (u >= 0.f ? u + 0.5f : inv * da);
}

// VEC activations as they lie in memory, widened when they are used.
template <typename T, int VEC>
struct alignas(sizeof(T) * VEC) RawVec {
  T v[VEC];
  __device__ __forceinline__ static RawVec at(const T* p) { return *reinterpret_cast<const RawVec*>(p); }
  __device__ __forceinline__ void widen(float (&out)[VEC]) const {
#pragma unroll
    for (int j = 0; j < VEC; ++j) out[j] = to_float<T>(v[j]);
  }
  __device__ __forceinline__ static void load(const T* p, float (&out)[VEC]) { at(p).widen(out); }
  __device__ __forceinline__ static void store(T* p, const float (&in)[VEC]) {
    RawVec raw;
#pragma unroll
    for (int j = 0; j < VEC; ++j) raw.v[j] = from_float<T>(in[j]);
    *reinterpret_cast<RawVec*>(p) = raw;
  }
};

template <>
struct RawVec<__nv_bfloat16, 2> {  // one word, so that a batch of them costs one register each
  uint32_t word;
  __device__ __forceinline__ static RawVec at(const __nv_bfloat16* p) { return {*reinterpret_cast<const uint32_t*>(p)}; }
  __device__ __forceinline__ void widen(float (&out)[2]) const {
    out[0] = __uint_as_float(word << 16);
    out[1] = __uint_as_float(word & 0xffff0000u);
  }
  __device__ __forceinline__ static void load(const __nv_bfloat16* p, float (&out)[2]) { at(p).widen(out); }
  __device__ __forceinline__ static void store(__nv_bfloat16* p, const float (&in)[2]) {
    *reinterpret_cast<uint32_t*>(p) = pack_bf16(in[0], in[1]);
  }
};

template <typename T, int VEC>
struct AverageStep {
  float zb[VEC], ub[VEC];
  __device__ __forceinline__ AverageStep(const AverageParams& p, int c) {
    RawVec<T, VEC>::load(reinterpret_cast<const T*>(p.z_bias) + c, zb);
    RawVec<T, VEC>::load(reinterpret_cast<const T*>(p.u_bias) + c, ub);
  }
  __device__ __forceinline__ void gates(const float (&z)[VEC], const float (&u)[VEC], float (&keep)[VEC],
                                        float (&add)[VEC]) const {
#pragma unroll
    for (int j = 0; j < VEC; ++j) average_gates(z[j] + zb[j], u[j] + ub[j], &keep[j], &add[j]);
  }
};
constexpr int kAverageBatch = 4;  // tokens loaded together, a batch ahead of the one that is computed


// state * silu(g)
template <typename T, int VEC>
__device__ __forceinline__ void average_emit(const float (&g)[VEC], T* out, const float (&state)[VEC]) {
  float v[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) v[j] = state[j] * silu(g[j]);
  RawVec<T, VEC>::store(out, v);
}

template <typename T, int VEC>
__global__ void average_decode_kernel(AverageParams p) {
  chain_wait();
  chain_release();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC, row = blockIdx.x;
  if (c >= p.width) return;
  float* slot = p.slots.at(row);
  if (slot == nullptr) return;
  const T* src = reinterpret_cast<const T*>(p.rows) + (long long)row * p.ld + c;
  const AverageStep<T, VEC> step(p, c);
  float state[VEC], keep[VEC], add[VEC], z[VEC], u[VEC], g[VEC];
  RawVec<T, VEC>::load(src, z);
  RawVec<T, VEC>::load(src + p.width, u);
  RawVec<T, VEC>::load(src + 2 * p.width, g);
  if (p.positions.at(row) == 0) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) state[j] = 0.f;
  } else {
    RawVec<float, VEC>::load(slot + c, state);
  }
  step.gates(z, u, keep, add);
#pragma unroll
  for (int j = 0; j < VEC; ++j) state[j] = keep[j] * state[j] + add[j];
  RawVec<float, VEC>::store(slot + c, state);
  average_emit<T, VEC>(g, reinterpret_cast<T*>(p.out) + (long long)row * p.ldo + c, state);
}

// What a segment does to a state before it: S -> product S + sum.
template <typename T, int VEC>
__global__ void __launch_bounds__(128, 8) average_summary_kernel(AverageParams p) {
  chain_wait();
  chain_release();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  Segment seg;
  if (c >= p.width || !p.seg.find(blockIdx.x, &seg) || seg.last) return;
  const AverageStep<T, VEC> step(p, c);
  float product[VEC], sum[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) product[j] = 1.f, sum[j] = 0.f;
  const T* src = reinterpret_cast<const T*>(p.rows) + seg.begin * p.ld + c;
  const int count = (int)(seg.end - seg.begin);
  struct Batch {
    RawVec<T, VEC> z[kAverageBatch], u[kAverageBatch];
  } batches[2];
  auto fetch = [&](int t0, Batch& to) {
#pragma unroll
    for (int i = 0; i < kAverageBatch; ++i)
      if (t0 + i < count) {
        to.z[i] = RawVec<T, VEC>::at(src + (t0 + i) * p.ld);
        to.u[i] = RawVec<T, VEC>::at(src + (t0 + i) * p.ld + p.width);
      }
  };
  auto advance = [&](int t0, const Batch& from) {
#pragma unroll
    for (int i = 0; i < kAverageBatch; ++i) {
      if (t0 + i >= count) break;
      float keep[VEC], add[VEC], a[VEC], b[VEC];
      from.z[i].widen(a);
      from.u[i].widen(b);
      step.gates(a, b, keep, add);
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        product[j] *= keep[j];
        sum[j] = keep[j] * sum[j] + add[j];
      }
    }
  };
  fetch(0, batches[0]);
  for (int t0 = 0; t0 < count; t0 += 2 * kAverageBatch) {
    fetch(t0 + kAverageBatch, batches[1]);
    advance(t0, batches[0]);
    fetch(t0 + 2 * kAverageBatch, batches[0]);
    advance(t0 + kAverageBatch, batches[1]);
  }
  float* dst = p.carry + (long long)blockIdx.x * 2 * p.width + c;
  RawVec<float, VEC>::store(dst, product);
  RawVec<float, VEC>::store(dst + p.width, sum);
}

// carry[segment][0] <- state before the segment.
__global__ void average_carry_kernel(AverageParams p) {
  chain_wait();
  chain_release();
  const int r = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.width) return;
  int first = 0;
  for (int i = 0; i < r; ++i) {
    const long long len = p.seg.cu_seqlens.at(i + 1) - p.seg.cu_seqlens.at(i);
    if (len > 0) first += (int)((len + p.seg.length - 1) / p.seg.length);
  }
  const long long begin = p.seg.cu_seqlens.at(r), len = p.seg.cu_seqlens.at(r + 1) - begin;
  if (len <= 0) return;
  const int pieces = (int)((len + p.seg.length - 1) / p.seg.length);
  const float* slot = p.slots.at(r);
  if (slot == nullptr) return;
  float state = p.positions.at(begin) == 0 ? 0.f : slot[c];
  float* at = p.carry + (long long)first * 2 * p.width + c;
  for (int i0 = 0; i0 < pieces; i0 += kCarryBatch, at += (long long)kCarryBatch * 2 * p.width) {
    float product[kCarryBatch], sum[kCarryBatch];
#pragma unroll
    for (int i = 0; i < kCarryBatch; ++i) {
      const bool more = i0 + i + 1 < pieces;
      product[i] = more ? at[(long long)i * 2 * p.width] : 0.f;
      sum[i] = more ? at[(long long)i * 2 * p.width + p.width] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < kCarryBatch; ++i) {
      if (i0 + i >= pieces) break;
      at[(long long)i * 2 * p.width] = state;
      state = product[i] * state + sum[i];
    }
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(128, 8) average_segment_kernel(AverageParams p) {
  chain_wait();
  chain_release();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  Segment seg;
  if (c >= p.width || !p.seg.find(blockIdx.x, &seg)) return;
  float* slot = p.slots.at(seg.request);
  if (slot == nullptr) return;
  const AverageStep<T, VEC> step(p, c);
  float state[VEC];
  if (p.carry != nullptr) {
    RawVec<float, VEC>::load(p.carry + (long long)blockIdx.x * 2 * p.width + c, state);
  } else if (p.positions.at(seg.begin) == 0) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) state[j] = 0.f;
  } else {
    RawVec<float, VEC>::load(slot + c, state);
  }
  const T* src = reinterpret_cast<const T*>(p.rows) + seg.begin * p.ld + c;
  T* out = reinterpret_cast<T*>(p.out) + seg.begin * p.ldo + c;
  const int count = (int)(seg.end - seg.begin);
  struct Batch {
    RawVec<T, VEC> z[kAverageBatch], u[kAverageBatch], g[kAverageBatch];
  } batches[2];
  auto fetch = [&](int t0, Batch& to) {
#pragma unroll
    for (int i = 0; i < kAverageBatch; ++i)
      if (t0 + i < count) {
        to.z[i] = RawVec<T, VEC>::at(src + (t0 + i) * p.ld);
        to.u[i] = RawVec<T, VEC>::at(src + (t0 + i) * p.ld + p.width);
        to.g[i] = RawVec<T, VEC>::at(src + (t0 + i) * p.ld + 2 * p.width);
      }
  };
  auto advance = [&](int t0, const Batch& from) {
#pragma unroll
    for (int i = 0; i < kAverageBatch; ++i) {
      if (t0 + i >= count) break;
      float keep[VEC], add[VEC], a[VEC], b[VEC];
      from.z[i].widen(a);
      from.u[i].widen(b);
      step.gates(a, b, keep, add);
#pragma unroll
      for (int j = 0; j < VEC; ++j) state[j] = keep[j] * state[j] + add[j];
      from.g[i].widen(a);
      average_emit<T, VEC>(a, out + (t0 + i) * p.ldo, state);
    }
  };
  fetch(0, batches[0]);
  for (int t0 = 0; t0 < count; t0 += 2 * kAverageBatch) {
    fetch(t0 + kAverageBatch, batches[1]);
    advance(t0, batches[0]);
    fetch(t0 + 2 * kAverageBatch, batches[0]);
    advance(t0 + kAverageBatch, batches[1]);
  }
  if (seg.last) RawVec<float, VEC>::store(slot + c, state);
}

// ---------------------------------------------------------------------------
// Host
// ---------------------------------------------------------------------------
template <typename K>
int allow_smem(K kernel, int bytes) {
  if (bytes > 48 * 1024) MIE_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
  return MIE_OK;
}

template <typename T>
int launch_outer_decode(const OuterParams& p, int vec, cudaStream_t stream) {
  const size_t smem = (size_t)(2 * p.dim + kOuterWarps * 32 * vec) * sizeof(float);
  const dim3 grid((unsigned)(p.tokens * p.heads), (unsigned)((p.vdim + 32 * vec - 1) / (32 * vec)));
  MIE_CUDA(vec == 4 ? launch_chained(outer_decode_kernel<T, 4>, grid, dim3(kOuterWarps * 32), smem, stream, p)
                    : launch_chained(outer_decode_kernel<T, 1>, grid, dim3(kOuterWarps * 32), smem, stream, p));
  MIE_LAUNCH_CHECK("outer_decode_kernel");
  return MIE_OK;
}

template <typename T>
int launch_outer_rows(const OuterParams& p, cudaStream_t stream) {
  const int smem = (2 * p.dim + kOuterWarps * 32 + 32 * p.dim) * (int)sizeof(float);
  if (int rc = allow_smem(outer_rows_kernel<T>, smem)) return rc;
  const dim3 grid((unsigned)(p.seg.requests * p.heads), (unsigned)((p.vdim + 31) / 32));
  MIE_CUDA(launch_chained(outer_rows_kernel<T>, grid, dim3(kOuterWarps * 32), (size_t)smem, stream, p));
  MIE_LAUNCH_CHECK("outer_rows_kernel");
  return MIE_OK;
}

template <int KD, int VD>
int launch_outer_chunks(const OuterParams& p, int segments, cudaStream_t stream) {
  constexpr int smem = OuterTile<KD, VD>::kSmem;
  const dim3 grid((unsigned)segments, (unsigned)p.heads, (unsigned)((p.vdim + VD * 64 - 1) / (VD * 64)));
  const dim3 block(OuterTile<KD, VD>::kThreads);
  if (p.carry != nullptr) {
    if (int rc = allow_smem(outer_chunk_kernel<KD, VD, false>, smem)) return rc;
    MIE_CUDA(launch_chained(outer_chunk_kernel<KD, VD, false>, grid, block, (size_t)smem, stream, p));
    MIE_LAUNCH_CHECK("outer_chunk_kernel");
    const dim3 flat((unsigned)(p.seg.requests * p.heads), (unsigned)((p.dim * p.vdim + 255) / 256));
    MIE_CUDA(launch_chained(outer_carry_kernel, flat, dim3(256), 0, stream, p));
    MIE_LAUNCH_CHECK("outer_carry_kernel");
  }
  if (int rc = allow_smem(outer_chunk_kernel<KD, VD, true>, smem)) return rc;
  MIE_CUDA(launch_chained(outer_chunk_kernel<KD, VD, true>, grid, block, (size_t)smem, stream, p));
  MIE_LAUNCH_CHECK("outer_chunk_kernel");
  return MIE_OK;
}

template <typename T, int VEC>
int launch_average(const AverageParams& p, bool decode, int segments, cudaStream_t stream) {
  const int threads = 128, per_block = threads * VEC;
  const unsigned columns = (unsigned)((p.width + per_block - 1) / per_block);
  if (decode) {
    MIE_CUDA(launch_chained(average_decode_kernel<T, VEC>, dim3((unsigned)p.tokens, columns), dim3(threads), 0, stream, p));
    MIE_LAUNCH_CHECK("average_decode_kernel");
    return MIE_OK;
  }
  const dim3 grid((unsigned)segments, columns);
  if (p.carry != nullptr) {
    MIE_CUDA(launch_chained(average_summary_kernel<T, VEC>, grid, dim3(threads), 0, stream, p));
    MIE_LAUNCH_CHECK("average_summary_kernel");
    MIE_CUDA(launch_chained(average_carry_kernel, dim3((unsigned)p.seg.requests, (unsigned)((p.width + 127) / 128)),
                            dim3(128), 0, stream, p));
    MIE_LAUNCH_CHECK("average_carry_kernel");
  }
  MIE_CUDA(launch_chained(average_segment_kernel<T, VEC>, grid, dim3(threads), 0, stream, p));
  MIE_LAUNCH_CHECK("average_segment_kernel");
  return MIE_OK;
}

Slots make_slots(float* state, int64_t stride, const mie_index_t& slots, int count, int* status) {
  Slots out;
  out.state = state;
  out.stride = stride;
  out.slots = IndexView(slots);
  out.count = count;
  out.status = status;
  return out;
}

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_outer_recurrence_chunked(int32_t dim, int32_t value_dim, int32_t dtype) {
  return dtype == MIE_DTYPE_BF16 && dim >= 8 && dim <= 128 && dim % 8 == 0 && value_dim >= 8 && value_dim % 8 == 0;
}

extern "C" int mie_outer_recurrence(const void* rows, int64_t ld, const float* decay, void* out, int64_t ldo,
                                    float* state, int64_t slot_stride, int32_t num_slots, mie_index_t slots,
                                    mie_index_t positions, mie_index_t cu_seqlens, int32_t requests,
                                    int32_t segment_tokens, float* carry, int64_t carry_floats, int32_t tokens,
                                    int32_t heads, int32_t dim, int32_t value_dim, int32_t dtype, int32_t* status,
                                    void* stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(rows && decay && out && state && slots.ptr && positions.ptr, "null pointer");
  MIE_CHECK_ARG(tokens >= 0 && heads >= 1 && dim >= 1 && dim <= 1024 && value_dim >= 1 && num_slots >= 1,
                "invalid sizes");
  if (tokens == 0) return MIE_OK;
  OuterParams p;
  p.rows = rows;
  p.ld = ld;
  p.decay = decay;
  p.out = out;
  p.ldo = ldo;
  p.slots = make_slots(state, slot_stride, slots, num_slots, status);
  p.positions = IndexView(positions);
  p.tokens = tokens;
  p.heads = heads;
  p.dim = dim;
  p.vdim = value_dim;
  p.seg.cu_seqlens = IndexView(cu_seqlens);
  p.seg.requests = requests;
  p.seg.length = segment_tokens > 0 ? segment_tokens : 0x40000000;
  p.carry = nullptr;
  if (!cu_seqlens.ptr) {  // one token per request
    const int act = dtype == MIE_DTYPE_BF16 ? 8 : 16;
    const bool vec = value_dim % 4 == 0 && (2 * heads * dim) % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 &&
                     slot_stride % 4 == 0 && aligned(rows, act) && aligned(out, act) && aligned(state, 16);
    if (dtype == MIE_DTYPE_BF16) return launch_outer_decode<__nv_bfloat16>(p, vec ? 4 : 1, stream);
    return launch_outer_decode<float>(p, vec ? 4 : 1, stream);
  }
  MIE_CHECK_ARG(requests >= 0 && segment_tokens >= 0, "invalid sizes");
  if (requests == 0) return MIE_OK;
  const bool chunked = mie_outer_recurrence_chunked(dim, value_dim, dtype) && ld % 8 == 0 && ldo % 2 == 0 &&
                       slot_stride % 2 == 0 && aligned(rows, 16) && aligned(out, 4) && aligned(state, 8);
  if (!chunked) {
    if (dtype == MIE_DTYPE_BF16) return launch_outer_rows<__nv_bfloat16>(p, stream);
    return launch_outer_rows<float>(p, stream);
  }
  int segments = requests;
  if (carry != nullptr && segment_tokens > 0) {
    segments = tokens / segment_tokens + requests;
    MIE_CHECK_ARG(segment_tokens % kOuterTokens == 0 && aligned(carry, 16), "segments are whole 64-token tiles");
    MIE_CHECK_ARG(carry_floats >= (long long)segments * heads * dim * value_dim, "the carry buffer is too small");
    p.carry = carry;
  } else {
    p.seg.length = 0x40000000;
  }
  if (value_dim <= 64)
    return dim <= 64 ? launch_outer_chunks<1, 1>(p, segments, stream) : launch_outer_chunks<2, 1>(p, segments, stream);
  return dim <= 64 ? launch_outer_chunks<1, 2>(p, segments, stream) : launch_outer_chunks<2, 2>(p, segments, stream);
}

extern "C" int mie_gated_average(const void* rows, int64_t ld, const void* z_bias, const void* u_bias, void* out,
                                 int64_t ldo, float* state, int64_t slot_stride, int32_t num_slots, mie_index_t slots,
                                 mie_index_t positions, mie_index_t cu_seqlens, int32_t requests,
                                 int32_t segment_tokens, float* carry, int64_t carry_floats, int32_t tokens,
                                 int32_t width, int32_t dtype, int32_t* status, void* stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  MIE_CHECK_ACT_DTYPE(dtype);
  MIE_CHECK_ARG(rows && z_bias && u_bias && out && state && slots.ptr && positions.ptr, "null pointer");
  MIE_CHECK_ARG(tokens >= 0 && width >= 1 && num_slots >= 1 && requests >= 0 && segment_tokens >= 0, "invalid sizes");
  const bool decode = !cu_seqlens.ptr;
  if (tokens == 0 || (!decode && requests == 0)) return MIE_OK;
  AverageParams p;
  p.rows = rows;
  p.ld = ld;
  p.z_bias = z_bias;
  p.u_bias = u_bias;
  p.out = out;
  p.ldo = ldo;
  p.slots = make_slots(state, slot_stride, slots, num_slots, status);
  p.positions = IndexView(positions);
  p.tokens = tokens;
  p.width = width;
  p.seg.cu_seqlens = IndexView(cu_seqlens);
  p.seg.requests = requests;
  p.seg.length = 0x40000000;
  p.carry = nullptr;
  int segments = requests;
  if (!decode && carry != nullptr && segment_tokens > 0) {
    segments = tokens / segment_tokens + requests;
    MIE_CHECK_ARG(carry_floats >= (long long)segments * 2 * width, "the carry buffer is too small");
    p.seg.length = segment_tokens;
    p.carry = carry;
  }
  const int act = dtype == MIE_DTYPE_BF16 ? 4 : 8;  // bytes of two activations
  const bool vec = width % 2 == 0 && ld % 2 == 0 && ldo % 2 == 0 && slot_stride % 2 == 0 && aligned(rows, act) &&
                   aligned(z_bias, act) && aligned(u_bias, act) && aligned(out, act) && aligned(state, 8) &&
                   aligned(carry, 8);
  if (dtype == MIE_DTYPE_BF16)
    return vec ? launch_average<__nv_bfloat16, 2>(p, decode, segments, stream)
               : launch_average<__nv_bfloat16, 1>(p, decode, segments, stream);
  return vec ? launch_average<float, 2>(p, decode, segments, stream)
             : launch_average<float, 1>(p, decode, segments, stream);
}
