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

__device__ __forceinline__ float sigmoid(float v) { return __fdividef(1.f, 1.f + expf(-v)); }
__device__ __forceinline__ float silu(float v) { return __fdividef(v, 1.f + expf(-v)); }
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoid(u); }

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

// The chunked form on tensor cores (bf16): one CTA per (segment, head, 64 value dims) walks its segment 64 tokens at
// a time with the state in registers.  With q, k, v of 64 tokens and the state S before them,
//
//   o_i  = decay^(i+1) S^T q_i + sum_(j <= i) decay^(i-j) (q_i . k_j) v_j
//   S   <- decay^n S + sum_j k_j (decay^(n-1-j) v_j)^T
//
// q, k, v are the bf16 activations; S, the decayed products and the decayed v enter as a rounded part plus its
// remainder (two MMAs), sums are fp32.  Four warps: warp w owns tokens 16w..16w+15 of the output and a quarter of the
// key dims of the state.
constexpr int kOuterTokens = 64;
constexpr int kOuterCols = 64;

template <int KD>  // 64-dim groups of a key row
struct OuterTile {
  static constexpr int kRow = 8192;  // 64 rows x 64 bf16, 128-byte rows, 16-byte units XOR-swizzled by row
  static constexpr int kOffQ = 0;
  static constexpr int kOffK = kOffQ + KD * kRow;
  static constexpr int kOffV = kOffK + KD * kRow;
  static constexpr int kOffW = kOffV + kRow;           // decayed v: rounded part, remainder
  static constexpr int kOffS = kOffW + 2 * kRow;       // state: rounded part, remainder
  static constexpr int kOffPow = kOffS + 2 * KD * kRow;
  static constexpr int kSmem = kOffPow + 80 * 4;
};

__device__ __forceinline__ uint32_t swizzled(int row, int unit) { return row * 128 + ((unit ^ (row & 7)) << 4); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) { return Mma16816<__nv_bfloat16>::pack(lo, hi); }

template <int KD, bool kEmit>
__global__ void __launch_bounds__(128) outer_chunk_kernel(OuterParams p) {
  using Tile = OuterTile<KD>;
  using T = __nv_bfloat16;
  using Mma = Mma16816<T>;
  extern __shared__ __align__(1024) uint8_t chunk_smem[];
  float* powers = reinterpret_cast<float*>(chunk_smem + Tile::kOffPow);
  const uint32_t base = smem_u32(chunk_smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, col0 = blockIdx.z * kOuterCols;
  chain_wait();
  chain_release();
  Segment seg;
  if (!p.seg.find(blockIdx.x, &seg)) return;
  if (!kEmit && seg.last) return;  // nobody needs what the last segment adds
  float* slot = p.slots.at(seg.request);
  if (slot == nullptr) return;
  const float decay = p.decay[h];
  if (tid <= kOuterTokens) powers[tid] = powf(decay, (float)tid);

  // State rows of this warp: m-tile mt covers key dims (warp * KD + mt) * 16 + {g, g + 8}.
  float s[KD][8][4];
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
    for (int mt = 0; mt < KD; ++mt)
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half)
          visit((warp * KD + mt) * 16 + g + half * 8, nt * 8 + 2 * t4, s[mt][nt][2 * half], s[mt][nt][2 * half + 1]);
  };
  each_pair([&](int d, int c, float& a, float& b) {
    a = b = 0.f;
    if (init != nullptr && d < p.dim && col0 + c < p.vdim) {
      const float2 v = *reinterpret_cast<const float2*>(init + (long long)d * p.vdim + col0 + c);
      a = v.x;
      b = v.y;
    }
  });

  // ldmatrix lane geometry: plain B operand ([n][k] rows), transposed B operand ([k][n] rows), transposed A operand.
  const int b_row = (lane & 7) + ((lane >> 4) & 1) * 8, b_sel = (lane >> 3) & 1;
  const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_sel = (lane >> 4) & 1;
  const int at_row = (lane & 7) + ((lane >> 4) & 1) * 8, at_sel = (lane >> 3) & 1;
  const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_sel = (lane >> 4) & 1;

  for (long long tok0 = seg.begin; tok0 < seg.end; tok0 += kOuterTokens) {
    const int n = (int)(seg.end - tok0 < kOuterTokens ? seg.end - tok0 : kOuterTokens);
    __syncthreads();  // the previous tile has been read (first pass: the powers are there)
    const T* rows = reinterpret_cast<const T*>(p.rows) + tok0 * p.ld;
    // q and k through silu; rows past the segment and dims past the head are zero.
    for (int i = tid; i < kOuterTokens * KD * 8; i += 128) {
      const int r = i / (KD * 8), u = i % (KD * 8);
      const bool in = r < n && u * 8 < p.dim;
      uint32_t kq[2][4];
#pragma unroll
      for (int which = kEmit ? 0 : 1; which < 2; ++which) {
        float v[8];
        if (in) {
          Vec<T, 8>::load(rows + (long long)r * p.ld + (which * p.heads + h) * p.dim + u * 8, v);
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) v[j] = 0.f;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) kq[which][j] = pack_bf16(silu(v[2 * j]), silu(v[2 * j + 1]));
        *reinterpret_cast<uint4*>(chunk_smem + (which == 0 ? Tile::kOffQ : Tile::kOffK) + (u >> 3) * Tile::kRow +
                                  swizzled(r, u & 7)) =
            make_uint4(kq[which][0], kq[which][1], kq[which][2], kq[which][3]);
      }
    }
    for (int i = tid; i < kOuterTokens * 8; i += 128) {
      const int r = i / 8, u = i % 8;
      float v[8];
      if (r < n && col0 + u * 8 < p.vdim) {
        Vec<T, 8>::load(rows + (long long)r * p.ld + 2 * p.heads * p.dim + h * p.vdim + col0 + u * 8, v);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = 0.f;
      }
      const float weight = r < n ? powers[n - 1 - r] : 0.f;
      uint32_t whole[4], high[4], low[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float a = round_bf16(silu(v[2 * j])), b = round_bf16(silu(v[2 * j + 1]));
        const float wa = a * weight, wb = b * weight;
        whole[j] = pack_bf16(a, b);
        high[j] = pack_bf16(wa, wb);
        low[j] = pack_bf16(wa - round_bf16(wa), wb - round_bf16(wb));
      }
      const uint32_t off = swizzled(r, u);
      *reinterpret_cast<uint4*>(chunk_smem + Tile::kOffV + off) = make_uint4(whole[0], whole[1], whole[2], whole[3]);
      *reinterpret_cast<uint4*>(chunk_smem + Tile::kOffW + off) = make_uint4(high[0], high[1], high[2], high[3]);
      *reinterpret_cast<uint4*>(chunk_smem + Tile::kOffW + Tile::kRow + off) = make_uint4(low[0], low[1], low[2], low[3]);
    }
    if (kEmit) {
      each_pair([&](int d, int c, float& a, float& b) {
        const uint32_t off = (d >> 6) * Tile::kRow + swizzled(d & 63, c >> 3) + (c & 7) * 2;
        *reinterpret_cast<uint32_t*>(chunk_smem + Tile::kOffS + off) = pack_bf16(a, b);
        *reinterpret_cast<uint32_t*>(chunk_smem + Tile::kOffS + KD * Tile::kRow + off) =
            pack_bf16(a - round_bf16(a), b - round_bf16(b));
      });
    }
    __syncthreads();

    if (kEmit && warp * 16 < n) {
      float o[8][4], a[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = a[i][j] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KD * 4; ++ks) {
        if (ks * 16 >= p.dim) break;
        const uint32_t group = (ks >> 2) * Tile::kRow;
        uint32_t q0, q1, q2, q3;
        ldmatrix_x4(q0, q1, q2, q3, base + Tile::kOffQ + group + swizzled(warp * 16 + a_row, (ks & 3) * 2 + a_sel));
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t r0, r1, r2, r3;
          if (np <= warp) {  // q . k, tokens up to this warp's
            ldmatrix_x4(r0, r1, r2, r3, base + Tile::kOffK + group + swizzled(np * 16 + b_row, (ks & 3) * 2 + b_sel));
            Mma::run(a[2 * np], q0, q1, q2, q3, r0, r1);
            Mma::run(a[2 * np + 1], q0, q1, q2, q3, r2, r3);
          }
#pragma unroll
          for (int part = 0; part < 2; ++part) {  // S^T q
            ldmatrix_x4_trans(r0, r1, r2, r3, base + Tile::kOffS + part * KD * Tile::kRow + group +
                                                  swizzled((ks & 3) * 16 + v_row, np * 2 + v_sel));
            Mma::run(o[2 * np], q0, q1, q2, q3, r0, r1);
            Mma::run(o[2 * np + 1], q0, q1, q2, q3, r2, r3);
          }
        }
      }
      const int i0 = warp * 16 + g, i1 = i0 + 8;
      const float d0 = powers[i0 + 1], d1 = powers[i1 + 1];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        o[nt][0] *= d0, o[nt][1] *= d0, o[nt][2] *= d1, o[nt][3] *= d1;
        const int j = nt * 8 + 2 * t4;
        a[nt][0] = i0 >= j ? a[nt][0] * powers[i0 - j] : 0.f;
        a[nt][1] = i0 >= j + 1 ? a[nt][1] * powers[i0 - j - 1] : 0.f;
        a[nt][2] = i1 >= j ? a[nt][2] * powers[i1 - j] : 0.f;
        a[nt][3] = i1 >= j + 1 ? a[nt][3] * powers[i1 - j - 1] : 0.f;
      }
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt > warp) break;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = a[2 * kt + (e >> 1)][(e & 1) * 2], y = a[2 * kt + (e >> 1)][(e & 1) * 2 + 1];
          hi[e] = pack_bf16(x, y);
          lo[e] = pack_bf16(x - round_bf16(x), y - round_bf16(y));
        }
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t r0, r1, r2, r3;
          ldmatrix_x4_trans(r0, r1, r2, r3, base + Tile::kOffV + swizzled(kt * 16 + v_row, np * 2 + v_sel));
          Mma::run(o[2 * np], hi[0], hi[1], hi[2], hi[3], r0, r1);
          Mma::run(o[2 * np + 1], hi[0], hi[1], hi[2], hi[3], r2, r3);
          Mma::run(o[2 * np], lo[0], lo[1], lo[2], lo[3], r0, r1);
          Mma::run(o[2 * np + 1], lo[0], lo[1], lo[2], lo[3], r2, r3);
        }
      }
      T* out = reinterpret_cast<T*>(p.out) + tok0 * p.ldo + h * p.vdim + col0;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const int c = nt * 8 + 2 * t4;
        if (col0 + c >= p.vdim) break;
        if (i0 < n) *reinterpret_cast<uint32_t*>(out + (long long)i0 * p.ldo + c) = pack_bf16(o[nt][0], o[nt][1]);
        if (i1 < n) *reinterpret_cast<uint32_t*>(out + (long long)i1 * p.ldo + c) = pack_bf16(o[nt][2], o[nt][3]);
      }
    }

    // State after the tile.
    const float whole = powers[n];
    each_pair([&](int, int, float& a, float& b) {
      a *= whole;
      b *= whole;
    });
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt * 16 >= n) break;
      uint32_t ka[KD][4];
#pragma unroll
      for (int mt = 0; mt < KD; ++mt) {
        const int unit = (warp * KD + mt) * 2 + at_sel;  // 16-byte unit of the key row
        ldmatrix_x4_trans(ka[mt][0], ka[mt][1], ka[mt][2], ka[mt][3],
                          base + Tile::kOffK + (unit >> 3) * Tile::kRow + swizzled(kt * 16 + at_row, unit & 7));
      }
#pragma unroll
      for (int np = 0; np < 4; ++np)
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          uint32_t r0, r1, r2, r3;
          ldmatrix_x4_trans(r0, r1, r2, r3,
                            base + Tile::kOffW + part * Tile::kRow + swizzled(kt * 16 + v_row, np * 2 + v_sel));
#pragma unroll
          for (int mt = 0; mt < KD; ++mt) {
            Mma::run(s[mt][2 * np], ka[mt][0], ka[mt][1], ka[mt][2], ka[mt][3], r0, r1);
            Mma::run(s[mt][2 * np + 1], ka[mt][0], ka[mt][1], ka[mt][2], ka[mt][3], r2, r3);
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
  for (int i = 0; i < pieces; ++i) {
    float* at = p.carry + ((long long)(first + i) * p.heads + h) * size + e;
    const float added = i + 1 < pieces ? *at : 0.f;
    *at = state;
    state = decay * state + added;
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

template <typename T, int VEC>
struct AverageStep {
  float zb[VEC], ub[VEC];
  __device__ __forceinline__ AverageStep(const AverageParams& p, int c) {
    Vec<T, VEC>::load(reinterpret_cast<const T*>(p.z_bias) + c, zb);
    Vec<T, VEC>::load(reinterpret_cast<const T*>(p.u_bias) + c, ub);
  }
  // keep = 1 - z, add = z * candidate
  __device__ __forceinline__ void gates(const T* row, int width, float (&keep)[VEC], float (&add)[VEC]) const {
    float z[VEC], u[VEC];
    Vec<T, VEC>::load(row, z);
    Vec<T, VEC>::load(row + width, u);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const float gate = sigmoid(z[j] + zb[j]);
      keep[j] = 1.f - gate;
      add[j] = gate * gru_candidate(u[j] + ub[j]);
    }
  }
};

template <typename T, int VEC>
__device__ __forceinline__ void average_emit(const T* row, int width, T* out, const float (&state)[VEC]) {
  float g[VEC];
  Vec<T, VEC>::load(row + 2 * width, g);
#pragma unroll
  for (int j = 0; j < VEC; ++j) g[j] = state[j] * silu(g[j]);
  Vec<T, VEC>::store(out, g);
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
  float state[VEC], keep[VEC], add[VEC];
  if (p.positions.at(row) == 0) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) state[j] = 0.f;
  } else {
    Vec<float, VEC>::load(slot + c, state);
  }
  step.gates(src, p.width, keep, add);
#pragma unroll
  for (int j = 0; j < VEC; ++j) state[j] = keep[j] * state[j] + add[j];
  Vec<float, VEC>::store(slot + c, state);
  average_emit<T, VEC>(src, p.width, reinterpret_cast<T*>(p.out) + (long long)row * p.ldo + c, state);
}

// What a segment does to a state before it: S -> product S + sum.
template <typename T, int VEC>
__global__ void average_summary_kernel(AverageParams p) {
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
#pragma unroll 8
  for (long long t = seg.begin; t < seg.end; ++t, src += p.ld) {
    float keep[VEC], add[VEC];
    step.gates(src, p.width, keep, add);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      product[j] *= keep[j];
      sum[j] = keep[j] * sum[j] + add[j];
    }
  }
  float* dst = p.carry + (long long)blockIdx.x * 2 * p.width + c;
  Vec<float, VEC>::store(dst, product);
  Vec<float, VEC>::store(dst + p.width, sum);
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
#pragma unroll 8
  for (int i = 0; i < pieces; ++i, at += 2 * p.width) {
    const float product = i + 1 < pieces ? at[0] : 0.f, sum = i + 1 < pieces ? at[p.width] : 0.f;
    at[0] = state;
    state = product * state + sum;
  }
}

template <typename T, int VEC>
__global__ void average_segment_kernel(AverageParams p) {
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
    Vec<float, VEC>::load(p.carry + (long long)blockIdx.x * 2 * p.width + c, state);
  } else if (p.positions.at(seg.begin) == 0) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) state[j] = 0.f;
  } else {
    Vec<float, VEC>::load(slot + c, state);
  }
  const T* src = reinterpret_cast<const T*>(p.rows) + seg.begin * p.ld + c;
  T* out = reinterpret_cast<T*>(p.out) + seg.begin * p.ldo + c;
#pragma unroll 4
  for (long long t = seg.begin; t < seg.end; ++t, src += p.ld, out += p.ldo) {
    float keep[VEC], add[VEC];
    step.gates(src, p.width, keep, add);
#pragma unroll
    for (int j = 0; j < VEC; ++j) state[j] = keep[j] * state[j] + add[j];
    average_emit<T, VEC>(src, p.width, out, state);
  }
  if (seg.last) Vec<float, VEC>::store(slot + c, state);
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

template <int KD>
int launch_outer_chunks(const OuterParams& p, int segments, cudaStream_t stream) {
  constexpr int smem = OuterTile<KD>::kSmem;
  const dim3 grid((unsigned)segments, (unsigned)p.heads, (unsigned)((p.vdim + kOuterCols - 1) / kOuterCols));
  if (p.carry != nullptr) {
    if (int rc = allow_smem(outer_chunk_kernel<KD, false>, smem)) return rc;
    MIE_CUDA(launch_chained(outer_chunk_kernel<KD, false>, grid, dim3(128), (size_t)smem, stream, p));
    MIE_LAUNCH_CHECK("outer_chunk_kernel");
    const dim3 flat((unsigned)(p.seg.requests * p.heads), (unsigned)((p.dim * p.vdim + 255) / 256));
    MIE_CUDA(launch_chained(outer_carry_kernel, flat, dim3(256), 0, stream, p));
    MIE_LAUNCH_CHECK("outer_carry_kernel");
  }
  if (int rc = allow_smem(outer_chunk_kernel<KD, true>, smem)) return rc;
  MIE_CUDA(launch_chained(outer_chunk_kernel<KD, true>, grid, dim3(128), (size_t)smem, stream, p));
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
  return dim <= 64 ? launch_outer_chunks<1>(p, segments, stream) : launch_outer_chunks<2>(p, segments, stream);
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
  const int act = dtype == MIE_DTYPE_BF16 ? 8 : 16;
  const bool vec = width % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && slot_stride % 4 == 0 && aligned(rows, act) &&
                   aligned(z_bias, act) && aligned(u_bias, act) && aligned(out, act) && aligned(state, 16) &&
                   aligned(carry, 16);
  if (dtype == MIE_DTYPE_BF16)
    return vec ? launch_average<__nv_bfloat16, 4>(p, decode, segments, stream)
               : launch_average<__nv_bfloat16, 1>(p, decode, segments, stream);
  return vec ? launch_average<float, 4>(p, decode, segments, stream)
             : launch_average<float, 1>(p, decode, segments, stream);
}
