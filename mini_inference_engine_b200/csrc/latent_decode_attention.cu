// Ragged paged decode attention over a latent cache: one cached row per token, read by every query head.  The key of
// a token is its whole row (latent | rotated part), the value the row's first `vdim` entries, so a row is fetched
// once for both products and for all heads.
//
// One persistent CTA per SM walks (request, chunk, group of heads) items of the shared split-KV plan in a fixed
// order: a producer warp streams 16-token slabs of the request's pages into a ring of 64-token stages with TMA
// (128-byte swizzle, no multicast) and runs ahead across items; eight warps compute on a stage together:
//   S = Q K^T    warp = (16 heads, 16 * MT keys, every other 16 dims); with one 16-head tile Q stays in registers.  The
//                pair that shares keys swaps halves of its sums               -> row maxima meet in shared memory
//   P            exp2 against the common running maximum, as a rounded bf16 part plus its remainder, to shared memory
//   O += P V     warp = one 64-dim box of the values, all heads, V read transposed from the same stage
// Scores, weights, sums and O are fp32.  The sink opens the running maximum and the denominator of a request's first
// chunk; partials are merged by merge_rows_kernel.
#include "decode_attention.cuh"

namespace mie {

// Defined in prefill_attention_umma.cu: cached 5-D slab map over pages [page, head, token, dim] (dim a multiple of
// 64) whose box is 16 tokens x `box_groups` 64-dim groups, and whether a page layout allows it.
int page_slab_map(const mie_view4_t& pages, int num_blocks, int kv_heads, int block_size, int dim, int box_groups,
                  int dtype, CUtensorMap* out);
bool pages_fit_slab_map(const mie_view4_t& v, int block_size, int dim);

namespace {

constexpr int kStageTokens = 64;
constexpr int kRing = 2;
constexpr int kComputeWarps = 8;
constexpr int kLatentThreads = (kComputeWarps + 1) * 32;
constexpr int kMaxKeyBoxes = 10;

struct LatentParams {
  const char* q;
  long long q_row, q_head;
  char* out;
  long long o_row, o_head;
  IndexView tables, lengths;
  Scratch sc;
  int batch, heads, block_size, num_blocks, table_width, dim, vdim, key_boxes, head_groups, slab;
  float scale_log2;
  long long window;
  const float* sinks;
  int* status;
};

// Shared memory: K ring | Q | P (rounded, remainder) | swapped sums | row maxima | row sums | barriers.
struct LatentLayout {
  int stage, q, p, swap, maxima, sums, bars, total;
};
__host__ __device__ inline LatentLayout latent_layout(int key_boxes, int mt) {
  LatentLayout l;
  l.stage = key_boxes * kStageTokens * 128;
  l.q = kRing * l.stage;
  l.p = l.q + key_boxes * mt * 16 * 128;
  l.swap = l.p + 2 * mt * 16 * 128;
  l.maxima = l.swap + kComputeWarps * 32 * mt * 4 * 4;
  l.sums = l.maxima + mt * 16 * 8 * 4;
  l.bars = l.sums + mt * 16 * 8 * 4;
  l.total = l.bars + 64;
  return l;
}

__device__ __forceinline__ void compute_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// What one item covers.
struct LatentItem {
  int request, chunk, group, chunks;
  long long first_seen, begin, end;  // first visible token, tokens of the chunk
};

// MT: 16-head tiles per item.  BOXES: upper limit of the key's 64-dim boxes.
template <int MT, int BOXES>
__global__ void __launch_bounds__(kLatentThreads, 1)
    latent_decode_kernel(const __grid_constant__ CUtensorMap map, const LatentParams p) {
  using T = __nv_bfloat16;
  using Mma = Mma16816<T>;
  extern __shared__ uint8_t latent_smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>(align_up((long long)reinterpret_cast<uintptr_t>(latent_smem_raw), 1024));
  const LatentLayout at = latent_layout(p.key_boxes, MT);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + at.bars);
  uint64_t* empty = full + kRing;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < kRing; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], kComputeWarps);
    }
    mbar_fence_init();
    tma_prefetch_desc(&map);
  }
  __syncthreads();
  chain_wait();
  chain_release();

  const int chunk = p.sc.header[0], total_items = p.sc.header[2];
  const long long capacity = (long long)p.table_width * p.block_size;
  auto item_of = [&](int number) {
    LatentItem it;
    const int pair = number / p.head_groups;  // below the plan's pair count, checked by the callers
    it.group = number % p.head_groups;
    it.request = p.sc.item_seq[pair];
    it.chunk = p.sc.item_chunk[pair];
    it.chunks = p.sc.offsets[it.request + 1] - p.sc.offsets[it.request];
    const long long len = read_length(p.lengths, IndexView(), it.request, capacity, nullptr);
    it.first_seen = p.window > 0 && len > p.window ? len - p.window : 0;
    it.begin = window_start(len, p.window) + (long long)it.chunk * chunk;
    it.end = len < it.begin + chunk ? len : it.begin + chunk;
    return it;
  };
  // Byte distance between 8-token groups and between 64-dim groups of a stage.
  const int tok_group = p.slab ? p.key_boxes * 1024 : 1024, dim_group = p.slab ? 1024 : kStageTokens * 128;

  if (warp == kComputeWarps) {
    // ---------------- producer ----------------
    const uint64_t policy = l2_evict_first_policy();
    int fill = 0;  // stages filled so far
    bool ok = true;
    for (int number = blockIdx.x; number < total_items && ok; number += gridDim.x) {
      const LatentItem it = item_of(number);
      for (long long tok0 = it.begin; tok0 < it.end && ok; tok0 += kStageTokens, ++fill) {
        const int s = fill % kRing;
        const int left = (int)(it.end - tok0 < kStageTokens ? it.end - tok0 : kStageTokens);
        const int slabs = (left + kTileTokens - 1) / kTileTokens;
        int page = 0, slot = 0;
        if (lane < slabs) {
          const long long tok = tok0 + lane * kTileTokens;
          const long long id = p.tables.at(it.request, tok / p.block_size);
          if (id < 0 || id >= p.num_blocks) raise_status(p.status, MIE_STATUS_BAD_PAGE);
          page = id < 0 || id >= p.num_blocks ? 0 : (int)id;
          slot = (int)(tok % p.block_size);
        }
        if (lane == 0) {
          ok = mbar_wait_bounded(&empty[s], ((fill / kRing) & 1u) ^ 1u);
          if (ok)
            mbar_expect_tx(&full[s], slabs * p.key_boxes * kBoxBytes);
          else
            raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (ok && lane < slabs) {
          uint8_t* dst = smem + s * at.stage;
          if (p.slab) {
            tma_load_5d_hint(dst + lane * p.key_boxes * kBoxBytes, &map, &full[s], 0, 0, 0, slot / 8, page, policy);
          } else {
            for (int x = 0; x < p.key_boxes; ++x)
              tma_load_4d_hint(dst + x * dim_group + lane * kBoxBytes, &map, &full[s], x * 64, slot, 0, page, policy);
          }
        }
        __syncwarp();
      }
    }
  } else {
    // ---------------- compute ----------------
    const int g = lane >> 2, t = lane & 3;
    // S: warp = (16-head tile mt_s, every other 16-dim step from k_half on, 16 * MT keys of pair kp); after the swap it
    // owns kKeys of them, group kg.
    constexpr int kKeys = 8 * MT;
    constexpr int kKeyGroups = 64 / kKeys;
    constexpr int kSteps = BOXES * 2;  // 16-dim steps of one half
    constexpr bool kHoldQ = MT == 1;
    const int mt_s = warp % MT, k_half = warp / MT % 2, kp = warp / (2 * MT);
    const int kg = 2 * kp + k_half;
    const int value_boxes = (p.vdim + 63) / 64;
    const int k_steps = (p.dim + 15) / 16;
    const uint32_t q_at = smem_u32(smem + at.q), p_at = smem_u32(smem + at.p);
    float* maxima = reinterpret_cast<float*>(smem + at.maxima);  // [head][key group]
    float* sums = reinterpret_cast<float*>(smem + at.sums);
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_sel = (lane >> 4) & 1;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_sel = (lane >> 4) & 1;
    const int k_row = (lane & 7) + ((lane >> 4) & 1) * 8, k_sel = (lane >> 3) & 1;  // sixteen keys x 16 dims per load
    float* swap = reinterpret_cast<float*>(smem + at.swap);
    int fill = 0;
    bool ok = true;
    for (int number = blockIdx.x; number < total_items; number += gridDim.x) {
      const LatentItem it = item_of(number);
      const int head0 = it.group * MT * 16;
      compute_sync();  // the previous item's Q, maxima and sums have been read
      for (int i = threadIdx.x; i < MT * 16 * p.key_boxes * 8; i += kComputeWarps * 32) {
        const int r = i / (p.key_boxes * 8), u = i % (p.key_boxes * 8);
        uint4 v = make_uint4(0, 0, 0, 0);
        if (head0 + r < p.heads && u * 8 < p.dim)
          v = *reinterpret_cast<const uint4*>(p.q + (it.request * p.q_row + (head0 + r) * p.q_head + u * 8) * 2);
        *reinterpret_cast<uint4*>(smem + at.q + (u >> 3) * (MT * 16 * 128) + r * 128 + (((u & 7) ^ (r & 7)) << 4)) = v;
      }
      // Running maximum (log2 units) of this thread's rows g, g + 8 of every 16-head tile; the denominators of its
      // own S rows over its own keys.
      float m[MT][2], l[2] = {0.f, 0.f}, o[MT][8][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        m[i][0] = m[i][1] = -INFINITY;
#pragma unroll
        for (int n = 0; n < 8; ++n) o[i][n][0] = o[i][n][1] = o[i][n][2] = o[i][n][3] = 0.f;
        if (p.sinks != nullptr && it.chunk == 0) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int head = head0 + i * 16 + g + e * 8;
            m[i][e] = head < p.heads ? p.sinks[head] * 1.4426950408889634f : 0.f;
            if (i == mt_s && kg == 0 && t == 0) l[e] = 1.f;
          }
        }
      }
      compute_sync();
      auto load_q = [&](int ks, uint32_t (&a)[4]) {
        ldmatrix_x4(a[0], a[1], a[2], a[3],
                    q_at + (ks >> 2) * (MT * 16 * 128) + (mt_s * 16 + a_row) * 128 +
                        ((((ks & 3) * 2 + a_sel) ^ (a_row & 7)) << 4));
      };
      uint32_t held[kHoldQ ? kSteps : 1][4];
      if (kHoldQ) {
#pragma unroll
        for (int i = 0; i < kSteps; ++i)
          if (2 * i + k_half < k_steps) load_q(2 * i + k_half, held[kHoldQ ? i : 0]);
      }
      for (long long tok0 = it.begin; tok0 < it.end; tok0 += kStageTokens, ++fill) {
        const int s = fill % kRing;
        const bool arrived = ok && mbar_wait_bounded(&full[s], (fill / kRing) & 1u);
        if (!__all_sync(0xffffffffu, arrived)) ok = false;  // later waits are skipped, the barriers below are not
        const int valid = (int)(it.end - tok0 < kStageTokens ? it.end - tok0 : kStageTokens);
        const uint32_t stage = smem_u32(smem + s * at.stage);
        if (valid < kStageTokens) {
          // Rows past the read length may hold anything (even NaN bits): zero them so that 0 * V stays 0.
          for (int i = threadIdx.x; i < (kStageTokens - valid) * p.key_boxes * 8; i += kComputeWarps * 32) {
            const int row = valid + i / (p.key_boxes * 8), u = i % (p.key_boxes * 8);
            *reinterpret_cast<uint4*>(smem + s * at.stage + (row >> 3) * tok_group + (u >> 3) * dim_group +
                                      (row & 7) * 128 + (u & 7) * 16) = make_uint4(0, 0, 0, 0);
          }
          fence_proxy_async_smem();
          compute_sync();
        }
        // Half sums of S for 16 heads x 16 * MT keys.
        float part[2 * MT][4];
#pragma unroll
        for (int n = 0; n < 2 * MT; ++n) part[n][0] = part[n][1] = part[n][2] = part[n][3] = 0.f;
#pragma unroll
        for (int i = 0; i < kSteps; ++i) {
          const int ks = 2 * i + k_half;
          if (ks < k_steps) {
            uint32_t(&q)[4] = held[kHoldQ ? i : 0];
            if (!kHoldQ) load_q(ks, q);
#pragma unroll
            for (int np = 0; np < MT; ++np) {
              const int key_row = (kp * MT + np) * 16 + k_row;
              uint32_t r0, r1, r2, r3;
              ldmatrix_x4(r0, r1, r2, r3,
                          stage + (key_row >> 3) * tok_group + (key_row & 7) * 128 + (ks >> 2) * dim_group +
                              ((((ks & 3) * 2 + k_sel) ^ (key_row & 7)) << 4));
              Mma::run(part[2 * np], q[0], q[1], q[2], q[3], r0, r1);
              Mma::run(part[2 * np + 1], q[0], q[1], q[2], q[3], r2, r3);
            }
          }
        }
        // Swap with the warp that has the other dims: each of the pair keeps half of the keys.
        float sa[MT][4];
#pragma unroll
        for (int n = 0; n < MT; ++n) {
          float4 give;
          if (k_half == 0) {
            give = make_float4(part[MT + n][0], part[MT + n][1], part[MT + n][2], part[MT + n][3]);
            sa[n][0] = part[n][0], sa[n][1] = part[n][1], sa[n][2] = part[n][2], sa[n][3] = part[n][3];
          } else {
            give = make_float4(part[n][0], part[n][1], part[n][2], part[n][3]);
            sa[n][0] = part[MT + n][0], sa[n][1] = part[MT + n][1], sa[n][2] = part[MT + n][2], sa[n][3] = part[MT + n][3];
          }
          *reinterpret_cast<float4*>(swap + ((warp * MT + n) * 32 + lane) * 4) = give;
        }
        asm volatile("bar.sync %0, 64;" ::"r"(2 + kp * MT + mt_s) : "memory");
#pragma unroll
        for (int n = 0; n < MT; ++n) {
          const int other = k_half == 0 ? warp + MT : warp - MT;
          const float4 v = *reinterpret_cast<const float4*>(swap + ((other * MT + n) * 32 + lane) * 4);
          sa[n][0] += v.x, sa[n][1] += v.y, sa[n][2] += v.z, sa[n][3] += v.w;
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < MT; ++n) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int key = kg * kKeys + n * 8 + 2 * t + (e & 1);
            float v = sa[n][e] * p.scale_log2;
            if (key >= valid || tok0 + key < it.first_seen) v = -INFINITY;
            sa[n][e] = v;
            mx[e >> 1] = fmaxf(mx[e >> 1], v);
          }
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
          mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
          if (t == 0) maxima[(mt_s * 16 + g + e * 8) * 8 + kg] = mx[e];
        }
        compute_sync();
        // Common maximum of every row; finite, since every stage holds a visible token.
        float alpha[MT][2];
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float* row = maxima + (i * 16 + g + e * 8) * 8;
            float top = m[i][e];
#pragma unroll
            for (int k = 0; k < kKeyGroups; ++k) top = fmaxf(top, row[k]);
            alpha[i][e] = exp2f(m[i][e] - top);
            m[i][e] = top;
          }
        float m_s[2], alpha_s[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          m_s[e] = mt_s == 0 ? m[0][e] : m[MT - 1][e];
          alpha_s[e] = mt_s == 0 ? alpha[0][e] : alpha[MT - 1][e];
          l[e] *= alpha_s[e];
        }
#pragma unroll
        for (int n = 0; n < MT; ++n) {
          const int key = kg * kKeys + n * 8 + 2 * t;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float w0 = exp2f(sa[n][2 * e] - m_s[e]), w1 = exp2f(sa[n][2 * e + 1] - m_s[e]);
            l[e] += w0 + w1;
            const int row = mt_s * 16 + g + e * 8;
            uint8_t* dst = smem + at.p + row * 128 + (((key >> 3) ^ (row & 7)) << 4) + (key & 7) * 2;
            *reinterpret_cast<uint32_t*>(dst) = Mma::pack(w0, w1);
            *reinterpret_cast<uint32_t*>(dst + MT * 16 * 128) = Mma::pack(w0 - round_bf16(w0), w1 - round_bf16(w1));
          }
        }
        compute_sync();
        if (warp < value_boxes) {
#pragma unroll
          for (int i = 0; i < MT; ++i)
#pragma unroll
            for (int n = 0; n < 8; ++n) {
              o[i][n][0] *= alpha[i][0], o[i][n][1] *= alpha[i][0];
              o[i][n][2] *= alpha[i][1], o[i][n][3] *= alpha[i][1];
            }
#pragma unroll
          for (int kt = 0; kt < 4; ++kt) {
            uint32_t w[MT][2][4];
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
              for (int part = 0; part < 2; ++part) {
                const int row = i * 16 + a_row;
                ldmatrix_x4(w[i][part][0], w[i][part][1], w[i][part][2], w[i][part][3],
                            p_at + part * (MT * 16 * 128) + row * 128 + (((kt * 2 + a_sel) ^ (row & 7)) << 4));
              }
            const int row = kt * 16 + v_row;
            const uint32_t v_base = stage + (row >> 3) * tok_group + warp * dim_group + (row & 7) * 128;
#pragma unroll
            for (int np = 0; np < 4; ++np) {
              uint32_t r0, r1, r2, r3;
              ldmatrix_x4_trans(r0, r1, r2, r3, v_base + (((np * 2 + v_sel) ^ (row & 7)) << 4));
#pragma unroll
              for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                  Mma::run(o[i][2 * np], w[i][part][0], w[i][part][1], w[i][part][2], w[i][part][3], r0, r1);
                  Mma::run(o[i][2 * np + 1], w[i][part][0], w[i][part][1], w[i][part][2], w[i][part][3], r2, r3);
                }
            }
          }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(&empty[s]);
      }
      // Denominators: over the quad, then over the key groups.
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        if (t == 0) sums[(mt_s * 16 + g + e * 8) * 8 + kg] = l[e];
      }
      compute_sync();
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int head = head0 + i * 16 + g + e * 8;
          if (head >= p.heads || warp >= value_boxes) continue;
          float total = 0.f;
#pragma unroll
          for (int k = 0; k < kKeyGroups; ++k) total += sums[(i * 16 + g + e * 8) * 8 + k];
          if (it.chunks == 1) {
            const float inv = 1.f / fmaxf(total, 1.17549435e-38f);
            T* row = reinterpret_cast<T*>(p.out) + it.request * p.o_row + head * p.o_head + warp * 64;
#pragma unroll
            for (int n = 0; n < 8; ++n)
              if (warp * 64 + n * 8 < p.vdim)
                *reinterpret_cast<uint32_t*>(row + n * 8 + 2 * t) =
                    Mma::pack(o[i][n][2 * e] * inv, o[i][n][2 * e + 1] * inv);
          } else {
            const long long part = ((long long)p.sc.offsets[it.request] + it.chunk) * p.heads + head;
            float* row = p.sc.part_o + part * p.vdim + warp * 64;
#pragma unroll
            for (int n = 0; n < 8; ++n)
              if (warp * 64 + n * 8 < p.vdim)
                *reinterpret_cast<float2*>(row + n * 8 + 2 * t) = make_float2(o[i][n][2 * e], o[i][n][2 * e + 1]);
            if (warp == 0 && t == 0) {
              p.sc.part_m[part] = m[i][e];
              p.sc.part_l[part] = total;
            }
          }
        }
    }
    if (!ok && lane == 0) raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
    // Requests with nothing to read (rejected metadata) get zeros.
    for (int e = blockIdx.x * kComputeWarps + warp; e < p.batch; e += gridDim.x * kComputeWarps) {
      if (p.sc.offsets[e + 1] != p.sc.offsets[e]) continue;
      for (int h = 0; h < p.heads; ++h)
        for (int d = 2 * lane; d < p.vdim; d += 64)
          *reinterpret_cast<uint32_t*>(reinterpret_cast<T*>(p.out) + e * p.o_row + h * p.o_head + d) = 0u;
    }
  }
}

template <int MT, int BOXES>
int launch_latent(const CUtensorMap& map, const LatentParams& p, cudaStream_t stream) {
  const int smem = latent_layout(p.key_boxes, MT).total + 1024;
  static int configured[64] = {0};
  int dev = 0;
  MIE_CUDA(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || configured[dev] < smem) {
    MIE_CUDA(cudaFuncSetAttribute(latent_decode_kernel<MT, BOXES>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    if (dev >= 0 && dev < 64) configured[dev] = smem;
  }
  MIE_CUDA(launch_chained(latent_decode_kernel<MT, BOXES>, dim3(sm_count()), dim3(kLatentThreads), (size_t)smem, stream,
                          map, p));
  MIE_LAUNCH_CHECK("latent_decode_kernel");
  return MIE_OK;
}

template <int MT>
int launch_latent_boxes(const CUtensorMap& map, const LatentParams& p, cudaStream_t stream) {
  if (p.key_boxes <= 4) return launch_latent<MT, 4>(map, p, stream);
  if (p.key_boxes <= 9) return launch_latent<MT, 9>(map, p, stream);
  return launch_latent<MT, kMaxKeyBoxes>(map, p, stream);
}

template <int VH>
int launch_latent_merge(const DecodeParams& p, cudaStream_t stream) {
  MIE_CUDA(launch_chained(merge_rows_kernel<__nv_bfloat16, VH>, dim3((unsigned)(p.batch * p.q_heads)),
                          dim3(kMergeWarps * 32), 0, stream, p));
  MIE_LAUNCH_CHECK("merge_rows_kernel");
  return MIE_OK;
}

int latent_pairs(int batch, long long max_total_tokens) {
  long long extra = max_total_tokens / kMinChunk;
  const long long most = 8ll * sm_count();
  return batch + 1 + (int)(extra < most ? extra : most);
}

}  // namespace
}  // namespace mie

using namespace mie;

extern "C" int mie_latent_decode_supported(int32_t dim, int32_t value_dim, int32_t block_size, int32_t dtype) {
  return dtype == MIE_DTYPE_BF16 && dim >= 8 && dim % 8 == 0 && dim <= kMaxKeyBoxes * 64 && value_dim >= 8 &&
         value_dim % 8 == 0 && value_dim <= dim && value_dim <= kComputeWarps * 64 && block_size >= kTileTokens &&
         block_size % kTileTokens == 0;
}

extern "C" int64_t mie_latent_decode_scratch_bytes(int32_t batch, int32_t heads, int32_t value_dim,
                                                   int64_t max_total_tokens) {
  if (batch < 0 || heads < 1 || value_dim < 1 || max_total_tokens < 0) return 0;
  return fixed_scratch_bytes(batch, 1) + 2048 +
         (int64_t)latent_pairs(batch, max_total_tokens) * per_chunk_bytes(heads, value_dim);
}

extern "C" int mie_latent_decode_attention(const void* query, int64_t q_row_stride, int64_t q_head_stride, void* out,
                                           int64_t o_row_stride, int64_t o_head_stride, mie_view4_t pages,
                                           mie_index_t block_tables, mie_index_t sequence_lengths, int32_t batch,
                                           int32_t heads, int32_t dim, int32_t value_dim, int32_t block_size,
                                           int32_t num_blocks, int32_t table_width, int32_t dtype, float scale,
                                           int64_t window, const float* sinks, int32_t split_policy, void* scratch,
                                           int64_t scratch_bytes, int32_t use_plan, int32_t* status, void* stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  MIE_CHECK_ARG(mie_latent_decode_supported(dim, value_dim, block_size, dtype),
                "latent decode attention takes bf16, rows of a multiple of 8 entries up to %d, values up to %d and "
                "pages of whole 16-token tiles (got %d, %d, page %d)", kMaxKeyBoxes * 64, kComputeWarps * 64, dim,
                value_dim, block_size);
  MIE_CHECK_ARG(batch >= 0 && heads >= 1, "invalid sizes");
  MIE_CHECK_ARG(query && out && pages.ptr && block_tables.ptr && sequence_lengths.ptr && scratch, "null pointer");
  MIE_CHECK_ARG(num_blocks >= 1 && table_width >= 1 && window >= 0 && split_policy >= 0, "invalid sizes");
  MIE_CHECK_ARG(pages.stride[3] == 1 && aligned16(pages.ptr), "pages must be 16-byte aligned rows");
  for (int i = 0; i < 3; ++i)
    MIE_CHECK_ARG(pages.stride[i] > 0 && pages.stride[i] % 8 == 0, "page strides must be multiples of 16 bytes");
  MIE_CHECK_ARG(q_row_stride % 8 == 0 && q_head_stride % 8 == 0 && aligned16(query) && o_row_stride % 2 == 0 &&
                    o_head_stride % 2 == 0 && (reinterpret_cast<uintptr_t>(out) & 3) == 0,
                "query rows must be 16-byte aligned, out rows 4-byte aligned");
  MIE_CHECK_ARG((reinterpret_cast<uintptr_t>(scratch) & 255) == 0, "scratch must be 256-byte aligned");
  if (batch == 0) return MIE_OK;
  Scratch sc = carve(scratch, scratch_bytes, batch, heads, 1, value_dim);
  MIE_CHECK_ARG(sc.cap > batch, "scratch of %lld bytes is too small for batch %d", (long long)scratch_bytes, batch);
  const int tiles = heads <= 16 ? 1 : 2;  // 16-head tiles per work item
  const int head_groups = (heads + tiles * 16 - 1) / (tiles * 16);
  const int key_boxes = (dim + 63) / 64;
  if (!use_plan) {
    plan_kernel<<<1, plan_threads(batch), 0, stream>>>(IndexView(sequence_lengths), IndexView(), batch,
                                                       (long long)table_width * block_size, head_groups, split_policy,
                                                       sm_count(), 128, (long long)window, sc, status);
    MIE_LAUNCH_CHECK("plan_kernel");
  }
  const bool slab = pages_fit_slab_map(pages, block_size, dim);
  CUtensorMap map;
  if (int rc = slab ? page_slab_map(pages, num_blocks, 1, block_size, dim, key_boxes, dtype, &map)
                    : page_tensor_map(pages, num_blocks, 1, block_size, dim, dtype, &map))
    return rc;
  const LatentParams p{(const char*)query, q_row_stride, q_head_stride, (char*)out, o_row_stride, o_head_stride,
                       IndexView(block_tables), IndexView(sequence_lengths), sc, batch, heads, block_size, num_blocks,
                       table_width, dim, value_dim, key_boxes, head_groups, slab ? 1 : 0, scale * 1.4426950408889634f,
                       window, sinks, status};
  if (int rc = tiles == 1 ? launch_latent_boxes<1>(map, p, stream) : launch_latent_boxes<2>(map, p, stream)) return rc;
  mie_view4_t q{const_cast<void*>(query), {q_row_stride, q_head_stride, 0, 1}};
  mie_view4_t o{out, {o_row_stride, o_head_stride, 0, 1}};
  const DecodeParams merge{View4(q), View4(o), p.tables, p.lengths, IndexView(), sc, batch, heads, 1, heads, block_size,
                           num_blocks, table_width, p.scale_log2, 0, status, nullptr, 0, nullptr, 0, 0, dim, value_dim,
                           head_groups, window, sinks};
  const int boxes = (value_dim + 63) / 64;
  return boxes <= 2 ? launch_latent_merge<2>(merge, stream)
                    : boxes <= 4 ? launch_latent_merge<4>(merge, stream) : launch_latent_merge<8>(merge, stream);
}
