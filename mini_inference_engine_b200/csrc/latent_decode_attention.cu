// Ragged paged decode attention over a latent cache: one cached row per token, read by every query head.  The key of
// a token is its whole row (latent | rotated part), the value the row's first `vdim` entries, so a row is fetched
// once for both products and for all heads.
//
// One persistent CTA per SM walks (request, chunk, up to 32 heads) items of the shared split-KV plan in a fixed order.
// Warp roles: 8 score warps, 1 TMA producer (16-token slabs of pages into a ring of 64-token stages, 128-byte swizzle,
// no multicast) that runs ahead across items, 1 tcgen05 issuer that owns the TMEM allocation.  Per stage:
//   S = K Q^T    mma.sync; a warp has 16 heads, 16 * MT keys and every other 16 dims (with one 16-head tile its Q
//                fragments stay in registers); the two warps that share keys swap halves of their sums
//   softmax      row maxima meet in shared memory; the common reference maximum moves only when a head's grows by more
//                than 2^8; the weights go to shared memory as a rounded bf16 part and its remainder, one row per head each
//   O += V^T P   tcgen05, A = 128 value dims of the stage read MN-major, B = the weight rows: rounded parts and
//                remainders accumulate in neighbouring TMEM columns (lane = dim) and are added at the end.  It runs while
//                the score warps are at the next stage
// (tcgen05 streams A at one row per cycle whatever the number of heads, mma.sync pays per 16 heads: for up to 32 heads
// the first product is cheaper on mma.sync and the second on tcgen05, and the two overlap.)  Every wait is bounded and
// reports MIE_STATUS_WAIT_TIMEOUT.  Scores, weights, sums and O are fp32.  The sink opens the running maximum and the
// denominator of a request's first chunk; partials are merged by merge_rows_kernel.
#include "decode_attention.cuh"
#include "umma.cuh"

namespace mie {

// Defined in prefill_attention_umma.cu: cached 5-D slab map over pages [page, head, token, dim] (dim a multiple of
// 64) whose box is 16 tokens x `box_groups` 64-dim groups, and whether a page layout allows it.
int page_slab_map(const mie_view4_t& pages, int num_blocks, int kv_heads, int block_size, int dim, int box_groups,
                  int dtype, CUtensorMap* out);
bool pages_fit_slab_map(const mie_view4_t& v, int block_size, int dim);

namespace {

constexpr int kStageTokens = 64;
constexpr int kScoreWarps = 8;
constexpr int kLatentThreads = (kScoreWarps + 2) * 32;
constexpr int kMaxKeyBoxes = 10;
constexpr int kMaxValueDims = 512;
constexpr int kItemHeads = 32;               // heads one work item covers at most
constexpr float kRescaleThreshold = 8.0f;    // log2 units
constexpr float kLog2e = 1.4426950408889634f;

struct LatentParams {
  const char* q;
  long long q_row, q_head;
  char* out;
  long long o_row, o_head;
  IndexView tables, lengths;
  Scratch sc;
  int batch, heads, block_size, num_blocks, table_width, dim, vdim, key_boxes, head_groups, ring, slab;
  float scale_log2;
  long long window;
  const float* sinks;
  int* status;
};

// Shared memory: ring of stages | Q [box][head][64] | P, two buffers of [rounded heads | remainders][64 keys] | swapped
// sums | two [head][key group] of maxima, one of denominators | factors per head | barriers.
struct LatentLayout {
  int stage, q, p, p_bytes, swap, maxima, sums, factors, bars, total;
};
__host__ __device__ inline LatentLayout latent_layout(int key_boxes, int ring, int tiles) {
  LatentLayout l;
  const int heads = tiles * 16;
  l.stage = key_boxes * kStageTokens * 128;
  l.q = ring * l.stage;
  l.p = l.q + key_boxes * heads * 128;
  l.p_bytes = 2 * heads * 128;
  l.swap = l.p + 2 * l.p_bytes;
  l.maxima = l.swap + kScoreWarps * 32 * tiles * 16;
  l.sums = l.maxima + 2 * heads * 8 * 4;
  l.factors = l.sums + heads * 8 * 4;
  l.bars = l.factors + heads * 4;
  l.total = l.bars + 256;
  return l;
}
constexpr int kMaxRing = 4;
enum LatentBar { kFull = 0, kEmpty = kMaxRing, kPFull = 2 * kMaxRing, kPvDone = kPFull + 2, kOFree = kPvDone + 2,
                 kLatentBars };

__device__ __forceinline__ void score_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ float ex2_approx(float x) {  // -inf gives +0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Columns of this thread's TMEM lane.
template <int N>
__device__ __forceinline__ void tmem_load(uint32_t addr, float (&v)[N]) {
  if constexpr (N == 16) {
    tmem_ld16(addr, v);
  } else {
#pragma unroll
    for (int c = 0; c < N; c += 32) tmem_ld32(addr + c, *reinterpret_cast<float(*)[32]>(&v[c]));
  }
  tmem_ld_wait();
}

// What one item covers.
struct LatentItem {
  int request, chunk, group, chunks;
  long long first_seen, begin, end;  // first visible token, tokens of the chunk
  __device__ __forceinline__ int valid(long long tok0) const {
    return (int)(end - tok0 < kStageTokens ? end - tok0 : kStageTokens);
  }
};

// MT: 16-head tiles per item.  BOXES: 64-dim boxes of the key (the last one zero-filled past the key's size).
template <int MT, int BOXES>
__global__ void __launch_bounds__(kLatentThreads, 1)
    latent_decode_kernel(const __grid_constant__ CUtensorMap map, const LatentParams p) {
  using T = __nv_bfloat16;
  using Mma = Mma16816<T>;
  constexpr int HN = MT * 16;
  extern __shared__ uint8_t latent_smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>(align_up((long long)reinterpret_cast<uintptr_t>(latent_smem_raw), 1024));
  const LatentLayout at = latent_layout(BOXES, p.ring, MT);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + at.bars);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + kLatentBars);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr uint32_t kTmemCols = kMaxValueDims / 128 * 2 * HN;  // 2 HN columns per group of 128 value dims
  if (threadIdx.x == 0) {
    for (int s = 0; s < p.ring; ++s) {
      mbar_init(&bars[kFull + s], 1);
      mbar_init(&bars[kEmpty + s], 1);
    }
    mbar_init(&bars[kOFree], kScoreWarps * 32);
    for (int b = 0; b < 2; ++b) {
      mbar_init(&bars[kPFull + b], kScoreWarps * 32);
      mbar_init(&bars[kPvDone + b], 1);
    }
    mbar_fence_init();
    tma_prefetch_desc(&map);
  }
  if (warp == kScoreWarps + 1) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_o = *tmem_slot;
  chain_wait();
  chain_release();

  const int chunk = p.sc.header[0], total_items = p.sc.header[2];
  const long long capacity = (long long)p.table_width * p.block_size;
  auto item_of = [&](int number) {
    LatentItem it;
    const int pair = number / p.head_groups;
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
  const int tok_group = p.slab ? BOXES * 1024 : 1024, dim_group = p.slab ? 1024 : kStageTokens * 128;
  const int value_groups = (p.vdim + 127) / 128;

  if (warp == kScoreWarps) {
    // ---------------- TMA producer ----------------
    const uint64_t policy = l2_evict_first_policy();
    int fill = 0;  // stages filled so far
    bool ok = true;
    for (int number = blockIdx.x; number < total_items && ok; number += gridDim.x) {
      const LatentItem it = item_of(number);
      for (long long tok0 = it.begin; tok0 < it.end && ok; tok0 += kStageTokens, ++fill) {
        const int s = fill % p.ring;
        const int slabs = (it.valid(tok0) + kTileTokens - 1) / kTileTokens;
        int page = 0, slot = 0;
        if (lane < slabs) {
          const long long tok = tok0 + lane * kTileTokens;
          const long long id = p.tables.at(it.request, tok / p.block_size);
          if (id < 0 || id >= p.num_blocks) raise_status(p.status, MIE_STATUS_BAD_PAGE);
          page = id < 0 || id >= p.num_blocks ? 0 : (int)id;
          slot = (int)(tok % p.block_size);
        }
        if (lane == 0) {
          ok = mbar_wait_bounded(&bars[kEmpty + s], ((fill / p.ring) & 1u) ^ 1u);
          if (ok)
            mbar_expect_tx(&bars[kFull + s], slabs * BOXES * kBoxBytes);
          else
            raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (ok && lane < slabs) {
          uint8_t* dst = smem + s * at.stage;
          if (p.slab) {
            tma_load_5d_hint(dst + lane * BOXES * kBoxBytes, &map, &bars[kFull + s], 0, 0, 0, slot / 8, page, policy);
          } else {
            for (int x = 0; x < BOXES; ++x)
              tma_load_4d_hint(dst + x * dim_group + lane * kBoxBytes, &map, &bars[kFull + s], x * 64, slot, 0, page, policy);
          }
        }
        __syncwarp();
      }
    }
  } else if (warp == kScoreWarps + 1) {
    // ---------------- tcgen05 issuer ----------------
    if (lane == 0) {
      constexpr uint32_t idesc = instr_desc_bf16(128, 2 * HN, 1, 0);  // A = V^T, MN-major; B = weight rows, K-major
      // Descriptor addresses count 16-byte units: every product's operands are a base plus small increments.
      const uint64_t slab_step = (2 * tok_group) >> 4, group_step = (2 * dim_group) >> 4;
      int tile = 0, items = 0;  // stages and items so far
      bool ok = true;
      for (int number = blockIdx.x; number < total_items && ok; number += gridDim.x, ++items) {
        const LatentItem it = item_of(number);
        for (long long tok0 = it.begin; tok0 < it.end && ok; tok0 += kStageTokens, ++tile) {
          const int s = tile % p.ring, b = tile & 1;
          ok = mbar_wait_bounded(&bars[kPFull + b], (tile >> 1) & 1u) &&
               mbar_wait_bounded(&bars[kFull + s], (tile / p.ring) & 1u) &&
               (tok0 > it.begin || items == 0 || mbar_wait_bounded(&bars[kOFree], (items - 1) & 1u));  // O has been read
          if (!ok) break;
          tc_fence_after();
          uint64_t values = smem_desc_mn128(smem_u32(smem + s * at.stage), dim_group, tok_group);
          uint64_t weights = smem_desc_k128(smem_u32(smem + at.p + b * at.p_bytes));
          const int slabs = (it.valid(tok0) + kTileTokens - 1) / kTileTokens;
          for (int kt = 0; kt < slabs; ++kt) {
#pragma unroll
            for (int d = 0; d < kMaxValueDims / 128; ++d)
              if (d < value_groups)
                umma_f16(tmem_o + d * 2 * HN, values + d * group_step, weights, idesc, tok0 > it.begin || kt > 0 ? 1u : 0u);
            values += slab_step;
            weights += 2;
          }
          umma_commit(&bars[kEmpty + s]);   // the stage is free once these MMAs have read it
          umma_commit(&bars[kPvDone + b]);  // O includes this stage
        }
      }
      if (!ok) raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
    }
  } else {
    // ---------------- scores, softmax, epilogue ----------------
    const int g = lane >> 2, t = lane & 3;
    // S: warp = (16-head tile mt_s, every other 16-dim step from k_half on, 16 * MT keys of pair kp); after the swap it
    // owns kKeys of them, group kg.
    constexpr int kKeys = 8 * MT;
    constexpr int kKeyGroups = kStageTokens / kKeys;
    constexpr int kSteps = BOXES * 2;  // 16-dim steps of one half
    constexpr int kAhead = 3;          // steps whose operands are loaded before they are used
    constexpr bool kHoldQ = MT == 1;
    const int mt_s = warp % MT, k_half = warp / MT % 2, kp = warp / (2 * MT);
    const int kg = 2 * kp + k_half;
    const uint32_t q_at = smem_u32(smem + at.q);
    float* swap = reinterpret_cast<float*>(smem + at.swap);
    float* maxima = reinterpret_cast<float*>(smem + at.maxima);    // [stage parity][head][key group]
    float* sums = reinterpret_cast<float*>(smem + at.sums);        // [head][key group]
    float* factors = reinterpret_cast<float*>(smem + at.factors);  // [head]
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_sel = (lane >> 4) & 1;
    const int k_row = (lane & 7) + ((lane >> 4) & 1) * 8, k_sel = (lane >> 3) & 1;  // sixteen keys x 16 dims per load
    const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;                   // O: TMEM lanes of this warp
    auto fetch_q = [&](const LatentItem& it) {
      for (int i = threadIdx.x; i < HN * BOXES * 8; i += kScoreWarps * 32) {
        const int r = i / (BOXES * 8), u = i % (BOXES * 8), head = it.group * HN + r;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (head < p.heads && u * 8 < p.dim)
          v = *reinterpret_cast<const uint4*>(p.q + (it.request * p.q_row + head * p.q_head + u * 8) * 2);
        *reinterpret_cast<uint4*>(smem + at.q + (u >> 3) * (HN * 128) + r * 128 + (((u & 7) ^ (r & 7)) << 4)) = v;
      }
    };
    int tile = 0;
    bool ok = true;  // a failed wait skips later waits, never a barrier
    LatentItem it;
    if ((int)blockIdx.x < total_items) {
      it = item_of(blockIdx.x);
      fetch_q(it);
    }
    for (int number = blockIdx.x; number < total_items; number += gridDim.x) {
      const int head0 = it.group * HN;
      score_sync();  // Q is there
      auto load_q = [&](int ks, uint32_t (&a)[4]) {
        ldmatrix_x4(a[0], a[1], a[2], a[3], q_at + (ks >> 2) * (HN * 128) + (mt_s * 16 + a_row) * 128 +
                                                ((((ks & 3) * 2 + a_sel) ^ (a_row & 7)) << 4));
      };
      uint32_t held[kHoldQ ? kSteps : 1][4];
      if (kHoldQ) {
#pragma unroll
        for (int i = 0; i < kSteps; ++i) load_q(2 * i + k_half, held[kHoldQ ? i : 0]);
      }
      // Reference maximum (log2 units) of rows g, g + 8 of every 16-head tile; the denominators of this thread's own
      // rows over its own keys.
      float m[MT][2], l[2] = {0.f, 0.f};
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          m[i][e] = -INFINITY;
          if (p.sinks != nullptr && it.chunk == 0) {
            const int head = head0 + i * 16 + g + e * 8;
            m[i][e] = head < p.heads ? p.sinks[head] * kLog2e : 0.f;
            if (i == mt_s && kg == 0 && t == 0) l[e] = 1.f;
          }
        }
      for (long long tok0 = it.begin; tok0 < it.end; tok0 += kStageTokens, ++tile) {
        const int s = tile % p.ring, b = tile & 1, valid = it.valid(tok0);
        if (ok && !mbar_wait_bounded(&bars[kFull + s], (tile / p.ring) & 1u)) ok = false;
        const uint32_t stage = smem_u32(smem + s * at.stage);
        // Half sums of S for 16 heads x 16 * MT keys.
        float part[2 * MT][4];
#pragma unroll
        for (int n = 0; n < 2 * MT; ++n) part[n][0] = part[n][1] = part[n][2] = part[n][3] = 0.f;
        uint32_t keys[kAhead][MT][4], rows[kHoldQ ? 1 : kAhead][4];
        auto load_keys = [&](int i) {
          const int ks = 2 * i + k_half;
          if (!kHoldQ) load_q(ks, rows[kHoldQ ? 0 : i % kAhead]);
#pragma unroll
          for (int np = 0; np < MT; ++np) {
            const int key_row = (kp * MT + np) * 16 + k_row;
            uint32_t(&k)[4] = keys[i % kAhead][np];
            ldmatrix_x4(k[0], k[1], k[2], k[3],
                        stage + (key_row >> 3) * tok_group + (key_row & 7) * 128 + (ks >> 2) * dim_group +
                            ((((ks & 3) * 2 + k_sel) ^ (key_row & 7)) << 4));
          }
        };
#pragma unroll
        for (int i = 0; i < kAhead - 1 && i < kSteps; ++i) load_keys(i);
#pragma unroll
        for (int i = 0; i < kSteps; ++i) {
          if (i + kAhead - 1 < kSteps) load_keys(i + kAhead - 1);
          const uint32_t(&q)[4] = kHoldQ ? held[i % (kHoldQ ? kSteps : 1)] : rows[kHoldQ ? 0 : i % kAhead];
#pragma unroll
          for (int np = 0; np < MT; ++np) {
            const uint32_t(&k)[4] = keys[i % kAhead][np];
            Mma::run(part[2 * np], q[0], q[1], q[2], q[3], k[0], k[1]);
            Mma::run(part[2 * np + 1], q[0], q[1], q[2], q[3], k[2], k[3]);
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
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < MT; ++n) {
          const int other = k_half == 0 ? warp + MT : warp - MT;
          const float4 v = *reinterpret_cast<const float4*>(swap + ((other * MT + n) * 32 + lane) * 4);
          sa[n][0] += v.x, sa[n][1] += v.y, sa[n][2] += v.z, sa[n][3] += v.w;
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int key = kg * kKeys + n * 8 + 2 * t + (e & 1);
            sa[n][e] = key >= valid || tok0 + key < it.first_seen ? -INFINITY : sa[n][e] * p.scale_log2;
            mx[e >> 1] = fmaxf(mx[e >> 1], sa[n][e]);
          }
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
          mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
          if (t == 0) maxima[(b * HN + mt_s * 16 + g + e * 8) * 8 + kg] = mx[e];
        }
        if (valid % kTileTokens != 0) {
          // Rows of the last slab past the read length may hold anything (even NaN bits): zero them so that 0 * V stays 0.
          const int end = (valid + kTileTokens - 1) / kTileTokens * kTileTokens;
          for (int i = threadIdx.x; i < (end - valid) * BOXES * 8; i += kScoreWarps * 32) {
            const int row = valid + i / (BOXES * 8), u = i % (BOXES * 8);
            *reinterpret_cast<uint4*>(smem + s * at.stage + (row >> 3) * tok_group + (u >> 3) * dim_group +
                                      (row & 7) * 128 + (u & 7) * 16) = make_uint4(0, 0, 0, 0);
          }
        }
        score_sync();
        // Reference maxima; every warp looks at every head, so all decide alike whether any of them moves.
        float next[MT][2];
        bool grow = false;
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float4* row = reinterpret_cast<const float4*>(maxima + (b * HN + i * 16 + g + e * 8) * 8);
            const float4 a = row[0];
            float top = fmaxf(fmaxf(a.x, a.y), fmaxf(a.z, a.w));
            if (kKeyGroups > 4) {
              const float4 c = row[1];
              top = fmaxf(top, fmaxf(fmaxf(c.x, c.y), fmaxf(c.z, c.w)));
            }
            // Finite: every stage holds a visible token.
            next[i][e] = top > m[i][e] + kRescaleThreshold ? top : m[i][e];
            grow = grow || next[i][e] != m[i][e];
          }
        if (__any_sync(0xffffffffu, grow)) {
          if (tok0 > it.begin) {
            // O must first hold every stage before this one; then its columns move to the new reference.
            if (ok && !mbar_wait_bounded(&bars[kPvDone + (b ^ 1)], ((tile - 1) >> 1) & 1u)) ok = false;
            tc_fence_after();
            if (warp == 0 && t == 0) {
#pragma unroll
              for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int e = 0; e < 2; ++e) factors[i * 16 + g + e * 8] = ex2_approx(m[i][e] - next[i][e]);
            }
            score_sync();
            for (int d = warp >> 2; d < value_groups; d += 2)
#pragma unroll
              for (int half = 0; half < 2; ++half) {
                const uint32_t addr = tmem_o + d * 2 * HN + half * HN + lane_addr;
                float v[HN];
                tmem_load<HN>(addr, v);
#pragma unroll
                for (int h = 0; h < HN; ++h) v[h] *= factors[h];
                if constexpr (HN == 16)
                  tmem_st16(addr, *reinterpret_cast<const uint32_t(*)[16]>(&v));
                else
                  tmem_st32(addr, *reinterpret_cast<const uint32_t(*)[32]>(&v));
              }
            tmem_st_wait();
            score_sync();  // `factors` may be written again
          }
#pragma unroll
          for (int i = 0; i < MT; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              if (i == mt_s) l[e] *= ex2_approx(m[i][e] - next[i][e]);
              m[i][e] = next[i][e];
            }
        }
        // P(tile) goes where P(tile - 2) was.
        if (ok && tile >= 2 && !mbar_wait_bounded(&bars[kPvDone + b], ((tile - 2) >> 1) & 1u)) ok = false;
#pragma unroll
        for (int n = 0; n < MT; ++n) {
          const int key = kg * kKeys + n * 8 + 2 * t;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float ref = mt_s == 0 ? m[0][e] : m[MT - 1][e];
            const float w0 = ex2_approx(sa[n][2 * e] - ref), w1 = ex2_approx(sa[n][2 * e + 1] - ref);
            l[e] += w0 + w1;
            const int row = mt_s * 16 + g + e * 8;
            uint8_t* dst = smem + at.p + b * at.p_bytes + row * 128 + (((key >> 3) ^ (row & 7)) << 4) + (key & 7) * 2;
            const uint32_t high = Mma::pack(w0, w1);
            const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high));
            *reinterpret_cast<uint32_t*>(dst) = high;
            *reinterpret_cast<uint32_t*>(dst + HN * 128) = Mma::pack(w0 - k.x, w1 - k.y);
          }
        }
        fence_proxy_async_smem();
        tc_fence_before();
        mbar_arrive(&bars[kPFull + b]);
      }
      const LatentItem done = it;
      // Denominators: over the quad, then over the key groups.
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        if (t == 0) sums[(mt_s * 16 + g + e * 8) * 8 + kg] = l[e];
      }
      if (number + (int)gridDim.x < total_items) {  // the next item's queries, while the last products run
        it = item_of(number + gridDim.x);
        fetch_q(it);
      }
      score_sync();
      const long long part0 = ((long long)p.sc.offsets[done.request] + done.chunk) * p.heads + head0;
      if (warp == 0 && t == 0) {
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int h = i * 16 + g + e * 8;
            float total = 0.f;
#pragma unroll
            for (int k = 0; k < kKeyGroups; ++k) total += sums[h * 8 + k];
            factors[h] = done.chunks == 1 ? 1.f / fmaxf(total, 1.17549435e-38f) : 1.f;
            if (done.chunks > 1 && head0 + h < p.heads) {
              p.sc.part_m[part0 + h] = m[i][e];
              p.sc.part_l[part0 + h] = total;
            }
          }
      }
      const int last = tile - 1;
      if (ok && !mbar_wait_bounded(&bars[kPvDone + (last & 1)], (last >> 1) & 1u)) ok = false;
      tc_fence_after();
      score_sync();
      for (int d = warp >> 2; d < value_groups; d += 2) {
        float v[HN], r[HN];
        tmem_load<HN>(tmem_o + d * 2 * HN + lane_addr, v);
        tmem_load<HN>(tmem_o + d * 2 * HN + HN + lane_addr, r);
        const int c = d * 128 + (warp & 3) * 32 + lane;
        if (c >= p.vdim) continue;
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          if (head0 + h >= p.heads) break;
          const float x = (v[h] + r[h]) * factors[h];
          if (done.chunks == 1)
            reinterpret_cast<T*>(p.out)[done.request * p.o_row + (head0 + h) * p.o_head + c] = __float2bfloat16_rn(x);
          else
            p.sc.part_o[(part0 + h) * p.vdim + c] = x;
        }
      }
      tc_fence_before();
      mbar_arrive(&bars[kOFree]);
    }
    if (!ok && lane == 0) raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
    // Requests with nothing to read (rejected metadata) get zeros.
    for (int e = blockIdx.x * kScoreWarps + warp; e < p.batch; e += gridDim.x * kScoreWarps) {
      if (p.sc.offsets[e + 1] != p.sc.offsets[e]) continue;
      for (int h = 0; h < p.heads; ++h)
        for (int d = 2 * lane; d < p.vdim; d += 64)
          *reinterpret_cast<uint32_t*>(reinterpret_cast<T*>(p.out) + e * p.o_row + h * p.o_head + d) = 0u;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kScoreWarps + 1) {
    tc_fence_after();
    tmem_dealloc(*tmem_slot, kTmemCols);
  }
}

template <int MT, int BOXES>
int launch_latent(const CUtensorMap& map, LatentParams p, cudaStream_t stream) {
  p.ring = 2;
  while (p.ring < kMaxRing && latent_layout(p.key_boxes, p.ring + 1, MT).total + 1024 <= 224 * 1024) ++p.ring;
  const int smem = latent_layout(p.key_boxes, p.ring, MT).total + 1024;
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
  switch (p.key_boxes) {
    case 1: return launch_latent<MT, 1>(map, p, stream);
    case 2: return launch_latent<MT, 2>(map, p, stream);
    case 3: return launch_latent<MT, 3>(map, p, stream);
    case 4: return launch_latent<MT, 4>(map, p, stream);
    case 5: return launch_latent<MT, 5>(map, p, stream);
    case 6: return launch_latent<MT, 6>(map, p, stream);
    case 7: return launch_latent<MT, 7>(map, p, stream);
    case 8: return launch_latent<MT, 8>(map, p, stream);
    case 9: return launch_latent<MT, 9>(map, p, stream);
    default: return launch_latent<MT, kMaxKeyBoxes>(map, p, stream);
  }
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
         value_dim % 8 == 0 && value_dim <= dim && value_dim <= kMaxValueDims && block_size >= kTileTokens &&
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
                "pages of whole 16-token tiles (got %d, %d, page %d)", kMaxKeyBoxes * 64, kMaxValueDims, dim,
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
  const int item_heads = heads <= 16 ? 16 : kItemHeads;
  const int head_groups = (heads + item_heads - 1) / item_heads;
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
                       table_width, dim, value_dim, key_boxes, head_groups, 2, slab ? 1 : 0, scale * 1.4426950408889634f,
                       window, sinks, status};
  if (int rc = item_heads == 16 ? launch_latent_boxes<1>(map, p, stream) : launch_latent_boxes<2>(map, p, stream)) return rc;
  mie_view4_t q{const_cast<void*>(query), {q_row_stride, q_head_stride, 0, 1}};
  mie_view4_t o{out, {o_row_stride, o_head_stride, 0, 1}};
  const DecodeParams merge{View4(q), View4(o), p.tables, p.lengths, IndexView(), sc, batch, heads, 1, heads, block_size,
                           num_blocks, table_width, p.scale_log2, 0, status, nullptr, 0, nullptr, 0, 0, dim, value_dim,
                           head_groups, window, sinks};
  const int boxes = (value_dim + 63) / 64;
  return boxes <= 2 ? launch_latent_merge<2>(merge, stream)
                    : boxes <= 4 ? launch_latent_merge<4>(merge, stream) : launch_latent_merge<8>(merge, stream);
}
