// Ragged paged decode attention over a latent cache: one cached row per token, read by every query head.  The key of
// a token is its whole row (latent | rotated part), the value the row's first `vdim` entries, so a row is fetched
// once for both products and for all heads.
//
// One persistent CTA per SM walks (request, chunk, up to 32 heads) items of the shared split-KV plan in a fixed order.
// The products run on tcgen05 with the cached rows as the A operand, so that their cost follows the number of heads:
//   S = K Q^T      64 keys x heads, K-major rows of the stage, into one of two TMEM buffers (lane = key)
//   softmax        a thread per key: common running maximum of every head (moved only when it grows by more than 2^8),
//                  exp2, the weights as a rounded bf16 part beside its remainder in one shared-memory row per key
//   O += V^T P     128 value dims x (2 x heads) per group, the same stage read MN-major; rounded parts and remainders
//                  accumulate in neighbouring TMEM columns (lane = dim) and are added at the end
// Warp roles: 4 softmax / epilogue warps, 1 TMA producer (16-token slabs of pages into a ring of 64-token stages,
// 128-byte swizzle, no multicast) that runs ahead across items, 1 MMA issuer that owns the TMEM allocation.  Every wait
// is bounded and reports MIE_STATUS_WAIT_TIMEOUT.  Scores, weights, sums and O are fp32.  The sink opens the running
// maximum and the denominator of a request's first chunk; partials are merged by merge_rows_kernel.
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
constexpr int kSoftmaxWarps = 4;
constexpr int kLatentThreads = (kSoftmaxWarps + 2) * 32;
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

// Shared memory: ring of stages | Q [box][head][64] | P, two buffers of [key][rounded heads | remainders] | warp maxima
// and sums [warp][head] | barriers.
struct LatentLayout {
  int stage, q, p, maxima, bars, total;
};
constexpr int kPBytes = kStageTokens * 128;
__host__ __device__ inline LatentLayout latent_layout(int key_boxes, int ring, int heads) {
  LatentLayout l;
  l.stage = key_boxes * kStageTokens * 128;
  l.q = ring * l.stage;
  l.p = l.q + key_boxes * heads * 128;
  l.maxima = l.p + 2 * kPBytes;
  l.bars = l.maxima + 2 * kSoftmaxWarps * heads * 4;
  l.total = l.bars + 256;
  return l;
}
constexpr int kMaxRing = 4;
enum LatentBar { kFull = 0, kEmpty = kMaxRing, kQFull = 2 * kMaxRing, kSFull, kPFull = kSFull + 2, kPvDone = kPFull + 2,
                 kOFree = kPvDone + 2, kLatentBars };

__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ float ex2_approx(float x) {  // -inf gives +0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Largest value of the warp in one instruction (warp-wide redux on fp32).
__device__ __forceinline__ float warp_most(float x) {
  float y;
  asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(y) : "f"(x));
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

template <int HN>  // heads per item, 16 or 32
__global__ void __launch_bounds__(kLatentThreads, 1)
    latent_decode_kernel(const __grid_constant__ CUtensorMap map, const LatentParams p) {
  using T = __nv_bfloat16;
  extern __shared__ uint8_t latent_smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>(align_up((long long)reinterpret_cast<uintptr_t>(latent_smem_raw), 1024));
  const LatentLayout at = latent_layout(p.key_boxes, p.ring, HN);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + at.bars);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + kLatentBars);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr uint32_t kTmemCols = 512;
  if (threadIdx.x == 0) {
    for (int s = 0; s < p.ring; ++s) {
      mbar_init(&bars[kFull + s], 1);
      mbar_init(&bars[kEmpty + s], 1);
    }
    mbar_init(&bars[kQFull], kSoftmaxWarps * 32);
    mbar_init(&bars[kOFree], kSoftmaxWarps * 32);
    for (int b = 0; b < 2; ++b) {
      mbar_init(&bars[kSFull + b], 1);
      mbar_init(&bars[kPFull + b], kSoftmaxWarps * 32);
      mbar_init(&bars[kPvDone + b], 1);
    }
    mbar_fence_init();
    tma_prefetch_desc(&map);
  }
  if (warp == kSoftmaxWarps + 1) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = *tmem_slot + 2 * HN;  // S: 2 x HN columns, O: 2 HN columns per group
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
  const int tok_group = p.slab ? p.key_boxes * 1024 : 1024, dim_group = p.slab ? 1024 : kStageTokens * 128;
  const int value_groups = (p.vdim + 127) / 128;

  if (warp == kSoftmaxWarps) {
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
            mbar_expect_tx(&bars[kFull + s], slabs * p.key_boxes * kBoxBytes);
          else
            raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (ok && lane < slabs) {
          uint8_t* dst = smem + s * at.stage;
          if (p.slab) {
            tma_load_5d_hint(dst + lane * p.key_boxes * kBoxBytes, &map, &bars[kFull + s], 0, 0, 0, slot / 8, page, policy);
          } else {
            for (int x = 0; x < p.key_boxes; ++x)
              tma_load_4d_hint(dst + x * dim_group + lane * kBoxBytes, &map, &bars[kFull + s], x * 64, slot, 0, page, policy);
          }
        }
        __syncwarp();
      }
    }
  } else if (warp == kSoftmaxWarps + 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      constexpr uint32_t idesc_s = instr_desc_bf16(64, HN, 0, 0);        // A = K rows, B = Q rows, both K-major
      constexpr uint32_t idesc_o = instr_desc_bf16(128, 2 * HN, 1, 1);   // A = V^T, B = P, both MN-major
      const int k_steps = (p.dim + 15) / 16;
      const uint32_t q_addr = smem_u32(smem + at.q), p_addr = smem_u32(smem + at.p);
      int tile = 0, items = 0;  // stages and items so far
      bool ok = true;
      for (int number = blockIdx.x; number < total_items && ok; number += gridDim.x, ++items) {
        const LatentItem it = item_of(number);
        const int tiles = (int)((it.end - it.begin + kStageTokens - 1) / kStageTokens);
        ok = mbar_wait_bounded(&bars[kQFull], items & 1u);
        // S(j) overwrites the buffer whose P(j - 2) was waited for before P V(j - 2) was issued.
        auto issue_s = [&](int j) {
          const int s = j % p.ring, b = j & 1;
          if (!mbar_wait_bounded(&bars[kFull + s], (j / p.ring) & 1u)) return false;
          tc_fence_after();
          const uint32_t k_addr = smem_u32(smem + s * at.stage);
          for (int ks = 0; ks < k_steps; ++ks)
            umma_f16(tmem_s + b * HN, smem_desc_k128(k_addr + (ks >> 2) * dim_group + (ks & 3) * 32, tok_group),
                     smem_desc_k128(q_addr + (ks >> 2) * (HN * 128) + (ks & 3) * 32), idesc_s, ks > 0 ? 1u : 0u);
          umma_commit(&bars[kSFull + b]);
          return true;
        };
        if (ok) ok = issue_s(tile);
        for (int j = 0; j < tiles && ok; ++j, ++tile) {
          const int s = tile % p.ring, b = tile & 1;
          if (j + 1 < tiles) ok = issue_s(tile + 1);
          if (ok) ok = mbar_wait_bounded(&bars[kPFull + b], (tile >> 1) & 1u);
          if (ok && j == 0 && items > 0) ok = mbar_wait_bounded(&bars[kOFree], (items - 1) & 1u);  // O has been read
          if (!ok) break;
          tc_fence_after();
          const uint32_t v_addr = smem_u32(smem + s * at.stage);
          const int slabs = (it.valid(it.begin + (long long)j * kStageTokens) + kTileTokens - 1) / kTileTokens;
          for (int kt = 0; kt < slabs; ++kt) {
            const uint64_t weights = smem_desc_mn128(p_addr + b * kPBytes + kt * 2048, 1024, 1024);
            for (int d = 0; d < value_groups; ++d)
              umma_f16(tmem_o + d * 2 * HN, smem_desc_mn128(v_addr + 2 * d * dim_group + kt * 2 * tok_group, dim_group, tok_group),
                       weights, idesc_o, j > 0 || kt > 0 ? 1u : 0u);
          }
          umma_commit(&bars[kEmpty + s]);   // the stage is free once these MMAs have read it
          umma_commit(&bars[kPvDone + b]);  // O includes this stage
        }
      }
      if (!ok) raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
    }
  } else {
    // ---------------- Softmax and epilogue: thread = key of a stage, then thread = value dim ----------------
    const uint32_t lane_addr = (uint32_t)(warp * 32) << 16;
    const int key = warp * 16 + lane;  // lanes 0 ... 15
    float* maxima = reinterpret_cast<float*>(smem + at.maxima);  // [warp][head], double-buffered by stage parity
    bool ok = true;
    auto load_q = [&](const LatentItem& it) {
      for (int i = threadIdx.x; i < HN * p.key_boxes * 8; i += kSoftmaxWarps * 32) {
        const int r = i / (p.key_boxes * 8), u = i % (p.key_boxes * 8), head = it.group * HN + r;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (head < p.heads && u * 8 < p.dim)
          v = *reinterpret_cast<const uint4*>(p.q + (it.request * p.q_row + head * p.q_head + u * 8) * 2);
        *reinterpret_cast<uint4*>(smem + at.q + (u >> 3) * (HN * 128) + r * 128 + (((u & 7) ^ (r & 7)) << 4)) = v;
      }
      fence_proxy_async_smem();
      mbar_arrive(&bars[kQFull]);
    };
    LatentItem it;
    int tile = 0;
    if ((int)blockIdx.x < total_items) {
      it = item_of(blockIdx.x);
      load_q(it);
    }
    for (int number = blockIdx.x; number < total_items; number += gridDim.x) {
      const int head0 = it.group * HN;
      float m[HN], l[HN];  // reference maximum (log2 units, the same in every thread); this key's share of the denominator
#pragma unroll
      for (int h = 0; h < HN; ++h) {
        m[h] = -INFINITY;
        l[h] = 0.f;
        if (p.sinks != nullptr && it.chunk == 0) {
          m[h] = head0 + h < p.heads ? p.sinks[head0 + h] * kLog2e : 0.f;
          if (threadIdx.x == 0) l[h] = 1.f;
        }
      }
      bool first = true;
      for (long long tok0 = it.begin; tok0 < it.end; tok0 += kStageTokens, ++tile) {
        const int b = tile & 1, valid = it.valid(tok0);
        if (ok && !mbar_wait_bounded(&bars[kSFull + b], (tile >> 1) & 1u)) ok = false;
        tc_fence_after();
        float s[HN];
        tmem_load<HN>(tmem_s + b * HN + lane_addr, s);
        const bool seen = lane < 16 && key < valid && tok0 + key >= it.first_seen;
        float* mine = maxima + b * kSoftmaxWarps * HN;
        float top = -INFINITY;
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          s[h] = seen ? s[h] * p.scale_log2 : -INFINITY;
          const float most = warp_most(s[h]);
          if (lane == h) top = most;
        }
        if (lane < HN) mine[warp * HN + lane] = top;
        if (valid % kTileTokens != 0) {
          // Rows of the last slab past the read length may hold anything (even NaN bits): zero them so that 0 * V stays 0.
          const int s0 = tile % p.ring, end = (valid + kTileTokens - 1) / kTileTokens * kTileTokens;
          for (int i = threadIdx.x; i < (end - valid) * p.key_boxes * 8; i += kSoftmaxWarps * 32) {
            const int row = valid + i / (p.key_boxes * 8), u = i % (p.key_boxes * 8);
            *reinterpret_cast<uint4*>(smem + s0 * at.stage + (row >> 3) * tok_group + (u >> 3) * dim_group +
                                      (row & 7) * 128 + (u & 7) * 16) = make_uint4(0, 0, 0, 0);
          }
        }
        softmax_sync();
        bool grow = false;  // the same in every thread
        float next[HN];
#pragma unroll
        for (int h = 0; h < HN; h += 4) {
          float4 a = *reinterpret_cast<const float4*>(mine + h);
#pragma unroll
          for (int w = 1; w < kSoftmaxWarps; ++w) {
            const float4 c = *reinterpret_cast<const float4*>(mine + w * HN + h);
            a.x = fmaxf(a.x, c.x), a.y = fmaxf(a.y, c.y), a.z = fmaxf(a.z, c.z), a.w = fmaxf(a.w, c.w);
          }
          next[h] = a.x, next[h + 1] = a.y, next[h + 2] = a.z, next[h + 3] = a.w;
        }
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          // Every stage holds a visible token, so the maximum is finite.
          if (next[h] <= m[h] + kRescaleThreshold) next[h] = m[h];
          grow = grow || next[h] != m[h];
        }
        if (grow) {
          if (!first) {
            // O must first hold every stage before this one; then its columns move to the new reference.
            if (ok && !mbar_wait_bounded(&bars[kPvDone + (b ^ 1)], ((tile - 1) >> 1) & 1u)) ok = false;
            tc_fence_after();
            for (int d = 0; d < value_groups; ++d)
#pragma unroll
              for (int part = 0; part < 2; ++part) {
                const uint32_t addr = tmem_o + d * 2 * HN + part * HN + lane_addr;
                float v[HN];
                tmem_load<HN>(addr, v);
#pragma unroll
                for (int h = 0; h < HN; ++h) v[h] *= ex2_approx(m[h] - next[h]);
                if constexpr (HN == 16)
                  tmem_st16(addr, *reinterpret_cast<const uint32_t(*)[16]>(&v));
                else
                  tmem_st32(addr, *reinterpret_cast<const uint32_t(*)[32]>(&v));
              }
            tmem_st_wait();
          }
#pragma unroll
          for (int h = 0; h < HN; ++h) {
            l[h] *= ex2_approx(m[h] - next[h]);  // 0 * 0 while nothing has been seen
            m[h] = next[h];
          }
        }
        first = false;
        // P(tile) goes where P(tile - 2) was.
        if (ok && tile >= 2 && !mbar_wait_bounded(&bars[kPvDone + b], ((tile - 2) >> 1) & 1u)) ok = false;
        if (lane < 16) {
          uint8_t* row = smem + at.p + b * kPBytes + key * 128;
#pragma unroll
          for (int h = 0; h < HN; h += 8) {
            uint32_t high[4], low[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              const float w0 = ex2_approx(s[h + 2 * j] - m[h + 2 * j]), w1 = ex2_approx(s[h + 2 * j + 1] - m[h + 2 * j + 1]);
              l[h + 2 * j] += w0;
              l[h + 2 * j + 1] += w1;
              high[j] = Mma16816<T>::pack(w0, w1);
              const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high[j]));
              low[j] = Mma16816<T>::pack(w0 - k.x, w1 - k.y);
            }
            *reinterpret_cast<uint4*>(row + (((h >> 3) ^ (key & 7)) << 4)) = make_uint4(high[0], high[1], high[2], high[3]);
            *reinterpret_cast<uint4*>(row + ((((HN + h) >> 3) ^ (key & 7)) << 4)) = make_uint4(low[0], low[1], low[2], low[3]);
          }
        }
        fence_proxy_async_smem();
        tc_fence_before();
        mbar_arrive(&bars[kPFull + b]);
      }
      const LatentItem done = it;
      if (number + (int)gridDim.x < total_items) {  // the next item's queries, while the last products run
        it = item_of(number + gridDim.x);
        load_q(it);
      }
      // Denominators: over the warp, then over the warps.
      float* sums = maxima + (tile & 1) * kSoftmaxWarps * HN;  // not the buffer the last stage's maxima are read from
      float mine = 0.f;
#pragma unroll
      for (int h = 0; h < HN; ++h) {
        const float total = warp_sum(l[h]);
        if (lane == h) mine = total;
      }
      if (lane < HN) sums[warp * HN + lane] = mine;
      softmax_sync();
      const int last = tile - 1;
      if (ok && !mbar_wait_bounded(&bars[kPvDone + (last & 1)], (last >> 1) & 1u)) ok = false;
      tc_fence_after();
#pragma unroll
      for (int h = 0; h < HN; ++h) {
        float total = 0.f;
#pragma unroll
        for (int w = 0; w < kSoftmaxWarps; ++w) total += sums[w * HN + h];
        l[h] = total;
      }
      const long long part0 = ((long long)p.sc.offsets[done.request] + done.chunk) * p.heads + head0;
      if (done.chunks > 1 && threadIdx.x == 0) {
#pragma unroll
        for (int h = 0; h < HN; ++h)
          if (head0 + h < p.heads) {
            p.sc.part_m[part0 + h] = m[h];
            p.sc.part_l[part0 + h] = l[h];
          }
      }
      for (int d = 0; d < value_groups; ++d) {
        float v[HN], r[HN];
        tmem_load<HN>(tmem_o + d * 2 * HN + lane_addr, v);
        tmem_load<HN>(tmem_o + d * 2 * HN + HN + lane_addr, r);
        const int c = d * 128 + warp * 32 + lane;
        if (c >= p.vdim) continue;
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          if (head0 + h >= p.heads) break;
          if (done.chunks == 1)
            reinterpret_cast<T*>(p.out)[done.request * p.o_row + (head0 + h) * p.o_head + c] =
                __float2bfloat16_rn((v[h] + r[h]) / fmaxf(l[h], 1.17549435e-38f));
          else
            p.sc.part_o[(part0 + h) * p.vdim + c] = v[h] + r[h];
        }
      }
      tc_fence_before();
      mbar_arrive(&bars[kOFree]);
      softmax_sync();  // `sums` has been read before the next item's maxima reuse it
    }
    if (!ok && lane == 0) raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
    // Requests with nothing to read (rejected metadata) get zeros.
    for (int e = blockIdx.x * kSoftmaxWarps + warp; e < p.batch; e += gridDim.x * kSoftmaxWarps) {
      if (p.sc.offsets[e + 1] != p.sc.offsets[e]) continue;
      for (int h = 0; h < p.heads; ++h)
        for (int d = 2 * lane; d < p.vdim; d += 64)
          *reinterpret_cast<uint32_t*>(reinterpret_cast<T*>(p.out) + e * p.o_row + h * p.o_head + d) = 0u;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kSoftmaxWarps + 1) {
    tc_fence_after();
    tmem_dealloc(*tmem_slot, kTmemCols);
  }
}

template <int HN>
int launch_latent(const CUtensorMap& map, LatentParams p, cudaStream_t stream) {
  p.ring = 2;
  while (p.ring < kMaxRing && latent_layout(p.key_boxes, p.ring + 1, HN).total + 1024 <= 200 * 1024) ++p.ring;
  const int smem = latent_layout(p.key_boxes, p.ring, HN).total + 1024;
  static int configured[64] = {0};
  int dev = 0;
  MIE_CUDA(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || configured[dev] < smem) {
    MIE_CUDA(cudaFuncSetAttribute(latent_decode_kernel<HN>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    if (dev >= 0 && dev < 64) configured[dev] = smem;
  }
  MIE_CUDA(launch_chained(latent_decode_kernel<HN>, dim3(sm_count()), dim3(kLatentThreads), (size_t)smem, stream, map, p));
  MIE_LAUNCH_CHECK("latent_decode_kernel");
  return MIE_OK;
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
  if (int rc = item_heads == 16 ? launch_latent<16>(map, p, stream) : launch_latent<32>(map, p, stream)) return rc;
  mie_view4_t q{const_cast<void*>(query), {q_row_stride, q_head_stride, 0, 1}};
  mie_view4_t o{out, {o_row_stride, o_head_stride, 0, 1}};
  const DecodeParams merge{View4(q), View4(o), p.tables, p.lengths, IndexView(), sc, batch, heads, 1, heads, block_size,
                           num_blocks, table_width, p.scale_log2, 0, status, nullptr, 0, nullptr, 0, 0, dim, value_dim,
                           head_groups, window, sinks};
  const int boxes = (value_dim + 63) / 64;
  return boxes <= 2 ? launch_latent_merge<2>(merge, stream)
                    : boxes <= 4 ? launch_latent_merge<4>(merge, stream) : launch_latent_merge<8>(merge, stream);
}
