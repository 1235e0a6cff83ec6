// Work planning and the streaming kernel of ragged paged decode attention, shared by the plain entry points
// (decode_attention.cu) and the ones with sinks, windows and other head sizes (sink_decode_attention.cu).
#pragma once

#include "common.cuh"

namespace mie {
namespace {

constexpr int kTileTokens = 16;
constexpr int kBoxBytes = kTileTokens * 128;            // one TMA box: 16 tokens x 64 dims, 128-byte swizzle
constexpr int kPidBatch = 128;                          // tiles whose page ids are staged at once
constexpr int kMinChunk = 64;
constexpr int kMaxChunk = 2048;
constexpr int kPlanThreads = 1024;
constexpr int kHeaderInts = 128;  // [0]=chunk [1]=seq_chunks [2]=items; [16..79] work counters
constexpr int kCounterBase = 16;
constexpr int kCounters = 64;
constexpr int kMaxGroupMerge = 4;  // query heads per KV head the merge kernel handles in one block

// Tile geometry for key rows of KH and value rows of VH 64-dim boxes.  A head size that is no multiple of 64
// leaves the rest of its last box zero-filled by TMA (no HBM traffic).  The ring holds about 24 KiB a warp.
template <int KH, int VH>
struct DecodeTile {
  static constexpr int kKBytes = KH * kBoxBytes;
  static constexpr int kStageBytes = (KH + VH) * kBoxBytes;
  static constexpr int kStages = KH + VH <= 6 ? 12 / (KH + VH) : 2;
  static constexpr int kWarps = KH + VH <= 6 ? 8 : 6;
  static constexpr size_t kSmem = (size_t)kWarps * kStages * kStageBytes + kWarps * kStages * 8 +
                                  (size_t)kWarps * kPidBatch * 4 + 1024;
};
constexpr int kHeadDim = 128;                           // of the plain kernel: two boxes of keys, two of values
constexpr int kWarps = DecodeTile<2, 2>::kWarps;

struct View4 {
  char* ptr;
  long long s[4];
  __host__ View4(const mie_view4_t& v) : ptr(reinterpret_cast<char*>(v.ptr)) {
    for (int i = 0; i < 4; ++i) s[i] = v.stride[i];
  }
};

struct Scratch {
  int* header;
  int* offsets;     // [batch + 1]
  int* item_seq;    // [cap]
  int* item_chunk;  // [cap]
  float* part_m;    // [cap][q_heads]
  float* part_l;    // [cap][q_heads]
  float* part_o;    // [cap][q_heads][head_dim]
  int cap;
};

template <typename T>
__device__ __forceinline__ float round_act(float v) {
  return to_float<T>(from_float<T>(v));
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
__host__ __device__ inline long long align_up(long long v, long long a) { return (v + a - 1) / a * a; }

// Attention read length of request b, or 0 (with a status bit) when the
// metadata is unusable.
__device__ __forceinline__ long long read_length(const IndexView& lengths, const IndexView& positions, int b,
                                                 long long capacity, int* status) {
  const long long len = lengths.at(b);
  if (len < 1 || len > capacity) {
    raise_status(status, MIE_STATUS_BAD_LENGTH);
    return 0;
  }
  if (!positions.valid()) return len;
  const long long pos = positions.at(b);
  if (pos < 0) {
    raise_status(status, MIE_STATUS_BAD_POSITION);
    return 0;
  }
  return pos + 1 < len ? pos + 1 : len;
}

// First token a windowed row reads: the last `window` tokens, from a tile border.  window 0: no window.
__device__ __forceinline__ long long window_start(long long read_len, long long window) {
  return window > 0 && read_len > window ? (read_len - window) / kTileTokens * kTileTokens : 0;
}

// ---------------------------------------------------------------------------
// Plan kernel: one CTA.
// ---------------------------------------------------------------------------
__device__ __forceinline__ long long block_sum_ll(long long v, long long* smem) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if (lane == 0) smem[warp] = v;
  __syncthreads();
  long long t = 0;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += smem[i];
  __syncthreads();
  return t;
}

// Split-KV planning.  The decode kernel is a dynamic queue of (request, chunk, KV head) items over
// `warps` persistent warps, so its time is close to
//     ceil(items / warps) x (time of one chunk + what a warp loses between two items),
// with items = kv_heads x sum_b ceil(length_b / chunk).  Policy 1 evaluates that with the batch's real
// lengths for a grid of chunk sizes and takes the cheapest: a chunk size that just misses a whole number of
// rounds costs a full extra round on a few warps (see the limit below for where this applies).
// `switch_tokens` is the between-items loss (queue pop,
// metadata, refilling the TMA ring, writing and later merging a partial) expressed in tokens of streaming;
// 128 tokens of one bf16 KV head (64 KB) reproduces the measured ranking of chunk sizes on an 8-way
// head shard (384 and 1024 tokens best, 512 and 192 worst).
constexpr int kPlanCands = 21;
// Candidate j (compile-time in the unrolled loops, so the divisions below are by constants).
__host__ __device__ constexpr int plan_chunk(int j) {
  constexpr int table[kPlanCands] = {64,  80,  96,  112, 128, 160, 192,  224,  256,  320, 384,
                                     448, 512, 640, 768, 896, 1024, 1280, 1536, 1792, 2048};
  return table[j];
}

__global__ void __launch_bounds__(kPlanThreads) plan_kernel(IndexView lengths, IndexView positions, int batch,
                                                            long long capacity_tokens, int kv_heads, int policy,
                                                            int warps, int switch_tokens, long long window, Scratch sc,
                                                            int* status) {
  __shared__ long long red[32];
  __shared__ int warp_tot[32];
  __shared__ int cand_part[32][kPlanCands];
  __shared__ int cand_count[kPlanCands];
  __shared__ int running_s;
  __shared__ long long chunk_s;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  chain_wait();
  chain_release();

  // With one thread per request (the usual launch) a request's length is read once and kept.
  const bool one_each = batch <= (int)blockDim.x;
  auto span = [&](int b, int* report) {  // tokens request b reads
    const long long rl = read_length(lengths, positions, b, capacity_tokens, report);
    return rl - window_start(rl, window);
  };
  long long own = 0, local = 0;
  if (one_each) {
    if (tid < batch) own = span(tid, status);
    local = own;
  } else {
    for (int b = tid; b < batch; b += blockDim.x) local += span(b, status);
  }
  const long long total = block_sum_ll(local, red);
  const long long room = sc.cap - batch;  // > 0, checked on the host

  long long chunk;
  if (policy == 0) {
    chunk = (1ll << 40);
  } else if (policy == 1) {
    int mine[kPlanCands];
#pragma unroll
    for (int j = 0; j < kPlanCands; ++j) mine[j] = 0;
    for (int b = tid; b < batch; b += blockDim.x) {
      const int rl = (int)(one_each ? own : span(b, nullptr));
#pragma unroll
      for (int j = 0; j < kPlanCands; ++j) mine[j] += (rl + plan_chunk(j) - 1) / plan_chunk(j);
    }
#pragma unroll
    for (int j = 0; j < kPlanCands; ++j) {
      int v = mine[j];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if (lane == 0) cand_part[warp][j] = v;
    }
    __syncthreads();
    if (tid < kPlanCands) {
      int t = 0;
      for (int w = 0; w < (int)(blockDim.x >> 5); ++w) t += cand_part[w][tid];
      cand_count[tid] = t;
    }
    __syncthreads();
    if (tid == 0) {
      // With several KV heads per rank and enough work for four items of at least 512 tokens per warp the kernel is bound by
      // HBM, not by the queue's rounds, and finer items measured better (C=256 at 1 / 2 ranks): there the
      // chunk stays at or below the four-items-per-warp size.  A single KV head per rank, or a batch too
      // small for that, is where whole rounds decide.
      long long limit = kMaxChunk;
      if (kv_heads >= 2) {
        const long long four = align_up((total * kv_heads + 4ll * warps - 1) / (4ll * warps), kTileTokens);
        if (four >= 512) limit = four;
      }
      long long best = plan_chunk(0);
      long long best_cost = -1;
#pragma unroll
      for (int j = kPlanCands - 1; j >= 0; --j) {  // larger chunks first: they win ties (fewer partials)
        if (plan_chunk(j) > limit && j > 0) continue;
        if (cand_count[j] > sc.cap) continue;      // more (request, chunk) pairs than the scratch holds
        const long long items = (long long)cand_count[j] * kv_heads;
        const long long rounds = (items + warps - 1) / warps;
        const long long cost = rounds * (plan_chunk(j) + switch_tokens);
        if (best_cost < 0 || cost < best_cost) {
          best_cost = cost;
          best = plan_chunk(j);
        }
      }
      chunk_s = best;
    }
    __syncthreads();
    chunk = chunk_s;
  } else {
    chunk = align_up(policy, kTileTokens);
  }
  // Never emit more (request, chunk) pairs than the caller's scratch holds.
  if (total / chunk + batch > sc.cap) {
    chunk = align_up((total + room - 1) / room, kTileTokens);  // still exact, only coarser
  }

  // Work list in request order, a request's chunks next to each other (queueing the full-sized chunks of
  // all requests first and the shorter last chunks at the end was measured 2 % slower at the same chunk size:
  // neighbouring items then no longer read neighbouring pages).
  if (tid == 0) running_s = 0;
  __syncthreads();
  for (int base = 0; base < batch; base += blockDim.x) {
    const int b = base + tid;
    int c = 0;
    if (b < batch) {
      const long long rl = one_each ? own : span(b, nullptr);
      c = (int)((rl + chunk - 1) / chunk);
    }
    int incl = c;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int n = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += n;
    }
    if (lane == 31) warp_tot[warp] = incl;
    __syncthreads();
    int before = running_s;
    for (int w = 0; w < warp; ++w) before += warp_tot[w];
    const int excl = before + incl - c;
    if (b < batch) {
      sc.offsets[b] = excl;
      for (int j = 0; j < c; ++j) {
        sc.item_seq[excl + j] = b;
        sc.item_chunk[excl + j] = j;
      }
    }
    __syncthreads();
    if (tid == 0) {
      int t = 0;
      for (int w = 0; w < (int)(blockDim.x >> 5); ++w) t += warp_tot[w];
      running_s += t;
    }
    __syncthreads();
  }
  const int pairs = running_s;
  if (tid == 0) {
    sc.offsets[batch] = pairs;
    sc.header[0] = (int)(chunk > 0x7fffffffll ? 0x7fffffff : chunk);
    sc.header[1] = pairs;
    sc.header[2] = pairs * kv_heads;
  }
  if (tid < kCounters) sc.header[kCounterBase + tid] = 0;
}

// ---------------------------------------------------------------------------
// Main kernel
// ---------------------------------------------------------------------------
struct DecodeParams {
  View4 q, out;
  IndexView tables, lengths, positions;
  Scratch sc;
  int batch, q_heads, kv_heads, group, block_size, num_blocks, table_width;
  float scale_log2;
  int counter_slot;
  int* status;
  uint8_t* out_q8;     // optional e4m3 copy of the output for the next FP8 GEMM: [batch][ldq8 bytes]
  long long ldq8;
  float* out_scales;   // [q_heads][out_scale_ld]: one scale per (head, request) = per 128 columns
  int out_scale_ld;
  int merge_head0;     // first head of the group handled by this merge launch
  // The extended kernel only: head sizes, work items per request and chunk (KV heads x query sub-groups of
  // eight), sliding window (0: none), one sink score per query head (null: none).
  int dim, vdim, item_heads;
  long long window;
  const float* sinks;
};

// kExt = false: head_dim 128, GQA group <= 8, scores rounded to the activation dtype as the reference's bf16
// product is.  kExt = true: other head sizes, any group, fp32 scores, sliding window, sinks, no e4m3 output.
template <typename T, int KH, int VH, bool kExt>
__global__ void __launch_bounds__(DecodeTile<KH, VH>::kWarps * 32, 1)
    decode_kernel(const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap,
                  const DecodeParams p) {
  using Tile = DecodeTile<KH, VH>;
  constexpr int kWarps = Tile::kWarps, kStages = Tile::kStages, kStageBytes = Tile::kStageBytes;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>(align_up((long long)reinterpret_cast<uintptr_t>(smem_raw), 1024));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  uint8_t* stages = smem + (size_t)warp * kStages * kStageBytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + (size_t)kWarps * kStages * kStageBytes) + warp * kStages;
  int* pids = reinterpret_cast<int*>(smem + (size_t)kWarps * kStages * kStageBytes + kWarps * kStages * 8) +
              warp * kPidBatch;

  if (lane == 0) {
    for (int s = 0; s < kStages; ++s) mbar_init(&bars[s], 1);
    mbar_fence_init();
    tma_prefetch_desc(&kmap);
    tma_prefetch_desc(&vmap);
  }
  __syncthreads();
  chain_wait();
  chain_release();

  const int g = lane >> 2, t = lane & 3;
  const int chunk = p.sc.header[0];
  const int total_items = p.sc.header[2];
  int* counter = p.sc.header + kCounterBase + p.counter_slot;
  const long long capacity_tokens = (long long)p.table_width * p.block_size;
  uint32_t parity = 0;
  const uint64_t stream_policy = l2_evict_first_policy();  // K/V pages are read once per step

  // ldmatrix lane geometry (constant per lane).
  const int k_tok = (lane & 7) + ((lane >> 4) & 1) * 8, k_sel = (lane >> 3) & 1;
  const int v_tok = (lane & 7) + ((lane >> 3) & 1) * 8, v_sel = (lane >> 4) & 1;
  const uint32_t k_row = k_tok * 128, k_key = k_tok & 7;
  const uint32_t v_row = v_tok * 128, v_key = v_tok & 7;

  while (true) {
    int item = 0;
    if (lane == 0) item = atomicAdd(counter, 1);
    item = __shfl_sync(0xffffffffu, item, 0);
    if (item >= total_items) break;
    const int item_heads = kExt ? p.item_heads : p.kv_heads;
    const int sci = item / item_heads, hi = item % item_heads;
    const int subs = kExt ? item_heads / p.kv_heads : 1;          // query sub-groups of a KV head
    const int h = kExt ? hi / subs : hi, sub0 = kExt ? (hi % subs) * 8 : 0;
    const int rows = kExt && p.group - sub0 > 8 ? 8 : p.group - sub0;  // query heads of this item
    const int b = p.sc.item_seq[sci], ck = p.sc.item_chunk[sci];
    const long long rl = read_length(p.lengths, p.positions, b, capacity_tokens, nullptr);
    const int nchunks = p.sc.offsets[b + 1] - p.sc.offsets[b];
    const long long first = kExt ? window_start(rl, p.window) : 0;
    const long long first_seen = kExt && p.window > 0 && rl > p.window ? rl - p.window : 0;
    const long long t_begin = first + (long long)ck * chunk;
    const long long t_end = rl < t_begin + chunk ? rl : t_begin + chunk;
    const int ntiles = (int)((t_end - t_begin + kTileTokens - 1) / kTileTokens);

    // Query fragments: rows g < group are real heads, the rest of the 16 MMA rows are zero.
    uint32_t qa[KH * 4][2];
    {
      const bool real = g < rows;
      const T* qrow = reinterpret_cast<const T*>(p.q.ptr) + (long long)b * p.q.s[0] +
                      (long long)(h * p.group + sub0 + (real ? g : 0)) * p.q.s[1];
#pragma unroll
      for (int ks = 0; ks < KH * 4; ++ks) {
        // Head sizes of the extended kernel are multiples of 8: an 8-dim half group is inside the row or past it.
        const bool in_lo = !kExt || ks * 16 < p.dim, in_hi = !kExt || ks * 16 + 8 < p.dim;
        const uint32_t lo = in_lo ? *reinterpret_cast<const uint32_t*>(qrow + ks * 16 + 2 * t) : 0u;
        const uint32_t hi = in_hi ? *reinterpret_cast<const uint32_t*>(qrow + ks * 16 + 8 + 2 * t) : 0u;
        qa[ks][0] = real ? lo : 0u;
        qa[ks][1] = real ? hi : 0u;
      }
    }

    float m = -INFINITY, l = 0.f;
    if (kExt && p.sinks != nullptr && ck == 0) {
      // The sink opens the softmax of a request's first chunk: running maximum and one unit of denominator.
      m = g < rows ? p.sinks[h * p.group + sub0 + g] * 1.4426950408889634f : 0.f;
      l = t == 0 ? 1.f : 0.f;
    }
    float o[VH * 8][4];
#pragma unroll
    for (int n = 0; n < VH * 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    bool timed_out = false;
    for (int batch0 = 0; batch0 < ntiles && !timed_out; batch0 += kPidBatch) {
      const int nb = ntiles - batch0 < kPidBatch ? ntiles - batch0 : kPidBatch;
      __syncwarp();
      for (int i = lane; i < nb; i += 32) {
        const long long tok = t_begin + (long long)(batch0 + i) * kTileTokens;
        long long pid = p.tables.at(b, tok / p.block_size);
        if (pid < 0 || pid >= p.num_blocks) {
          raise_status(p.status, MIE_STATUS_BAD_PAGE);
          pid = 0;
        }
        pids[i] = (int)pid;
      }
      __syncwarp();
      auto issue = [&](int i) {
        const int s = i % kStages;
        const long long tok = t_begin + (long long)(batch0 + i) * kTileTokens;
        const int tok_in_page = (int)(tok % p.block_size);
        uint8_t* dst = stages + (size_t)s * kStageBytes;
        mbar_expect_tx(&bars[s], kStageBytes);
#pragma unroll
        for (int x = 0; x < KH; ++x)
          tma_load_4d_hint(dst + x * kBoxBytes, &kmap, &bars[s], x * 64, tok_in_page, h, pids[i], stream_policy);
#pragma unroll
        for (int x = 0; x < VH; ++x)
          tma_load_4d_hint(dst + (KH + x) * kBoxBytes, &vmap, &bars[s], x * 64, tok_in_page, h, pids[i],
                           stream_policy);
      };
      if (lane == 0) {
        for (int i = 0; i < kStages && i < nb; ++i) issue(i);
      }
      for (int i = 0; i < nb; ++i) {
        const int s = i % kStages;
        const bool arrived = mbar_wait_bounded(&bars[s], (parity >> s) & 1u);
        if (!__all_sync(0xffffffffu, arrived)) {
          timed_out = true;
          break;
        }
        parity ^= 1u << s;
        const uint32_t kbase = smem_u32(stages + (size_t)s * kStageBytes);
        const uint32_t vbase = kbase + Tile::kKBytes;
        const long long tok0 = t_begin + (long long)(batch0 + i) * kTileTokens;
        const int valid = (int)(t_end - tok0 < kTileTokens ? t_end - tok0 : kTileTokens);

        if (valid < kTileTokens) {
          // Rows past the read length may hold anything (even NaN bits): zero
          // them in V so that 0 * V stays 0.  K rows are masked by select below.
          uint8_t* vt = stages + (size_t)s * kStageBytes + Tile::kKBytes;
          for (int c = lane; c < VH * kTileTokens * 8; c += 32) {
            const int half = c / (kTileTokens * 8), rem = c % (kTileTokens * 8);
            const int row = rem / 8;
            if (row >= valid) {
              *reinterpret_cast<uint4*>(vt + half * kBoxBytes + row * 128 + (rem % 8) * 16) =
                  make_uint4(0, 0, 0, 0);
            }
          }
          fence_proxy_async_smem();
          __syncwarp();
        }

        // S = Q K^T for 16 tokens: two n-tiles, two accumulator sets to shorten the chain.
        float sa[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        float sb[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int ks = 0; ks < KH * 4; ++ks) {
          const uint32_t addr =
              kbase + (ks >> 2) * kBoxBytes + k_row + (((((ks & 3) * 2) | k_sel) ^ k_key) << 4);
          uint32_t r0, r1, r2, r3;
          ldmatrix_x4(r0, r1, r2, r3, addr);
          if (ks & 1) {
            Mma16816<T>::run(sb[0], qa[ks][0], 0u, qa[ks][1], 0u, r0, r1);
            Mma16816<T>::run(sb[1], qa[ks][0], 0u, qa[ks][1], 0u, r2, r3);
          } else {
            Mma16816<T>::run(sa[0], qa[ks][0], 0u, qa[ks][1], 0u, r0, r1);
            Mma16816<T>::run(sa[1], qa[ks][0], 0u, qa[ks][1], 0u, r2, r3);
          }
        }
        // This lane's four scores of head g: tokens 2t, 2t+1, 8+2t, 9+2t.  The reference keeps the
        // Q.K^T product in the activation dtype (a bf16/fp16 bmm per page) before the fp32 softmax;
        // rounding the fp32 dot product once reproduces that.
        float sv[4];
        sv[0] = (kExt ? sa[0][0] + sb[0][0] : round_act<T>(sa[0][0] + sb[0][0])) * p.scale_log2;
        sv[1] = (kExt ? sa[0][1] + sb[0][1] : round_act<T>(sa[0][1] + sb[0][1])) * p.scale_log2;
        sv[2] = (kExt ? sa[1][0] + sb[1][0] : round_act<T>(sa[1][0] + sb[1][0])) * p.scale_log2;
        sv[3] = (kExt ? sa[1][1] + sb[1][1] : round_act<T>(sa[1][1] + sb[1][1])) * p.scale_log2;
        const int tk = 2 * t;
        if (tk >= valid) sv[0] = -INFINITY;
        if (tk + 1 >= valid) sv[1] = -INFINITY;
        if (tk + 8 >= valid) sv[2] = -INFINITY;
        if (tk + 9 >= valid) sv[3] = -INFINITY;
        if (kExt && tok0 < first_seen) {  // the window's first tile: at least one of its tokens is inside
          const int hidden = (int)(first_seen - tok0);
          if (tk < hidden) sv[0] = -INFINITY;
          if (tk + 1 < hidden) sv[1] = -INFINITY;
          if (tk + 8 < hidden) sv[2] = -INFINITY;
          if (tk + 9 < hidden) sv[3] = -INFINITY;
        }
        float mx = fmaxf(fmaxf(sv[0], sv[1]), fmaxf(sv[2], sv[3]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m, mx);  // finite: every tile has a token that is seen
        const float alpha = exp2f(m - m_new);
        const float p0 = exp2f(sv[0] - m_new), p1 = exp2f(sv[1] - m_new);
        const float p2 = exp2f(sv[2] - m_new), p3 = exp2f(sv[3] - m_new);
        l = l * alpha + ((p0 + p1) + (p2 + p3));
        m = m_new;
        // P.V runs on the tensor cores in the activation dtype; the reference multiplies fp32 weights by
        // fp32 V, so P is split into a rounded part and its remainder (two MMAs) to keep ~16 more bits.
        const uint32_t pa0 = Mma16816<T>::pack(p0, p1), pa2 = Mma16816<T>::pack(p2, p3);
        const uint32_t pb0 = Mma16816<T>::pack(p0 - round_act<T>(p0), p1 - round_act<T>(p1));
        const uint32_t pb2 = Mma16816<T>::pack(p2 - round_act<T>(p2), p3 - round_act<T>(p3));
#pragma unroll
        for (int n = 0; n < VH * 8; ++n) {
          o[n][0] *= alpha;
          o[n][1] *= alpha;
        }
        // O += P V
#pragma unroll
        for (int np = 0; np < VH * 4; ++np) {
          const uint32_t addr =
              vbase + (np >> 2) * kBoxBytes + v_row + (((((np & 3) * 2) | v_sel) ^ v_key) << 4);
          uint32_t r0, r1, r2, r3;
          ldmatrix_x4_trans(r0, r1, r2, r3, addr);
          Mma16816<T>::run(o[2 * np], pa0, 0u, pa2, 0u, r0, r1);
          Mma16816<T>::run(o[2 * np + 1], pa0, 0u, pa2, 0u, r2, r3);
          Mma16816<T>::run(o[2 * np], pb0, 0u, pb2, 0u, r0, r1);
          Mma16816<T>::run(o[2 * np + 1], pb0, 0u, pb2, 0u, r2, r3);
        }
        __syncwarp();
        if (lane == 0 && i + kStages < nb) issue(i + kStages);
      }
    }
    if (timed_out) {
      if (lane == 0) raise_status(p.status, MIE_STATUS_WAIT_TIMEOUT);
      break;
    }

    // Row sum over the quad, then write the result (final or partial).
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    const bool head_live = g < rows;
    const int head = h * p.group + sub0 + (head_live ? g : 0);
    const int out_dim = kExt ? p.vdim : kHeadDim;
    if (nchunks == 1) {
      const float inv = 1.f / fmaxf(l, 1.17549435e-38f);
      T* orow = reinterpret_cast<T*>(p.out.ptr) + (long long)b * p.out.s[0] + (long long)head * p.out.s[1];
      float amax = 0.f;
#pragma unroll
      for (int n = 0; n < VH * 8; ++n) {
        if (n * 8 >= out_dim) break;
        o[n][0] = round_act<T>(o[n][0] * inv);  // the stored (and quantised) value is the rounded one
        o[n][1] = round_act<T>(o[n][1] * inv);
        amax = fmaxf(amax, fmaxf(fabsf(o[n][0]), fabsf(o[n][1])));
        if (head_live) *reinterpret_cast<uint32_t*>(orow + n * 8 + 2 * t) = Mma16816<T>::pack(o[n][0], o[n][1]);
      }
      if (!kExt && p.out_q8 != nullptr) {
        amax = fmaxf(amax, __shfl_xor_sync(0xffffffffu, amax, 1));
        amax = fmaxf(amax, __shfl_xor_sync(0xffffffffu, amax, 2));
        const float scale = __fdiv_rn(amax, 448.0f), denom = fmaxf(scale, 1e-12f);
        if (head_live) {
          uint8_t* qrow = p.out_q8 + (long long)b * p.ldq8 + head * kHeadDim;
#pragma unroll
          for (int n = 0; n < VH * 8; ++n) {
            *reinterpret_cast<__nv_fp8x2_storage_t*>(qrow + n * 8 + 2 * t) = __nv_cvt_float2_to_fp8x2(
                make_float2(__fdiv_rn(o[n][0], denom), __fdiv_rn(o[n][1], denom)), __NV_SATFINITE, __NV_E4M3);
          }
          if (t == 0) p.out_scales[(long long)head * p.out_scale_ld + b] = scale;
        }
      }
    } else {
      const long long first_row = (long long)p.sc.offsets[b] * p.q_heads;
      if (head_live) {
        const long long row = first_row + (long long)ck * p.q_heads + head;
        float* po = p.sc.part_o + row * out_dim;
#pragma unroll
        for (int n = 0; n < VH * 8; ++n) {
          if (n * 8 >= out_dim) break;
          *reinterpret_cast<float2*>(po + n * 8 + 2 * t) = make_float2(o[n][0], o[n][1]);
        }
        if (t == 0) {
          p.sc.part_m[row] = m;
          p.sc.part_l[row] = l;
        }
      }
    }
  }

  // Requests with nothing to read (rejected metadata) get zeros.
  const int warps_total = gridDim.x * kWarps;
  for (int e = blockIdx.x * kWarps + warp; e < p.batch; e += warps_total) {
    if (p.sc.offsets[e + 1] != p.sc.offsets[e]) continue;
    for (int hq = 0; hq < p.q_heads; ++hq) {
      T* orow = reinterpret_cast<T*>(p.out.ptr) + (long long)e * p.out.s[0] + (long long)hq * p.out.s[1];
      if (kExt) {
        for (int d = 2 * lane; d < p.vdim; d += 64) *reinterpret_cast<uint32_t*>(orow + d) = 0u;
        continue;
      }
      *reinterpret_cast<uint2*>(orow + 4 * lane) = make_uint2(0u, 0u);
      if (p.out_q8 != nullptr) {
        *reinterpret_cast<uint32_t*>(p.out_q8 + (long long)e * p.ldq8 + hq * kHeadDim + 4 * lane) = 0u;
        if (lane == 0) p.out_scales[(long long)hq * p.out_scale_ld + e] = 0.f;
      }
    }
  }
}

// Split-KV partials of the extended kernels: one block per (request, query head), values of up to VH 64-dim boxes.
constexpr int kMergeWarps = 4;

template <typename T, int VH>
__global__ void __launch_bounds__(kMergeWarps * 32) merge_rows_kernel(DecodeParams p) {
  __shared__ float part[kMergeWarps][2 + VH * 64];
  chain_wait();
  chain_release();
  const int b = blockIdx.x / p.q_heads, head = blockIdx.x % p.q_heads;
  const int first = p.sc.offsets[b], n = p.sc.offsets[b + 1] - first;
  if (n <= 1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float big = -INFINITY, lsum = 0.f, acc[VH][2];
#pragma unroll
  for (int x = 0; x < VH; ++x) acc[x][0] = acc[x][1] = 0.f;
#pragma unroll 4
  for (int i = warp; i < n; i += kMergeWarps) {
    const long long row = ((long long)first + i) * p.q_heads + head;
    const float mi = p.sc.part_m[row], li = p.sc.part_l[row];
    const float mn = fmaxf(big, mi);
    const float wo = exp2f(big - mn), wi = exp2f(mi - mn);
    lsum = lsum * wo + li * wi;
    big = mn;
#pragma unroll
    for (int x = 0; x < VH; ++x) {
      const int d = x * 64 + 2 * lane;
      if (d < p.vdim) {
        const float2 o = *reinterpret_cast<const float2*>(p.sc.part_o + row * p.vdim + d);
        acc[x][0] = acc[x][0] * wo + o.x * wi;
        acc[x][1] = acc[x][1] * wo + o.y * wi;
      }
    }
  }
  float* mine = part[warp];
  if (lane == 0) {
    mine[0] = big;
    mine[1] = lsum;
  }
#pragma unroll
  for (int x = 0; x < VH; ++x) {
    mine[2 + x * 64 + 2 * lane] = acc[x][0];
    mine[2 + x * 64 + 2 * lane + 1] = acc[x][1];
  }
  __syncthreads();
  if (warp != 0) return;
  big = -INFINITY;
  for (int w = 0; w < kMergeWarps; ++w) big = fmaxf(big, part[w][0]);
  lsum = 0.f;
#pragma unroll
  for (int x = 0; x < VH; ++x) acc[x][0] = acc[x][1] = 0.f;
  for (int w = 0; w < kMergeWarps; ++w) {
    const float mw = part[w][0];
    if (mw == -INFINITY) continue;  // this warp had no chunk
    const float wt = exp2f(mw - big);
    lsum += part[w][1] * wt;
#pragma unroll
    for (int x = 0; x < VH; ++x) {
      acc[x][0] += part[w][2 + x * 64 + 2 * lane] * wt;
      acc[x][1] += part[w][2 + x * 64 + 2 * lane + 1] * wt;
    }
  }
  const float inv = 1.f / fmaxf(lsum, 1.17549435e-38f);
  T* orow = reinterpret_cast<T*>(p.out.ptr) + (long long)b * p.out.s[0] + (long long)head * p.out.s[1];
#pragma unroll
  for (int x = 0; x < VH; ++x) {
    const int d = x * 64 + 2 * lane;
    if (d < p.vdim) *reinterpret_cast<uint32_t*>(orow + d) = Mma16816<T>::pack(acc[x][0] * inv, acc[x][1] * inv);
  }
}

long long fixed_scratch_bytes(int batch, int kv_heads) {
  (void)kv_heads;
  return kHeaderInts * 4 + align_up((long long)(batch + 1) * 4, 256);
}
long long per_chunk_bytes(int q_heads, int head_dim) { return 8 + (long long)q_heads * (head_dim + 2) * 4; }

// (request, chunk) pairs `mie_decode_scratch_bytes` makes room for beyond one per request: four items per
// warp.  The plan kernel considers more items per warp only while they fit the scratch it was given.
// One thread per request, at least two warps, at most the kernel's bound: a small batch does not pay for
// block-wide reductions over 32 warps.
int plan_threads(int batch) {
  const int threads = (batch + 31) / 32 * 32;
  return threads < 64 ? 64 : threads > kPlanThreads ? kPlanThreads : threads;
}

int target_seq_chunks(int kv_heads) {
  const int items = sm_count() * kWarps * 4;
  return (items + kv_heads - 1) / kv_heads;
}

Scratch carve(void* scratch, long long bytes, int batch, int q_heads, int kv_heads, int head_dim) {
  Scratch s;
  char* base = reinterpret_cast<char*>(scratch);
  s.header = reinterpret_cast<int*>(base);
  s.offsets = reinterpret_cast<int*>(base + kHeaderInts * 4);
  long long off = fixed_scratch_bytes(batch, kv_heads);
  const long long avail = bytes - off - 1024;
  long long cap = avail / per_chunk_bytes(q_heads, head_dim);
  if (cap > 0x3fffffff) cap = 0x3fffffff;
  s.cap = (int)(cap > 0 ? cap : 0);
  s.item_seq = reinterpret_cast<int*>(base + off);
  off += align_up((long long)s.cap * 4, 256);
  s.item_chunk = reinterpret_cast<int*>(base + off);
  off += align_up((long long)s.cap * 4, 256);
  s.part_m = reinterpret_cast<float*>(base + off);
  off += align_up((long long)s.cap * q_heads * 4, 256);
  s.part_l = reinterpret_cast<float*>(base + off);
  off += align_up((long long)s.cap * q_heads * 4, 256);
  s.part_o = reinterpret_cast<float*>(base + off);
  return s;
}

}  // namespace

// Defined in decode_attention.cu: cached 4-D tensor map over [pages, kv_heads, page, dim], box 16 tokens x 64 dims.
int page_tensor_map(const mie_view4_t& pages, int num_blocks, int kv_heads, int block_size, int dim, int dtype,
                    CUtensorMap* out);

}  // namespace mie
