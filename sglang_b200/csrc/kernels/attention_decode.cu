// Decode attention for sm_100a with the MMA operands SWAPPED: the 128 KEYS of a tile are the UMMA M dimension, the (few) query heads that
// share a KV head are the UMMA N dimension.
//
// Why (profiles/attention_persist_r1.md): in the query-major kernel (attention_tc.cu) a decode item uses G = 4
// of the 128 rows of every S / O tile, one softmax warp of four does all the exponentials (64 per thread per 64-key tile), the Q box drags
// 32 KB through TMA to use 1 KB, and the tensor pipe spends 512 cycles per 16 KB of KV on rows that carry nothing.  Transposed:
//
//     S^T[128 keys, NQ]  = K_tile[128 keys, 128 d] . Q^T            (A = K from smem, K-major;  B = Q, NQ = 16 padded query rows)
//     O^T[128 d,   NQ]  += V_tile^T[128 d, 128 keys] . P^T            (A = V from smem, MN-major; B = P^T from smem, K-major)
//
//   * every TMEM lane / softmax thread owns ONE KEY: G exponentials per thread per 128-key tile, all 128 threads busy;
//   * tensor time per 64 KB of KV: 16 MMAs of 128x16x16 (~0.2 us) instead of 2 x 12 of 128x64/128x16 — the kernel is pure streaming;
//   * Q is 2 x [16 rows x 128 B] = 4 KB of smem (G rows live), which pays for a 3-deep ring of 32 KB K and V tiles: 192 KB of KV in
//     flight per SM, one persistent CTA per SM, work items (request, kv head, split) from an atomic queue;
//   * only the pages that hold keys < seq_len are fetched (expect_tx is sized per tile), so the ragged tail costs pages, not tiles;
//   * row max: warp shuffle + one named barrier per tile; row SUM is kept per thread and reduced once per item; lazy O rescale (FA4).
//
// Hand-offs use one barrier per *meaning* (no waiting on a shared barrier by tile parity — see the o_final note in attention_tc.cu).
//
// Stands in for the reference's trtllm-gen decode kernel (python/sglang/srt/layers/attention/trtllm_mha_backend.py:1470) and the Triton
// split-KV decode kernel (kernels/ops/attention/decode_attention.py:472).
#include <math.h>

// Round-2 experiments that did NOT pay and were removed again (numbers: profiles/attn_decode_r2.md, profiles/tma_gather_r2.md):
//   * two softmax groups on alternating tiles (the consumer was not the limiter);
//   * separate K / V producer warps + one 5-D TMA box per V page (fewer issues per thread; same speed, slower on ragged batches);
//   * an L2 prefetcher warp running ahead of the work queue (extra TMA traffic cost more than the added bytes in flight gave).
// The kernel sits on the loaded-latency curve of the paged gather: throughput ~ bytes in flight per SM, and 192 KB of smem rings is all there is.
#include "common.cuh"
#include "tma_host.h"

#include <algorithm>

namespace sglb {

constexpr int DA_D = 128;                 // head dim
constexpr int DA_KT = 128;                // keys per tile (UMMA M)
constexpr int DA_NQ = 16;                 // padded query rows (UMMA N)
constexpr int DA_THREADS = 192;           // warp 0 producer, warp 1 MMA, warps 2-5 softmax (one key per thread)
constexpr int DA_STAGES = 3;
constexpr int DA_TILE_BYTES = DA_KT * DA_D * 2;          // 32 KB  (K or V tile: two 64-wide d halves of [128 keys x 128 B])
constexpr int DA_HALF_BYTES = DA_TILE_BYTES / 2;
constexpr int DA_Q_BYTES = 2 * DA_NQ * 128;              // 4 KB   (two d halves of [16 rows x 128 B])
constexpr int DA_P_BYTES = 2 * DA_NQ * 128;              // 4 KB   (two 64-key chunks of [16 rows x 128 B]), double buffered
constexpr int DA_SMEM_BYTES = 2 * DA_STAGES * DA_TILE_BYTES + 2 * DA_Q_BYTES + 2 * DA_P_BYTES + 1024 /*align*/ + 1024 /*barriers + scratch*/;
constexpr float DA_RESCALE_THRESHOLD = 8.0f;

constexpr int DA_PLAIN = 0, DA_CAP = 1, DA_DIFF = 2;      // MODE of a kernel instance

struct DecodeParams {
  __nv_bfloat16* out;     // [B, Hq, D]
  float* part_o;          // [splits, B, Hq, D]
  float* part_lse;        // [splits, B, Hq]
  float* lse;             // optional [B, Hq]
  const int* page_table;
  const int* req_slots;
  const int* seq_lens;
  int pt_stride, Hq, Hkv, G, page_size, num_splits, B;
  float scale_log2, logit_cap;
  const float* slopes;      // optional [Hq]: distance bias, score -= slopes[h] * (seq_len - 1 - key position), applied after the cap
  const float* log_rates;   // optional [Hq], with slopes: the bias is slopes[h] * ln(1 + log_rates[h] * distance) instead of linear (no cap)
  int window;
  int chunk;                // > 0: only keys of the query's own chunk of this many positions
  DiffCombine diff;         // DIFF instances: query heads 2h, 2h + 1 are combined in the epilogue (see attention_tc.cu)
  int keep_first;           // with a window: keys below this position stay visible (their tiles are walked first)
  int total_items;
  int* sched;             // [0] next item, [1] CTAs finished (the last one re-arms both)
  long long* prof;        // PROF builds: [ctas][32] per-role cycle accounting (tools/attn_decode_bench.py prof)
};

template <int GMAX, int MODE, bool PROF>
__global__ void __launch_bounds__(DA_THREADS, 1)
attn_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                   const DecodeParams p) {
  constexpr bool HAS_CAP = MODE == DA_CAP, DIFF = MODE == DA_DIFF;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = p.G;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sK = smem;                                              // [STAGES][32 KB]
  uint8_t* sV = smem + DA_STAGES * DA_TILE_BYTES;                  // [STAGES][32 KB]
  uint8_t* sQ = smem + 2 * DA_STAGES * DA_TILE_BYTES;              // 2 x 4 KB: the next item's Q lands while the current item computes
  uint8_t* sP = sQ + 2 * DA_Q_BYTES;                               // 2 x 4 KB
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + 2 * DA_P_BYTES);
  uint64_t* q_full = bars;             // [2] Q of the item landed                   (slot = item ordinal & 1, phase = ordinal >> 1)
  uint64_t* q_empty = bars + 30;       // [2] last S of the item has read Q  (bars 27..29 hold the 6 debug words)
  uint64_t* k_full = bars + 2;         // [STAGES]
  uint64_t* k_empty = bars + 5;        // [STAGES]
  uint64_t* v_full = bars + 8;         // [STAGES]
  uint64_t* v_empty = bars + 11;       // [STAGES]
  uint64_t* s_full = bars + 14;        // [2] S^T of a tile is in TMEM
  uint64_t* p_full = bars + 16;        // [2] P^T of a tile is in smem (128 arrivals)
  uint64_t* o_done = bars + 18;        // every PV tile (lazy-rescale hand-off)
  uint64_t* o_final = bars + 19;       // last PV of an item                         (phase = item ordinal)
  uint64_t* o_free = bars + 20;        // epilogue has read O^T (4 arrivals)         (phase = item ordinal)
  uint64_t* item_full = bars + 21;     // [2]
  uint64_t* item_empty = bars + 23;    // [2]  (MMA thread + 4 softmax warps)
  volatile int* s_item = reinterpret_cast<volatile int*>(bars + 25);        // [2]
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 26);
  volatile uint32_t* dbg = reinterpret_cast<volatile uint32_t*>(bars + 27); // [6] role state for the timeout dump
  float* red = reinterpret_cast<float*>(bars + 32);                         // [2][4 warps][GMAX] row-max exchange, then [4][GMAX] sums
#define DA_WAIT(bar_, par_) mbar_wait((bar_), (par_), dbg, 6)

  // PROF builds: the elected thread of each role charges the cycles of a statement to a slot of its local table
  long long pacc[12];
  if constexpr (PROF) {
#pragma unroll
    for (int i = 0; i < 12; ++i) pacc[i] = 0;
  }
#define DA_T(slot, ...)                                                        \
  do {                                                                         \
    if constexpr (PROF) { const long long t0__ = clock64(); __VA_ARGS__; pacc[slot] += clock64() - t0__; } \
    else { __VA_ARGS__; }                                                      \
  } while (0)
#define DA_DBG(code_, a_, b_) dbg[warp] = ((uint32_t)(code_) << 28) | (((uint32_t)(a_) & 0x3fff) << 14) | ((uint32_t)(b_) & 0x3fff)

  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
    mbar_init(&q_full[0], 1); mbar_init(&q_full[1], 1); mbar_init(&q_empty[0], 1); mbar_init(&q_empty[1], 1);
    for (int i = 0; i < DA_STAGES; ++i) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 128); mbar_init(&item_full[i], 1); mbar_init(&item_empty[i], 5); }
    mbar_init(o_done, 1); mbar_init(o_final, 1); mbar_init(o_free, 4);
    fence_barrier_init();
  }
  if (lane == 0) dbg[warp] = 0;
  // zero Q / P (rows >= G stay zero for the whole kernel) and the V ring (a tile's unfetched tail pages must hold finite numbers: their
  // probabilities are exactly 0, and 0 x NaN would poison O)
  for (int i = threadIdx.x; i < (2 * DA_Q_BYTES + 2 * DA_P_BYTES) / 16; i += DA_THREADS) reinterpret_cast<U4*>(sQ)[i] = U4{0, 0, 0, 0};
  for (int i = threadIdx.x; i < DA_STAGES * DA_TILE_BYTES / 16; i += DA_THREADS) reinterpret_cast<U4*>(sV)[i] = U4{0, 0, 0, 0};
  fence_proxy_async_smem();
  if (warp == 1) { tmem_alloc(tmem_ptr, 64); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;
  const uint32_t tmem_S = tmem_base;                 // S^T buffers: cols [0,16) and [16,32)
  const uint32_t tmem_O = tmem_base + 32;            // O^T: cols [32,48)

  // geometry of a work item: pure function of its id, evaluated identically by every role
  // key tiles are walked by a running index L: tiles of kept first tokens wholly before the window's first tile (tile L), then the window's (L + tile_skip)
  struct Item {
    int b, kvh, split, seq_len, kv_hi, tile_begin, n_tiles, keep_tiles, tile_skip;
    __device__ __forceinline__ int tile(int j) const { const int L = tile_begin + j; return L < keep_tiles ? L : L + tile_skip; }
  };
  auto decode_item = [&](int idx) {
    Item it;
    const int per_b = p.Hkv * p.num_splits;
    it.b = idx / per_b;
    const int y = idx - it.b * per_b;
    it.kvh = y / p.num_splits; it.split = y - it.kvh * p.num_splits;
    it.seq_len = p.seq_lens[it.b];
    it.kv_hi = it.seq_len;
    int kv_lo = 0;
    if (p.window > 0) kv_lo = max(0, it.seq_len - p.window);
    if (p.chunk > 0) kv_lo = (it.seq_len - 1) / p.chunk * p.chunk;
    const int tile_lo = kv_lo / DA_KT;
    it.keep_tiles = min((p.keep_first + DA_KT - 1) / DA_KT, tile_lo);
    it.tile_skip = tile_lo - it.keep_tiles;
    const int tile_hi = (it.kv_hi + DA_KT - 1) / DA_KT - it.tile_skip;
    const int per_split = (tile_hi + p.num_splits - 1) / p.num_splits;
    it.tile_begin = it.split * per_split;
    it.n_tiles = max(0, min(tile_hi, it.tile_begin + per_split) - it.tile_begin);
    return it;
  };

  if (warp == 0 && lane == 0) {
    // ------------------------------------------------------------ scheduler + TMA producer
    uint32_t n_it = 0, n_q = 0, g = 0;
    const int ps = p.page_size, pages_per_tile = DA_KT / ps;
    int next_idx = atomicAdd(p.sched, 1);
    for (;;) {
      const int slot = n_it & 1;
      DA_T(0, DA_WAIT(&item_empty[slot], ((n_it >> 1) & 1) ^ 1));
      // the queue atomic is a ~1 us L2 round trip: fetch the NEXT item's index now and consume it one iteration later, so the round trip
      // overlaps this item's TMA issue instead of stalling the only thread that feeds the ring
      const int idx = next_idx;
      if (idx < p.total_items) next_idx = atomicAdd(p.sched, 1);
      DA_DBG(1, n_it, g);
      s_item[slot] = idx;
      mbar_arrive(&item_full[slot]);
      ++n_it;
      if (idx >= p.total_items) break;
      const Item it = decode_item(idx);
      if (it.n_tiles == 0) continue;
      {
        const int qs = n_q & 1;
        uint8_t* qdst = sQ + qs * DA_Q_BYTES;
        DA_T(1, DA_WAIT(&q_empty[qs], ((n_q >> 1) & 1) ^ 1));
        mbar_expect_tx(&q_full[qs], 2 * G * 128);
        tma_load_4d(qdst, &tmQ, &q_full[qs], 0, 0, it.kvh, it.b);
        tma_load_4d(qdst + DA_NQ * 128, &tmQ, &q_full[qs], 64, 0, it.kvh, it.b);
        ++n_q;
      }
      const int* pt = p.page_table + (size_t)p.req_slots[it.b] * p.pt_stride;
      for (int j = 0; j < it.n_tiles; ++j, ++g) {
        const int st = g % DA_STAGES;
        const uint32_t ph = (g / DA_STAGES) & 1;
        const int key0 = it.tile(j) * DA_KT;
        const int n_pages = min(pages_per_tile, (it.kv_hi - key0 + ps - 1) / ps);     // only pages that hold live keys
        const int pg0 = key0 / ps;
        const uint32_t bytes = (uint32_t)n_pages * ps * 256;
        DA_T(2, DA_WAIT(&k_empty[st], ph ^ 1));
        if constexpr (PROF) pacc[4] += 1;
        mbar_expect_tx(&k_full[st], bytes);
        for (int i = 0; i < n_pages; ++i) {
          const int page = pt[pg0 + i];
          uint8_t* dst = sK + st * DA_TILE_BYTES + i * ps * 128;
          tma_load_3d(dst, &tmK, &k_full[st], 0, it.kvh, page * ps);
          tma_load_3d(dst + DA_HALF_BYTES, &tmK, &k_full[st], 64, it.kvh, page * ps);
        }
        DA_T(3, DA_WAIT(&v_empty[st], ph ^ 1));
        mbar_expect_tx(&v_full[st], bytes);
        for (int i = 0; i < n_pages; ++i) {
          const int page = pt[pg0 + i];
          uint8_t* dst = sV + st * DA_TILE_BYTES + i * ps * 128;
          tma_load_3d(dst, &tmV, &v_full[st], 0, it.kvh, page * ps);
          tma_load_3d(dst + DA_HALF_BYTES, &tmV, &v_full[st], 64, it.kvh, page * ps);
        }
      }
    }
  } else if (warp == 1 && lane == 0) {
    // ------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_s = make_idesc(UMMA_BF16, UMMA_BF16, DA_KT, DA_NQ, 0, 0);      // A = K (K-major), B = Q (K-major)
    constexpr uint32_t idesc_o = make_idesc(UMMA_BF16, UMMA_BF16, DA_D, DA_NQ, 1, 0);       // A = V^T (MN-major: d contiguous), B = P^T
    uint32_t n_it = 0, n_q = 0, g = 0;
    for (;;) {
      const int slot = n_it & 1;
      DA_T(0, DA_WAIT(&item_full[slot], (n_it >> 1) & 1));
      const int idx = s_item[slot];
      mbar_arrive(&item_empty[slot]);
      ++n_it;
      if (idx >= p.total_items) break;
      const Item it = decode_item(idx);
      if (it.n_tiles == 0) continue;
      const int n_tiles = it.n_tiles;
      const int qs = n_q & 1;
      const uint32_t q_addr = smem_u32(sQ + qs * DA_Q_BYTES);
      DA_DBG(2, n_q, g);
      auto issue_S = [&](uint32_t gt, bool last) {
        const int st = gt % DA_STAGES;
        DA_T(1, DA_WAIT(&k_full[st], (gt / DA_STAGES) & 1));
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sK + st * DA_TILE_BYTES);
#pragma unroll
        for (int k = 0; k < DA_D / 16; ++k) {
          const uint32_t koff = (k >> 2) * DA_HALF_BYTES + (k & 3) * 32;
          const uint32_t qoff = (k >> 2) * (DA_NQ * 128) + (k & 3) * 32;
          umma_f16_ss(tmem_S + (gt & 1) * DA_NQ, make_smem_desc_sw128(k_addr + koff, 0, 1024), make_smem_desc_sw128(q_addr + qoff, 0, 1024),
                      idesc_s, k != 0);
        }
        umma_commit(&k_empty[st]);
        umma_commit(&s_full[gt & 1]);
        if (last) umma_commit(&q_empty[qs]);
      };
      DA_T(5, DA_WAIT(&q_full[qs], (n_q >> 1) & 1));
      issue_S(g, n_tiles == 1);
      for (int j = 0; j < n_tiles; ++j) {
        const uint32_t gt = g + j;
        const int st = gt % DA_STAGES;
        if (j + 1 < n_tiles) issue_S(gt + 1, j + 2 == n_tiles);
        DA_T(2, DA_WAIT(&p_full[gt & 1], (gt >> 1) & 1));
        DA_T(3, DA_WAIT(&v_full[st], (gt / DA_STAGES) & 1));
        if (j == 0) DA_T(4, DA_WAIT(o_free, (n_q & 1) ^ 1));       // the previous item's epilogue has read O^T
        tc_fence_after();
        const uint32_t v_addr = smem_u32(sV + st * DA_TILE_BYTES);
        const uint32_t p_addr = smem_u32(sP + (gt & 1) * DA_P_BYTES);
#pragma unroll
        for (int k = 0; k < DA_KT / 16; ++k)      // 16 keys per step: A rows advance 16 x 128 B, B (P^T, K-major) advances 32 B inside a 64-key chunk
          umma_f16_ss(tmem_O, make_smem_desc_sw128(v_addr + k * 2048, DA_HALF_BYTES, 1024),
                      make_smem_desc_sw128(p_addr + (k >> 2) * (DA_NQ * 128) + (k & 3) * 32, 0, 1024), idesc_o, (j | k) != 0);
        umma_commit(&v_empty[st]);
        umma_commit(o_done);
        if (j + 1 == n_tiles) umma_commit(o_final);
      }
      g += n_tiles;
      ++n_q;
    }
  } else if (warp >= 2) {
    // ------------------------------------------------------------ softmax (thread = key) + epilogue (thread = output dim)
    const int q4 = warp & 3;                              // TMEM lane quadrant of this warp
    const int row = (q4 << 5) + lane;                     // key index inside the tile / output dim in the epilogue
    const uint32_t lane_addr = (uint32_t)(q4 << 5) << 16;
    const float scale_log2 = p.scale_log2;
    const float cap = p.logit_cap, inv_cap = (HAS_CAP && p.logit_cap > 0.f) ? 1.f / p.logit_cap : 0.f;
    const float scale_nat = scale_log2 * 0.6931471805599453f, inv_scale_nat = 1.f / scale_nat;
    uint32_t n_it = 0, n_q = 0, g = 0;
    for (;;) {
      const int slot = n_it & 1;
      DA_T(0, DA_WAIT(&item_full[slot], (n_it >> 1) & 1));
      const int idx = s_item[slot];
      __syncwarp();
      if (lane == 0) mbar_arrive(&item_empty[slot]);
      ++n_it;
      if (idx >= p.total_items) break;
      const Item it = decode_item(idx);
      if (it.n_tiles == 0) {
        if (p.num_splits > 1) {          // empty split: neutral partial (the merge kernel ignores lse = -inf)
          for (int gq = 0; gq < G; ++gq) {
            const size_t r = ((size_t)it.split * p.B + it.b) * p.Hq + it.kvh * G + gq;
            p.part_o[r * DA_D + row] = 0.f;
            if (row == 0) p.part_lse[r] = -INFINITY;
          }
        }
        continue;
      }
      const int n_tiles = it.n_tiles;
      if (lane == 0) DA_DBG(3, n_q, g);
      const int kv_first = p.chunk > 0 ? (it.seq_len - 1) / p.chunk * p.chunk : p.window > 0 ? it.seq_len - p.window : 0;
      float slope[GMAX];
#pragma unroll
      for (int i = 0; i < GMAX; ++i) slope[i] = (HAS_CAP && p.slopes && i < G) ? p.slopes[it.kvh * G + i] : 0.f;
      float rate[GMAX];
#pragma unroll
      for (int i = 0; i < GMAX; ++i) rate[i] = (HAS_CAP && p.log_rates && i < G) ? p.log_rates[it.kvh * G + i] : 0.f;
      const bool log_bias = HAS_CAP && p.log_rates != nullptr;
      float m_run[GMAX], l_part[GMAX];
#pragma unroll
      for (int i = 0; i < GMAX; ++i) { m_run[i] = -INFINITY; l_part[i] = 0.f; }
      for (int j = 0; j < n_tiles; ++j) {
        const uint32_t gt = g + j;
        DA_T(1, DA_WAIT(&s_full[gt & 1], (gt >> 1) & 1));
        if constexpr (PROF) pacc[8] += 1;
        long long tp__ = 0;
        if constexpr (PROF) tp__ = clock64();
        tc_fence_after();
        uint32_t sr[GMAX];
        {
          const uint32_t a = tmem_S + lane_addr + (gt & 1) * DA_NQ;
          if constexpr (GMAX == 4) {
            asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(sr[0]), "=r"(sr[1]), "=r"(sr[2]), "=r"(sr[3]) : "r"(a) : "memory");
          } else if constexpr (GMAX == 8) {
            asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                         : "=r"(sr[0]), "=r"(sr[1]), "=r"(sr[2]), "=r"(sr[3]), "=r"(sr[4]), "=r"(sr[5]), "=r"(sr[6]), "=r"(sr[7]) : "r"(a) : "memory");
          } else {
            asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                         : "=r"(sr[0]), "=r"(sr[1]), "=r"(sr[2]), "=r"(sr[3]), "=r"(sr[4]), "=r"(sr[5]), "=r"(sr[6]), "=r"(sr[7]), "=r"(sr[8]),
                           "=r"(sr[9]), "=r"(sr[10]), "=r"(sr[11]), "=r"(sr[12]), "=r"(sr[13]), "=r"(sr[14]), "=r"(sr[15]) : "r"(a) : "memory");
          }
          tmem_ld_wait();
        }
        if constexpr (PROF) { const long long t__ = clock64(); pacc[2] += t__ - tp__; tp__ = t__; }
        const int key = it.tile(j) * DA_KT + row;
        const bool live = key < it.kv_hi && (key >= kv_first || key < p.keep_first);
        const float dist = fmaxf((float)(it.seq_len - 1 - key), 0.f);
        float sv[GMAX], wmax[GMAX];
#pragma unroll
        for (int i = 0; i < GMAX; ++i) {
          float x = __uint_as_float(sr[i]);
          if (HAS_CAP) {
            float y = x * scale_nat;
            if (cap > 0.f) y = cap * tanhf(y * inv_cap);
            const float bias = log_bias ? slope[i] * 0.6931471805599453f * __log2f(fmaf(rate[i], dist, 1.f)) : slope[i] * (float)(it.seq_len - 1 - key);
            x = (y - bias) * inv_scale_nat;
          }
          sv[i] = live ? x * scale_log2 : -INFINITY;
          wmax[i] = warp_max(sv[i]);
        }
        float* rbuf = red + (gt & 1) * (4 * GMAX);
        if (lane == 0) {
#pragma unroll
          for (int i = 0; i < GMAX; ++i) rbuf[q4 * GMAX + i] = wmax[i];
        }
        asm volatile("bar.sync 1, 128;" ::: "memory");
        if constexpr (PROF) { const long long t__ = clock64(); pacc[3] += t__ - tp__; tp__ = t__; }
        bool need = false;
        float m_new[GMAX];
#pragma unroll
        for (int i = 0; i < GMAX; ++i) {
          const float tmax = fmaxf(fmaxf(rbuf[i], rbuf[GMAX + i]), fmaxf(rbuf[2 * GMAX + i], rbuf[3 * GMAX + i]));
          m_new[i] = fmaxf(m_run[i], tmax);
          need |= (m_new[i] > m_run[i] + DA_RESCALE_THRESHOLD);     // same value in every thread (m_run and tmax are CTA-uniform)
        }
        if (j == 0) {
#pragma unroll
          for (int i = 0; i < GMAX; ++i) m_run[i] = m_new[i];
        } else if (need) {
          // lazy rescale of O^T (lane = output dim, column = query row): wait for PV(j-1), scale the columns, write back
          DA_WAIT(o_done, (gt - 1) & 1);
          tc_fence_after();
          uint32_t orow[16];
          asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                       : "=r"(orow[0]), "=r"(orow[1]), "=r"(orow[2]), "=r"(orow[3]), "=r"(orow[4]), "=r"(orow[5]), "=r"(orow[6]), "=r"(orow[7]),
                         "=r"(orow[8]), "=r"(orow[9]), "=r"(orow[10]), "=r"(orow[11]), "=r"(orow[12]), "=r"(orow[13]), "=r"(orow[14]), "=r"(orow[15])
                       : "r"(tmem_O + lane_addr) : "memory");
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < GMAX; ++i) {
            const float f = (m_new[i] == -INFINITY) ? 1.f : exp2f(m_run[i] - m_new[i]);
            orow[i] = __float_as_uint(__uint_as_float(orow[i]) * f);
            l_part[i] *= f;
            m_run[i] = m_new[i];
          }
          tmem_st_32x32b_x16(tmem_O + lane_addr, orow);
          tmem_st_wait();
        }
        if constexpr (PROF) { const long long t__ = clock64(); pacc[4] += t__ - tp__; tp__ = t__; }
        // P^T[query row i][key] (bf16, K-major, 128-byte swizzle): rows >= G stay zero
        uint8_t* pbuf = sP + (gt & 1) * DA_P_BYTES + (row >> 6) * (DA_NQ * 128);
        const int c = row & 63;
#pragma unroll
        for (int i = 0; i < GMAX; ++i) {
          if (i < G) {
            const float mm = (m_run[i] == -INFINITY) ? 0.f : m_run[i];
            const float pv = ex2_approx(sv[i] - mm);
            l_part[i] += pv;
            const uint32_t off = i * 128 + ((((uint32_t)c >> 3) ^ (i & 7)) << 4) + (c & 7) * 2;
            *reinterpret_cast<__nv_bfloat16*>(pbuf + off) = __float2bfloat16(pv);
          }
        }
        fence_proxy_async_smem();               // generic-proxy stores -> visible to the tensor core's smem reads
        tc_fence_before();
        if constexpr (PROF) { const long long t__ = clock64(); pacc[5] += t__ - tp__; tp__ = t__; }
        mbar_arrive(&p_full[gt & 1]);
        if constexpr (PROF) pacc[6] += clock64() - tp__;
      }
      g += n_tiles;

      // ---- epilogue: row sums across the 128 key-threads, then O^T / l -> out (thread = output dim)
      long long te__ = 0;
      if constexpr (PROF) te__ = clock64();
      if (lane == 0) DA_DBG(4, n_q, g);
      float lsum[GMAX];
#pragma unroll
      for (int i = 0; i < GMAX; ++i) lsum[i] = warp_sum(l_part[i]);
      float* sbuf = red + 2 * (4 * GMAX);
      if (lane == 0) {
#pragma unroll
        for (int i = 0; i < GMAX; ++i) sbuf[q4 * GMAX + i] = lsum[i];
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      DA_WAIT(o_final, n_q & 1);
      ++n_q;
      tc_fence_after();
      uint32_t orow[16];
      asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                   : "=r"(orow[0]), "=r"(orow[1]), "=r"(orow[2]), "=r"(orow[3]), "=r"(orow[4]), "=r"(orow[5]), "=r"(orow[6]), "=r"(orow[7]),
                     "=r"(orow[8]), "=r"(orow[9]), "=r"(orow[10]), "=r"(orow[11]), "=r"(orow[12]), "=r"(orow[13]), "=r"(orow[14]), "=r"(orow[15])
                   : "r"(tmem_O + lane_addr) : "memory");
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(o_free);        // O^T sits in registers: the next item may overwrite the accumulator
      if (DIFF && p.num_splits == 1) {
        // pairs of columns: combine, mean square over the output dims (= the 128 threads; red's row-max buffers are idle here), scale, store
        constexpr int NP = GMAX / 2;
        float ov[NP];
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const float l0 = sbuf[2 * i] + sbuf[GMAX + 2 * i] + sbuf[2 * GMAX + 2 * i] + sbuf[3 * GMAX + 2 * i];
          const float l1 = sbuf[2 * i + 1] + sbuf[GMAX + 2 * i + 1] + sbuf[2 * GMAX + 2 * i + 1] + sbuf[3 * GMAX + 2 * i + 1];
          const float a = l0 > 0.f ? __uint_as_float(orow[2 * i]) / l0 : 0.f, c = l1 > 0.f ? __uint_as_float(orow[2 * i + 1]) / l1 : 0.f;
          ov[i] = a - p.diff.lam * c;
          const float ss = warp_sum(ov[i] * ov[i]);
          if (lane == 0) red[q4 * NP + i] = ss;
        }
        asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const float ss = red[i] + red[NP + i] + red[2 * NP + i] + red[3 * NP + i];
          if (2 * i < G && row < p.diff.dv)
            p.out[((size_t)it.b * (p.Hq >> 1) + ((it.kvh * G) >> 1) + i) * p.diff.dv + row] =
                __float2bfloat16(ov[i] * (p.diff.post / sqrtf(ss / (float)p.diff.dv + p.diff.eps)));
        }
      }
#pragma unroll
      for (int i = 0; i < GMAX; ++i) {
        if (i < G && !(DIFF && p.num_splits == 1)) {
          const float l = sbuf[i] + sbuf[GMAX + i] + sbuf[2 * GMAX + i] + sbuf[3 * GMAX + i];
          const float inv_l = l > 0.f ? 1.f / l : 0.f;
          const float o = __uint_as_float(orow[i]) * inv_l;
          const int head = it.kvh * G + i;
          if (p.num_splits == 1) {
            p.out[((size_t)it.b * p.Hq + head) * DA_D + row] = __float2bfloat16(o);
            if (p.lse && row == 0) p.lse[(size_t)it.b * p.Hq + head] = l > 0.f ? (m_run[i] + log2f(l)) * 0.6931471805599453f : -INFINITY;
          } else {
            const size_t r = ((size_t)it.split * p.B + it.b) * p.Hq + head;
            p.part_o[r * DA_D + row] = o;
            if (row == 0) p.part_lse[r] = l > 0.f ? (m_run[i] + log2f(l)) * 0.6931471805599453f : -INFINITY;
          }
        }
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");      // sbuf is reused by the next item's epilogue
      if constexpr (PROF) pacc[7] += clock64() - te__;
    }
  }
#undef DA_WAIT
#undef DA_DBG
#undef DA_T
  if constexpr (PROF) {
    if (p.prof != nullptr && lane == 0 && warp <= 2) {
#pragma unroll
      for (int i = 0; i < 10; ++i) p.prof[((size_t)blockIdx.x * 4 + warp) * 10 + i] = pacc[i];      // 4 slots per CTA (the tool's layout)
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 64);
  if (threadIdx.x == 0) {
    __threadfence();
    const int done = atomicAdd(p.sched + 1, 1);
    if (done == (int)gridDim.x - 1) { p.sched[0] = 0; p.sched[1] = 0; __threadfence(); }
  }
}

// defined in attention_tc.cu
void attn_merge_splits(const float* part_o, const float* part_lse, void* out, float* lse, int rows, int num_splits, const DiffCombine* diff, cudaStream_t stream);

bool attn_decode_tc_supported(int Hq, int Hkv, int D, int page_size) {
  if (D != DA_D || Hkv <= 0 || Hq % Hkv) return false;
  const int G = Hq / Hkv;
  return G >= 1 && G <= 16 && page_size >= 8 && page_size <= 128 && (page_size & (page_size - 1)) == 0;
}

static long long* g_da_prof = nullptr;
void attn_decode_set_prof(long long* buf) { g_da_prof = buf; }

void attn_decode_tc(const void* q, const void* k_cache, const void* v_cache, void* out, float* lse, float* part_o, float* part_lse,
                    const int* page_table, int pt_stride, const int* req_slots, const int* seq_lens, int B, int q_stride, int Hq, int Hkv,
                    int D, int num_slots, int page_size, int num_splits, float scale, int window, float logit_cap, int* sched, int num_sms,
                    cudaStream_t stream, const float* slopes, const float* log_rates, int keep_first, int kv_stride, int chunk,
                    const DiffCombine* diff) {
  if (!attn_decode_tc_supported(Hq, Hkv, D, page_size)) throw std::runtime_error("sglb attn_decode_tc: unsupported shape");
  if (sched == nullptr) throw std::runtime_error("sglb attn_decode_tc: needs the work-queue counters");
  const int G = Hq / Hkv;
  // Q viewed as [T][Hkv][G][D]; one box = the G query rows of one (token, kv head), one 64-wide d half
  uint64_t dq[4] = {(uint64_t)D, (uint64_t)G, (uint64_t)Hkv, (uint64_t)B};
  uint64_t sq[3] = {(uint64_t)D * 2, (uint64_t)G * D * 2, (uint64_t)q_stride * 2};
  uint32_t bq[4] = {64, (uint32_t)G, 1, 1};
  CUtensorMap tmQ = make_tmap(q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, dq, sq, bq, CU_TENSOR_MAP_SWIZZLE_128B);
  uint64_t dk[3] = {(uint64_t)D, (uint64_t)Hkv, (uint64_t)num_slots};
  if (kv_stride <= 0) kv_stride = Hkv * D;      // elements between two slots' rows
  if (kv_stride < Hkv * D || (kv_stride % 8) != 0) throw std::runtime_error("sglb attn_decode_tc: cache rows must be 16-byte multiples at least Hkv * D wide");
  uint64_t sk[2] = {(uint64_t)D * 2, (uint64_t)kv_stride * 2};
  uint32_t bk[3] = {64, 1, (uint32_t)page_size};
  CUtensorMap tmK = make_tmap(k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dk, sk, bk, CU_TENSOR_MAP_SWIZZLE_128B);
  CUtensorMap tmV = make_tmap(v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dk, sk, bk, CU_TENSOR_MAP_SWIZZLE_128B);
  DecodeParams p;
  p.out = (__nv_bfloat16*)out; p.part_o = part_o; p.part_lse = part_lse; p.lse = lse;
  p.page_table = page_table; p.req_slots = req_slots; p.seq_lens = seq_lens;
  p.pt_stride = pt_stride; p.Hq = Hq; p.Hkv = Hkv; p.G = G; p.page_size = page_size; p.num_splits = num_splits; p.B = B;
  p.scale_log2 = scale * 1.4426950408889634f; p.logit_cap = logit_cap; p.window = window; p.slopes = slopes;
  p.log_rates = slopes ? log_rates : nullptr; p.keep_first = window > 0 ? std::max(keep_first, 0) : 0;
  if (p.log_rates && logit_cap > 0.f) throw std::runtime_error("sglb attn_decode_tc: the logarithmic distance bias takes no soft cap");
  p.chunk = chunk > 0 ? chunk : 0;
  if (p.chunk && window > 0) throw std::runtime_error("sglb attn_decode_tc: chunked attention has no window");
  p.diff = diff ? *diff : DiffCombine{};
  if (diff && (G % 2 || lse || logit_cap > 0.f || slopes || diff->dv < 1 || diff->dv > DA_D))
    throw std::runtime_error("sglb attn_decode_tc: the differential form pairs query heads of a group, without cap, bias or lse; at most 128 value columns");
  p.total_items = B * Hkv * num_splits; p.sched = sched; p.prof = g_da_prof;
  const int ctas = std::min(p.total_items, num_sms);
  const bool capped = logit_cap > 0.f || slopes != nullptr;
#define SGLB_DA_LAUNCH(GM_, CAP_)                                                                                                    \
  do {                                                                                                                              \
    static bool configured = false;                                                                                                 \
    if (!configured) {                                                                                                              \
      SGLB_CUDA_CHECK(cudaFuncSetAttribute(attn_decode_kernel<GM_, CAP_, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, DA_SMEM_BYTES)); \
      configured = true;                                                                                                            \
    }                                                                                                                               \
    attn_decode_kernel<GM_, CAP_, false><<<ctas, DA_THREADS, DA_SMEM_BYTES, stream>>>(tmQ, tmK, tmV, p);                            \
  } while (0)
  if (g_da_prof != nullptr && G <= 4 && !capped && !diff) {      // instrumented build (per-role cycle accounting), bench tool only
    static bool configured = false;
    if (!configured) {
      SGLB_CUDA_CHECK(cudaFuncSetAttribute(attn_decode_kernel<4, DA_PLAIN, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, DA_SMEM_BYTES));
      configured = true;
    }
    attn_decode_kernel<4, DA_PLAIN, true><<<ctas, DA_THREADS, DA_SMEM_BYTES, stream>>>(tmQ, tmK, tmV, p);
  } else
  if (G <= 4) { if (diff) SGLB_DA_LAUNCH(4, DA_DIFF); else if (capped) SGLB_DA_LAUNCH(4, DA_CAP); else SGLB_DA_LAUNCH(4, DA_PLAIN); }
  else if (G <= 8) { if (diff) SGLB_DA_LAUNCH(8, DA_DIFF); else if (capped) SGLB_DA_LAUNCH(8, DA_CAP); else SGLB_DA_LAUNCH(8, DA_PLAIN); }
  else { if (diff) SGLB_DA_LAUNCH(16, DA_DIFF); else if (capped) SGLB_DA_LAUNCH(16, DA_CAP); else SGLB_DA_LAUNCH(16, DA_PLAIN); }
#undef SGLB_DA_LAUNCH
  SGLB_CUDA_CHECK(cudaGetLastError());
  if (num_splits > 1) attn_merge_splits(part_o, part_lse, out, lse, B * Hq, num_splits, diff, stream);
}

}  // namespace sglb
