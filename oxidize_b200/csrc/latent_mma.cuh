// Latent attention in absorbed form on the tensor cores: all heads of a query attend over the same cached rows.
//
// The work is turned around so that the cached rows are the wide operand: a tile of 128 rows (keys) is the M dimension of
// S^T[keys, rows] = K Q^T, and the latent values are the M dimension (128 at a time) of O^T[values, rows] = V^T P^T, where K
// and V are ONE tile in shared memory: V^T is the same 128-byte-swizzled tile read as an MN-major operand.  N is a block of
// 32 query rows ((token, head) pairs, token-major), so a decode step of 32 heads is one instruction shape and the kernel is a
// stream of cache rows: every CTA owns (sequence, block of query rows, split of the keys), TMA warps bring the pages in
// (column chunks of 64 values, in pairs of chunks so that a pair is one 128-value block of the second product), one warp
// issues tcgen05.mma, two warpgroups do the softmax on S^T read from tensor memory (16 rows each).  A slot of the ring is
// given back as soon as the second product has read its block, so the copies of the next tile run under this one's end.
//
// Softmax: a thread holds one key of 16 rows.  Running maxima are moved by the first tile and then only when a score exceeds
// one by more than 2^8, which one vote settles; row maxima are found with a transposing butterfly, and O^T is then rescaled
// in tensor memory.  The result is exact either way.  The key splits of a row block are one thread-block cluster: each leaves
// its partial O^T in its own shared memory (the ring is idle by then), and every CTA merges a share of the rows out of its
// peers' memory.
#pragma once
#include "common.cuh"

namespace oxb {

constexpr int LM_KEYS = 128;             // keys per tile
constexpr int LM_NR = 32;                // query rows per CTA
constexpr int LM_CN = 16;                // of them per softmax warpgroup
constexpr int LM_CHUNK = LM_KEYS * 128;  // bytes of one 64-value column chunk of a tile
constexpr int LM_PAIR = 2 * LM_CHUNK;
constexpr int LM_TMA_WARPS = 4;          // each brings every fourth page of a tile
// warps: softmax and output, then TMA, then MMA
constexpr int LM_SOFT_WARPS = 4 * (LM_NR / LM_CN), LM_WARP_MMA = LM_SOFT_WARPS + LM_TMA_WARPS, LM_WARPS = LM_WARP_MMA + 1, LM_THREADS = 32 * LM_WARPS;
constexpr int LM_MAX_SLOTS = 16;
constexpr int LM_DYN_SMEM = 224 * 1024;
constexpr float LM_LAZY = 8.f;               // log2 of the factor by which scores may exceed the running maximum

struct LatentMmaArgs {
  const int* block_tables;  // [B, max_blocks]
  const int* seq_lens;      // [B]
  const int* query_start;   // [B + 1]
  const float* sink;        // [H] or null
  __nv_bfloat16* out;       // [H, T, pad]
  int max_blocks, T, H, pad, width, page, num_blocks, window;
  int n_splits;             // CTAs of a cluster
  int pairs, rest, slots;   // 128-value blocks of the latent part, further 64-value chunks, ring slots (pairs)
  int rest_slots, p_bufs;   // buffers of the further chunks and of P
  float scale_log2;
};

// An MN-major operand (64 contiguous values per 128-byte row, rows = the K dimension) with the 128-byte swizzle: 64-value
// chunks lie the descriptor's leading offset apart, groups of 8 rows its stride offset (1024 bytes).
constexpr uint32_t UMMA_A_MN_MAJOR = 1u << 15, UMMA_B_MN_MAJOR = 1u << 16;  // instruction descriptor bits

__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
      "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
// Reduce v[j] (j < 16) over the 32 lanes; lane L returns the result of j = L % 16.  v is used up.
template <class Op>
__device__ __forceinline__ float butterfly_rows(float* v, int lane, Op op) {
#pragma unroll
  for (int j = 0; j < 16; ++j) v[j] = op(v[j], __shfl_xor_sync(0xffffffffu, v[j], 16));
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) {
#pragma unroll
    for (int j = 0; j < o; ++j) {
      const bool up = (lane & o) != 0;
      const float give = up ? v[j] : v[j + o], keep = up ? v[j + o] : v[j];
      v[j] = op(keep, __shfl_xor_sync(0xffffffffu, give, o));
    }
  }
  return v[0];
}

// Merge of a cluster's key splits with the log-sum-exp weights exp2(m_s - M) / sum: this CTA takes rows rank, rank + n, ...
constexpr int LM_MAX_SPLITS = 16;  // clusters of more than 8 CTAs where the device takes them
__device__ __forceinline__ void merge_splits(const LatentMmaArgs& a, const uint8_t* part, const float2* part_ml,
                                             const long long* row_out, int rank, int tiles, int per) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t part_addr = smem_u32(part), ml_addr = smem_u32(part_ml);
  for (int row = rank + warp * a.n_splits; row < LM_NR; row += LM_WARPS * a.n_splits) {
    const long long o = row_out[row];
    if (o < 0) continue;
    // lane s holds split s
    float ms = -INFINITY, ls = 0.f;
    if (lane < a.n_splits && lane * per < tiles) {
      const uint32_t src = dsmem_map(ml_addr + row * 8, lane);
      ms = dsmem_ld_f32(src);
      ls = dsmem_ld_f32(src + 4);
    }
    const float M = warp_max(ms);
    float w = ms == -INFINITY ? 0.f : exp2f(ms - M);  // 0: that split saw no key of this row
    const float den = warp_sum(w * ls);
    w *= den > 0.f ? 1.f / den : 0.f;
    float wv[LM_MAX_SPLITS];
#pragma unroll
    for (int s = 0; s < LM_MAX_SPLITS; ++s) wv[s] = __shfl_sync(0xffffffffu, w, s);
    for (int d = lane * 4; d < a.pad; d += 128) {
      float4 v[LM_MAX_SPLITS];
#pragma unroll
      for (int s = 0; s < LM_MAX_SPLITS; ++s) {
        v[s] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s < a.n_splits && s * per < tiles) v[s] = dsmem_ld_f32x4(dsmem_map(part_addr + (row * a.pad + d) * 4, s));
      }
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < LM_MAX_SPLITS; ++s) {
        acc.x += wv[s] * v[s].x;
        acc.y += wv[s] * v[s].y;
        acc.z += wv[s] * v[s].z;
        acc.w += wv[s] * v[s].w;
      }
      *reinterpret_cast<uint2*>(a.out + o + d) = make_uint2(pack_bf16x2(acc.x, acc.y), pack_bf16x2(acc.z, acc.w));
    }
  }
}

static __global__ void __launch_bounds__(LM_THREADS, 1)
latent_attention_mma_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ,
                            const LatentMmaArgs a) {
  constexpr int NR = LM_NR;
  extern __shared__ uint8_t lm_raw[];
  // s_full / p_full / pv_done: one per parity of the tile (S^T is double-buffered)
  __shared__ uint64_t full[LM_MAX_SLOTS], empty[LM_MAX_SLOTS], rest_full[2], rest_empty[2], q_full, s_full[2], p_full[2], pv_done[2];
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  __shared__ int2 row_keys[NR];                 // first and last key that a row sees
  __shared__ __align__(8) float2 part_ml[NR];   // maximum and sum of this split
  __shared__ long long row_out[NR];             // offset of a row's output, < 0: no such row
  __shared__ float wmax[LM_SOFT_WARPS][LM_CN];                // per-warp maxima of a tile, then per-warp sums
  __shared__ __align__(16) float mrow[LM_SOFT_WARPS][LM_CN];  // running maxima (a copy per warp)
  __shared__ __align__(16) float frow[LM_SOFT_WARPS][LM_CN];  // factors of a rescale / normalisation

  // (broadcast from lane 0: the role branches and what is computed inside them are then known to be warp-uniform)
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const int b = blockIdx.y;
  const int rb = blockIdx.x / a.n_splits, split = blockIdx.x % a.n_splits;
  const int q0 = a.query_start[b], qlen = a.query_start[b + 1] - q0;
  const int R = qlen * a.H, row_base = rb * NR;
  const int seq_len = a.seq_lens[b];
  if (row_base >= R || seq_len < qlen) {  // no such rows (or a padding sequence of a captured step): nothing is written
    pdl_wait();
    return;
  }
  const int pos0 = seq_len - qlen;
  const int last_row = min(R, row_base + NR) - 1;
  const int hi = pos0 + last_row / a.H;
  const int lo = a.window > 0 ? max(0, pos0 + row_base / a.H - a.window + 1) : 0;
  const int page_lo = lo / a.page, page_hi = hi / a.page;
  const int ppt = LM_KEYS / a.page;  // pages per tile
  const int tiles = (page_hi - page_lo + ppt) / ppt;
  const int per = (tiles + a.n_splits - 1) / a.n_splits;
  const int t_begin = min(tiles, split * per), t_end = min(tiles, t_begin + per);

  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lm_raw) + 1023) & ~uintptr_t(1023));
  const int nch = (a.width + 63) / 64;
  uint8_t* s_rest = smem + a.slots * LM_PAIR;                     // [rest_slots][rest chunks]
  uint8_t* s_q = s_rest + a.rest_slots * a.rest * LM_CHUNK;       // [nch][NR][128 bytes]
  uint8_t* s_p = s_q + nch * NR * 128;                            // [p_bufs][2][NR][128 bytes]: 64 keys per row
  uint32_t tmem_cols = 64;
  while ((int)tmem_cols < NR * (2 + a.pairs)) tmem_cols <<= 1;

  if (threadIdx.x == 0) {
    for (int i = 0; i < a.slots; ++i) {
      mbar_init(&full[i], LM_TMA_WARPS);
      mbar_init(&empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&rest_full[i], LM_TMA_WARPS);
      mbar_init(&rest_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 32 * LM_SOFT_WARPS);
      mbar_init(&pv_done[i], 1);
    }
    mbar_init(&q_full, 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  if (threadIdx.x < NR) {
    const int r0 = row_base + (int)threadIdx.x, r = min(r0, R - 1);  // rows past the end see what the last row sees
    const int p = pos0 + r / a.H;
    row_keys[threadIdx.x] = make_int2(a.window > 0 ? max(0, p - a.window + 1) : 0, p);
    row_out[threadIdx.x] = r0 < R ? ((long long)(r % a.H) * a.T + q0 + r / a.H) * a.pad : -1;
  }
  if (warp == LM_WARP_MMA) {
    tmem_alloc(&tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();  // (only now: a CTA of the next kernel must not take the tensor memory that this one still waits for)
  const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_slot, 0);  // columns: S^T (two buffers of NR), then the blocks of O^T
  pdl_wait();  // queries and this step's cache rows come from the upstream kernels

  if (warp >= LM_SOFT_WARPS && warp < LM_WARP_MMA) {
    // ---------------- TMA: warp-uniform loops, one elected lane issues
    const int w = warp - LM_SOFT_WARPS;
    const bool leader = elect_one();
    if (leader && w == 0) {
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmQ);
      mbar_expect_tx(&q_full, nch * NR * 128);
      for (int c = 0; c < nch; ++c) tma_load_2d(s_q + c * NR * 128, &tmQ, &q_full, c * 64, q0 * a.H + row_base);
    }
    const int* bt = a.block_tables + (size_t)b * a.max_blocks;
    const int mine = (ppt + LM_TMA_WARPS - 1 - w) / LM_TMA_WARPS;  // pages of this warp: w, w + LM_TMA_WARPS, ...
    int slot = 0, use = 0;  // ring position and how often it has been round
    bool ok = true;
    for (int t = t_begin; t < t_end && ok; ++t) {
      const int i = t - t_begin;
      int blk = a.num_blocks;  // pages past the last one: a row outside the pool, which the copy fills with zeros
      if (lane < ppt && page_lo + t * ppt + lane <= page_hi) {
        blk = bt[page_lo + t * ppt + lane];
        if ((unsigned)blk >= (unsigned)a.num_blocks) {
          oxb_report(OXB_BAD_BLOCK_ID, blk);
          blk = 0;
        }
      }
      for (int p = 0; p < a.pairs + (a.rest > 0 ? 1 : 0); ++p) {
        const bool is_rest = p == a.pairs;
        const int rs = a.rest_slots == 2 ? i & 1 : 0, ru = a.rest_slots == 2 ? i >> 1 : i;
        uint64_t* fb = is_rest ? &rest_full[rs] : &full[slot];
        const int round = is_rest ? ru : use;
        if (round > 0)
          ok = mbar_wait_bounded(is_rest ? &rest_empty[rs] : &empty[slot], (round - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        uint8_t* dst = is_rest ? s_rest + rs * a.rest * LM_CHUNK : smem + slot * LM_PAIR;
        const int c0 = 2 * p, nc = (is_rest ? nch : min(nch, c0 + 2)) - c0;
        if (leader) mbar_expect_tx(fb, nc * mine * a.page * 128);
        for (int g = w; g < ppt; g += LM_TMA_WARPS) {
          const int row = __shfl_sync(0xffffffffu, blk, g) * a.page;
          uint8_t* d = dst + g * a.page * 128;
          if (leader) {
            tma_load_2d(d, &tmK, fb, c0 * 64, row);
            for (int c = 1; c < nc; ++c) tma_load_2d(d + c * LM_CHUNK, &tmK, fb, (c0 + c) * 64, row);
          }
        }
        __syncwarp();
        if (!is_rest && ++slot == a.slots) {
          slot = 0;
          ++use;
        }
      }
    }
  } else if (warp == LM_WARP_MMA) {
    // ---------------- MMA
    const bool leader = elect_one();
    constexpr uint32_t idesc_s = umma_idesc_bf16(LM_KEYS, NR);
    constexpr uint32_t idesc_o = umma_idesc_bf16(128, NR) | UMMA_A_MN_MAJOR;
    const uint32_t base = smem_u32(smem), q_addr = smem_u32(s_q), p_addr = smem_u32(s_p), r_addr = smem_u32(s_rest);
    const int ksteps = a.width / 16, n = t_end - t_begin;
    int slot = 0, use = 0;  // of the first product; the second follows in the same order
    // S^T of tile i
    auto first = [&](int i) -> bool {
      for (int p = 0; p < a.pairs + (a.rest > 0 ? 1 : 0); ++p) {
        const bool is_rest = p == a.pairs;
        const int rs = a.rest_slots == 2 ? i & 1 : 0, ru = a.rest_slots == 2 ? i >> 1 : i;
        const bool ok = mbar_wait_bounded(is_rest ? &rest_full[rs] : &full[slot], (is_rest ? ru : use) & 1, &abort_flag,
                                          OXB_TIMEOUT_TMA_FULL, blockIdx.x);
        if (!__all_sync(0xffffffffu, ok)) return false;
        tc_fence_after();
        const uint32_t kd = umma_desc_lo(is_rest ? r_addr + rs * a.rest * LM_CHUNK : base + slot * LM_PAIR);
        const uint32_t qd = umma_desc_lo(q_addr + 2 * p * (NR * 128)), d = tmem + NR * (i & 1);
        const int left = ksteps - 8 * p;
        if (left >= 8 && !is_rest) {
#pragma unroll
          for (int k = 0; k < 8; ++k)  // a 64-value chunk is four k-steps of 32 bytes
            umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc_s>(
                leader, d, kd + (k >> 2) * (LM_CHUNK >> 4) + 2 * (k & 3), qd + (k >> 2) * (NR * 128 >> 4) + 2 * (k & 3), k > 0 || p > 0);
        } else {
          for (int k = 0; k < left; ++k)
            umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc_s>(
                leader, d, kd + (k >> 2) * (LM_CHUNK >> 4) + 2 * (k & 3), qd + (k >> 2) * (NR * 128 >> 4) + 2 * (k & 3), k > 0 || p > 0);
        }
        if (is_rest) umma_commit_if(leader, &rest_empty[rs]);
        if (!is_rest && ++slot == a.slots) {
          slot = 0;
          ++use;
        }
      }
      umma_commit_if(leader, &s_full[i & 1]);
      return true;
    };
    // O^T += V^T P^T of tile i
    int vslot = 0;
    auto second = [&](int i) -> bool {
      const bool ok = mbar_wait_bounded(&p_full[i & 1], (i >> 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      if (!__all_sync(0xffffffffu, ok)) return false;
      tc_fence_after();
      const uint32_t pd = umma_desc_lo(p_addr + (a.p_bufs == 2 ? i & 1 : 0) * (2 * NR * 128));
      for (int p = 0; p < a.pairs; ++p) {
        const uint32_t vd = umma_desc_lo(base + vslot * LM_PAIR, LM_CHUNK);
#pragma unroll
        for (int k = 0; k < LM_KEYS / 16; ++k)  // 16 keys: 2 KB of the value tile, 32 bytes of a P row (64 keys per row)
          umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc_o>(
              leader, tmem + NR * (2 + p), vd + k * (2048 >> 4), pd + (k >> 2) * (NR * 128 >> 4) + 2 * (k & 3), i > 0 || k > 0);
        umma_commit_if(leader, &empty[vslot]);
        if (++vslot == a.slots) vslot = 0;
      }
      umma_commit_if(leader, &pv_done[i & 1]);
      return true;
    };
    bool ok = n > 0 && mbar_wait_bounded(&q_full, 0, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
    ok = __all_sync(0xffffffffu, ok);
    // the next tile's first product goes ahead of this tile's second one where the ring holds two tiles
    const bool ahead = a.slots >= 2 * a.pairs;
    if (ok) ok = first(0);
    for (int i = 0; i < n && ok; ++i) {
      if (ahead && i + 1 < n) ok = first(i + 1);
      if (ok) ok = second(i);
      if (ok && !ahead && i + 1 < n) ok = first(i + 1);
    }
    __syncwarp();
  } else {
    // ---------------- softmax: thread = key of the tile (its tensor-memory lane); warpgroup g has query rows n0 .. n0 + 15
    const int g = warp >> 2, n0 = g * LM_CN, w0 = g * 4;
    const uint32_t lanes = ((uint32_t)((warp & 3) * 32) << 16) + n0;
    const int key_in = threadIdx.x & 127, my = lane & 15;  // my: the row whose maximum this lane keeps
    auto group_sync = [&]() { asm volatile("bar.sync %0, 128;" ::"r"(1 + g) : "memory"); };
    // widest key range that every row of the group sees: tiles inside it need no mask
    const int all_lo = row_keys[n0 + LM_CN - 1].x, all_hi = row_keys[n0].y;
    const float sink = (a.sink != nullptr && split == 0) ? a.sink[(row_base + n0 + my) % a.H] * 1.4426950408889634f : -INFINITY;
    float m = sink;  // running maximum of row n0 + my (log2 units), the same in every warp of the group
    float l[LM_CN];
#pragma unroll
    for (int j = 0; j < LM_CN; ++j) l[j] = 0.f;
    const int n = t_end - t_begin;
    for (int i = 0; i < n; ++i) {
      // (no early exit on a failed wait: every thread passes every barrier, later waits return at once)
      mbar_wait_bounded(&s_full[i & 1], (i >> 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      __syncwarp();
      tc_fence_after();
      float s[LM_CN];
      tmem_ld16(tmem + lanes + NR * (i & 1), reinterpret_cast<uint32_t*>(s));
      tmem_ld_wait();
      const int key0 = (page_lo + (t_begin + i) * ppt) * a.page;
#pragma unroll
      for (int j = 0; j < LM_CN; ++j) s[j] *= a.scale_log2;
      if (!(key0 >= all_lo && key0 + LM_KEYS - 1 <= all_hi)) {
        const int key = key0 + key_in;
#pragma unroll
        for (int j = 0; j < LM_CN; ++j) {
          const int2 rk = row_keys[n0 + j];
          if (key < rk.x || key > rk.y) s[j] = -INFINITY;
        }
      }
      // running maxima of the group's rows; usually no score exceeds them by the lazy margin, which one vote settles
      float mm[LM_CN];
      auto load_max = [&]() {
#pragma unroll
        for (int j = 0; j < LM_CN; j += 4) {
          const float4 v = *reinterpret_cast<const float4*>(&mrow[warp][j]);
          mm[j] = v.x;
          mm[j + 1] = v.y;
          mm[j + 2] = v.z;
          mm[j + 3] = v.w;
        }
      };
      bool over = i == 0 || m == -INFINITY;
      if (i > 0) {
        load_max();
#pragma unroll
        for (int j = 0; j < LM_CN; ++j) over |= s[j] > mm[j] + LM_LAZY;
      }
      int any_over;
      asm volatile(
          "{\n\t.reg .pred p, q;\n\tsetp.ne.s32 p, %1, 0;\n\tbarrier.cta.red.or.pred q, %2, 128, p;\n\tselp.s32 %0, 1, 0, q;\n\t}"
          : "=r"(any_over)
          : "r"((int)over), "r"(1 + g)
          : "memory");
      bool any_move = false;
      if (any_over) {
        float v[LM_CN];
#pragma unroll
        for (int j = 0; j < LM_CN; ++j) v[j] = s[j];
        const float wm = butterfly_rows(v, lane, [](float x, float y) { return fmaxf(x, y); });
        if (lane < LM_CN) wmax[warp][lane] = wm;
        group_sync();
        const float tm = fmaxf(fmaxf(wmax[w0][my], wmax[w0 + 1][my]), fmaxf(wmax[w0 + 2][my], wmax[w0 + 3][my]));
        // the first tile sets the maximum, later ones move it past the margin only
        const bool move = tm > m + (i == 0 ? 0.f : LM_LAZY) || (m == -INFINITY && tm > -INFINITY);
        const float m_new = move ? tm : m;
        if (lane < LM_CN) {
          frow[warp][lane] = move ? exp2f(m - m_new) : 1.f;  // 0 when nothing was accumulated
          mrow[warp][lane] = m_new == -INFINITY ? 0.f : m_new;
        }
        m = m_new;
        any_move = __any_sync(0xffffffffu, move) && i > 0;
        __syncwarp();
        load_max();
      }
#pragma unroll
      for (int j = 0; j < LM_CN; ++j) s[j] = exp2f(s[j] - mm[j]);
      // O^T is rescaled once every earlier second product is complete; a P buffer is free once its last reader is
      const int done = (any_move || a.p_bufs == 1) ? i - 1 : i - 2;
      if (done >= 0) mbar_wait_bounded(&pv_done[done & 1], (done >> 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      __syncwarp();
      if (any_move) {
        tc_fence_after();
#pragma unroll
        for (int j = 0; j < LM_CN; ++j) l[j] *= frow[warp][j];
        for (int p = 0; p < a.pairs; ++p) {
          uint32_t r[16];
          const uint32_t addr = tmem + lanes + NR * (2 + p);
          tmem_ld16(addr, r);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * frow[warp][j]);
          tmem_st16(addr, r);
        }
        tmem_st_wait();
      }
      // P^T as the second product's B operand: row = 128 bytes of 64 keys, 16-byte pieces swizzled by the row
      uint8_t* pb = s_p + (a.p_bufs == 2 ? i & 1 : 0) * (2 * NR * 128) + (key_in >> 6) * (NR * 128) + n0 * 128;
      const int piece = (key_in & 63) >> 3, in = (key_in & 7) * 2;
#pragma unroll
      for (int j = 0; j < LM_CN; ++j) {
        l[j] += s[j];
        *reinterpret_cast<__nv_bfloat16*>(pb + j * 128 + ((piece ^ (j & 7)) << 4) + in) = __float2bfloat16(s[j]);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      tc_fence_before();
      mbar_arrive(&p_full[i & 1]);
    }
    // ---------------- sums over the keys, then the output
    const float ws = butterfly_rows(l, lane, [](float x, float y) { return x + y; });
    if (n > 0) mbar_wait_bounded(&pv_done[(n - 1) & 1], ((n - 1) >> 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
    __syncwarp();
    tc_fence_after();
    group_sync();
    if (lane < LM_CN) wmax[warp][lane] = ws;
    group_sync();
    float L = (wmax[w0][my] + wmax[w0 + 1][my]) + (wmax[w0 + 2][my] + wmax[w0 + 3][my]);
    if (sink > -INFINITY) L += exp2f(sink - m);  // the sink's share of the denominator, once
    if (a.n_splits > 1) {
      // O^T of this split into shared memory as [row][pad], next to its maxima and sums
      if (warp == w0 && lane < LM_CN) part_ml[n0 + lane] = make_float2(m, L);
      float* part = reinterpret_cast<float*>(smem);
      asm volatile("bar.sync 3, 256;" ::: "memory");  // both groups are past their last product: the ring is idle
      for (int p = 0; n > 0 && p < a.pairs; ++p) {
        uint32_t r[16];
        tmem_ld16(tmem + lanes + NR * (2 + p), r);
        tmem_ld_wait();
        const int d = p * 128 + key_in;
        if (d < a.pad) {
#pragma unroll
          for (int j = 0; j < 16; ++j) part[(n0 + j) * a.pad + d] = __uint_as_float(r[j]);
        }
      }
    } else {
      if (lane < LM_CN) frow[warp][lane] = L > 0.f ? 1.f / L : 0.f;
      __syncwarp();
      // neighbouring lanes (values d, d + 1) swap one row of each pair of rows, so that a lane stores two values of one row
      const bool odd = lane & 1;
      for (int p = 0; p < a.pairs; ++p) {
        uint32_t r[16];
        tmem_ld16(tmem + lanes + NR * (2 + p), r);
        tmem_ld_wait();
        const int d = p * 128 + (key_in & ~1);
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
          const float lo_v = __uint_as_float(r[j]) * frow[warp][j], hi_v = __uint_as_float(r[j + 1]) * frow[warp][j + 1];
          const float got = __shfl_xor_sync(0xffffffffu, odd ? lo_v : hi_v, 1);
          const float v0 = odd ? got : lo_v, v1 = odd ? hi_v : got;
          const long long o = row_out[n0 + j + (odd ? 1 : 0)];
          if (o >= 0 && d < a.pad) *reinterpret_cast<uint32_t*>(a.out + o + d) = pack_bf16x2(v0, v1);
        }
      }
    }
  }
  if (a.n_splits > 1) {
    __syncwarp();
    cluster_sync_all();
    merge_splits(a, smem, part_ml, row_out, split, tiles, per);
    __syncwarp();
    cluster_sync_all();  // every peer has finished reading this CTA's partial
  }
  if (abort_flag) {
    // a wait gave up: give copies that may still be in flight time to land before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == LM_WARP_MMA) tmem_dealloc(tmem, tmem_cols);
}
struct LatentMmaPlan {
  int ok, pairs, rest, slots, rest_slots, p_bufs, smem;
};

// Shared-memory plan for rows of `width` values of which the first `pad` are the latent part: the ring gets what queries, P
// and the chunks past the latent blocks leave; these are double-buffered where the ring then holds two tiles.
inline LatentMmaPlan latent_mma_plan(int pad, int width, int page) {
  LatentMmaPlan p{0, (pad + 127) / 128, 0, 0, 2, 2, 0};
  const int nch = (width + 63) / 64, pbuf = 2 * LM_NR * 128;
  p.rest = nch > 2 * p.pairs ? nch - 2 * p.pairs : 0;
  const int fixed = nch * LM_NR * 128 + 1024;
  p.slots = (LM_DYN_SMEM - fixed - 2 * p.rest * LM_CHUNK - 2 * pbuf) / LM_PAIR;
  if (p.slots < 2 * p.pairs) {
    p.rest_slots = p.p_bufs = 1;
    p.slots = (LM_DYN_SMEM - fixed - p.rest * LM_CHUNK - pbuf) / LM_PAIR;
  }
  if (p.slots > 4 * p.pairs) p.slots = 4 * p.pairs;
  if (p.slots > LM_MAX_SLOTS) p.slots = LM_MAX_SLOTS;
  p.smem = p.slots * LM_PAIR + p.rest_slots * p.rest * LM_CHUNK + p.p_bufs * pbuf + fixed;
  p.ok = p.slots >= p.pairs && page % 8 == 0 && LM_KEYS % page == 0 && width % 16 == 0 && LM_NR * (2 + p.pairs) <= 512;
  return p;
}

}  // namespace oxb
