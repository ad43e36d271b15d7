// Latent attention in absorbed form on the tensor cores: all heads of a query attend over the same cached rows.
//
// The work is turned around so that the cached rows are the wide operand: a tile of 128 rows (keys) is the M dimension of
// S^T[keys, rows] = K Q^T, and the latent values are the M dimension of O^T[values, rows] = V^T P^T, where K and V are ONE
// tile in shared memory: V^T is the same 128-byte-swizzled tile read as an MN-major operand.  N is a block of NR query rows
// ((token, head) pairs, token-major), so a decode step of 32 heads is one instruction shape and the kernel is a stream of
// cache rows: every CTA owns (sequence, block of query rows, split of the keys), one warp brings the pages in with TMA
// (column chunks of 64 values, in pairs of chunks so that a pair is one 128-value block of the second product), one warp
// issues tcgen05.mma, four warps do the softmax on S^T read from tensor memory.  A slot of the ring is given back as soon
// as the second product has read its block, so the copies of the next tile run while this one is finished.
//
// Softmax: a thread holds one key of every row; row maxima are found with a transposing butterfly (31 shuffles for 32
// rows).  The running maximum is only moved when a tile exceeds it by more than 2^8, so O^T is rarely rescaled; the
// result is exact either way.  Partial (max, sum, O) of key splits are merged by whichever CTA finishes last.
#pragma once
#include "common.cuh"

namespace oxb {

constexpr int LM_KEYS = 128;                 // keys per tile
constexpr int LM_CHUNK = LM_KEYS * 128;      // bytes of one 64-value column chunk of a tile
constexpr int LM_PAIR = 2 * LM_CHUNK;
constexpr int LM_THREADS = 192;              // warps 0-3 softmax and output, 4 TMA, 5 MMA
constexpr int LM_MAX_SLOTS = 8;
constexpr float LM_LAZY = 8.f;               // log2 of the factor by which scores may exceed the running maximum

struct LatentMmaArgs {
  const int* block_tables;  // [B, max_blocks]
  const int* seq_lens;      // [B]
  const int* query_start;   // [B + 1]
  const float* sink;        // [H] or null
  __nv_bfloat16* out;       // [H, T, pad]
  float* ws_o;              // [tasks, NR, pad] (key splits only)
  float* ws_ml;             // [tasks, NR, 2]
  int* counters;            // [B * row blocks] zero-initialised tickets
  int max_blocks, T, H, pad, width, page, num_blocks, window;
  int n_splits, row_blocks;
  int pairs, rest, slots;   // 128-value blocks of the latent part, further 64-value chunks, ring slots (pairs)
  float scale_log2;
};

// MN-major operand (64 contiguous values per 128-byte row, rows = the K dimension) with the 128-byte swizzle: 64-value
// chunks `chunk_bytes` apart (leading offset), groups of 8 rows 1024 bytes apart (stride offset)
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr, uint32_t chunk_bytes) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)((chunk_bytes >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
constexpr uint32_t UMMA_A_MN_MAJOR = 1u << 15;
constexpr uint32_t UMMA_B_MN_MAJOR = 1u << 16;

__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
      "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}

// Reduce v[n] over the 32 lanes for every n < NR; lane L returns the result of n = L % NR.  v is used up.
template <int NR, class Op>
__device__ __forceinline__ float butterfly_rows(float* v, int lane, Op op) {
  if constexpr (NR == 16) {
#pragma unroll
    for (int j = 0; j < 16; ++j) v[j] = op(v[j], __shfl_xor_sync(0xffffffffu, v[j], 16));
  }
#pragma unroll
  for (int o = NR / 2; o > 0; o >>= 1) {
#pragma unroll
    for (int j = 0; j < o; ++j) {
      const bool up = (lane & o) != 0;
      const float give = up ? v[j] : v[j + o], keep = up ? v[j + o] : v[j];
      v[j] = op(keep, __shfl_xor_sync(0xffffffffu, give, o));
    }
  }
  return v[0];
}

template <int NR>
__global__ void __launch_bounds__(LM_THREADS, 1)
latent_attention_mma_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ,
                            const LatentMmaArgs a) {
  static_assert(NR == 16 || NR == 32, "rows per block");
  extern __shared__ uint8_t lm_raw[];
  __shared__ uint64_t full[LM_MAX_SLOTS], empty[LM_MAX_SLOTS], rest_full, rest_empty, q_full, s_full, p_full, pv_done;
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  __shared__ int ticket;
  __shared__ int2 row_keys[NR];        // first and last key that a row sees
  __shared__ float wmax[4][NR];        // per-warp maxima of a tile, then per-warp sums
  __shared__ __align__(16) float mrow[4][NR];  // running maxima (a copy per warp)
  __shared__ __align__(16) float frow[4][NR];  // factors of a rescale / normalisation
  pdl_launch_dependents();

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
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
  uint8_t* s_rest = smem + a.slots * LM_PAIR;
  uint8_t* s_q = s_rest + a.rest * LM_CHUNK;       // [nch][NR][128 bytes]
  uint8_t* s_p = s_q + nch * NR * 128;             // [2][NR][128 bytes]: 64 keys per 128-byte row
  uint32_t tmem_cols = 32;
  while ((int)tmem_cols < NR * (1 + a.pairs)) tmem_cols <<= 1;

  if (threadIdx.x == 0) {
    for (int i = 0; i < a.slots; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(&rest_full, 1);
    mbar_init(&rest_empty, 1);
    mbar_init(&q_full, 1);
    mbar_init(&s_full, 1);
    mbar_init(&p_full, 128);
    mbar_init(&pv_done, 1);
    abort_flag = 0;
    ticket = 0;
    mbar_fence_init();
  }
  if (threadIdx.x < NR) {
    const int r = min(row_base + (int)threadIdx.x, R - 1);  // rows past the end see what the last row sees; never stored
    const int p = pos0 + r / a.H;
    row_keys[threadIdx.x] = make_int2(a.window > 0 ? max(0, p - a.window + 1) : 0, p);
  }
  if (warp == 5) {
    tmem_alloc(&tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  pdl_wait();  // queries and this step's cache rows come from the upstream kernels

  if (warp == 4) {
    // ---------------- TMA: lane p brings page p of the tile
    if (lane == 0) {
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmQ);
      mbar_expect_tx(&q_full, nch * NR * 128);
      for (int c = 0; c < nch; ++c) tma_load_2d(s_q + c * NR * 128, &tmQ, &q_full, c * 64, q0 * a.H + row_base);
    }
    const int* bt = a.block_tables + (size_t)b * a.max_blocks;
    int cnt = 0;  // pairs issued
    bool ok = true;
    for (int t = t_begin; t < t_end && ok; ++t) {
      int blk = 0;
      if (lane < ppt) {
        blk = bt[min(page_lo + t * ppt + lane, page_hi)];  // pages past the last one: any valid page, its keys are masked
        if ((unsigned)blk >= (unsigned)a.num_blocks) {
          oxb_report(OXB_BAD_BLOCK_ID, blk);
          blk = 0;
        }
      }
      const int row = blk * a.page;
      for (int p = 0; p < a.pairs + (a.rest > 0 ? 1 : 0) && ok; ++p) {
        const bool is_rest = p == a.pairs;
        const int slot = cnt % a.slots;
        uint64_t* fb = is_rest ? &rest_full : &full[slot];
        if (is_rest) {
          const int i = t - t_begin;
          if (i > 0) ok = mbar_wait_bounded(&rest_empty, (i - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
        } else {
          if (cnt >= a.slots) ok = mbar_wait_bounded(&empty[slot], (cnt / a.slots - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
          ++cnt;
        }
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        uint8_t* dst = is_rest ? s_rest : smem + slot * LM_PAIR;
        const int c0 = 2 * p, c1 = is_rest ? nch : min(nch, c0 + 2);
        if (lane == 0) mbar_expect_tx(fb, (c1 - c0) * LM_CHUNK);
        __syncwarp();
        if (lane < ppt)
          for (int c = c0; c < c1; ++c) tma_load_2d(dst + (c - c0) * LM_CHUNK + lane * a.page * 128, &tmK, fb, c * 64, row);
        __syncwarp();
      }
    }
  } else if (warp == 5) {
    // ---------------- MMA
    const bool leader = elect_one();
    constexpr uint32_t idesc_s = umma_idesc_bf16(128, NR);
    constexpr uint32_t idesc_o = umma_idesc_bf16(128, NR) | UMMA_A_MN_MAJOR;
    const uint32_t base = smem_u32(smem), q_addr = smem_u32(s_q), p_addr = smem_u32(s_p), r_addr = smem_u32(s_rest);
    const int ksteps = a.width / 16;
    int cnt = 0;
    bool ok = t_begin < t_end && mbar_wait_bounded(&q_full, 0, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
    ok = __all_sync(0xffffffffu, ok);
    for (int t = t_begin; t < t_end && ok; ++t) {
      const int i = t - t_begin;
      for (int p = 0; p < a.pairs + (a.rest > 0 ? 1 : 0); ++p) {
        const bool is_rest = p == a.pairs;
        const int slot = (cnt + p) % a.slots;
        ok = is_rest ? mbar_wait_bounded(&rest_full, i & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x)
                     : mbar_wait_bounded(&full[slot], ((cnt + p) / a.slots) & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        if (leader) {
          const uint32_t src = is_rest ? r_addr : base + slot * LM_PAIR;
          const int k0 = p * 8, k1 = is_rest ? ksteps : min(ksteps, k0 + 8);
          for (int k = k0; k < k1; ++k)
            umma_bf16(tmem, umma_desc_k_sw128(src + ((k - k0) >> 2) * LM_CHUNK) + 2 * (k & 3),
                      umma_desc_k_sw128(q_addr + (k >> 2) * (NR * 128)) + 2 * (k & 3), idesc_s, k > 0 ? 1u : 0u);
          if (is_rest) umma_commit(&rest_empty);
        }
        __syncwarp();
      }
      if (!ok) break;
      if (leader) umma_commit(&s_full);
      ok = __all_sync(0xffffffffu, mbar_wait_bounded(&p_full, i & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x));
      if (!ok) break;
      tc_fence_after();
      for (int p = 0; p < a.pairs; ++p) {
        const int slot = (cnt + p) % a.slots;
        if (leader) {
          const uint64_t vdesc = umma_desc_mn_sw128(base + slot * LM_PAIR, LM_CHUNK);
#pragma unroll
          for (int k = 0; k < LM_KEYS / 16; ++k)
            umma_bf16(tmem + NR * (1 + p), vdesc + (uint64_t)(k * (2048 >> 4)),
                      umma_desc_k_sw128(p_addr + (k >> 2) * (NR * 128)) + 2 * (k & 3), idesc_o, (i > 0 || k > 0) ? 1u : 0u);
          umma_commit(&empty[slot]);
        }
      }
      if (leader) umma_commit(&pv_done);
      __syncwarp();
      cnt += a.pairs;
    }
  } else {
    // ---------------- softmax: thread = key of the tile (its tensor-memory lane)
    const uint32_t lanes = (uint32_t)(warp * 32) << 16;
    const int tid = threadIdx.x;
    // widest key range that every row of the block sees: tiles inside it need no mask
    const int all_lo = row_keys[NR - 1].x, all_hi = row_keys[0].y;
    const int my_h = (row_base + lane % NR) % a.H;
    const float sink = (a.sink != nullptr && split == 0) ? a.sink[my_h] * 1.4426950408889634f : -INFINITY;
    float m = sink;  // running maximum of row lane % NR (log2 units), the same in every warp
    float l[NR];
#pragma unroll
    for (int n = 0; n < NR; ++n) l[n] = 0.f;
    for (int t = t_begin; t < t_end; ++t) {
      const int i = t - t_begin;
      // (no early exit on a failed wait: every thread passes every barrier, later waits return at once)
      mbar_wait_bounded(&s_full, i & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      __syncwarp();
      tc_fence_after();
      float s[NR];
#pragma unroll
      for (int c = 0; c < NR / 16; ++c) tmem_ld16(tmem + lanes + 16 * c, reinterpret_cast<uint32_t*>(s) + 16 * c);
      tmem_ld_wait();
      const int key0 = (page_lo + t * ppt) * a.page, key = key0 + tid;
      const bool inside = key0 >= all_lo && key0 + LM_KEYS - 1 <= all_hi;
#pragma unroll
      for (int n = 0; n < NR; ++n) {
        s[n] *= a.scale_log2;
        if (!inside) {
          const int2 rk = row_keys[n];
          if (key < rk.x || key > rk.y) s[n] = -INFINITY;
        }
      }
      {
        float v[NR];
#pragma unroll
        for (int n = 0; n < NR; ++n) v[n] = s[n];
        const float wm = butterfly_rows<NR>(v, lane, [](float x, float y) { return fmaxf(x, y); });
        if (lane < NR) wmax[warp][lane] = wm;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      const int n_ = lane % NR;
      const float tm = fmaxf(fmaxf(wmax[0][n_], wmax[1][n_]), fmaxf(wmax[2][n_], wmax[3][n_]));
      const bool move = tm > m + LM_LAZY || (m == -INFINITY && tm > -INFINITY);
      const float m_new = move ? tm : m;
      const float f = move ? exp2f(m - m_new) : 1.f;  // 0 when nothing was accumulated
      m = m_new;
      if (lane < NR) mrow[warp][lane] = m == -INFINITY ? 0.f : m;
      const bool any_move = __any_sync(0xffffffffu, move);
      if (any_move && lane < NR) frow[warp][lane] = f;
      __syncwarp();
      if (i > 0) {
        mbar_wait_bounded(&pv_done, (i - 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);  // P is free, O^T is complete
        __syncwarp();
      }
      if (any_move) {
#pragma unroll
        for (int n = 0; n < NR; ++n) l[n] *= frow[warp][n];
        if (i > 0) {
          tc_fence_after();
          for (int p = 0; p < a.pairs; ++p) {
#pragma unroll
            for (int c = 0; c < NR / 16; ++c) {
              uint32_t r[16];
              const uint32_t addr = tmem + lanes + NR * (1 + p) + 16 * c;
              tmem_ld16(addr, r);
              tmem_ld_wait();
#pragma unroll
              for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * frow[warp][16 * c + j]);
              tmem_st16(addr, r);
            }
          }
          tmem_st_wait();
        }
      }
      // P^T as the second product's B operand: row n = 128 bytes of 64 keys, 16-byte pieces swizzled by the row
      uint8_t* pb = s_p + (tid >> 6) * (NR * 128);
      const int piece = (tid & 63) >> 3, in = (tid & 7) * 2;
#pragma unroll
      for (int n = 0; n < NR; ++n) {
        const float p = exp2f(s[n] - mrow[warp][n]);
        l[n] += p;
        *reinterpret_cast<__nv_bfloat16*>(pb + n * 128 + ((piece ^ (n & 7)) << 4) + in) = __float2bfloat16(p);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      tc_fence_before();
      mbar_arrive(&p_full);
    }
    // ---------------- sums over the keys, then the output
    const float ws = butterfly_rows<NR>(l, lane, [](float x, float y) { return x + y; });
    if (t_end > t_begin) mbar_wait_bounded(&pv_done, (t_end - t_begin - 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
    __syncwarp();
    tc_fence_after();
    asm volatile("bar.sync 1, 128;" ::: "memory");
    if (lane < NR) wmax[warp][lane] = ws;
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const int n_ = lane % NR;
    float L = (wmax[0][n_] + wmax[1][n_]) + (wmax[2][n_] + wmax[3][n_]);
    if (sink > -INFINITY) L += exp2f(sink - m);  // the sink's share of the denominator, once
    const int rows = min(NR, R - row_base);
    if (a.n_splits == 1) {
      if (lane < NR) frow[warp][lane] = L > 0.f ? 1.f / L : 0.f;
      __syncwarp();
      for (int p = 0; p < a.pairs; ++p) {
        const int d = p * 128 + tid;
#pragma unroll
        for (int c = 0; c < NR / 16; ++c) {
          uint32_t r[16];
          tmem_ld16(tmem + lanes + NR * (1 + p) + 16 * c, r);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const int n = 16 * c + j;
            if (n < rows && d < a.pad) {
              const int g = row_base + n;
              a.out[((size_t)(g % a.H) * a.T + q0 + g / a.H) * a.pad + d] = __float2bfloat16(__uint_as_float(r[j]) * frow[warp][n]);
            }
          }
        }
      }
    } else {
      const size_t task0 = ((size_t)b * a.row_blocks + rb) * a.n_splits;
      float* po = a.ws_o + (task0 + split) * NR * a.pad;
      if (warp == 0 && lane < NR) {
        a.ws_ml[((task0 + split) * NR + lane) * 2] = m;
        a.ws_ml[((task0 + split) * NR + lane) * 2 + 1] = L;
      }
      if (t_end > t_begin) {
        for (int p = 0; p < a.pairs; ++p) {
          const int d = p * 128 + tid;
#pragma unroll
          for (int c = 0; c < NR / 16; ++c) {
            uint32_t r[16];
            tmem_ld16(tmem + lanes + NR * (1 + p) + 16 * c, r);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j)
              if (16 * c + j < rows && d < a.pad) po[(size_t)(16 * c + j) * a.pad + d] = __uint_as_float(r[j]);
          }
        }
      }
      __threadfence();
      asm volatile("bar.sync 1, 128;" ::: "memory");
      int* cnt = a.counters + (size_t)b * a.row_blocks + rb;
      if (tid == 0) ticket = atomicAdd(cnt, 1);
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (ticket == a.n_splits - 1) {
        __threadfence();
        for (int n = warp; n < rows; n += 4) {  // a warp per row
          float M = -INFINITY;
          for (int s = 0; s < a.n_splits; ++s) M = fmaxf(M, __ldcg(a.ws_ml + ((task0 + s) * NR + n) * 2));
          float den = 0.f;
          for (int s = 0; s < a.n_splits; ++s) {
            const float ms = __ldcg(a.ws_ml + ((task0 + s) * NR + n) * 2);
            if (ms > -INFINITY) den += exp2f(ms - M) * __ldcg(a.ws_ml + ((task0 + s) * NR + n) * 2 + 1);
          }
          const float inv = den > 0.f ? 1.f / den : 0.f;
          const int g = row_base + n;
          __nv_bfloat16* o = a.out + ((size_t)(g % a.H) * a.T + q0 + g / a.H) * a.pad;
          for (int d = lane * 4; d < a.pad; d += 128) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int s = 0; s < a.n_splits; ++s) {
              const float ms = __ldcg(a.ws_ml + ((task0 + s) * NR + n) * 2);
              if (ms == -INFINITY || (s * per >= tiles)) continue;  // that split saw no key of this row (or had no tile)
              const float w = exp2f(ms - M) * inv;
              const float4 v = __ldcg(reinterpret_cast<const float4*>(a.ws_o + ((task0 + s) * NR + n) * (size_t)a.pad + d));
              acc.x += w * v.x;
              acc.y += w * v.y;
              acc.z += w * v.z;
              acc.w += w * v.w;
            }
            *reinterpret_cast<uint2*>(o + d) = make_uint2(pack_bf16x2(acc.x, acc.y), pack_bf16x2(acc.z, acc.w));
          }
        }
        if (tid == 0) *cnt = 0;  // re-armed for the next launch / graph replay
      }
    }
  }
  if (abort_flag) {
    // a wait gave up: give copies that may still be in flight time to land before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) tmem_dealloc(tmem, tmem_cols);
}

struct LatentMmaPlan {
  int ok, pairs, rest, slots, smem;
};

// Shared-memory plan for rows of `width` values of which the first `pad` are the latent part.
inline LatentMmaPlan latent_mma_plan(int nr, int pad, int width, int page) {
  LatentMmaPlan p{0, (pad + 127) / 128, 0, 0, 0};
  const int nch = (width + 63) / 64;
  p.rest = nch > 2 * p.pairs ? nch - 2 * p.pairs : 0;
  const int fixed = p.rest * LM_CHUNK + nch * nr * 128 + 2 * nr * 128 + 1024;
  const int budget = 225 * 1024;  // the static variables of the kernel share the 227 KB
  p.slots = (budget - fixed) / LM_PAIR;
  if (p.slots > 2 * p.pairs) p.slots = 2 * p.pairs;
  if (p.slots > LM_MAX_SLOTS) p.slots = LM_MAX_SLOTS;
  p.smem = p.slots * LM_PAIR + fixed;
  p.ok = p.slots >= p.pairs && page % 8 == 0 && LM_KEYS % page == 0 && width % 16 == 0 && nr * (1 + p.pairs) <= 512;
  return p;
}

}  // namespace oxb
