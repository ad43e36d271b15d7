// Attention on the scores of all heads together (joint.cuh) for long portions, in three kernels.
//
// joint_scores_kernel: scores of four heads for 128 tokens per CTA, products on tcgen05 with the keys as rows: a thread has a key, a
// warp a tile.  What it caps goes out as the operand registers that the mixing wants: a high and a low half each, the four heads of
// a (token, key) in 16 bytes.
// joint_mix_kernel: a warp mixes one token's scores with 32 keys at a time over all heads (hi hi + hi lo + lo hi, float32 sums)
// and leaves exp2(score - m) in bfloat16, its sum and m, the largest score rounded up to a whole power of two.
// joint_values_kernel: weights times values, a head and 128 tokens per CTA, on tcgen05 with the weights as the operand in tensor
// memory.  Between tiles with different m they are multiplied by powers of two, which rounds nothing.
//
// Keys and values are the same rows, which come by TMA out of the cache pages: four tiles of 32 keys per place of the scores' ring,
// two per place of the values'.  Of the 32 keys of a tile a lane of the mixing has 2 t4, 2 t4 + 1 and those 8, 16 and 24 further,
// 16 bytes of weights in all.
#pragma once
#include "joint.cuh"
#include "latent_mma.cuh"
#include "latent_prefill.cuh"
#include "retention.cuh"

namespace oxb {

constexpr int JP_ROWS = 16, JP_KEYS = 32;  // tokens of a block, keys of a tile
constexpr int JP_M = 128;                  // tokens of a CTA
constexpr int JC_PLACE = 128, JC_CHUNK = JC_PLACE * 128, JC_PLACES = 2;  // joint_scores_kernel: keys of a place, bytes of 64 columns
constexpr int JC_WARPS = 16, JC_THREADS = JC_WARPS * 32 + 64;
constexpr int JM_WARPS = 8, JM_TILES = 8;  // joint_mix_kernel: tiles per warp
constexpr int JV_PLACE = 64, JV_CHUNK = JV_PLACE * 128, JV_PLACES = 4, JV_THREADS = 128 + 64;
constexpr float JP_NONE = -1e30f;  // m of a tile without a visible key

struct JointPrefillArgs {
  JointArgs a;
  const int* block_seq;  // [blocks] sequence of every block of 16 tokens
  const int* block_row;  // [blocks] its first row
  const int* wide;       // [wide blocks, 2]: first block of 16, number of them (up to 8, of one sequence)
  uint4* scores;         // [blocks, tiles, quads of heads, 16, 32]
  uint4* weights;        // [blocks, tiles, H, 16, 4]
  float2* stats;         // [blocks, tiles, H, 16]: m, sum
  int tiles;             // most tiles of a block
  int block0;            // the first block of this launch: scratch is numbered from there
  int blocks;
};

// What a block of tokens sees: `kept` tiles of 32 keys from position 0 on, then the tiles from `lo` through `hi`.
struct JointSpan {
  int pos0, rows, kept, lo, hi;
};
__device__ __forceinline__ JointSpan joint_span(const JointArgs& a, int b, int row0) {
  JointSpan s;
  const int left = a.query_start[b + 1] - row0;
  s.rows = min(JP_ROWS, left);
  s.pos0 = a.seq_lens[b] - left;
  s.lo = a.window > 0 ? max(0, s.pos0 - a.window + 1) / JP_KEYS : 0;
  s.hi = (s.pos0 + s.rows - 1) / JP_KEYS;
  s.kept = min((a.keep_first + JP_KEYS - 1) / JP_KEYS, s.lo);
  return s;
}

// The tiles that the blocks first .. last of a sequence see together, in order, and which of them one block sees.
struct JointTiles {
  int kept, lo, n, last_page;
  __device__ __forceinline__ JointTiles(const JointSpan& first, const JointSpan& last)
      : kept(first.kept), lo(first.lo), n(first.kept + last.hi - first.lo + 1), last_page((last.pos0 + last.rows - 1) >> 4) {}
  __device__ __forceinline__ int tile(int i) const { return i < kept ? i : lo + i - kept; }
};
struct JointOwn {
  int head, lo, hi;  // i < head or lo <= i <= hi
  __device__ __forceinline__ JointOwn(const JointTiles& all, const JointSpan& s, bool any)
      : head(s.kept), lo(all.kept + s.lo - all.lo), hi(any ? all.kept + s.hi - all.lo : -1) {}
  __device__ __forceinline__ bool has(int i) const { return i <= hi && (i < head || i >= lo); }
  __device__ __forceinline__ int number(int i) const { return i < head ? i : head + i - lo; }  // among the block's own
};

// The pages of tiles i .. i + n/2, by number; -1 past the end, where a place keeps what is there.
struct JointLoader {
  const JointArgs& a;
  const JointTiles& all;
  const int* bt;
  __device__ __forceinline__ int pages(int i, int most) const {
    int n = 0;
    for (int p = 0; p < most; ++p) n += page(i, p) >= 0;
    return n;
  }
  __device__ __forceinline__ int page(int i, int p) const {
    const int t = i + (p >> 1), n = 2 * all.tile(t) + (p & 1);
    return t < all.n && n <= all.last_page ? n : -1;
  }
  __device__ __forceinline__ int row(int page, int g) const {  // of the cache, in rows of 16 per key head
    int id = bt[page];
    if ((unsigned)id >= (unsigned)a.num_blocks) {
      oxb_report(OXB_BAD_BLOCK_ID, id);
      id = 0;
    }
    return (id * a.G + g) * 16;
  }
};

// ----------------------------------------------------------------------------- scores
__host__ __device__ inline int joint_scores_smem(int W) {  // queries of four heads, keys, factors of the keys (rows of 16 bytes)
  return (4 * JP_M + JC_PLACES * JC_PLACE) * ((W + 63) / 64) * 128 + JC_PLACES * JC_PLACE * 16 + 1024;
}

// grid (wide blocks, quads of heads, parts of the tiles).  Sixteen warps cap, one loads, one multiplies.  Tensor memory: tokens
// 64 s .. 64 s + 63 of head h at 256 s + 64 h.
static __global__ void __launch_bounds__(JC_THREADS, 1)
joint_scores_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmT,
                    const JointPrefillArgs x, const int same) {
  extern __shared__ uint8_t jc_raw[];
  __shared__ uint64_t q_full, k_full[JC_PLACES], k_empty[JC_PLACES], t_empty[JC_PLACES], s_full[2], s_empty[2];
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  const JointArgs& a = x.a;
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const int H = a.H, per = H / a.G, quad = blockIdx.y, quads = gridDim.y, chunks = (a.W + 63) / 64;
  const int blk0 = x.wide[2 * blockIdx.x], n_blk = x.wide[2 * blockIdx.x + 1], b = x.block_seq[blk0], row0 = x.block_row[blk0];
  const JointTiles all(joint_span(a, b, row0), joint_span(a, b, x.block_row[blk0 + n_blk - 1]));
  const int places = (all.n + 3) / 4, share = (places + gridDim.z - 1) / gridDim.z;
  const int u0 = blockIdx.z * share, u1 = min(places, u0 + share);
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(jc_raw) + 1023) & ~uintptr_t(1023));
  if (u0 >= u1) {
    pdl_wait();
    return;
  }
  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    for (int i = 0; i < JC_PLACES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&t_empty[i], JC_WARPS);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], JC_WARPS);
    }
    abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == JC_WARPS + 1) {
    tmem_alloc(&tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();  // (only now: a CTA of the next kernel must not take the tensor memory that this one still waits for)
  const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_slot, 0);
  pdl_wait();

  // item j: place u0 + j / nk, key head j % nk of the quad; it lies in place j % JC_PLACES of the ring
  const int nk = same ? 1 : 4, items = (u1 - u0) * nk, halves = (n_blk + 3) / 4;
  uint8_t *sK = smem + 4 * chunks * JP_M * 128, *sT = sK + JC_PLACES * chunks * JC_CHUNK;
  if (warp == JC_WARPS) {
    const JointLoader ld{a, all, a.block_tables + (size_t)b * a.max_blocks};
    const bool leader = elect_one();
    if (leader) {
      mbar_expect_tx(&q_full, 4 * chunks * JP_M * 128);
      for (int h = 0; h < 4; ++h)
        for (int c = 0; c < chunks; ++c) tma_load_2d(smem + (h * chunks + c) * JP_M * 128, &tmQ, &q_full, (quad * 4 + h) * a.W + c * 64, row0);
    }
    bool ok = true;
    for (int j = 0; j < items && ok; ++j) {
      const int s = j % JC_PLACES, turn = j / JC_PLACES, i = 4 * (u0 + j / nk), g = min(quad * 4 + j % nk, H - 1) / per;
      if (turn > 0)
        ok = mbar_wait_bounded(&k_empty[s], (turn - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x) &&
             mbar_wait_bounded(&t_empty[s], (turn - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (leader) {
        mbar_expect_tx(&k_full[s], ld.pages(i, 8) * (chunks * 2048 + 256));
        for (int p = 0; p < 8; ++p) {
          const int page = ld.page(i, p);
          if (page < 0) continue;
          const int row = ld.row(page, g);
          for (int c = 0; c < chunks; ++c) tma_load_2d(sK + (s * chunks + c) * JC_CHUNK + p * 2048, &tmK, &k_full[s], c * 64, row);
          tma_load_2d(sT + (s * JC_PLACE + p * 16) * 16, &tmT, &k_full[s], a.W / 2, row);  // (coordinates in words)
        }
      }
      __syncwarp();
    }
  } else if (warp == JC_WARPS + 1) {
    const bool leader = elect_one();
    constexpr uint32_t idesc = umma_idesc_bf16(JC_PLACE, 64);
    const uint32_t qa = smem_u32(smem), ka = smem_u32(sK);
    bool ok = __all_sync(0xffffffffu, mbar_wait_bounded(&q_full, 0, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x));
    for (int j = 0; j < items && ok; ++j) {
      const int s = j % JC_PLACES, t = j / nk, heads = same ? 4 : 1, h0 = same ? 0 : j % nk;
      ok = mbar_wait_bounded(&k_full[s], (j / JC_PLACES) & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
      for (int half = 0; half < halves; ++half) {
        if (j % nk == 0 && t > 0) ok = mbar_wait_bounded(&s_empty[half], (t - 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x) && ok;
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        for (int h = h0; h < h0 + heads; ++h)
          for (int c = 0; c < chunks; ++c) {
            const uint32_t qd = umma_desc_lo(qa + (h * chunks + c) * JP_M * 128 + half * 8192), kd = umma_desc_lo(ka + (s * chunks + c) * JC_CHUNK);
            const int left = min(4, a.W / 16 - 4 * c);
            for (int k = 0; k < left; ++k)
              umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc>(leader, tmem + 256 * half + 64 * h, kd + 2 * k, qd + 2 * k, k > 0 || c > 0);
          }
        if (j % nk == nk - 1) umma_commit_if(leader, &s_full[half]);
      }
      if (ok) umma_commit_if(leader, &k_empty[s]);
    }
    __syncwarp();
  } else {
    // ---------------- thread = key, warp = a tile of the place and a block of the half
    const int quarter = warp & 3, group = warp >> 2;
    const uint32_t lanes = (uint32_t)(quarter * 32) << 16;
    const JointCap cap = joint_cap(a);
    for (int u = u0; u < u1; ++u) {
      const int t = u - u0, i = 4 * u + quarter;
      float f[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {  // what the keys' rows are divided by
        if (c < nk) {
          const int j = t * nk + c, s = j % JC_PLACES;
          mbar_wait_bounded(&k_full[s], (j / JC_PLACES) & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
          __syncwarp();
          f[c] = *reinterpret_cast<const float*>(sT + (s * JC_PLACE + quarter * 32 + lane) * 16) * cap.factor;
          __syncwarp();
          if (lane == 0) mbar_arrive(&t_empty[s]);
        } else {
          f[c] = f[0];
        }
      }
      for (int half = 0; half < halves; ++half) {
        mbar_wait_bounded(&s_full[half], t & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
        __syncwarp();
        tc_fence_after();
        const int bi = 4 * half + group;
        if (bi < n_blk) {
          const JointOwn own(all, joint_span(a, b, x.block_row[blk0 + bi]), true);
          if (i < all.n && own.has(i)) {
            float s[4][16];
#pragma unroll
            for (int h = 0; h < 4; ++h) tmem_ld16(tmem + lanes + 256 * half + 64 * h + 16 * group, reinterpret_cast<uint32_t*>(s[h]));
            tmem_ld_wait();
            uint4* to = x.scores + (((size_t)(blk0 + bi - x.block0) * x.tiles + own.number(i)) * quads + quad) * (JP_ROWS * JP_KEYS) + lane;
#pragma unroll
            for (int k = 0; k < 16; ++k) {
              float v[4];
#pragma unroll
              for (int h = 0; h < 4; ++h) v[h] = s[h][k] * f[h];
              if (cap.cap > 0.f) {
#pragma unroll
                for (int h = 0; h < 4; ++h) v[h] = joint_capped_of(v[h], cap);
              }
              uint4 o;
              split_bf16x2(v[0], v[1], o.x, o.z);
              split_bf16x2(v[2], v[3], o.y, o.w);
              to[k * JP_KEYS] = o;
            }
          }
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&s_empty[half]);
      }
    }
  }
  if (abort_flag) {
    // a wait gave up: give copies that may still be in flight time to land before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == JC_WARPS + 1) tmem_dealloc(tmem, 512);
}

// ----------------------------------------------------------------------------- mixing
// grid (blocks x 2, parts of JM_TILES tiles): a warp has a token.  HPW = heads / 16 rounded up.
template <int HPW>
__global__ void __launch_bounds__(JM_WARPS * 32, 2) joint_mix_kernel(const JointPrefillArgs x) {
  constexpr int HP = 16 * HPW, MIXB = HP * 2 + 16;
  __shared__ __align__(16) uint8_t sMix[2 * HP * MIXB];  // [2 (hi, lo)][HP] rows of HP halves
  pdl_launch_dependents();
  const JointArgs& a = x.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
  const int H = a.H, quads = (H + 3) / 4, blk = x.block0 + (blockIdx.x >> 1), b = x.block_seq[blk], q = (blockIdx.x & 1) * JM_WARPS + warp;
  const JointSpan sp = joint_span(a, b, x.block_row[blk]);
  const int n_tiles = sp.kept + sp.hi - sp.lo + 1, i0 = blockIdx.y * JM_TILES, i1 = min(n_tiles, i0 + JM_TILES);
  if (i0 >= n_tiles || (blockIdx.x & 1) * JM_WARPS >= sp.rows) {
    pdl_wait();
    return;
  }
  bool rest = false;  // the matrix has a low half (one that is kept in 16 bits has none)
  for (int i = tid; i < HP * HP; i += JM_WARPS * 32) {
    // column c of a k-step: heads 4 t, 4 t + 1 at 2 t, 2 t + 1, heads 4 t + 2, 4 t + 3 eight further
    const int h = i / HP, c = i % HP, g = c / 16 * 16 + c % 8 / 2 * 4 + c % 16 / 8 * 2 + (c & 1);
    const float w = (h < H && g < H) ? (a.mix != nullptr ? a.mix[h * H + g] : (g == h ? 1.f : 0.f)) : 0.f;
    const __nv_bfloat16 hi = __float2bfloat16(w);
    *reinterpret_cast<__nv_bfloat16*>(sMix + h * MIXB + c * 2) = hi;
    *reinterpret_cast<__nv_bfloat16*>(sMix + (HP + h) * MIXB + c * 2) = __float2bfloat16(w - __bfloat162float(hi));
    rest = rest || w != __bfloat162float(hi);
  }
  const int pos = sp.pos0 + q;
  float far[HPW][2];
#pragma unroll
  for (int m = 0; m < HPW; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = m * 16 + g8 + 8 * e;
      far[m][e] = (a.bias != nullptr && h < H) ? a.bias[(size_t)h * a.distances + a.distances - 1] : 0.f;
    }
  rest = __syncthreads_or(rest);
  const uint32_t mix_at = smem_u32(sMix) + ((mi & 1) * 8 + lr) * MIXB + (mi >> 1) * 16;
  uint32_t wh[HPW][HPW][4];
#pragma unroll
  for (int ks = 0; ks < HPW; ++ks)
#pragma unroll
    for (int m = 0; m < HPW; ++m) ldmatrix_x4(mix_at + m * 16 * MIXB + ks * 32, wh[ks][m][0], wh[ks][m][1], wh[ks][m][2], wh[ks][m][3]);
  pdl_wait();
  if (q >= sp.rows) return;
  const size_t at = (size_t)(blk - x.block0) * x.tiles + i0;
  const uint4* scores = x.scores + (at * quads + t4) * (JP_ROWS * JP_KEYS) + q * JP_KEYS + g8;
  uint4* weights = x.weights + (at * H + g8) * (JP_ROWS * 4) + q * 4 + t4;
  float2* stats = x.stats + (at * H + g8) * JP_ROWS + q;
  for (int i = i0; i < i1; ++i) {
    const int key0 = (i < sp.kept ? i : sp.lo + i - sp.kept) * JP_KEYS;
    const bool near = a.bias != nullptr && pos - key0 - (JP_KEYS - 1) < a.distances - 1;
    float acc[HPW][4][4];
#pragma unroll
    for (int m = 0; m < HPW; ++m)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[m][j][e] = near ? 0.f : far[m][e >> 1];
#pragma unroll
    for (int ks = 0; ks < HPW; ++ks) {
      uint4 s[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        s[j] = 4 * ks + t4 < quads ? __ldcs(scores + (size_t)4 * ks * (JP_ROWS * JP_KEYS) + 8 * j) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
#pragma unroll
        for (int m = 0; m < HPW; ++m) mma_bf16_16816(acc[m][j], wh[ks][m], s[j].z, s[j].w);
#pragma unroll
        for (int m = 0; m < HPW; ++m) mma_bf16_16816(acc[m][j], wh[ks][m], s[j].x, s[j].y);
      }
      if (rest) {
#pragma unroll
        for (int m = 0; m < HPW; ++m) {
          uint32_t wl[4];
          ldmatrix_x4(mix_at + (HP + m * 16) * MIXB + ks * 32, wl[0], wl[1], wl[2], wl[3]);
#pragma unroll
          for (int j = 0; j < 4; ++j) mma_bf16_16816(acc[m][j], wl, s[j].x, s[j].y);
        }
      }
    }
    scores += (size_t)quads * (JP_ROWS * JP_KEYS);
    const bool whole = key0 + JP_KEYS - 1 <= pos && (a.window <= 0 || key0 > pos - a.window || key0 + JP_KEYS <= a.keep_first);
    if (near || !whole) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int key = key0 + 8 * (j >> 1) + 2 * t4 + (j & 1), dist = min(max(pos - key, 0), a.distances - 1);
        const bool ok = key <= pos && (a.window <= 0 || key > pos - a.window || key < a.keep_first);
#pragma unroll
        for (int m = 0; m < HPW; ++m)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float& v = acc[m][j >> 1][2 * e + (j & 1)];
            if (near) v += a.bias[(size_t)min(m * 16 + g8 + 8 * e, H - 1) * a.distances + dist];
            v = ok ? v : -INFINITY;
          }
      }
    }
    float top[HPW][2], sum[HPW][2];
#pragma unroll
    for (int m = 0; m < HPW; ++m)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        top[m][e] = -INFINITY;
#pragma unroll
        for (int j = 0; j < 4; ++j) top[m][e] = fmaxf(top[m][e], fmaxf(acc[m][j][2 * e], acc[m][j][2 * e + 1]));
      }
#pragma unroll
    for (int d = 1; d < 4; d <<= 1)
#pragma unroll
      for (int m = 0; m < HPW; ++m)
#pragma unroll
        for (int e = 0; e < 2; ++e) top[m][e] = fmaxf(top[m][e], __shfl_xor_sync(0xffffffffu, top[m][e], d));
#pragma unroll
    for (int m = 0; m < HPW; ++m)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float base = top[m][e] == -INFINITY ? 0.f : ceilf(top[m][e] * 1.4426950408889634f);
        top[m][e] = top[m][e] == -INFINITY ? JP_NONE : base;
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = joint_exp2(fmaf(acc[m][j >> 1][2 * e + (j & 1)], 1.4426950408889634f, -base));
        sum[m][e] = ((v[0] + v[1]) + (v[2] + v[3])) + ((v[4] + v[5]) + (v[6] + v[7]));
        if (m * 16 + 8 * e + g8 < H)
          weights[(m * 16 + 8 * e) * (JP_ROWS * 4)] =
              make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
      }
#pragma unroll
    for (int d = 1; d < 4; d <<= 1)
#pragma unroll
      for (int m = 0; m < HPW; ++m)
#pragma unroll
        for (int e = 0; e < 2; ++e) sum[m][e] += __shfl_xor_sync(0xffffffffu, sum[m][e], d);
    if (t4 == 0) {
#pragma unroll
      for (int m = 0; m < HPW; ++m)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          if (m * 16 + 8 * e + g8 < H) stats[(m * 16 + 8 * e) * JP_ROWS] = make_float2(top[m][e], sum[m][e]);
    }
    weights += H * JP_ROWS * 4;
    stats += H * JP_ROWS;
  }
}

// ----------------------------------------------------------------------------- values
__host__ __device__ inline int joint_values_smem(int W) { return JV_PLACES * ((W + 63) / 64) * JV_CHUNK + 1024; }

__device__ __forceinline__ float joint_pow2(float e) {  // of a whole number up to 0
  return e < -126.f ? 0.f : __int_as_float(((int)e + 127) << 23);
}

// grid (wide blocks, H).  Four warps bring the weights to tensor memory (thread = token), one loads values, one multiplies.  Tensor
// memory: O at 0, the weights of place u at 128 + 32 (u % 2).
static __global__ void __launch_bounds__(JV_THREADS, 2)
joint_values_kernel(const __grid_constant__ CUtensorMap tmV, const JointPrefillArgs x) {
  extern __shared__ uint8_t jv_raw[];
  __shared__ uint64_t v_full[JV_PLACES], v_empty[JV_PLACES], p_full[2], pv_done[2];
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  const JointArgs& a = x.a;
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0);
  const int H = a.H, h = blockIdx.y, blk0 = x.wide[2 * blockIdx.x], n_blk = x.wide[2 * blockIdx.x + 1], b = x.block_seq[blk0];
  const JointTiles all(joint_span(a, b, x.block_row[blk0]), joint_span(a, b, x.block_row[blk0 + n_blk - 1]));
  const int places = (all.n + 1) / 2, chunks = (a.W + 63) / 64;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(jv_raw) + 1023) & ~uintptr_t(1023));
  // (places whose pages end early: their rows are multiplied by weights of zero)
  for (int i = threadIdx.x; i < JV_PLACES * chunks * JV_CHUNK / 16; i += JV_THREADS) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  if (threadIdx.x == 0) {
    for (int i = 0; i < JV_PLACES; ++i) {
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&p_full[i], 128);
      mbar_init(&pv_done[i], 1);
    }
    abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(&tmem_slot, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();  // (only now: a CTA of the next kernel must not take the tensor memory that this one still waits for)
  const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_slot, 0);
  pdl_wait();

  if (warp == 4) {
    const JointLoader ld{a, all, a.block_tables + (size_t)b * a.max_blocks};
    const bool leader = elect_one();
    const int g = h / (H / a.G);
    bool ok = true;
    for (int u = 0; u < places && ok; ++u) {
      const int s = u % JV_PLACES, turn = u / JV_PLACES;
      if (turn > 0) ok = mbar_wait_bounded(&v_empty[s], (turn - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (leader) {
        mbar_expect_tx(&v_full[s], ld.pages(2 * u, 4) * chunks * 2048);
        for (int p = 0; p < 4; ++p) {
          const int page = ld.page(2 * u, p);
          if (page < 0) continue;
          const int row = ld.row(page, g);
          for (int c = 0; c < chunks; ++c) tma_load_2d(smem + (s * chunks + c) * JV_CHUNK + p * 2048, &tmV, &v_full[s], c * 64, row);
        }
      }
      __syncwarp();
    }
  } else if (warp == 5) {
    const bool leader = elect_one();
    const uint32_t idesc = umma_idesc_bf16(JP_M, a.W) | UMMA_B_MN_MAJOR, va = smem_u32(smem);
    bool ok = true;
    for (int u = 0; u < places && ok; ++u) {
      const int s = u % JV_PLACES;
      ok = mbar_wait_bounded(&v_full[s], (u / JV_PLACES) & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x) &&
           mbar_wait_bounded(&p_full[u & 1], (u >> 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const uint32_t vd = umma_desc_lo(va + s * chunks * JV_CHUNK, JV_CHUNK);
#pragma unroll
      for (int k = 0; k < JV_PLACE / 16; ++k)  // 16 keys: 8 columns of weights, 2 KB of the values
        umma_bf16_ts_if(leader, tmem, tmem + 128 + 32 * (u & 1) + 8 * k, vd + k * (2048 >> 4), UMMA_DESC_HI_SW128, idesc, u > 0 || k > 0);
      umma_commit_if(leader, &pv_done[u & 1]);
      umma_commit_if(leader, &v_empty[s]);
    }
    __syncwarp();
  } else {
    const int r = threadIdx.x, bi = min(r / JP_ROWS, n_blk - 1), rb = r - bi * JP_ROWS, row0 = x.block_row[blk0 + bi];
    const uint32_t lanes = (uint32_t)(warp * 32) << 16;
    const JointSpan sp = joint_span(a, b, row0);
    const bool on = rb < sp.rows;
    const JointOwn own(all, sp, on);
    const size_t at = (size_t)(blk0 + bi - x.block0) * x.tiles * H + h, step = (size_t)H;
    const uint4* wp = x.weights + at * 64 + (on ? rb : 0) * 4;
    const float2* mp = x.stats + at * JP_ROWS + (on ? rb : 0);
    const float sink = a.sink != nullptr ? a.sink[h] * 1.4426950408889634f : -INFINITY;
    float M = sink == -INFINITY ? JP_NONE : ceilf(sink), L = 0.f;
    const int n_own = on ? sp.kept + sp.hi - sp.lo + 1 : 0;
    for (int i = 0; i < n_own; i += 8) {
      float2 st[8];
      float top = M;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        st[j] = i + j < n_own ? mp[(size_t)(i + j) * step * JP_ROWS] : make_float2(JP_NONE, 0.f);
        top = fmaxf(top, st[j].x);
      }
      L *= joint_pow2(M - top);
      M = top;
#pragma unroll
      for (int j = 0; j < 8; ++j) L = fmaf(st[j].y, joint_pow2(st[j].x - top), L);
    }
    if (sink != -INFINITY) L += exp2f(sink - M);
    struct Fetched {
      uint4 w[2][4];
      float m[2];
    };
    auto fetch = [&](int u) {  // of the place's two tiles, what is this token's
      Fetched f;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const bool my = own.has(2 * u + e);
#pragma unroll
        for (int g = 0; g < 4; ++g) f.w[e][g] = my ? wp[g] : make_uint4(0, 0, 0, 0);
        f.m[e] = my ? mp->x : JP_NONE;
        if (my) {
          wp += step * 64;
          mp += step * JP_ROWS;
        }
      }
      return f;
    };
    Fetched next = fetch(0), after = fetch(1);  // (two places ahead; none is own.has() past the last)
    for (int u = 0; u < places; ++u) {
      const Fetched now = next;
      next = after;
      after = fetch(u + 2);
      uint32_t pk[32];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float f = joint_pow2(now.m[e] - M);
        const __nv_bfloat162 f2 = __floats2bfloat162_rn(f, f);
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          const uint32_t src[4] = {now.w[e][g].x, now.w[e][g].y, now.w[e][g].z, now.w[e][g].w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const __nv_bfloat162 y = __hmul2(*reinterpret_cast<const __nv_bfloat162*>(&src[j]), f2);
            pk[16 * e + 4 * j + g] = *reinterpret_cast<const uint32_t*>(&y);
          }
        }
      }
      // (no early exit on a failed wait: every thread arrives at every barrier, later waits return at once)
      if (u > 1) mbar_wait_bounded(&pv_done[u & 1], ((u >> 1) - 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      __syncwarp();
      tc_fence_after();
      tmem_st16(tmem + lanes + 128 + 32 * (u & 1), pk);
      tmem_st16(tmem + lanes + 128 + 32 * (u & 1) + 16, pk + 16);
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_full[u & 1]);
    }
    mbar_wait_bounded(&pv_done[(places - 1) & 1], ((places - 1) >> 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
    __syncwarp();
    tc_fence_after();
    const float inv = L > 0.f ? a.out_scale / L : 0.f;
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(row0 + (on ? rb : 0)) * a.ld_out + (size_t)h * a.W;
    for (int c = 0; c < a.W / 16; ++c) {
      uint32_t o[16];
      tmem_ld16(tmem + lanes + 16 * c, o);
      tmem_ld_wait();
      if (on) {
        uint32_t p[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) p[j] = pack_bf16x2(__uint_as_float(o[2 * j]) * inv, __uint_as_float(o[2 * j + 1]) * inv);
        *reinterpret_cast<uint4*>(out + 16 * c) = make_uint4(p[0], p[1], p[2], p[3]);
        *reinterpret_cast<uint4*>(out + 16 * c + 8) = make_uint4(p[4], p[5], p[6], p[7]);
      }
    }
  }
  if (abort_flag) {
    // a wait gave up: give copies that may still be in flight time to land before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) tmem_dealloc(tmem, 256);
}

}  // namespace oxb
