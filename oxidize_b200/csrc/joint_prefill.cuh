// Attention on the scores of all heads together (joint.cuh) for long portions, in two kernels.
//
// joint_scores_kernel: a CTA has 16 tokens of a sequence and all heads.  For 32 keys at a time every warp takes the scores of
// its heads, which meet in shared memory; then every warp mixes one token's (the mixing matrix and the scores as a high and a
// low half each, hi hi + hi lo + lo hi, float32 sums) and leaves exp2(score - m) in bfloat16, its sum and m, the largest score
// rounded up to a whole power of two.
// joint_values_kernel: weights times values, a head and 128 tokens per CTA.  Between tiles with different m the weights are
// multiplied by powers of two, which rounds nothing.
//
// Weights lie as the second kernel's operand registers want them: of the 32 keys of a tile a lane has 2 t4, 2 t4 + 1 and those
// 8, 16 and 24 further, 16 bytes in all.
#pragma once
#include "joint.cuh"
#include "retention.cuh"

namespace oxb {

constexpr int JP_ROWS = 16, JP_KEYS = 32, JP_WARPS = 16, JP_QROW = 40, JP_HEAD = JP_ROWS * JP_QROW + 4;
constexpr int JV_WARPS = 8, JV_STAGES = 6;
constexpr float JP_NONE = -1e30f;  // m of a tile without a visible key

struct JointPrefillArgs {
  JointArgs a;
  const int* block_seq;  // [blocks] sequence of every block of 16 tokens
  const int* block_row;  // [blocks] its first row
  const int* wide;       // [wide blocks, 2]: first block of 16, number of them (up to 8, of one sequence)
  uint4* weights;        // [blocks, tiles, H, 16, 4]
  float2* stats;         // [blocks, tiles, H, 16]: m, sum
  int tiles;             // most tiles of a block
  int block0;            // the first block of this launch: scratch is numbered from there
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

__host__ __device__ inline int joint_scores_smem(int HD, int HPW) {
  const int hp = 16 * HPW;
  return JP_WARPS * 2 * 16 * (HD * 2 + 16) + hp * JP_HEAD * 4 + 2 * hp * (hp + 8) * 2 + JP_WARPS * 2 * 8;
}

// grid (blocks of 16 tokens).  HPW heads per warp (H <= 16 HPW); SAME: a warp's heads share a key head.
template <int HD, int HPW, bool SAME>
__global__ void __launch_bounds__(JP_WARPS * 32, 1) joint_scores_kernel(const JointPrefillArgs x) {
  constexpr int ROWB = HD * 2 + 16, STAGE = 16 * ROWB, KS = HD / 16, HP = 16 * HPW, MIXB = HP * 2 + 16;
  constexpr int ITEMS = SAME ? 2 : 2 * HPW;  // pages a warp reads per tile
  extern __shared__ __align__(16) uint8_t jp_smem[];
  pdl_launch_dependents();
  const JointArgs& a = x.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
  const int H = a.H, per = H / a.G, blk = x.block0 + blockIdx.x, b = x.block_seq[blk], row0 = x.block_row[blk];
  const JointSpan sp = joint_span(a, b, row0);
  uint8_t* ring = jp_smem + warp * 2 * STAGE;
  float* sS = reinterpret_cast<float*>(jp_smem + JP_WARPS * 2 * STAGE);  // [HP][16][40]
  uint8_t* sMix = reinterpret_cast<uint8_t*>(sS + HP * JP_HEAD);          // [2 (hi, lo)][HP] rows of HP halves
  uint64_t* full = reinterpret_cast<uint64_t*>(sMix + 2 * HP * MIXB) + warp * 2;
  __shared__ int gave_up;
  if (tid == 0) gave_up = 0;
  if (lane == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    mbar_fence_init();
  }
  __syncwarp();
  for (int i = tid; i < HP * JP_HEAD; i += JP_WARPS * 32) sS[i] = 0.f;    // (heads that do not exist count for nothing)
  bool rest = false;  // the matrix has a low half (one that is kept in 16 bits has none)
  for (int i = tid; i < HP * HP; i += JP_WARPS * 32) {
    const int h = i / HP, g = i % HP;
    const float w = (h < H && g < H) ? (a.mix != nullptr ? a.mix[h * H + g] : (g == h ? 1.f : 0.f)) : 0.f;
    const __nv_bfloat16 hi = __float2bfloat16(w);
    *reinterpret_cast<__nv_bfloat16*>(sMix + h * MIXB + g * 2) = hi;
    *reinterpret_cast<__nv_bfloat16*>(sMix + (HP + h) * MIXB + g * 2) = __float2bfloat16(w - __bfloat162float(hi));
    rest = rest || w != __bfloat162float(hi);
  }
  const int h0 = warp * HPW, n_tiles = sp.kept + sp.hi - sp.lo + 1, last_page = (sp.pos0 + sp.rows - 1) >> 4;
  const int* bt = a.block_tables + (size_t)b * a.max_blocks;
  auto tile_of = [&](int i) { return i < sp.kept ? i : sp.lo + i - sp.kept; };
  const bool works = h0 < H;
  pdl_wait();
  uint32_t qf[HPW][KS][4];
#pragma unroll
  for (int j = 0; j < HPW; ++j)
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const bool on = h0 + j < H && g8 + 8 * i < sp.rows;
        const __nv_bfloat16* qp = reinterpret_cast<const __nv_bfloat16*>(a.q) +
                                  ((size_t)(row0 + (on ? g8 + 8 * i : 0)) * H + (on ? h0 + j : 0)) * HD + ks * 16 + 2 * t4;
        qf[j][ks][i] = on ? *reinterpret_cast<const uint32_t*>(qp) : 0u;
        qf[j][ks][i + 2] = on ? *reinterpret_cast<const uint32_t*>(qp + 8) : 0u;
      }
  // a warp's pages in order: tile, page of the tile, head (heads of one key head together); the it-th of tile i goes to place it % 2
  auto load = [&](int i, int it) {
    const int page = 2 * tile_of(i) + it / (ITEMS / 2), head = h0 + (SAME ? 0 : it % HPW);
    if (page > last_page || (!SAME && head >= H)) return;
    int id = bt[page];
    if ((unsigned)id >= (unsigned)a.num_blocks) {
      if (lane == 0) oxb_report(OXB_BAD_BLOCK_ID, id);
      id = 0;
    }
    if (lane == 0) {
      mbar_expect_tx(full + (it & 1), STAGE);
      bulk_load(ring + (it & 1) * STAGE, reinterpret_cast<const uint8_t*>(a.cache) + ((size_t)id * a.G + head / per) * STAGE, STAGE, full + (it & 1));
    }
  };
  const JointCap cap = joint_cap(a);
  if (works) load(0, 0);
  const uint32_t mix_at = smem_u32(sMix) + ((mi & 1) * 8 + lr) * MIXB + (mi >> 1) * 16;
  const int pos = sp.pos0 + warp;  // this warp's token in the second half of a round
  float far[HPW][2];
#pragma unroll
  for (int m = 0; m < HPW; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int h = m * 16 + g8 + 8 * i;
      far[m][i] = (a.bias != nullptr && h < H) ? a.bias[(size_t)h * a.distances + a.distances - 1] : 0.f;
    }
  // this lane's pieces of a tile: head 8 (2 m + e) further is 8 * 16 rows further
  uint4* weights = x.weights + ((size_t)blockIdx.x * x.tiles * H + g8) * (JP_ROWS * 4) + warp * 4 + t4;
  float2* stats = x.stats + ((size_t)blockIdx.x * x.tiles * H + g8) * JP_ROWS + warp;
  rest = __syncthreads_or(rest);
  for (int i = 0; i < n_tiles; ++i) {
    const int tile = tile_of(i);
    if (works) {
#pragma unroll
      for (int it = 0; it < ITEMS; ++it) {
        const int half = it / (ITEMS / 2);
        if (it + 1 < ITEMS) load(i, it + 1);
        else if (i + 1 < n_tiles) load(i + 1, 0);
        if (2 * tile + half <= last_page && (SAME || h0 + it % HPW < H)) {
          mbar_wait_bounded(full + (it & 1), (i * (ITEMS / 2) + it / 2) & 1, &gave_up, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
          const uint8_t* st = ring + (it & 1) * STAGE;
          const uint32_t addr = smem_u32(st) + ((mi >> 1) * 8 + lr) * ROWB + (mi & 1) * 16;
          constexpr int NH = SAME ? HPW : 1;
          float s[NH][2][4];
#pragma unroll
          for (int j = 0; j < NH; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[j][0][e] = s[j][1][e] = 0.f;
#pragma unroll
          for (int ks = 0; ks < KS; ++ks) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(addr + ks * 32, b0, b1, b2, b3);
#pragma unroll
            for (int j = 0; j < NH; ++j) {
              mma_bf16_16816(s[j][0], qf[SAME ? j : it % HPW][ks], b0, b1);
              mma_bf16_16816(s[j][1], qf[SAME ? j : it % HPW][ks], b2, b3);
            }
          }
          const float* inv = reinterpret_cast<const float*>(st + 2 * t4 * ROWB + HD * 2);
          float f[2][2];
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 2; ++e) f[nt][e] = inv[(nt * 8 + e) * (ROWB / 4)] * cap.factor;
#pragma unroll
          for (int j = 0; j < NH; ++j)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
              for (int e = 0; e < 4; ++e) s[j][nt][e] *= f[nt][e & 1];
          if (cap.cap > 0.f) {
#pragma unroll
            for (int j = 0; j < NH; ++j)
#pragma unroll
              for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[j][nt][e] = joint_capped_of(s[j][nt][e], cap);
          }
          float* dst = sS + (h0 + (SAME ? 0 : it % HPW)) * JP_HEAD + g8 * JP_QROW + half * 16 + 2 * t4;
#pragma unroll
          for (int j = 0; j < NH; ++j)  // (a head past the last has zeros for queries, and so for scores)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
              for (int e = 0; e < 2; ++e)
                *reinterpret_cast<float2*>(dst + j * JP_HEAD + 8 * e * JP_QROW + nt * 8) = make_float2(s[j][nt][2 * e], s[j][nt][2 * e + 1]);
        }
        __syncwarp();
      }
    }
    __syncthreads();
    float acc[HPW][4][4];
    const int key0 = tile * JP_KEYS;
    const bool near = a.bias != nullptr && pos - key0 - (JP_KEYS - 1) < a.distances - 1;
    if (warp < sp.rows) {
#pragma unroll
      for (int m = 0; m < HPW; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[m][j][e] = near ? 0.f : far[m][e >> 1];
#pragma unroll
      for (int ks = 0; ks < HPW; ++ks) {
        uint32_t wh[HPW][4];
#pragma unroll
        for (int m = 0; m < HPW; ++m) ldmatrix_x4(mix_at + m * 16 * MIXB + ks * 32, wh[m][0], wh[m][1], wh[m][2], wh[m][3]);
        const float* src = sS + (ks * 16 + 2 * t4) * JP_HEAD + warp * JP_QROW + g8;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t bh[2], bl[2];
          split_bf16x2(src[8 * j], src[JP_HEAD + 8 * j], bh[0], bl[0]);
          split_bf16x2(src[8 * JP_HEAD + 8 * j], src[9 * JP_HEAD + 8 * j], bh[1], bl[1]);
#pragma unroll
          for (int m = 0; m < HPW; ++m) mma_bf16_16816(acc[m][j], wh[m], bl[0], bl[1]);
#pragma unroll
          for (int m = 0; m < HPW; ++m) mma_bf16_16816(acc[m][j], wh[m], bh[0], bh[1]);
          if (rest) {
#pragma unroll
            for (int m = 0; m < HPW; ++m) {
              uint32_t wl[4];
              ldmatrix_x4(mix_at + (HP + m * 16) * MIXB + ks * 32, wl[0], wl[1], wl[2], wl[3]);
              mma_bf16_16816(acc[m][j], wl, bh[0], bh[1]);
            }
          }
        }
      }
    }
    __syncthreads();  // the scores are in registers: the next tile's may follow while this one's weights are made
    if (warp < sp.rows) {
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
          sum[m][e] = 0.f;
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            v[j] = joint_exp2(fmaf(acc[m][j >> 1][2 * e + (j & 1)], 1.4426950408889634f, -base));
            sum[m][e] += v[j];
          }
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
    }
    weights += H * JP_ROWS * 4;
    stats += H * JP_ROWS;
  }
}

__host__ __device__ inline int joint_values_smem(int HD) {
  return JV_STAGES * JP_KEYS * (HD * 2 + 16) + JV_WARPS * JP_ROWS * 2 * 4 + 2 * JV_STAGES * 8;
}

__device__ __forceinline__ float joint_pow2(float e) {  // of a whole number up to 0
  return e < -126.f ? 0.f : __int_as_float(((int)e + 127) << 23);
}

// grid (wide blocks, H).  A warp has 16 tokens.
template <int HD>
__global__ void __launch_bounds__(JV_WARPS * 32, 2) joint_values_kernel(const JointPrefillArgs x) {
  constexpr int ROWB = HD * 2 + 16, NT = HD / 8, STAGE = JP_KEYS * ROWB;
  extern __shared__ __align__(16) uint8_t jv_smem[];
  pdl_launch_dependents();
  const JointArgs& a = x.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
  const int H = a.H, h = blockIdx.y, g = h / (H / a.G), blk0 = x.wide[2 * blockIdx.x], n_blk = x.wide[2 * blockIdx.x + 1];
  const int b = x.block_seq[blk0], last = blk0 + n_blk - 1, blk = min(blk0 + warp, last), row0 = x.block_row[blk];
  const bool works = warp < n_blk;
  const JointSpan first = joint_span(a, b, x.block_row[blk0]), end = joint_span(a, b, x.block_row[last]), sp = joint_span(a, b, row0);
  float* sM = reinterpret_cast<float*>(jv_smem + JV_STAGES * STAGE) + warp * JP_ROWS * 2;  // [16] m of the row, [16] 1 / sum
  const int* bt = a.block_tables + (size_t)b * a.max_blocks;
  const int n_tiles = first.kept + end.hi - first.lo + 1, last_page = (end.pos0 + end.rows - 1) >> 4;
  auto tile_of = [&](int i) { return i < first.kept ? i : first.lo + i - first.kept; };
  uint64_t *full = reinterpret_cast<uint64_t*>(jv_smem + JV_STAGES * STAGE + JV_WARPS * JP_ROWS * 2 * 4), *empty = full + JV_STAGES;
  __shared__ int gave_up;
  // tile i of all, both pages, by one thread; places of pages past the portion keep what they hold (zeros, or another tile)
  auto load = [&](int i) {
    uint8_t* st = jv_smem + (i % JV_STAGES) * STAGE;
    const int page = 2 * tile_of(i), pages = page + 1 <= last_page ? 2 : 1;
    mbar_expect_tx(full + i % JV_STAGES, pages * (STAGE / 2));
    for (int k = 0; k < pages; ++k) {
      int id = bt[page + k];
      if ((unsigned)id >= (unsigned)a.num_blocks) {
        oxb_report(OXB_BAD_BLOCK_ID, id);
        id = 0;
      }
      bulk_load(st + k * (STAGE / 2), reinterpret_cast<const uint8_t*>(a.cache) + ((size_t)id * a.G + g) * (STAGE / 2), STAGE / 2, full + i % JV_STAGES);
    }
  };
  for (int i = tid; i < JV_STAGES * STAGE / 16; i += JV_WARPS * 32) reinterpret_cast<uint4*>(jv_smem)[i] = make_uint4(0, 0, 0, 0);
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  if (tid == 0) {
    gave_up = 0;
    for (int i = 0; i < JV_STAGES; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, JV_WARPS);
    }
    mbar_fence_init();
  }
  __syncthreads();
  pdl_wait();
  if (tid == 0)
    for (int i = 0; i < JV_STAGES && i < n_tiles; ++i) load(i);
  // this warp's weights and stats of a tile: 16 rows of 64 bytes, 16 pairs
  const uint4* weights = x.weights + ((size_t)(blk - x.block0) * x.tiles * H + h) * (JP_ROWS * 4) + t4;
  const float2* stats = x.stats + ((size_t)(blk - x.block0) * x.tiles * H + h) * JP_ROWS;
  const int own = sp.kept + sp.hi - sp.lo + 1;
  if (works) {  // a lane has row lane % 16 and every other tile
    const float sink = a.sink != nullptr ? a.sink[h] * 1.4426950408889634f : -INFINITY;
    const bool on = (lane & 15) < sp.rows;
    float M = sink == -INFINITY ? JP_NONE : ceilf(sink), L = 0.f;
    for (int i = lane >> 4; i < own && on; i += 2) {
      const float2 st = stats[(size_t)i * H * JP_ROWS + (lane & 15)];
      const float top = fmaxf(M, st.x);
      L = L * joint_pow2(M - top) + st.y * joint_pow2(st.x - top);
      M = top;
    }
    const float other = __shfl_xor_sync(0xffffffffu, M, 16), top = fmaxf(M, other);
    L *= joint_pow2(M - top);
    L += __shfl_xor_sync(0xffffffffu, L, 16);
    if (sink != -INFINITY) L += exp2f(sink - top);
    if (lane < JP_ROWS) {
      sM[lane] = top;
      sM[JP_ROWS + lane] = L > 0.f ? a.out_scale / L : 0.f;
    }
    __syncwarp();
  }
  float o[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
  const float M[2] = {works ? sM[g8] : 0.f, works ? sM[g8 + 8] : 0.f};
  // tiles 0 .. kept0 - 1 of all and own_lo .. own_hi are this warp's, in that order
  const int kept0 = min(sp.kept, first.kept), own_lo = first.kept + max(sp.lo, first.lo) - first.lo, own_hi = works ? first.kept + sp.hi - first.lo : -1;
  const int extra = sp.kept - kept0;  // (kept tiles that lie in the range of the first block's window)
  const bool on[2] = {works && g8 < sp.rows, works && g8 + 8 < sp.rows};
  const uint4* wp = weights + g8 * 4;
  const float2* mp = stats + g8;
  const size_t step = (size_t)H * JP_ROWS;
  auto mine = [&](int i) { return i <= own_hi && (i < kept0 + extra || i >= own_lo); };
  uint4 w[2][2];
  float m[2][2];
  auto fetch = [&](int i, uint4 (&fw)[2], float (&fm)[2]) {  // of this warp's next tile, if i is one
    const bool my = mine(i);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      fw[e] = on[e] && my ? wp[8 * e * 4] : make_uint4(0, 0, 0, 0);
      fm[e] = on[e] && my ? mp[8 * e].x : JP_NONE;
    }
    if (my) {
      wp += step * 4;
      mp += step;
    }
  };
  auto multiply = [&](int i, uint4 (&fw)[2], float (&fm)[2]) {
    const bool my = mine(i);
    uint32_t p[2][4];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float f = joint_pow2(fm[e] - M[e]);
      const __nv_bfloat162 f2 = __floats2bfloat162_rn(f, f);
      const uint32_t src[4] = {fw[e].x, fw[e].y, fw[e].z, fw[e].w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const __nv_bfloat162 y = __hmul2(*reinterpret_cast<const __nv_bfloat162*>(&src[j]), f2);
        p[e][j] = *reinterpret_cast<const uint32_t*>(&y);
      }
    }
    fetch(i + 2, fw, fm);
    // (every warp waits, whether the tile is its own or not: none may be a whole turn of the places ahead)
    mbar_wait_bounded(full + i % JV_STAGES, (i / JV_STAGES) & 1, &gave_up, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
    if (my) {
      const uint32_t addr = smem_u32(jv_smem + (i % JV_STAGES) * STAGE) + ((mi & 1) * 8 + lr) * ROWB + (mi >> 1) * 16;
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        const uint32_t av[4] = {p[0][2 * ks], p[1][2 * ks], p[0][2 * ks + 1], p[1][2 * ks + 1]};
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(addr + ks * 16 * ROWB + nt * 16, b0, b1, b2, b3);
          mma_bf16_16816(o[nt], av, b0, b1);
          mma_bf16_16816(o[nt + 1], av, b2, b3);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(empty + i % JV_STAGES);
    const int done = i - 2;  // the next tile of its place, once every warp is done with it
    if (tid == 0 && done >= 0 && done + JV_STAGES < n_tiles) {
      mbar_wait_bounded(empty + done % JV_STAGES, (done / JV_STAGES) & 1, &gave_up, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
      load(done + JV_STAGES);
    }
  };
  fetch(0, w[0], m[0]);
  fetch(1, w[1], m[1]);
  for (int i = 0; i < n_tiles; i += 2) {
    multiply(i, w[0], m[0]);
    if (i + 1 < n_tiles) multiply(i + 1, w[1], m[1]);
  }
  if (!works) return;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = g8 + 8 * e;
    if (r >= sp.rows) continue;
    const float inv = sM[JP_ROWS + r];
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(row0 + r) * a.ld_out + (size_t)h * HD + 2 * t4;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) *reinterpret_cast<uint32_t*>(out + nt * 8) = pack_bf16x2(o[nt][2 * e] * inv, o[nt][2 * e + 1] * inv);
  }
}

}  // namespace oxb
