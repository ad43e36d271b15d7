// Attention on the scores of all heads together (joint.cuh) for long portions, in three kernels.
//
// joint_scores_kernel: capped scores of four heads for 64 tokens per CTA, left as the operand registers that the mixing wants: a
// high and a low half each, the four heads of a (token, key) in 16 bytes.
// joint_mix_kernel: a warp mixes one token's scores with 32 keys at a time over all heads (hi hi + hi lo + lo hi, float32 sums)
// and leaves exp2(score - m) in bfloat16, its sum and m, the largest score rounded up to a whole power of two.
// joint_values_kernel: weights times values, a head and 128 tokens per CTA.  Between tiles with different m the weights are
// multiplied by powers of two, which rounds nothing.
//
// Weights lie as the last kernel's operand registers want them: of the 32 keys of a tile a lane has 2 t4, 2 t4 + 1 and those
// 8, 16 and 24 further, 16 bytes in all.
#pragma once
#include "joint.cuh"
#include "retention.cuh"

namespace oxb {

constexpr int JP_ROWS = 16, JP_KEYS = 32;   // tokens of a block, keys of a tile
constexpr int JC_WARPS = 8, JC_BLOCKS = 4;  // joint_scores_kernel: a warp has a block and a page of the tile
constexpr int JM_WARPS = 8, JM_TILES = 8;   // joint_mix_kernel: tiles per warp
constexpr int JV_WARPS = 8, JV_STAGES = 6;
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

template <int HD, bool SAME>
__host__ __device__ constexpr int joint_scores_stages() { return SAME ? 4 : 2; }
template <int HD, bool SAME>
__host__ __device__ constexpr int joint_scores_smem() {
  return 4 * JC_BLOCKS * JP_ROWS * (HD * 2 + 16) + joint_scores_stages<HD, SAME>() * (SAME ? 1 : 4) * JP_KEYS * (HD * 2 + 16) + 2 * 8 * 4;
}

// grid (wide blocks x 2, quads of heads, parts of the tiles).  SAME: the four heads share a key head.
template <int HD, bool SAME>
__global__ void __launch_bounds__(JC_WARPS * 32, SAME ? 2 : 1) joint_scores_kernel(const JointPrefillArgs x) {
  constexpr int ROWB = HD * 2 + 16, PAGE = 16 * ROWB, KS = HD / 16, NK = SAME ? 1 : 4, STAGES = joint_scores_stages<HD, SAME>();
  constexpr int QROWS = JC_BLOCKS * JP_ROWS, STAGE = 2 * NK * PAGE;
  extern __shared__ __align__(16) uint8_t jc_smem[];
  __shared__ int gave_up;
  pdl_launch_dependents();
  const JointArgs& a = x.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
  const int H = a.H, per = H / a.G, quad = blockIdx.y, quads = gridDim.y;
  const int blk0 = x.wide[2 * (blockIdx.x >> 1)] + (blockIdx.x & 1) * JC_BLOCKS;
  const int n_blk = min(JC_BLOCKS, x.wide[2 * (blockIdx.x >> 1)] + x.wide[2 * (blockIdx.x >> 1) + 1] - blk0);
  if (n_blk <= 0) {
    pdl_wait();
    return;
  }
  const int b = x.block_seq[blk0], row0 = x.block_row[blk0], qg = warp % JC_BLOCKS, half = warp / JC_BLOCKS;
  const JointSpan last = joint_span(a, b, x.block_row[blk0 + n_blk - 1]);
  const JointTiles all(joint_span(a, b, row0), last);
  const JointOwn own(all, joint_span(a, b, x.block_row[min(blk0 + qg, blk0 + n_blk - 1)]), qg < n_blk);
  const int share = (all.n + gridDim.z - 1) / gridDim.z, i0 = blockIdx.z * share, i1 = min(all.n, i0 + share);
  uint8_t *sQ = jc_smem, *ring = sQ + 4 * QROWS * ROWB;  // [4 heads][64] rows; [stages][2 pages][NK]
  uint64_t *full = reinterpret_cast<uint64_t*>(ring + STAGES * STAGE), *empty = full + STAGES;
  const int* bt = a.block_tables + (size_t)b * a.max_blocks;
  const int rows = last.pos0 + last.rows - joint_span(a, b, row0).pos0;
  if (tid == 0) {
    gave_up = 0;
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, JC_WARPS);
    }
    mbar_fence_init();
  }
  auto load = [&](int i) {  // by one thread
    const int k = (i - i0) % STAGES, page = 2 * all.tile(i), pages = page + 1 <= all.last_page ? 2 : 1;
    mbar_expect_tx(full + k, pages * NK * PAGE);
    for (int p = 0; p < pages; ++p) {
      int id = bt[page + p];
      if ((unsigned)id >= (unsigned)a.num_blocks) {
        oxb_report(OXB_BAD_BLOCK_ID, id);
        id = 0;
      }
      for (int c = 0; c < NK; ++c)
        bulk_load(ring + k * STAGE + (p * NK + c) * PAGE,
                  reinterpret_cast<const uint8_t*>(a.cache) + ((size_t)id * a.G + min(quad * 4 + c, H - 1) / per) * PAGE, PAGE, full + k);
    }
  };
  pdl_wait();
  if (tid == 0)
    for (int i = i0; i < i0 + STAGES && i < i1; ++i) load(i);
  for (int i = tid; i < 4 * QROWS * (HD / 8); i += JC_WARPS * 32) {
    const int c = i % (HD / 8), r = i / (HD / 8) % QROWS, h = i / (HD / 8) / QROWS;
    uint8_t* dst = sQ + (h * QROWS + r) * ROWB + c * 16;
    if (r < rows && quad * 4 + h < H)
      cp_async16(dst, reinterpret_cast<const __nv_bfloat16*>(a.q) + ((size_t)(row0 + r) * H + quad * 4 + h) * HD + c * 8);
    else
      *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);  // (a head past the last has scores of zero)
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  const JointCap cap = joint_cap(a);
  const uint32_t q_at = smem_u32(sQ) + (qg * JP_ROWS + (mi & 1) * 8 + lr) * ROWB + (mi >> 1) * 16;
  uint4* dst = x.scores + ((size_t)(blk0 + qg - x.block0) * x.tiles * quads + quad) * (JP_ROWS * JP_KEYS) + g8 * JP_KEYS + half * 16 + 2 * t4;
  for (int i = i0; i < i1; ++i) {
    const int k = (i - i0) % STAGES, turn = (i - i0) / STAGES;
    const int done = i - 1;  // the next tile of its place, once every warp is done with it
    if (tid == 0 && done >= i0 && done + STAGES < i1) {
      mbar_wait_bounded(empty + (done - i0) % STAGES, ((done - i0) / STAGES) & 1, &gave_up, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
      load(done + STAGES);
    }
    mbar_wait_bounded(full + k, turn & 1, &gave_up, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
    if (own.has(i) && 2 * all.tile(i) + half <= all.last_page) {
      const uint8_t* st = ring + k * STAGE + half * NK * PAGE;
      const uint32_t k_at = smem_u32(st) + ((mi >> 1) * 8 + lr) * ROWB + (mi & 1) * 16;
      float s[4][2][4];
#pragma unroll
      for (int h = 0; h < 4; ++h)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[h][0][e] = s[h][1][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t kb[4];
        if (SAME) ldmatrix_x4(k_at + ks * 32, kb[0], kb[1], kb[2], kb[3]);
#pragma unroll
        for (int h = 0; h < 4; ++h) {
          uint32_t qa[4];
          ldmatrix_x4(q_at + h * QROWS * ROWB + ks * 32, qa[0], qa[1], qa[2], qa[3]);
          if (!SAME) ldmatrix_x4(k_at + h * PAGE + ks * 32, kb[0], kb[1], kb[2], kb[3]);
          mma_bf16_16816(s[h][0], qa, kb[0], kb[1]);
          mma_bf16_16816(s[h][1], qa, kb[2], kb[3]);
        }
      }
      const float* inv = reinterpret_cast<const float*>(st + 2 * t4 * ROWB + HD * 2);
#pragma unroll
      for (int h = 0; h < 4; ++h)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[h][nt][e] *= inv[((SAME ? 0 : h) * PAGE + (nt * 8 + (e & 1)) * ROWB) / 4] * cap.factor;
      if (cap.cap > 0.f) {
#pragma unroll
        for (int h = 0; h < 4; ++h)
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[h][nt][e] = joint_capped_of(s[h][nt][e], cap);
      }
      uint4* to = dst + (size_t)own.number(i) * quads * (JP_ROWS * JP_KEYS);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {  // row g8 + 8 (e >> 1), key 2 t4 + (e & 1) of tile nt
          uint4 o;
          split_bf16x2(s[0][nt][e], s[1][nt][e], o.x, o.z);
          split_bf16x2(s[2][nt][e], s[3][nt][e], o.y, o.w);
          to[(e >> 1) * 8 * JP_KEYS + nt * 8 + (e & 1)] = o;
        }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(empty + k);
  }
}

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
  const JointTiles all(first, end);
  const JointOwn owned(all, sp, works);
  const int n_tiles = all.n;
  uint64_t *full = reinterpret_cast<uint64_t*>(jv_smem + JV_STAGES * STAGE + JV_WARPS * JP_ROWS * 2 * 4), *empty = full + JV_STAGES;
  __shared__ int gave_up;
  // tile i of all, both pages, by one thread; places of pages past the portion keep what they hold (zeros, or another tile)
  auto load = [&](int i) {
    uint8_t* st = jv_smem + (i % JV_STAGES) * STAGE;
    const int page = 2 * all.tile(i), pages = page + 1 <= all.last_page ? 2 : 1;
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
    for (int i0 = lane >> 4; i0 < own && on; i0 += 16) {
      float2 st[8];
      float top = M;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        st[j] = i0 + 2 * j < own ? stats[(size_t)(i0 + 2 * j) * H * JP_ROWS + (lane & 15)] : make_float2(JP_NONE, 0.f);
        top = fmaxf(top, st[j].x);
      }
      L *= joint_pow2(M - top);
      M = top;
#pragma unroll
      for (int j = 0; j < 8; ++j) L = fmaf(st[j].y, joint_pow2(st[j].x - top), L);
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
  const bool on[2] = {works && g8 < sp.rows, works && g8 + 8 < sp.rows};
  const uint4* wp = weights + g8 * 4;
  const float2* mp = stats + g8;
  const size_t step = (size_t)H * JP_ROWS;
  uint4 w[2][2];
  float m[2][2];
  auto fetch = [&](int i, uint4 (&fw)[2], float (&fm)[2]) {  // of this warp's next tile, if i is one
    const bool my = owned.has(i);
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
    const bool my = owned.has(i);
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
