// Attention on the scores of all heads together (joint.cuh) for long portions, in two kernels.
//
// joint_scores_kernel: a CTA has 16 tokens of a sequence and all heads.  For 32 keys at a time every warp takes the scores of
// its heads, which meet in shared memory; then every warp mixes one token's (the mixing matrix and the scores as a high and a
// low half each, three products for one, float32 sums) and leaves exp2(score - m) in bfloat16, its sum and m, the largest score
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
constexpr int JV_WARPS = 8, JV_STAGES = 4;
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
  return JP_WARPS * 2 * 16 * (HD * 2 + 16) + hp * JP_HEAD * 4 + 2 * hp * (hp + 8) * 2;
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
  uint8_t* sMix = reinterpret_cast<uint8_t*>(sS + HP * JP_HEAD);          // [2 (hi, lo)][HP] rows of HP halves, in binary logarithms
  for (int i = tid; i < HP * JP_HEAD; i += JP_WARPS * 32) sS[i] = 0.f;    // (heads that do not exist count for nothing)
  for (int i = tid; i < HP * HP; i += JP_WARPS * 32) {
    const int h = i / HP, g = i % HP;
    const float w = (h < H && g < H) ? (a.mix != nullptr ? a.mix[h * H + g] : (g == h ? 1.f : 0.f)) * 1.4426950408889634f : 0.f;
    const __nv_bfloat16 hi = __float2bfloat16(w);
    *reinterpret_cast<__nv_bfloat16*>(sMix + h * MIXB + g * 2) = hi;
    *reinterpret_cast<__nv_bfloat16*>(sMix + (HP + h) * MIXB + g * 2) = __float2bfloat16(w - __bfloat162float(hi));
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
  // a warp's pages in order: tile, page of the tile, head (heads of one key head together)
  auto load = [&](int item, int slot) {
    const int i = item / ITEMS, page = 2 * tile_of(i) + (item % ITEMS) / (ITEMS / 2), head = h0 + (SAME ? 0 : item % HPW);
    if (page > last_page || head >= H) return;
    int id = bt[page];
    if ((unsigned)id >= (unsigned)a.num_blocks) {
      if (lane == 0) oxb_report(OXB_BAD_BLOCK_ID, id);
      id = 0;
    }
    joint_load_page<HD>(ring + slot * STAGE, a, id, head / per, lane);
  };
  const JointCap cap = joint_cap(a);
  const int items = works ? n_tiles * ITEMS : 0;
  if (items > 0) load(0, 0);
  cp_async_commit();
  const uint32_t mix_at = smem_u32(sMix) + ((mi & 1) * 8 + lr) * MIXB + (mi >> 1) * 16;
  const int pos = sp.pos0 + warp;  // this warp's token in the second half of a round
  float far[HPW][2];
#pragma unroll
  for (int m = 0; m < HPW; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int h = m * 16 + g8 + 8 * i;
      far[m][i] = (a.bias != nullptr && h < H) ? a.bias[(size_t)h * a.distances + a.distances - 1] * 1.4426950408889634f : 0.f;
    }
  // this lane's pieces of a tile: head 8 (2 m + e) further is 8 * 16 rows further
  uint4* weights = x.weights + ((size_t)blockIdx.x * x.tiles * H + g8) * (JP_ROWS * 4) + warp * 4 + t4;
  float2* stats = x.stats + ((size_t)blockIdx.x * x.tiles * H + g8) * JP_ROWS + warp;
  __syncthreads();
  for (int i = 0; i < n_tiles; ++i) {
    const int tile = tile_of(i);
    if (works) {
#pragma unroll
      for (int it = 0; it < ITEMS; ++it) {
        const int item = i * ITEMS + it, half = it / (ITEMS / 2);
        if (item + 1 < items) load(item + 1, (it + 1) & 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncwarp();
        if (2 * tile + half <= last_page) {
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
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int key = nt * 8 + 2 * t4;
            const float f0 = *reinterpret_cast<const float*>(st + key * ROWB + HD * 2) * cap.factor;
            const float f1 = *reinterpret_cast<const float*>(st + (key + 1) * ROWB + HD * 2) * cap.factor;
#pragma unroll
            for (int j = 0; j < NH; ++j) {
              const int h = h0 + (SAME ? j : it % HPW);
              if (h >= H) continue;
#pragma unroll
              for (int e = 0; e < 2; ++e)
                *reinterpret_cast<float2*>(sS + h * JP_HEAD + (g8 + 8 * e) * JP_QROW + half * 16 + key) =
                    make_float2(joint_capped_fast(s[j][nt][2 * e], f0, cap), joint_capped_fast(s[j][nt][2 * e + 1], f1, cap));
            }
          }
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
        uint32_t wh[HPW][4], wl[HPW][4];
#pragma unroll
        for (int m = 0; m < HPW; ++m) {
          ldmatrix_x4(mix_at + m * 16 * MIXB + ks * 32, wh[m][0], wh[m][1], wh[m][2], wh[m][3]);
          ldmatrix_x4(mix_at + (HP + m * 16) * MIXB + ks * 32, wl[m][0], wl[m][1], wl[m][2], wl[m][3]);
        }
        const float* src = sS + (ks * 16 + 2 * t4) * JP_HEAD + warp * JP_QROW + g8;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t bh[2], bl[2];
          split_bf16x2(src[8 * j], src[JP_HEAD + 8 * j], bh[0], bl[0]);
          split_bf16x2(src[8 * JP_HEAD + 8 * j], src[9 * JP_HEAD + 8 * j], bh[1], bl[1]);
#pragma unroll
          for (int m = 0; m < HPW; ++m) mma_bf16_16816(acc[m][j], wh[m], bl[0], bl[1]);
#pragma unroll
          for (int m = 0; m < HPW; ++m) mma_bf16_16816(acc[m][j], wl[m], bh[0], bh[1]);
#pragma unroll
          for (int m = 0; m < HPW; ++m) mma_bf16_16816(acc[m][j], wh[m], bh[0], bh[1]);
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
              if (near) v = fmaf(a.bias[(size_t)min(m * 16 + g8 + 8 * e, H - 1) * a.distances + dist], 1.4426950408889634f, v);
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
          const float base = top[m][e] == -INFINITY ? 0.f : ceilf(top[m][e]);
          top[m][e] = top[m][e] == -INFINITY ? JP_NONE : base;
          float v[8];
          sum[m][e] = 0.f;
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            v[j] = joint_exp2(acc[m][j >> 1][2 * e + (j & 1)] - base);
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

__host__ __device__ inline int joint_values_smem(int HD) { return JV_STAGES * JP_KEYS * (HD * 2 + 16) + JV_WARPS * JP_ROWS * 2 * 4; }

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
  pdl_wait();
  auto load = [&](int i) {
    uint8_t* st = jv_smem + (i % JV_STAGES) * STAGE;
    constexpr int PIECES = 16 * ROWB / 16;  // of a page
    for (int c = tid; c < 2 * PIECES; c += JV_WARPS * 32) {
      const int page = 2 * tile_of(i) + c / PIECES;
      uint8_t* dst = st + c * 16;
      int id = page <= last_page ? bt[page] : -1;
      if (id >= a.num_blocks) {
        oxb_report(OXB_BAD_BLOCK_ID, id);
        id = -1;
      }
      if (id >= 0) cp_async16(dst, reinterpret_cast<const uint8_t*>(a.cache) + ((size_t)id * a.G + g) * 16 * ROWB + (c % PIECES) * 16);
      else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
  };
#pragma unroll
  for (int i = 0; i < JV_STAGES - 1; ++i) {
    if (i < n_tiles) load(i);
    cp_async_commit();
  }
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
  // this warp's number of a tile, -1: not one of its own
  auto mine = [&](int i) {
    if (!works || i >= n_tiles) return -1;
    const int tile = tile_of(i);
    return tile < sp.kept ? tile : (tile >= sp.lo && tile <= sp.hi ? sp.kept + tile - sp.lo : -1);
  };
  uint4 w[2][2];
  float m[2][2];
  auto fetch = [&](int i, uint4 (&fw)[2], float (&fm)[2]) {
    const int k = mine(i);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool on = k >= 0 && g8 + 8 * e < sp.rows;
      const size_t at = on ? (size_t)k * H * JP_ROWS + g8 + 8 * e : 0;
      fw[e] = on ? weights[at * 4] : make_uint4(0, 0, 0, 0);
      fm[e] = on ? stats[at].x : JP_NONE;
    }
  };
  auto step = [&](int i, uint4 (&fw)[2], float (&fm)[2]) {
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
    cp_async_wait<JV_STAGES - 2>();
    __syncthreads();
    if (i + JV_STAGES - 1 < n_tiles) load(i + JV_STAGES - 1);
    cp_async_commit();
    if (mine(i) < 0) return;
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
  };
  fetch(0, w[0], m[0]);
  fetch(1, w[1], m[1]);
  for (int i = 0; i < n_tiles; i += 2) {
    step(i, w[0], m[0]);
    if (i + 1 < n_tiles) step(i + 1, w[1], m[1]);
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
