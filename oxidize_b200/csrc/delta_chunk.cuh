// Gated delta rule of long portions: chunks of 64 tokens on the tensor cores.
//
// Inside a chunk that starts from state S0, with the running sums G_t of the decays' logarithms (per key channel, or one number
// per head), the recurrence is a triangular system: with
//     L_ts = beta_t sum_d k_t k_s exp(G_t - G_s)  (s < t),    P_ts = sum_d q_t k_s exp(G_t - G_s)  (s <= t),
//     U = (I + L)^-1 diag(beta) (V - (exp(G) K) S0),   O = (exp(G) Q) S0 + P U,   S' = exp(G_end) S0 + (exp(G_end - G) K)^T U.
// delta_prepare_kernel, all chunks at once: convolutions, unit vectors, decays, L, P, the inverse, and from it
//     W = (I + L)^-1 diag(beta) exp(G) K  and  U0 = (I + L)^-1 diag(beta) V.
// delta_state_kernel, chunk after chunk, the values of a head dealt out to CTAs: U = U0 - W S, then S'.
// delta_output_kernel, all chunks at once: O, its norm and gate.
//
// A portion is worked off in rounds of as many chunks as the scratch holds.
//
// G is kept in binary logarithms, as running sums within blocks of 16 tokens and the blocks' totals, so that what lies between
// two tokens is never the small difference of two large sums; a token's logarithm ends at -72.  In L and P a block off the
// diagonal takes its rows relative to the start of their block and its columns relative to that point, so that no exponent is
// positive; a block on the diagonal takes both relative to its start unless a channel loses more than 2^-60 in it, in which
// case its columns are multiplied by one token's decay at a time.  Every float32 factor enters the bf16 products as a high and
// a low half, and hi hi + hi lo + lo hi is summed in float32 (see retention.cuh).
#pragma once
#include <type_traits>

#include "delta.cuh"
#include "retention.cuh"

namespace oxb {

constexpr int DC = 64;                // tokens per chunk
constexpr int DC_LD = DC + 4;         // floats of a row of L and of the inverse
constexpr int DC_PROW = DC * 2 + 16;  // bytes of a row of 64 halves in shared memory

// Scratch of one (chunk, head), in bytes: arrays as they stand in shared memory (rows padded by 16 bytes), one bulk copy each.
// Pairs of halves lie behind each other (hi, lo).
struct DeltaPlan {
  int w, kb, u0, gend, qt, s, p, u, bytes;  // offsets
};
constexpr int DC_USLICE = DC * (16 * 4 + 16);  // bytes of 16 values of U0, [64][16 + padding]
__host__ __device__ inline DeltaPlan delta_plan(int K, int V) {
  const int rk = 2 * DC * (K * 2 + 16), rv = V * 2 + 16;
  DeltaPlan p;
  p.w = 0;
  p.kb = p.w + rk;
  p.u0 = p.kb + rk;
  p.gend = p.u0 + V / 16 * DC_USLICE;
  p.qt = p.gend + K * 4;
  p.s = p.qt + rk;
  p.p = p.s + 2 * K * rv;
  p.u = p.p + 2 * DC * DC_PROW;
  p.bytes = p.u + 2 * DC * rv;
  return p;
}

struct DeltaChunkArgs {
  DeltaArgs a;
  uint8_t* ws;        // B * round * H blocks of delta_plan(K, V).bytes
  int chunk0, round;  // chunks [chunk0, chunk0 + round) of every portion
};
__device__ __forceinline__ uint8_t* delta_block(const DeltaChunkArgs& x, int bytes, int b, int chunk, int h) {
  return x.ws + ((size_t)(b * x.round + chunk - x.chunk0) * x.a.H + h) * bytes;
}

__device__ __forceinline__ void delta_split8(const float* v, void* hi_at, void* lo_at) {
  uint32_t hi[4], lo[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) split_bf16x2(v[2 * e], v[2 * e + 1], hi[e], lo[e]);
  *reinterpret_cast<uint4*>(hi_at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
  *reinterpret_cast<uint4*>(lo_at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
}
__device__ __forceinline__ void delta_load8(const float* p, float* v) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
__device__ __forceinline__ void delta_load4(const __nv_bfloat16* p, float* v) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
}

// 2^x, 0 where that is no normal number
__device__ __forceinline__ float delta_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ----------------------------------------------------------------------------- chunks by themselves
constexpr int DP_THREADS = 512, DP_WARPS = DP_THREADS / 32, DP_TAPS = 4, DP_RAW = DC + DP_TAPS - 1;
constexpr float DP_FLOOR = -72.f;  // 2^ of it is far below the rounding of anything it is added to
constexpr float DP_RANGE = -60.f;  // what a block on the diagonal may lose

struct DeltaPrepSmem {
  int k, q, g, kt, tp, l, t, misc, total;  // byte offsets
};
__host__ __device__ inline DeltaPrepSmem delta_prep_smem(int K, int V) {
  DeltaPrepSmem s;
  const int f32 = DC * (K + 8) * 4, vhalves = 2 * DC * (V * 2 + 16), rawv = DP_RAW * V * 2, tp = 2 * DC * DC_PROW;
  s.k = 0;
  s.q = s.k + f32;
  s.g = s.q + f32;                               // decays; later v as halves
  s.kt = s.g + (f32 > vhalves ? f32 : vhalves);  // raw rows of q and k; later exp(G) k as halves
  s.tp = s.kt + f32;                             // raw rows of v; later the inverse times beta as halves
  s.l = s.tp + ((tp > rawv ? tp : rawv) + 15) / 16 * 16;
  s.t = s.l + DC * DC_LD * 4;
  s.misc = s.t + DC * DC_LD * 4;
  s.total = s.misc + (DC + 4 * K + 8) * 4;       // beta | totals of blocks | flags of blocks
  return s;
}

// (The kernels of this file run most of their code once per warp, and instructions that are run once come no faster than they are
// fetched: loops stay rolled wherever registers allow it.)

// Taps of this lane's four channels, zeros on the oldest rows of shorter convolutions.
__device__ __forceinline__ void delta_taps4(const DeltaArgs& a, int C, int ch, float4 (&w)[DP_TAPS]) {
#pragma unroll
  for (int i = 0; i < DP_TAPS; ++i) {
    const int tap = i - (DP_TAPS - a.taps);
    w[i] = (tap >= 0 && a.taps <= DP_TAPS) ? *reinterpret_cast<const float4*>(a.conv + (size_t)tap * C + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
}
// Those channels of token t of the chunk after convolution and silu, out of raw rows in shared memory (`raw`: three tokens ahead
// of the chunk, rows `row` values apart; zeros past the portion), or, for longer convolutions, out of global memory.
__device__ __forceinline__ void delta_conv4(const DeltaArgs& a, const float4 (&w)[DP_TAPS], const __nv_bfloat16* raw, int row,
                                            const __nv_bfloat16* z, const float* ring, int C, int pos0, int c0, int t, int n, int ch,
                                            float* y) {
  if (a.taps <= DP_TAPS) {
    y[0] = y[1] = y[2] = y[3] = 0.f;
#pragma unroll
    for (int i = 0; i < DP_TAPS; ++i) {
      float x[4];
      delta_load4(raw + (t + i) * row, x);
      y[0] = fmaf(w[i].x, x[0], y[0]);
      y[1] = fmaf(w[i].y, x[1], y[1]);
      y[2] = fmaf(w[i].z, x[2], y[2]);
      y[3] = fmaf(w[i].w, x[3], y[3]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] *= delta_sigmoid_fast(y[e]);
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = t < n ? delta_conv(a, z, ring, C, pos0, c0 + t, ch + e) : 0.f;
  }
}

// Products of a low-rank projection: 16 rows (this lane's two: r0, r1) by nt <= NT tiles of 8 columns (`up`: this lane's row of
// the first).  Which values of a k-step a lane holds is free, as long as both operands agree: four neighbouring ones.
template <int NT, int STEPS>
__device__ __forceinline__ void delta_low_rank_steps(const __nv_bfloat16* r0, const __nv_bfloat16* r1, const __nv_bfloat16* up, int rank,
                                                     int nt, float (&acc)[NT][4]) {
  uint2 x0[STEPS], x1[STEPS], w[STEPS][NT];
#pragma unroll
  for (int j = 0; j < STEPS; ++j) {
    x0[j] = *reinterpret_cast<const uint2*>(r0 + 16 * j);
    x1[j] = *reinterpret_cast<const uint2*>(r1 + 16 * j);
#pragma unroll
    for (int i = 0; i < NT; ++i) w[j][i] = i < nt ? *reinterpret_cast<const uint2*>(up + (size_t)i * 8 * rank + 16 * j) : make_uint2(0, 0);
  }
#pragma unroll
  for (int j = 0; j < STEPS; ++j) {
    const uint32_t av[4] = {x0[j].x, x1[j].x, x0[j].y, x1[j].y};
#pragma unroll
    for (int i = 0; i < NT; ++i) mma_bf16_16816(acc[i], av, w[j][i].x, w[j][i].y);
  }
}
template <int NT>
__device__ __forceinline__ void delta_low_rank(const __nv_bfloat16* r0, const __nv_bfloat16* r1, const __nv_bfloat16* up, int rank, int nt,
                                               float (&acc)[NT][4]) {
  int ks = 0;
  for (; ks + 64 <= rank; ks += 64) delta_low_rank_steps<NT, 4>(r0 + ks, r1 + ks, up + ks, rank, nt, acc);
  for (; ks < rank; ks += 16) delta_low_rank_steps<NT, 1>(r0 + ks, r1 + ks, up + ks, rank, nt, acc);
}

// grid (chunks of the round, H, B); CH: a decay per key channel.
template <int KT, bool CH>
__global__ void __launch_bounds__(DP_THREADS, 1) delta_prepare_kernel(const DeltaChunkArgs x) {
  constexpr int K = KT * 16, KF = K + 8, K8 = K / 8, CPL = K / 32;
  constexpr int RB = K * 2 + 16, HALF = DC * RB;  // bytes of a row of halves, of 64 rows
  extern __shared__ __align__(16) uint8_t dp_smem[];
  pdl_launch_dependents();
  const DeltaArgs& a = x.a;
  const int b = blockIdx.z, h = blockIdx.y, chunk = x.chunk0 + blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int q0 = a.query_start[b], n_all = a.query_start[b + 1] - q0, slot = a.slots[b], c0 = chunk * DC;
  if (n_all < a.min_rows || n_all > a.max_rows || c0 >= n_all || (unsigned)slot >= (unsigned)a.num_slots) {
    pdl_wait();
    return;
  }
  const int n = min(DC, n_all - c0), V = a.V, V8 = V / 8, C = 2 * a.G * K + a.H * V, kvh = h / (a.H / a.G);
  const int pos0 = a.seq_lens[b] - n_all;
  const DeltaPlan pl = delta_plan(K, V);
  const DeltaPrepSmem sm = delta_prep_smem(K, V);
  uint8_t* block = delta_block(x, pl.bytes, b, chunk, h);
  float *sK = reinterpret_cast<float*>(dp_smem + sm.k), *sQ = reinterpret_cast<float*>(dp_smem + sm.q);
  float* sG = reinterpret_cast<float*>(dp_smem + sm.g);  // [64][KF], or [64] with one decay per head: sums within blocks of 16
  float *sL = reinterpret_cast<float*>(dp_smem + sm.l), *sT = reinterpret_cast<float*>(dp_smem + sm.t);
  float *beta = reinterpret_cast<float*>(dp_smem + sm.misc), *total = beta + DC;  // total: [4][K], or [4]
  int* wild = reinterpret_cast<int*>(total + 4 * K);                              // [4] blocks whose decays leave the range
  __nv_bfloat16 *raw_qk = reinterpret_cast<__nv_bfloat16*>(dp_smem + sm.kt), *raw_v = reinterpret_cast<__nv_bfloat16*>(dp_smem + sm.tp);
  const int RV = V * 2 + 16, VHALF = DC * RV;
  const float* ring = a.window + (size_t)slot * a.taps * C;
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)q0 * a.ld;
  if (tid < 4) wild[tid] = 0;
  pdl_wait();
  // ---- raw rows of q | k and of v, from three tokens ahead of the chunk on
  if (a.taps <= DP_TAPS) {
    const __nv_bfloat16 *zq = z + kvh * K, *zv = z + 2 * a.G * K + h * V;
#pragma unroll 1
    for (int r = warp; r < DP_RAW; r += DP_WARPS) {
      const int j = c0 - (DP_TAPS - 1) + r;
      const bool now = j >= 0 && j < n_all, past = j < 0 && pos0 + j >= 0 && j > -a.taps;
      const float* old = ring + (past ? (size_t)((pos0 + j) % a.taps) * C : 0);
#pragma unroll 1
      for (int p = lane; p < 2 * K8 + V8; p += 32) {
        const bool is_v = p >= 2 * K8;
        const int off = is_v ? (p - 2 * K8) * 8 : (p < K8 ? p * 8 : a.G * K + (p - K8) * 8);
        __nv_bfloat16* dst = is_v ? raw_v + r * V + off : raw_qk + (r * 2 * K8 + p) * 8;
        if (now) {
          cp_async16(dst, (is_v ? zv : zq) + (size_t)j * a.ld + off);
        } else if (past) {  // (an earlier step's projections: 16-bit values)
          float v[8];
          delta_load8(old + (is_v ? 2 * a.G * K + h * V : kvh * K) + off, v);
          *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
        } else {
          *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
      }
    }
  }
  cp_async_commit();
  // ---- decays and step sizes
  if (tid < DC) beta[tid] = tid < n ? delta_sigmoid(lat_f32(z[(size_t)(c0 + tid) * a.ld + a.beta_off + h])) : 0.f;
  const float rate = expf(a.a_log[h]) * 1.4426950408889634f;
  if (CH) {  // 16 tokens x K / 4 channels per warp
    const int mt = warp & 3, d0 = (warp >> 2) * (K / 4);
    float acc[K / 32][4];
#pragma unroll
    for (int i = 0; i < K / 32; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const __nv_bfloat16* rows = z + (size_t)c0 * a.ld + a.decay_off + 4 * t4;
    delta_low_rank<K / 32>(rows + (size_t)min(mt * 16 + g, n - 1) * a.ld, rows + (size_t)min(mt * 16 + g + 8, n - 1) * a.ld,
                           reinterpret_cast<const __nv_bfloat16*>(a.decay_up) + (size_t)(h * K + d0 + g) * a.decay_rank + 4 * t4, a.decay_rank,
                           K / 32, acc);
#pragma unroll
    for (int i = 0; i < K / 32; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2)
        *reinterpret_cast<float2*>(sG + (mt * 16 + g + 8 * (e >> 1)) * KF + d0 + i * 8 + 2 * t4) = make_float2(acc[i][e], acc[i][e + 1]);
  } else if (warp == 0) {
    float v[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 2 * lane + i;
      v[i] = t < n ? fmaxf(-rate * delta_softplus(lat_f32(z[(size_t)(c0 + t) * a.ld + a.decay_off + h]) + a.dt_bias[h]), DP_FLOOR) : 0.f;
    }
    v[1] += v[0];
    float s = v[1];
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) {  // (eight lanes have a block)
      const float y = __shfl_up_sync(0xffffffffu, s, o);
      if ((lane & 7) >= o) s += y;
    }
    const float before = __shfl_up_sync(0xffffffffu, s, 1);
    sG[2 * lane] = ((lane & 7) ? before : 0.f) + v[0];
    sG[2 * lane + 1] = s;
    if ((lane & 7) == 7) total[lane >> 3] = s;
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- q and k: convolution, silu, unit vectors; a warp has four tokens, a lane four channels
#pragma unroll 1
  for (int side = 0; side < 2; ++side) {
    const int d = lane * 4, dc = min(d, K - 4), ch = (side ? a.G + kvh : kvh) * K + dc;
    float* dst = (side ? sK : sQ) + d;
    float4 w[DP_TAPS];
    delta_taps4(a, C, ch, w);
#pragma unroll 2
    for (int t = warp * 4; t < warp * 4 + 4; ++t) {
      float y[4];
      delta_conv4(a, w, raw_qk + side * K + dc, 2 * K, z, ring, C, pos0, c0, t, n, ch, y);
      const float ss = d < K ? (y[0] * y[0] + y[1] * y[1]) + (y[2] * y[2] + y[3] * y[3]) : 0.f;
      const float f = t < n ? rsqrtf(warp_sum(ss) + 1e-6f) * (side ? 1.f : a.q_scale) : 0.f;
      if (d < K) *reinterpret_cast<float4*>(dst + t * KF) = make_float4(y[0] * f, y[1] * f, y[2] * f, y[3] * f);
    }
  }
  if (CH) {  // running sums (512 threads: four blocks of up to 128 channels)
    const int d = tid % K, blk = tid / K;
    if (blk < 4) {
      const float dt = a.dt_bias[h * K + d];
      float sum = 0.f;
#pragma unroll 2
      for (int t = blk * 16; t < blk * 16 + 16; ++t) {
        const float v = fmaxf(-rate * delta_softplus(sG[t * KF + d] + dt), DP_FLOOR);
        sum += t < n ? v : 0.f;
        sG[t * KF + d] = sum;
      }
      total[blk * K + d] = sum;
      if (sum < DP_RANGE) wild[blk] = 1;
    }
  }
  __syncthreads();
  // logarithm of the decay behind token t through the end of block `block1` - 1, channels d and d + 1
  auto until2 = [&](int t, int block1, int d) {
    float2 v, w;
    const int blk = t >> 4;
    if (CH) {
      v = *reinterpret_cast<const float2*>(total + blk * K + d);
      w = *reinterpret_cast<const float2*>(sG + t * KF + d);
    } else {
      v.x = v.y = total[blk];
      w.x = w.y = sG[t];
    }
    v.x -= w.x;
    v.y -= w.y;
    for (int i = blk + 1; i < block1; ++i) {
      v.x += total[CH ? i * K + d : i];
      v.y += total[CH ? i * K + d + 1 : i];
    }
    return v;
  };
  constexpr int PR = DC_PROW / 2;
  __nv_bfloat16 *p_hi = reinterpret_cast<__nv_bfloat16*>(block + pl.p), *p_lo = p_hi + DC * PR;
  if (warp < 10) {
    // ---- L and P, blocks of 16 x 16, operands from the float32 rows
    const int mt = warp < 1 ? 0 : (warp < 3 ? 1 : (warp < 6 ? 2 : 3)), np = warp - mt * (mt + 1) / 2;
    const bool diag = mt == np;
    if (!(CH && diag && wild[mt])) {
      float accK[2][4], accQ[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) accK[i][0] = accK[i][1] = accK[i][2] = accK[i][3] = accQ[i][0] = accQ[i][1] = accQ[i][2] = accQ[i][3] = 0.f;
#pragma unroll 1
      for (int ks = 0; ks < KT; ++ks) {
        uint32_t kh[4], kl[4], qh[4], ql[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {  // (row g + 8 (j & 1), values 2 t4 + 8 (j >> 1))
          const int t = mt * 16 + g + 8 * (j & 1), d = ks * 16 + 2 * t4 + 8 * (j >> 1);
          float2 kv = *reinterpret_cast<const float2*>(sK + t * KF + d), qv = *reinterpret_cast<const float2*>(sQ + t * KF + d);
          if (CH) {
            const float2 l = *reinterpret_cast<const float2*>(sG + t * KF + d);
            const float fx = delta_exp2(l.x), fy = delta_exp2(l.y);
            kv = make_float2(kv.x * fx, kv.y * fy);
            qv = make_float2(qv.x * fx, qv.y * fy);
          }
          split_bf16x2(kv.x, kv.y, kh[j], kl[j]);
          split_bf16x2(qv.x, qv.y, qh[j], ql[j]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int j = 0; j < 2; ++j) {  // (column g of tile i, values 2 t4 + 8 j)
            const int s = np * 16 + 8 * i + g, d = ks * 16 + 2 * t4 + 8 * j;
            float2 kv = *reinterpret_cast<const float2*>(sK + s * KF + d);
            if (CH) {
              float2 l;
              if (diag) {
                l = *reinterpret_cast<const float2*>(sG + s * KF + d);
                l = make_float2(-l.x, -l.y);
              } else {
                l = until2(s, mt, d);
              }
              kv = make_float2(kv.x * delta_exp2(l.x), kv.y * delta_exp2(l.y));
            }
            split_bf16x2(kv.x, kv.y, bh[j], bl[j]);
          }
          mma_bf16_16816(accK[i], kh, bh[0], bh[1]);
          mma_bf16_16816(accQ[i], qh, bh[0], bh[1]);
          mma_bf16_16816(accK[i], kh, bl[0], bl[1]);
          mma_bf16_16816(accQ[i], qh, bl[0], bl[1]);
          mma_bf16_16816(accK[i], kl, bh[0], bh[1]);
          mma_bf16_16816(accQ[i], ql, bh[0], bh[1]);
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int t = mt * 16 + g + 8 * (e >> 1), s = np * 16 + 8 * i + 2 * t4;
          float f0 = 1.f, f1 = 1.f;
          if (!CH) {
            if (diag) {
              f0 = delta_exp2(fminf(sG[t] - sG[s], 0.f));  // (positive only where the triangle is cut off)
              f1 = delta_exp2(fminf(sG[t] - sG[s + 1], 0.f));
            } else {
              f0 = delta_exp2(sG[t] + until2(s, mt, 0).x);
              f1 = delta_exp2(sG[t] + until2(s + 1, mt, 0).x);
            }
          }
          const bool on0 = !diag || s <= t, on1 = !diag || s + 1 <= t;
          uint32_t hi, lo;
          split_bf16x2(on0 ? accQ[i][e] * f0 : 0.f, on1 ? accQ[i][e + 1] * f1 : 0.f, hi, lo);
          *reinterpret_cast<uint32_t*>(p_hi + t * PR + s) = hi;
          *reinterpret_cast<uint32_t*>(p_lo + t * PR + s) = lo;
          *reinterpret_cast<float2*>(sL + t * DC_LD + s) = make_float2(on0 ? accK[i][e] * f0 * beta[t] : 0.f, on1 ? accK[i][e + 1] * f1 * beta[t] : 0.f);
        }
    }
  } else {
    // ---- meanwhile: exp(G) k for this kernel, exp(G) q and exp(G_end - G) k for the others
#pragma unroll 1
    for (int i = tid - 320; i < DC * K8; i += DP_THREADS - 320) {
      const int t = i / K8, p = i % K8;
      float kv[8], qv[8], f[8], r[8], y[8], l[8];
      delta_load8(sK + t * KF + p * 8, kv);
      delta_load8(sQ + t * KF + p * 8, qv);
      const int blk = t >> 4;
      if (CH) {
        delta_load8(sG + t * KF + p * 8, l);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          f[e] = l[e];
          r[e] = -l[e];
        }
#pragma unroll
        for (int i = 0; i < DC / 16; ++i) {
          delta_load8(total + i * K + p * 8, l);
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            if (i < blk) f[e] += l[e];
            else r[e] += l[e];
          }
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          f[e] = delta_exp2(f[e]);
          r[e] = delta_exp2(r[e]);
        }
      } else {
        float u = sG[t], w = -u;
#pragma unroll
        for (int i = 0; i < DC / 16; ++i) {
          if (i < blk) u += total[i];
          else w += total[i];
        }
        u = delta_exp2(u);
        w = delta_exp2(w);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = u, r[e] = w;
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = kv[e] * f[e];
      uint8_t* at = dp_smem + sm.kt + t * RB + p * 16;
      delta_split8(y, at, at + HALF);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = qv[e] * f[e];
      at = block + pl.qt + t * RB + p * 16;
      delta_split8(y, at, at + HALF);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = kv[e] * r[e];
      at = block + pl.kb + t * RB + p * 16;
      delta_split8(y, at, at + HALF);
    }
    for (int d = tid - 320; d < K; d += DP_THREADS - 320) {
      float s = 0.f;
      for (int i = 0; i < DC / 16; ++i) s += total[CH ? i * K + d : i];
      reinterpret_cast<float*>(block + pl.gend)[d] = delta_exp2(s);
    }
  }
  if (CH && wild[warp >> 2]) {  // a block on the diagonal column by column: a warp has four columns, a lane CPL channels
    const int t0 = (warp >> 2) * 16, s0 = t0 + (warp & 3) * 4;
    float w[4][CPL];
#pragma unroll
    for (int s = 0; s < 4; ++s)
#pragma unroll
      for (int i = 0; i < CPL; ++i) w[s][i] = 0.f;
#pragma unroll 1
    for (int t = t0; t < t0 + 16; ++t) {
      float sum[8];  // k . w, q . w of the four columns
#pragma unroll
      for (int s = 0; s < 8; ++s) sum[s] = 0.f;
      if (t >= s0) {
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
          const int d = lane + 32 * i;
          const float kt = sK[t * KF + d], qt = sQ[t * KF + d];
          const float f = t > s0 ? delta_exp2(sG[t * KF + d] - sG[(t - 1) * KF + d]) : 0.f;
#pragma unroll
          for (int s = 0; s < 4; ++s) {
            w[s][i] = t == s0 + s ? kt : w[s][i] * f;  // (zero ahead of its own token)
            sum[s] = fmaf(kt, w[s][i], sum[s]);
            sum[4 + s] = fmaf(qt, w[s][i], sum[4 + s]);
          }
        }
      }
      // every lane's eight sums to eight totals, total l >> 2 in lane l
#pragma unroll
      for (int m = 16, c = 4; m >= 4; m >>= 1, c >>= 1) {
        const bool up = lane & m;
#pragma unroll
        for (int i = 0; i < c; ++i) {
          const float keep = up ? sum[c + i] : sum[i], send = up ? sum[i] : sum[c + i];
          sum[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
        }
      }
      sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], 2);
      sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], 1);
      const int s = s0 + (lane >> 2 & 3);
      if ((lane & 3) == 0) {
        if (lane < 16) {
          sL[t * DC_LD + s] = s < t ? sum[0] * beta[t] : 0.f;
        } else {
          const float v = s <= t ? sum[0] : 0.f;
          const __nv_bfloat16 hi = __float2bfloat16(v);
          p_hi[t * PR + s] = hi;
          p_lo[t * PR + s] = __float2bfloat16(v - __bfloat162float(hi));
        }
      }
    }
  }
  __syncthreads();
  // ---- the inverse of I + L: blocks of 16 on the diagonal by substitution, the others from them
  if (warp < 2) {
    const int t0 = tid & ~15, c = tid & 15;
    float *col = sT + t0 * DC_LD + t0 + c, *rows = sL + t0 * DC_LD + t0;
#pragma unroll
    for (int r = 0; r < 16; ++r) col[r * DC_LD] = r == c ? 1.f : 0.f;
#pragma unroll 1
    for (int r = 1; r < 16; ++r) {  // (rows at and past r are zero, but for the one on the diagonal)
      float s[4];
#pragma unroll
      for (int i = 0; i < 16; i += 4) {
        const float4 l = *reinterpret_cast<const float4*>(rows + r * DC_LD + i);
        s[i >> 2] = (l.x * col[i * DC_LD] + l.y * col[(i + 1) * DC_LD]) + (l.z * col[(i + 2) * DC_LD] + l.w * col[(i + 3) * DC_LD]);
      }
      if (r > c) col[r * DC_LD] = -((s[0] + s[1]) + (s[2] + s[3]));
    }
  } else {  // (meanwhile) v: convolution and silu, as halves where the decays were
    const int d = lane * 4, dc = min(d, V - 4), ch = 2 * a.G * K + h * V + dc;
    float4 w[DP_TAPS];
    delta_taps4(a, C, ch, w);
#pragma unroll 1
    for (int t = warp - 2; t < DC; t += DP_WARPS - 2) {
      float y[4];
      delta_conv4(a, w, raw_v + dc, V, z, ring, C, pos0, c0, t, n, ch, y);
      if (d >= V) continue;
      uint32_t h0, l0, h1, l1;
      split_bf16x2(t < n ? y[0] : 0.f, t < n ? y[1] : 0.f, h0, l0);
      split_bf16x2(t < n ? y[2] : 0.f, t < n ? y[3] : 0.f, h1, l1);
      uint8_t* at = dp_smem + sm.g + t * RV + d * 2;
      *reinterpret_cast<uint2*>(at) = make_uint2(h0, h1);
      *reinterpret_cast<uint2*>(at + VHALF) = make_uint2(l0, l1);
    }
  }
  __syncthreads();
#pragma unroll 1
  for (int dist = 1; dist < 4; ++dist) {
    // block (i, i - dist): first sum_k L_ik T_kj into the (unused) mirror block above the diagonal, then - T_ii times that
#pragma unroll 1
    for (int step = 0; step < 2; ++step) {
#pragma unroll 1
      for (int u = tid; u < (4 - dist) * 256; u += DP_THREADS) {
        const int j = u >> 8, i = j + dist, r = u >> 4 & 15, c = u & 15;
        const float* x = step ? sT + (i * 16 + r) * DC_LD + i * 16 : sL + (i * 16 + r) * DC_LD + j * 16;
        const float* y = step ? sL + j * 16 * DC_LD + i * 16 + c : sT + j * 16 * DC_LD + j * 16 + c;
        float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
        for (int m = 0; m < (step ? 1 : dist); ++m, x += 16, y += 16 * DC_LD) {
#pragma unroll
          for (int k = 0; k < 16; k += 4) {
            const float4 v = *reinterpret_cast<const float4*>(x + k);
            s[0] = fmaf(v.x, y[k * DC_LD], s[0]);
            s[1] = fmaf(v.y, y[(k + 1) * DC_LD], s[1]);
            s[2] = fmaf(v.z, y[(k + 2) * DC_LD], s[2]);
            s[3] = fmaf(v.w, y[(k + 3) * DC_LD], s[3]);
          }
        }
        const float sum = (s[0] + s[1]) + (s[2] + s[3]);
        if (step) sT[(i * 16 + r) * DC_LD + j * 16 + c] = -sum;
        else sL[(j * 16 + r) * DC_LD + i * 16 + c] = sum;
      }
      __syncthreads();
    }
  }
  {  // times beta, as halves: 64 rows of eight pieces
    const int t = tid >> 3, p = tid & 7;
    if (p * 8 <= (t | 15)) {
      float v[8];
      delta_load8(sT + t * DC_LD + p * 8, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= beta[p * 8 + e];
      uint8_t* at = dp_smem + sm.tp + t * DC_PROW + p * 16;
      delta_split8(v, at, at + DC * DC_PROW);
    }
  }
  __syncthreads();
  // ---- W = T exp(G) k and U0 = T v (T: the inverse times beta), all 64 tokens of 16 columns per warp
  {
    const int mi = lane >> 3, r8 = lane & 7, nk = K / 16, nv = V / 16;
    const uint32_t A = smem_u32(dp_smem + sm.tp) + ((mi & 1) * 8 + r8) * DC_PROW + (mi >> 1) * 16;
    for (int u = warp; u < nk + nv; u += DP_WARPS) {
      const bool is_w = u < nk;
      const int rb = is_w ? RB : RV, col = is_w ? u : u - nk;
      const uint32_t Bm = smem_u32(dp_smem + (is_w ? sm.kt : sm.g)) + ((mi & 1) * 8 + r8) * rb + (mi >> 1) * 16 + col * 32;
      float acc[4][2][4];
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int i = 0; i < 2; ++i) acc[mt][i][0] = acc[mt][i][1] = acc[mt][i][2] = acc[mt][i][3] = 0.f;
#pragma unroll 1
      for (int ks = 0; ks < 4; ++ks) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(Bm + ks * 16 * rb, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(Bm + DC * rb + ks * 16 * rb, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
          if (mt < ks) continue;  // (the same for all)
          uint32_t ah[4], al[4];
          ldmatrix_x4(A + mt * 16 * DC_PROW + ks * 32, ah[0], ah[1], ah[2], ah[3]);
          ldmatrix_x4(A + (DC + mt * 16) * DC_PROW + ks * 32, al[0], al[1], al[2], al[3]);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16_16816(acc[mt][i], ah, bh[2 * i], bh[2 * i + 1]);
            mma_bf16_16816(acc[mt][i], ah, bl[2 * i], bl[2 * i + 1]);
            mma_bf16_16816(acc[mt][i], al, bh[2 * i], bh[2 * i + 1]);
          }
        }
      }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int e = 0; e < 4; e += 2) {
            const int t = mt * 16 + g + 8 * (e >> 1), c = col * 16 + 8 * i + 2 * t4;
            if (is_w) {
              uint32_t hi, lo;
              split_bf16x2(acc[mt][i][e], acc[mt][i][e + 1], hi, lo);
              uint8_t* at = block + pl.w + t * RB + c * 2;
              *reinterpret_cast<uint32_t*>(at) = hi;
              *reinterpret_cast<uint32_t*>(at + HALF) = lo;
            } else {
              *reinterpret_cast<float2*>(block + pl.u0 + col * DC_USLICE + t * 80 + (8 * i + 2 * t4) * 4) = make_float2(acc[mt][i][e], acc[mt][i][e + 1]);
            }
          }
    }
  }
}

// ----------------------------------------------------------------------------- the state, chunk after chunk
constexpr int DS_THREADS = 512;
__host__ __device__ inline int delta_state_stage(int K, int NV) { return 4 * DC * (K * 2 + 16) + NV / 16 * DC_USLICE + K * 4; }
__host__ __device__ inline int delta_state_smem(int K, int NV) {
  return 2 * delta_state_stage(K, NV) + 2 * K * (NV * 2 + 16) + 2 * DC * (NV * 2 + 16);
}

// grid (V / NV, H, B): a CTA has NV values of one head's state; warp w has rows 16 (w % KT) .. and values 16 (w / KT) .. of it in
// accumulator registers, and a tile of U of 16 tokens x 8 values.
template <int KT, int NV>
__global__ void __launch_bounds__(DS_THREADS, 1) delta_state_kernel(const DeltaChunkArgs x) {
  constexpr int K = KT * 16, RB = K * 2 + 16, RN = NV * 2 + 16, US = NV / 16 * DC_USLICE;
  extern __shared__ __align__(16) uint8_t dt_smem[];
  __shared__ uint64_t full[2];
  __shared__ volatile int abort_flag;
  pdl_launch_dependents();
  const DeltaArgs& a = x.a;
  const int v0 = blockIdx.x * NV, h = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const int q0 = a.query_start[b], n = a.query_start[b + 1] - q0, slot = a.slots[b];
  const int V = a.V, chunk1 = min((n + DC - 1) / DC, x.chunk0 + x.round);
  pdl_wait();
  if (n < a.min_rows || n > a.max_rows || x.chunk0 >= chunk1 || (unsigned)slot >= (unsigned)a.num_slots) return;
  const DeltaPlan pl = delta_plan(K, V);
  const int stage_bytes = delta_state_stage(K, NV);
  uint8_t* sS = dt_smem + 2 * stage_bytes;  // [hi, lo][K][RN]
  uint8_t* sU = sS + 2 * K * RN;            // [hi, lo][64][RN]
  const int RV = V * 2 + 16;
  if (tid == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  auto fetch = [&](int c) {  // one thread: W, Kb [hi, lo][64][RB] | U0, slices of 16 values | gend [K]
    const uint8_t* block = delta_block(x, pl.bytes, b, c, h);
    const int i = (c - x.chunk0) & 1;
    uint8_t* dst = dt_smem + i * stage_bytes;
    mbar_expect_tx(&full[i], stage_bytes);
    bulk_load(dst, block, 4 * DC * RB, &full[i]);
    bulk_load(dst + 4 * DC * RB, block + pl.u0 + v0 / 16 * DC_USLICE, US, &full[i]);
    bulk_load(dst + 4 * DC * RB + US, block + pl.gend, K * 4, &full[i]);
  };
  if (tid == 0) fetch(x.chunk0);
  const int srow = warp % KT, scol = warp / KT;
  const bool owner = scol < NV / 16;  // this warp has a part of the state
  const bool resumed = a.seq_lens[b] > n || x.chunk0 > 0;
  float S[2][4];
  float* st = a.state + ((size_t)slot * a.H + h) * K * V + (size_t)(srow * 16 + g) * V + v0 + scol * 16 + 2 * t4;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const float2 y = (owner && resumed) ? __ldcg(reinterpret_cast<const float2*>(st + (size_t)(e >> 1) * 8 * V + 8 * i)) : make_float2(0.f, 0.f);
      S[i][e] = y.x;
      S[i][e + 1] = y.y;
    }
  auto put_state = [&](uint8_t* block) {  // halves: for the next products, and for the outputs
    if (!owner) return;
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        uint32_t hi, lo;
        split_bf16x2(S[i][e], S[i][e + 1], hi, lo);
        const int k = srow * 16 + g + 8 * (e >> 1), c = scol * 16 + 8 * i + 2 * t4;
        *reinterpret_cast<uint32_t*>(sS + k * RN + c * 2) = hi;
        *reinterpret_cast<uint32_t*>(sS + K * RN + k * RN + c * 2) = lo;
        uint8_t* at = block + pl.s + k * RV + (v0 + c) * 2;
        *reinterpret_cast<uint32_t*>(at) = hi;
        *reinterpret_cast<uint32_t*>(at + K * RV) = lo;
      }
  };
  const uint32_t base = smem_u32(dt_smem), s_u = smem_u32(sS), u_u = smem_u32(sU);
  const int mt = warp & 3, un = (warp >> 2) * 8;  // this warp's tile of U
  const bool has_u = un < NV;
  const uint32_t wa = (mt * 16 + (mi & 1) * 8 + r8) * RB + (mi >> 1) * 16;
  const uint32_t sb = lane * RN + un * 2;                                      // transposed: 32 keys x 8 values
  const uint32_t ka = ((mi >> 1) * 8 + r8) * RB + srow * 32 + (mi & 1) * 16;   // transposed: 16 keys x 16 tokens
  const uint32_t ub = ((mi & 1) * 8 + r8) * RN + scol * 32 + (mi >> 1) * 16;
  for (int c = x.chunk0; c < chunk1; ++c) {
    uint8_t* block = delta_block(x, pl.bytes, b, c, h);
    put_state(block);
    __syncthreads();  // the state is in shared memory; the other buffer has been read
    if (tid == 0 && c + 1 < chunk1) fetch(c + 1);
    const int step = c - x.chunk0, stage = (step & 1) * stage_bytes;
    mbar_wait_bounded(&full[step & 1], step >> 1 & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
    __syncwarp();
    const uint32_t W = base + stage, Kb = W + 2 * DC * RB;
    const uint8_t* extra = dt_smem + stage + 4 * DC * RB;
    if (has_u) {
      float acc[3][4];
#pragma unroll
      for (int j = 0; j < 3; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KT; ks += 2) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(s_u + sb + ks * 16 * RN, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(s_u + K * RN + sb + ks * 16 * RN, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          uint32_t ah[4], al[4];
          ldmatrix_x4(W + wa + (ks + j) * 32, ah[0], ah[1], ah[2], ah[3]);
          ldmatrix_x4(W + DC * RB + wa + (ks + j) * 32, al[0], al[1], al[2], al[3]);
          mma_bf16_16816(acc[0], ah, bh[2 * j], bh[2 * j + 1]);
          mma_bf16_16816(acc[1], ah, bl[2 * j], bl[2 * j + 1]);
          mma_bf16_16816(acc[2], al, bh[2 * j], bh[2 * j + 1]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int t = mt * 16 + g + 8 * (e >> 1), cc = un + 2 * t4;
        const float2 u0 = *reinterpret_cast<const float2*>(extra + (cc >> 4) * DC_USLICE + t * 80 + (cc & 15) * 4);
        uint32_t hi, lo;
        split_bf16x2(u0.x - (acc[0][e] + (acc[1][e] + acc[2][e])), u0.y - (acc[0][e + 1] + (acc[1][e + 1] + acc[2][e + 1])), hi, lo);
        *reinterpret_cast<uint32_t*>(sU + t * RN + cc * 2) = hi;
        *reinterpret_cast<uint32_t*>(sU + DC * RN + t * RN + cc * 2) = lo;
        uint8_t* at = block + pl.u + t * RV + (v0 + cc) * 2;
        *reinterpret_cast<uint32_t*>(at) = hi;
        *reinterpret_cast<uint32_t*>(at + DC * RV) = lo;
      }
    }
    __syncthreads();  // U is complete; the state's halves have been read
    if (owner) {
      const float* ge = reinterpret_cast<const float*>(extra + US) + srow * 16 + g;
      float acc[2][2][4];  // (the low halves' products in accumulators of their own)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        S[i][0] *= ge[0];
        S[i][1] *= ge[0];
        S[i][2] *= ge[8];
        S[i][3] *= ge[8];
#pragma unroll
        for (int j = 0; j < 2; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
      }
#pragma unroll
      for (int ks = 0; ks < DC / 16; ++ks) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        ldmatrix_x4_trans(Kb + ka + ks * 16 * RB, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4_trans(Kb + DC * RB + ka + ks * 16 * RB, al[0], al[1], al[2], al[3]);
        ldmatrix_x4_trans(u_u + ub + ks * 16 * RN, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(u_u + DC * RN + ub + ks * 16 * RN, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma_bf16_16816(S[i], ah, bh[2 * i], bh[2 * i + 1]);
          mma_bf16_16816(acc[i][0], ah, bl[2 * i], bl[2 * i + 1]);
          mma_bf16_16816(acc[i][1], al, bh[2 * i], bh[2 * i + 1]);
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][e] += acc[i][0][e] + acc[i][1][e];
    }
  }
  if (owner) {
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) *reinterpret_cast<float2*>(st + (size_t)(e >> 1) * 8 * V + 8 * i) = make_float2(S[i][e], S[i][e + 1]);
  }
  if (abort_flag) {
    // a wait gave up: give copies that may still be in flight time to land before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
}

// ----------------------------------------------------------------------------- outputs
constexpr int DO_THREADS = 512;
__host__ __device__ inline int delta_output_smem(int K, int V) {
  return 2 * DC * (K * 2 + 16) + 2 * K * (V * 2 + 16) + 2 * DC * DC_PROW + 2 * DC * (V * 2 + 16) + 4 * DC * 4;
}

// grid (chunks of the round, H, B); warp w: tokens 16 (w % 4) .., values 32 (w / 4) ..
template <int KT>
__global__ void __launch_bounds__(DO_THREADS, 1) delta_output_kernel(const DeltaChunkArgs x) {
  constexpr int K = KT * 16, RB = K * 2 + 16;
  extern __shared__ __align__(16) uint8_t do_smem[];
  __shared__ uint64_t full[2];
  __shared__ volatile int abort_flag;
  pdl_launch_dependents();
  const DeltaArgs& a = x.a;
  const int b = blockIdx.z, h = blockIdx.y, chunk = x.chunk0 + blockIdx.x, c0 = chunk * DC;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const int q0 = a.query_start[b], n_all = a.query_start[b + 1] - q0, slot = a.slots[b];
  const int V = a.V, RV = V * 2 + 16;
  pdl_wait();
  if (n_all < a.min_rows || n_all > a.max_rows || c0 >= n_all) return;
  const int n = min(DC, n_all - c0);
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(q0 + c0) * a.ld_out + (size_t)h * V;
  if ((unsigned)slot >= (unsigned)a.num_slots) {
    if (slot >= 0 && tid == 0) oxb_report(OXB_BAD_SLOT, slot);
    for (int i = tid; i < n * V; i += DO_THREADS) out[(size_t)(i / V) * a.ld_out + i % V] = __float2bfloat16(0.f);
    return;
  }
  const DeltaPlan pl = delta_plan(K, V);
  const uint8_t* block = delta_block(x, pl.bytes, b, chunk, h);
  uint8_t* sq = do_smem;                   // [hi, lo][64][RB]
  uint8_t* ss = sq + 2 * DC * RB;          // [hi, lo][K][RV]
  uint8_t* sp = ss + 2 * K * RV;           // [hi, lo][64][DC_PROW]
  uint8_t* su = sp + 2 * DC * DC_PROW;     // [hi, lo][64][RV]
  float* red = reinterpret_cast<float*>(su + 2 * DC * RV);  // [4][64]
  if (tid == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    abort_flag = 0;
    mbar_fence_init();
    const uint32_t first = 2 * DC * RB + 2 * K * RV, second = 2 * DC * DC_PROW + 2 * DC * RV;
    mbar_expect_tx(&full[0], first);
    bulk_load(do_smem, block + pl.qt, first, &full[0]);  // (q and the state lie behind each other, P and U as well)
    mbar_expect_tx(&full[1], second);
    bulk_load(sp, block + pl.p, second, &full[1]);
  }
  __syncthreads();
  const int mt = warp & 3, vn = (warp >> 2) * 32, nt = min(4, max(0, (V - vn) / 8));  // 8-value tiles of this warp (even)
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)(q0 + c0) * a.ld;
  // ---- gates, in the layout of the outputs
  float gate[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) gate[i][0] = gate[i][1] = gate[i][2] = gate[i][3] = 0.f;
  const int ta = min(mt * 16 + g, n - 1), tb = min(mt * 16 + g + 8, n - 1);
  if (a.gate_up != nullptr) {
    const __nv_bfloat16* up = reinterpret_cast<const __nv_bfloat16*>(a.gate_up) + (size_t)(h * V + vn + g) * a.gate_rank + 4 * t4;
    if (nt > 0) delta_low_rank<4>(z + (size_t)ta * a.ld + a.gate_off + 4 * t4, z + (size_t)tb * a.ld + a.gate_off + 4 * t4, up, a.gate_rank, nt, gate);
  } else {
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (i < nt) {
        const int c = a.gate_off + h * V + vn + 8 * i + 2 * t4;
        const float2 y0 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(z + (size_t)ta * a.ld + c));
        const float2 y1 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(z + (size_t)tb * a.ld + c));
        gate[i][0] = y0.x, gate[i][1] = y0.y, gate[i][2] = y1.x, gate[i][3] = y1.y;
      }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) gate[i][e] = (a.gate_up != nullptr ? 1.f : gate[i][e]) * delta_sigmoid_fast(gate[i][e]);
  float O[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) O[i][0] = O[i][1] = O[i][2] = O[i][3] = 0.f;
  auto product = [&](uint32_t A, int arow, int abytes, uint32_t Bm, int bbytes, int steps) {
    const uint32_t ao = A + (mt * 16 + (mi & 1) * 8 + r8) * arow + (mi >> 1) * 16;
    const uint32_t bo = Bm + ((mi & 1) * 8 + r8) * RV + (mi >> 1) * 16 + vn * 2;
#pragma unroll 2
    for (int ks = 0; ks < steps; ++ks) {
      uint32_t ah[4], al[4];
      ldmatrix_x4(ao + ks * 32, ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(ao + abytes + ks * 32, al[0], al[1], al[2], al[3]);
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        if (i >= nt) continue;
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bo + ks * 16 * RV + i * 16, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(bo + bbytes + ks * 16 * RV + i * 16, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          mma_bf16_16816(O[i + j], ah, bh[2 * j], bh[2 * j + 1]);
          mma_bf16_16816(O[i + j], ah, bl[2 * j], bl[2 * j + 1]);
          mma_bf16_16816(O[i + j], al, bh[2 * j], bh[2 * j + 1]);
        }
      }
    }
  };
  mbar_wait_bounded(&full[0], 0, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
  __syncwarp();
  product(smem_u32(sq), RB, DC * RB, smem_u32(ss), K * RV, KT);
  mbar_wait_bounded(&full[1], 0, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
  __syncwarp();
  product(smem_u32(sp), DC_PROW, DC * DC_PROW, smem_u32(su), DC * RV, mt + 1);
  // ---- norm over the head's values: this warp's, then across the four warps of the same tokens
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) s += O[i][2 * e] * O[i][2 * e] + O[i][2 * e + 1] * O[i][2 * e + 1];
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    if (t4 == 0) red[(warp >> 2) * DC + mt * 16 + g + 8 * e] = s;
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int t = mt * 16 + g + 8 * e;
    const float inv = rsqrtf((red[t] + red[DC + t] + red[2 * DC + t] + red[3 * DC + t]) / (float)a.v_dim + a.eps) * a.out_scale;
    if (t >= n) continue;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      if (i >= nt) continue;
      const int c = vn + 8 * i + 2 * t4;
      const float2 w = *reinterpret_cast<const float2*>(a.norm + c);
      *reinterpret_cast<uint32_t*>(out + (size_t)t * a.ld_out + c) =
          pack_bf16x2(O[i][2 * e] * inv * w.x * gate[i][2 * e], O[i][2 * e + 1] * inv * w.y * gate[i][2 * e + 1]);
    }
  }
}

}  // namespace oxb
