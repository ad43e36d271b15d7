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
// Exponents are never positive: a block of L and P that lies off the diagonal takes G relative to the last token ahead of its
// rows (rows exp(G_t - G_ref), columns exp(G_ref - G_s)); blocks of 16 on the diagonal multiply a column by one token's decay
// at a time.  G is kept as running sums within blocks of 16 and the blocks' totals, so that what lies between two tokens is
// never the small difference of two large sums; a token's logarithm ends at -50.  Every float32 factor enters the bf16 products as a high and a low half, and hi hi + hi lo + lo hi is summed in
// float32 (see retention.cuh).
#pragma once
#include "delta.cuh"
#include "retention.cuh"

namespace oxb {

constexpr int DC = 64;              // tokens per chunk
constexpr int DC_LD = DC + 4;       // floats of a row of L and of the inverse
constexpr int DC_PROW = DC * 2 + 16;  // bytes of a row of 64 halves in shared memory

// Scratch of one (chunk, head), in bytes.
struct DeltaPlan {
  int w, kb, qt, p, u0, u, s, gend, bytes;  // offsets; pairs of halves lie behind each other (hi, lo)
};
__host__ __device__ inline DeltaPlan delta_plan(int K, int V) {
  DeltaPlan p;
  p.w = 0;
  p.kb = p.w + 2 * DC * K * 2;
  p.qt = p.kb + 2 * DC * K * 2;
  p.p = p.qt + 2 * DC * K * 2;
  p.u0 = p.p + 2 * DC * DC * 2;
  p.u = p.u0 + DC * V * 4;
  p.s = p.u + 2 * DC * V * 2;
  p.gend = p.s + 2 * K * V * 2;
  p.bytes = p.gend + K * 4;
  return p;
}

struct DeltaChunkArgs {
  DeltaArgs a;
  uint8_t* ws;  // (T / 64 + B) * H blocks of delta_plan(K, V).bytes
};
// (sequence b's first block: its chunks never need more than the rows ahead of it and one each)
__device__ __forceinline__ uint8_t* delta_block(const DeltaChunkArgs& x, int bytes, int q0, int b, int chunk, int h) {
  return x.ws + ((size_t)(q0 / DC + b + chunk) * x.a.H + h) * bytes;
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

// ----------------------------------------------------------------------------- chunks by themselves
constexpr int DP_THREADS = 512, DP_TAPS = 4;
constexpr float DP_FLOOR = -50.f;  // exp of it is far below the rounding of anything it is added to

struct DeltaPrepSmem {
  int k, q, g, stage, l, misc, total;  // byte offsets
  int rows_q, cols, t, tp, kt, v;      // offsets of what shares the staging area
};
__host__ __device__ inline DeltaPrepSmem delta_prep_smem(int K, int V) {
  DeltaPrepSmem s;
  const int f32 = DC * (K + 4) * 4, half = DC * (K * 2 + 16), vhalf = DC * (V * 2 + 16);
  s.k = 0;
  s.q = s.k + f32;
  s.g = s.q + f32;
  s.stage = s.g + f32;
  // first: rows of k (hi, lo) | rows of q | columns; then: inverse (float32) | inverse * beta (hi, lo) | exp(G) k | v
  s.rows_q = 2 * half;
  s.cols = 4 * half;
  s.t = 0;
  s.tp = DC * DC_LD * 4;
  s.kt = s.tp + 2 * DC * DC_PROW;
  s.v = s.kt + 2 * half;
  const int a = 6 * half, b = s.v + 2 * vhalf;
  s.l = s.stage + (a > b ? a : b);
  s.misc = s.l + DC * DC_LD * 4;
  s.total = s.misc + (DC + 4 * K) * 4;  // beta | totals of blocks
  return s;
}

// Eight channels of the convolution and silu for tokens [j0, j0 + 8) of a portion (rows at or past n: zero); put(token, values).
template <typename F>
__device__ __forceinline__ void delta_conv8(const DeltaArgs& a, const __nv_bfloat16* z, const float* ring, int C, int pos0, int j0, int n,
                                            int ch, F put) {
  if (a.taps <= DP_TAPS) {
    float w[DP_TAPS][8], x[DP_TAPS][8];
#pragma unroll
    for (int i = 0; i < DP_TAPS; ++i) {  // (shorter convolutions: zeros on the oldest rows)
      const int tap = i - (DP_TAPS - a.taps);
      if (tap >= 0) delta_load8(a.conv + (size_t)tap * C + ch, w[i]);
      else
#pragma unroll
        for (int e = 0; e < 8; ++e) w[i][e] = 0.f;
    }
    auto fetch = [&](int j, float* v) {
      const int p = pos0 + j;
      if (j >= 0 && j < n) head_load8(z + (size_t)j * a.ld + ch, v);
      else if (j < 0 && p >= 0 && j >= 1 - a.taps) delta_load8(ring + (size_t)(p % a.taps) * C + ch, v);
      else
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = 0.f;
    };
#pragma unroll
    for (int i = 0; i < DP_TAPS - 1; ++i) fetch(j0 - (DP_TAPS - 1) + i, x[i]);
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      fetch(j0 + t, x[(t + DP_TAPS - 1) % DP_TAPS]);
      float y[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < DP_TAPS; ++i) s = fmaf(w[i][e], x[(t + i) % DP_TAPS][e], s);
        y[e] = j0 + t < n ? delta_silu(s) : 0.f;
      }
      put(t, y);
    }
  } else {
    for (int t = 0; t < 8; ++t) {
      float y[8];
      for (int e = 0; e < 8; ++e) y[e] = j0 + t < n ? delta_conv(a, z, ring, C, pos0, j0 + t, ch + e) : 0.f;
      put(t, y);
    }
  }
}

// A 16 x 16 tile (two accumulators of 8 columns) of rows . columns^T over K values, both as halves.
template <int KT>
__device__ __forceinline__ void delta_tile(uint32_t rows_hi, uint32_t rows_lo, uint32_t cols_hi, uint32_t cols_lo, int row_bytes, int lane,
                                           float (&acc)[2][4]) {
  const int mi = lane >> 3, r8 = lane & 7;
  const uint32_t ao = ((mi & 1) * 8 + r8) * row_bytes + (mi >> 1) * 16, bo = ((mi >> 1) * 8 + r8) * row_bytes + (mi & 1) * 16;
#pragma unroll
  for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int ks = 0; ks < KT; ++ks) {
    uint32_t ah[4], al[4], bh[4], bl[4];
    ldmatrix_x4(rows_hi + ao + ks * 32, ah[0], ah[1], ah[2], ah[3]);
    ldmatrix_x4(rows_lo + ao + ks * 32, al[0], al[1], al[2], al[3]);
    ldmatrix_x4(cols_hi + bo + ks * 32, bh[0], bh[1], bh[2], bh[3]);
    ldmatrix_x4(cols_lo + bo + ks * 32, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mma_bf16_16816(acc[i], ah, bh[2 * i], bh[2 * i + 1]);
      mma_bf16_16816(acc[i], ah, bl[2 * i], bl[2 * i + 1]);
      mma_bf16_16816(acc[i], al, bh[2 * i], bh[2 * i + 1]);
    }
  }
}

// grid (chunks of the longest portion, H, B); CH: a decay per key channel.
template <int KT, bool CH>
__global__ void __launch_bounds__(DP_THREADS, 1) delta_prepare_kernel(const DeltaChunkArgs x) {
  constexpr int K = KT * 16, KF = K + 4, K8 = K / 8, CPL = K / 32;
  constexpr int RB = K * 2 + 16;  // bytes of a row of halves
  extern __shared__ __align__(16) uint8_t dp_smem[];
  pdl_launch_dependents();
  const DeltaArgs& a = x.a;
  const int b = blockIdx.z, h = blockIdx.y, chunk = blockIdx.x;
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
  uint8_t* block = delta_block(x, pl.bytes, q0, b, chunk, h);
  float *sK = reinterpret_cast<float*>(dp_smem + sm.k), *sQ = reinterpret_cast<float*>(dp_smem + sm.q);
  float* sG = reinterpret_cast<float*>(dp_smem + sm.g);  // [64][KF], or [64] with one decay per head: sums within blocks of 16
  uint8_t* stage = dp_smem + sm.stage;
  float *sL = reinterpret_cast<float*>(dp_smem + sm.l), *beta = reinterpret_cast<float*>(dp_smem + sm.misc), *total = beta + DC;  // [4][K], or [4]
  const int half = DC * RB, RV = V * 2 + 16;
  const float* ring = a.window + (size_t)slot * a.taps * C;
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)q0 * a.ld;
  pdl_wait();
  // ---- convolutions of q and k, decays, step sizes
  for (int i = tid; i < 2 * K8 * 8; i += DP_THREADS) {
    const int c = i % (2 * K8), j0 = i / (2 * K8) * 8;
    float* dst = (c < K8 ? sQ + c * 8 : sK + (c - K8) * 8) + j0 * KF;
    delta_conv8(a, z, ring, C, pos0, c0 + j0, n_all, c < K8 ? kvh * K + c * 8 : (a.G + kvh) * K + (c - K8) * 8,
                [&](int t, const float* y) {
                  *reinterpret_cast<float4*>(dst + t * KF) = make_float4(y[0], y[1], y[2], y[3]);
                  *reinterpret_cast<float4*>(dst + t * KF + 4) = make_float4(y[4], y[5], y[6], y[7]);
                });
  }
  if (tid < DC) beta[tid] = tid < n ? delta_sigmoid(lat_f32(z[(size_t)(c0 + tid) * a.ld + a.beta_off + h])) : 0.f;
  const float rate = expf(a.a_log[h]);
  if (CH) {  // z . decay_up^T for 16 tokens x K / 4 channels per warp
    const int mt = warp & 3, nt0 = (warp >> 2) * (K / 32);
    float acc[K / 32][4];
#pragma unroll
    for (int i = 0; i < K / 32; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const __nv_bfloat16* r0 = z + (size_t)(c0 + min(mt * 16 + g, n - 1)) * a.ld + a.decay_off + 4 * t4;
    const __nv_bfloat16* r1 = z + (size_t)(c0 + min(mt * 16 + g + 8, n - 1)) * a.ld + a.decay_off + 4 * t4;
    const __nv_bfloat16* up = reinterpret_cast<const __nv_bfloat16*>(a.decay_up) + (size_t)(h * K + nt0 * 8 + g) * a.decay_rank + 4 * t4;
    for (int ks = 0; ks < a.decay_rank; ks += 16) {  // (which values of a k-step a lane holds is free, as long as both operands agree)
      const uint2 x0 = *reinterpret_cast<const uint2*>(r0 + ks), x1 = *reinterpret_cast<const uint2*>(r1 + ks);
      const uint32_t av[4] = {x0.x, x1.x, x0.y, x1.y};
#pragma unroll
      for (int i = 0; i < K / 32; ++i) {
        const uint2 w = *reinterpret_cast<const uint2*>(up + (size_t)i * 8 * a.decay_rank + ks);
        mma_bf16_16816(acc[i], av, w.x, w.y);
      }
    }
#pragma unroll
    for (int i = 0; i < K / 32; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = mt * 16 + g + 8 * (e >> 1), d = (nt0 + i) * 8 + 2 * t4 + (e & 1);
        sG[t * KF + d] = t < n ? fmaxf(-rate * delta_softplus(acc[i][e] + a.dt_bias[h * K + d]), DP_FLOOR) : 0.f;
      }
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
  __syncthreads();
  // ---- unit vectors; running sums of the decays
  for (int t = warp; t < DC; t += DP_THREADS / 32) {
    float qv[CPL], kv[CPL], qq = 0.f, kk = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      qv[i] = sQ[t * KF + lane + 32 * i];
      kv[i] = sK[t * KF + lane + 32 * i];
      qq += qv[i] * qv[i];
      kk += kv[i] * kv[i];
    }
    const float iq = rsqrtf(warp_sum(qq) + 1e-6f) * a.q_scale, ik = rsqrtf(warp_sum(kk) + 1e-6f);
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      sQ[t * KF + lane + 32 * i] = qv[i] * iq;
      sK[t * KF + lane + 32 * i] = kv[i] * ik;
    }
  }
  if (CH) {
    const int d = tid % K, blk = tid / K;  // (512 threads: four blocks of up to 128 channels)
    if (blk < 4) {
      float v[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) v[i] = sG[(blk * 16 + i) * KF + d];
#pragma unroll
      for (int i = 1; i < 16; ++i) v[i] += v[i - 1];
#pragma unroll
      for (int i = 1; i < 16; ++i) sG[(blk * 16 + i) * KF + d] = v[i];
      total[blk * K + d] = v[15];
    }
  }
  __syncthreads();
  auto add_totals8 = [&](int from, int to, int p, float* v) {  // totals of blocks [from, to)
    for (int i = from; i < to; ++i) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] += total[CH ? i * K + p * 8 + e : i];
    }
  };
  auto since8 = [&](int block0, int t, int p, float* v) {  // decay from the start of block `block0` through token t, eight channels
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = sG[CH ? t * KF + p * 8 + e : t];
    add_totals8(block0, t >> 4, p, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = expf(v[e]);
  };
  auto until8 = [&](int t, int block1, int p, float* v) {  // decay behind token t through the end of block `block1` - 1
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = total[CH ? (t >> 4) * K + p * 8 + e : t >> 4] - sG[CH ? t * KF + p * 8 + e : t];
    add_totals8((t >> 4) + 1, block1, p, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = expf(v[e]);
  };
  auto between = [&](int s, int t) {  // decay behind token s through token t >= s (one decay per head)
    if (s >> 4 == t >> 4) return expf(sG[t] - sG[s]);
    float v = sG[t] + (total[s >> 4] - sG[s]);
    for (int i = (s >> 4) + 1; i < t >> 4; ++i) v += total[i];
    return expf(v);
  };
  // ---- rows and columns of L and P as halves
  // with a decay per channel, rows 0-31 of the staging area: tokens 32-63 and 0-31 around token 31; rows 32-47: 16-31 and 0-15
  // around 15; rows 48-63: 48-63 and 32-47 around 47
  for (int i = tid; i < DC * K8; i += DP_THREADS) {
    const int r = i / K8, p = i % K8;
    const uint32_t o = r * RB + p * 16;
    const int row = CH ? (r < 32 ? 32 + r : (r < 48 ? r - 16 : r)) : r, col = r < 32 ? r : (r < 48 ? r - 32 : r - 16);
    float kv[8], qv[8];
    delta_load8(sK + row * KF + p * 8, kv);
    delta_load8(sQ + row * KF + p * 8, qv);
    if (CH) {
      const int ref = r < 32 ? 2 : (r < 48 ? 1 : 3);  // the block that starts behind token 31, 15, 47
      float f[8];
      since8(ref, row, p, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        kv[e] *= f[e];
        qv[e] *= f[e];
      }
      delta_split8(kv, stage + o, stage + half + o);
      delta_split8(qv, stage + sm.rows_q + o, stage + sm.rows_q + half + o);
      delta_load8(sK + col * KF + p * 8, kv);
      until8(col, ref, p, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) kv[e] *= f[e];
      delta_split8(kv, stage + sm.cols + o, stage + sm.cols + half + o);
    } else {
      delta_split8(kv, stage + o, stage + half + o);
      delta_split8(qv, stage + sm.rows_q + o, stage + sm.rows_q + half + o);
    }
  }
  __nv_bfloat16 *p_hi = reinterpret_cast<__nv_bfloat16*>(block + pl.p), *p_lo = p_hi + DC * DC;
  __syncthreads();
  {
    const uint32_t st = smem_u32(stage);
    const int tasks = CH ? 12 : 20;
    for (int u = warp; u < tasks; u += DP_THREADS / 32) {
      const bool is_q = u >= tasks / 2;
      const int v = is_q ? u - tasks / 2 : u;
      int mt, np, rr, cr;  // 16-token blocks of the rows and columns, and where they stand
      if (CH) {
        mt = v < 4 ? 2 + (v >> 1) : (v == 4 ? 1 : 3);
        np = v < 4 ? (v & 1) : (v == 4 ? 0 : 2);
        rr = v < 4 ? (v >> 1) * 16 : (v == 4 ? 32 : 48);
        cr = v < 4 ? (v & 1) * 16 : (v == 4 ? 32 : 48);
      } else {
        mt = v < 1 ? 0 : (v < 3 ? 1 : (v < 6 ? 2 : 3));
        np = v - mt * (mt + 1) / 2;
        rr = mt * 16;
        cr = np * 16;
      }
      const uint32_t rows = st + (is_q ? sm.rows_q : 0) + rr * RB, cols = st + (CH ? sm.cols : 0) + cr * RB;
      float acc[2][4];
      delta_tile<KT>(rows, rows + half, cols, cols + half, RB, lane, acc);
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int t = mt * 16 + g + 8 * (e >> 1), s = np * 16 + 8 * i + 2 * t4;
          float v0 = acc[i][e], v1 = acc[i][e + 1];
          if (!CH) {
            v0 = s <= t ? v0 * between(s, t) : 0.f;
            v1 = s + 1 <= t ? v1 * between(s + 1, t) : 0.f;
          }
          if (is_q) {
            uint32_t hi, lo;
            split_bf16x2(v0, v1, hi, lo);
            *reinterpret_cast<uint32_t*>(p_hi + t * DC + s) = hi;
            *reinterpret_cast<uint32_t*>(p_lo + t * DC + s) = lo;
          } else {
            sL[t * DC_LD + s] = v0 * beta[t];
            sL[t * DC_LD + s + 1] = v1 * beta[t];
          }
        }
    }
  }
  if (CH) {  // blocks of 16 on the diagonal: a warp has four columns of one block, a lane CPL channels
    const int t0 = (warp >> 2) * 16, s0 = t0 + (warp & 3) * 4;
    float w[4][CPL];
#pragma unroll
    for (int s = 0; s < 4; ++s)
#pragma unroll
      for (int i = 0; i < CPL; ++i) w[s][i] = 0.f;
    for (int t = t0; t < t0 + 16; ++t) {
      float sum[8];  // k . w, q . w of the four columns
#pragma unroll
      for (int s = 0; s < 8; ++s) sum[s] = 0.f;
      if (t >= s0) {
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
          const int d = lane + 32 * i;
          const float kt = sK[t * KF + d], qt = sQ[t * KF + d];
          const float f = t > s0 ? expf(sG[t * KF + d] - sG[(t - 1) * KF + d]) : 0.f;
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
          p_hi[t * DC + s] = hi;
          p_lo[t * DC + s] = __float2bfloat16(v - __bfloat162float(hi));
        }
      }
    }
  }
  __syncthreads();
  // ---- the inverse of I + L: blocks of 16 on the diagonal by substitution, the others from them
  float* sT = reinterpret_cast<float*>(stage + sm.t);
  if (tid < DC) {
    const int t0 = tid & ~15, c = tid & 15;
    float v[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < 16; ++i)
        if (i < r) s = fmaf(sL[(t0 + r) * DC_LD + t0 + i], v[i], s);
      v[r] = r < c ? 0.f : (r == c ? 1.f : -s);
      sT[(t0 + r) * DC_LD + t0 + c] = v[r];
    }
  } else if (tid >= 128) {  // (meanwhile) v into its halves, and exp(G) k
    for (int i = tid - 128; i < V8 * 8; i += DP_THREADS - 128) {
      const int c = i % V8, j0 = i / V8 * 8;
      delta_conv8(a, z, ring, C, pos0, c0 + j0, n_all, 2 * a.G * K + h * V + c * 8, [&](int t, const float* y) {
        uint8_t* at = stage + sm.v + (j0 + t) * RV + c * 16;
        delta_split8(y, at, at + DC * RV);
      });
    }
    for (int i = tid - 128; i < DC * K8; i += DP_THREADS - 128) {
      const int t = i / K8, p = i % K8;
      float kv[8], f[8];
      delta_load8(sK + t * KF + p * 8, kv);
      since8(0, t, p, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) kv[e] *= f[e];
      uint8_t* at = stage + sm.kt + t * RB + p * 16;
      delta_split8(kv, at, at + half);
    }
  }
  __syncthreads();
  for (int dist = 1; dist < 4; ++dist) {
    // block (i, i - dist): first sum_k L_ik T_kj into the (unused) mirror block above the diagonal, then - T_ii times that
    for (int u = tid; u < (4 - dist) * 256; u += DP_THREADS) {
      const int j = u >> 8, i = j + dist, r = u >> 4 & 15, c = u & 15;
      float s = 0.f;
      for (int m = j * 16; m < i * 16; ++m) s = fmaf(sL[(i * 16 + r) * DC_LD + m], sT[m * DC_LD + j * 16 + c], s);
      sL[(j * 16 + r) * DC_LD + i * 16 + c] = s;
    }
    __syncthreads();
    for (int u = tid; u < (4 - dist) * 256; u += DP_THREADS) {
      const int j = u >> 8, i = j + dist, r = u >> 4 & 15, c = u & 15;
      float s = 0.f;
#pragma unroll
      for (int m = 0; m < 16; ++m) s = fmaf(sT[(i * 16 + r) * DC_LD + i * 16 + m], sL[(j * 16 + m) * DC_LD + i * 16 + c], s);
      sT[(i * 16 + r) * DC_LD + j * 16 + c] = -s;
    }
    __syncthreads();
  }
  for (int i = tid; i < DC * DC / 8; i += DP_THREADS) {  // times beta, as halves
    const int t = i / 8, p = i % 8;
    if (p * 8 > (t | 15)) continue;
    float v[8];
    delta_load8(sT + t * DC_LD + p * 8, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= beta[p * 8 + e];
    uint8_t* at = stage + sm.tp + t * DC_PROW + p * 16;
    delta_split8(v, at, at + DC * DC_PROW);
  }
  // ---- exp(G) q and exp(G_end - G) k for the other kernels
  for (int i = tid; i < DC * K8; i += DP_THREADS) {
    const int t = i / K8, p = i % K8;
    float v[8], f[8];
    since8(0, t, p, f);
    delta_load8(sQ + t * KF + p * 8, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= f[e];
    uint8_t* at = block + pl.qt + (t * K + p * 8) * 2;
    delta_split8(v, at, at + DC * K * 2);
    delta_load8(sK + t * KF + p * 8, v);
    until8(t, DC / 16, p, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= f[e];
    at = block + pl.kb + (t * K + p * 8) * 2;
    delta_split8(v, at, at + DC * K * 2);
  }
  if (tid < K) {
    float s = 0.f;
    for (int i = 0; i < DC / 16; ++i) s += total[CH ? i * K + tid : i];
    reinterpret_cast<float*>(block + pl.gend)[tid] = expf(s);
  }
  __syncthreads();
  // ---- W = T exp(G) k and U0 = T v (T: the inverse times beta), 16 x 16 tiles
  {
    const int mi = lane >> 3, r8 = lane & 7, nk = K / 16, nv = V / 16;
    const uint32_t tp = smem_u32(stage + sm.tp), kt = smem_u32(stage + sm.kt), vt = smem_u32(stage + sm.v);
    for (int u = warp; u < 4 * (nk + nv); u += DP_THREADS / 32) {
      const int mt = 3 - (u & 3), nt = u >> 2;
      const bool is_w = nt < nk;
      const int rb = is_w ? RB : RV, col = is_w ? nt : nt - nk;
      const uint32_t A = tp + (mt * 16 + (mi & 1) * 8 + r8) * DC_PROW + (mi >> 1) * 16;
      const uint32_t Bm = (is_w ? kt : vt) + ((mi & 1) * 8 + r8) * rb + (mi >> 1) * 16 + col * 32;
      float acc[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
      for (int ks = 0; ks <= mt; ++ks) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        ldmatrix_x4(A + ks * 32, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(A + DC * DC_PROW + ks * 32, al[0], al[1], al[2], al[3]);
        ldmatrix_x4_trans(Bm + ks * 16 * rb, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(Bm + DC * rb + ks * 16 * rb, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma_bf16_16816(acc[i], ah, bh[2 * i], bh[2 * i + 1]);
          mma_bf16_16816(acc[i], ah, bl[2 * i], bl[2 * i + 1]);
          mma_bf16_16816(acc[i], al, bh[2 * i], bh[2 * i + 1]);
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int t = mt * 16 + g + 8 * (e >> 1), c = col * 16 + 8 * i + 2 * t4;
          if (is_w) {
            uint32_t hi, lo;
            split_bf16x2(acc[i][e], acc[i][e + 1], hi, lo);
            uint8_t* at = block + pl.w + (t * K + c) * 2;
            *reinterpret_cast<uint32_t*>(at) = hi;
            *reinterpret_cast<uint32_t*>(at + DC * K * 2) = lo;
          } else {
            *reinterpret_cast<float2*>(block + pl.u0 + (t * V + c) * 4) = make_float2(acc[i][e], acc[i][e + 1]);
          }
        }
    }
  }
}

// ----------------------------------------------------------------------------- the state, chunk after chunk
constexpr int DS_THREADS = 256;
__host__ __device__ inline int delta_state_smem(int K, int NV) {
  return 2 * 4 * DC * (K * 2 + 16) + 2 * K * (NV * 2 + 16) + 2 * DC * (NV * 2 + 16);
}

// grid (V / NV, H, B): a CTA has NV values of one head's state, warp w its rows 16 w .. 16 w + 15 in accumulator registers.
template <int KT, int NV>
__global__ void __launch_bounds__(DS_THREADS, 1) delta_state_kernel(const DeltaChunkArgs x) {
  constexpr int K = KT * 16, RB = K * 2 + 16, RN = NV * 2 + 16, NT = NV / 8, K8 = K / 8;
  constexpr int UT = NV / 16;  // tiles of 8 values that a warp has of U: 16 tokens x NV / 2 values
  extern __shared__ __align__(16) uint8_t dt_smem[];
  pdl_launch_dependents();
  const DeltaArgs& a = x.a;
  const int v0 = blockIdx.x * NV, h = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const int q0 = a.query_start[b], n = a.query_start[b + 1] - q0, slot = a.slots[b];
  if (n < a.min_rows || n > a.max_rows || n <= 0 || (unsigned)slot >= (unsigned)a.num_slots) {
    pdl_wait();
    return;
  }
  const int V = a.V, chunks = (n + DC - 1) / DC;
  const DeltaPlan pl = delta_plan(K, V);
  uint8_t* ops = dt_smem;               // [2][W hi, lo, Kb hi, lo][64][RB]
  uint8_t* sS = ops + 8 * DC * RB;      // [hi, lo][K][RN]
  uint8_t* sU = sS + 2 * K * RN;        // [hi, lo][64][RN]
  const bool rows = warp < KT;          // this warp has rows of the state
  float S[NT][4];
  float* st = a.state + ((size_t)slot * a.H + h) * K * V + (size_t)(warp * 16 + g) * V + v0 + 2 * t4;
  const bool resumed = a.seq_lens[b] > n;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {  // (written by an earlier step: no need to wait for this step's kernels)
      const float2 y = (rows && resumed) ? *reinterpret_cast<const float2*>(st + (size_t)(e >> 1) * 8 * V + 8 * i) : make_float2(0.f, 0.f);
      S[i][e] = y.x;
      S[i][e + 1] = y.y;
    }
  pdl_wait();
  auto fetch = [&](int c) {
    const uint8_t* block = delta_block(x, pl.bytes, q0, b, c, h);
    uint8_t* dst = ops + (c & 1) * 4 * DC * RB;
    for (int i = tid; i < 4 * DC * K8; i += DS_THREADS) {  // (W and Kb lie behind each other: 256 rows of halves)
      const int r = i / K8, p = i % K8;
      cp_async16(dst + r * RB + p * 16, block + (size_t)i * 16);
    }
    cp_async_commit();
  };
  auto put_state = [&](uint8_t* block) {  // halves of this warp's rows: for the next products, and for the outputs
    if (!rows) return;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        uint32_t hi, lo;
        split_bf16x2(S[i][e], S[i][e + 1], hi, lo);
        const int k = warp * 16 + g + 8 * (e >> 1), c = 8 * i + 2 * t4;
        *reinterpret_cast<uint32_t*>(sS + k * RN + c * 2) = hi;
        *reinterpret_cast<uint32_t*>(sS + K * RN + k * RN + c * 2) = lo;
        uint8_t* at = block + pl.s + ((size_t)k * V + v0 + c) * 2;
        *reinterpret_cast<uint32_t*>(at) = hi;
        *reinterpret_cast<uint32_t*>(at + (size_t)K * V * 2) = lo;
      }
  };
  const uint32_t ops_u = smem_u32(ops), s_u = smem_u32(sS), u_u = smem_u32(sU);
  const int mt = warp & 3, un = (warp >> 2) * (NV / 2);  // this warp's tile of U
  const uint32_t wa = (mt * 16 + (mi & 1) * 8 + r8) * RB + (mi >> 1) * 16;
  const uint32_t sb = ((mi & 1) * 8 + r8) * RN + (NV == 32 ? un * 2 + (mi >> 1) * 16 : (mi >> 1) * 16);
  const uint32_t ka = ((mi >> 1) * 8 + r8) * RB + warp * 32 + (mi & 1) * 16;  // transposed: 16 keys x 16 tokens
  const uint32_t ub = ((mi & 1) * 8 + r8) * RN + (mi >> 1) * 16;
  fetch(0);
  for (int c = 0; c < chunks; ++c) {
    uint8_t* block = delta_block(x, pl.bytes, q0, b, c, h);
    put_state(block);
    float u0[UT][4];
    const float* up = reinterpret_cast<const float*>(block + pl.u0) + (size_t)(mt * 16 + g) * V + v0 + un + 2 * t4;
#pragma unroll
    for (int i = 0; i < UT; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const float2 y = *reinterpret_cast<const float2*>(up + (size_t)(e >> 1) * 8 * V + 8 * i);
        u0[i][e] = y.x;
        u0[i][e + 1] = y.y;
      }
    float ge[2] = {0.f, 0.f};
    if (rows) {
      const float* gp = reinterpret_cast<const float*>(block + pl.gend) + warp * 16 + g;
      ge[0] = gp[0];
      ge[1] = gp[8];
    }
    if (c + 1 < chunks) {
      fetch(c + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();  // this chunk's operands and the state are in shared memory
    const uint32_t W = ops_u + (c & 1) * 4 * DC * RB, Kb = W + 2 * DC * RB;
    float acc[UT][3][4];
#pragma unroll
    for (int i = 0; i < UT; ++i)
#pragma unroll
      for (int j = 0; j < 3; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KT; ++ks) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      ldmatrix_x4(W + wa + ks * 32, ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(W + DC * RB + wa + ks * 32, al[0], al[1], al[2], al[3]);
      ldmatrix_x4_trans(s_u + sb + ks * 16 * RN, bh[0], bh[1], bh[2], bh[3]);
      ldmatrix_x4_trans(s_u + K * RN + sb + ks * 16 * RN, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
      for (int i = 0; i < UT; ++i) {
        const bool second = NV == 32 ? i == 1 : un > 0;
        const uint32_t b0 = second ? bh[2] : bh[0], b1 = second ? bh[3] : bh[1], l0 = second ? bl[2] : bl[0], l1 = second ? bl[3] : bl[1];
        mma_bf16_16816(acc[i][0], ah, b0, b1);
        mma_bf16_16816(acc[i][1], ah, l0, l1);
        mma_bf16_16816(acc[i][2], al, b0, b1);
      }
    }
#pragma unroll
    for (int i = 0; i < UT; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        uint32_t hi, lo;
        split_bf16x2(u0[i][e] - (acc[i][0][e] + (acc[i][1][e] + acc[i][2][e])),
                     u0[i][e + 1] - (acc[i][0][e + 1] + (acc[i][1][e + 1] + acc[i][2][e + 1])), hi, lo);
        const int t = mt * 16 + g + 8 * (e >> 1), cc = un + 8 * i + 2 * t4;
        *reinterpret_cast<uint32_t*>(sU + t * RN + cc * 2) = hi;
        *reinterpret_cast<uint32_t*>(sU + DC * RN + t * RN + cc * 2) = lo;
        uint8_t* at = block + pl.u + ((size_t)t * V + v0 + cc) * 2;
        *reinterpret_cast<uint32_t*>(at) = hi;
        *reinterpret_cast<uint32_t*>(at + (size_t)DC * V * 2) = lo;
      }
    __syncthreads();  // U is complete; the state's halves have been read
    if (rows) {
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        S[i][0] *= ge[0];
        S[i][1] *= ge[0];
        S[i][2] *= ge[1];
        S[i][3] *= ge[1];
      }
#pragma unroll
      for (int ks = 0; ks < DC / 16; ++ks) {
        uint32_t ah[4], al[4];
        ldmatrix_x4_trans(Kb + ka + ks * 16 * RB, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4_trans(Kb + DC * RB + ka + ks * 16 * RB, al[0], al[1], al[2], al[3]);
#pragma unroll
        for (int i = 0; i < NT; i += 2) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(u_u + ub + ks * 16 * RN + i * 16, bh[0], bh[1], bh[2], bh[3]);
          ldmatrix_x4_trans(u_u + DC * RN + ub + ks * 16 * RN + i * 16, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            mma_bf16_16816(S[i + j], ah, bh[2 * j], bh[2 * j + 1]);
            mma_bf16_16816(S[i + j], ah, bl[2 * j], bl[2 * j + 1]);
            mma_bf16_16816(S[i + j], al, bh[2 * j], bh[2 * j + 1]);
          }
        }
      }
    }
    __syncthreads();  // this chunk's operands have been read: their buffer takes the chunk after next
  }
  if (rows) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) *reinterpret_cast<float2*>(st + (size_t)(e >> 1) * 8 * V + 8 * i) = make_float2(S[i][e], S[i][e + 1]);
  }
}

// ----------------------------------------------------------------------------- outputs
constexpr int DO_THREADS = 512;
__host__ __device__ inline int delta_output_smem(int K, int V) {
  return 2 * DC * (K * 2 + 16) + 2 * K * (V * 2 + 16) + 2 * DC * DC_PROW + 2 * DC * (V * 2 + 16) + 4 * DC * 4;
}

// grid (chunks of the longest portion, H, B); warp w: tokens 16 (w % 4) .., values 32 (w / 4) ..
template <int KT>
__global__ void __launch_bounds__(DO_THREADS, 1) delta_output_kernel(const DeltaChunkArgs x) {
  constexpr int K = KT * 16, RB = K * 2 + 16, K8 = K / 8;
  extern __shared__ __align__(16) uint8_t do_smem[];
  pdl_launch_dependents();
  const DeltaArgs& a = x.a;
  const int b = blockIdx.z, h = blockIdx.y, chunk = blockIdx.x, c0 = chunk * DC;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const int q0 = a.query_start[b], n_all = a.query_start[b + 1] - q0, slot = a.slots[b];
  const int V = a.V, V8 = V / 8, RV = V * 2 + 16;
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
  const uint8_t* block = delta_block(x, pl.bytes, q0, b, chunk, h);
  uint8_t* sq = do_smem;                   // [hi, lo][64][RB]
  uint8_t* ss = sq + 2 * DC * RB;          // [hi, lo][K][RV]
  uint8_t* sp = ss + 2 * K * RV;           // [hi, lo][64][DC_PROW]
  uint8_t* su = sp + 2 * DC * DC_PROW;     // [hi, lo][64][RV]
  float* red = reinterpret_cast<float*>(su + 2 * DC * RV);  // [4][64]
  for (int i = tid; i < 2 * DC * K8; i += DO_THREADS) cp_async16(sq + i / K8 * RB + i % K8 * 16, block + pl.qt + (size_t)i * 16);
  for (int i = tid; i < 2 * K * V8; i += DO_THREADS) cp_async16(ss + i / V8 * RV + i % V8 * 16, block + pl.s + (size_t)i * 16);
  cp_async_commit();
  for (int i = tid; i < 2 * DC * 8; i += DO_THREADS) cp_async16(sp + i / 8 * DC_PROW + i % 8 * 16, block + pl.p + (size_t)i * 16);
  for (int i = tid; i < 2 * DC * V8; i += DO_THREADS) cp_async16(su + i / V8 * RV + i % V8 * 16, block + pl.u + (size_t)i * 16);
  cp_async_commit();
  const int mt = warp & 3, vn = (warp >> 2) * 32, nt = min(4, max(0, (V - vn) / 8));  // 8-value tiles of this warp (even)
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)(q0 + c0) * a.ld;
  // ---- gates, in the layout of the outputs
  float gate[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) gate[i][0] = gate[i][1] = gate[i][2] = gate[i][3] = 0.f;
  const int ta = min(mt * 16 + g, n - 1), tb = min(mt * 16 + g + 8, n - 1);
  if (a.gate_up != nullptr) {
    const __nv_bfloat16 *r0 = z + (size_t)ta * a.ld + a.gate_off + 4 * t4, *r1 = z + (size_t)tb * a.ld + a.gate_off + 4 * t4;
    const __nv_bfloat16* up = reinterpret_cast<const __nv_bfloat16*>(a.gate_up) + (size_t)(h * V + vn + g) * a.gate_rank + 4 * t4;
    for (int ks = 0; ks < a.gate_rank; ks += 16) {
      const uint2 x0 = *reinterpret_cast<const uint2*>(r0 + ks), x1 = *reinterpret_cast<const uint2*>(r1 + ks);
      const uint32_t av[4] = {x0.x, x1.x, x0.y, x1.y};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (i >= nt) continue;  // (the same for the whole warp)
        const uint2 w = *reinterpret_cast<const uint2*>(up + (size_t)i * 8 * a.gate_rank + ks);
        mma_bf16_16816(gate[i], av, w.x, w.y);
      }
    }
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
    for (int e = 0; e < 4; ++e) gate[i][e] = (a.gate_up != nullptr ? 1.f : gate[i][e]) / (1.f + expf(-gate[i][e]));
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
  cp_async_wait<1>();
  __syncthreads();
  product(smem_u32(sq), RB, DC * RB, smem_u32(ss), K * RV, KT);
  cp_async_wait<0>();
  __syncthreads();
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
