// RWKV time mixing of long portions: chunks of 64 tokens on the tensor cores.
//
// Inside a chunk that starts from state S, with the running sums G_t of the decays' logarithms (per key channel),
//     o_t = (exp(G_(t-1)) r_t)^T S + sum_(s<t) A_ts v_s + (r_t . u k_t) v_t,   A_ts = sum_d r_t k_s exp(G_(t-1) - G_s),
//     S' = exp(G_end) S + sum_s (exp(G_end - G_s) k_s) v_s^T.
// wkv_state_kernel goes from chunk to chunk; the rows of the state do not depend on one another, so a CTA owns 32 key channels
// of a head with their state in accumulator registers, and leaves the state in front of every chunk as the operand that
// wkv_output_kernel (all chunks at once) multiplies with.  The transposed product, [values, channels], makes the accumulators of
// the one the operand registers of the other.
//
// G is kept in binary logarithms, as running sums within blocks of 16 tokens and the blocks' totals, so that what lies between
// two tokens is never the small difference of two large sums; a token's logarithm ends at -72.  In A a block off the diagonal
// takes its rows relative to the start of their block and its columns relative to that point, so that no exponent is positive;
// a block on the diagonal takes both relative to its start unless a channel loses more than 2^-60 in it, in which case its
// entries are summed up one by one.  Every float32 factor enters the bf16 products as a high and a low half (see retention.cuh).
//
// A portion is worked off in rounds of as many chunks as the scratch holds; between them the state is where it always is.
#pragma once
#include "delta_chunk.cuh"
#include "wkv.cuh"

namespace oxb {

constexpr int WC = 64;       // tokens per chunk
constexpr int WC_CH = 32;    // key channels per CTA of wkv_state_kernel
constexpr int WC_PROW = WC * 2 + 16;  // bytes of a row of 64 halves

struct WkvChunkArgs {
  WkvArgs a;
  uint4* ws;          // states in front of the chunks: B * round * H blocks of K * V / 4 pieces
  int chunk0, round;  // chunks [chunk0, chunk0 + round) of every portion
};

constexpr int WST_WARPS = 8, WST_THREADS = WST_WARPS * 32, WST_ROWS = WC / WST_WARPS;  // tokens per warp
__host__ __device__ inline int wkv_state_smem(int K) {
  return 2 * WC * (K * 2 + 16) + 2 * WC * (WC_CH * 2 + 16) + 2 * (WST_WARPS + 1) * WC_CH * 4;
}

// This thread's tokens from t0 on of channel `col`: logarithms and keys, zeros past the portion.
__device__ __forceinline__ void wkv_fetch(const WkvArgs& a, const __nv_bfloat16* z, const float* decay, int t0, int n, int col, float* l,
                                          __nv_bfloat16* k) {
  const size_t hk = (size_t)a.H * a.K;
#pragma unroll
  for (int i = 0; i < WST_ROWS; ++i) {
    const bool have = t0 + i < n;
    l[i] = have ? decay[(size_t)(t0 + i) * hk + col] : 0.f;
    k[i] = have ? z[(size_t)(t0 + i) * a.ld + hk + col] : __float2bfloat16(0.f);
  }
}

// grid (K / 32, H, B).  Every warp owns 16 MT values of a head (MT * 128 = V rounded up).
template <int MT>
__global__ void __launch_bounds__(WST_THREADS) wkv_state_kernel(const WkvChunkArgs x) {
  extern __shared__ __align__(16) uint8_t wst_smem[];
  pdl_launch_dependents();
  const WkvArgs& a = x.a;
  const int b = blockIdx.z, h = blockIdx.y, ch0 = blockIdx.x * WC_CH, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3, K = a.K, V = K;
  const int q0 = a.query_start[b], n_all = a.query_start[b + 1] - q0, slot = a.slots[b], c0 = x.chunk0 * WC;
  if (n_all < a.min_rows || n_all > a.max_rows || c0 >= n_all || (unsigned)slot >= (unsigned)a.num_slots) {
    pdl_wait();
    return;
  }
  const int RV = V * 2 + 16, RK = WC_CH * 2 + 16, vtiles = V / 16;
  uint8_t* sv = wst_smem;                   // [2][64] rows of V halves
  uint8_t* skh = sv + 2 * WC * RV;          // [2 (hi, lo)][64] rows of 32 halves
  float* total = reinterpret_cast<float*>(skh + 2 * WC * RK);  // [2][8 + 1][32] logarithms of what the warps' tokens decay by, and the chunk's decay
  float* S0 = a.state + ((size_t)slot * a.H + h) * K * V;
  const bool fresh = a.seq_lens[b] == n_all && x.chunk0 == 0;
  const size_t hk = (size_t)a.H * K;
  pdl_wait();
  // values: rows g, g + 8 of tile m; channels: columns 2 t4, 2 t4 + 1 of tile i
  float s[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = (warp * MT + m) * 16 + g + 8 * (e >> 1), c = ch0 + 8 * i + 2 * t4 + (e & 1);
        s[m][i][e] = (!fresh && v < V) ? S0[(size_t)c * V + v] : 0.f;
      }
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)q0 * a.ld + (size_t)h * K;
  const float* decay = a.log_decay + (size_t)q0 * hk + (size_t)h * K;
  const int chunks = min((n_all - c0 + WC - 1) / WC, x.round), col = ch0 + lane;
  auto load_v = [&](int c) {  // chunk c of the round
    uint8_t* dst = sv + (c & 1) * WC * RV;
    for (int i = tid; i < WC * (V / 8); i += WST_THREADS) {
      const int r = i / (V / 8), p = i % (V / 8), t = c0 + c * WC + r;
      if (t < n_all) cp_async16(dst + r * RV + p * 16, z + (size_t)t * a.ld + 2 * hk + p * 8);
      else *reinterpret_cast<uint4*>(dst + r * RV + p * 16) = make_uint4(0, 0, 0, 0);
    }
  };
  float l2[2][WST_ROWS];  // two chunks' inputs on their way
  __nv_bfloat16 k2[2][WST_ROWS];
  wkv_fetch(a, z, decay, c0 + warp * WST_ROWS, n_all, col, l2[0], k2[0]);
  wkv_fetch(a, z, decay, c0 + WC + warp * WST_ROWS, n_all, col, l2[1], k2[1]);
  load_v(0);
  cp_async_commit();
  uint4* ws = x.ws + ((size_t)b * x.round * a.H + h) * (K * V / 4);
  auto chunk = [&](int c, float (&l)[WST_ROWS], __nv_bfloat16 (&k)[WST_ROWS]) {
    // ---- the state in front of the chunk, as operand registers: (channels 16 j .., values 8 n ..) of this lane
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int vt = warp * MT + m;
      if (vt >= vtiles) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          uint4 o;
          split_bf16x2(s[m][2 * j][2 * e], s[m][2 * j][2 * e + 1], o.x, o.z);
          split_bf16x2(s[m][2 * j + 1][2 * e], s[m][2 * j + 1][2 * e + 1], o.y, o.w);
          ws[((size_t)(ch0 / 16 + j) * (V / 8) + 2 * vt + e) * 32 + lane] = o;
        }
    }
    ws += (size_t)a.H * (K * V / 4);
    // ---- running sums of this thread's tokens; the keys relative to the end of the chunk
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < WST_ROWS; ++i) {
      sum += fmaxf(l[i] * 1.4426950408889634f, DP_FLOOR);
      l[i] = sum;
    }
    float* tot = total + (c & 1) * (WST_WARPS + 1) * WC_CH;
    tot[warp * WC_CH + lane] = sum;
    __syncthreads();  // (also: every warp is done with the previous chunk's operands)
    float rest = sum;
    for (int i = warp + 1; i < WST_WARPS; ++i) rest += tot[i * WC_CH + lane];
    if (warp == 0) tot[WST_WARPS * WC_CH + lane] = delta_exp2(rest);
#pragma unroll
    for (int i = 0; i < WST_ROWS; ++i) {
      const float y = __bfloat162float(k[i]) * delta_exp2(rest - l[i]);
      const __nv_bfloat16 hi = __float2bfloat16(y);
      uint8_t* at = skh + (warp * WST_ROWS + i) * RK + lane * 2;
      *reinterpret_cast<__nv_bfloat16*>(at) = hi;
      *reinterpret_cast<__nv_bfloat16*>(at + WC * RK) = __float2bfloat16(y - __bfloat162float(hi));
    }
    cp_async_wait<0>();
    __syncthreads();
    if (c + 2 < chunks) wkv_fetch(a, z, decay, c0 + (c + 2) * WC + warp * WST_ROWS, n_all, col, l, k);
    if (c + 1 < chunks) load_v(c + 1);
    cp_async_commit();
    // ---- S' = exp(G_end) S + V^T k
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 d = *reinterpret_cast<const float2*>(tot + WST_WARPS * WC_CH + 8 * i + 2 * t4);
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[m][i][e] *= e & 1 ? d.y : d.x;
    }
    const uint32_t v_base = smem_u32(sv + (c & 1) * WC * RV), k_base = smem_u32(skh);
    const int mi = lane >> 3, r = lane & 7;
#pragma unroll
    for (int ks = 0; ks < WC / 16; ++ks) {
      uint32_t bh[4][2], bl[4][2];
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        const uint32_t at = k_base + (ks * 16 + (mi & 1) * 8 + r) * RK + (i + (mi >> 1)) * 16;
        ldmatrix_x4_trans(at, bh[i][0], bh[i][1], bh[i + 1][0], bh[i + 1][1]);
        ldmatrix_x4_trans(at + WC * RK, bl[i][0], bl[i][1], bl[i + 1][0], bl[i + 1][1]);
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int vt = warp * MT + m;
        if (vt >= vtiles) continue;
        uint32_t av[4];  // [values, tokens] out of rows of tokens
        ldmatrix_x4_trans(v_base + (ks * 16 + (mi >> 1) * 8 + r) * RV + vt * 32 + (mi & 1) * 16, av[0], av[1], av[2], av[3]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          mma_bf16_16816(s[m][i], av, bl[i][0], bl[i][1]);
          mma_bf16_16816(s[m][i], av, bh[i][0], bh[i][1]);
        }
      }
    }
  };
  for (int c = 0; c < chunks; c += 2) {
    chunk(c, l2[0], k2[0]);
    if (c + 1 < chunks) chunk(c + 1, l2[1], k2[1]);
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = (warp * MT + m) * 16 + g + 8 * (e >> 1), c = ch0 + 8 * i + 2 * t4 + (e & 1);
        if (v < V) S0[(size_t)c * V + v] = s[m][i][e];
      }
}

constexpr int WO_THREADS = 256;
struct WkvOutputSmem {
  int g, rr, k, a, misc, total;  // byte offsets
};
__host__ __device__ inline WkvOutputSmem wkv_output_smem(int K) {
  WkvOutputSmem s;
  const int row = WC * (K * 2 + 16);
  s.g = 0;                         // logarithms; once A is there: v
  s.rr = s.g + WC * (K + 8) * 4;   // r times decays as halves (hi, lo)
  s.k = s.rr + 2 * row;
  s.a = s.k + row;                 // r; then A as halves (hi, lo)
  s.misc = s.a + (2 * WC * WC_PROW > row ? 2 * WC * WC_PROW : row);
  s.total = s.misc + (4 * K + WC + 8 * WC + 4) * 4;  // totals of blocks | diagonal | sums of squares per warp | flags
  return s;
}

// grid (chunks of the round, H, B).  A warp owns NT tiles of 8 values and all tokens of the chunk.
template <int KT>
__global__ void __launch_bounds__(WO_THREADS, 2) wkv_output_kernel(const WkvChunkArgs x) {
  constexpr int K = KT * 16, V = K, KF = K + 8, K8 = K / 8, RB = K * 2 + 16, HALF = WC * RB, NT = (V / 8 + 7) / 8;
  extern __shared__ __align__(16) uint8_t wo_smem[];
  pdl_launch_dependents();
  const WkvArgs& a = x.a;
  const int b = blockIdx.z, h = blockIdx.y, chunk = x.chunk0 + blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
  const int q0 = a.query_start[b], n_all = a.query_start[b + 1] - q0, slot = a.slots[b], c0 = chunk * WC;
  if (n_all < a.min_rows || n_all > a.max_rows || c0 >= n_all) {
    pdl_wait();
    return;
  }
  const int n = min(WC, n_all - c0);
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(q0 + c0) * a.ld_out + (size_t)h * V;
  if ((unsigned)slot >= (unsigned)a.num_slots) {
    if (slot >= 0 && tid == 0) oxb_report(OXB_BAD_SLOT, slot);
    pdl_wait();
    for (int i = tid; i < n * V; i += WO_THREADS) out[(size_t)(i / V) * a.ld_out + i % V] = __float2bfloat16(0.f);
    return;
  }
  const WkvOutputSmem sm = wkv_output_smem(K);
  float* sG = reinterpret_cast<float*>(wo_smem + sm.g);  // [64][KF] logarithms, then their sums within blocks of 16
  uint8_t *sRR = wo_smem + sm.rr, *sA = wo_smem + sm.a;
  uint8_t *sR = sA, *sK = wo_smem + sm.k, *sV = wo_smem + sm.g;
  float *total = reinterpret_cast<float*>(wo_smem + sm.misc), *diag = total + 4 * K, *sums = diag + WC;
  int* wild = reinterpret_cast<int*>(sums + 8 * WC);  // [4] blocks whose decays leave the range
  const size_t hk = (size_t)a.H * K;
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)(q0 + c0) * a.ld + (size_t)h * K;
  const float* decay = a.log_decay + (size_t)(q0 + c0) * hk + (size_t)h * K;
  if (tid < 4) wild[tid] = 0;
  pdl_wait();
  for (int i = tid; i < WC * (K / 4); i += WO_THREADS) {
    const int t = i / (K / 4), p = i % (K / 4);
    float* dst = sG + t * KF + p * 4;
    if (t < n) cp_async16(dst, decay + (size_t)t * hk + p * 4);
    else *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  cp_async_commit();
  auto load_rows = [&](int what, uint8_t* to) {
    for (int i = tid; i < WC * K8; i += WO_THREADS) {
      const int t = i / K8, p = i % K8;
      uint8_t* dst = to + t * RB + p * 16;
      if (t < n) cp_async16(dst, z + (size_t)t * a.ld + what * hk + p * 8);
      else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
  };
  load_rows(0, sR);
  load_rows(1, sK);
  cp_async_commit();
  cp_async_wait<1>();
  __syncthreads();
  for (int i = tid; i < 4 * K; i += WO_THREADS) {
    const int blk = i / K, d = i % K;
    float sum = 0.f;
#pragma unroll
    for (int t = blk * 16; t < blk * 16 + 16; ++t) {
      sum += fmaxf(sG[t * KF + d] * 1.4426950408889634f, DP_FLOOR);
      sG[t * KF + d] = sum;
    }
    total[i] = sum;
    if (sum < DP_RANGE) wild[blk] = 1;
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- r relative to its block's start (eight channels of a token at a time), and the bonus of the current token
  for (int i = tid; i < WC * K8; i += WO_THREADS) {
    const int t = i / K8, p = i % K8;
    const uint4 u = *reinterpret_cast<const uint4*>(sR + t * RB + p * 16);
    const uint32_t us[4] = {u.x, u.y, u.z, u.w};
    float l[8], v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) l[e] = 0.f;
    if (t & 15) delta_load8(sG + (t - 1) * KF + p * 8, l);
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const float2 f = unpack_bf16x2(us[e >> 1]);
      v[e] = f.x * delta_exp2(l[e]);
      v[e + 1] = f.y * delta_exp2(l[e + 1]);
    }
    delta_split8(v, sRR + t * RB + p * 16, sRR + HALF + t * RB + p * 16);
  }
  for (int t = warp; t < WC; t += WO_THREADS / 32) {
    float s = 0.f;
    for (int d = lane; d < K; d += 32)
      s = fmaf(__bfloat162float(reinterpret_cast<const __nv_bfloat16*>(sR + t * RB)[d]) * a.bonus[(size_t)h * K + d],
               __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(sK + t * RB)[d]), s);
    s = warp_sum(s);
    if (lane == 0) diag[t] = s;
  }
  __syncthreads();
  // ---- A, blocks of 16 x 16
  for (int task = warp; task < 10; task += WO_THREADS / 32) {
    const int mt = task < 1 ? 0 : (task < 3 ? 1 : (task < 6 ? 2 : 3)), np = task - mt * (mt + 1) / 2;
    const bool on_diag = mt == np;
    if (on_diag && wild[mt]) {
      for (int i = lane; i < 256; i += 32) {
        uint8_t* at = sA + (mt * 16 + i / 16) * WC_PROW + (np * 16 + i % 16) * 2;
        *reinterpret_cast<__nv_bfloat16*>(at) = *reinterpret_cast<__nv_bfloat16*>(at + WC * WC_PROW) = __float2bfloat16(0.f);
      }
      __syncwarp();
      for (int t = mt * 16; t < mt * 16 + 16; ++t)
        for (int s = mt * 16; s <= t; ++s) {
          float y = 0.f;
          if (s == t) {
            y = diag[t];
          } else {
            for (int d = lane; d < K; d += 32)
              y = fmaf(t < n ? __bfloat162float(z[(size_t)t * a.ld + d]) * delta_exp2(sG[(t - 1) * KF + d] - sG[s * KF + d]) : 0.f,
                       __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(sK + s * RB)[d]), y);
            y = warp_sum(y);
          }
          if (lane == 0) {
            const __nv_bfloat16 hi = __float2bfloat16(y);
            uint8_t* at = sA + t * WC_PROW + s * 2;
            *reinterpret_cast<__nv_bfloat16*>(at) = hi;
            *reinterpret_cast<__nv_bfloat16*>(at + WC * WC_PROW) = __float2bfloat16(y - __bfloat162float(hi));
          }
        }
      continue;
    }
    float acc[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const uint32_t r_at = smem_u32(sRR) + (mt * 16 + (mi & 1) * 8 + lr) * RB + (mi >> 1) * 16;
#pragma unroll 2
    for (int ks = 0; ks < KT; ++ks) {
      uint32_t ah[4], al[4];
      ldmatrix_x4(r_at + ks * 32, ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(r_at + HALF + ks * 32, al[0], al[1], al[2], al[3]);
      float2 between[2];  // logarithms of the decays from the columns' block on to the rows'
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int d = ks * 16 + 2 * t4 + 8 * j;
        between[j] = make_float2(0.f, 0.f);
        for (int i = np; i < mt; ++i) {
          const float2 v = *reinterpret_cast<const float2*>(total + i * K + d);
          between[j].x += v.x;
          between[j].y += v.y;
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {  // (column g of tile i, values 2 t4 + 8 j)
          const int s = np * 16 + 8 * i + g, d = ks * 16 + 2 * t4 + 8 * j;
          const float2 kv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sK + s * RB + d * 2));
          const float2 l = *reinterpret_cast<const float2*>(sG + s * KF + d);
          split_bf16x2(kv.x * delta_exp2(between[j].x - l.x), kv.y * delta_exp2(between[j].y - l.y), bh[j], bl[j]);
        }
        mma_bf16_16816(acc[i], ah, bl[0], bl[1]);
        mma_bf16_16816(acc[i], al, bh[0], bh[1]);
        mma_bf16_16816(acc[i], ah, bh[0], bh[1]);
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int t = mt * 16 + g + 8 * (e >> 1), s = np * 16 + 8 * i + 2 * t4;
        float v0 = acc[i][e], v1 = acc[i][e + 1];
        if (on_diag) {
          v0 = s < t ? v0 : (s == t ? diag[t] : 0.f);
          v1 = s + 1 < t ? v1 : (s + 1 == t ? diag[t] : 0.f);
        }
        uint32_t hi, lo;
        split_bf16x2(v0, v1, hi, lo);
        *reinterpret_cast<uint32_t*>(sA + t * WC_PROW + s * 2) = hi;
        *reinterpret_cast<uint32_t*>(sA + WC * WC_PROW + t * WC_PROW + s * 2) = lo;
      }
  }
  __syncthreads();
  // ---- r relative to the chunk's start, while v arrives
  load_rows(2, sV);
  cp_async_commit();
  for (int i = 16 * K8 + tid; i < WC * K8; i += WO_THREADS) {
    const int t = i / K8, p = i % K8;
    uint8_t *at_hi = sRR + t * RB + p * 16, *at_lo = at_hi + HALF;
    const uint4 uh = *reinterpret_cast<const uint4*>(at_hi), ul = *reinterpret_cast<const uint4*>(at_lo);
    const uint32_t hs[4] = {uh.x, uh.y, uh.z, uh.w}, ls[4] = {ul.x, ul.y, ul.z, ul.w};
    float l[8], v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) l[e] = 0.f;
    for (int j = 0; j < t >> 4; ++j) {
      delta_load8(total + j * K + p * 8, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) l[e] += v[e];
    }
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const float2 x0 = unpack_bf16x2(hs[e >> 1]), x1 = unpack_bf16x2(ls[e >> 1]);
      v[e] = (x0.x + x1.x) * delta_exp2(l[e]);
      v[e + 1] = (x0.y + x1.y) * delta_exp2(l[e + 1]);
    }
    delta_split8(v, at_hi, at_lo);
  }
  const int nt0 = warp * NT;  // (warps past the last value have nothing to multiply)
  constexpr int AHEAD = KT < 4 ? KT : 4;  // k-steps of the state on their way
  const uint4* ws = x.ws + (((size_t)b * x.round + blockIdx.x) * a.H + h) * (K * V / 4) + lane;
  uint4 s[AHEAD][NT];
#pragma unroll
  for (int ks = 0; ks < AHEAD; ++ks)
#pragma unroll
    for (int i = 0; i < NT; ++i) s[ks][i] = ws[((size_t)ks * (V / 8) + min(nt0 + i, V / 8 - 1)) * 32];
  cp_async_wait<0>();
  __syncthreads();
  float o[4][NT][4];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
  if (nt0 * 8 < V) {
    const uint32_t a_at = smem_u32(sA) + ((mi & 1) * 8 + lr) * WC_PROW + (mi >> 1) * 16;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t bv[NT][2];
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int nt = min(nt0 + i, V / 8 - 1);
        uint32_t d0, d1;
        ldmatrix_x4_trans(smem_u32(sV) + (ks * 16 + (mi & 1) * 8 + lr) * RB + nt * 16, bv[i][0], bv[i][1], d0, d1);
      }
#pragma unroll
      for (int m = ks; m < 4; ++m) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(a_at + m * 16 * WC_PROW + ks * 32, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(a_at + (WC + m * 16) * WC_PROW + ks * 32, al[0], al[1], al[2], al[3]);
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          mma_bf16_16816(o[m][i], al, bv[i][0], bv[i][1]);
          mma_bf16_16816(o[m][i], ah, bv[i][0], bv[i][1]);
        }
      }
    }
    const uint32_t r_at = smem_u32(sRR) + ((mi & 1) * 8 + lr) * RB + (mi >> 1) * 16;
#pragma unroll
    for (int ks = 0; ks < KT; ++ks) {
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(r_at + m * 16 * RB + ks * 32, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(r_at + HALF + m * 16 * RB + ks * 32, al[0], al[1], al[2], al[3]);
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          const uint4 v = s[ks % AHEAD][i];
          mma_bf16_16816(o[m][i], ah, v.z, v.w);
          mma_bf16_16816(o[m][i], al, v.x, v.y);
          mma_bf16_16816(o[m][i], ah, v.x, v.y);
        }
      }
      if (ks + AHEAD < KT) {
#pragma unroll
        for (int i = 0; i < NT; ++i) s[ks % AHEAD][i] = ws[((size_t)(ks + AHEAD) * (V / 8) + min(nt0 + i, V / 8 - 1)) * 32];
      }
    }
  }
  // ---- every row over its root mean square, norm and gate
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NT; ++i)
        if (nt0 + i < V / 8) ss += o[m][i][e] * o[m][i][e] + o[m][i][e + 1] * o[m][i][e + 1];
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (t4 == 0) sums[warp * WC + m * 16 + g + 8 * (e >> 1)] = ss;
    }
  uint32_t gates[4][2][NT];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int t = m * 16 + g + 8 * e;
        gates[m][e][i] = t < n && nt0 + i < V / 8 ? *reinterpret_cast<const uint32_t*>(z + (size_t)t * a.ld + 3 * hk + (nt0 + i) * 8 + 2 * t4) : 0u;
      }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int t = m * 16 + g + 8 * (e >> 1);
      if (t >= n) continue;
      float ss = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) ss += sums[w * WC + t];
      const float inv = rsqrtf(ss / (float)a.dim + a.eps);
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = (nt0 + i) * 8 + 2 * t4;
        if (nt0 + i >= V / 8) continue;
        const float2 gate = unpack_bf16x2(gates[m][e >> 1][i]);
        const float2 w = *reinterpret_cast<const float2*>(a.norm + (size_t)h * V + c);
        *reinterpret_cast<uint32_t*>(out + (size_t)t * a.ld_out + c) =
            pack_bf16x2(o[m][i][e] * inv * w.x * gate.x * delta_sigmoid_fast(gate.x), o[m][i][e + 1] * inv * w.y * gate.y * delta_sigmoid_fast(gate.y));
      }
    }
}

}  // namespace oxb
