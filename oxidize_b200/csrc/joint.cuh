// Attention on the scores of all heads together: a query head's score with a key is
//     s_g = cap tanh(q_g . k_g scale / cap)   (k over its root mean square),   s_h <- sum_g mix[h, g] s_g + bias[h, distance],
// under a softmax with a sink logit per head, in a window with kept first positions.  One cached row is key and value: row
// [width + tail] holds the key as projected, which is the value, and behind it the float that turns it into the normed key.
//
// joint_attention_simt_kernel: any type, width, page and number of heads that fits shared memory.
// joint_decode_kernel: one token per cluster, keys dealt out to its CTAs (decoded tokens and short portions).
// joint_prefill.cuh: long portions.
#pragma once
#include "attention.cuh"
#include "latent.cuh"

namespace oxb {

struct JointArgs {
  const void* q;            // [T, H, W], over their root mean square
  void* out;                // [T, H * W], rows ld_out apart
  int ld_out;
  float out_scale;
  const void* cache;        // layer base [blocks, G, page, W + tail]
  const int* block_tables;  // [B, max_blocks]
  const int* seq_lens;      // [B]
  const int* query_start;   // [B + 1]
  const float* sink;        // [H] or null
  const float* mix;         // [H, H] or null
  const float* bias;        // [H, distances] or null
  int distances;
  int B, max_blocks, T, H, G, W, tail, page, num_blocks, window, keep_first;
  float scale, cap;         // cap 0: scores as they are
  int max_rows;             // sequences that feed more rows belong to other kernels
};

__device__ __forceinline__ float joint_capped(const JointArgs& a, float s) { return a.cap > 0.f ? a.cap * tanhf(s / a.cap) : s; }

constexpr int JS_KEYS = 64;  // keys per round
static inline size_t joint_simt_smem(int H, int W) { return (size_t)(2 * H * W + 2 * H * JS_KEYS + H * H + 3 * H) * sizeof(float); }

// One CTA per token.  The keys a query sees are numbered 0, 1, ...: kept first positions ahead of the window, then the window.
template <typename T>
__global__ void __launch_bounds__(256) joint_attention_simt_kernel(const JointArgs a) {
  extern __shared__ float js[];
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, H = a.H, W = a.W, per = H / a.G;
  float *q = js, *acc = q + H * W, *s = acc + H * W, *p = s + H * JS_KEYS, *mix = p + H * JS_KEYS, *m = mix + H * H, *l = m + H, *corr = l + H;
  const int b = sequence_of(a.query_start, a.B, t);
  const int pos = a.seq_lens[b] - (a.query_start[b + 1] - t);
  pdl_wait();
  if (a.query_start[b + 1] - a.query_start[b] > a.max_rows) return;
  for (int i = tid; i < H * W; i += 256) {
    q[i] = lat_f32(reinterpret_cast<const T*>(a.q)[(size_t)t * H * W + i]) * a.scale;
    acc[i] = 0.f;
  }
  for (int i = tid; i < H * H; i += 256) mix[i] = a.mix != nullptr ? a.mix[i] : (i / H == i % H ? 1.f : 0.f);
  for (int h = tid; h < H; h += 256) {
    m[h] = a.sink != nullptr ? a.sink[h] : -INFINITY;
    l[h] = a.sink != nullptr ? 1.f : 0.f;
  }
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0, first = min(a.keep_first, lo), total = first + pos - lo + 1;
  const int* bt = a.block_tables + (size_t)b * a.max_blocks;
  const int ld = W + a.tail;
  auto key_row = [&](int e, int g) {
    const int k = e < first ? e : lo + e - first;
    int blk = bt[k / a.page];
    if ((unsigned)blk >= (unsigned)a.num_blocks) {
      if (lane == 0) oxb_report(OXB_BAD_BLOCK_ID, blk);
      blk = 0;
    }
    return reinterpret_cast<const T*>(a.cache) + (((size_t)blk * a.G + g) * a.page + k % a.page) * ld;
  };
  __syncthreads();
  for (int e0 = 0; e0 < total; e0 += JS_KEYS) {
    const int n = min(JS_KEYS, total - e0);
    for (int i = warp; i < n * a.G; i += 8) {
      const int e = i / a.G, g = i % a.G;
      const T* k = key_row(e0 + e, g);
      const float inv = *reinterpret_cast<const float*>(k + W);
      for (int h = g * per; h < (g + 1) * per; ++h) {
        float d = 0.f;
        for (int c = lane; c < W; c += 32) d = fmaf(q[h * W + c], lat_f32(k[c]), d);
        d = warp_sum(d);
        if (lane == 0) s[h * JS_KEYS + e] = joint_capped(a, d * inv);
      }
    }
    __syncthreads();
    for (int i = tid; i < H * n; i += 256) {
      const int h = i / n, e = i % n, k = e0 + e < first ? e0 + e : lo + e0 + e - first;
      float v = a.bias != nullptr ? a.bias[(size_t)h * a.distances + min(pos - k, a.distances - 1)] : 0.f;
      for (int g = 0; g < H; ++g) v = fmaf(mix[h * H + g], s[g * JS_KEYS + e], v);
      p[h * JS_KEYS + e] = v;
    }
    __syncthreads();
    for (int h = warp; h < H; h += 8) {
      float top = -INFINITY, sum = 0.f;
      for (int e = lane; e < n; e += 32) top = fmaxf(top, p[h * JS_KEYS + e]);
      top = fmaxf(warp_max(top), m[h]);
      for (int e = lane; e < n; e += 32) {
        const float x = expf(p[h * JS_KEYS + e] - top);
        p[h * JS_KEYS + e] = x;
        sum += x;
      }
      sum = warp_sum(sum);
      const float c = expf(m[h] - top);
      __syncwarp();
      if (lane == 0) {
        corr[h] = c;
        m[h] = top;
        l[h] = l[h] * c + sum;
      }
    }
    __syncthreads();
    for (int i = tid; i < H * W; i += 256) {
      const int h = i / W, c = i % W;
      float o = acc[i] * corr[h];
      for (int e = 0; e < n; ++e) o = fmaf(p[h * JS_KEYS + e], lat_f32(key_row(e0 + e, h / per)[c]), o);
      acc[i] = o;
    }
    __syncthreads();
  }
  T* out = reinterpret_cast<T*>(a.out) + (size_t)t * a.ld_out;
  for (int i = tid; i < H * W; i += 256) out[i] = lat_from<T>(l[i / W] > 0.f ? acc[i] * a.out_scale / l[i / W] : 0.f);
}

// ----------------------------------------------------------------------------- decoded tokens
__device__ __forceinline__ float joint_exp2(float x) {  // 0 where that is no normal number
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float joint_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// cap tanh(f s / cap) for scores of bfloat16 factors, tanh(x) = 1 - 2 / (1 + exp(2 x)): `f` carries the factor 2 log2(e) / cap
// (joint_factor), absolute error about 1e-7 cap.
struct JointCap {
  float cap, factor;
};
__device__ __forceinline__ JointCap joint_cap(const JointArgs& a) {
  return JointCap{a.cap, a.cap > 0.f ? a.scale * 2.f * 1.4426950408889634f / a.cap : a.scale};
}
__device__ __forceinline__ float joint_capped_of(float x, const JointCap& c) { return fmaf(-2.f * c.cap, joint_rcp(1.f + joint_exp2(x)), c.cap); }
__device__ __forceinline__ float joint_capped_fast(float s, float f, const JointCap& c) {
  return c.cap > 0.f ? joint_capped_of(s * f, c) : s * f;
}

// A page of one key head: 16 rows of HD values and their tails, as it stands in the cache (rows HD * 2 + 16 bytes apart, which
// ldmatrix reads without bank conflicts).  One warp.
template <int HD>
__device__ __forceinline__ void joint_load_page(uint8_t* stage, const JointArgs& a, int blk, int g, int lane) {
  constexpr int BYTES = 16 * (HD * 2 + 16);
  const uint8_t* src = reinterpret_cast<const uint8_t*>(a.cache) + ((size_t)blk * a.G + g) * BYTES;
#pragma unroll
  for (int c = lane; c < BYTES / 16; c += 32) cp_async16(stage + c * 16, src + c * 16);
}

constexpr int JD_WARPS = 8, JD_PAGES = 4, JD_KEYS = 16 * JD_PAGES, JD_SROW = JD_KEYS + 4, JD_PROW = JD_KEYS + 8;
struct JointDecodeSmem {
  int s, o, mix, p, stat, total;  // byte offsets; the warps' pages come first
};
// Whether a warp's pages of a round stay in shared memory, and how many warps share a key head.
__host__ __device__ inline bool joint_decode_resident(int G, int HD) { return G <= JD_WARPS && HD <= 128; }
__host__ __device__ inline int joint_decode_parts(int G, bool res) { return res && G < JD_WARPS ? JD_WARPS / G : 1; }
__host__ __device__ inline JointDecodeSmem joint_decode_smem(int H, int G, int HD) {
  const bool res = joint_decode_resident(G, HD);
  const int parts = joint_decode_parts(G, res), h4 = (H + 3) / 4 * 4;
  JointDecodeSmem m;
  m.s = JD_WARPS * (res ? JD_PAGES : 2) * 16 * (HD * 2 + 16);
  m.o = m.s + H * JD_SROW * 4;
  m.mix = m.o + parts * H * HD * 4;
  m.p = m.mix + H * h4 * 4;
  m.stat = m.p + (H * JD_PROW * 2 + 15) / 16 * 16;
  m.total = m.stat + 3 * h4 * 4;
  return m;
}

// grid (splits, T), the splits of a token one cluster.  A round covers 64 keys: every warp takes the scores of its key heads
// (where there are fewer than eight, of some of their pages), the CTA mixes them and takes the softmax step, and every warp
// weighs its pages as values.  RES (up to eight key heads of up to 128 values): a warp's pages of a round stay in shared memory in between, and those
// of the next round take their places one by one; else they pass through two places and are read a second time, out of the L2.
template <int HD, bool RES>
__global__ void __launch_bounds__(JD_WARPS * 32, (HD <= 128 && !RES) ? 2 : 1) joint_decode_kernel(const JointArgs a) {
  constexpr int ROWB = HD * 2 + 16, STAGE = 16 * ROWB, KS = HD / 16, NT = HD / 8, STAGES = RES ? JD_PAGES : 2;
  extern __shared__ __align__(16) uint8_t jd_smem[];
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3, lr = lane & 7;
  const int t = blockIdx.y, split = blockIdx.x, splits = gridDim.x;
  const int H = a.H, G = a.G, per = H / G, h4 = (H + 3) / 4 * 4, parts = joint_decode_parts(G, RES), units = G * parts;
  const int b = sequence_of(a.query_start, a.B, t), rows = a.query_start[b + 1] - a.query_start[b];
  if (rows > a.max_rows) {  // (the whole cluster leaves)
    pdl_wait();
    return;
  }
  const int pos = a.seq_lens[b] - (a.query_start[b + 1] - t);
  const JointDecodeSmem sm = joint_decode_smem(H, G, HD);
  float *sS = reinterpret_cast<float*>(jd_smem + sm.s), *sO = reinterpret_cast<float*>(jd_smem + sm.o), *sMix = reinterpret_cast<float*>(jd_smem + sm.mix);
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(jd_smem + sm.p);
  float *m_run = reinterpret_cast<float*>(jd_smem + sm.stat), *l_run = m_run + h4, *corr = l_run + h4;
  uint8_t* ring = jd_smem + warp * STAGES * STAGE;
  for (int i = tid; i < H * h4; i += JD_WARPS * 32) {  // [g][h], in binary logarithms
    const int g = i / h4, h = i % h4;
    sMix[i] = h < H ? (a.mix != nullptr ? a.mix[h * H + g] : (g == h ? 1.f : 0.f)) * 1.4426950408889634f : 0.f;
  }
  for (int i = tid; i < parts * H * HD; i += JD_WARPS * 32) sO[i] = 0.f;
  if (tid < h4) {
    m_run[tid] = -INFINITY;
    l_run[tid] = 0.f;
  }
  // the pages this token sees: those of kept first positions ahead of the window's, then the window's
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0, page_lo = lo >> 4;
  const int kept = min((a.keep_first + 15) >> 4, page_lo), n_pages = pos < 0 ? 0 : kept + (pos >> 4) - page_lo + 1;
  const int share = (n_pages + splits - 1) / splits, p0 = split * share, p1 = min(n_pages, p0 + share);
  const int* bt = a.block_tables + (size_t)b * a.max_blocks;
  auto page_of = [&](int i) { return i < kept ? i : page_lo + i - kept; };
  const JointCap cap = joint_cap(a);
  auto load = [&](int page, int u, int slot) {
    int blk = bt[page_of(page)];
    if ((unsigned)blk >= (unsigned)a.num_blocks) {
      if (lane == 0) oxb_report(OXB_BAD_BLOCK_ID, blk);
      blk = 0;
    }
    joint_load_page<HD>(ring + slot * STAGE, a, blk, u / parts, lane);
  };
  uint32_t qf[KS][4];
  auto load_q = [&](int g) {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.q) + ((size_t)t * H + g * per) * HD + 2 * t4;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const bool on = g8 + 8 * i < per;
        const __nv_bfloat16* qp = q + (size_t)(on ? g8 + 8 * i : 0) * HD + ks * 16;
        qf[ks][i] = on ? *reinterpret_cast<const uint32_t*>(qp) : 0u;
        qf[ks][i + 2] = on ? *reinterpret_cast<const uint32_t*>(qp + 8) : 0u;
      }
  };
  auto scores = [&](int g, int p, int slot) {
    const uint8_t* st = ring + slot * STAGE;
    const uint32_t addr = smem_u32(st) + ((mi >> 1) * 8 + lr) * ROWB + (mi & 1) * 16;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4(addr + ks * 32, b0, b1, b2, b3);
      mma_bf16_16816(s[0], qf[ks], b0, b1);
      mma_bf16_16816(s[1], qf[ks], b2, b3);
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int key = nt * 8 + 2 * t4;
      const float f0 = *reinterpret_cast<const float*>(st + key * ROWB + HD * 2) * cap.factor;
      const float f1 = *reinterpret_cast<const float*>(st + (key + 1) * ROWB + HD * 2) * cap.factor;
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (g8 + 8 * i < per)
          *reinterpret_cast<float2*>(sS + (g * per + g8 + 8 * i) * JD_SROW + p * 16 + key) =
              make_float2(joint_capped_fast(s[nt][2 * i], f0, cap), joint_capped_fast(s[nt][2 * i + 1], f1, cap));
    }
  };
  float o[NT][4];
  auto clear = [&]() {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
  };
  auto values = [&](int g, int p, int slot) {
    uint32_t pf[4];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const bool on = g8 + 8 * i < per;
      const __nv_bfloat16* src = sP + (g * per + (on ? g8 + 8 * i : 0)) * JD_PROW + p * 16 + 2 * t4;
      pf[i] = on ? *reinterpret_cast<const uint32_t*>(src) : 0u;
      pf[i + 2] = on ? *reinterpret_cast<const uint32_t*>(src + 8) : 0u;
    }
    const uint32_t addr = smem_u32(ring + slot * STAGE) + ((mi & 1) * 8 + lr) * ROWB + (mi >> 1) * 16;
#pragma unroll
    for (int nt = 0; nt < NT; nt += 2) {
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4_trans(addr + nt * 16, b0, b1, b2, b3);
      mma_bf16_16816(o[nt], pf, b0, b1);
      mma_bf16_16816(o[nt + 1], pf, b2, b3);
    }
  };
  // O <- corr O + o; RES: a warp has one unit, whose O stays in o
  auto flush = [&](int unit) {
    const int g = unit / parts;
    float* dst = sO + ((size_t)(unit % parts) * H + g * per) * HD + 2 * t4;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = g8 + 8 * i;
      if (r >= per) continue;
      const float c = RES ? 0.f : corr[g * per + r];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        float2* at = reinterpret_cast<float2*>(dst + r * HD + nt * 8);
        const float2 x = RES ? make_float2(0.f, 0.f) : *at;
        *at = make_float2(fmaf(c, x.x, o[nt][2 * i]), fmaf(c, x.y, o[nt][2 * i + 1]));
      }
    }
  };
  // ---- mixing and softmax of a round: a warp has four heads and all keys, a lane keys `lane` and `lane` + 32
  auto mix_round = [&](int r0, int npg) {
    bool ok[2];
    int dist[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int pg = (lane >> 4) + 2 * j, key = page_of(r0 + min(pg, npg - 1)) * 16 + (lane & 15);
      ok[j] = pg < npg && key <= pos && (a.window <= 0 || key > pos - a.window || key < a.keep_first);
      dist[j] = min(max(pos - key, 0), a.distances - 1);
    }
    for (int h0 = 4 * warp; h0 < H; h0 += 4 * JD_WARPS) {
      float v[2][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float* bias = a.bias + (size_t)min(h0 + i, H - 1) * a.distances;
#pragma unroll
        for (int j = 0; j < 2; ++j) v[j][i] = a.bias != nullptr ? bias[dist[j]] * 1.4426950408889634f : 0.f;
      }
#pragma unroll 8
      for (int g = 0; g < H; ++g) {
        const float4 w = *reinterpret_cast<const float4*>(sMix + g * h4 + h0);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float x = sS[g * JD_SROW + lane + 32 * j];
          v[j][0] = fmaf(w.x, x, v[j][0]);
          v[j][1] = fmaf(w.y, x, v[j][1]);
          v[j][2] = fmaf(w.z, x, v[j][2]);
          v[j][3] = fmaf(w.w, x, v[j][3]);
        }
      }
      float old[4], top[4], sum[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[0][i] = ok[0] ? v[0][i] : -INFINITY;
        v[1][i] = ok[1] ? v[1][i] : -INFINITY;
        old[i] = m_run[h0 + i];  // (rows up to h4 exist)
        top[i] = fmaxf(v[0][i], v[1][i]);
      }
#pragma unroll
      for (int d = 16; d > 0; d >>= 1)
#pragma unroll
        for (int i = 0; i < 4; ++i) top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], d));
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        top[i] = fmaxf(top[i], old[i]);
        const float base = top[i] == -INFINITY ? 0.f : top[i];
        v[0][i] = joint_exp2(v[0][i] - base);
        v[1][i] = joint_exp2(v[1][i] - base);
        old[i] = joint_exp2(old[i] - base);
        sum[i] = v[0][i] + v[1][i];
      }
#pragma unroll
      for (int d = 16; d > 0; d >>= 1)
#pragma unroll
        for (int i = 0; i < 4; ++i) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], d);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (h0 + i >= H) continue;
        sP[(h0 + i) * JD_PROW + lane] = __float2bfloat16(v[0][i]);
        sP[(h0 + i) * JD_PROW + lane + 32] = __float2bfloat16(v[1][i]);
        if (lane == 0) {
          m_run[h0 + i] = top[i];
          l_run[h0 + i] = l_run[h0 + i] * old[i] + sum[i];
          corr[h0 + i] = old[i];
        }
      }
      __syncwarp();
    }
  };
  __syncthreads();
  pdl_wait();
  if constexpr (RES) {
    const int u = warp, g = u / parts, part = u % parts;
    const bool works = u < units;
    clear();
    // page k of a round (k-th of this warp's) lies in place k
    auto mine = [&](int k, int r0) { return works && k * parts + part < min(JD_PAGES, p1 - r0); };
#pragma unroll
    for (int k = 0; k < JD_PAGES; ++k) {
      if (p0 < p1 && mine(k, p0)) load(p0 + k * parts + part, u, k);
      cp_async_commit();
    }
    if (works) load_q(g);
    for (int r0 = p0; r0 < p1; r0 += JD_PAGES) {
      const int npg = min(JD_PAGES, p1 - r0);
      cp_async_wait<3>();
      __syncwarp();
      if (mine(0, r0)) scores(g, part, 0);
      cp_async_wait<2>();
      __syncwarp();
      if (mine(1, r0)) scores(g, parts + part, 1);
      cp_async_wait<1>();
      __syncwarp();
      if (mine(2, r0)) scores(g, 2 * parts + part, 2);
      cp_async_wait<0>();
      __syncwarp();
      if (mine(3, r0)) scores(g, 3 * parts + part, 3);
      __syncthreads();
      mix_round(r0, npg);
      __syncthreads();
      if (works) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          if (g8 + 8 * i >= per) continue;
          const float c = corr[g * per + g8 + 8 * i];
#pragma unroll
          for (int nt = 0; nt < NT; ++nt) {
            o[nt][2 * i] *= c;
            o[nt][2 * i + 1] *= c;
          }
        }
      }
#pragma unroll
      for (int k = 0; k < JD_PAGES; ++k) {
        if (mine(k, r0)) values(g, k * parts + part, k);
        __syncwarp();
        if (r0 + JD_PAGES < p1 && mine(k, r0 + JD_PAGES)) load(r0 + JD_PAGES + k * parts + part, u, k);
        cp_async_commit();
      }
    }
    if (works) flush(u);
  } else {
    int slot = 0;
    auto first_unit = [&](int& u, int& p) {
      u = warp;
      p = 0;
    };
    auto next_unit = [&](int npg, int& u, int& p) {
      if (++p >= npg) {
        u += JD_WARPS;
        p = 0;
      }
    };
    if (p0 < p1 && warp < units) load(p0, warp, 0);
    cp_async_commit();
    for (int r0 = p0; r0 < p1; r0 += JD_PAGES) {
      const int npg = min(JD_PAGES, p1 - r0);
      int u, p, held = -1;
      first_unit(u, p);
      while (u < units) {
        int nu = u, np = p;
        next_unit(npg, nu, np);
        if (nu < units) load(r0 + np, nu, slot ^ 1);
        cp_async_commit();
        if (u != held) load_q(held = u);
        cp_async_wait<1>();
        __syncwarp();
        scores(u, p, slot);
        __syncwarp();
        slot ^= 1;
        u = nu;
        p = np;
      }
      if (warp < units) load(r0, warp, slot);  // the first page of the values is on its way during the mixing
      cp_async_commit();
      __syncthreads();
      mix_round(r0, npg);
      __syncthreads();
      first_unit(u, p);
      while (u < units) {
        int nu = u, np = p;
        next_unit(npg, nu, np);
        if (nu < units) load(r0 + np, nu, slot ^ 1);
        cp_async_commit();
        if (p == 0) clear();
        cp_async_wait<1>();
        __syncwarp();
        values(u, p, slot);
        __syncwarp();
        slot ^= 1;
        if (nu != u) flush(u);
        u = nu;
        p = np;
      }
      if (r0 + JD_PAGES < p1 && warp < units) load(r0 + JD_PAGES, warp, slot);
      cp_async_commit();
      // (the next round's scores overwrite sS, which nobody reads any more; its mixing starts behind a barrier)
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  if (parts > 1) {
    for (int i = tid; i < H * HD; i += JD_WARPS * 32) {
      float s = sO[i];
      for (int k = 1; k < parts; ++k) s += sO[(size_t)k * H * HD + i];
      sO[i] = s;
    }
    __syncthreads();
  }
  if (splits > 1) cluster_sync_all();
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)t * a.ld_out;
  for (int i = split * JD_WARPS * 32 + tid; i < H * HD / 4; i += splits * JD_WARPS * 32) {
    const int h = 4 * i / HD;
    const float sink = a.sink != nullptr ? a.sink[h] * 1.4426950408889634f : -INFINITY;
    float4 v;
    float L, M = sink;
    if (splits == 1) {
      M = fmaxf(M, m_run[h]);
      const float w = m_run[h] == -INFINITY ? 0.f : exp2f(m_run[h] - M);
      v = *reinterpret_cast<const float4*>(sO + 4 * i);
      v = make_float4(w * v.x, w * v.y, w * v.z, w * v.w);
      L = w * l_run[h];
    } else {
      const uint32_t m_at = smem_u32(m_run + h), l_at = smem_u32(l_run + h), o_at = smem_u32(sO + 4 * i);
#pragma unroll 4
      for (int r = 0; r < splits; ++r) M = fmaxf(M, dsmem_ld_f32(dsmem_map(m_at, r)));
      v = make_float4(0.f, 0.f, 0.f, 0.f);
      L = 0.f;
#pragma unroll 4
      for (int r = 0; r < splits; ++r) {
        const float m = dsmem_ld_f32(dsmem_map(m_at, r)), w = m == -INFINITY ? 0.f : exp2f(m - M);
        const float4 x = dsmem_ld_f32x4(dsmem_map(o_at, r));
        L = fmaf(w, dsmem_ld_f32(dsmem_map(l_at, r)), L);
        v = make_float4(fmaf(w, x.x, v.x), fmaf(w, x.y, v.y), fmaf(w, x.z, v.z), fmaf(w, x.w, v.w));
      }
    }
    if (sink != -INFINITY) L += exp2f(sink - M);
    const float inv = L > 0.f ? a.out_scale / L : 0.f;
    *reinterpret_cast<uint2*>(out + 4 * i) = make_uint2(pack_bf16x2(v.x * inv, v.y * inv), pack_bf16x2(v.z * inv, v.w * inv));
  }
  if (splits > 1) cluster_sync_all();  // every peer has finished reading this CTA's partial
}

}  // namespace oxb
