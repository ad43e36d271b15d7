// Grouped-query attention of models that list their layers: what surrounds the attention step (norms, rotation, cache rows),
// the plain form of the step itself, and the elementwise and routing pieces of their feed-forward blocks.
//
// Heads are stored with `width` values each, the first `dim` of which are the head's own and the rest zeros.
#pragma once
#include "latent.cuh"
#include "residual_norm.cuh"

namespace oxb {

struct HeadPrepArgs {
  const void* z;        // [T, ld]: q (H heads), k (G heads), v (G heads)
  int ld;
  const int* positions; // [T]
  const int* slots;     // [T] block * page + offset, < 0: no cache row
  const float* cos_sin; // [max_pos, rot]: cos of the rot / 2 pairs, then sin
  int max_pos, rot, pairing /*0 split-half, 1 adjacent*/;
  const float *q_norm, *k_norm;  // norm weights, or null: [width] (per head) or [heads * width] (over the projection)
  int full;             // 1: one norm over all heads
  float eps;
  int H, G, dim, width;
  void* q;              // [T, H, width]
  void* cache;          // layer base [blocks, G, 2, page, width]
  int page, num_blocks;
  int per_cta;          // heads (of q, k and v together) per CTA
  float temp_coef, temp_every;  // queries times 1 + temp_coef ln(floor((pos + 1) / temp_every) + 1); 0: off
  const void* v_first;  // values that are mixed into this layer's, rows ld_first apart, heads first_width apart; or null
  int ld_first, first_width, v_dim;
  const float* v_mix;   // [1]: their share
  int unit;             // 1: queries and keys over their root mean square per head, without a weight
  // 1: there are no values; the cache has one row per key head, [blocks, G, page, width + tail], the key as projected and behind
  // it the float that turns it into the normed key
  int shared, tail;
};

constexpr int HEAD_PREP_WARPS = 8;

template <int N>
__device__ __forceinline__ void head_load(const float* p, float* v) {
#pragma unroll
  for (int j = 0; j < N; ++j) v[j] = p[j];
}
template <int N>
__device__ __forceinline__ void head_load(const __nv_bfloat16* p, float* v) {
  if constexpr (N == 1) {
    v[0] = __bfloat162float(*p);
  } else if constexpr (N == 2) {
    const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p));
    v[0] = f.x;
    v[1] = f.y;
  } else {
#pragma unroll
    for (int j = 0; j < N; j += 4) {
      const uint2 u = *reinterpret_cast<const uint2*>(p + j);
      const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
      v[j] = a.x;
      v[j + 1] = a.y;
      v[j + 2] = b.x;
      v[j + 3] = b.y;
    }
  }
}
template <int N>
__device__ __forceinline__ void head_store(float* p, const float* v) {
#pragma unroll
  for (int j = 0; j < N; ++j) p[j] = v[j];
}
template <int N>
__device__ __forceinline__ void head_store(__nv_bfloat16* p, const float* v) {
  if constexpr (N == 1) {
    *p = __float2bfloat16(v[0]);
  } else if constexpr (N == 2) {
    *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v[0], v[1]);
  } else {
#pragma unroll
    for (int j = 0; j < N; j += 4)
      *reinterpret_cast<uint2*>(p + j) = make_uint2(pack_bf16x2(v[j], v[j + 1]), pack_bf16x2(v[j + 2], v[j + 3]));
  }
}

// Rotation of the VPL values from `d0` on of a head that stands in shared memory.
template <int VPL>
__device__ __forceinline__ void head_rotate(const float* row, const float* cs, int d0, int rot, int pairing, float* v) {
  const int half = rot >> 1;
#pragma unroll
  for (int j = 0; j < VPL; ++j) {
    const int d = d0 + j;
    if (d >= rot) continue;
    int p, o;
    bool first;
    if (pairing == 0) {
      first = d < half;
      p = first ? d : d - half;
      o = first ? d + half : p;
    } else {
      first = (d & 1) == 0;
      p = d >> 1;
      o = d ^ 1;
    }
    const float c = cs[p], s = cs[half + p];
    v[j] = first ? v[j] * c - row[o] * s : v[j] * c + row[o] * s;
  }
}

// grid (T, head groups), one warp per head at a time, VPL neighbouring values per lane (32 * VPL >= width).  A norm over all
// heads is summed up by every CTA that needs it.  Dynamic shared memory: one row of floats per warp.
template <typename T, int VPL>
__global__ void __launch_bounds__(HEAD_PREP_WARPS * 32) head_prep_kernel(const HeadPrepArgs a) {
  extern __shared__ float hp_rows[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int W = a.width, d0 = lane * VPL;
  const T* z = reinterpret_cast<const T*>(a.z) + (size_t)t * a.ld;
  const bool norm = a.unit || a.q_norm != nullptr, on = d0 < W;
  const int h0 = blockIdx.y * a.per_cta, h1 = min(h0 + a.per_cta, a.H + (a.shared ? 1 : 2) * a.G);
  float inv_q = 0.f, inv_k = 0.f;
  if (norm && !a.unit && a.full && h0 < a.H + a.G) {
    float sq = 0.f, sk = 0.f;
    const int f0 = h0 < a.H ? 0 : a.H, f1 = h1 > a.H ? a.H + a.G : a.H;
#pragma unroll 4
    for (int h = f0 + warp; h < f1; h += HEAD_PREP_WARPS) {
      float v[VPL], s = 0.f;
      if (on) {
        head_load<VPL>(z + (size_t)h * W + d0, v);
#pragma unroll
        for (int j = 0; j < VPL; ++j) s += v[j] * v[j];
      }
      if (h < a.H) sq += s;
      else sk += s;
    }
    inv_q = rsqrtf(block_sum(sq, red) / (float)(a.H * a.dim) + a.eps);
    inv_k = rsqrtf(block_sum(sk, red) / (float)(a.G * a.dim) + a.eps);
  }
  int pos = a.positions[t];
  pos = pos < 0 ? 0 : (pos >= a.max_pos ? a.max_pos - 1 : pos);
  const float* cs = a.cos_sin + (size_t)pos * a.rot;
  const int slot = a.slots[t], blk = slot < 0 ? -1 : slot / a.page, off = slot < 0 ? 0 : slot % a.page;
  const float temp = a.temp_coef != 0.f ? 1.f + a.temp_coef * logf(floorf((float)(a.positions[t] + 1) / a.temp_every) + 1.f) : 1.f;
  const bool keep = blk >= 0 && blk < a.num_blocks;
  if (blk >= a.num_blocks && threadIdx.x == 0 && blockIdx.y == 0) oxb_report(OXB_BAD_SLOT, slot);  // never write outside the pool
  float* row = hp_rows + warp * W;
  for (int h = h0 + warp; h < h1; h += HEAD_PREP_WARPS) {
    const bool is_q = h < a.H, is_v = h >= a.H + a.G;
    if (!is_q && !keep) continue;
    float v[VPL];
#pragma unroll
    for (int j = 0; j < VPL; ++j) v[j] = 0.f;
    if (on) head_load<VPL>(z + (size_t)h * W + d0, v);
    float inv = is_q ? inv_q : inv_k;
    if (!is_v) {
      if (norm) {
        if (a.unit || !a.full) {
          float s = 0.f;
#pragma unroll
          for (int j = 0; j < VPL; ++j) s += v[j] * v[j];
          inv = rsqrtf(warp_sum(s) / (float)a.dim + a.eps);
        }
        if (a.unit) {
          if (!a.shared || is_q) {
#pragma unroll
            for (int j = 0; j < VPL; ++j) v[j] *= inv;
          }
        } else {
          const float* w = (is_q ? a.q_norm : a.k_norm) + (a.full ? (size_t)(is_q ? h : h - a.H) * W : 0);
          if (on) {
#pragma unroll
            for (int j = 0; j < VPL; ++j) v[j] *= inv * w[d0 + j];
          }
        }
      }
      if (on && d0 < a.rot) head_store<VPL>(row + d0, v);
      __syncwarp();
      if (on) head_rotate<VPL>(row, cs, d0, a.rot, a.pairing, v);
      __syncwarp();
      if (is_q) {
#pragma unroll
        for (int j = 0; j < VPL; ++j) v[j] *= temp;
      }
    }
    if (!on) continue;
    if (is_v && a.v_first != nullptr) {
      const float mix = *a.v_mix;
      const T* f = reinterpret_cast<const T*>(a.v_first) + (size_t)t * a.ld_first + (size_t)(h - a.H - a.G) * a.first_width;
#pragma unroll
      for (int j = 0; j < VPL; ++j)
        if (d0 + j < a.v_dim) v[j] = (1.f - mix) * v[j] + mix * lat_f32(f[d0 + j]);
    }
    T* dst;
    if (is_q) {
      dst = reinterpret_cast<T*>(a.q) + ((size_t)t * a.H + h) * W;
    } else if (a.shared) {
      dst = reinterpret_cast<T*>(a.cache) + (((size_t)blk * a.G + h - a.H) * a.page + off) * (W + a.tail);
      if (lane == 0) *reinterpret_cast<float*>(dst + W) = inv;
    } else {
      const int g = is_v ? h - a.H - a.G : h - a.H;
      dst = reinterpret_cast<T*>(a.cache) + ((((size_t)blk * a.G + g) * 2 + is_v) * a.page + off) * W;
    }
    head_store<VPL>(dst + d0, v);
  }
}

struct GqaSimtArgs {
  const void* q;            // [T, H, width]
  void* out;                // [T, H * width], rows ld_out apart
  const void* cache;        // layer base [blocks, G, 2, page, width]
  const int* block_tables;  // [B, max_blocks]
  const int* seq_lens;      // [B]
  const int* query_start;   // [B + 1]
  const float* sink;        // [H] or null
  int B, max_blocks, T, H, G, width, page, num_blocks, window, ld_out;
  float scale, out_scale;
  HeadGate gate;
};

// The plain attention step (any type, width and page): one warp per (token, head), keys one after the other; NC * 32 >= width.
template <typename T, int NC>
__global__ void __launch_bounds__(128) gqa_attention_simt_kernel(const GqaSimtArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int task = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (task >= a.T * a.H) return;
  const int t = task / a.H, h = task % a.H, g = h / (a.H / a.G);
  int b = 0, hi_b = a.B - 1;  // the sequence that holds row t
  while (b < hi_b) {
    const int mid = (b + hi_b + 1) >> 1;
    if (a.query_start[mid] <= t) b = mid;
    else hi_b = mid - 1;
  }
  const int pos = a.seq_lens[b] - (a.query_start[b + 1] - t);  // position of row t
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const T* q = reinterpret_cast<const T*>(a.q) + ((size_t)t * a.H + h) * a.width;
  float qv[NC], acc[NC];
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int d = lane + 32 * i;
    qv[i] = d < a.width ? lat_f32(q[d]) * a.scale : 0.f;
    acc[i] = 0.f;
  }
  float m = a.sink != nullptr ? a.sink[h] : -INFINITY;
  float l = a.sink != nullptr ? 1.f : 0.f;
  const int* bt = a.block_tables + (size_t)b * a.max_blocks;
  for (int k = lo; k <= pos; ++k) {
    int blk = bt[k / a.page];
    if ((unsigned)blk >= (unsigned)a.num_blocks) {
      if (lane == 0) oxb_report(OXB_BAD_BLOCK_ID, blk);
      blk = 0;
    }
    const T* kr = reinterpret_cast<const T*>(a.cache) + (((size_t)blk * a.G + g) * 2 * a.page + k % a.page) * a.width;
    const T* vr = kr + (size_t)a.page * a.width;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int d = lane + 32 * i;
      if (d < a.width) s += qv[i] * lat_f32(kr[d]);
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s);
    const float c = expf(m - mn), p = expf(s - mn);  // m is -inf before the first key only
    l = l * c + p;
    m = mn;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int d = lane + 32 * i;
      acc[i] = acc[i] * c + (d < a.width ? p * lat_f32(vr[d]) : 0.f);
    }
  }
  float inv = l > 0.f ? a.out_scale / l : 0.f;
  const T* gates = a.gate.rows == nullptr ? nullptr : reinterpret_cast<const T*>(a.gate.rows) + (size_t)t * a.gate.ld;
  if (gates != nullptr && !a.gate.per_value) inv *= head_gate_of(lat_f32(gates[h]));
  T* o = reinterpret_cast<T*>(a.out) + (size_t)t * a.ld_out + (size_t)h * a.width;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int d = lane + 32 * i;
    if (d < a.width)
      o[d] = lat_from<T>(acc[i] * inv * (gates != nullptr && a.gate.per_value ? head_gate_of(lat_f32(gates[h * a.width + d])) : 1.f));
  }
}

// ----------------------------------------------------------------------------- feed-forward pieces in float32
// silu(gate) * up of [T, 2I] rows
static __global__ void silu_mul_f32_kernel(const float* __restrict__ gu, float* __restrict__ out, const int* __restrict__ n_rows,
                                           int T, int I) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t total = (size_t)(n_rows != nullptr ? *n_rows : T) * I;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / I, c = i % I;
    const float g = gu[t * 2 * I + c];
    out[i] = g / (1.f + expf(-g)) * gu[t * 2 * I + I + c];
  }
}

// out[t] = sum_k w[t, k] * y[inv[t, k]] (+ shared) over H values; rows of y are ld apart
static __global__ void moe_combine_f32_kernel(const float* __restrict__ y, int ld, const int* __restrict__ inv,
                                              const float* __restrict__ w, int k, const float* __restrict__ shared,
                                              float* __restrict__ out, int H) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float acc = shared != nullptr ? shared[(size_t)t * H + i] : 0.f;
    for (int j = 0; j < k; ++j) {
      const int r = inv[(size_t)t * k + j];
      if (r >= 0) acc += w[(size_t)t * k + j] * y[(size_t)r * ld + i];
    }
    out[(size_t)t * H + i] = acc;
  }
}

// ----------------------------------------------------------------------------- router logits
// logits [T, E] float32 = X [T, K] . W [E, K]^T in bf16 products with float32 sums that are never rounded to 16 bits.
// A CTA owns 16 tokens x 8 NT experts; its eight warps share the inner dimension (steps of 16) and meet in shared memory.
__device__ __forceinline__ void router_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int NT>
__global__ void __launch_bounds__(256)
router_logits_kernel(const __nv_bfloat16* __restrict__ X, const __nv_bfloat16* __restrict__ W, float* __restrict__ out, int T, int E,
                     int K) {
  __shared__ float part[8][16][8 * NT + 1];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int t0 = blockIdx.x * 16, e0 = blockIdx.y * 8 * NT;
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
  pdl_wait();
  // values 2 t4 .. and 2 t4 + 8 .. of a k-step; which k a lane's values are is free as long as both operands agree, so a
  // lane reads four neighbouring ones: [4 t4, 4 t4 + 4)
  const __nv_bfloat16 *x0 = X + (size_t)min(t0 + g, T - 1) * K + 4 * t4, *x1 = X + (size_t)min(t0 + g + 8, T - 1) * K + 4 * t4;
  const __nv_bfloat16* w[NT];
#pragma unroll
  for (int n = 0; n < NT; ++n) w[n] = W + (size_t)min(e0 + 8 * n + g, E - 1) * K + 4 * t4;
#pragma unroll 4
  for (int k = warp * 16; k < K; k += 128) {
    const uint2 a0 = *reinterpret_cast<const uint2*>(x0 + k), a1 = *reinterpret_cast<const uint2*>(x1 + k);
    const uint32_t a[4] = {a0.x, a1.x, a0.y, a1.y};
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const uint2 b = *reinterpret_cast<const uint2*>(w[n] + k);
      router_mma(acc[n], a, b.x, b.y);
    }
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) part[warp][g + 8 * (i >> 1)][8 * n + 2 * t4 + (i & 1)] = acc[n][i];
  __syncthreads();
  for (int i = threadIdx.x; i < 16 * 8 * NT; i += 256) {
    const int r = i / (8 * NT), c = i % (8 * NT);
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) s += part[j][r][c];
    if (t0 + r < T && e0 + c < E) out[(size_t)(t0 + r) * E + e0 + c] = s;
  }
}

// Any inner size: one warp per (token, expert).
template <typename T>
__global__ void __launch_bounds__(256)
router_logits_any_kernel(const T* __restrict__ X, const T* __restrict__ W, float* __restrict__ out, int rows, int E, int K) {
  pdl_launch_dependents();
  pdl_wait();
  const int task = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (task >= rows * E) return;
  const T *x = X + (size_t)(task / E) * K, *w = W + (size_t)(task % E) * K;
  float s = 0.f;
  for (int k = lane; k < K; k += 32) s += lat_f32(x[k]) * lat_f32(w[k]);
  s = warp_sum(s);
  if (lane == 0) out[task] = s;
}

}  // namespace oxb
