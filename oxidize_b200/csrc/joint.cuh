// Attention on the scores of all heads together: a query head's score with a key is
//     s_g = cap tanh(q_g . k_g scale / cap)   (k over its root mean square),   s_h <- sum_g mix[h, g] s_g + bias[h, distance],
// under a softmax with a sink logit per head, in a window with kept first positions.  One cached row is key and value: row
// [width + tail] holds the key as projected, which is the value, and behind it the float that turns it into the normed key.
//
// joint_attention_simt_kernel: any type, width, page and number of heads that fits shared memory.
#pragma once
#include "attention.cuh"
#include "latent.cuh"
#include "wkv.cuh"

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

}  // namespace oxb
