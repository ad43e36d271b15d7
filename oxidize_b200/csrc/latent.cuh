// Latent attention over a paged cache of shared rows: what surrounds the matrix products of one layer.
//
// A cached row is [latent (rank values, padded to a multiple of 16) | rotated key part (padded likewise)], one per token,
// shared by all heads.  latent_prep_kernel turns a layer's projections into this step's rows and into the queries;
// latent_attention_simt_kernel is the plain form of the attention step (any type and size: the float32 path), the
// tensor-core forms are in latent_mma.cuh.  A query may be limited to a window of latest positions, and a per-head sink
// logit may join the softmax denominator.
#pragma once
#include "common.cuh"

namespace oxb {

__device__ __forceinline__ float lat_f32(float v) { return v; }
__device__ __forceinline__ float lat_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T lat_from(float v);
template <>
__device__ __forceinline__ float lat_from<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 lat_from<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

struct LatentPrepArgs {
  const void* qkv;      // [T, ld]: H * (nope + rot) query values, then (where rows are written) rank + rot values
  int ld;
  const int* positions; // [T]
  const int* slots;     // [T] block * page + offset (< 0: no row), or null: this layer writes no rows
  const float* cos_sin; // [max_pos, rot]: cos of the rot / 2 pairs, then sin
  int max_pos, rot, pairing /*0 split-half, 1 adjacent*/;
  const float* norm_w;  // [rank]
  float eps;
  int T, H, nope, rank, pad, width;  // pad: first value of the rotated part of a row, width: values per row
  void* q_nope;         // absorbed form: [H, T, nope_ld], the operand of the per-head products with W_uk
  int nope_ld;
  void* q_rows;         // absorbed form: [T, H, width], of which the rotated part is written here
  void* q_full;         // expanded form (instead of the two above): [T, H, full_ld], the rotated part at full_rot, zeros elsewhere
  int full_ld, full_rot;
  void* cache;          // layer base [blocks, page, width]
  int page, num_blocks;
  int vec8;             // sizes and strides allow pieces of eight values (bf16)
};

constexpr int LAT_PREP_HEADS = 8;  // query heads per CTA

// element i of the rotation of v[0..rot)
template <typename T>
__device__ __forceinline__ float lat_rotated(const T* v, int i, const float* cs, int rot, int pairing) {
  const int half = rot >> 1;
  if (pairing == 0) {
    const int p = i < half ? i : i - half;
    const float c = cs[p], s = cs[half + p];
    const float x = lat_f32(v[i]), o = lat_f32(v[i < half ? i + half : p]);
    return i < half ? x * c - o * s : x * c + o * s;
  }
  const int p = i >> 1;
  const float c = cs[p], s = cs[half + p];
  const float x = lat_f32(v[i]), o = lat_f32(v[i ^ 1]);
  return (i & 1) ? x * c + o * s : x * c - o * s;
}

// Eight neighbouring values of the rotation at once (split-half pairing, rot a multiple of 16, 16-byte aligned).
__device__ __forceinline__ uint4 lat_rotated8(const __nv_bfloat16* v, int i, const float* cs, int rot) {
  const int half = rot >> 1;
  const bool lo = i < half;
  const int p = lo ? i : i - half;
  const uint4 xv = *reinterpret_cast<const uint4*>(v + i), ov = *reinterpret_cast<const uint4*>(v + (lo ? i + half : p));
  const uint32_t xs[4] = {xv.x, xv.y, xv.z, xv.w}, os[4] = {ov.x, ov.y, ov.z, ov.w};
  float c[8], sn[8];
#pragma unroll
  for (int j = 0; j < 8; j += 4) {
    *reinterpret_cast<float4*>(c + j) = *reinterpret_cast<const float4*>(cs + p + j);
    *reinterpret_cast<float4*>(sn + j) = *reinterpret_cast<const float4*>(cs + half + p + j);
  }
  uint32_t r[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 x = unpack_bf16x2(xs[j]), o = unpack_bf16x2(os[j]);
    const float sgn = lo ? -1.f : 1.f;
    r[j] = pack_bf16x2(x.x * c[2 * j] + sgn * o.x * sn[2 * j], x.y * c[2 * j + 1] + sgn * o.y * sn[2 * j + 1]);
  }
  return make_uint4(r[0], r[1], r[2], r[3]);
}

// The query heads of one CTA in pieces of eight values; every size and stride involved is a multiple of eight.
__device__ __forceinline__ void latent_prep_queries8(const LatentPrepArgs& a, const __nv_bfloat16* row, const float* cs, int t, int h0,
                                                     int h1) {
  const int qk = a.nope + a.rot;
  const bool full = a.q_full != nullptr;
  const int n1 = (full ? a.full_ld : a.nope_ld) / 8, n2 = full ? 0 : (a.width - a.rank) / 8, per = n1 + n2;
  for (int i = threadIdx.x; i < (h1 - h0) * per; i += blockDim.x) {
    const int h = h0 + i / per, c = i % per;
    const __nv_bfloat16* q = row + (size_t)h * qk;
    uint4 v = make_uint4(0, 0, 0, 0);
    uint4* dst;
    int e;  // value of the rotated part, < 0 or >= rot: none
    if (c < n1) {
      const int d = 8 * c;
      dst = full ? reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(a.q_full) + ((size_t)t * a.H + h) * a.full_ld + d)
                 : reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(a.q_nope) + ((size_t)h * a.T + t) * a.nope_ld + d);
      if (d < a.nope) v = *reinterpret_cast<const uint4*>(q + d);
      e = full ? d - a.full_rot : -1;
    } else {
      const int d = a.rank + 8 * (c - n1);
      dst = reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(a.q_rows) + ((size_t)t * a.H + h) * a.width + d);
      e = d - a.pad;
    }
    if (e >= 0 && e < a.rot) v = lat_rotated8(q + a.nope, e, cs, a.rot);
    *dst = v;
  }
}

// grid (T, 1 + ceil(H / LAT_PREP_HEADS)): CTA (t, 0) makes token t's cache row, the others its query heads
template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepArgs a) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x;
  const T* row = reinterpret_cast<const T*>(a.qkv) + (size_t)t * a.ld;
  int pos = a.positions[t];
  pos = pos < 0 ? 0 : (pos >= a.max_pos ? a.max_pos - 1 : pos);
  const float* cs = a.cos_sin + (size_t)pos * a.rot;
  const int qk = a.nope + a.rot;
  if (blockIdx.y == 0) {
    if (a.slots == nullptr) return;
    const int slot = a.slots[t];
    if (slot < 0) return;
    const int blk = slot / a.page;
    if (blk >= a.num_blocks) {  // never write outside the pool
      if (tid == 0) oxb_report(OXB_BAD_SLOT, slot);
      return;
    }
    const T* lat = row + (size_t)a.H * qk;
    float ss = 0.f;
    for (int i = tid; i < a.rank; i += blockDim.x) {
      const float v = lat_f32(lat[i]);
      ss += v * v;
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)a.rank + a.eps);
    T* dst = reinterpret_cast<T*>(a.cache) + ((size_t)blk * a.page + slot % a.page) * a.width;
    for (int i = tid; i < a.width; i += blockDim.x) {
      float v = 0.f;
      if (i < a.rank) v = lat_f32(lat[i]) * inv * a.norm_w[i];
      else if (i >= a.pad && i < a.pad + a.rot) v = lat_rotated(lat + a.rank, i - a.pad, cs, a.rot, a.pairing);
      dst[i] = lat_from<T>(v);
    }
    return;
  }
  const int h0 = (blockIdx.y - 1) * LAT_PREP_HEADS, h1 = min(a.H, h0 + LAT_PREP_HEADS);
  if constexpr (sizeof(T) == 2) {
    if (a.vec8) {
      latent_prep_queries8(a, row, cs, t, h0, h1);
      return;
    }
  }
  for (int h = h0; h < h1; ++h) {
    const T* q = row + (size_t)h * qk;
    if (a.q_full != nullptr) {
      T* dst = reinterpret_cast<T*>(a.q_full) + ((size_t)t * a.H + h) * a.full_ld;
      for (int i = tid; i < a.full_ld; i += blockDim.x)
        dst[i] = i < a.nope ? q[i]
                            : lat_from<T>((i >= a.full_rot && i < a.full_rot + a.rot)
                                              ? lat_rotated(q + a.nope, i - a.full_rot, cs, a.rot, a.pairing)
                                              : 0.f);
      continue;
    }
    T* qn = reinterpret_cast<T*>(a.q_nope) + ((size_t)h * a.T + t) * a.nope_ld;
    for (int i = tid; i < a.nope_ld; i += blockDim.x) qn[i] = i < a.nope ? q[i] : lat_from<T>(0.f);
    T* qr = reinterpret_cast<T*>(a.q_rows) + ((size_t)t * a.H + h) * a.width;
    for (int i = a.rank + tid; i < a.width; i += blockDim.x)  // also the padding between the two parts
      qr[i] = lat_from<T>((i >= a.pad && i < a.pad + a.rot) ? lat_rotated(q + a.nope, i - a.pad, cs, a.rot, a.pairing) : 0.f);
  }
}

struct LatentAttnArgs {
  const void* q;            // [T, H, width]
  void* out;                // [H, T, pad]: attended latents, head-major (operand of the per-head products with W_uv)
  const void* cache;        // layer base [blocks, page, width]
  const int* block_tables;  // [B, max_blocks]
  const int* seq_lens;      // [B]
  const int* query_start;   // [B + 1]
  const float* sink;        // [H] or null
  int B, max_blocks, T, H, pad, width, page, num_blocks, window;
  float scale;
};

// One warp per (token, head), keys one after the other; NC * 32 >= width.
template <typename T, int NC>
__global__ void __launch_bounds__(128) latent_attention_simt_kernel(const LatentAttnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int task = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (task >= a.T * a.H) return;
  const int t = task / a.H, h = task % a.H;
  int lo_b = 0, hi_b = a.B - 1;  // the sequence that holds row t
  while (lo_b < hi_b) {
    const int mid = (lo_b + hi_b + 1) >> 1;
    if (a.query_start[mid] <= t) lo_b = mid;
    else hi_b = mid - 1;
  }
  const int b = lo_b;
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
    const T* row = reinterpret_cast<const T*>(a.cache) + ((size_t)blk * a.page + k % a.page) * a.width;
    float v[NC], s = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int d = lane + 32 * i;
      v[i] = d < a.width ? lat_f32(row[d]) : 0.f;
      s += qv[i] * v[i];
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s);
    const float c = expf(m - mn), p = expf(s - mn);  // m is -inf before the first key only
    l = l * c + p;
    m = mn;
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] = acc[i] * c + p * v[i];
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* o = reinterpret_cast<T*>(a.out) + ((size_t)h * a.T + t) * a.pad;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int d = lane + 32 * i;
    if (d < a.pad) o[d] = lat_from<T>(acc[i] * inv);
  }
}

}  // namespace oxb
