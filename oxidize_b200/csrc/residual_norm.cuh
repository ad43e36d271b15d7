// Norm after the sum: x <- norm(alpha * x + y) with the residual stream x in float32, and the same rows in the
// activation type for the matrix products that follow, in one kernel.  Layer norm (mean removed, weight and bias) or RMS
// norm; the variance is the mean of the squared deviations, taken in a second pass over the row held in registers.
#pragma once
#include "common.cuh"

namespace oxb {

struct ResidualNormArgs {
  const float* res;  // [T, H] or null
  const void* y;     // [T, H] in the activation type, or null
  float alpha;
  const float *w, *b;  // [H]; b may be null
  float* x_out;        // [T, H] or null (may be res: the rows are read before they are written)
  void* a_out;         // [T, H] in the activation type, or null
  int H;
  float eps;
  int layer_norm;  // 1: layer norm, 0: RMS norm
};

__device__ __forceinline__ float4 rn_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 rn_load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void rn_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void rn_store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float rn_load(const float* p) { return *p; }
__device__ __forceinline__ float rn_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void rn_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void rn_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// One CTA per row; every thread owns CH groups of four neighbouring values (H % 4 == 0, H <= 4 * CH * threads).
template <typename A, int CH>
__global__ void __launch_bounds__(1024) residual_norm_kernel(const ResidualNormArgs a) {
  __shared__ float red[32];
  const int H4 = a.H >> 2;
  const size_t base = (size_t)blockIdx.x * a.H;
  float4 v[CH], w[CH], b[CH];
  pdl_launch_dependents();
#pragma unroll
  for (int c = 0; c < CH; ++c) {  // weights are static: fetched ahead of the dependency
    const int i = threadIdx.x + c * blockDim.x;
    w[c] = b[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < H4) {
      w[c] = rn_load4(a.w + 4 * i);
      if (a.b != nullptr) b[c] = rn_load4(a.b + 4 * i);
    }
  }
  pdl_wait();
  float sum = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    v[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < H4) {
      float4 r = v[c], y = v[c];
      if (a.y != nullptr) y = rn_load4(reinterpret_cast<const A*>(a.y) + base + 4 * i);
      if (a.res != nullptr) r = rn_load4(a.res + base + 4 * i);
      v[c] = make_float4(a.alpha * r.x + y.x, a.alpha * r.y + y.y, a.alpha * r.z + y.z, a.alpha * r.w + y.w);
    }
    sum += (v[c].x + v[c].y) + (v[c].z + v[c].w);
  }
  const float mean = a.layer_norm ? block_sum(sum, red) / (float)a.H : 0.f;
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    if (threadIdx.x + c * blockDim.x < H4) {
      v[c] = make_float4(v[c].x - mean, v[c].y - mean, v[c].z - mean, v[c].w - mean);
      ss += (v[c].x * v[c].x + v[c].y * v[c].y) + (v[c].z * v[c].z + v[c].w * v[c].w);
    }
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.H + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < H4) {
      const float4 o = make_float4(v[c].x * inv * w[c].x + b[c].x, v[c].y * inv * w[c].y + b[c].y,
                                   v[c].z * inv * w[c].z + b[c].z, v[c].w * inv * w[c].w + b[c].w);
      if (a.x_out != nullptr) rn_store4(a.x_out + base + 4 * i, o);
      if (a.a_out != nullptr) rn_store4(reinterpret_cast<A*>(a.a_out) + base + 4 * i, o);
    }
  }
}

// Any width: the row is staged in shared memory (dynamic, H floats).
template <typename A>
__global__ void __launch_bounds__(256) residual_norm_any_kernel(const ResidualNormArgs a) {
  extern __shared__ float rn_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const size_t base = (size_t)blockIdx.x * a.H;
  float sum = 0.f;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    float v = a.res != nullptr ? a.alpha * a.res[base + i] : 0.f;
    if (a.y != nullptr) v += rn_load(reinterpret_cast<const A*>(a.y) + base + i);
    rn_row[i] = v;
    sum += v;
  }
  const float mean = a.layer_norm ? block_sum(sum, red) / (float)a.H : 0.f;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    const float v = rn_row[i] - mean;
    ss += v * v;
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.H + a.eps);
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    const float o = (rn_row[i] - mean) * inv * a.w[i] + (a.b != nullptr ? a.b[i] : 0.f);
    if (a.x_out != nullptr) a.x_out[base + i] = o;
    if (a.a_out != nullptr) rn_store(reinterpret_cast<A*>(a.a_out) + base + i, o);
  }
}

template <typename A>
int residual_norm_launch(const ResidualNormArgs& a, int T, cudaStream_t stream) {
  if (a.H % 4 == 0 && a.H <= 16384) {
    // many rows: few threads with several groups each, so that several rows are resident per SM; few rows: the row is spread
    // over as many threads as there are groups
    const int H4 = a.H / 4, lim = T >= 512 ? 256 : 1024, ch = H4 <= lim ? 1 : (H4 <= 2 * lim ? 2 : 4);
    const int threads = ((H4 + ch - 1) / ch + 31) / 32 * 32;
    if (ch == 1) oxb_launch(residual_norm_kernel<A, 1>, dim3(T), dim3(threads), 0, stream, a);
    else if (ch == 2) oxb_launch(residual_norm_kernel<A, 2>, dim3(T), dim3(threads), 0, stream, a);
    else oxb_launch(residual_norm_kernel<A, 4>, dim3(T), dim3(threads), 0, stream, a);
  } else {
    if (a.H > 12 * 1024) return (int)cudaErrorInvalidValue;  // 48 KB of shared memory
    oxb_launch(residual_norm_any_kernel<A>, dim3(T), dim3(256), (size_t)a.H * sizeof(float), stream, a);
  }
  OXB_CHECK_LAUNCH();
  return 0;
}

// Norms on both sides of a branch: x = res + rms(y) * w_post, then the next branch's input rms(x) * w_next in the activation
// type, in one kernel (the stream x in float32; w_next null: the sum alone; y null: the norm alone).
struct BranchNormArgs {
  const float* res;              // [T, H]
  const void* y;                 // [T, H] in the activation type, or null
  const float *w_post, *w_next;  // [H]
  float* x_out;                  // [T, H] or null
  void* a_out;                   // [T, H] in the activation type, or null
  int H;
  float eps;
};

// One CTA per row; every thread owns CH groups of four neighbouring values (H % 4 == 0, H <= 4 * CH * threads).
template <typename A, int CH>
__global__ void __launch_bounds__(1024) branch_norm_kernel(const BranchNormArgs a) {
  __shared__ float red[32];
  const int H4 = a.H >> 2;
  const size_t base = (size_t)blockIdx.x * a.H;
  float4 y[CH], v[CH], w[CH], n[CH];
  pdl_launch_dependents();
#pragma unroll
  for (int c = 0; c < CH; ++c) {  // weights are static: fetched ahead of the dependency
    const int i = threadIdx.x + c * blockDim.x;
    w[c] = n[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < H4) {
      if (a.w_post != nullptr) w[c] = rn_load4(a.w_post + 4 * i);
      if (a.w_next != nullptr) n[c] = rn_load4(a.w_next + 4 * i);
    }
  }
  pdl_wait();
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    y[c] = v[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < H4) {
      v[c] = rn_load4(a.res + base + 4 * i);
      if (a.y != nullptr) y[c] = rn_load4(reinterpret_cast<const A*>(a.y) + base + 4 * i);
    }
    ss += (y[c].x * y[c].x + y[c].y * y[c].y) + (y[c].z * y[c].z + y[c].w * y[c].w);
  }
  if (a.y != nullptr) {
    const float inv = rsqrtf(block_sum(ss, red) / (float)a.H + a.eps);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = threadIdx.x + c * blockDim.x;
      v[c] = make_float4(v[c].x + y[c].x * inv * w[c].x, v[c].y + y[c].y * inv * w[c].y, v[c].z + y[c].z * inv * w[c].z,
                         v[c].w + y[c].w * inv * w[c].w);
      if (i < H4 && a.x_out != nullptr) rn_store4(a.x_out + base + 4 * i, v[c]);
    }
  }
  if (a.a_out == nullptr) return;
  ss = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) ss += (v[c].x * v[c].x + v[c].y * v[c].y) + (v[c].z * v[c].z + v[c].w * v[c].w);
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.H + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < H4)
      rn_store4(reinterpret_cast<A*>(a.a_out) + base + 4 * i,
                make_float4(v[c].x * inv * n[c].x, v[c].y * inv * n[c].y, v[c].z * inv * n[c].z, v[c].w * inv * n[c].w));
  }
}

// Any width: the row is staged in shared memory (dynamic, H floats).
template <typename A>
__global__ void __launch_bounds__(256) branch_norm_any_kernel(const BranchNormArgs a) {
  extern __shared__ float rn_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const size_t base = (size_t)blockIdx.x * a.H;
  const A* y = reinterpret_cast<const A*>(a.y);
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    rn_row[i] = y != nullptr ? rn_load(y + base + i) : 0.f;
    ss += rn_row[i] * rn_row[i];
  }
  const float inv_y = y != nullptr ? rsqrtf(block_sum(ss, red) / (float)a.H + a.eps) : 0.f;
  ss = 0.f;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    float v = a.res[base + i];
    if (y != nullptr) v += rn_row[i] * inv_y * a.w_post[i];
    rn_row[i] = v;
    if (a.x_out != nullptr) a.x_out[base + i] = v;
    ss += v * v;
  }
  if (a.a_out == nullptr) return;
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.H + a.eps);
  for (int i = threadIdx.x; i < a.H; i += blockDim.x)
    rn_store(reinterpret_cast<A*>(a.a_out) + base + i, rn_row[i] * inv * a.w_next[i]);
}

// Both branches of a layer join the stream and the next layer's norm follows, in one kernel:
//     x = res + mixer + ffn,   a = rms(x) * w_next  in the activation type.
// The mixer's output is y0, or s0 rms(y0) w0 + s1 rms(y1) w1 where two mixers have norms of their own; the feed-forward
// output is f, or the weighted sum of routed rows, sum_j weights[t, j] f[index[t, j]].
struct JointNormArgs {
  const float* res;     // [T, H]
  const void *y0, *y1;  // [T, H] in the activation type, or null
  const float *w0, *w1; // [H]; null: y0 as it is
  float s0, s1;
  const void* f;        // [T, H], or rows ldf apart with index; or null
  const int* index;     // [T, k] or null; < 0: none
  const float* weights; // [T, k]
  int k, ldf;
  const float* w_next;  // [H] or null: the sum alone
  float* x_out;         // [T, H] or null
  void* a_out;          // [T, H] in the activation type, or null
  int H;
  float eps;
};

// One CTA per row; every thread owns CH groups of four neighbouring values (H % 4 == 0, H <= 4 * CH * threads).
template <typename A, int CH>
__global__ void __launch_bounds__(1024) joint_norm_kernel(const JointNormArgs a) {
  __shared__ float red[32];
  const int H4 = a.H >> 2, t = blockIdx.x;
  const size_t base = (size_t)t * a.H;
  float4 v[CH], n[CH];
  pdl_launch_dependents();
#pragma unroll
  for (int c = 0; c < CH; ++c) {  // weights are static: fetched ahead of the dependency
    const int i = threadIdx.x + c * blockDim.x;
    n[c] = (i < H4 && a.w_next != nullptr) ? rn_load4(a.w_next + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    v[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < H4) v[c] = rn_load4(a.res + base + 4 * i);
  }
  if (a.f != nullptr) {
    const A* f = reinterpret_cast<const A*>(a.f);
    const int k = a.index != nullptr ? a.k : 1;
    for (int j = 0; j < k; ++j) {
      const int r = a.index != nullptr ? a.index[(size_t)t * k + j] : t;
      if (r < 0) continue;
      const float w = a.index != nullptr ? a.weights[(size_t)t * k + j] : 1.f;
#pragma unroll
      for (int c = 0; c < CH; ++c) {
        const int i = threadIdx.x + c * blockDim.x;
        if (i < H4) {
          const float4 y = rn_load4(f + (size_t)r * a.ldf + 4 * i);
          v[c] = make_float4(fmaf(w, y.x, v[c].x), fmaf(w, y.y, v[c].y), fmaf(w, y.z, v[c].z), fmaf(w, y.w, v[c].w));
        }
      }
    }
  }
#pragma unroll
  for (int side = 0; side < 2; ++side) {
    const A* yp = reinterpret_cast<const A*>(side == 0 ? a.y0 : a.y1);
    const float* wp = side == 0 ? a.w0 : a.w1;
    if (yp == nullptr) continue;
    float4 y[CH];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = threadIdx.x + c * blockDim.x;
      y[c] = i < H4 ? rn_load4(yp + base + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += (y[c].x * y[c].x + y[c].y * y[c].y) + (y[c].z * y[c].z + y[c].w * y[c].w);
    }
    const float inv = wp != nullptr ? rsqrtf(block_sum(ss, red) / (float)a.H + a.eps) * (side == 0 ? a.s0 : a.s1) : 1.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = threadIdx.x + c * blockDim.x;
      if (i >= H4) continue;
      const float4 w = wp != nullptr ? rn_load4(wp + 4 * i) : make_float4(1.f, 1.f, 1.f, 1.f);
      v[c] = make_float4(v[c].x + y[c].x * inv * w.x, v[c].y + y[c].y * inv * w.y, v[c].z + y[c].z * inv * w.z,
                         v[c].w + y[c].w * inv * w.w);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < H4 && a.x_out != nullptr) rn_store4(a.x_out + base + 4 * i, v[c]);
    ss += (v[c].x * v[c].x + v[c].y * v[c].y) + (v[c].z * v[c].z + v[c].w * v[c].w);
  }
  if (a.a_out == nullptr) return;
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.H + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < H4)
      rn_store4(reinterpret_cast<A*>(a.a_out) + base + 4 * i,
                make_float4(v[c].x * inv * n[c].x, v[c].y * inv * n[c].y, v[c].z * inv * n[c].z, v[c].w * inv * n[c].w));
  }
}

// Any width: the row is staged in shared memory (dynamic, H floats).
template <typename A>
__global__ void __launch_bounds__(256) joint_norm_any_kernel(const JointNormArgs a) {
  extern __shared__ float rn_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const size_t base = (size_t)t * a.H;
  const A *y0 = reinterpret_cast<const A*>(a.y0), *y1 = reinterpret_cast<const A*>(a.y1), *f = reinterpret_cast<const A*>(a.f);
  float i0 = 1.f, i1 = 1.f;
  if (a.w0 != nullptr) {
    float ss0 = 0.f, ss1 = 0.f;
    for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
      const float u = rn_load(y0 + base + i), w = rn_load(y1 + base + i);
      ss0 += u * u;
      ss1 += w * w;
    }
    i0 = rsqrtf(block_sum(ss0, red) / (float)a.H + a.eps) * a.s0;
    i1 = rsqrtf(block_sum(ss1, red) / (float)a.H + a.eps) * a.s1;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    float v = a.res[base + i];
    if (f != nullptr && a.index == nullptr) v += rn_load(f + (size_t)t * a.ldf + i);
    if (f != nullptr && a.index != nullptr)
      for (int j = 0; j < a.k; ++j) {
        const int r = a.index[(size_t)t * a.k + j];
        if (r >= 0) v = fmaf(a.weights[(size_t)t * a.k + j], rn_load(f + (size_t)r * a.ldf + i), v);
      }
    if (y0 != nullptr) v += rn_load(y0 + base + i) * i0 * (a.w0 != nullptr ? a.w0[i] : 1.f);
    if (y1 != nullptr) v += rn_load(y1 + base + i) * i1 * (a.w1 != nullptr ? a.w1[i] : 1.f);
    rn_row[i] = v;
    if (a.x_out != nullptr) a.x_out[base + i] = v;
    ss += v * v;
  }
  if (a.a_out == nullptr) return;
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.H + a.eps);
  for (int i = threadIdx.x; i < a.H; i += blockDim.x)
    rn_store(reinterpret_cast<A*>(a.a_out) + base + i, rn_row[i] * inv * a.w_next[i]);
}

template <typename A>
int joint_norm_launch(const JointNormArgs& a, int T, cudaStream_t stream) {
  if (a.H % 4 == 0 && a.ldf % 4 == 0 && a.H <= 16384) {
    const int H4 = a.H / 4, lim = T >= 512 ? 256 : 1024, ch = H4 <= lim ? 1 : (H4 <= 2 * lim ? 2 : 4);
    const int threads = ((H4 + ch - 1) / ch + 31) / 32 * 32;
    if (ch == 1) oxb_launch(joint_norm_kernel<A, 1>, dim3(T), dim3(threads), 0, stream, a);
    else if (ch == 2) oxb_launch(joint_norm_kernel<A, 2>, dim3(T), dim3(threads), 0, stream, a);
    else oxb_launch(joint_norm_kernel<A, 4>, dim3(T), dim3(threads), 0, stream, a);
  } else {
    if (a.H > 12 * 1024) return (int)cudaErrorInvalidValue;  // 48 KB of shared memory
    oxb_launch(joint_norm_any_kernel<A>, dim3(T), dim3(256), (size_t)a.H * sizeof(float), stream, a);
  }
  OXB_CHECK_LAUNCH();
  return 0;
}

// A branch's output joins the stream through an RMS norm in groups, x = res + norm(y) w, every one of `groups` consecutive parts
// over its own root mean square; y may be the weighted sum of routed rows, sum_j weights[t, j] y[index[t, j]].  With `depth`, x
// becomes the n-th of the kept results and what goes on is depth[0] first + sum_(j < n) depth[j + 1] results[j] + depth[n + 1] x.
// Without a branch (y null): a = norm(res) w.
struct AddNormedArgs {
  const float* res;     // [T, H]
  const void* y;        // [T, H] in the activation type, or rows ldy apart with index; or null
  const int* index;     // [T, k] or null; < 0: none
  const float* weights; // [T, k]
  int k, ldy;
  const float* w;       // [H]
  int groups;
  float eps;
  const float* first;   // [T, H]
  float* results;       // [n + 1, T, H]
  size_t step;          // T * H
  int n;
  const float* depth;   // [n + 2] or null
  float* x_out;         // [T, H] or null
  void* a_out;          // [T, H] in the activation type, or null
  int H;
};

// One CTA per row; every thread owns CH groups of four neighbouring values (H <= 4 * CH * threads); a part is a multiple of 128
// values, so that a warp's values lie in one part.
template <typename A, int CH>
__global__ void __launch_bounds__(1024) add_normed_kernel(const AddNormedArgs a) {
  __shared__ float part[128];  // sums of 128 values each
  const int H4 = a.H >> 2, t = blockIdx.x, lane = threadIdx.x & 31;
  const size_t base = (size_t)t * a.H;
  float4 y[CH], w[CH];
  pdl_launch_dependents();
#pragma unroll
  for (int c = 0; c < CH; ++c) {  // weights are static: fetched ahead of the dependency
    const int i = threadIdx.x + c * blockDim.x;
    w[c] = y[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < H4) w[c] = rn_load4(a.w + 4 * i);
  }
  pdl_wait();
  float4 v[CH];
  const A* yp = reinterpret_cast<const A*>(a.y);
  const int k = a.index != nullptr ? a.k : 1;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    v[c] = i < H4 ? rn_load4(a.res + base + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    if (yp == nullptr) y[c] = v[c];
  }
  for (int j = 0; j < k && yp != nullptr; ++j) {
    const int r = a.index != nullptr ? a.index[(size_t)t * k + j] : t;
    if (r < 0) continue;
    const float g = a.index != nullptr ? a.weights[(size_t)t * k + j] : 1.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = threadIdx.x + c * blockDim.x;
      if (i < H4) {
        const float4 f = rn_load4(yp + (size_t)r * a.ldy + 4 * i);
        y[c] = make_float4(fmaf(g, f.x, y[c].x), fmaf(g, f.y, y[c].y), fmaf(g, f.z, y[c].z), fmaf(g, f.w, y[c].w));
      }
    }
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    const float ss = warp_sum((y[c].x * y[c].x + y[c].y * y[c].y) + (y[c].z * y[c].z + y[c].w * y[c].w));
    if (lane == 0 && i < H4) part[i >> 5] = ss;
  }
  __syncthreads();
  const int per = a.H / a.groups;  // values of a part
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i >= H4) continue;
    const int g0 = 4 * i / per * (per >> 7);
    float ss = 0.f;
    for (int j = 0; j < per >> 7; ++j) ss += part[g0 + j];
    const float inv = rsqrtf(ss / (float)per + a.eps);
    y[c] = make_float4(y[c].x * inv * w[c].x, y[c].y * inv * w[c].y, y[c].z * inv * w[c].z, y[c].w * inv * w[c].w);
    if (yp == nullptr) v[c] = y[c];
    else v[c] = make_float4(v[c].x + y[c].x, v[c].y + y[c].y, v[c].z + y[c].z, v[c].w + y[c].w);
  }
  if (a.depth != nullptr) {
    const float d0 = a.depth[0], dn = a.depth[a.n + 1];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = threadIdx.x + c * blockDim.x;
      if (i >= H4) continue;
      const float* row = a.results + base + 4 * i;
      rn_store4(a.results + a.n * a.step + base + 4 * i, v[c]);
      const float4 f = rn_load4(a.first + base + 4 * i);
      float4 s = make_float4(d0 * f.x, d0 * f.y, d0 * f.z, d0 * f.w);
#pragma unroll 8
      for (int j = 0; j < a.n; ++j) {
        const float4 r = rn_load4(row + j * a.step);
        const float d = a.depth[j + 1];
        s = make_float4(fmaf(d, r.x, s.x), fmaf(d, r.y, s.y), fmaf(d, r.z, s.z), fmaf(d, r.w, s.w));
      }
      v[c] = make_float4(fmaf(dn, v[c].x, s.x), fmaf(dn, v[c].y, s.y), fmaf(dn, v[c].z, s.z), fmaf(dn, v[c].w, s.w));
    }
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i >= H4) continue;
    if (a.x_out != nullptr) rn_store4(a.x_out + base + 4 * i, v[c]);
    if (a.a_out != nullptr) rn_store4(reinterpret_cast<A*>(a.a_out) + base + 4 * i, v[c]);
  }
}

// Any width and part: the row is staged in shared memory (dynamic, H + groups floats).
template <typename A>
__global__ void __launch_bounds__(256) add_normed_any_kernel(const AddNormedArgs a) {
  extern __shared__ float rn_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per = a.H / a.groups;
  const size_t base = (size_t)t * a.H;
  const A* y = reinterpret_cast<const A*>(a.y);
  float* inv = rn_row + a.H;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    float v = 0.f;
    if (y == nullptr) v = a.res[base + i];
    else if (a.index == nullptr) v = rn_load(y + (size_t)t * a.ldy + i);
    else
      for (int j = 0; j < a.k; ++j) {
        const int r = a.index[(size_t)t * a.k + j];
        if (r >= 0) v = fmaf(a.weights[(size_t)t * a.k + j], rn_load(y + (size_t)r * a.ldy + i), v);
      }
    rn_row[i] = v;
  }
  __syncthreads();
  if (a.groups >= 8) {
    for (int g = warp; g < a.groups; g += blockDim.x >> 5) {
      float ss = 0.f;
      for (int i = lane; i < per; i += 32) ss += rn_row[g * per + i] * rn_row[g * per + i];
      ss = warp_sum(ss);
      if (lane == 0) inv[g] = rsqrtf(ss / (float)per + a.eps);
    }
  } else {
    for (int g = 0; g < a.groups; ++g) {
      float ss = 0.f;
      for (int i = threadIdx.x; i < per; i += blockDim.x) ss += rn_row[g * per + i] * rn_row[g * per + i];
      ss = block_sum(ss, red);
      if (threadIdx.x == 0) inv[g] = rsqrtf(ss / (float)per + a.eps);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) {
    float v = rn_row[i] * inv[i / per] * a.w[i];
    if (y != nullptr) v += a.res[base + i];
    if (a.depth != nullptr) {
      a.results[a.n * a.step + base + i] = v;
      float s = a.depth[0] * a.first[base + i];
      for (int j = 0; j < a.n; ++j) s = fmaf(a.depth[j + 1], a.results[j * a.step + base + i], s);
      v = fmaf(a.depth[a.n + 1], v, s);
    }
    if (a.x_out != nullptr) a.x_out[base + i] = v;
    if (a.a_out != nullptr) rn_store(reinterpret_cast<A*>(a.a_out) + base + i, v);
  }
}

template <typename A>
int add_normed_launch(const AddNormedArgs& a, int T, cudaStream_t stream) {
  if (a.H % a.groups == 0 && (a.H / a.groups) % 128 == 0 && a.ldy % 4 == 0 && a.H <= 16384) {
    const int H4 = a.H / 4, lim = T >= 512 ? 256 : 1024, ch = H4 <= lim ? 1 : (H4 <= 2 * lim ? 2 : 4);
    const int threads = ((H4 + ch - 1) / ch + 31) / 32 * 32;
    if (ch == 1) oxb_launch(add_normed_kernel<A, 1>, dim3(T), dim3(threads), 0, stream, a);
    else if (ch == 2) oxb_launch(add_normed_kernel<A, 2>, dim3(T), dim3(threads), 0, stream, a);
    else oxb_launch(add_normed_kernel<A, 4>, dim3(T), dim3(threads), 0, stream, a);
  } else {
    if (a.H % a.groups != 0 || a.H + a.groups > 12 * 1024) return (int)cudaErrorInvalidValue;  // 48 KB of shared memory
    oxb_launch(add_normed_any_kernel<A>, dim3(T), dim3(256), (size_t)(a.H + a.groups) * sizeof(float), stream, a);
  }
  OXB_CHECK_LAUNCH();
  return 0;
}

template <typename A>
int branch_norm_launch(const BranchNormArgs& a, int T, cudaStream_t stream) {
  if (a.H % 4 == 0 && a.H <= 16384) {
    const int H4 = a.H / 4, lim = T >= 512 ? 256 : 1024, ch = H4 <= lim ? 1 : (H4 <= 2 * lim ? 2 : 4);
    const int threads = ((H4 + ch - 1) / ch + 31) / 32 * 32;
    if (ch == 1) oxb_launch(branch_norm_kernel<A, 1>, dim3(T), dim3(threads), 0, stream, a);
    else if (ch == 2) oxb_launch(branch_norm_kernel<A, 2>, dim3(T), dim3(threads), 0, stream, a);
    else oxb_launch(branch_norm_kernel<A, 4>, dim3(T), dim3(threads), 0, stream, a);
  } else {
    if (a.H > 12 * 1024) return (int)cudaErrorInvalidValue;  // 48 KB of shared memory
    oxb_launch(branch_norm_any_kernel<A>, dim3(T), dim3(256), (size_t)a.H * sizeof(float), stream, a);
  }
  OXB_CHECK_LAUNCH();
  return 0;
}

}  // namespace oxb
