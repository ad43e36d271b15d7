// Float32 matrix product on the CUDA cores, Y[g] [T, N] = act(X[g] [T, K] . W[g] [N, K]^T + bias): the float32 compute
// path, in which no operand or product is rounded to a shorter type.  64 x 64 tile per CTA, 4 x 4 results per thread,
// k-slices of 16 double-buffered through shared memory.
#pragma once
#include "common.cuh"

namespace oxb {

constexpr int F32_TILE = 64, F32_K = 16;

struct GemmF32Args {
  const float *x, *w, *bias;
  float* y;
  int T, N, K, ldx, ldw, ldy;
  long long xs, ws, ys;  // strides of a group
  int act;               // 0 none, 1 square of relu
  // routed groups: group g multiplies rows [offsets[g], offsets[g + 1]) of Y; row r of Y reads row perm[r] of X (perm null: r)
  const int *offsets, *perm;
};

static __global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32Args a) {
  __shared__ float sx[2][F32_K][F32_TILE + 4], sw[2][F32_K][F32_TILE + 4];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x;
  const int g0 = a.offsets != nullptr ? a.offsets[blockIdx.z] : 0;
  const int T = a.offsets != nullptr ? a.offsets[blockIdx.z + 1] : a.T;  // rows end here
  const float* X = a.x + (size_t)blockIdx.z * a.xs;
  const float* W = a.w + (size_t)blockIdx.z * a.ws;
  float* Y = a.y + (size_t)blockIdx.z * a.ys;
  const int t0 = g0 + blockIdx.y * F32_TILE, n0 = blockIdx.x * F32_TILE;
  if (t0 >= T) return;
  const int lr = tid >> 4, lk = tid & 15;  // loads: 16 rows x 16 k per pass, 4 passes
  float rx[4], rw[4];
  size_t xrow[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + lr + 16 * i;
    xrow[i] = t < T ? (a.perm != nullptr ? a.perm[t] : t) : 0;
  }
  auto fetch = [&](int k0) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = lr + 16 * i, k = k0 + lk;
      rx[i] = (t0 + r < T && k < a.K) ? X[xrow[i] * a.ldx + k] : 0.f;
      rw[i] = (n0 + r < a.N && k < a.K) ? W[(size_t)(n0 + r) * a.ldw + k] : 0.f;
    }
  };
  auto put = [&](int s) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      sx[s][lk][lr + 16 * i] = rx[i];
      sw[s][lk][lr + 16 * i] = rw[i];
    }
  };
  float acc[4][4] = {};
  const int tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
  fetch(0);
  put(0);
  __syncthreads();
  int s = 0;
  for (int k0 = 0; k0 < a.K; k0 += F32_K) {
    const bool more = k0 + F32_K < a.K;
    if (more) fetch(k0 + F32_K);
#pragma unroll
    for (int k = 0; k < F32_K; ++k) {
      const float4 xv = *reinterpret_cast<const float4*>(&sx[s][k][tr]);
      const float4 wv = *reinterpret_cast<const float4*>(&sw[s][k][tc]);
      const float xa[4] = {xv.x, xv.y, xv.z, xv.w}, wa[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xa[i], wa[j], acc[i][j]);
    }
    if (more) put(s ^ 1);
    __syncthreads();
    s ^= 1;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (t0 + tr + i >= T) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tc + j;
      if (n >= a.N) break;
      float v = acc[i][j] + (a.bias != nullptr ? a.bias[n] : 0.f);
      if (a.act == 1) {
        v = fmaxf(v, 0.f);
        v *= v;
      }
      Y[(size_t)(t0 + tr + i) * a.ldy + n] = v;
    }
  }
}

}  // namespace oxb
