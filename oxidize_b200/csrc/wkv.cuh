// RWKV time mixing: linear attention with one decay per key channel and token, a learned bonus for the current token and one
// [K, V] float32 state per sequence and head,
//     o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_(t-1) + k_t v_t^T,   y_t = o_t / rms(o_t) * norm * silu(gate_t),
// where r, k, v, the gate and the decay are projections of five mixes of a token's input with the one ahead of it, and
// w = exp(-exp(W_2 tanh(W_1 x) + w_0)).  A sequence whose rows start at position 0 starts from nothing.
//
// token_shift_kernel: the mixes.  wkv_decay_kernel: logarithms of the decays.  wkv_step_kernel: token by token, the state in
// registers (decoded tokens, and the float32 path).  wkv_chunk.cuh: chunks of 64 tokens on the tensor cores.
#pragma once
#include "attention.cuh"
#include "latent.cuh"
#include "residual_norm.cuh"

namespace oxb {

struct TokenShiftArgs {
  const float* x;          // [T, H]
  const float* mu;         // [n, H]
  const int* query_start;  // [B + 1]
  const int* seq_lens;     // [B]
  const int* slots;        // [B] state slot, < 0: none
  float* window;           // [num_slots, H]: a sequence's last input
  int num_slots;
  void* out;               // [n, T, ld] in the activation type, zeros behind the H values of a row
  int B, T, H, n, ld;
};

// out[i] = x + (x_before - x) mu[i].  grid (T, channel blocks); the CTA of a sequence's first row reads what earlier steps left
// in the window and then leaves the portion's last row there.
template <typename A, int VEC>
__global__ void __launch_bounds__(256) token_shift_kernel(const TokenShiftArgs a) {
  pdl_launch_dependents();
  const int t = blockIdx.x, i = (blockIdx.y * 256 + threadIdx.x) * VEC;
  const int b = sequence_of(a.query_start, a.B, t), t0 = a.query_start[b], t1 = a.query_start[b + 1], slot = a.slots[b];
  const bool have = (unsigned)slot < (unsigned)a.num_slots, first = t == t0;
  if (slot >= a.num_slots && first && blockIdx.y == 0 && threadIdx.x == 0) oxb_report(OXB_BAD_SLOT, slot);
  if (i >= a.H) {
    pdl_wait();
    if (i < a.ld)
      for (int n = 0; n < a.n; ++n)
#pragma unroll
        for (int j = 0; j < VEC; ++j) rn_store(reinterpret_cast<A*>(a.out) + ((size_t)n * a.T + t) * a.ld + i + j, 0.f);
    return;
  }
  float* win = a.window + (size_t)(have ? slot : 0) * a.H + i;
  const bool carried = first && have && a.seq_lens[b] > t1 - t0;
  float x[VEC], p[VEC], m[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) p[j] = 0.f;
  if (carried) {  // (written by an earlier step: no need to wait for this step's kernels)
#pragma unroll
    for (int j = 0; j < VEC; ++j) p[j] = win[j];
  }
  pdl_wait();
  const float* row = a.x + (size_t)t * a.H + i;
#pragma unroll
  for (int j = 0; j < VEC; ++j) x[j] = row[j];
  if (!first) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) p[j] = row[j - a.H];
  } else if (have) {
    const float* last = a.x + (size_t)(t1 - 1) * a.H + i;
#pragma unroll
    for (int j = 0; j < VEC; ++j) win[j] = last[j];
  }
  A* out = reinterpret_cast<A*>(a.out) + (size_t)t * a.ld + i;
  for (int n = 0; n < a.n; ++n, out += (size_t)a.T * a.ld) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) m[j] = a.mu[(size_t)n * a.H + i + j];
    if constexpr (VEC == 4) {
      rn_store4(out, make_float4(fmaf(p[0] - x[0], m[0], x[0]), fmaf(p[1] - x[1], m[1], x[1]), fmaf(p[2] - x[2], m[2], x[2]),
                                 fmaf(p[3] - x[3], m[3], x[3])));
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) rn_store(out + j, fmaf(p[j] - x[j], m[j], x[j]));
    }
  }
}

// log decays [T, N] float32 = -exp(tanh(low [T, rank]) . up [N, rank]^T + base [N]).
// float32: one thread per value, a token per blockIdx.y; dynamic shared memory: rank floats.
template <typename A>
__global__ void __launch_bounds__(256) wkv_decay_any_kernel(const A* __restrict__ low, const A* __restrict__ up,
                                                            const float* __restrict__ base, float* __restrict__ out, int N, int rank) {
  extern __shared__ float tanh_row[];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
  for (int i = threadIdx.x; i < rank; i += 256) tanh_row[i] = tanhf(lat_f32(low[(size_t)t * rank + i]));
  __syncthreads();
  if (c >= N) return;
  float s = 0.f;
  for (int i = 0; i < rank; ++i) s = fmaf(tanh_row[i], lat_f32(up[(size_t)c * rank + i]), s);
  out[(size_t)t * N + c] = -expf(s + base[c]);
}

// bfloat16 on the tensor cores, tanh as two halves: a CTA has 16 tokens x 256 columns, a warp 32 of them.  rank % 16 == 0,
// N % 32 == 0; dynamic shared memory: 2 * 16 * (rank + 8) halves.
static __global__ void __launch_bounds__(256)
wkv_decay_kernel(const __nv_bfloat16* __restrict__ low, const __nv_bfloat16* __restrict__ up, const float* __restrict__ base,
                 float* __restrict__ out, int T, int N, int rank) {
  extern __shared__ __align__(16) __nv_bfloat16 th[];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, ld = rank + 8;
  const int c0 = (blockIdx.x * 8 + warp) * 32, t0 = blockIdx.y * 16;
  const bool on = c0 < N;
  if (on) {  // (weights are static: on their way ahead of the dependency)
    for (int k = lane * 8; k < 32 * rank; k += 256) asm volatile("prefetch.global.L2 [%0];" ::"l"(up + (size_t)c0 * rank + k));
  }
  pdl_wait();
  for (int i = threadIdx.x; i < 16 * rank; i += 256) {
    const int r = i / rank, k = i % rank;
    const float x = tanhf(__bfloat162float(low[(size_t)min(t0 + r, T - 1) * rank + k]));
    const __nv_bfloat16 hi = __float2bfloat16(x);
    th[r * ld + k] = hi;
    th[(16 + r) * ld + k] = __float2bfloat16(x - __bfloat162float(hi));
  }
  __syncthreads();
  if (!on) return;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  for (int ks = 0; ks < rank; ks += 16) {
    uint2 w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) w[i] = *reinterpret_cast<const uint2*>(up + (size_t)(c0 + 8 * i + g) * rank + ks + 4 * t4);
#pragma unroll
    for (int half = 1; half >= 0; --half) {
      const uint2 x0 = *reinterpret_cast<const uint2*>(th + (16 * half + g) * ld + ks + 4 * t4);
      const uint2 x1 = *reinterpret_cast<const uint2*>(th + (16 * half + g + 8) * ld + ks + 4 * t4);
      const uint32_t a[4] = {x0.x, x1.x, x0.y, x1.y};
#pragma unroll
      for (int i = 0; i < 4; ++i) mma_bf16_16816(acc[i], a, w[i].x, w[i].y);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int t = t0 + g + 8 * (e >> 1), c = c0 + 8 * i + 2 * t4;
      if (t < T)
        *reinterpret_cast<float2*>(out + (size_t)t * N + c) = make_float2(-expf(acc[i][e] + base[c]), -expf(acc[i][e + 1] + base[c + 1]));
    }
}

struct WkvArgs {
  const void* z;           // [T, ld]: r | k | v | gate, H heads of K (= V) values each
  int ld;
  const float* log_decay;  // [T, H * K]
  const int* query_start;  // [B + 1]
  const int* seq_lens;     // [B]
  const int* slots;        // [B] state slot, < 0: none (rows of zeros come out)
  const float* bonus;      // [H * K]
  const float* norm;       // [H * V]
  float* state;            // [num_slots, H, K, V]
  int num_slots;
  void* out;               // [T, ld_out], H heads of V values
  int ld_out;
  int H, K, dim;
  float eps;
  int min_rows, max_rows;  // sequences that feed fewer or more rows belong to the other kernel
};

__device__ __forceinline__ float wkv_silu(float x) { return x / (1.f + expf(-x)); }

// grid (H, B).  Thread (r, c) owns values 4 c .. 4 c + 3 of the state's rows r, r + R, ...; dynamic shared memory:
// 4 K + R V floats.
template <typename T, int NK, int THREADS>
__global__ void __launch_bounds__(THREADS) wkv_step_kernel(const WkvArgs a) {
  extern __shared__ __align__(16) float ws_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  const int q0 = a.query_start[b], n = a.query_start[b + 1] - q0, slot = a.slots[b];
  if (n < a.min_rows || n > a.max_rows || n <= 0) {
    pdl_wait();
    return;
  }
  const int K = a.K, V = K, cols = V >> 2, R = THREADS / cols, r = tid / cols, c = tid % cols;
  const bool on = r < R;
  T* out = reinterpret_cast<T*>(a.out) + (size_t)q0 * a.ld_out + (size_t)h * V;
  if ((unsigned)slot >= (unsigned)a.num_slots) {
    if (slot >= 0 && tid == 0) oxb_report(OXB_BAD_SLOT, slot);
    pdl_wait();
    for (int i = tid; i < n * V; i += THREADS) out[(size_t)(i / V) * a.ld_out + i % V] = lat_from<T>(0.f);
    return;
  }
  float *sr = ws_smem, *sk = sr + K, *sw = sk + K, *sv = sw + K, *part = sv + V;
  float4* S = reinterpret_cast<float4*>(a.state + ((size_t)slot * a.H + h) * K * V);
  const int pos0 = a.seq_lens[b] - n;
  float4 s[NK];
#pragma unroll
  for (int i = 0; i < NK; ++i) {  // (written by an earlier step: no need to wait for this step's kernels)
    const int k = i * R + r;
    s[i] = (on && k < K && pos0 > 0) ? S[(size_t)k * cols + c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float* bonus = a.bonus + (size_t)h * K;
  const float norm = tid < V ? a.norm[(size_t)h * V + tid] : 0.f;
  pdl_wait();
  const size_t hk = (size_t)a.H * K;
  for (int j = 0; j < n; ++j) {
    const T* row = reinterpret_cast<const T*>(a.z) + (size_t)(q0 + j) * a.ld + (size_t)h * K;
    const float* decay = a.log_decay + (size_t)(q0 + j) * hk + (size_t)h * K;
    for (int i = tid; i < 4 * K; i += THREADS) {  // r, k, decay, v
      const int what = i / K, d = i - what * K;
      ws_smem[i] = what == 2 ? expf(decay[d]) : lat_f32(row[(what == 3 ? 2 : what) * hk + d]);
    }
    const float gate = tid < V ? wkv_silu(lat_f32(row[3 * hk + tid])) : 0.f;
    __syncthreads();
    float own = 0.f;  // what the current token gives through the bonus
    for (int d = lane; d < K; d += 32) own = fmaf(sr[d] * bonus[d], sk[d], own);
    own = warp_sum(own);
    if (on) {
      const float4 v = *reinterpret_cast<const float4*>(sv + 4 * c);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < NK; ++i) {
        const int k = i * R + r;
        if (k < K) {
          const float kk = sk[k], qq = sr[k], w = sw[k];
          o.x = fmaf(qq, s[i].x, o.x);
          o.y = fmaf(qq, s[i].y, o.y);
          o.z = fmaf(qq, s[i].z, o.z);
          o.w = fmaf(qq, s[i].w, o.w);
          s[i].x = fmaf(w, s[i].x, kk * v.x);
          s[i].y = fmaf(w, s[i].y, kk * v.y);
          s[i].z = fmaf(w, s[i].z, kk * v.z);
          s[i].w = fmaf(w, s[i].w, kk * v.w);
          if (j == n - 1) S[(size_t)k * cols + c] = s[i];
        }
      }
      *reinterpret_cast<float4*>(part + r * V + 4 * c) = o;
    }
    __syncthreads();
    float o = 0.f;
    if (tid < V) {
      o = own * sv[tid];
      for (int i = 0; i < R; ++i) o += part[i * V + tid];
    }
    const float inv = rsqrtf(block_sum(o * o, red) / (float)a.dim + a.eps);
    if (tid < V) out[(size_t)j * a.ld_out + tid] = lat_from<T>(o * inv * norm * gate);
  }
}

}  // namespace oxb
