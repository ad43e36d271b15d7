// Gated delta rule: linear attention with one [K, V] float32 state per sequence and head,
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q,   y = o / rms(o) * norm * gate,
// where q, k and v have passed a short causal convolution and silu, q and k are unit vectors (q also scaled by dim^-1/2), the
// decay g = exp(-exp(A_log) softplus(a + dt_bias)) is one number per head or one per key channel, and the gate is silu of a
// projection or sigmoid of a low-rank one.  A sequence whose rows start at position 0 starts from nothing.
//
// The inputs of the convolutions are kept in a ring of `taps` rows per sequence: position p's row is row p % taps, so that the
// row a decoded token writes is none of those it reads.
//
// delta_step_kernel: token by token, the state in registers (decoded tokens, short portions, and the float32 path).
// delta_chunk.cuh: chunks of 64 tokens on the tensor cores.
#pragma once
#include "latent.cuh"

namespace oxb {

struct DeltaArgs {
  const void* z;           // [T, ld]: q | k (G heads of K values each) | v (H heads of V values) | gate | decay | beta
  int ld, gate_off, decay_off, beta_off;
  const int* query_start;  // [B + 1]
  const int* seq_lens;     // [B]
  const int* slots;        // [B] state slot, < 0: none (rows of zeros come out)
  const float* conv;       // [taps, C], C = 2 G K + H V, the last row on the current token
  int taps;
  const float* a_log;      // [H]
  const float* dt_bias;    // [H], or [H * K] with a decay per channel
  const void* decay_up;    // [H * K, decay_rank] or null: a decay per head
  int decay_rank;
  const void* gate_up;     // [H * V, gate_rank] or null: silu gate
  int gate_rank;
  const float* norm;       // [V]
  float* state;            // [num_slots, H, K, V]
  float* window;           // [num_slots, taps, C]
  int num_slots;
  void* out;               // [T, ld_out], H heads of V values
  int ld_out;
  float out_scale;
  int H, G, K, V, v_dim;
  float q_scale, eps;
  int min_rows, max_rows;  // sequences that feed fewer or more rows belong to the other kernels
  int write_window;        // 1: the step kernel keeps the convolution inputs (one row per sequence only)
};

__device__ __forceinline__ float delta_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float delta_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
// (for activations and output gates of the 16-bit path)
__device__ __forceinline__ float delta_sigmoid_fast(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ float delta_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// Dot product of n values (n % 8 == 0, both rows aligned to 8 values).
__device__ __forceinline__ float delta_dot(const float* a, const float* b, int n) {
  float s = 0.f;
#pragma unroll 4
  for (int i = 0; i < n; i += 4) {
    const float4 x = *reinterpret_cast<const float4*>(a + i), y = *reinterpret_cast<const float4*>(b + i);
    s += (x.x * y.x + x.y * y.y) + (x.z * y.z + x.w * y.w);
  }
  return s;
}
__device__ __forceinline__ float delta_dot(const __nv_bfloat16* a, const __nv_bfloat16* b, int n) {
  float s = 0.f;
#pragma unroll 4
  for (int i = 0; i < n; i += 8) {
    const uint4 x = *reinterpret_cast<const uint4*>(a + i), y = *reinterpret_cast<const uint4*>(b + i);
    const uint32_t xs[4] = {x.x, x.y, x.z, x.w}, ys[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 p = unpack_bf16x2(xs[j]), q = unpack_bf16x2(ys[j]);
      s += p.x * q.x + p.y * q.y;
    }
  }
  return s;
}

// Channel `ch` after the convolution over the rows that end at row j of a sequence's portion, and silu.
template <typename T>
__device__ __forceinline__ float delta_conv(const DeltaArgs& a, const T* z, const float* ring, int C, int pos0, int j, int ch) {
  float s = 0.f;
  for (int i = 0; i < a.taps; ++i) {
    const int r = j - (a.taps - 1) + i, p = pos0 + r;  // row of the portion, position
    if (p < 0) continue;
    const float x = r >= 0 ? lat_f32(z[(size_t)r * a.ld + ch]) : ring[(size_t)(p % a.taps) * C + ch];
    s = fmaf(a.conv[(size_t)i * C + ch], x, s);
  }
  return delta_silu(s);
}

// Output gate of value c of head h (z: the token's row).
template <typename T>
__device__ __forceinline__ float delta_gate(const DeltaArgs& a, const T* z, int h, int c) {
  if (a.gate_up == nullptr) return delta_silu(lat_f32(z[a.gate_off + h * a.V + c]));
  return delta_sigmoid(delta_dot(z + a.gate_off, reinterpret_cast<const T*>(a.gate_up) + (size_t)(h * a.V + c) * a.gate_rank, a.gate_rank));
}

// Logarithm of the decay of key channel d of head h (of the whole head without decay_up).
template <typename T>
__device__ __forceinline__ float delta_log_decay(const DeltaArgs& a, const T* z, int h, int d) {
  const float x = a.decay_up == nullptr
                      ? lat_f32(z[a.decay_off + h]) + a.dt_bias[h]
                      : delta_dot(z + a.decay_off, reinterpret_cast<const T*>(a.decay_up) + (size_t)(h * a.K + d) * a.decay_rank,
                                  a.decay_rank) + a.dt_bias[h * a.K + d];
  return -expf(a.a_log[h]) * delta_softplus(x);
}

// Channel i of the 2 K + V that head h reads: q, k, v.
__device__ __forceinline__ int delta_channel(const DeltaArgs& a, int h, int i) {
  const int g = h / (a.H / a.G);
  return i < a.K ? g * a.K + i : (i < 2 * a.K ? (a.G + g) * a.K + i - a.K : 2 * a.G * a.K + h * a.V + i - 2 * a.K);
}

// grid (H, B).  Thread (r, c) owns values 4 c .. 4 c + 3 of the state's rows r, r + R, ...; dynamic shared memory:
// 3 K + 3 V + 2 R V floats.
template <typename T, int NK, int THREADS>
__global__ void __launch_bounds__(THREADS) delta_step_kernel(const DeltaArgs a) {
  extern __shared__ __align__(16) float ds_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  const int q0 = a.query_start[b], n = a.query_start[b + 1] - q0, slot = a.slots[b];
  if (n < a.min_rows || n > a.max_rows || n <= 0) {
    pdl_wait();
    return;
  }
  const int K = a.K, V = a.V, cols = V >> 2, R = THREADS / cols, r = tid / cols, c = tid % cols;
  const bool on = r < R;
  T* out = reinterpret_cast<T*>(a.out) + (size_t)q0 * a.ld_out + (size_t)h * V;
  if ((unsigned)slot >= (unsigned)a.num_slots) {
    if (slot >= 0 && tid == 0) oxb_report(OXB_BAD_SLOT, slot);
    pdl_wait();
    for (int i = tid; i < n * V; i += THREADS) out[(size_t)(i / V) * a.ld_out + i % V] = lat_from<T>(0.f);
    return;
  }
  float *sq = ds_smem, *sk = sq + K, *sg = sk + K, *sv = sg + K, *gate = sv + V, *su = gate + V, *pa = su + V, *po = pa + R * V;
  float4* S = reinterpret_cast<float4*>(a.state + ((size_t)slot * a.H + h) * K * V);
  const int pos0 = a.seq_lens[b] - n, C = 2 * a.G * K + a.H * V;
  float* ring = a.window + (size_t)slot * a.taps * C;
  float4 s[NK];
#pragma unroll
  for (int i = 0; i < NK; ++i) {  // (written by an earlier step: no need to wait for this step's kernels)
    const int k = i * R + r;
    s[i] = (on && k < K && pos0 > 0) ? S[(size_t)k * cols + c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  const T* z = reinterpret_cast<const T*>(a.z) + (size_t)q0 * a.ld;
  const int tasks = 2 * K + V, decays = a.decay_up != nullptr ? K : 1;
  for (int j = 0; j < n; ++j) {
    const T* row = z + (size_t)j * a.ld;
    for (int i = tid; i < tasks + decays + V; i += THREADS) {
      if (i < tasks) {
        (i < 2 * K ? sq[i] : sv[i - 2 * K]) = delta_conv(a, z, ring, C, pos0, j, delta_channel(a, h, i));
      } else if (i < tasks + decays) {
        sg[i - tasks] = expf(delta_log_decay(a, row, h, i - tasks));
      } else {
        gate[i - tasks - decays] = delta_gate(a, row, h, i - tasks - decays);
      }
    }
    const float beta = delta_sigmoid(lat_f32(row[a.beta_off + h]));
    __syncthreads();
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int d = lane; d < K; d += 32) {
      const float x = sq[d], y = sk[d];
      qq += x * x;
      kk += y * y;
      qk += x * y;
    }
    const float iq = rsqrtf(warp_sum(qq) + 1e-6f) * a.q_scale, ik = rsqrtf(warp_sum(kk) + 1e-6f);
    const float dot = warp_sum(qk) * iq * ik;
    if (on) {
      float4 p = make_float4(0.f, 0.f, 0.f, 0.f), o = p;
#pragma unroll
      for (int i = 0; i < NK; ++i) {
        const int k = i * R + r;
        if (k < K) {
          const float g = sg[decays == 1 ? 0 : k], kv = sk[k] * ik, qv = sq[k] * iq;
          s[i] = make_float4(g * s[i].x, g * s[i].y, g * s[i].z, g * s[i].w);
          p.x = fmaf(kv, s[i].x, p.x);
          p.y = fmaf(kv, s[i].y, p.y);
          p.z = fmaf(kv, s[i].z, p.z);
          p.w = fmaf(kv, s[i].w, p.w);
          o.x = fmaf(qv, s[i].x, o.x);
          o.y = fmaf(qv, s[i].y, o.y);
          o.z = fmaf(qv, s[i].z, o.z);
          o.w = fmaf(qv, s[i].w, o.w);
        }
      }
      *reinterpret_cast<float4*>(pa + r * V + 4 * c) = p;
      *reinterpret_cast<float4*>(po + r * V + 4 * c) = o;
    }
    __syncthreads();
    float o = 0.f;
    if (tid < V) {
      float p = 0.f;
      for (int i = 0; i < R; ++i) {
        p += pa[i * V + tid];
        o += po[i * V + tid];
      }
      const float u = beta * (sv[tid] - p);
      su[tid] = u;
      o = fmaf(dot, u, o);  // the read-out sees this token's write: (S + k u^T)^T q = S^T q + (k . q) u
    }
    __syncthreads();
    if (on) {
      const float4 u = *reinterpret_cast<const float4*>(su + 4 * c);
#pragma unroll
      for (int i = 0; i < NK; ++i) {
        const int k = i * R + r;
        if (k < K) {
          const float kv = sk[k] * ik;
          s[i] = make_float4(fmaf(kv, u.x, s[i].x), fmaf(kv, u.y, s[i].y), fmaf(kv, u.z, s[i].z), fmaf(kv, u.w, s[i].w));
          if (j == n - 1) S[(size_t)k * cols + c] = s[i];
        }
      }
    }
    const float inv = rsqrtf(block_sum(o * o, red) / (float)a.v_dim + a.eps) * a.out_scale;
    if (tid < V) out[(size_t)j * a.ld_out + tid] = lat_from<T>(o * inv * a.norm[tid] * gate[tid]);
    if (j + 1 < n) __syncthreads();
  }
  if (a.write_window) {  // n = 1: the row written is none of those that other heads' CTAs read
    const int first = h % (a.H / a.G) == 0 ? 0 : 2 * K;
    for (int i = first + tid; i < tasks; i += THREADS) {
      const int ch = delta_channel(a, h, i);
      ring[(size_t)(pos0 % a.taps) * C + ch] = lat_f32(z[ch]);
    }
  }
}

// Keeps the last rows of every sequence's portion in its ring (after the kernels that read it).  grid (channel blocks, B).
template <typename T>
__global__ void __launch_bounds__(256) delta_window_kernel(const DeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, q0 = a.query_start[b], n = a.query_start[b + 1] - q0, slot = a.slots[b];
  const int C = 2 * a.G * a.K + a.H * a.V, ch = blockIdx.x * 256 + threadIdx.x;
  if (n <= 0 || (unsigned)slot >= (unsigned)a.num_slots || ch >= C) return;
  const T* z = reinterpret_cast<const T*>(a.z) + (size_t)q0 * a.ld;
  float* ring = a.window + (size_t)slot * a.taps * C;
  const int pos0 = a.seq_lens[b] - n;
  for (int j = max(0, n - a.taps); j < n; ++j) ring[(size_t)((pos0 + j) % a.taps) * C + ch] = lat_f32(z[(size_t)j * a.ld + ch]);
}

}  // namespace oxb
