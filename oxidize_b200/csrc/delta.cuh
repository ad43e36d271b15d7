// Gated delta rule: linear attention with one [K, V] float32 state per sequence and head,
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q,   y = o / rms(o) * norm * gate,
// where q, k and v have passed a short causal convolution and silu, q and k are unit vectors (q also scaled by dim^-1/2), the
// decay g = exp(-exp(A_log) softplus(a + dt_bias)) is one number per head or one per key channel, and the gate is silu of a
// projection or sigmoid of a low-rank one.  A sequence whose rows start at position 0 starts from nothing.
//
// The inputs of the convolutions are kept in a ring of `taps` rows per sequence: position p's row is row p % taps, so that the
// row a decoded token writes is none of those it reads.
//
// delta_step_kernel: token by token, the state in registers (short portions, and the float32 path).
// delta_decode_kernel: the same for single rows, with what can be loaded ahead on its way before this step's projections are there.
// delta_chunk.cuh: chunks of 64 tokens on the tensor cores.
#pragma once
#include "attention.cuh"
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

// Low-rank decays and gates of single-row steps: out [T, H * K | H * V] float32 = z's low-rank columns . [decay_up; gate_up]^T.
// A warp has 16 tokens x 32 columns.  grid (columns / 256, tokens / 16)
static __global__ void __launch_bounds__(256) delta_low_rank_kernel(const DeltaArgs a, float* __restrict__ out, int T) {
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int nd = a.decay_up != nullptr ? a.H * a.K : 0, ng = a.gate_up != nullptr ? a.H * a.V : 0;
  const int c0 = (blockIdx.x * 8 + warp) * 32, t0 = blockIdx.y * 16;
  const bool on = c0 < nd + ng, is_d = c0 < nd;  // (nd is a multiple of 32)
  const int rank = is_d ? a.decay_rank : a.gate_rank, col = is_d ? c0 : c0 - nd, cols = is_d ? nd : ng;
  const __nv_bfloat16* up = reinterpret_cast<const __nv_bfloat16*>(is_d ? a.decay_up : a.gate_up) + 4 * t4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  if (on) {  // (weights are static: on their way ahead of the dependency)
#pragma unroll
    for (int i = 0; i < 4; ++i)
      for (int k = 0; k < rank; k += 64) {
        const __nv_bfloat16* p = up + (size_t)min(col + 8 * i + g, cols - 1) * rank + k;
        asm volatile("prefetch.global.L2 [%0];" ::"l"(p));
      }
  }
  pdl_wait();
  if (!on) return;
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (is_d ? a.decay_off : a.gate_off) + 4 * t4;
  const __nv_bfloat16 *r0 = z + (size_t)min(t0 + g, T - 1) * a.ld, *r1 = z + (size_t)min(t0 + g + 8, T - 1) * a.ld;
#pragma unroll 4
  for (int ks = 0; ks < rank; ks += 16) {
    const uint2 x0 = *reinterpret_cast<const uint2*>(r0 + ks), x1 = *reinterpret_cast<const uint2*>(r1 + ks);
    const uint32_t av[4] = {x0.x, x1.x, x0.y, x1.y};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const uint2 w = *reinterpret_cast<const uint2*>(up + (size_t)min(col + 8 * i + g, cols - 1) * rank + ks);
      mma_bf16_16816(acc[i], av, w.x, w.y);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int t = t0 + g + 8 * (e >> 1), c = c0 + 8 * i + 2 * t4;
      if (t < T && c < nd + ng) *reinterpret_cast<float2*>(out + (size_t)t * (nd + ng) + c) = make_float2(acc[i][e], acc[i][e + 1]);
    }
}

// Steps of one row per sequence (decoding), taps <= 4 and 2 K + V <= CH * 512, 2 V <= 512: everything that does not come out of this step's
// projections (state, ring, weights) is loaded ahead of the dependency, and what does in one go.  `low`: what
// delta_low_rank_kernel left, or null without low-rank projections.  EXACT: the threads have all of the state's rows.  grid (H, B), threads as in
// delta_step_kernel; dynamic shared memory: 3 K + 2 V + 2 R V floats.
template <int NK, int CH, bool EXACT>
__global__ void __launch_bounds__(512, NK <= 8 ? 2 : 1) delta_decode_kernel(const DeltaArgs a, const float* __restrict__ low) {
  constexpr int THREADS = 512, TAPS = 4;
  extern __shared__ __align__(16) float ds_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  const int q0 = a.query_start[b], n = a.query_start[b + 1] - q0, slot = a.slots[b];
  if (n != 1) {
    pdl_wait();
    return;
  }
  const int V = a.V, cols = V >> 2, R = THREADS / cols, K = EXACT ? NK * R : a.K, r = tid / cols, c = tid % cols;
  const bool on = EXACT || r < R;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)q0 * a.ld_out + (size_t)h * V;
  if ((unsigned)slot >= (unsigned)a.num_slots) {
    if (slot >= 0 && tid == 0) oxb_report(OXB_BAD_SLOT, slot);
    pdl_wait();
    for (int i = tid; i < V; i += THREADS) out[i] = __float2bfloat16(0.f);
    return;
  }
  float *sq = ds_smem, *sk = sq + K, *sg = sk + K, *sv = sg + K, *su = sv + V, *pa = su + V, *po = pa + R * V;
  float4* S = reinterpret_cast<float4*>(a.state + ((size_t)slot * a.H + h) * K * V) + tid;  // (row r, column c: thread order)
  const int step = R * cols;
  const int pos = a.seq_lens[b] - 1, C = 2 * a.G * K + a.H * V, tasks = 2 * K + V, taps = a.taps;
  float* ring = a.window + (size_t)slot * taps * C;
  float4 s[NK];
#pragma unroll
  for (int i = 0; i < NK; ++i) {  // (written by an earlier step: no need to wait for this step's kernels)
    const int k = i * R + r;
    s[i] = (on && (EXACT || k < K) && pos > 0) ? S[i * step] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  // this thread's channels: what the earlier rows of the ring give to the convolution, and the current row's weight
  float past[CH], w_now[CH];
  int ch[CH];
#pragma unroll
  for (int e = 0; e < CH; ++e) {
    const int i = tid + e * THREADS;
    ch[e] = i < tasks ? delta_channel(a, h, i) : -1;
    past[e] = 0.f;
    w_now[e] = ch[e] >= 0 ? a.conv[(size_t)(taps - 1) * C + ch[e]] : 0.f;
    float x[TAPS - 1], w[TAPS - 1];
#pragma unroll
    for (int j = 1; j < TAPS; ++j) {  // j rows back
      const bool have = ch[e] >= 0 && j < taps && pos - j >= 0;
      x[j - 1] = have ? ring[(size_t)((pos - j) % taps) * C + ch[e]] : 0.f;
      w[j - 1] = have ? a.conv[(size_t)(taps - 1 - j) * C + ch[e]] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) past[e] = fmaf(w[j], x[j], past[e]);
  }
  const bool low_d = a.decay_up != nullptr, low_g = a.gate_up != nullptr;
  const int nd = low_d ? a.H * K : 0, decays = low_d ? K : 1;
  const float rate = expf(a.a_log[h]);
  const float dt = tid < decays ? a.dt_bias[low_d ? h * K + tid : h] : 0.f;
  const bool reads = tid >= V && tid < 2 * V;
  const float norm = reads ? a.norm[tid - V] : 0.f;
  pdl_wait();
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)q0 * a.ld;
  const float* lr = low + (size_t)q0 * (nd + (low_g ? a.H * V : 0));
  float now[CH];
#pragma unroll
  for (int e = 0; e < CH; ++e) now[e] = ch[e] >= 0 ? __bfloat162float(z[ch[e]]) : 0.f;
  const float zd = tid < decays ? (low_d ? lr[h * K + tid] : __bfloat162float(z[a.decay_off + h])) : 0.f;
  const float zg = reads ? (low_g ? lr[nd + h * V + tid - V] : __bfloat162float(z[a.gate_off + h * V + tid - V])) : 0.f;
  const float beta = delta_sigmoid(__bfloat162float(z[a.beta_off + h]));
#pragma unroll
  for (int e = 0; e < CH; ++e) {
    const int i = tid + e * THREADS;
    const float x = fmaf(w_now[e], now[e], past[e]);
    if (i < tasks) (i < 2 * K ? sq[i] : sv[i - 2 * K]) = x * delta_sigmoid_fast(x);
  }
  if (tid < decays) sg[tid] = expf(-rate * delta_softplus(zd + dt));
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
      if (EXACT || k < K) {
        const float g = sg[low_d ? k : 0], kv = sk[k] * ik, qv = sq[k] * iq;
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
  // threads 0 .. V - 1 sum up what the key recalls, the next V what the query reads
  const int v = reads ? tid - V : tid;
  float o = 0.f;
  if (tid < 2 * V) {
    const float* part = (reads ? po : pa) + v;
#pragma unroll 8
    for (int i = 0; i < R; ++i) o += part[i * V];
    if (!reads) su[v] = beta * (sv[v] - o);
  }
  __syncthreads();
  if (on) {
    const float4 u = *reinterpret_cast<const float4*>(su + 4 * c);
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int k = i * R + r;
      if (EXACT || k < K) {
        const float kv = sk[k] * ik;
        S[i * step] = make_float4(fmaf(kv, u.x, s[i].x), fmaf(kv, u.y, s[i].y), fmaf(kv, u.z, s[i].z), fmaf(kv, u.w, s[i].w));
      }
    }
  }
  const bool keep = h % (a.H / a.G) == 0;  // the row written to the ring is none of those that other heads' CTAs read
#pragma unroll
  for (int e = 0; e < CH; ++e)
    if (ch[e] >= 0 && (keep || tid + e * THREADS >= 2 * K)) ring[(size_t)(pos % taps) * C + ch[e]] = now[e];
  if (reads) o = fmaf(dot, su[v], o);  // the read-out sees this token's write
  const float inv = rsqrtf(block_sum(reads ? o * o : 0.f, red) / (float)a.v_dim + a.eps) * a.out_scale;
  if (reads) out[v] = __float2bfloat16(o * inv * norm * (low_g ? 1.f : zg) * delta_sigmoid_fast(zg));
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
