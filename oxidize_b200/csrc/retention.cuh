// Retention: linear attention with a fixed decay per head and one [K, V] float32 state per sequence and head,
//     S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   y_t = o_t / rms(o_t) * silu(gate_t),
// with q and k rotated and k scaled on the way in.  A sequence whose rows start at position 0 starts from a zero state.
//
// retention_step_kernel: token by token, the state in registers (decoded tokens, and the float32 path).
// retention_chunk_kernel: chunks of 64 tokens on the tensor cores.  Inside a chunk that starts from state S
//     o_t = decay^(t+1) S^T q_t + sum_(s<=t) decay^(t-s) (q_t . k_s) v_s,   S' = decay^n S + sum_s decay^(n-1-s) k_s v_s^T.
// Every float32 factor (rotated q and k, decayed scores, decayed values, the state) enters the bf16 products as a high and a
// low half, x = hi + lo, and hi hi + hi lo + lo hi is summed in float32; v itself is a bf16 projection and needs one half.
// A long portion is cut into segments: a first launch computes what each segment adds to the state, the second starts every
// segment from the decayed sum of what lies before it.
#pragma once
#include "attention.cuh"
#include "latent.cuh"

namespace oxb {

struct RetentionArgs {
  const void* z;           // [T, ld]: q | k (H heads of K values each), v | gate (H heads of V values each)
  int ld;
  const int* query_start;  // [B + 1]
  const int* seq_lens;     // [B]
  const int* slots;        // [B] state slot, < 0: none (rows of zeros come out)
  const float* cos_sin;    // [max_pos, rot]
  int max_pos, rot, pairing;
  const float* decay;      // [H]
  float* state;            // [num_slots, H, K, V]
  int num_slots;
  void* out;               // [T, ld_out], H heads of V values
  int ld_out;
  float out_scale;
  int H, K, V, v_dim;
  float k_scale, eps;
  int min_rows, max_rows;  // sequences that feed fewer or more rows belong to the other kernel
  float* ws;               // [B, H, segments, K * V]: the state ahead of the portion, then what each segment but the last adds
};

// Rotated value d of a head's row; cs: the position's table row.
template <typename T>
__device__ __forceinline__ float ret_rotated(const T* v, int d, const float* cs, int rot, int pairing) {
  return d < rot ? lat_rotated(v, d, cs, rot, pairing) : lat_f32(v[d]);
}

// grid (H, B).  Thread (r, c) owns values 4 c .. 4 c + 3 of the state's rows r, r + R, ...; dynamic shared memory:
// 2 K + V + R V floats.
template <typename T, int NK, int THREADS>
__global__ void __launch_bounds__(THREADS) retention_step_kernel(const RetentionArgs a) {
  extern __shared__ float rs_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
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
  float *sq = rs_smem, *sk = sq + K, *sv = sk + K, *part = sv + V;
  float4* S = reinterpret_cast<float4*>(a.state + ((size_t)slot * a.H + h) * K * V);
  const int pos0 = a.seq_lens[b] - n;
  float4 s[NK];
#pragma unroll
  for (int i = 0; i < NK; ++i) {  // (written by an earlier step: no need to wait for this step's kernels)
    const int k = i * R + r;
    s[i] = (on && k < K && pos0 > 0) ? S[(size_t)k * cols + c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float decay = a.decay[h];
  pdl_wait();
  for (int j = 0; j < n; ++j) {
    const T* row = reinterpret_cast<const T*>(a.z) + (size_t)(q0 + j) * a.ld;
    const float* cs = a.cos_sin + (size_t)min(max(pos0 + j, 0), a.max_pos - 1) * a.rot;
    for (int d = tid; d < K; d += THREADS) {
      sq[d] = ret_rotated(row + (size_t)h * K, d, cs, a.rot, a.pairing);
      sk[d] = ret_rotated(row + (size_t)(a.H + h) * K, d, cs, a.rot, a.pairing) * a.k_scale;
    }
    const T* vg = row + (size_t)2 * a.H * K + (size_t)h * V;
    float gate = 0.f;
    if (tid < V) {
      sv[tid] = lat_f32(vg[tid]);
      gate = lat_f32(vg[(size_t)a.H * V + tid]);
    }
    __syncthreads();
    if (on) {
      const float4 v = *reinterpret_cast<const float4*>(sv + 4 * c);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < NK; ++i) {
        const int k = i * R + r;
        if (k < K) {
          const float kk = sk[k], qq = sq[k];
          s[i].x = fmaf(kk, v.x, decay * s[i].x);
          s[i].y = fmaf(kk, v.y, decay * s[i].y);
          s[i].z = fmaf(kk, v.z, decay * s[i].z);
          s[i].w = fmaf(kk, v.w, decay * s[i].w);
          o.x = fmaf(qq, s[i].x, o.x);
          o.y = fmaf(qq, s[i].y, o.y);
          o.z = fmaf(qq, s[i].z, o.z);
          o.w = fmaf(qq, s[i].w, o.w);
          if (j == n - 1) S[(size_t)k * cols + c] = s[i];
        }
      }
      *reinterpret_cast<float4*>(part + r * V + 4 * c) = o;
    }
    __syncthreads();
    float o = 0.f;
    if (tid < V)
      for (int i = 0; i < R; ++i) o += part[i * V + tid];
    const float inv = rsqrtf(block_sum(o * o, red) / (float)a.v_dim + a.eps);
    if (tid < V) out[(size_t)j * a.ld_out + tid] = lat_from<T>(o * inv * (gate / (1.f + expf(-gate))) * a.out_scale);
  }
}

// ----------------------------------------------------------------------------- chunks on the tensor cores
constexpr int RC = 64;                // tokens per chunk
constexpr int RC_PROW = RC * 2 + 16;  // bytes of a row of scores

struct RetentionPlan {
  int row_k, row_v, raw, smem;  // bytes: padded q / k row, padded v row, raw q | k rows, everything
};
__host__ __device__ inline RetentionPlan retention_plan(int K, int V) {
  RetentionPlan p;
  p.row_k = K * 2 + 16;
  p.row_v = V * 2 + 16;
  p.raw = RC * 2 * K * 2;
  p.smem = 4 * RC * p.row_k + p.raw + 2 * RC * p.row_v + 2 * RC * RC_PROW + (V / 16) * RC * 4 + (RC + 16) * 4;
  return p;
}

__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}

__device__ __forceinline__ void head_load8(const __nv_bfloat16* p, float* v) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = unpack_bf16x2(w[j]);
    v[2 * j] = f.x;
    v[2 * j + 1] = f.y;
  }
}

// eight values of the rotation of a raw row in shared memory, times `scale`, as high and low halves
__device__ __forceinline__ void ret_piece(const __nv_bfloat16* row, int d0, const float* cs, int rot, int pairing, float scale,
                                          uint4* hi, uint4* lo) {
  float v[8];
  if (d0 >= rot) {
    head_load8(row + d0, v);
  } else {
    const int half = rot >> 1;
    if (pairing == 0 && half % 8 == 0) {
      const bool first = d0 < half;
      const int p = first ? d0 : d0 - half;
      float o[8], c[8], s[8];
      head_load8(row + d0, v);
      head_load8(row + (first ? d0 + half : p), o);
#pragma unroll
      for (int j = 0; j < 8; j += 4) {
        *reinterpret_cast<float4*>(c + j) = *reinterpret_cast<const float4*>(cs + p + j);
        *reinterpret_cast<float4*>(s + j) = *reinterpret_cast<const float4*>(cs + half + p + j);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = first ? v[j] * c[j] - o[j] * s[j] : v[j] * c[j] + o[j] * s[j];
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = ret_rotated(row, d0 + j, cs, rot, pairing);
    }
  }
  uint32_t h[4], l[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) split_bf16x2(v[2 * j] * scale, v[2 * j + 1] * scale, h[j], l[j]);
  *hi = make_uint4(h[0], h[1], h[2], h[3]);
  *lo = make_uint4(l[0], l[1], l[2], l[3]);
}

// grid (H, B, segments), V / 16 warps: warp w owns values 16 w .. 16 w + 15 of the state (as S^T in accumulator registers)
// and of the outputs.  OUT = false: the segment's addition to the state only.
template <int KT, bool OUT>
__global__ void __launch_bounds__(256) retention_chunk_kernel(const RetentionArgs a) {
  constexpr int K = KT * 16;
  extern __shared__ __align__(16) uint8_t rc_smem[];
  pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, seg = blockIdx.z, nseg = OUT ? gridDim.z : gridDim.z + 1;
  const int tid = threadIdx.x, threads = blockDim.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int q0 = a.query_start[b], n_all = a.query_start[b + 1] - q0, slot = a.slots[b];
  const int L = ((n_all + nseg - 1) / nseg + RC - 1) / RC * RC;  // tokens per segment
  const int s0 = seg * L, s1 = min(n_all, s0 + L);
  const bool mine = n_all >= a.min_rows && n_all <= a.max_rows && s0 < n_all && (OUT || s1 < n_all);
  if (!mine || (unsigned)slot >= (unsigned)a.num_slots) {
    if (mine && slot >= 0 && tid == 0) oxb_report(OXB_BAD_SLOT, slot);
    pdl_wait();
    if (mine && OUT) {
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(q0 + s0) * a.ld_out + (size_t)h * a.V;
      for (int i = tid; i < (s1 - s0) * a.V; i += threads) out[(size_t)(i / a.V) * a.ld_out + i % a.V] = __float2bfloat16(0.f);
    }
    return;
  }
  const int V = a.V, pos0 = a.seq_lens[b] - n_all;
  const RetentionPlan pl = retention_plan(K, V);
  uint8_t* s_qh = rc_smem;
  uint8_t* s_ql = s_qh + RC * pl.row_k;
  uint8_t* s_kh = s_ql + RC * pl.row_k;
  uint8_t* s_kl = s_kh + RC * pl.row_k;
  uint8_t* s_raw = s_kl + RC * pl.row_k;  // [q, k][64][K]
  uint8_t* s_v = s_raw + pl.raw;          // [2][64][row_v]
  uint8_t* s_ph = s_v + 2 * RC * pl.row_v;
  uint8_t* s_pl = s_ph + RC * RC_PROW;
  float* s_red = reinterpret_cast<float*>(s_pl + RC * RC_PROW);  // [warps][64]
  float* s_dec = s_red + (V / 16) * RC;                         // decay^0 .. decay^64
  const float l2 = log2f(a.decay[h]);
  for (int i = tid; i <= RC; i += threads) s_dec[i] = exp2f(l2 * (float)i);

  float S[2 * KT][4];
  float* st = a.state + ((size_t)slot * a.H + h) * K * V + warp * 16 + g;
#pragma unroll
  for (int i = 0; i < 2 * KT; ++i) S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
  float* ws = a.ws + (((size_t)b * a.H + h) * nseg) * K * V + tid;  // (blocks are laid out thread by thread)
  const bool single = n_all <= L;  // nobody else reads or writes this state
  if (pos0 > 0 && (OUT ? single : seg == 0)) {  // (written by an earlier step: no need to wait for this step's kernels)
#pragma unroll
    for (int i = 0; i < 2 * KT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] = st[(size_t)(8 * i + 2 * t4 + (e & 1)) * V + 8 * (e >> 1)];
  }
  pdl_wait();
  if (!OUT && seg == 0) {  // the last segment of the second launch overwrites the state: the others read this copy
#pragma unroll
    for (int i = 0; i < 2 * KT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        ws[(4 * i + e) * threads] = S[i][e];
        S[i][e] = 0.f;
      }
  }
  if (OUT && !single) {
    for (int j = 0; j <= seg; ++j) {
      const float f = exp2f(l2 * (float)(j == 0 ? s0 : (seg - j) * L));
      const float* w = ws + (size_t)j * K * V;
#pragma unroll
      for (int i = 0; i < 2 * KT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][e] = fmaf(f, w[(4 * i + e) * threads], S[i][e]);
    }
  }

  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)q0 * a.ld;
  constexpr int K8 = K / 8;
  const int V8 = V / 8;
  auto fetch = [&](int c0, int buf) {  // raw rows of the chunk that starts at token c0
    const int n = min(RC, s1 - c0);
    if (OUT) {
      for (int i = tid; i < n * K8; i += threads)
        cp_async16(s_raw + i * 16, z + (size_t)(c0 + i / K8) * a.ld + (size_t)h * K + i % K8 * 8);
    }
    for (int i = tid; i < n * K8; i += threads)
      cp_async16(s_raw + (RC * K8 + i) * 16, z + (size_t)(c0 + i / K8) * a.ld + (size_t)(a.H + h) * K + i % K8 * 8);
    uint8_t* v = s_v + buf * RC * pl.row_v;
    for (int i = tid; i < RC * V8; i += threads) {
      const int r = i / V8, c = i % V8;
      if (r < n) cp_async16(v + r * pl.row_v + c * 16, z + (size_t)(c0 + r) * a.ld + (size_t)2 * a.H * K + (size_t)h * V + c * 8);
      else *reinterpret_cast<uint4*>(v + r * pl.row_v + c * 16) = make_uint4(0, 0, 0, 0);
    }
    cp_async_commit();
  };
  fetch(s0, 0);
  const int mi = lane >> 3, r8 = lane & 7;
  const uint32_t a_off = ((mi & 1) * 8 + r8) * pl.row_k + (mi >> 1) * 16;  // A operand: 16 rows x 16 values
  const uint32_t p_off = ((mi & 1) * 8 + r8) * RC_PROW + (mi >> 1) * 16;
  const uint32_t t_off = ((mi & 1) * 8 + r8) * pl.row_v + (mi >> 1) * 16;  // transposed: 16 tokens x 16 values
  const uint32_t qh = smem_u32(s_qh), ql = smem_u32(s_ql), kh = smem_u32(s_kh), kl = smem_u32(s_kl), ph = smem_u32(s_ph),
                 pl_ = smem_u32(s_pl);
  int buf = 0;
  for (int c0 = s0; c0 < s1; c0 += RC, buf ^= 1) {
    const int n = min(RC, s1 - c0);
    cp_async_wait<0>();
    __syncthreads();  // the raw rows are here; everything of the previous chunk has been read
    for (int i = tid; i < RC * K8; i += threads) {
      const int r = i / K8, d0 = i % K8 * 8;
      const uint32_t o = r * pl.row_k + d0 * 2;
      uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
      const float* cs = a.cos_sin + (size_t)min(max(pos0 + c0 + r, 0), a.max_pos - 1) * a.rot;
      if (r < n) ret_piece(reinterpret_cast<__nv_bfloat16*>(s_raw) + (RC + r) * K, d0, cs, a.rot, a.pairing, a.k_scale, &hi, &lo);
      *reinterpret_cast<uint4*>(s_kh + o) = hi;
      *reinterpret_cast<uint4*>(s_kl + o) = lo;
      if (OUT) {
        hi = lo = make_uint4(0, 0, 0, 0);
        if (r < n) ret_piece(reinterpret_cast<__nv_bfloat16*>(s_raw) + r * K, d0, cs, a.rot, a.pairing, 1.f, &hi, &lo);
        *reinterpret_cast<uint4*>(s_qh + o) = hi;
        *reinterpret_cast<uint4*>(s_ql + o) = lo;
      }
    }
    __syncthreads();
    if (c0 + RC < s1) fetch(c0 + RC, buf ^ 1);

    float O[4][2][4];
    if (OUT) {
      // decayed scores: 16 x 8 tiles on and below the diagonal, dealt out to the warps
      for (int u = warp; u < 20; u += threads >> 5) {
        const int mt = u < 2 ? 0 : (u < 6 ? 1 : (u < 12 ? 2 : 3)), nt = u - mt * (mt + 1);
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        const uint32_t kb = (nt * 8 + r8) * pl.row_k + mi * 16, qb = mt * 16 * pl.row_k + a_off;
#pragma unroll
        for (int kp = 0; kp < KT / 2; ++kp) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4(kh + kb + kp * 64, bh[0], bh[1], bh[2], bh[3]);
          ldmatrix_x4(kl + kb + kp * 64, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            uint32_t ah[4], al[4];
            ldmatrix_x4(qh + qb + kp * 64 + e * 32, ah[0], ah[1], ah[2], ah[3]);
            ldmatrix_x4(ql + qb + kp * 64 + e * 32, al[0], al[1], al[2], al[3]);
            mma_bf16_16816(acc, ah, bh[2 * e], bh[2 * e + 1]);
            mma_bf16_16816(acc, ah, bl[2 * e], bl[2 * e + 1]);
            mma_bf16_16816(acc, al, bh[2 * e], bh[2 * e + 1]);
          }
        }
        const int s = nt * 8 + 2 * t4;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = mt * 16 + g + 8 * i;
          const float p0 = s <= t ? acc[2 * i] * s_dec[t - s] : 0.f, p1 = s + 1 <= t ? acc[2 * i + 1] * s_dec[t - s - 1] : 0.f;
          uint32_t hi, lo;
          split_bf16x2(p0, p1, hi, lo);
          *reinterpret_cast<uint32_t*>(s_ph + t * RC_PROW + s * 2) = hi;
          *reinterpret_cast<uint32_t*>(s_pl + t * RC_PROW + s * 2) = lo;
        }
      }
      // what the state holds of earlier chunks
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int i = 0; i < 2; ++i) O[mt][i][0] = O[mt][i][1] = O[mt][i][2] = O[mt][i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KT; ++ks) {
        uint32_t bh[4], bl[4];  // [value half][k half]: an accumulator tile of S^T is a B operand of q S
        split_bf16x2(S[2 * ks][0], S[2 * ks][1], bh[0], bl[0]);
        split_bf16x2(S[2 * ks + 1][0], S[2 * ks + 1][1], bh[1], bl[1]);
        split_bf16x2(S[2 * ks][2], S[2 * ks][3], bh[2], bl[2]);
        split_bf16x2(S[2 * ks + 1][2], S[2 * ks + 1][3], bh[3], bl[3]);
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
          uint32_t ah[4], al[4];
          ldmatrix_x4(qh + mt * 16 * pl.row_k + a_off + ks * 32, ah[0], ah[1], ah[2], ah[3]);
          ldmatrix_x4(ql + mt * 16 * pl.row_k + a_off + ks * 32, al[0], al[1], al[2], al[3]);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16_16816(O[mt][i], ah, bh[2 * i], bh[2 * i + 1]);
            mma_bf16_16816(O[mt][i], ah, bl[2 * i], bl[2 * i + 1]);
            mma_bf16_16816(O[mt][i], al, bh[2 * i], bh[2 * i + 1]);
          }
        }
      }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) {
        const float f0 = s_dec[mt * 16 + g + 1], f1 = s_dec[mt * 16 + g + 9];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          O[mt][i][0] *= f0;
          O[mt][i][1] *= f0;
          O[mt][i][2] *= f1;
          O[mt][i][3] *= f1;
        }
      }
      __syncthreads();  // scores are complete
    }
    const float fn = s_dec[n];
#pragma unroll
    for (int i = 0; i < 2 * KT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] *= fn;
    const uint32_t vb = smem_u32(s_v) + buf * RC * pl.row_v + t_off + warp * 32;
#pragma unroll
    for (int ks = 0; ks < RC / 16; ++ks) {
      uint32_t v[4];  // (tokens 0-7, values 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15)
      ldmatrix_x4_trans(vb + ks * 16 * pl.row_v, v[0], v[1], v[2], v[3]);
      if (OUT) {
#pragma unroll
        for (int mt = ks; mt < 4; ++mt) {
          uint32_t ah[4], al[4];
          ldmatrix_x4(ph + mt * 16 * RC_PROW + p_off + ks * 32, ah[0], ah[1], ah[2], ah[3]);
          ldmatrix_x4(pl_ + mt * 16 * RC_PROW + p_off + ks * 32, al[0], al[1], al[2], al[3]);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16_16816(O[mt][i], ah, v[2 * i], v[2 * i + 1]);
            mma_bf16_16816(O[mt][i], al, v[2 * i], v[2 * i + 1]);
          }
        }
      }
      // the same registers, scaled by the decay to the chunk's end, are the A operand of S^T += v^T k
      const int s = ks * 16 + 2 * t4;
      float f[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int sj = s + (j & 1) + 8 * (j >> 1);
        f[j] = sj < n ? s_dec[n - 1 - sj] : 0.f;
      }
      uint32_t ah[4], al[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {  // A order: (values 0-7, tokens 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15)
        const float2 x = unpack_bf16x2(v[(j & 1) * 2 + (j >> 1)]);
        split_bf16x2(x.x * f[2 * (j >> 1)], x.y * f[2 * (j >> 1) + 1], ah[j], al[j]);
      }
      const uint32_t ko = ks * 16 * pl.row_k + a_off;
#pragma unroll
      for (int dt = 0; dt < KT; ++dt) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(kh + ko + dt * 32, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(kl + ko + dt * 32, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma_bf16_16816(S[2 * dt + e], ah, bh[2 * e], bh[2 * e + 1]);
          mma_bf16_16816(S[2 * dt + e], al, bh[2 * e], bh[2 * e + 1]);
          mma_bf16_16816(S[2 * dt + e], ah, bl[2 * e], bl[2 * e + 1]);
        }
      }
    }
    if (OUT) {
      // root mean square over all values of the head: this warp's 16, then across the warps
      uint32_t gate[4][2][2];
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = mt * 16 + g + 8 * i;
          const __nv_bfloat16* gp = z + (size_t)(c0 + t) * a.ld + (size_t)2 * a.H * K + (size_t)(a.H + h) * V + warp * 16 + 2 * t4;
          gate[mt][i][0] = t < n ? *reinterpret_cast<const uint32_t*>(gp) : 0u;
          gate[mt][i][1] = t < n ? *reinterpret_cast<const uint32_t*>(gp + 8) : 0u;
          float ss = O[mt][0][2 * i] * O[mt][0][2 * i] + O[mt][0][2 * i + 1] * O[mt][0][2 * i + 1] +
                     O[mt][1][2 * i] * O[mt][1][2 * i] + O[mt][1][2 * i + 1] * O[mt][1][2 * i + 1];
          ss += __shfl_xor_sync(0xffffffffu, ss, 1);
          ss += __shfl_xor_sync(0xffffffffu, ss, 2);
          if (t4 == 0) s_red[warp * RC + t] = ss;
        }
      __syncthreads();
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = mt * 16 + g + 8 * i;
          float ss = 0.f;
          for (int w = 0; w < threads >> 5; ++w) ss += s_red[w * RC + t];
          const float inv = rsqrtf(ss / (float)a.v_dim + a.eps) * a.out_scale;
          if (t < n) {
            __nv_bfloat16* op = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(q0 + c0 + t) * a.ld_out + (size_t)h * V + warp * 16 + 2 * t4;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const float2 gg = unpack_bf16x2(gate[mt][i][e]);
              *reinterpret_cast<uint32_t*>(op + 8 * e) =
                  pack_bf16x2(O[mt][e][2 * i] * inv * (gg.x / (1.f + expf(-gg.x))), O[mt][e][2 * i + 1] * inv * (gg.y / (1.f + expf(-gg.y))));
            }
          }
        }
    }
  }
  if (OUT) {
    if (s1 == n_all) {
#pragma unroll
      for (int i = 0; i < 2 * KT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[(size_t)(8 * i + 2 * t4 + (e & 1)) * V + 8 * (e >> 1)] = S[i][e];
    }
  } else {
    float* w = ws + (size_t)(seg + 1) * K * V;
#pragma unroll
    for (int i = 0; i < 2 * KT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) w[(4 * i + e) * threads] = S[i][e];
  }
}

}  // namespace oxb
