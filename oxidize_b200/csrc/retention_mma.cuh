// Retention of long portions on tcgen05: chunks of 128 tokens per CTA, one (sequence, head, segment) each.
//
// The chunk form and the split of every float32 factor into two bf16 halves are those of retention.cuh.  Per chunk
//     P  = q k^T                (tensor memory, M = tokens, N = tokens)      O1 = q S      (M = tokens, N = values)
//     O2 = decayed P . V        (P written back to tensor memory as the A operand, high and low halves)
//     dS = decayed k^T V        (k read as an MN-major operand, M = keys)
// and o_t = decay^(t+1) O1 + O2, S' = decay^n S + dS.  The state stands in registers, a row per lane and a share of its values
// per thread; its two halves go to shared memory as the MN-major B operand of the next chunk's O1.  A tile of 64 values is 128
// rows of 128 bytes with the 128-byte swizzle, tiles 16 KB apart.
#pragma once
#include "latent_mma.cuh"
#include "retention.cuh"

namespace oxb {

constexpr int RM = 128;             // tokens per chunk
constexpr int RM_TILE = RM * 128;   // bytes of a 64-value tile
constexpr int RM_THREADS = 512;     // warp w: tensor-memory lanes 32 (w % 4) .. + 31, 16-value groups w / 4 and w / 4 + 4

struct RetentionMmaPlan {
  int kt, vt, smem;  // 64-value tiles of a key and a value row; bytes of dynamic shared memory, 0: not covered
};
__host__ __device__ inline RetentionMmaPlan retention_mma_plan(int K, int V) {
  RetentionMmaPlan p{(K + 63) / 64, (V + 63) / 64, 0};
  if (K % 16 == 0 && V % 16 == 0 && K > 0 && V > 0 && K <= 128 && V <= 128) p.smem = (4 * p.kt + 3 * p.vt) * RM_TILE + 1024;
  return p;
}

// shared-memory A and B operands (low descriptor words), runtime instruction descriptor; called by a whole warp
__device__ __forceinline__ void umma_bf16_ss_if(bool issue, uint32_t tmem_d, uint32_t alo, uint32_t blo, uint32_t idesc, bool accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t.reg .b64 da, db;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "mov.b64 da, {%1, %6};\n\t"
      "mov.b64 db, {%2, %6};\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(alo), "r"(blo), "r"(idesc), "r"((uint32_t)accumulate), "r"((uint32_t)issue), "r"(UMMA_DESC_HI_SW128)
      : "memory");
}
// the same with A in tensor memory
__device__ __forceinline__ void umma_bf16_tm_if(bool issue, uint32_t tmem_d, uint32_t tmem_a, uint32_t blo, uint32_t idesc, bool accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t.reg .b64 db;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "mov.b64 db, {%2, %6};\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], db, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "r"(blo), "r"(idesc), "r"((uint32_t)accumulate), "r"((uint32_t)issue), "r"(UMMA_DESC_HI_SW128)
      : "memory");
}

// byte offset of 8-value piece `p` of row `row`
__device__ __forceinline__ uint32_t rm_piece(int row, int p) {
  return (uint32_t)((p >> 3) * RM_TILE + row * 128 + (((p & 7) ^ (row & 7)) << 4));
}

// grid (H, B, segments); OUT = false: what a segment adds to the state only (see retention_chunk_kernel).
template <bool OUT>
__global__ void __launch_bounds__(RM_THREADS, 1) retention_mma_kernel(const RetentionArgs a) {
  extern __shared__ uint8_t rm_raw[];
  __shared__ uint64_t p_done, o_done, end_done;
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  const int h = blockIdx.x, b = blockIdx.y, seg = blockIdx.z, nseg = OUT ? gridDim.z : gridDim.z + 1;
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
  const int q0 = a.query_start[b], n_all = a.query_start[b + 1] - q0, slot = a.slots[b];
  const int L = ((n_all + nseg - 1) / nseg + RM - 1) / RM * RM;  // tokens per segment
  const int s0 = seg * L, s1 = min(n_all, s0 + L), K = a.K, V = a.V;
  const bool mine = n_all >= a.min_rows && n_all <= a.max_rows && s0 < n_all && (OUT || s1 < n_all);
  if (!mine || (unsigned)slot >= (unsigned)a.num_slots) {
    if (mine && slot >= 0 && tid == 0) oxb_report(OXB_BAD_SLOT, slot);
    pdl_wait();
    if (mine && OUT) {
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(q0 + s0) * a.ld_out + (size_t)h * V;
      for (int i = tid; i < (s1 - s0) * V; i += RM_THREADS) out[(size_t)(i / V) * a.ld_out + i % V] = __float2bfloat16(0.f);
    }
    return;
  }
  const int pos0 = a.seq_lens[b] - n_all;
  const RetentionMmaPlan pl = retention_mma_plan(K, V);
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rm_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* s_kh = smem;                       // (k first: a short k's second MN-major tile, whose rows are not used, lies in k_lo)
  uint8_t* s_kl = s_kh + pl.kt * RM_TILE;
  uint8_t* s_v = s_kl + pl.kt * RM_TILE;
  uint8_t* s_qh = s_v + pl.vt * RM_TILE;
  uint8_t* s_ql = s_qh + pl.kt * RM_TILE;
  uint8_t* s_sh = s_ql + pl.kt * RM_TILE;     // state, rows = keys
  uint8_t* s_sl = s_sh + pl.vt * RM_TILE;
  float* s_red = reinterpret_cast<float*>(s_qh);  // [4][128], while q is not needed

  if (tid == 0) {
    mbar_init(&p_done, 1);
    mbar_init(&o_done, 1);
    mbar_init(&end_done, 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  const float l2 = log2f(a.decay[h]);
  const int t = (warp & 3) * 32 + lane, cq = warp >> 2;  // this thread's tensor-memory lane and first group
  const bool key = t < K;
  float S[2][16];  // state row t, groups cq and cq + 4
  float* st = a.state + ((size_t)slot * a.H + h) * K * V + (size_t)t * V;
  float* ws = a.ws + (((size_t)b * a.H + h) * nseg) * K * V + (size_t)t * V;
  const bool single = n_all <= L;  // nobody else reads or writes this state
  const bool from_state = pos0 > 0 && (OUT ? single : seg == 0);  // (written by an earlier step: no need to wait)
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 16; j += 4) {
      const int v = 16 * (cq + 4 * i) + j;
      const float4 x = (from_state && key && v < V) ? *reinterpret_cast<const float4*>(st + v) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i][j] = x.x;
      S[i][j + 1] = x.y;
      S[i][j + 2] = x.z;
      S[i][j + 3] = x.w;
    }
  pdl_wait();
  if (warp == 1) {
    tmem_alloc(&tmem_slot, OUT ? 512 : 128);
    tmem_relinquish();
  }
  if (!OUT && seg == 0) {  // the last segment of the second launch overwrites the state: the others read this copy
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 16; j += 4) {
        const int v = 16 * (cq + 4 * i) + j;
        if (key && v < V) *reinterpret_cast<float4*>(ws + v) = make_float4(S[i][j], S[i][j + 1], S[i][j + 2], S[i][j + 3]);
        S[i][j] = S[i][j + 1] = S[i][j + 2] = S[i][j + 3] = 0.f;
      }
  }
  if (OUT && !single) {
    for (int g = 0; g <= seg; ++g) {
      const float f = exp2f(l2 * (float)(g == 0 ? s0 : (seg - g) * L));
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 16; j += 4) {
          const int v = 16 * (cq + 4 * i) + j;
          if (key && v < V) {
            const float4 x = *reinterpret_cast<const float4*>(ws + (size_t)g * K * V + v);
            S[i][j] = fmaf(f, x.x, S[i][j]);
            S[i][j + 1] = fmaf(f, x.y, S[i][j + 1]);
            S[i][j + 2] = fmaf(f, x.z, S[i][j + 2]);
            S[i][j + 3] = fmaf(f, x.w, S[i][j + 3]);
          }
        }
    }
  }
  auto put_state = [&]() {  // both halves of this thread's share of the state
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int g = cq + 4 * i;
      if (!key || 16 * g >= V) continue;
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split_bf16x2(S[i][8 * p + 2 * e], S[i][8 * p + 2 * e + 1], hi[e], lo[e]);
        const uint32_t o = rm_piece(t, 2 * g + p);
        *reinterpret_cast<uint4*>(s_sh + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(s_sl + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
  };
  bool carry = pos0 > 0 || seg > 0;  // something lies in the state
  if (OUT && carry) put_state();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();  // (only now: a CTA of the next kernel must not take the tensor memory that this one waits for)
  const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_slot, 0);
  // columns: scores, later the halves of decayed P (64 each) | O1 | O2 | dS
  const uint32_t tm_p = tmem, tm_o1 = tmem + 128, tm_o2 = tmem + 256, tm_ds = OUT ? tmem + 384 : tmem;
  const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
  const bool issuer = warp == 0 && elect_one();
  const uint32_t idesc_p = umma_idesc_bf16(RM, RM), idesc_v = umma_idesc_bf16(RM, V) | UMMA_B_MN_MAJOR;
  const uint32_t idesc_s = idesc_v | UMMA_A_MN_MAJOR;
  const uint32_t kh = umma_desc_lo(smem_u32(s_kh)), kl = umma_desc_lo(smem_u32(s_kl)), qh = umma_desc_lo(smem_u32(s_qh)),
                 ql = umma_desc_lo(smem_u32(s_ql));
  const uint32_t khm = umma_desc_lo(smem_u32(s_kh), RM_TILE), klm = umma_desc_lo(smem_u32(s_kl), RM_TILE),
                 vd = umma_desc_lo(smem_u32(s_v), RM_TILE), shd = umma_desc_lo(smem_u32(s_sh), RM_TILE),
                 sld = umma_desc_lo(smem_u32(s_sl), RM_TILE);
  constexpr int STEP = 2048 >> 4;  // 16 rows of an MN-major tile

  const int K8 = K / 8, V8 = V / 8;
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)q0 * a.ld;
  uint32_t phase = 0;
  for (int c0 = s0; c0 < s1; c0 += RM, phase ^= 1) {
    const int n = min(RM, s1 - c0), ksteps = (n + 15) / 16;
    // ---- rows of the chunk: rotated, split; v as it is
    for (int i = tid; i < RM * V8; i += RM_THREADS) {
      const int r = i / V8, p = i % V8;
      const uint32_t o = rm_piece(r, p);
      if (r < n) cp_async16(s_v + o, z + (size_t)(c0 + r) * a.ld + (size_t)2 * a.H * K + (size_t)h * V + p * 8);
      else *reinterpret_cast<uint4*>(s_v + o) = make_uint4(0, 0, 0, 0);
    }
    cp_async_commit();
#pragma unroll 2
    for (int i = tid; i < RM * K8; i += RM_THREADS) {
      const int r = i / K8, p = i % K8;
      const uint32_t o = rm_piece(r, p);
      uint4 hi = make_uint4(0, 0, 0, 0), lo = hi, qhi = hi, qlo = hi;
      if (r < n) {
        const __nv_bfloat16* row = z + (size_t)(c0 + r) * a.ld + (size_t)h * K;
        const float* cs = a.cos_sin + (size_t)min(max(pos0 + c0 + r, 0), a.max_pos - 1) * a.rot;
        ret_piece(row + (size_t)a.H * K, p * 8, cs, a.rot, a.pairing, OUT ? a.k_scale : a.k_scale * exp2f(l2 * (float)(n - 1 - r)), &hi, &lo);
        if (OUT) ret_piece(row, p * 8, cs, a.rot, a.pairing, 1.f, &qhi, &qlo);
      }
      *reinterpret_cast<uint4*>(s_kh + o) = hi;
      *reinterpret_cast<uint4*>(s_kl + o) = lo;
      if (OUT) {
        *reinterpret_cast<uint4*>(s_qh + o) = qhi;
        *reinterpret_cast<uint4*>(s_ql + o) = qlo;
      }
    }
    cp_async_wait<0>();
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    __syncthreads();
    tc_fence_after();

    if (OUT) {
      if (warp == 0) {
        int acc = 0;
        for (int term = 0; term < 3; ++term) {
          const uint32_t A = term == 2 ? ql : qh, B = term == 1 ? kl : kh;
          for (int ks = 0; ks < K / 16; ++ks, acc = 1) {
            const uint32_t off = (ks >> 2) * (RM_TILE >> 4) + 2 * (ks & 3);
            umma_bf16_ss_if(issuer, tm_p, A + off, B + off, idesc_p, acc);
          }
        }
        umma_commit_if(issuer, &p_done);
        if (carry) {
          acc = 0;
          for (int term = 0; term < 3; ++term) {
            const uint32_t A = term == 2 ? ql : qh, B = term == 1 ? sld : shd;
            for (int ks = 0; ks < K / 16; ++ks, acc = 1)
              umma_bf16_ss_if(issuer, tm_o1, A + (ks >> 2) * (RM_TILE >> 4) + 2 * (ks & 3), B + ks * STEP, idesc_v, acc);
          }
        }
        umma_commit_if(issuer, &o_done);
        __syncwarp();
      }
      // ---- decayed scores: row t, groups of 16 columns
      mbar_wait_bounded(&p_done, phase, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      __syncwarp();
      tc_fence_after();
      float s[2][16];
#pragma unroll
      for (int i = 0; i < 2; ++i) tmem_ld16(tm_p + lanes + 16 * (cq + 4 * i), reinterpret_cast<uint32_t*>(s[i]));
      tmem_ld_wait();
      // k, decayed to the chunk's end, in place (its products with q are done)
      for (int i = tid; i < RM * K8; i += RM_THREADS) {
        const int r = i / K8;
        const uint32_t o = rm_piece(r, i % K8);
        if (r >= n) continue;
        const float f = exp2f(l2 * (float)(n - 1 - r));
        const uint4 h4 = *reinterpret_cast<const uint4*>(s_kh + o), l4 = *reinterpret_cast<const uint4*>(s_kl + o);
        const uint32_t hs[4] = {h4.x, h4.y, h4.z, h4.w}, ls[4] = {l4.x, l4.y, l4.z, l4.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 x = unpack_bf16x2(hs[e]), y = unpack_bf16x2(ls[e]);
          split_bf16x2((x.x + y.x) * f, (x.y + y.y) * f, hi[e], lo[e]);
        }
        *reinterpret_cast<uint4*>(s_kh + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(s_kl + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      tc_fence_before();
      __syncthreads();  // every score has been read: their columns take the halves of P
      tc_fence_after();
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int g = cq + 4 * i;
        uint32_t hi[8], lo[8];
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
          const int d = t - (16 * g + j);  // tokens between key and query
          split_bf16x2(d >= 0 ? s[i][j] * exp2f(l2 * (float)d) : 0.f, d >= 1 ? s[i][j + 1] * exp2f(l2 * (float)(d - 1)) : 0.f, hi[j >> 1],
                       lo[j >> 1]);
        }
        tmem_st4(tm_p + lanes + 8 * g, hi[0], hi[1], hi[2], hi[3]);
        tmem_st4(tm_p + lanes + 8 * g + 4, hi[4], hi[5], hi[6], hi[7]);
        tmem_st4(tm_p + lanes + 64 + 8 * g, lo[0], lo[1], lo[2], lo[3]);
        tmem_st4(tm_p + lanes + 64 + 8 * g + 4, lo[4], lo[5], lo[6], lo[7]);
      }
      tmem_st_wait();
      tc_fence_before();
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncthreads();
      tc_fence_after();
    }
    if (warp == 0) {
      if (OUT) {
        for (int half = 0; half < 2; ++half)
          for (int ks = 0; ks < ksteps; ++ks)
            umma_bf16_tm_if(issuer, tm_o2, tm_p + 64 * half + 8 * ks, vd + ks * STEP, idesc_v, half > 0 || ks > 0);
      }
      for (int half = 0; half < 2; ++half)
        for (int ks = 0; ks < ksteps; ++ks)
          umma_bf16_ss_if(issuer, tm_ds, (half ? klm : khm) + ks * STEP, vd + ks * STEP, idesc_s, half > 0 || ks > 0);
      umma_commit_if(issuer, &end_done);
      __syncwarp();
    }
    uint4 gate[2][2];
    const __nv_bfloat16* gp = z + (size_t)(c0 + t) * a.ld + (size_t)2 * a.H * K + (size_t)(a.H + h) * V;
    if (OUT) {
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          const int v = 16 * (cq + 4 * i) + 8 * p;
          gate[i][p] = (t < n && v < V) ? *reinterpret_cast<const uint4*>(gp + v) : make_uint4(0, 0, 0, 0);
        }
      mbar_wait_bounded(&o_done, phase, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
    }
    mbar_wait_bounded(&end_done, phase, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
    __syncwarp();
    tc_fence_after();
    float o[2][16];
    {
      const float fn = exp2f(l2 * (float)n);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int g = cq + 4 * i;
        if (16 * g >= V) continue;  // (the same for the whole warp)
        float x[16];
        tmem_ld16(tm_ds + lanes + 16 * g, reinterpret_cast<uint32_t*>(x));
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; ++j) S[i][j] = fmaf(fn, S[i][j], x[j]);
      }
    }
    if (OUT) {
      float ss = 0.f;
      const float ft = exp2f(l2 * (float)(t + 1));
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int g = cq + 4 * i;
        if (16 * g >= V) continue;
        float x[16];
        tmem_ld16(tm_o2 + lanes + 16 * g, reinterpret_cast<uint32_t*>(o[i]));
        if (carry) tmem_ld16(tm_o1 + lanes + 16 * g, reinterpret_cast<uint32_t*>(x));
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          if (carry) o[i][j] = fmaf(ft, x[j], o[i][j]);
          ss += o[i][j] * o[i][j];
        }
      }
      s_red[cq * RM + t] = ss;
      if (c0 + RM < s1) put_state();
    }
    tc_fence_before();
    __syncthreads();
    if (OUT) {
      const float inv = rsqrtf((s_red[t] + s_red[RM + t] + s_red[2 * RM + t] + s_red[3 * RM + t]) / (float)a.v_dim + a.eps) * a.out_scale;
      if (t < n) {
        __nv_bfloat16* op = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(q0 + c0 + t) * a.ld_out + (size_t)h * V;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int g = cq + 4 * i;
          if (16 * g >= V) continue;
#pragma unroll
          for (int p = 0; p < 2; ++p) {
            const uint32_t gs[4] = {gate[i][p].x, gate[i][p].y, gate[i][p].z, gate[i][p].w};
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 gg = unpack_bf16x2(gs[e]);
              w[e] = pack_bf16x2(o[i][8 * p + 2 * e] * inv * (gg.x / (1.f + expf(-gg.x))),
                                 o[i][8 * p + 2 * e + 1] * inv * (gg.y / (1.f + expf(-gg.y))));
            }
            *reinterpret_cast<uint4*>(op + 16 * g + 8 * p) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
      }
      __syncthreads();  // the sums have been read: q may come in
    }
    carry = true;
  }
  float* dst = OUT ? st : ws + (size_t)(seg + 1) * K * V;
  if (!OUT || s1 == n_all) {
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 16; j += 4) {
        const int v = 16 * (cq + 4 * i) + j;
        if (key && v < V) *reinterpret_cast<float4*>(dst + v) = make_float4(S[i][j], S[i][j + 1], S[i][j + 2], S[i][j + 3]);
      }
  }
  if (abort_flag) {
    // a wait gave up: give products that may still be in flight time to end before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, OUT ? 512 : 128);
}

}  // namespace oxb
