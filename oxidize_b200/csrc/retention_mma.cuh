// Retention of long portions on tcgen05: chunks of 128 tokens per CTA, one (sequence, head, segment) each.
//
// The chunk form and the split of every float32 factor into two bf16 halves are those of retention.cuh.  Per chunk
//     P  = q k^T                (tensor memory, M = tokens, N = tokens)      O1 = q S      (M = tokens, N = values)
//     O2 = decayed P . V        (P written back to tensor memory as the A operand, high and low halves)
//     dS = decayed k^T V        (k read as an MN-major operand, M = keys)
// and o_t = decay^(t+1) O1 + O2, S' = decay^n S + dS.  The state stands in tensor memory, a row per lane, decayed ahead of the
// product that adds dS to it; its two halves go to shared memory as the MN-major B operand of the next chunk's O1.  A tile of 64 values is 128
// rows of 128 bytes with the 128-byte swizzle, tiles 16 KB apart.
#pragma once
#include "latent_mma.cuh"
#include "retention.cuh"

namespace oxb {

constexpr int RM = 128;             // tokens per chunk
constexpr int RM_TILE = RM * 128;   // bytes of a 64-value tile
constexpr int RM_WS = 128 * 128;    // floats of a segment's block of scratch
// Data warp w (of 16): tensor-memory lanes 32 (w % 4) .. + 31, 16-value groups w / 4 and w / 4 + 4; one more warp issues the products.
constexpr int RM_WARP_MMA = 16;
constexpr int RM_THREADS = 544, RM_DATA = 512;

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

// Eight values, times `scale`, as two halves at two places.
__device__ __forceinline__ void rm_store(uint8_t* hi_at, uint8_t* lo_at, const float* v, float scale) {
  uint32_t hi[4], lo[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) split_bf16x2(v[2 * e] * scale, v[2 * e + 1] * scale, hi[e], lo[e]);
  *reinterpret_cast<uint4*>(hi_at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
  *reinterpret_cast<uint4*>(lo_at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
}
// Two pieces of eight values that rotate into each other, to o0 and o1 of the tiles hi and lo.
__device__ __forceinline__ void rm_rotate(const uint4 xu, const uint4 yu, const float* c, const float* s, uint8_t* hi, uint8_t* lo,
                                          uint32_t o0, uint32_t o1, float scale) {
  const uint32_t xs[4] = {xu.x, xu.y, xu.z, xu.w}, ys[4] = {yu.x, yu.y, yu.z, yu.w};
  float u[8], v[8];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 x = unpack_bf16x2(xs[e]), y = unpack_bf16x2(ys[e]);
    u[2 * e] = x.x * c[2 * e] - y.x * s[2 * e];
    u[2 * e + 1] = x.y * c[2 * e + 1] - y.y * s[2 * e + 1];
    v[2 * e] = y.x * c[2 * e] + x.x * s[2 * e];
    v[2 * e + 1] = y.y * c[2 * e + 1] + x.y * s[2 * e + 1];
  }
  rm_store(hi + o0, lo + o0, u, scale);
  rm_store(hi + o1, lo + o1, v, scale);
}

// grid (H, B, segments); OUT = false: what a segment adds to the state only (see retention_chunk_kernel).
template <bool OUT>
__global__ void __launch_bounds__(RM_THREADS, 1) retention_mma_kernel(const RetentionArgs a) {
  extern __shared__ uint8_t rm_raw[];
  // data -> products: rows are in shared memory, k is decayed, P is in tensor memory; products -> data: P, O1, O2 and dS
  __shared__ uint64_t rows_full, kd_full, pp_full, p_done, o_done, end_done;
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  __shared__ float s_dec[RM + 4];  // decay^0 .. decay^128
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
    mbar_init(&rows_full, RM_WARP_MMA);
    mbar_init(&kd_full, RM_WARP_MMA);
    mbar_init(&pp_full, RM_WARP_MMA);
    mbar_init(&p_done, 1);
    mbar_init(&o_done, 1);
    mbar_init(&end_done, 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  const float l2 = log2f(a.decay[h]);
  if (tid <= RM) s_dec[tid] = exp2f(l2 * (float)tid);
  const int quad = warp & 3, t = quad * 32 + lane, cq = warp >> 2;  // this thread's tensor-memory lane and first group
  const bool data = warp < RM_WARP_MMA, key = data && t < K;
  float* st = a.state + ((size_t)slot * a.H + h) * K * V + (size_t)t * V;
  // (a segment's block of the scratch is laid out thread by thread: eight pieces of four values for each of 512 threads)
  float4* ws = reinterpret_cast<float4*>(a.ws + (((size_t)b * a.H + h) * nseg) * RM_WS) + tid;
  auto put_state = [&](int g, const float* x) {  // both halves of 16 values of this thread's state row
    if (!key || 16 * g >= V) return;
#pragma unroll
    for (int p = 0; p < 2; ++p) {
      const uint32_t o = rm_piece(t, 2 * g + p);
      rm_store(s_sh + o, s_sl + o, x + 8 * p, 1.f);
    }
  };
  const bool single = n_all <= L;  // nobody else reads or writes this state
  const bool from_state = pos0 > 0 && (OUT ? single : seg == 0);  // (written by an earlier step: no need to wait)
  const bool carry0 = pos0 > 0 || seg > 0;                        // something lies in the state
  float S[2][16];  // state row t, groups cq and cq + 4
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
  if (warp == RM_WARP_MMA) {
    tmem_alloc(&tmem_slot, OUT ? 512 : 128);
    tmem_relinquish();
  }
  if (data && !OUT && seg == 0) {  // the last segment of the second launch overwrites the state: the others read this copy
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 16; j += 4) {
        ws[(4 * i + (j >> 2)) * RM_DATA] = make_float4(S[i][j], S[i][j + 1], S[i][j + 2], S[i][j + 3]);
        S[i][j] = S[i][j + 1] = S[i][j + 2] = S[i][j + 3] = 0.f;
      }
  }
  if (data && OUT && !single) {
#pragma unroll 2
    for (int g = 0; g <= seg; ++g) {
      const float f = exp2f(l2 * (float)(g == 0 ? s0 : (seg - g) * L));
      const float4* w = ws + (size_t)g * (RM_WS / 4);
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 16; j += 4) {
          const float4 x = w[(4 * i + (j >> 2)) * RM_DATA];
          S[i][j] = fmaf(f, x.x, S[i][j]);
          S[i][j + 1] = fmaf(f, x.y, S[i][j + 1]);
          S[i][j + 2] = fmaf(f, x.z, S[i][j + 2]);
          S[i][j + 3] = fmaf(f, x.w, S[i][j + 3]);
        }
    }
  }
  if (OUT && carry0) {
    put_state(cq, S[0]);
    put_state(cq + 4, S[1]);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();  // (only now: a CTA of the next kernel must not take the tensor memory that this one waits for)
  const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_slot, 0);
  // columns: scores, later the halves of decayed P (64 each) | O1 | O2 | state
  const uint32_t tm_p = tmem, tm_o1 = tmem + 128, tm_o2 = tmem + 256, tm_ds = OUT ? tmem + 384 : tmem;
  const uint32_t lanes = (uint32_t)(quad * 32) << 16;

  if (warp == RM_WARP_MMA) {
    // ---------------- products
    const bool issuer = elect_one();
    const uint32_t idesc_v = umma_idesc_bf16(RM, V) | UMMA_B_MN_MAJOR, idesc_s = idesc_v | UMMA_A_MN_MAJOR;
    constexpr uint32_t idesc_p = umma_idesc_bf16(RM, RM);
    constexpr uint32_t STEP = 2048 >> 4;  // 16 rows of an MN-major tile
    const uint32_t kh = umma_desc_lo(smem_u32(s_kh)), kl = umma_desc_lo(smem_u32(s_kl)), qh = umma_desc_lo(smem_u32(s_qh)),
                   ql = umma_desc_lo(smem_u32(s_ql));
    const uint32_t khm = umma_desc_lo(smem_u32(s_kh), RM_TILE), klm = umma_desc_lo(smem_u32(s_kl), RM_TILE),
                   vd = umma_desc_lo(smem_u32(s_v), RM_TILE), shd = umma_desc_lo(smem_u32(s_sh), RM_TILE),
                   sld = umma_desc_lo(smem_u32(s_sl), RM_TILE);
    auto k_step = [](int ks) { return (uint32_t)((ks >> 2) * (RM_TILE >> 4) + 2 * (ks & 3)); };  // 16 values of a K-major row
    auto scores = [&](uint32_t A, uint32_t B, bool first) {
      if (K == 128) {
#pragma unroll
        for (int ks = 0; ks < 8; ++ks)
          umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc_p>(issuer, tm_p, A + k_step(ks), B + k_step(ks), !first || ks > 0);
      } else {
        for (int ks = 0; ks < K / 16; ++ks)
          umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc_p>(issuer, tm_p, A + k_step(ks), B + k_step(ks), !first || ks > 0);
      }
    };
    auto of_state = [&](uint32_t A, uint32_t B, bool first) {
      if (K == 128) {
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) umma_bf16_ss_if(issuer, tm_o1, A + k_step(ks), B + ks * STEP, idesc_v, !first || ks > 0);
      } else {
        for (int ks = 0; ks < K / 16; ++ks) umma_bf16_ss_if(issuer, tm_o1, A + k_step(ks), B + ks * STEP, idesc_v, !first || ks > 0);
      }
    };
    auto ready = [&](uint64_t* bar, uint32_t phase) {
      const bool ok = mbar_wait_bounded(bar, phase, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
      const bool all = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      return all;
    };
    uint32_t phase = 0;
    bool carry = carry0;
    for (int c0 = s0; c0 < s1; c0 += RM, phase ^= 1, carry = true) {
      const int ksteps = (min(RM, s1 - c0) + 15) / 16;
      if (!ready(&rows_full, phase)) break;
      if (OUT) {
        scores(qh, kh, true);
        scores(qh, kl, false);
        scores(ql, kh, false);
        umma_commit_if(issuer, &p_done);
        if (carry) {
          of_state(qh, shd, true);
          of_state(qh, sld, false);
          of_state(ql, shd, false);
        }
        umma_commit_if(issuer, &o_done);
        if (!ready(&pp_full, phase)) break;
        for (int half = 0; half < 2; ++half)
          for (int ks = 0; ks < ksteps; ++ks)
            umma_bf16_tm_if(issuer, tm_o2, tm_p + 64 * half + 8 * ks, vd + ks * STEP, idesc_v, half > 0 || ks > 0);
        if (!ready(&kd_full, phase)) break;
      }
      for (int half = 0; half < 2; ++half)
        for (int ks = 0; ks < ksteps; ++ks)
          umma_bf16_ss_if(issuer, tm_ds, (half ? klm : khm) + ks * STEP, vd + ks * STEP, idesc_s, true);
      umma_commit_if(issuer, &end_done);
    }
    __syncwarp();
  } else {
    // ---------------- data: rows into shared memory, decayed scores, outputs and state
    {  // the state, decayed over the first chunk
      const float f = s_dec[min(RM, s1 - s0)];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (16 * (cq + 4 * i) >= V) continue;  // (the same for the whole warp)
#pragma unroll
        for (int j = 0; j < 16; ++j) S[i][j] *= f;
        tmem_st16(tm_ds + lanes + 16 * (cq + 4 * i), reinterpret_cast<const uint32_t*>(S[i]));
      }
      tmem_st_wait();
      tc_fence_before();
    }
    const int K8 = K / 8, V8 = V / 8;
    const int units = (a.pairing == 0 && a.rot % 16 == 0) ? a.rot / 16 : 0;  // pieces that rotate with a whole other piece
    const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(a.z) + (size_t)q0 * a.ld;
    const int row = tid >> 2, sub = tid & 3;  // loads: four threads per token
    auto arrive = [&](uint64_t* bar) {        // this warp's writes are done
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    auto quarter_sync = [&]() { asm volatile("bar.sync %0, 128;" ::"r"(1 + quad) : "memory"); };  // the warps of the same lanes
    auto data_sync = [&]() { asm volatile("bar.sync 5, 512;" ::: "memory"); };
    uint32_t phase = 0;
    bool carry = carry0;
    for (int c0 = s0; c0 < s1; c0 += RM, phase ^= 1, carry = true) {
      const int n = min(RM, s1 - c0);
      const bool live = row < n;
      {
        // ---- this thread's pieces of its token: v as it is, q and k rotated and split
        const __nv_bfloat16* zr = z + (size_t)(c0 + (live ? row : 0)) * a.ld;
        const uint4 *vr = reinterpret_cast<const uint4*>(zr + (size_t)2 * a.H * K + (size_t)h * V),
                    *qr = reinterpret_cast<const uint4*>(zr + (size_t)h * K), *kr = qr + (size_t)a.H * K8;
        for (int p = sub; p < V8; p += 4) {
          if (live) cp_async16(s_v + rm_piece(row, p), vr + p);
          else *reinterpret_cast<uint4*>(s_v + rm_piece(row, p)) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
        const float* cs = a.cos_sin + (size_t)min(max(pos0 + c0 + row, 0), a.max_pos - 1) * a.rot;
        const float kscale = live ? (OUT ? a.k_scale : a.k_scale * s_dec[max(n - 1 - row, 0)]) : 0.f, qscale = live ? 1.f : 0.f;
        for (int p = sub; p < units; p += 4) {
          const int p2 = p + units;
          const uint4 k0v = kr[p], k1v = kr[p2];
          uint4 q0v = k0v, q1v = k1v;
          if (OUT) {
            q0v = qr[p];
            q1v = qr[p2];
          }
          float c[8], sn[8];
#pragma unroll
          for (int j = 0; j < 8; j += 4) {
            *reinterpret_cast<float4*>(c + j) = *reinterpret_cast<const float4*>(cs + 8 * p + j);
            *reinterpret_cast<float4*>(sn + j) = *reinterpret_cast<const float4*>(cs + 8 * p2 + j);
          }
          const uint32_t o0 = rm_piece(row, p), o1 = rm_piece(row, p2);
          rm_rotate(k0v, k1v, c, sn, s_kh, s_kl, o0, o1, kscale);
          if (OUT) rm_rotate(q0v, q1v, c, sn, s_qh, s_ql, o0, o1, qscale);
        }
        for (int p = 2 * units + sub; p < K8; p += 4) {  // pieces that do not rotate, or not with a whole piece
          uint4 hi, lo;
          ret_piece(reinterpret_cast<const __nv_bfloat16*>(kr), p * 8, cs, a.rot, a.pairing, kscale, &hi, &lo);
          *reinterpret_cast<uint4*>(s_kh + rm_piece(row, p)) = hi;
          *reinterpret_cast<uint4*>(s_kl + rm_piece(row, p)) = lo;
          if (OUT) {
            ret_piece(reinterpret_cast<const __nv_bfloat16*>(qr), p * 8, cs, a.rot, a.pairing, qscale, &hi, &lo);
            *reinterpret_cast<uint4*>(s_qh + rm_piece(row, p)) = hi;
            *reinterpret_cast<uint4*>(s_ql + rm_piece(row, p)) = lo;
          }
        }
        cp_async_wait<0>();
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        arrive(&rows_full);
      }
      if (OUT) {
        mbar_wait_bounded(&p_done, phase, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
        __syncwarp();
        tc_fence_after();
        // ---- decayed scores: row t, groups of 16 columns (keys); in whole groups ahead of the query nothing is masked
        float s[2][16];
#pragma unroll
        for (int i = 0; i < 2; ++i) tmem_ld16(tm_p + lanes + 16 * (cq + 4 * i), reinterpret_cast<uint32_t*>(s[i]));
        tmem_ld_wait();
        tc_fence_before();
        quarter_sync();  // these lanes' scores have been read: their columns take the halves of P
        tc_fence_after();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int g = cq + 4 * i;
          uint32_t hi[8], lo[8];
          if (16 * g > quad * 32 + 31) {  // (the same for the whole warp, as the next case is)
#pragma unroll
            for (int j = 0; j < 8; ++j) hi[j] = lo[j] = 0u;
          } else if (16 * g + 15 <= quad * 32) {
            const float* dec = s_dec + (t - 16 * g - 15);
#pragma unroll
            for (int j = 0; j < 16; j += 2) split_bf16x2(s[i][j] * dec[15 - j], s[i][j + 1] * dec[14 - j], hi[j >> 1], lo[j >> 1]);
          } else {
            const int d0 = t - 16 * g;
#pragma unroll
            for (int j = 0; j < 16; j += 2)
              split_bf16x2(d0 >= j ? s[i][j] * s_dec[max(d0 - j, 0)] : 0.f, d0 > j ? s[i][j + 1] * s_dec[max(d0 - j - 1, 0)] : 0.f, hi[j >> 1],
                           lo[j >> 1]);
          }
          tmem_st4(tm_p + lanes + 8 * g, hi[0], hi[1], hi[2], hi[3]);
          tmem_st4(tm_p + lanes + 8 * g + 4, hi[4], hi[5], hi[6], hi[7]);
          tmem_st4(tm_p + lanes + 64 + 8 * g, lo[0], lo[1], lo[2], lo[3]);
          tmem_st4(tm_p + lanes + 64 + 8 * g + 4, lo[4], lo[5], lo[6], lo[7]);
        }
        tmem_st_wait();
        tc_fence_before();
        arrive(&pp_full);
        // ---- k, decayed to the chunk's end, in place (its products with q are done)
        if (live) {
          const float f = s_dec[n - 1 - row];
          for (int p = sub; p < K8; p += 4) {
            const uint32_t o = rm_piece(row, p);
            const uint4 h4 = *reinterpret_cast<const uint4*>(s_kh + o), l4 = *reinterpret_cast<const uint4*>(s_kl + o);
            const uint32_t hs[4] = {h4.x, h4.y, h4.z, h4.w}, ls[4] = {l4.x, l4.y, l4.z, l4.w};
            float v[8];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 x = unpack_bf16x2(hs[e]), y = unpack_bf16x2(ls[e]);
              v[2 * e] = x.x + y.x;
              v[2 * e + 1] = x.y + y.y;
            }
            rm_store(s_kh + o, s_kl + o, v, f);
          }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        arrive(&kd_full);
      }
      uint4 gate[2][2];
      if (OUT) {
        const __nv_bfloat16* gp = z + (size_t)(c0 + t) * a.ld + (size_t)2 * a.H * K + (size_t)(a.H + h) * V;
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
      // ---- the state after this chunk: for the next one's products, or the end
      const bool last = c0 + RM >= s1;
      const float fn = last ? 1.f : s_dec[min(RM, s1 - c0 - RM)];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int g = cq + 4 * i;
        if (16 * g >= V || (OUT && last && s1 < n_all)) continue;  // (the same for the whole warp)
        float x[16];
        tmem_ld16(tm_ds + lanes + 16 * g, reinterpret_cast<uint32_t*>(x));
        tmem_ld_wait();
        if (last) {
          float4* w = ws + (size_t)(seg + 1) * (RM_WS / 4);
#pragma unroll
          for (int j = 0; j < 16; j += 4) {
            const float4 y = make_float4(x[j], x[j + 1], x[j + 2], x[j + 3]);
            if (!OUT) w[(4 * i + (j >> 2)) * RM_DATA] = y;
            else if (key) *reinterpret_cast<float4*>(st + 16 * g + j) = y;
          }
          continue;
        }
        if (OUT) put_state(g, x);
#pragma unroll
        for (int j = 0; j < 16; ++j) x[j] *= fn;
        tmem_st16(tm_ds + lanes + 16 * g, reinterpret_cast<const uint32_t*>(x));
      }
      tmem_st_wait();
      if (OUT) {
        float o[2][16], ss = 0.f;
        const float ft = s_dec[t + 1];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int g = cq + 4 * i;
          if (16 * g >= V) continue;
          tmem_ld16(tm_o2 + lanes + 16 * g, reinterpret_cast<uint32_t*>(o[i]));
          if (carry) {
            float x[16];
            tmem_ld16(tm_o1 + lanes + 16 * g, reinterpret_cast<uint32_t*>(x));
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) o[i][j] = fmaf(ft, x[j], o[i][j]);
          } else {
            tmem_ld_wait();
          }
#pragma unroll
          for (int j = 0; j < 16; ++j) ss += o[i][j] * o[i][j];
        }
        s_red[cq * RM + t] = ss;
        quarter_sync();
        const float inv = rsqrtf((s_red[t] + s_red[RM + t] + s_red[2 * RM + t] + s_red[3 * RM + t]) / (float)a.v_dim + a.eps) * a.out_scale;
        tc_fence_before();
        data_sync();  // the sums and everything of this chunk in tensor and shared memory have been read: the next rows may come in
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
                w[e] = pack_bf16x2(o[i][8 * p + 2 * e] * inv * __fdividef(gg.x, 1.f + __expf(-gg.x)),
                                   o[i][8 * p + 2 * e + 1] * inv * __fdividef(gg.y, 1.f + __expf(-gg.y)));
              }
              *reinterpret_cast<uint4*>(op + 16 * g + 8 * p) = make_uint4(w[0], w[1], w[2], w[3]);
            }
          }
        }
      } else {
        tc_fence_before();
        data_sync();
      }
    }
  }
  if (abort_flag) {
    // a wait gave up: give products that may still be in flight time to end before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == RM_WARP_MMA) tmem_dealloc(tmem, OUT ? 512 : 128);
}

}  // namespace oxb
