// Attention for long portions of a prompt: flash attention with tcgen05 over dense rows of per-head keys and values.
//
// Latent attention: keys and values are expanded per head (one matrix product over the sequence's visible rows).  Against the absorbed form
// (latent_mma.cuh) this trades (2 rank + rot) products per query, key and head for (nope + rot + v).
//
// Grouped-query attention: the visible rows' keys and values are gathered as they are, `group` query heads share a key head,
// and there is no separate rotated part.
//
// latent_gather_kernel / kv_gather_kernel copy the visible rows out of the pages into dense matrices ([rows, latent] and [rows, rot], or
// [rows, keys of all heads | values of all heads]); the
// expansion is the library's GEMM; latent_prefill_kernel attends.  A CTA owns one head and 256 query tokens of a sequence as
// two tiles of 128 rows: S = Q K^T (M = 128 tokens, N = 64 keys) goes to tensor memory, a warpgroup per tile does the softmax
// with one thread per row and writes P back to tensor memory as the A operand of O += P V (V read MN-major).  The two tiles
// alternate on the tensor core, so one's softmax runs under the other's products; K and V tiles are double-buffered by TMA.
#pragma once
#include "latent_mma.cuh"

namespace oxb {

// dense copies of the rows [span_lo[b], ...) of every sequence: lat [rows, pad], rot [rows, rot16]; sequence b's rows start
// at span_off[b] (span_off[B] = rows)
static __global__ void __launch_bounds__(128)
latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_tables, const int* __restrict__ span_lo,
                     const int* __restrict__ span_off, int B, int max_blocks, int pad, int width, int page, int num_blocks,
                     __nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ rot) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= span_off[B]) return;
  int b = 0, hi = B - 1;
  while (b < hi) {
    const int mid = (b + hi + 1) >> 1;
    if (span_off[mid] <= row) b = mid;
    else hi = mid - 1;
  }
  const int pos = span_lo[b] + row - span_off[b];
  int blk = block_tables[(size_t)b * max_blocks + pos / page];
  if ((unsigned)blk >= (unsigned)num_blocks) {
    if (lane == 0) oxb_report(OXB_BAD_BLOCK_ID, blk);
    blk = 0;
  }
  const uint4* src = reinterpret_cast<const uint4*>(cache + ((size_t)blk * page + pos % page) * width);
  const int p8 = pad / 8, r8 = (width - pad) / 8;
  uint4* l = reinterpret_cast<uint4*>(lat + (size_t)row * pad);
  uint4* r = reinterpret_cast<uint4*>(rot + (size_t)row * (width - pad));
  for (int i = lane; i < p8 + r8; i += 32) (i < p8 ? l[i] : r[i - p8]) = src[i];
}

// dense copies of the K / V pages' rows [span_lo[b], ...) of every sequence: out [rows, K of all heads | V of all heads]
static __global__ void __launch_bounds__(128)
kv_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_tables, const int* __restrict__ span_lo,
                 const int* __restrict__ span_off, int B, int max_blocks, int heads, int width, int page, int num_blocks,
                 __nv_bfloat16* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= span_off[B]) return;
  int b = 0, hi = B - 1;
  while (b < hi) {
    const int mid = (b + hi + 1) >> 1;
    if (span_off[mid] <= row) b = mid;
    else hi = mid - 1;
  }
  const int pos = span_lo[b] + row - span_off[b];
  int blk = block_tables[(size_t)b * max_blocks + pos / page];
  if ((unsigned)blk >= (unsigned)num_blocks) {
    if (lane == 0) oxb_report(OXB_BAD_BLOCK_ID, blk);
    blk = 0;
  }
  const int w8 = width / 8, n = 2 * heads * w8;
  const uint4* src = reinterpret_cast<const uint4*>(cache) + ((size_t)blk * 2 * heads * page + pos % page) * w8;
  uint4* dst = reinterpret_cast<uint4*>(out) + (size_t)row * n;
  for (int i = lane; i < n; i += 32) {
    const int head = i / w8, plane = head >= heads;  // (pages are [heads][K, V][page][width])
    dst[i] = src[(size_t)((head - plane * heads) * 2 + plane) * page * w8 + i % w8];
  }
}

constexpr int LP_KEYS = 64;       // keys per tile
constexpr int LP_M = 128;         // query tokens per tile, two tiles per CTA
constexpr int LP_QCHUNK = LP_M * 128, LP_KCHUNK = LP_KEYS * 128;  // bytes of a 64-value column chunk
constexpr int LP_WARP_TMA = 8, LP_WARP_MMA = 9, LP_THREADS = 320;
constexpr int LP_MAX_V = 128;

struct LatentPrefillArgs {
  const int* query_start;   // [B + 1]
  const int* seq_lens;      // [B]
  const int* span_lo;       // [B] first position of the dense rows
  const int* span_off;      // [B + 1] first dense row of every sequence
  const float* sink;        // [H] or null
  __nv_bfloat16* out;       // [T, H * v], rows ld_out apart
  int H, window, group;     // group: query heads per key head
  int ld_out;
  float out_scale;
  HeadGate gate;
  int nope16, rot16, full_ld;  // k-steps of 16 values of the two key parts; values per head of a query row
  int nope_ld, v_off, v_ld, v; // expanded row: head h's key at h * nope_ld, its value at v_off + h * v_ld
  float scale_log2;
};

__device__ __forceinline__ void umma_bf16_ts_if(bool issue, uint32_t tmem_d, uint32_t tmem_a, uint32_t blo, uint32_t bhi,
                                                uint32_t idesc, bool accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t.reg .b64 db;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "mov.b64 db, {%2, %6};\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], db, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "r"(blo), "r"(idesc), "r"((uint32_t)accumulate), "r"((uint32_t)issue), "r"(bhi)
      : "memory");
}

// Host: chunks and shared memory for a head's sizes; 0 bytes when the kernel does not cover them.
struct LatentPrefillPlan {
  int nope_ch, rot_ch, v_ch, smem;
};
inline LatentPrefillPlan latent_prefill_plan(int nope, int rot, int v) {
  LatentPrefillPlan p{(nope + 63) / 64, (rot + 63) / 64, (v + 63) / 64, 0};
  const int q = p.nope_ch + p.rot_ch;
  const int bytes = 2 * q * LP_QCHUNK + 2 * q * LP_KCHUNK + 2 * p.v_ch * LP_KCHUNK + 1024;
  if (v <= LP_MAX_V && bytes <= LM_DYN_SMEM) p.smem = bytes;
  return p;
}

static __global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmKV,
                      const __grid_constant__ CUtensorMap tmR, const LatentPrefillArgs a) {
  extern __shared__ uint8_t lp_raw[];
  __shared__ uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], p_full[2], pv_done[2];
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0);
  const int h = blockIdx.y, b = blockIdx.z;
  const int q0 = a.query_start[b], qlen = a.query_start[b + 1] - q0;
  const int m0 = blockIdx.x * 2 * LP_M;  // first token (of the sequence's rows) of this CTA
  const int seq_len = a.seq_lens[b];
  if (m0 >= qlen || seq_len < qlen) {
    pdl_wait();
    return;
  }
  const int pos0 = seq_len - qlen + m0;                    // position of row 0
  const int hi = min(pos0 + 2 * LP_M, seq_len) - 1;        // last key of the last row
  const int lo = a.window > 0 ? max(0, pos0 - a.window + 1) : 0;
  const int tiles = (hi - lo) / LP_KEYS + 1;
  const int krow0 = a.span_off[b] + lo - a.span_lo[b];     // dense row of key `lo`

  const int nope_ch = (a.nope16 + 3) / 4, rot_ch = (a.rot16 + 3) / 4, q_ch = nope_ch + rot_ch, v_ch = (a.v + 63) / 64;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lp_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* s_q = smem;                                     // [2 tiles][q_ch][128 rows][128 bytes]
  uint8_t* s_k = s_q + 2 * q_ch * LP_QCHUNK;               // [2][q_ch][64 keys][128 bytes]
  uint8_t* s_v = s_k + 2 * q_ch * LP_KCHUNK;               // [2][v_ch][64 keys][128 bytes]

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 128);
      mbar_init(&pv_done[i], 1);
    }
    abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == LP_WARP_MMA) {
    tmem_alloc(&tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();  // (only now: a CTA of the next kernel must not take the tensor memory that this one still waits for)
  // tensor-memory columns of tile t: S at 64 t, P at 128 + 32 t, O at 256 + 128 t
  const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_slot, 0);
  pdl_wait();

  if (warp == LP_WARP_TMA) {
    const bool leader = elect_one();
    if (leader) {
      mbar_expect_tx(&q_full, 2 * q_ch * LP_QCHUNK);
      for (int t = 0; t < 2; ++t)
        for (int c = 0; c < q_ch; ++c) {
          const int col = h * a.full_ld + (c < nope_ch ? c * 64 : a.nope16 * 16 + (c - nope_ch) * 64);
          tma_load_2d(s_q + (t * q_ch + c) * LP_QCHUNK, &tmQ, &q_full, col, q0 + m0 + t * LP_M);
        }
    }
    bool ok = true;
    for (int i = 0; i < tiles && ok; ++i) {
      const int s = i & 1, row = krow0 + i * LP_KEYS;
      if (i > 1) ok = mbar_wait_bounded(&k_empty[s], ((i >> 1) - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (leader) {
        mbar_expect_tx(&k_full[s], q_ch * LP_KCHUNK);
        uint8_t* d = s_k + s * q_ch * LP_KCHUNK;
        for (int c = 0; c < nope_ch; ++c) tma_load_2d(d + c * LP_KCHUNK, &tmKV, &k_full[s], (h / a.group) * a.nope_ld + c * 64, row);
        for (int c = 0; c < rot_ch; ++c) tma_load_2d(d + (nope_ch + c) * LP_KCHUNK, &tmR, &k_full[s], c * 64, row);
      }
      if (i > 1) ok = mbar_wait_bounded(&v_empty[s], ((i >> 1) - 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_EMPTY, blockIdx.x);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (leader) {
        mbar_expect_tx(&v_full[s], v_ch * LP_KCHUNK);
        for (int c = 0; c < v_ch; ++c)
          tma_load_2d(s_v + (s * v_ch + c) * LP_KCHUNK, &tmKV, &v_full[s], a.v_off + (h / a.group) * a.v_ld + c * 64, row);
      }
      __syncwarp();
    }
  } else if (warp == LP_WARP_MMA) {
    const bool leader = elect_one();
    constexpr uint32_t idesc_s = umma_idesc_bf16(LP_M, LP_KEYS);
    const uint32_t idesc_o = umma_idesc_bf16(LP_M, (a.v + 15) / 16 * 16) | UMMA_B_MN_MAJOR;
    const uint32_t qa = smem_u32(s_q), ka = smem_u32(s_k), va = smem_u32(s_v);
    auto first = [&](int i, int t) {  // S of tile t against keys i
      const uint32_t k0 = ka + (i & 1) * q_ch * LP_KCHUNK, q00 = qa + t * q_ch * LP_QCHUNK;
      for (int c = 0; c < q_ch; ++c) {
        const uint32_t qd = umma_desc_lo(q00 + c * LP_QCHUNK), kd = umma_desc_lo(k0 + c * LP_KCHUNK);
        const int left = c < nope_ch ? a.nope16 - 4 * c : a.rot16 - 4 * (c - nope_ch);
        if (left >= 4) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc_s>(leader, tmem + 64 * t, qd + 2 * k, kd + 2 * k, k > 0 || c > 0);
        } else {
          for (int k = 0; k < left; ++k)
            umma_bf16_if<UMMA_DESC_HI_SW128, UMMA_DESC_HI_SW128, idesc_s>(leader, tmem + 64 * t, qd + 2 * k, kd + 2 * k, k > 0 || c > 0);
        }
      }
      umma_commit_if(leader, &s_full[t]);
      if (t == 1) umma_commit_if(leader, &k_empty[i & 1]);
    };
    bool ok = mbar_wait_bounded(&q_full, 0, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x) &&
              mbar_wait_bounded(&k_full[0], 0, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    if (ok) {
      first(0, 0);
      first(0, 1);
    }
    for (int i = 0; i < tiles && ok; ++i) {
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        ok = mbar_wait_bounded(&p_full[t], i & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);  // S is free, P is written
        if (t == 0) {
          if (i + 1 < tiles)
            ok = mbar_wait_bounded(&k_full[(i + 1) & 1], ((i + 1) >> 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x) && ok;
          ok = mbar_wait_bounded(&v_full[i & 1], (i >> 1) & 1, &abort_flag, OXB_TIMEOUT_TMA_FULL, blockIdx.x) && ok;
        }
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        if (i + 1 < tiles) first(i + 1, t);
        const uint32_t vd = umma_desc_lo(va + (i & 1) * v_ch * LP_KCHUNK, LP_KCHUNK);
#pragma unroll
        for (int k = 0; k < LP_KEYS / 16; ++k)  // 16 keys: 8 columns of P, 2 KB of the value tile
          umma_bf16_ts_if(leader, tmem + 256 + 128 * t, tmem + 128 + 32 * t + 8 * k, vd + k * (2048 >> 4), UMMA_DESC_HI_SW128, idesc_o,
                          i > 0 || k > 0);
        umma_commit_if(leader, &pv_done[t]);
        if (t == 1) umma_commit_if(leader, &v_empty[i & 1]);
      }
    }
    __syncwarp();
  } else {
    // ---------------- softmax: warpgroup t = query tile, thread = query token
    const int t = warp >> 2, r = m0 + t * LP_M + (threadIdx.x & 127);
    const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t s_col = tmem + lanes + 64 * t, p_col = tmem + lanes + 128 + 32 * t, o_col = tmem + lanes + 256 + 128 * t;
    const int pos = seq_len - qlen + min(r, qlen - 1);  // rows past the end repeat the last one; never stored
    const int first_key = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const int w_lo = __reduce_max_sync(0xffffffffu, first_key), w_hi = __reduce_min_sync(0xffffffffu, pos);  // keys every row sees
    const float sink = a.sink != nullptr ? a.sink[h] * 1.4426950408889634f : -INFINITY;
    float m = sink, l = 0.f;
    const int v16 = (a.v + 15) / 16;
    for (int i = 0; i < tiles; ++i) {
      // (no early exit on a failed wait: every thread arrives at every barrier, later waits return at once)
      mbar_wait_bounded(&s_full[t], i & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
      __syncwarp();
      tc_fence_after();
      float s[LP_KEYS];
#pragma unroll
      for (int c = 0; c < LP_KEYS / 16; ++c) tmem_ld16(s_col + 16 * c, reinterpret_cast<uint32_t*>(s) + 16 * c);
      tmem_ld_wait();
      const int key0 = lo + i * LP_KEYS;
      if (key0 < w_lo || key0 + LP_KEYS - 1 > w_hi) {
        const int ka = first_key - key0, kb = pos - key0;
#pragma unroll
        for (int j = 0; j < LP_KEYS; ++j)
          if (j < ka || j > kb) s[j] = -INFINITY;
      }
      float mx[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int j = 4; j < LP_KEYS; ++j) mx[j & 3] = fmaxf(mx[j & 3], s[j]);
      const float tm = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * a.scale_log2;
      const bool move = tm > m + (i == 0 ? 0.f : LM_LAZY) || (m == -INFINITY && tm > -INFINITY);
      const float m_new = move ? tm : m;
      const float f = move ? exp2f(m - m_new) : 1.f;  // 0 when nothing was accumulated
      m = m_new;
      l *= f;
      const float base = m == -INFINITY ? 0.f : m;
      uint32_t pk[LP_KEYS / 2];
      float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < LP_KEYS; j += 2) {
        const float p0 = exp2f(fmaf(s[j], a.scale_log2, -base)), p1 = exp2f(fmaf(s[j + 1], a.scale_log2, -base));
        sum[j & 2] += p0;
        sum[(j & 2) + 1] += p1;
        pk[j >> 1] = pack_bf16x2(p0, p1);
      }
      l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
      if (i > 0) mbar_wait_bounded(&pv_done[t], (i - 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);  // P is free, O complete
      __syncwarp();
      tc_fence_after();
      if (i > 0 && __any_sync(0xffffffffu, move)) {
        for (int c = 0; c < v16; ++c) {
          uint32_t o[16];
          tmem_ld16(o_col + 16 * c, o);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
          tmem_st16(o_col + 16 * c, o);
        }
      }
      tmem_st16(p_col, pk);
      tmem_st16(p_col + 16, pk + 16);
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_full[t]);
    }
    mbar_wait_bounded(&pv_done[t], (tiles - 1) & 1, &abort_flag, OXB_TIMEOUT_ACCUM, blockIdx.x);
    __syncwarp();
    tc_fence_after();
    if (sink > -INFINITY) l += exp2f(sink - m);  // the sink's share of the denominator, once
    float inv = l > 0.f ? a.out_scale / l : 0.f;
    const __nv_bfloat16* gates = reinterpret_cast<const __nv_bfloat16*>(a.gate.rows);  // this row's
    if (gates != nullptr) {
      gates += (size_t)(q0 + min(r, qlen - 1)) * a.gate.ld;
      if (!a.gate.per_value) {
        inv *= head_gate_of(__bfloat162float(gates[h]));
        gates = nullptr;
      } else {
        gates += h * a.v;
      }
    }
    __nv_bfloat16* o_row = a.out + (size_t)(q0 + r) * a.ld_out + h * a.v;
    for (int c = 0; c < v16; ++c) {
      uint32_t o[16];
      tmem_ld16(o_col + 16 * c, o);
      tmem_ld_wait();
      if (r < qlen) {
        if (gates != nullptr) {  // (v a multiple of 16)
#pragma unroll
          for (int j = 0; j < 16; j += 8) {
            const uint4 u = *reinterpret_cast<const uint4*>(gates + 16 * c + j);
            const uint32_t us[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 z = unpack_bf16x2(us[e]);
              o[j + 2 * e] = __float_as_uint(__uint_as_float(o[j + 2 * e]) * head_gate_of(z.x));
              o[j + 2 * e + 1] = __float_as_uint(__uint_as_float(o[j + 2 * e + 1]) * head_gate_of(z.y));
            }
          }
        }
        if ((a.v | a.ld_out) % 8 == 0) {
#pragma unroll
          for (int j = 0; j < 16; j += 8) {
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e)
              w[e] = pack_bf16x2(__uint_as_float(o[j + 2 * e]) * inv, __uint_as_float(o[j + 2 * e + 1]) * inv);
            if (16 * c + j < a.v) *reinterpret_cast<uint4*>(o_row + 16 * c + j) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (16 * c + j < a.v) o_row[16 * c + j] = __float2bfloat16(__uint_as_float(o[j]) * inv);
        }
      }
    }
  }
  if (abort_flag) {
    // a wait gave up: give copies that may still be in flight time to land before the CTA exits
    for (int i = 0; i < 64; ++i) __nanosleep(2000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == LP_WARP_MMA) tmem_dealloc(tmem, 512);
}

}  // namespace oxb
