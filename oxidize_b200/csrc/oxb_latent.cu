// liboxb, entry points of models with latent attention and norms after the sum (latent.cuh, residual_norm.cuh) and of the
// float32 compute path (gemm_f32.cuh).
#include "common.cuh"
#include "gemm_f32.cuh"
#include "latent.cuh"
#include "latent_mma.cuh"
#include "latent_prefill.cuh"
#include "residual_norm.cuh"
using namespace oxb;

// dtype codes of the activation type: 0 float32, 2 bfloat16
OXB_API int oxb_residual_norm(const float* res, const void* y, float alpha, const float* w, const float* b, float* x_out,
                              void* a_out, int dtype, int T, int H, float eps, int layer_norm, cudaStream_t stream) {
  if (T <= 0) return 0;
  const ResidualNormArgs a{res, y, alpha, w, b, x_out, a_out, H, eps, layer_norm};
  return dtype == 0 ? residual_norm_launch<float>(a, T, stream) : residual_norm_launch<__nv_bfloat16>(a, T, stream);
}

OXB_API int oxb_gemm_f32(const float* x, const float* w, float* y, const float* bias, int T, int N, int K, int ldx, int ldw,
                         int ldy, int groups, long long xs, long long ws, long long ys, int act, cudaStream_t stream) {
  if (T <= 0 || N <= 0 || K <= 0 || groups <= 0) return 0;
  const GemmF32Args a{x, w, bias, y, T, N, K, ldx, ldw, ldy, xs, ws, ys, act, nullptr, nullptr};
  oxb_launch(gemm_f32_kernel, dim3((N + F32_TILE - 1) / F32_TILE, (T + F32_TILE - 1) / F32_TILE, groups), dim3(256), 0, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}

// Routed groups: y[r] = x[perm[r]] . W_g^T for the rows r of every group g (offsets [groups + 1], perm null: x[r]);
// max_rows bounds the rows of one group.
OXB_API int oxb_gemm_f32_rows(const float* x, const float* w, float* y, const int* offsets, const int* perm, int groups,
                              int max_rows, int N, int K, int ldx, int ldy, int act, cudaStream_t stream) {
  if (max_rows <= 0 || N <= 0 || K <= 0 || groups <= 0) return 0;
  const GemmF32Args a{x, w, nullptr, y, 0, N, K, ldx, K, ldy, 0, (long long)N * K, 0, act, offsets, perm};
  oxb_launch(gemm_f32_kernel, dim3((N + F32_TILE - 1) / F32_TILE, (max_rows + F32_TILE - 1) / F32_TILE, groups), dim3(256), 0,
             stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}

OXB_API int oxb_latent_prep(const void* qkv, int ld, int dtype, const int* positions, const int* slots, const float* cos_sin,
                            int max_pos, int rot, int pairing, const float* norm_w, float eps, int T, int H, int nope, int rank,
                            int pad, int width, void* q_nope, int nope_ld, void* q_rows, void* q_full, int full_ld, int full_rot, void* cache,
                            int page, int num_blocks, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot <= 0 || rot % 2 != 0 || rank > pad || pad + rot > width || page <= 0) return (int)cudaErrorInvalidValue;
  const LatentPrepArgs a{qkv, ld, positions, slots, cos_sin, max_pos, rot, pairing, norm_w, eps, T, H, nope, rank, pad, width,
                         q_nope, nope_ld, q_rows, q_full, full_ld, full_rot, cache, page, num_blocks,
                         (ld | nope | rank | pad | width | nope_ld | full_ld | full_rot) % 8 == 0 && rot % 16 == 0 && pairing == 0 &&
                             (reinterpret_cast<uintptr_t>(qkv) & 15) == 0};
  const dim3 grid(T, 1 + (H + LAT_PREP_HEADS - 1) / LAT_PREP_HEADS);
  if (dtype == 0) oxb_launch(latent_prep_kernel<float>, grid, dim3(128), 0, stream, a);
  else oxb_launch(latent_prep_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}

template <typename T>
static int latent_simt_launch(const LatentAttnArgs& a, cudaStream_t stream) {
  const dim3 grid((a.T * a.H + 3) / 4);
  if (a.width <= 128) oxb_launch(latent_attention_simt_kernel<T, 4>, grid, dim3(128), 0, stream, a);
  else if (a.width <= 320) oxb_launch(latent_attention_simt_kernel<T, 10>, grid, dim3(128), 0, stream, a);
  else if (a.width <= 640) oxb_launch(latent_attention_simt_kernel<T, 20>, grid, dim3(128), 0, stream, a);
  else if (a.width <= 1280) oxb_launch(latent_attention_simt_kernel<T, 40>, grid, dim3(128), 0, stream, a);
  else return (int)cudaErrorInvalidValue;
  OXB_CHECK_LAUNCH();
  return 0;
}

OXB_API int oxb_latent_attention_simt(const void* q, void* out, const void* cache, int dtype, const int* block_tables,
                                      const int* seq_lens, const int* query_start, const float* sink, int B, int max_blocks,
                                      int T, int H, int pad, int width, int page, int num_blocks, int window, float scale,
                                      cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  const LatentAttnArgs a{q, out, cache, block_tables, seq_lens, query_start, sink, B, max_blocks, T, H, pad, width, page,
                         num_blocks, window, scale};
  return dtype == 0 ? latent_simt_launch<float>(a, stream) : latent_simt_launch<__nv_bfloat16>(a, stream);
}

// 1 when latent_attention_mma_kernel covers rows of this shape (else: the plain kernel)
OXB_API int oxb_latent_mma_supported(int pad, int width, int page) { return latent_mma_plan(pad, width, page).ok; }

// Shared memory and cluster sizes of latent_attention_mma_kernel, set up once per device; returns the largest cluster it
// can be launched with (its key splits), or 0 on an error.
static int latent_mma_max_splits() {
  static int cached[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return 0;
  if (cached[dev]) return cached[dev];
  if (cudaFuncSetAttribute(latent_attention_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LM_DYN_SMEM) != cudaSuccess)
    return 0;
  cached[dev] = 8;
  if (cudaFuncSetAttribute(latent_attention_mma_kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) == cudaSuccess) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(LM_MAX_SPLITS, 1, 1);
    cfg.blockDim = dim3(LM_THREADS);
    cfg.dynamicSmemBytes = LM_DYN_SMEM;
    cudaLaunchAttribute at;
    at.id = cudaLaunchAttributeClusterDimension;
    at.val.clusterDim.x = LM_MAX_SPLITS;
    at.val.clusterDim.y = 1;
    at.val.clusterDim.z = 1;
    cfg.attrs = &at;
    cfg.numAttrs = 1;
    int n = 0;
    if (cudaOccupancyMaxActiveClusters(&n, latent_attention_mma_kernel, &cfg) == cudaSuccess && n > 0) cached[dev] = LM_MAX_SPLITS;
  }
  cudaGetLastError();
  return cached[dev];
}
OXB_API int oxb_latent_max_splits() { return latent_mma_max_splits(); }

// Latent attention, absorbed form, bf16: q [T, H, width] and the cache rows [num_blocks * page, width]; the B sequences
// have at most max_query_len rows each.  n_splits CTAs (at most oxb_latent_max_splits()) share the keys of a block of 32 rows.
OXB_API int oxb_latent_attention_mma(const void* q, void* out, const void* cache, const int* block_tables, const int* seq_lens,
                                     const int* query_start, const float* sink, int B, int max_blocks, int T, int H, int pad,
                                     int width, int page, int num_blocks, int window, float scale, int max_query_len,
                                     int n_splits, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_query_len <= 0) return 0;
  const LatentMmaPlan pl = latent_mma_plan(pad, width, page);
  if (!pl.ok || B > 65535) return (int)cudaErrorInvalidValue;
  const int max_splits = latent_mma_max_splits();
  if (max_splits == 0) return (int)cudaErrorInvalidDevice;
  if (n_splits > max_splits) n_splits = max_splits;
  CUtensorMap tk, tq;
  int e = oxb_make_tmap_2d(&tk, cache, (uint64_t)num_blocks * page, width, (uint64_t)width * 2, page, 64, 2);
  if (e) return e;
  e = oxb_make_tmap_2d(&tq, q, (uint64_t)T * H, width, (uint64_t)width * 2, LM_NR, 64, 2);
  if (e) return e;
  LatentMmaArgs a;
  a.block_tables = block_tables;
  a.seq_lens = seq_lens;
  a.query_start = query_start;
  a.sink = sink;
  a.out = reinterpret_cast<__nv_bfloat16*>(out);
  a.max_blocks = max_blocks;
  a.T = T;
  a.H = H;
  a.pad = pad;
  a.width = width;
  a.page = page;
  a.num_blocks = num_blocks;
  a.window = window;
  a.n_splits = n_splits < 1 ? 1 : n_splits;
  a.pairs = pl.pairs;
  a.rest = pl.rest;
  a.slots = pl.slots;
  a.rest_slots = pl.rest_slots;
  a.p_bufs = pl.p_bufs;
  a.scale_log2 = scale * 1.4426950408889634f;
  const dim3 grid((max_query_len * H + LM_NR - 1) / LM_NR * a.n_splits, B);
  const cudaError_t le =
      a.n_splits > 1 ? oxb_launch_cluster(latent_attention_mma_kernel, grid, dim3(LM_THREADS), dim3(a.n_splits, 1, 1),
                                          (size_t)pl.smem, stream, tk, tq, a)
                     : oxb_launch(latent_attention_mma_kernel, grid, dim3(LM_THREADS), (size_t)pl.smem, stream, tk, tq, a);
  if (le != cudaSuccess) return (int)le;
  OXB_CHECK_LAUNCH();
  return 0;
}

// Dense copies of the cache rows that the sequences of a step see (latent_gather_kernel); `rows` = span_off[B].
OXB_API int oxb_latent_gather(const void* cache, const int* block_tables, const int* span_lo, const int* span_off, int B, int rows,
                              int max_blocks, int pad, int width, int page, int num_blocks, void* lat, void* rot,
                              cudaStream_t stream) {
  if (rows <= 0 || B <= 0) return 0;
  if (pad % 8 != 0 || width % 8 != 0 || page <= 0) return (int)cudaErrorInvalidValue;
  oxb_launch(latent_gather_kernel, dim3((rows + 3) / 4), dim3(128), 0, stream, reinterpret_cast<const __nv_bfloat16*>(cache),
             block_tables, span_lo, span_off, B, max_blocks, pad, width, page, num_blocks, reinterpret_cast<__nv_bfloat16*>(lat),
             reinterpret_cast<__nv_bfloat16*>(rot));
  OXB_CHECK_LAUNCH();
  return 0;
}

// 1 when latent_prefill_kernel covers heads of these sizes
OXB_API int oxb_latent_prefill_supported(int nope, int rot, int v) { return latent_prefill_plan(nope, rot, v).smem > 0; }

static int prefill_launch(LatentPrefillArgs a, const void* q, const void* kv, const void* rot_rows, int B, int T, int rows, int kv_ld,
                          int max_query_len, const LatentPrefillPlan& pl, cudaStream_t stream) {
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
  if (!configured[dev]) {
    const cudaError_t ce = cudaFuncSetAttribute(latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LM_DYN_SMEM);
    if (ce != cudaSuccess) return (int)ce;
    configured[dev] = true;
  }
  CUtensorMap tq, tkv, tr;
  int e = oxb_make_tmap_2d(&tq, q, T, (uint64_t)a.H * a.full_ld, (uint64_t)a.H * a.full_ld * 2, LP_M, 64, 2);
  if (e) return e;
  e = oxb_make_tmap_2d(&tkv, kv, rows, kv_ld, (uint64_t)kv_ld * 2, LP_KEYS, 64, 2);
  if (e) return e;
  tr = tkv;  // (never read without a rotated part)
  if (a.rot16 > 0) e = oxb_make_tmap_2d(&tr, rot_rows, rows, 16 * a.rot16, (uint64_t)a.rot16 * 32, LP_KEYS, 64, 2);
  if (e) return e;
  const dim3 grid((max_query_len + 2 * LP_M - 1) / (2 * LP_M), a.H, B);
  const cudaError_t le = oxb_launch(latent_prefill_kernel, grid, dim3(LP_THREADS), (size_t)pl.smem, stream, tq, tkv, tr, a);
  if (le != cudaSuccess) return (int)le;
  OXB_CHECK_LAUNCH();
  return 0;
}

// Attention of long portions over expanded keys and values: q [T, H, full_ld] (nope | rotated part, each padded with zeros
// to a multiple of 16), kv [rows, kv_ld] (head h's key at h * nope_ld, its value at v_off + h * v_ld, all multiples of 8),
// rot [rows, rot padded to 16]; out [T, H * v].
OXB_API int oxb_latent_prefill(const void* q, const void* kv, const void* rot_rows, void* out, const int* query_start,
                               const int* seq_lens, const int* span_lo, const int* span_off, const float* sink, int B, int T, int H,
                               int rows, int nope, int rot, int v, int kv_ld, int nope_ld, int v_off, int v_ld, int window,
                               float scale, int max_query_len, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_query_len <= 0 || rows <= 0) return 0;
  const LatentPrefillPlan pl = latent_prefill_plan(nope, rot, v);
  if (pl.smem == 0 || kv_ld % 8 != 0 || nope_ld % 8 != 0 || v_off % 8 != 0 || v_ld % 8 != 0 || H > 65535 || B > 65535)
    return (int)cudaErrorInvalidValue;
  LatentPrefillArgs a;
  a.query_start = query_start;
  a.seq_lens = seq_lens;
  a.span_lo = span_lo;
  a.span_off = span_off;
  a.sink = sink;
  a.out = reinterpret_cast<__nv_bfloat16*>(out);
  a.H = H;
  a.window = window;
  a.group = 1;
  a.ld_out = H * v;
  a.out_scale = 1.f;
  a.gate = HeadGate{nullptr, 0, 0};
  a.nope16 = (nope + 15) / 16;
  a.rot16 = (rot + 15) / 16;
  a.full_ld = 16 * (a.nope16 + a.rot16);
  a.nope_ld = nope_ld;
  a.v_off = v_off;
  a.v_ld = v_ld;
  a.v = v;
  a.scale_log2 = scale * 1.4426950408889634f;
  return prefill_launch(a, q, kv, rot_rows, B, T, rows, kv_ld, max_query_len, pl, stream);
}

// Dense rows [keys of all heads | values of all heads] of the K / V pages that the sequences of a step see
// (kv_gather_kernel); `rows` = span_off[B].
OXB_API int oxb_kv_gather(const void* cache, const int* block_tables, const int* span_lo, const int* span_off, int B, int rows,
                          int max_blocks, int heads, int width, int page, int num_blocks, void* out, cudaStream_t stream) {
  if (rows <= 0 || B <= 0) return 0;
  if (width % 8 != 0 || page <= 0) return (int)cudaErrorInvalidValue;
  oxb_launch(kv_gather_kernel, dim3((rows + 3) / 4), dim3(128), 0, stream, reinterpret_cast<const __nv_bfloat16*>(cache), block_tables,
             span_lo, span_off, B, max_blocks, heads, width, page, num_blocks, reinterpret_cast<__nv_bfloat16*>(out));
  OXB_CHECK_LAUNCH();
  return 0;
}

// Grouped-query attention of long portions: q [T, H, width], kv as oxb_kv_gather leaves it, out [T, H * width] with rows
// ld_out apart; width a multiple of 16.
OXB_API int oxb_gqa_prefill(const void* q, const void* kv, void* out, int ld_out, float out_scale, const int* query_start,
                            const int* seq_lens, const int* span_lo, const int* span_off, const float* sink, int B, int T, int H,
                            int G, int rows, int width, int window, float scale, int max_query_len, const void* gate, int ld_gate,
                            int gate_per_value, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_query_len <= 0 || rows <= 0) return 0;
  const LatentPrefillPlan pl = latent_prefill_plan(width, 0, width);
  if (pl.smem == 0 || width % 16 != 0 || G <= 0 || H % G != 0 || H > 65535 || B > 65535 ||
      (gate != nullptr && gate_per_value && (ld_gate % 8 != 0 || (reinterpret_cast<uintptr_t>(gate) & 15) != 0)))
    return (int)cudaErrorInvalidValue;
  LatentPrefillArgs a;
  a.query_start = query_start;
  a.seq_lens = seq_lens;
  a.span_lo = span_lo;
  a.span_off = span_off;
  a.sink = sink;
  a.out = reinterpret_cast<__nv_bfloat16*>(out);
  a.H = H;
  a.window = window;
  a.group = H / G;
  a.ld_out = ld_out;
  a.out_scale = out_scale;
  a.gate = HeadGate{gate, ld_gate, gate_per_value};
  a.nope16 = width / 16;
  a.rot16 = 0;
  a.full_ld = width;
  a.nope_ld = width;
  a.v_off = G * width;
  a.v_ld = width;
  a.v = width;
  a.scale_log2 = scale * 1.4426950408889634f;
  return prefill_launch(a, q, kv, nullptr, B, T, rows, 2 * G * width, max_query_len, pl, stream);
}
