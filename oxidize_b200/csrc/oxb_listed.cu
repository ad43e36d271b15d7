// liboxb, entry points of grouped-query attention and retention in models that list their layers (listed.cuh, retention.cuh),
// of norms on both sides of a branch (residual_norm.cuh) and of float32 router logits.
#include "common.cuh"
#include "listed.cuh"
#include "residual_norm.cuh"
#include "retention.cuh"
#include "retention_mma.cuh"
using namespace oxb;

// dtype codes of the activation type: 0 float32, 2 bfloat16
OXB_API int oxb_branch_norm(const float* res, const void* y, const float* w_post, const float* w_next, float* x_out, void* a_out,
                            int dtype, int T, int H, float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  const BranchNormArgs a{res, y, w_post, w_next, x_out, a_out, H, eps};
  return dtype == 0 ? branch_norm_launch<float>(a, T, stream) : branch_norm_launch<__nv_bfloat16>(a, T, stream);
}

OXB_API int oxb_joint_norm(const float* res, const void* y0, const void* y1, const float* w0, const float* w1, float s0, float s1,
                           const void* f, int ldf, const int* index, const float* weights, int k, const float* w_next, float* x_out,
                           void* a_out, int dtype, int T, int H, float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((w0 != nullptr) != (w1 != nullptr) || (w0 != nullptr && (y0 == nullptr || y1 == nullptr))) return (int)cudaErrorInvalidValue;
  const JointNormArgs a{res, y0, y1, w0, w1, s0, s1, f, index, weights, k, ldf, w_next, x_out, a_out, H, eps};
  return dtype == 0 ? joint_norm_launch<float>(a, T, stream) : joint_norm_launch<__nv_bfloat16>(a, T, stream);
}

OXB_API int oxb_add_normed(const float* res, const void* y, int ldy, const int* index, const float* weights, int k, const float* w,
                           int groups, float eps, const float* first, float* results, int n, const float* depth, float* x_out,
                           void* a_out, int dtype, int T, int H, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (groups <= 0 || H <= 0 || (depth != nullptr && (first == nullptr || results == nullptr || n < 0 || y == nullptr)))
    return (int)cudaErrorInvalidValue;
  const AddNormedArgs a{res, y, index, weights, k, ldy, w, groups, eps, first, results, (size_t)T * H, n, depth, x_out, a_out, H};
  return dtype == 0 ? add_normed_launch<float>(a, T, stream) : add_normed_launch<__nv_bfloat16>(a, T, stream);
}

template <typename T>
static int head_prep_launch(HeadPrepArgs a, int rows, cudaStream_t stream) {
  // few tokens: their heads are spread over CTAs, a head per warp
  const int heads = a.H + (a.shared ? 1 : 2) * a.G, groups = (heads + HEAD_PREP_WARPS - 1) / HEAD_PREP_WARPS;
  const int split = rows * groups <= 4 * oxb_sm_count() ? groups : 1;
  a.per_cta = (heads + split - 1) / split;
  const dim3 grid(rows, split), block(HEAD_PREP_WARPS * 32);
  const size_t smem = (size_t)HEAD_PREP_WARPS * a.width * sizeof(float);
  if (a.width <= 32) oxb_launch(head_prep_kernel<T, 1>, grid, block, smem, stream, a);
  else if (a.width <= 64) oxb_launch(head_prep_kernel<T, 2>, grid, block, smem, stream, a);
  else if (a.width <= 128) oxb_launch(head_prep_kernel<T, 4>, grid, block, smem, stream, a);
  else if (a.width <= 256) oxb_launch(head_prep_kernel<T, 8>, grid, block, smem, stream, a);
  else if (a.width <= 512) oxb_launch(head_prep_kernel<T, 16>, grid, block, smem, stream, a);
  else return (int)cudaErrorInvalidValue;
  OXB_CHECK_LAUNCH();
  return 0;
}

// Norms, rotation, queries and cache rows of a step's q | k | v projections (head_prep_kernel); width a multiple of 32.
OXB_API int oxb_head_prep(const void* z, int ld, int dtype, const int* positions, const int* slots, const float* cos_sin, int max_pos,
                          int rot, int pairing, const float* q_norm, const float* k_norm, int full, float eps, int T, int H, int G,
                          int dim, int width, void* q, void* cache, int page, int num_blocks, float temp_coef, float temp_every,
                          const void* v_first, int ld_first, int first_width, int v_dim, const float* v_mix, int unit, int shared,
                          int tail, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot < 0 || rot % 2 != 0 || rot > width || width % 32 != 0 || page <= 0 || H <= 0 || G <= 0 || (temp_coef != 0.f && !(temp_every > 0.f)) || (shared && (!unit || tail * (dtype == 0 ? 4 : 2) < 4)) ||
      (v_first != nullptr && (v_mix == nullptr || v_dim > first_width)))
    return (int)cudaErrorInvalidValue;
  const HeadPrepArgs a{z, ld, positions, slots, cos_sin, max_pos, rot, pairing, q_norm, k_norm, full, eps, H, G, dim, width,
                       q, cache, page, num_blocks, 0, temp_coef, temp_every, v_first, ld_first, first_width, v_dim, v_mix, unit, shared, tail};
  return dtype == 0 ? head_prep_launch<float>(a, T, stream) : head_prep_launch<__nv_bfloat16>(a, T, stream);
}

template <typename T>
static int gqa_simt_launch(const GqaSimtArgs& a, cudaStream_t stream) {
  const dim3 grid((a.T * a.H + 3) / 4);
  if (a.width <= 64) oxb_launch(gqa_attention_simt_kernel<T, 2>, grid, dim3(128), 0, stream, a);
  else if (a.width <= 128) oxb_launch(gqa_attention_simt_kernel<T, 4>, grid, dim3(128), 0, stream, a);
  else if (a.width <= 256) oxb_launch(gqa_attention_simt_kernel<T, 8>, grid, dim3(128), 0, stream, a);
  else if (a.width <= 512) oxb_launch(gqa_attention_simt_kernel<T, 16>, grid, dim3(128), 0, stream, a);
  else return (int)cudaErrorInvalidValue;
  OXB_CHECK_LAUNCH();
  return 0;
}

OXB_API int oxb_gqa_attention_simt(const void* q, void* out, int ld_out, float out_scale, const void* cache, int dtype,
                                   const int* block_tables, const int* seq_lens, const int* query_start, const float* sink, int B,
                                   int max_blocks, int T, int H, int G, int width, int page, int num_blocks, int window, float scale,
                                   const void* gate, int ld_gate, int gate_per_value, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (G <= 0 || H % G != 0 || page <= 0) return (int)cudaErrorInvalidValue;
  const GqaSimtArgs a{q, out, cache, block_tables, seq_lens, query_start, sink, B, max_blocks, T, H, G, width, page, num_blocks,
                      window, ld_out, scale, out_scale, HeadGate{gate, ld_gate, gate_per_value}};
  return dtype == 0 ? gqa_simt_launch<float>(a, stream) : gqa_simt_launch<__nv_bfloat16>(a, stream);
}

// ----------------------------------------------------------------------------- retention
template <typename T, int NK, int THREADS>
static int retention_step_go(const RetentionArgs& a, int B, cudaStream_t stream) {
  const int R = THREADS / (a.V / 4);
  oxb_launch(retention_step_kernel<T, NK, THREADS>, dim3(a.H, B), dim3(THREADS), (size_t)(2 * a.K + a.V + R * a.V) * sizeof(float), stream,
             a);
  OXB_CHECK_LAUNCH();
  return 0;
}
template <typename T>
static int retention_step_launch(const RetentionArgs& a, int B, cudaStream_t stream) {
  const int cols = a.V / 4;
  if (a.V <= 256) {
    const int nk = (a.K + 256 / cols - 1) / (256 / cols);
    if (nk <= 4) return retention_step_go<T, 4, 256>(a, B, stream);
    if (nk <= 8) return retention_step_go<T, 8, 256>(a, B, stream);
    if (nk <= 16) return retention_step_go<T, 16, 256>(a, B, stream);
    if (nk <= 32) return retention_step_go<T, 32, 256>(a, B, stream);
  }
  if (a.V <= 1024 && (a.K + 1024 / cols - 1) / (1024 / cols) <= 32) return retention_step_go<T, 32, 1024>(a, B, stream);
  return (int)cudaErrorInvalidValue;
}

template <int KT>
static int retention_chunk_go(const RetentionArgs& a, int B, int nseg, cudaStream_t stream) {
  const int smem = retention_plan(KT * 16, a.V).smem, threads = a.V / 16 * 32;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
  if (!configured[dev]) {
    const int most = retention_plan(KT * 16, 128).smem;
    cudaError_t e = cudaFuncSetAttribute(retention_chunk_kernel<KT, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(retention_chunk_kernel<KT, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e != cudaSuccess) return (int)e;
    configured[dev] = true;
  }
  if (nseg > 1) {
    oxb_launch(retention_chunk_kernel<KT, false>, dim3(a.H, B, nseg - 1), dim3(threads), (size_t)smem, stream, a);
    OXB_CHECK_LAUNCH();
  }
  oxb_launch(retention_chunk_kernel<KT, true>, dim3(a.H, B, nseg), dim3(threads), (size_t)smem, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}

static int retention_mma_go(const RetentionArgs& a, int B, int nseg, cudaStream_t stream) {
  const int smem = retention_mma_plan(a.K, a.V).smem;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
  if (!configured[dev]) {
    const int most = retention_mma_plan(128, 128).smem;
    cudaError_t e = cudaFuncSetAttribute(retention_mma_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(retention_mma_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e != cudaSuccess) return (int)e;
    configured[dev] = true;
  }
  cudaError_t le = cudaSuccess;
  if (nseg > 1) le = oxb_launch(retention_mma_kernel<false>, dim3(a.H, B, nseg - 1), dim3(RM_THREADS), (size_t)smem, stream, a);
  if (le == cudaSuccess) le = oxb_launch(retention_mma_kernel<true>, dim3(a.H, B, nseg), dim3(RM_THREADS), (size_t)smem, stream, a);
  if (le != cudaSuccess) return (int)le;
  OXB_CHECK_LAUNCH();
  return 0;
}

// 1 when retention_mma_kernel covers heads of these widths
OXB_API int oxb_retention_mma_supported(int K, int V) { return retention_mma_plan(K, V).smem > 0; }

// 1 when retention_chunk_kernel covers heads of these widths
OXB_API int oxb_retention_chunk_supported(int K, int V) {
  return (K == 32 || K == 64 || K == 96 || K == 128 || K == 192) && V % 16 == 0 && V > 0 && V <= 128 &&
         retention_plan(K, V).smem <= 227 * 1024;
}

// Retention of a step: z [T, ld] holds q | k (H heads of K values) and v | gate (H heads of V values), the state
// [num_slots, H, K, V] float32 is read and updated.  chunk 0: retention_step_kernel, 1: retention_chunk_kernel, 2:
// retention_mma_kernel (both bf16) in n_seg segments with scratch ws [B * H * n_seg * (K * V; 16384 in form 2)] floats (unused with one segment); only sequences that feed
// min_rows .. max_rows rows take part.
OXB_API int oxb_retention(const void* z, int ld, int dtype, const int* query_start, const int* seq_lens, const int* slots,
                          const float* cos_sin, int max_pos, int rot, int pairing, const float* decay, float* state, int num_slots,
                          void* out, int ld_out, float out_scale, int B, int H, int K, int V, int v_dim, float k_scale, float eps,
                          int min_rows, int max_rows, int chunk, int n_seg, float* ws, cudaStream_t stream) {
  if (B <= 0 || H <= 0) return 0;
  if (rot < 0 || rot % 2 != 0 || rot > K || V % 4 != 0 || V <= 0 || K <= 0 || B > 65535 || slots == nullptr)
    return (int)cudaErrorInvalidValue;
  const RetentionArgs a{z, ld, query_start, seq_lens, slots, cos_sin, max_pos, rot, pairing, decay, state, num_slots,
                        out, ld_out, out_scale, H, K, V, v_dim, k_scale, eps, min_rows, max_rows, ws};
  if (!chunk) return dtype == 0 ? retention_step_launch<float>(a, B, stream) : retention_step_launch<__nv_bfloat16>(a, B, stream);
  if (dtype != 2 || n_seg < 1 || n_seg > 64 || (n_seg > 1 && ws == nullptr) || ld % 8 != 0 || ld_out % 8 != 0 ||
      ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15) != 0)
    return (int)cudaErrorInvalidValue;
  if (chunk == 2) return oxb_retention_mma_supported(K, V) ? retention_mma_go(a, B, n_seg, stream) : (int)cudaErrorInvalidValue;
  if (!oxb_retention_chunk_supported(K, V)) return (int)cudaErrorInvalidValue;
  switch (K) {
    case 32: return retention_chunk_go<2>(a, B, n_seg, stream);
    case 64: return retention_chunk_go<4>(a, B, n_seg, stream);
    case 96: return retention_chunk_go<6>(a, B, n_seg, stream);
    case 128: return retention_chunk_go<8>(a, B, n_seg, stream);
    default: return retention_chunk_go<12>(a, B, n_seg, stream);
  }
}

// ----------------------------------------------------------------------------- feed-forward pieces
OXB_API int oxb_silu_mul_f32(const float* gu, float* out, const int* n_rows, int T, int I, cudaStream_t stream) {
  if (T <= 0 || I <= 0) return 0;
  const size_t blocks = ((size_t)T * I + 255) / 256;
  oxb_launch(silu_mul_f32_kernel, dim3((unsigned)(blocks < 4096 ? blocks : 4096)), dim3(256), 0, stream, gu, out, n_rows, T, I);
  OXB_CHECK_LAUNCH();
  return 0;
}

OXB_API int oxb_moe_combine_f32(const float* y, int ld, const int* inv, const float* w, int k, const float* shared, float* out, int T,
                                int H, cudaStream_t stream) {
  if (T <= 0) return 0;
  oxb_launch(moe_combine_f32_kernel, dim3(T), dim3(256), 0, stream, y, ld, inv, w, k, shared, out, H);
  OXB_CHECK_LAUNCH();
  return 0;
}

// logits [T, E] float32 = x [T, K] . w [E, K]^T, both in the activation type
OXB_API int oxb_router_logits(const void* x, const void* w, int dtype, float* out, int T, int E, int K, cudaStream_t stream) {
  if (T <= 0 || E <= 0 || K <= 0) return 0;
  if (dtype == 2 && K % 16 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 7) == 0) {
    const __nv_bfloat16 *xb = reinterpret_cast<const __nv_bfloat16*>(x), *wb = reinterpret_cast<const __nv_bfloat16*>(w);
    const int rows = (T + 15) / 16;
    if (rows * ((E + 31) / 32) >= 2 * oxb_sm_count())
      oxb_launch(router_logits_kernel<4>, dim3(rows, (E + 31) / 32), dim3(256), 0, stream, xb, wb, out, T, E, K);
    else
      oxb_launch(router_logits_kernel<1>, dim3(rows, (E + 7) / 8), dim3(256), 0, stream, xb, wb, out, T, E, K);
  } else {
    const dim3 grid((unsigned)(((size_t)T * E + 7) / 8));
    if (dtype == 0)
      oxb_launch(router_logits_any_kernel<float>, grid, dim3(256), 0, stream, reinterpret_cast<const float*>(x),
                 reinterpret_cast<const float*>(w), out, T, E, K);
    else
      oxb_launch(router_logits_any_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, reinterpret_cast<const __nv_bfloat16*>(x),
                 reinterpret_cast<const __nv_bfloat16*>(w), out, T, E, K);
  }
  OXB_CHECK_LAUNCH();
  return 0;
}
