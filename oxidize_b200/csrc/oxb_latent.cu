// liboxb, entry points of models with latent attention and norms after the sum (latent.cuh, residual_norm.cuh) and of the
// float32 compute path (gemm_f32.cuh).
#include "common.cuh"
#include "gemm_f32.cuh"
#include "latent.cuh"
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
  const GemmF32Args a{x, w, bias, y, T, N, K, ldx, ldw, ldy, xs, ws, ys, act};
  oxb_launch(gemm_f32_kernel, dim3((N + F32_TILE - 1) / F32_TILE, (T + F32_TILE - 1) / F32_TILE, groups), dim3(256), 0, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}

OXB_API int oxb_latent_prep(const void* qkv, int ld, int dtype, const int* positions, const int* slots, const float* cos_sin,
                            int max_pos, int rot, int pairing, const float* norm_w, float eps, int T, int H, int nope, int rank,
                            int pad, int width, void* q_nope, int nope_ld, void* q_rows, void* q_full, int full_ld, void* cache,
                            int page, int num_blocks, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot <= 0 || rot % 2 != 0 || rank > pad || pad + rot > width || page <= 0) return (int)cudaErrorInvalidValue;
  const LatentPrepArgs a{qkv, ld, positions, slots, cos_sin, max_pos, rot, pairing, norm_w, eps, T, H, nope, rank, pad, width,
                         q_nope, nope_ld, q_rows, q_full, full_ld, cache, page, num_blocks};
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
