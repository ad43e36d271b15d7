// liboxb, entry points of attention on the scores of all heads together (joint.cuh).
#include "common.cuh"
#include "joint.cuh"
using namespace oxb;

template <typename T>
static int joint_simt_launch(const JointArgs& a, cudaStream_t stream) {
  const size_t smem = joint_simt_smem(a.H, a.W);
  if (smem > 227 * 1024) return (int)cudaErrorInvalidValue;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
  if (!configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(joint_attention_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured[dev] = true;
  }
  oxb_launch(joint_attention_simt_kernel<T>, dim3(a.T), dim3(256), smem, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}

static int joint_check(const JointArgs& a) {
  return a.G <= 0 || a.H % a.G != 0 || a.page <= 0 || a.W <= 0 || a.keep_first < 0 || (a.bias != nullptr && a.distances <= 0);
}

// Attention of a step's queries over the cache, any shape; dtype codes of q, out and cache: 0 float32, 2 bfloat16
OXB_API int oxb_joint_simt(const void* q, void* out, int ld_out, float out_scale, const void* cache, int dtype, const int* block_tables,
                           const int* seq_lens, const int* query_start, const float* sink, const float* mix, const float* bias,
                           int distances, int B, int max_blocks, int T, int H, int G, int W, int tail, int page, int num_blocks,
                           int window, int keep_first, float scale, float cap, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  const JointArgs a{q, out, ld_out, out_scale, cache, block_tables, seq_lens, query_start, sink, mix, bias, distances,
                    B, max_blocks, T, H, G, W, tail, page, num_blocks, window, keep_first, scale, cap};
  if (joint_check(a)) return (int)cudaErrorInvalidValue;
  return dtype == 0 ? joint_simt_launch<float>(a, stream) : joint_simt_launch<__nv_bfloat16>(a, stream);
}
