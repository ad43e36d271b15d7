// liboxb, entry points of attention on the scores of all heads together (joint.cuh, joint_prefill.cuh).
#include "common.cuh"
#include "joint.cuh"
#include "joint_prefill.cuh"
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

// Attention of a step's queries over the cache, any shape, of sequences that feed up to max_rows rows; dtype codes of q, out and cache: 0 float32, 2 bfloat16
OXB_API int oxb_joint_simt(const void* q, void* out, int ld_out, float out_scale, const void* cache, int dtype, const int* block_tables,
                           const int* seq_lens, const int* query_start, const float* sink, const float* mix, const float* bias,
                           int distances, int B, int max_blocks, int T, int H, int G, int W, int tail, int page, int num_blocks,
                           int window, int keep_first, float scale, float cap, int max_rows, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  const JointArgs a{q, out, ld_out, out_scale, cache, block_tables, seq_lens, query_start, sink, mix, bias, distances,
                    B, max_blocks, T, H, G, W, tail, page, num_blocks, window, keep_first, scale, cap, max_rows};
  if (joint_check(a)) return (int)cudaErrorInvalidValue;
  return dtype == 0 ? joint_simt_launch<float>(a, stream) : joint_simt_launch<__nv_bfloat16>(a, stream);
}

// ----------------------------------------------------------------------------- decoded tokens
constexpr int JD_MAX_SPLITS = 16;  // clusters of more than 8 CTAs where the device takes them

// Largest cluster of joint_decode_kernel; sets the kernel up once per device.
template <int HD, bool RES>
static int joint_decode_setup(int smem) {
  static int most[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return 0;
  if (most[dev] == 0) {
    cudaError_t e = cudaFuncSetAttribute(joint_decode_kernel<HD, RES>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return 0;
    most[dev] = 8;
    if (cudaFuncSetAttribute(joint_decode_kernel<HD, RES>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) == cudaSuccess) {
      cudaLaunchConfig_t cfg = {};
      cfg.gridDim = dim3(JD_MAX_SPLITS, 1, 1);
      cfg.blockDim = dim3(JD_WARPS * 32);
      cfg.dynamicSmemBytes = 227 * 1024;  // (whatever a later call needs)
      cudaLaunchAttribute at;
      at.id = cudaLaunchAttributeClusterDimension;
      at.val.clusterDim.x = JD_MAX_SPLITS;
      at.val.clusterDim.y = 1;
      at.val.clusterDim.z = 1;
      cfg.attrs = &at;
      cfg.numAttrs = 1;
      int n = 0;
      if (cudaOccupancyMaxActiveClusters(&n, joint_decode_kernel<HD, RES>, &cfg) == cudaSuccess && n > 0) most[dev] = JD_MAX_SPLITS;
    }
    cudaGetLastError();
  }
  return smem > 227 * 1024 ? 0 : most[dev];
}

template <int HD, bool RES>
static int joint_decode_launch(const JointArgs& a, int splits, cudaStream_t stream) {
  const int smem = joint_decode_smem(a.H, a.G, HD).total, most = joint_decode_setup<HD, RES>(smem);
  if (most == 0) return (int)cudaErrorInvalidValue;
  if (splits > most) splits = most;
  const dim3 grid(splits, a.T), block(JD_WARPS * 32);
  const cudaError_t e = splits > 1 ? oxb_launch_cluster(joint_decode_kernel<HD, RES>, grid, block, dim3(splits, 1, 1), (size_t)smem, stream, a)
                                   : oxb_launch(joint_decode_kernel<HD, RES>, grid, block, (size_t)smem, stream, a);
  if (e != cudaSuccess) return (int)e;
  OXB_CHECK_LAUNCH();
  return 0;
}

template <int HD>
static int joint_decode_go(const JointArgs& a, int splits, cudaStream_t stream) {
  if constexpr (HD <= 128) {
    if (joint_decode_resident(a.G, HD)) return joint_decode_launch<HD, true>(a, splits, stream);
  }
  return joint_decode_launch<HD, false>(a, splits, stream);
}

// 1 when joint_decode_kernel covers these heads (bf16, pages of 16 tokens)
OXB_API int oxb_joint_decode_supported(int H, int G, int W) {
  const bool width = W == 32 || W == 64 || W == 96 || W == 128 || W == 192 || W == 256;
  return width && G > 0 && H % G == 0 && H / G <= 16 && H <= 256 && joint_decode_smem(H, G, W).total <= 227 * 1024;
}

// The same in bf16 on pages of 16 tokens, the keys of a token dealt out to `splits` CTAs.
OXB_API int oxb_joint_decode(const void* q, void* out, int ld_out, float out_scale, const void* cache, const int* block_tables,
                             const int* seq_lens, const int* query_start, const float* sink, const float* mix, const float* bias,
                             int distances, int B, int max_blocks, int T, int H, int G, int W, int tail, int page, int num_blocks,
                             int window, int keep_first, float scale, float cap, int max_rows, int splits, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  const JointArgs a{q, out, ld_out, out_scale, cache, block_tables, seq_lens, query_start, sink, mix, bias, distances,
                    B, max_blocks, T, H, G, W, tail, page, num_blocks, window, keep_first, scale, cap, max_rows};
  if (joint_check(a) || !oxb_joint_decode_supported(H, G, W) || page != 16 || tail != 8 || T > 65535 || splits < 1 || ld_out % 4 != 0 ||
      (reinterpret_cast<uintptr_t>(out) & 7) != 0 || ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) != 0)
    return (int)cudaErrorInvalidValue;
  switch (W) {
    case 32: return joint_decode_go<32>(a, splits, stream);
    case 64: return joint_decode_go<64>(a, splits, stream);
    case 96: return joint_decode_go<96>(a, splits, stream);
    case 128: return joint_decode_go<128>(a, splits, stream);
    case 192: return joint_decode_go<192>(a, splits, stream);
    default: return joint_decode_go<256>(a, splits, stream);
  }
}

// ----------------------------------------------------------------------------- long portions
static int joint_prefill_go(const JointPrefillArgs& x, int wide_blocks, cudaStream_t stream) {
  const JointArgs& a = x.a;
  const int quads = (a.H + 3) / 4, same = a.H / a.G % 4 == 0;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
  if (!configured[dev]) {
    constexpr cudaFuncAttribute attr = cudaFuncAttributeMaxDynamicSharedMemorySize;
    cudaError_t e = cudaFuncSetAttribute(joint_scores_kernel, attr, joint_scores_smem(128));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(joint_values_kernel, attr, joint_values_smem(128));
    if (e != cudaSuccess) return (int)e;
    configured[dev] = true;
  }
  CUtensorMap tq, tk, tt;
  const uint64_t rows = (uint64_t)a.num_blocks * a.G * 16, pitch = (uint64_t)(a.W + a.tail) * 2;
  int e = oxb_make_tmap_2d(&tq, a.q, a.T, (uint64_t)a.H * a.W, (uint64_t)a.H * a.W * 2, JP_M, 64, 2);
  if (e == 0) e = oxb_make_tmap_2d(&tk, a.cache, rows, a.W + a.tail, pitch, 16, 64, 2);
  if (e == 0) e = oxb_make_tmap_bytes(&tt, a.cache, rows, pitch, 16, 16);
  if (e) return e;
  // the tiles of 128 tokens are dealt out to as many CTAs as run at once
  int parts = oxb_sm_count() / (wide_blocks * quads);
  if (parts > x.tiles / 16) parts = x.tiles / 16;
  if (parts < 1) parts = 1;
  const dim3 mix((unsigned)x.blocks * 2, (x.tiles + JM_TILES - 1) / JM_TILES);
  cudaError_t le = oxb_launch(joint_scores_kernel, dim3(wide_blocks, quads, parts), dim3(JC_THREADS), (size_t)joint_scores_smem(a.W),
                              stream, tq, tk, tt, x, same);
  if (le == cudaSuccess)
    le = a.H <= 16 ? oxb_launch(joint_mix_kernel<1>, mix, dim3(JM_WARPS * 32), 0, stream, x)
                   : oxb_launch(joint_mix_kernel<2>, mix, dim3(JM_WARPS * 32), 0, stream, x);
  if (le == cudaSuccess)
    le = oxb_launch(joint_values_kernel, dim3(wide_blocks, a.H), dim3(JV_THREADS), (size_t)joint_values_smem(a.W), stream, tk, x);
  if (le != cudaSuccess) return (int)le;
  OXB_CHECK_LAUNCH();
  return 0;
}

// 1 when the kernels for long portions cover these heads (bf16, pages of 16 tokens)
OXB_API int oxb_joint_prefill_supported(int H, int G, int W) {
  return W >= 16 && W <= 128 && W % 16 == 0 && G > 0 && H % G == 0 && H <= 32;
}

// The same in bf16 on pages of 16 tokens for the given blocks of 16 tokens (block0 .. block0 + blocks, of long portions), which
// wide [wide_blocks, 2] groups by up to eight of one sequence; scratch scores blocks * (H / 4 rounded up) *
// tiles * 8192 bytes, weights blocks * H * 16 * tiles * 64 bytes and stats blocks * H * 16 * tiles * 8 bytes, tiles: the most tiles
// of 32 keys that a block sees.
OXB_API int oxb_joint_prefill(const void* q, void* out, int ld_out, float out_scale, const void* cache, const int* block_tables,
                              const int* seq_lens, const int* query_start, const float* sink, const float* mix, const float* bias,
                              int distances, int B, int max_blocks, int T, int H, int G, int W, int tail, int page, int num_blocks,
                              int window, int keep_first, float scale, float cap, const int* block_seq, const int* block_row,
                              const int* wide, int block0, int blocks, int wide_blocks, void* scores, void* weights, void* stats,
                              int tiles, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || blocks <= 0 || wide_blocks <= 0) return 0;
  const JointArgs a{q, out, ld_out, out_scale, cache, block_tables, seq_lens, query_start, sink, mix, bias, distances,
                    B, max_blocks, T, H, G, W, tail, page, num_blocks, window, keep_first, scale, cap, 0};
  if (joint_check(a) || !oxb_joint_prefill_supported(H, G, W) || page != 16 || tail != 8 || tiles <= 0 || ld_out % 8 != 0 ||
      (reinterpret_cast<uintptr_t>(out) & 15) != 0 ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(scores) | reinterpret_cast<uintptr_t>(weights) |
        reinterpret_cast<uintptr_t>(stats)) & 15) != 0)
    return (int)cudaErrorInvalidValue;
  const JointPrefillArgs x{a, block_seq, block_row, wide, reinterpret_cast<uint4*>(scores), reinterpret_cast<uint4*>(weights),
                           reinterpret_cast<float2*>(stats), tiles, block0, blocks};
  return joint_prefill_go(x, wide_blocks, stream);
}
