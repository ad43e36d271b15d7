// liboxb, entry points of RWKV time mixing (wkv.cuh, wkv_chunk.cuh).
#include "common.cuh"
#include "wkv.cuh"
#include "wkv_chunk.cuh"
using namespace oxb;

// dtype codes of the activation type: 0 float32, 2 bfloat16
template <typename A>
static int token_shift_launch(const TokenShiftArgs& a, cudaStream_t stream) {
  if (a.H % 4 == 0) oxb_launch(token_shift_kernel<A, 4>, dim3(a.T, (a.ld + 1023) / 1024), dim3(256), 0, stream, a);
  else oxb_launch(token_shift_kernel<A, 1>, dim3(a.T, (a.ld + 255) / 256), dim3(256), 0, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}

// out [n, T, ld]: mixes of every row of x [T, H] with the one ahead of it in its sequence (token_shift_kernel); ld % 4 == 0.
OXB_API int oxb_token_shift(const float* x, const float* mu, const int* query_start, const int* seq_lens, const int* slots, float* window,
                            int num_slots, void* out, int dtype, int B, int T, int H, int n, int ld, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || n <= 0) return 0;
  if (H <= 0 || ld < H || ld % 4 != 0 || slots == nullptr || (H + 255) / 256 > 65535) return (int)cudaErrorInvalidValue;
  const TokenShiftArgs a{x, mu, query_start, seq_lens, slots, window, num_slots, out, B, T, H, n, ld};
  return dtype == 0 ? token_shift_launch<float>(a, stream) : token_shift_launch<__nv_bfloat16>(a, stream);
}

// out [T, N] float32: logarithms of the decays from the first of their projections, low [T, rank].
OXB_API int oxb_wkv_decay(const void* low, const void* up, const float* base, float* out, int dtype, int T, int N, int rank,
                          cudaStream_t stream) {
  if (T <= 0 || N <= 0) return 0;
  if (rank <= 0 || rank > 4096) return (int)cudaErrorInvalidValue;
  if (dtype == 2 && rank % 16 == 0 && N % 32 == 0 && rank <= 512 && T <= 16 * 65535 &&
      ((reinterpret_cast<uintptr_t>(low) | reinterpret_cast<uintptr_t>(up)) & 7) == 0) {
    oxb_launch(wkv_decay_kernel, dim3((N + 255) / 256, (T + 15) / 16), dim3(256), (size_t)2 * 16 * (rank + 8) * 2, stream,
               reinterpret_cast<const __nv_bfloat16*>(low), reinterpret_cast<const __nv_bfloat16*>(up), base, out, T, N, rank);
  } else {
    const int most = 65535;  // rows of a launch
    for (int t = 0; t < T; t += most) {
      const dim3 grid((N + 255) / 256, T - t < most ? T - t : most);
      if (dtype == 0)
        oxb_launch(wkv_decay_any_kernel<float>, grid, dim3(256), (size_t)rank * 4, stream, reinterpret_cast<const float*>(low) + (size_t)t * rank,
                   reinterpret_cast<const float*>(up), base, out + (size_t)t * N, N, rank);
      else
        oxb_launch(wkv_decay_any_kernel<__nv_bfloat16>, grid, dim3(256), (size_t)rank * 4, stream,
                   reinterpret_cast<const __nv_bfloat16*>(low) + (size_t)t * rank, reinterpret_cast<const __nv_bfloat16*>(up), base,
                   out + (size_t)t * N, N, rank);
    }
  }
  OXB_CHECK_LAUNCH();
  return 0;
}

template <typename T, int NK, int THREADS>
static int wkv_step_go(const WkvArgs& a, int B, cudaStream_t stream) {
  const int R = THREADS / (a.K / 4);
  const size_t smem = (size_t)(4 * a.K + R * a.K) * sizeof(float);
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  oxb_launch(wkv_step_kernel<T, NK, THREADS>, dim3(a.H, B), dim3(THREADS), smem, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}
template <typename T>
static int wkv_step_launch(const WkvArgs& a, int B, cudaStream_t stream) {
  const int cols = a.K / 4;
  if (a.K <= 256) {
    const int nk = (a.K + 256 / cols - 1) / (256 / cols);
    if (nk <= 4) return wkv_step_go<T, 4, 256>(a, B, stream);
    if (nk <= 8) return wkv_step_go<T, 8, 256>(a, B, stream);
    if (nk <= 16) return wkv_step_go<T, 16, 256>(a, B, stream);
    return wkv_step_go<T, 32, 512>(a, B, stream);
  }
  if (a.K <= 512) return wkv_step_go<T, 64, 1024>(a, B, stream);
  return (int)cudaErrorInvalidValue;
}

template <int KT>
static int wkv_chunk_go(WkvChunkArgs x, int B, int longest, cudaStream_t stream) {
  constexpr int K = KT * 16, MT = (K / 16 + WST_WARPS - 1) / WST_WARPS;
  const int chunks = (longest + WC - 1) / WC, state = wkv_state_smem(K), output = wkv_output_smem(K).total;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
  if (!configured[dev]) {
    cudaError_t e = cudaFuncSetAttribute(wkv_state_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, wkv_state_smem(128));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(wkv_output_kernel<KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, output);
    if (e != cudaSuccess) return (int)e;
    configured[dev] = true;
  }
  for (x.chunk0 = 0; x.chunk0 < chunks; x.chunk0 += x.round) {
    cudaError_t e = oxb_launch(wkv_state_kernel<MT>, dim3(K / WC_CH, x.a.H, B), dim3(WST_THREADS), (size_t)state, stream, x);
    if (e == cudaSuccess)
      e = oxb_launch(wkv_output_kernel<KT>, dim3(chunks - x.chunk0 < x.round ? chunks - x.chunk0 : x.round, x.a.H, B), dim3(WO_THREADS),
                     (size_t)output, stream, x);
    if (e != cudaSuccess) return (int)e;
    OXB_CHECK_LAUNCH();
  }
  return 0;
}

// Bytes of scratch per (chunk of 64 tokens, head) of heads that the chunk kernels cover, 0: not covered
OXB_API int oxb_wkv_chunk_bytes(int K) { return K == 32 || K == 64 || K == 96 || K == 128 ? K * K * 4 : 0; }

// Time mixing of a step: z [T, ld] holds r | k | v | gate (H heads of K values each), the state [num_slots, H, K, K] float32 is
// read and updated.  Only sequences that feed min_rows .. max_rows rows take part.  round 0: wkv_step_kernel; else (bf16) the chunk
// kernels, portions of up to `longest` rows in rounds of that many chunks with scratch ws of B * round * H *
// oxb_wkv_chunk_bytes(K) bytes.
OXB_API int oxb_wkv(const void* z, int ld, int dtype, const float* log_decay, const int* query_start, const int* seq_lens,
                    const int* slots, const float* bonus, const float* norm, float* state, int num_slots, void* out, int ld_out, int B,
                    int H, int K, int dim, float eps, int min_rows, int max_rows, int longest, int round, void* ws, cudaStream_t stream) {
  if (B <= 0 || H <= 0) return 0;
  if (K <= 0 || K % 32 != 0 || dim <= 0 || dim > K || B > 65535 || slots == nullptr) return (int)cudaErrorInvalidValue;
  const WkvArgs a{z, ld, log_decay, query_start, seq_lens, slots, bonus, norm, state, num_slots, out, ld_out, H, K, dim, eps, min_rows, max_rows};
  if (round == 0) return dtype == 0 ? wkv_step_launch<float>(a, B, stream) : wkv_step_launch<__nv_bfloat16>(a, B, stream);
  if (dtype != 2 || ws == nullptr || oxb_wkv_chunk_bytes(K) == 0 || round < 0 || longest <= 0 || H > 65535 || ld % 8 != 0 || ld_out % 2 != 0 ||
      (((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(log_decay) | reinterpret_cast<uintptr_t>(ws)) & 15) != 0))
    return (int)cudaErrorInvalidValue;
  const WkvChunkArgs x{a, reinterpret_cast<uint4*>(ws), 0, round};
  switch (K) {
    case 32: return wkv_chunk_go<2>(x, B, longest, stream);
    case 64: return wkv_chunk_go<4>(x, B, longest, stream);
    case 96: return wkv_chunk_go<6>(x, B, longest, stream);
    default: return wkv_chunk_go<8>(x, B, longest, stream);
  }
}
