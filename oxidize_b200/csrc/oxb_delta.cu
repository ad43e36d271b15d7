// liboxb, entry points of the gated delta rule (delta.cuh, delta_chunk.cuh).
#include "common.cuh"
#include "delta.cuh"
#include "delta_chunk.cuh"
using namespace oxb;

template <typename T, int NK, int THREADS>
static int delta_step_go(const DeltaArgs& a, int B, cudaStream_t stream) {
  const int R = THREADS / (a.V / 4);
  const size_t smem = (size_t)(3 * a.K + 3 * a.V + 2 * R * a.V) * sizeof(float);
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  oxb_launch(delta_step_kernel<T, NK, THREADS>, dim3(a.H, B), dim3(THREADS), smem, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}
template <typename T>
static int delta_step_launch(const DeltaArgs& a, int B, cudaStream_t stream) {
  const int cols = a.V / 4;
  if (a.V <= 256) {
    const int nk = (a.K + 256 / cols - 1) / (256 / cols);
    if (nk <= 4) return delta_step_go<T, 4, 256>(a, B, stream);
    if (nk <= 8) return delta_step_go<T, 8, 256>(a, B, stream);
    if (nk <= 16) return delta_step_go<T, 16, 256>(a, B, stream);
    if (nk <= 32) return delta_step_go<T, 32, 256>(a, B, stream);
  }
  if (a.V <= 1024 && (a.K + 1024 / cols - 1) / (1024 / cols) <= 32) return delta_step_go<T, 32, 1024>(a, B, stream);
  return (int)cudaErrorInvalidValue;
}

template <int NK, int CH>
static int delta_decode_go(const DeltaArgs& a, int B, const float* low, cudaStream_t stream) {
  const int R = 512 / (a.V / 4);
  const size_t smem = (size_t)(3 * a.K + 2 * a.V + 2 * R * a.V) * sizeof(float);
  if (512 % (a.V / 4) == 0 && a.K == NK * R) oxb_launch(delta_decode_kernel<NK, CH, true>, dim3(a.H, B), dim3(512), smem, stream, a, low);
  else oxb_launch(delta_decode_kernel<NK, CH, false>, dim3(a.H, B), dim3(512), smem, stream, a, low);
  OXB_CHECK_LAUNCH();
  return 0;
}

// Steps of one row per sequence; `low`: B x (H K (+) H V) floats of scratch with low-rank projections, -1: not covered
static int delta_decode_launch(const DeltaArgs& a, int B, float* low, cudaStream_t stream) {
  const int n = (a.decay_up != nullptr ? a.H * a.K : 0) + (a.gate_up != nullptr ? a.H * a.V : 0);
  if (a.taps > 4 || a.V > 256 || a.K > 256 || (n > 0 && low == nullptr) || (a.decay_up != nullptr && (a.K % 32 != 0 || a.decay_rank % 16 != 0)) ||
      (a.gate_up != nullptr && a.gate_rank % 16 != 0))
    return -1;
  if (n > 0) {
    oxb_launch(delta_low_rank_kernel, dim3((n + 255) / 256, (B + 15) / 16), dim3(256), 0, stream, a, low, B);
    OXB_CHECK_LAUNCH();
  }
  const int R = 512 / (a.V / 4), nk = (a.K + R - 1) / R;
  const bool one = 2 * a.K + a.V <= 512;
  if (nk <= 2) return one ? delta_decode_go<2, 1>(a, B, low, stream) : delta_decode_go<2, 2>(a, B, low, stream);
  if (nk <= 4) return one ? delta_decode_go<4, 1>(a, B, low, stream) : delta_decode_go<4, 2>(a, B, low, stream);
  if (nk <= 8) return one ? delta_decode_go<8, 1>(a, B, low, stream) : delta_decode_go<8, 2>(a, B, low, stream);
  if (nk <= 16) return delta_decode_go<16, 2>(a, B, low, stream);
  return delta_decode_go<32, 2>(a, B, low, stream);
}

template <int KT, bool CH>
static int delta_chunk_go(DeltaChunkArgs x, int B, int longest, int nv, cudaStream_t stream) {
  constexpr int K = KT * 16;
  const int V = x.a.V, chunks = (longest + DC - 1) / DC;
  const int most[4] = {delta_prep_smem(K, 128).total, delta_state_smem(K, 32), delta_state_smem(K, 16), delta_output_smem(K, 128)};
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
  if (!configured[dev]) {
    constexpr cudaFuncAttribute attr = cudaFuncAttributeMaxDynamicSharedMemorySize;
    cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<KT, CH>, attr, most[0]);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_state_kernel<KT, 32>, attr, most[1]);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_state_kernel<KT, 16>, attr, most[2]);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_output_kernel<KT>, attr, most[3]);
    if (e != cudaSuccess) return (int)e;
    configured[dev] = true;
  }
  for (x.chunk0 = 0; x.chunk0 < chunks; x.chunk0 += x.round) {
    const dim3 units(chunks - x.chunk0 < x.round ? chunks - x.chunk0 : x.round, x.a.H, B), slices(V / nv, x.a.H, B);
    cudaError_t e = oxb_launch(delta_prepare_kernel<KT, CH>, units, dim3(DP_THREADS), (size_t)delta_prep_smem(K, V).total, stream, x);
    if (e == cudaSuccess)
      e = nv == 32 ? oxb_launch(delta_state_kernel<KT, 32>, slices, dim3(DS_THREADS), (size_t)most[1], stream, x)
                   : oxb_launch(delta_state_kernel<KT, 16>, slices, dim3(DS_THREADS), (size_t)most[2], stream, x);
    if (e == cudaSuccess)
      e = oxb_launch(delta_output_kernel<KT>, units, dim3(DO_THREADS), (size_t)delta_output_smem(K, V), stream, x);
    if (e != cudaSuccess) return (int)e;
    OXB_CHECK_LAUNCH();
  }
  return 0;
}

// Bytes of scratch per (chunk of 64 tokens, head) of heads that the chunk kernels cover, 0: not covered
OXB_API int oxb_delta_chunk_bytes(int K, int V) {
  const bool ok = (K == 32 || K == 64 || K == 96 || K == 128) && V > 0 && V % 16 == 0 && V <= 128;
  return ok ? delta_plan(K, V).bytes : 0;
}

// Gated delta rule of a step: z [T, ld] holds q | k (G heads of K values) | v (H heads of V values) and, at the given columns,
// gate, decay and beta; the state [num_slots, H, K, V] float32 is read and updated, the ring of convolution inputs [num_slots,
// taps, channels] read.  Only sequences that feed min_rows .. max_rows rows take part.  write_window (single-row steps): the
// ring is updated too; elsewhere oxb_delta_window does that afterwards; in bf16 these steps take delta_decode_kernel, with scratch
// ws of B * H * (K + V) floats where a projection has a low rank.  chunk_values 0: delta_step_kernel; else (bf16) the chunk
// kernels with that many values of the state per CTA (16 or 32), portions of up to `longest` rows, in rounds of `round`
// chunks with scratch ws of B * round * H * oxb_delta_chunk_bytes(K, V) bytes.
OXB_API int oxb_delta(const void* z, int ld, int dtype, int gate_off, int decay_off, int beta_off, const int* query_start,
                      const int* seq_lens, const int* slots, const float* conv, int taps, const float* a_log, const float* dt_bias,
                      const void* decay_up, int decay_rank, const void* gate_up, int gate_rank, const float* norm, float* state,
                      float* window, int num_slots, void* out, int ld_out, float out_scale, int B, int H, int G, int K, int V,
                      int v_dim, float q_scale, float eps, int min_rows, int max_rows, int write_window, int chunk_values,
                      int longest, int round, void* ws, cudaStream_t stream) {
  if (B <= 0 || H <= 0) return 0;
  if (G <= 0 || H % G != 0 || V % 4 != 0 || V <= 0 || K <= 0 || taps <= 0 || B > 65535 || slots == nullptr ||
      (decay_up != nullptr && (decay_rank % 8 != 0 || decay_off % 8 != 0)) || (gate_up != nullptr && (gate_rank % 8 != 0 || gate_off % 8 != 0)) ||
      ld % 8 != 0 || (reinterpret_cast<uintptr_t>(z) & 15) != 0)
    return (int)cudaErrorInvalidValue;
  const DeltaArgs a{z, ld, gate_off, decay_off, beta_off, query_start, seq_lens, slots, conv, taps, a_log, dt_bias, decay_up, decay_rank,
                    gate_up, gate_rank, norm, state, window, num_slots, out, ld_out, out_scale, H, G, K, V, v_dim, q_scale, eps,
                    min_rows, max_rows, write_window};
  if (chunk_values == 0 && write_window && dtype == 2) {
    const int e = delta_decode_launch(a, B, reinterpret_cast<float*>(ws), stream);
    if (e != -1) return e;
  }
  if (chunk_values == 0) return dtype == 0 ? delta_step_launch<float>(a, B, stream) : delta_step_launch<__nv_bfloat16>(a, B, stream);
  if (dtype != 2 || ws == nullptr || write_window || oxb_delta_chunk_bytes(K, V) == 0 || (chunk_values != 16 && chunk_values != 32) ||
      V % chunk_values != 0 || longest <= 0 || round <= 0 || H > 65535 || ld_out % 2 != 0 || (reinterpret_cast<uintptr_t>(out) & 3) != 0 ||
      (decay_up != nullptr && decay_rank % 16 != 0) || (gate_up != nullptr && gate_rank % 16 != 0) || gate_off % 2 != 0)
    return (int)cudaErrorInvalidValue;
  const DeltaChunkArgs x{a, reinterpret_cast<uint8_t*>(ws), 0, round};
  switch (K * 2 + (decay_up != nullptr)) {
    case 64: return delta_chunk_go<2, false>(x, B, longest, chunk_values, stream);
    case 65: return delta_chunk_go<2, true>(x, B, longest, chunk_values, stream);
    case 128: return delta_chunk_go<4, false>(x, B, longest, chunk_values, stream);
    case 129: return delta_chunk_go<4, true>(x, B, longest, chunk_values, stream);
    case 192: return delta_chunk_go<6, false>(x, B, longest, chunk_values, stream);
    case 193: return delta_chunk_go<6, true>(x, B, longest, chunk_values, stream);
    case 256: return delta_chunk_go<8, false>(x, B, longest, chunk_values, stream);
    default: return delta_chunk_go<8, true>(x, B, longest, chunk_values, stream);
  }
}

OXB_API int oxb_delta_window(const void* z, int ld, int dtype, const int* query_start, const int* seq_lens, const int* slots, int taps,
                             float* window, int num_slots, int B, int H, int G, int K, int V, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (taps <= 0 || B > 65535 || slots == nullptr) return (int)cudaErrorInvalidValue;
  DeltaArgs a{};
  a.z = z, a.ld = ld, a.query_start = query_start, a.seq_lens = seq_lens, a.slots = slots, a.taps = taps, a.window = window;
  a.num_slots = num_slots, a.H = H, a.G = G, a.K = K, a.V = V;
  const dim3 grid((2 * G * K + H * V + 255) / 256, B);
  if (dtype == 0) oxb_launch(delta_window_kernel<float>, grid, dim3(256), 0, stream, a);
  else oxb_launch(delta_window_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, a);
  OXB_CHECK_LAUNCH();
  return 0;
}
