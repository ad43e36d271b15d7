// Shared device helpers for the sm_100a kernels: bf16 packing, warp/block reductions,
// mbarrier / TMA / tcgen05 PTX wrappers, bounded waits and the per-device status word.
//
// Every wait in these kernels is bounded.  When a wait gives up it records a code in the
// global status word (read by the host after the step) and lets the kernel run to its
// normal end, so a logic error or a missing peer never hangs the GPU.
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define OXB_API extern "C" __attribute__((visibility("default")))

#define OXB_CHECK_LAUNCH()                      \
  do {                                          \
    cudaError_t e__ = cudaGetLastError();       \
    if (e__ != cudaSuccess) return (int)e__;    \
  } while (0)

// status codes written to the device status word
enum OxbStatus : int {
  OXB_OK = 0,
  OXB_TIMEOUT_TMA_FULL = 1,
  OXB_TIMEOUT_TMA_EMPTY = 2,
  OXB_TIMEOUT_ACCUM = 3,
  OXB_TIMEOUT_PEER_FLAG = 4,
  OXB_TIMEOUT_SPLITK = 5,
  OXB_BAD_BLOCK_ID = 6,   // a block table entry outside the KV pool (access skipped)
  OXB_BAD_SLOT = 7,       // a KV write slot outside the KV pool (write skipped)
  OXB_BAD_ARGUMENT = 8,   // a kernel argument outside its documented range (work skipped)
};

// Device status word; the host reads it with oxb_status().  The translation units of the library are compiled
// independently (no relocatable device code: whole-kernel optimisations such as per-warpgroup register budgets need the
// compiler to see a complete program), so each unit has its own copy and registers a reader for it; oxb_status() merges
// the copies (first non-zero code, summed count).
static __device__ int g_oxb_status[4];  // [0]=code, [1]=detail (block / stage / rank), [2]=count
struct OxbStatusUnit {
  int (*read)(int* out4, int reset);
  OxbStatusUnit* next;
};
void oxb_register_status_unit(OxbStatusUnit* u);  // oxb.cu
namespace {
int oxb_status_of_this_unit(int* out4, int reset) {
  cudaError_t e = cudaMemcpyFromSymbol(out4, g_oxb_status, 4 * sizeof(int));
  if (e == cudaSuccess && reset) {
    const int z[4] = {0, 0, 0, 0};
    e = cudaMemcpyToSymbol(g_oxb_status, z, sizeof(z));
  }
  return (int)e;
}
struct OxbStatusRegistration {
  OxbStatusUnit unit;
  OxbStatusRegistration() {
    unit.read = &oxb_status_of_this_unit;
    unit.next = nullptr;
    oxb_register_status_unit(&unit);
  }
} g_oxb_status_registration;
}  // namespace

__device__ __forceinline__ void oxb_report(int code, int detail) {
  if (atomicCAS(&g_oxb_status[0], 0, code) == 0) g_oxb_status[1] = detail;
  atomicAdd(&g_oxb_status[2], 1);
}

// ----------------------------------------------------------------------------- numerics
__device__ __forceinline__ float bf16_to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float2 unpack_bf16x2(uint32_t u) {
  __nv_bfloat162 v = *reinterpret_cast<__nv_bfloat162*>(&u);
  return __bfloat1622float2(v);
}

// Gates on attention outputs, out *= sigmoid(gate): one per head (rows [T, heads]), or one per value (rows [T, heads * width]).
struct HeadGate {
  const void* rows;  // in the activation type, or null
  int ld, per_value;
};
__device__ __forceinline__ float head_gate_of(float z) { return 1.f / (1.f + expf(-z)); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// block-wide sum; `scratch` must hold >= 32 floats; all threads get the result
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float r = (lane < nwarps) ? scratch[lane] : 0.f;
  r = warp_sum(r);
  return r;
}

// The sequence that holds row t.
__device__ __forceinline__ int sequence_of(const int* query_start, int B, int t) {
  int b = 0, hi = B - 1;
  while (b < hi) {
    const int mid = (b + hi + 1) >> 1;
    if (query_start[mid] <= t) b = mid;
    else hi = mid - 1;
  }
  return b;
}

// ----------------------------------------------------------------------------- smem / mbarrier
__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_fence_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok != 0;
}

// Bounded wait: gives up after ~`limit` polls (each poll itself blocks for a short hardware
// time slice), reports `code`, raises the CTA-wide abort flag and returns false.  Once the
// abort flag is up every later wait returns at once, so the kernel drains quickly.
__device__ __forceinline__ bool mbar_wait_bounded(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int code,
                                                  int detail, uint32_t limit = 4000000u) {
  for (uint32_t i = 0; i < limit; ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if (*abort_flag) return false;
    if (i > 1024) __nanosleep(64);
  }
  *abort_flag = 1;
  oxb_report(code, detail);
  return false;
}

// ----------------------------------------------------------------------------- TMA
__device__ __forceinline__ void tma_prefetch_desc(const CUtensorMap* d) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(d)) : "memory");
}
// Ask the memory system to bring one tile of a tensor map into the L2 (no shared memory, no barrier):
// used before the grid dependency resolves, so that the weight stream keeps HBM busy while the
// upstream kernel drains.
__device__ __forceinline__ void tma_prefetch_l2_2d(const CUtensorMap* d, int c0, int c1) {
  asm volatile("cp.async.bulk.prefetch.tensor.2d.L2.global [%0, {%1, %2}];" ::"l"(reinterpret_cast<uint64_t>(d)), "r"(c0),
               "r"(c1)
               : "memory");
}
// 2-D tiled load into this CTA's own shared memory (every CTA fetches its own tiles)
// `bytes` (a multiple of 16) of this GPU's own memory; both addresses on 16-byte boundaries
__device__ __forceinline__ void bulk_load(void* smem_dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(smem_dst)), "l"(src),
               "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void tma_load_2d(void* smem_dst, const CUtensorMap* d, uint64_t* bar, int c0, int c1) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(d)), "r"(smem_u32(bar)), "r"(c0), "r"(c1)
      : "memory");
}
__device__ __forceinline__ void tma_load_2d_hint(void* smem_dst, const CUtensorMap* d, uint64_t* bar, int c0, int c1,
                                                 uint64_t policy) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint [%0], [%1, {%3, %4}], [%2], %5;"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(d)), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "l"(policy)
      : "memory");
}
__device__ __forceinline__ uint64_t l2_policy_evict_first() {
  uint64_t p;
  asm volatile("createpolicy.fractional.L2::evict_first.b64 %0, 1.0;" : "=l"(p));
  return p;
}
__device__ __forceinline__ uint64_t l2_policy_evict_last() {
  uint64_t p;
  asm volatile("createpolicy.fractional.L2::evict_last.b64 %0, 1.0;" : "=l"(p));
  return p;
}

// ----------------------------------------------------------------------------- tcgen05 / TMEM
__device__ __forceinline__ void tmem_alloc(uint32_t* smem_out, uint32_t ncols) {  // whole warp
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(smem_out)), "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tmem_relinquish() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {  // whole warp
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }

// K-major operand tile in shared memory with the 128-byte swizzle: rows of 128 bytes,
// 8-row groups 1024 bytes apart (SBO), LBO field 1, descriptor version 1 (Blackwell).
__device__ __forceinline__ uint64_t umma_desc_k_sw128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)1 << 16;                 // leading byte offset (unused with swizzle) = 1
  d |= (uint64_t)(1024 >> 4) << 32;       // stride byte offset between 8-row groups
  d |= (uint64_t)1 << 46;                 // version
  d |= (uint64_t)2 << 61;                 // SWIZZLE_128B
  return d;
}

// instruction descriptor for kind::f16, bf16 x bf16 -> f32, both operands K-major
__host__ __device__ constexpr uint32_t umma_idesc_bf16(int M, int N) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(M >> 4) << 24);
}
__device__ __forceinline__ void umma_bf16(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// The same with the issuing lane chosen by a predicate instead of a branch (called by the whole warp) and the descriptors
// given as their low words, which hold the address; the high words (layout) are constants: short, warp-uniform operands.
template <uint32_t AHI, uint32_t BHI, uint32_t IDESC>
__device__ __forceinline__ void umma_bf16_if(bool issue, uint32_t tmem_d, uint32_t alo, uint32_t blo, bool accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t.reg .b64 da, db;\n\t"
      "setp.ne.b32 p, %3, 0;\n\t"
      "setp.ne.b32 q, %4, 0;\n\t"
      "mov.b64 da, {%1, %5};\n\t"
      "mov.b64 db, {%2, %6};\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %7, p;\n\t}"
      ::"r"(tmem_d), "r"(alo), "r"(blo), "r"((uint32_t)accumulate), "r"((uint32_t)issue), "n"(AHI), "n"(BHI), "n"(IDESC)
      : "memory");
}
// low word of a shared-memory descriptor: address and leading byte offset, both in 16-byte units
__device__ __forceinline__ uint32_t umma_desc_lo(uint32_t smem_addr, uint32_t leading_bytes = 16) {
  return ((smem_addr & 0x3FFFF) >> 4) | ((leading_bytes >> 4) << 16);
}
// high word: stride byte offset 1024 (8 rows of 128 bytes), version 1, 128-byte swizzle
constexpr uint32_t UMMA_DESC_HI_SW128 = (1024u >> 4) | (1u << 14) | (2u << 29);
// A operand in tensor memory (row = lane, two bf16 per 32-bit column), B through a shared-memory descriptor
__device__ __forceinline__ void umma_bf16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// 32 lanes x 4 consecutive 32-bit columns: thread i of the warp writes lane (base_lane + i)
__device__ __forceinline__ void tmem_st4(uint32_t taddr, uint32_t a, uint32_t b, uint32_t c, uint32_t d) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x4.b32 [%0], {%1, %2, %3, %4};" ::"r"(taddr), "r"(a), "r"(b), "r"(c), "r"(d)
               : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}

__device__ __forceinline__ void umma_commit_if(bool issue, uint64_t* bar) {
  asm volatile(
      "{\n\t.reg .pred q;\n\t"
      "setp.ne.b32 q, %1, 0;\n\t"
      "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}"
      ::"r"(smem_u32(bar)), "r"((uint32_t)issue)
      : "memory");
}

// 32 lanes x 16 consecutive 32-bit columns: thread i of the warp reads lane (base_lane + i)
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr));
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }

__device__ __forceinline__ bool elect_one() {
  uint32_t pred;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "elect.sync _|p, 0xffffffff;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(pred));
  return pred != 0;
}

// programmatic dependent launch: wait for the upstream grid's memory / let dependents start
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

// ----------------------------------------------------------------------------- host side
typedef CUresult (*PFN_encodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                    const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                    CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
PFN_encodeTiled oxb_get_encode_tiled();
int oxb_sm_count();  // SM count of the current device
// Byte view of packed weight rows: [rows, row_bytes] uint8, no swizzle (box_bytes <= 256, 16-byte multiples)
int oxb_make_tmap_bytes(CUtensorMap* out, const void* base, uint64_t rows, uint64_t row_bytes, uint32_t box_rows,
                        uint32_t box_bytes);
extern int g_oxb_ar_ll_min_world;          // rank counts from which the fused all-reduce uses the LL two-shot exchange
extern int g_oxb_gemv_max_t;               // packed-weight calls of at most this many tokens take the dp4a GEMV
extern int g_oxb_gemv_wide;                // 1: also for matrices with K >= 2N (default 0: those go to the tensor-core kernel)
extern unsigned long long* g_oxb_ar_trace;    // optional device buffers for in-kernel phase timestamps
extern unsigned long long* g_oxb_attn_trace;
// 2-D row-major tensor [rows, cols] of `elem_bytes` elements, box [box_rows, box_cols], 128B swizzle
int oxb_make_tmap_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t cols, uint64_t row_stride_bytes,
                     uint32_t box_rows, uint32_t box_cols, int elem_bytes);

// Programmatic dependent launch: a kernel started with this helper may begin (block scheduling,
// shared-memory / barrier / TMEM set-up, loads of *static* data such as weights) while the previous
// kernel in the stream is still draining; it must execute pdl_wait() before it touches anything the
// previous kernel produced.  Kernels call pdl_launch_dependents() at their top so that the next
// one can do the same.  With the switch off the launch is an ordinary stream-ordered one, in
// which case griddepcontrol.* are no-ops.
extern int g_oxb_pdl;  // 1 = on (default), 0 = off (OXB_PDL=0 or oxb_set_pdl(0))
template <typename... KArgs, typename... Args>
inline cudaError_t oxb_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                              Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = g_oxb_pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

// Same, as thread-block clusters of `cluster` CTAs (cluster.x*y*z <= 8 is portable; up to 16 needs
// cudaFuncAttributeNonPortableClusterSizeAllowed on the kernel).
template <typename... KArgs, typename... Args>
inline cudaError_t oxb_launch_cluster(void (*kernel)(KArgs...), dim3 grid, dim3 block, dim3 cluster, size_t smem,
                                      cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster.x;
  attr[0].val.clusterDim.y = cluster.y;
  attr[0].val.clusterDim.z = cluster.z;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = g_oxb_pdl ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

// ---- thread-block cluster helpers (distributed shared memory)
__device__ __forceinline__ uint32_t cluster_nctarank() {
  uint32_t v;
  asm volatile("mov.u32 %0, %%cluster_nctarank;" : "=r"(v));
  return v;
}
__device__ __forceinline__ uint32_t cluster_ctarank() {
  uint32_t v;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(v));
  return v;
}
// every thread of every CTA of the cluster must call this the same number of times (warp-convergent)
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// address of the same shared-memory location in CTA `rank` of the cluster
__device__ __forceinline__ uint32_t dsmem_map(uint32_t local_smem_addr, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local_smem_addr), "r"(rank));
  return r;
}
__device__ __forceinline__ float dsmem_ld_f32(uint32_t cluster_addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(cluster_addr) : "memory");
  return v;
}
__device__ __forceinline__ float4 dsmem_ld_f32x4(uint32_t cluster_addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];"
               : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(cluster_addr) : "memory");
  return v;
}
