// Shared device helpers for the sm_100a kernels: mbarrier, TMA, tcgen05/TMEM
// wrappers (inline PTX) and waits with an iteration limit.
//
// Every wait in this library is bounded.  When a limit is hit the waiting thread
// records a code in a per-launch status word (global memory), raises the CTA's
// shared abort flag, and every role of the CTA falls through to the common
// teardown (wait for the CTA's own bulk copies, free TMEM, return), so that a
// protocol bug or a missing peer shows up as an error status on the host rather
// than as a hung GPU.
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_fp8.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace b200 {

// status codes written to the status word
enum : int {
  ST_OK = 0,
  ST_TIMEOUT_FULL = 1,      // consumer waited for a TMA stage
  ST_TIMEOUT_EMPTY = 2,     // producer waited for a free stage
  ST_TIMEOUT_TMEM_FULL = 3, // epilogue waited for the accumulator
  ST_TIMEOUT_TMEM_EMPTY = 4,
  ST_TIMEOUT_FLAG = 5,      // waited for a peer / other CTA flag
  ST_BAD_INDEX = 6,         // bounds-checked build: index out of range
  ST_TIMEOUT_DRAIN = 7,
};

// Bounds-checked build (-DB200_BOUNDS_CHECK): the attention kernels always clamp a block id that falls
// outside the pool; this build also counts such ids, and page indices past the end of a block-table row,
// per translation unit, so that tests can assert that none occurred.
#ifdef B200_BOUNDS_CHECK
static __device__ unsigned int b200_bad_index_count = 0;
#define B200_NOTE_BAD_INDEX() atomicAdd(&b200_bad_index_count, 1u)
#define B200_TAKE_BAD_INDEX_COUNT(out)                                                          \
  do {                                                                                          \
    unsigned int _zero = 0;                                                                     \
    if (cudaMemcpyFromSymbol((out), b200_bad_index_count, sizeof(unsigned int)) != cudaSuccess) return -1; \
    if (cudaMemcpyToSymbol(b200_bad_index_count, &_zero, sizeof(unsigned int)) != cudaSuccess) return -1;  \
  } while (0)
#else
#define B200_NOTE_BAD_INDEX() ((void)0)
#define B200_TAKE_BAD_INDEX_COUNT(out) (*(out) = 0u)
#endif

#ifndef B200_WAIT_LIMIT_NS
#define B200_WAIT_LIMIT_NS 1000000000ull     // one second
#endif

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

__device__ __forceinline__ uint32_t elect_one() {
  uint32_t pred = 0;
  asm volatile(
      "{\n\t"
      ".reg .pred P;\n\t"
      "elect.sync _|P, 0xffffffff;\n\t"
      "selp.b32 %0, 1, 0, P;\n\t"
      "}\n"
      : "=r"(pred));
  return pred;
}

// ---------------------------------------------------------------- mbarrier
__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_fence_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes)
               : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ uint32_t mbar_test(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t"
      ".reg .pred P;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 P, [%1], %2;\n\t"
      "selp.b32 %0, 1, 0, P;\n\t"
      "}\n"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok;
}

// try_wait with a suspend-time hint: the thread may be parked by the hardware for up to `ns`
// nanoseconds instead of burning issue slots (and power) in a polling loop.
__device__ __forceinline__ uint32_t mbar_try_wait(uint64_t* bar, uint32_t parity, uint32_t ns) {
  uint32_t ok;
  asm volatile(
      "{\n\t"
      ".reg .pred P;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 P, [%1], %2, %3;\n\t"
      "selp.b32 %0, 1, 0, P;\n\t"
      "}\n"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity), "r"(ns)
      : "memory");
  return ok;
}
__device__ __forceinline__ unsigned long long global_timer_ns() {
  unsigned long long t;
  asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
  return t;
}

// Bounded wait.  Returns true when the phase completed, false on timeout or when another role of
// the CTA already aborted.  A few immediate polls cover the common case of a barrier that is
// (almost) ready; after that the thread parks in try_wait and the bound is wall time
// (B200_WAIT_LIMIT_NS), checked every few wake-ups together with the CTA's abort flag.
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag,
                                          int* status, int code) {
#pragma unroll 1
  for (int it = 0; it < 32; ++it)
    if (mbar_test(bar, parity)) return true;
  const unsigned long long t0 = global_timer_ns();
#pragma unroll 1
  for (uint32_t it = 0;; ++it) {
    if (mbar_try_wait(bar, parity, 2000u)) return true;
    if ((it & 7u) == 7u) {
      if (*abort_flag) return false;
      if (global_timer_ns() - t0 > B200_WAIT_LIMIT_NS) break;
    }
  }
  *abort_flag = 1;
  if (status) atomicCAS(status, ST_OK, code);
  return false;
}

// ---------------------------------------------------------------------- TMA
__device__ __forceinline__ void tma_prefetch_desc(const CUtensorMap* m) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(m)) : "memory");
}
// 2D tiled load, global -> this CTA's shared memory (no cluster multicast)
__device__ __forceinline__ void tma_load_2d(void* smem_dst, const CUtensorMap* m, uint64_t* bar, int x,
                                            int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      :
      : "r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y)
      : "memory");
}
__device__ __forceinline__ void tma_load_2d_hint(void* smem_dst, const CUtensorMap* m, uint64_t* bar, int x,
                                                 int y, uint64_t policy) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint "
      "[%0], [%1, {%3, %4}], [%2], %5;"
      :
      : "r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y),
        "l"(policy)
      : "memory");
}
__device__ __forceinline__ void tma_load_3d(void* smem_dst, const CUtensorMap* m, uint64_t* bar, int x,
                                            int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      :
      : "r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y),
        "r"(z)
      : "memory");
}
constexpr uint64_t L2_EVICT_NORMAL = 0x1000000000000000ull;
constexpr uint64_t L2_EVICT_FIRST = 0x12F0000000000000ull;
constexpr uint64_t L2_EVICT_LAST = 0x14F0000000000000ull;

// ------------------------------------------------------------------ tcgen05
__device__ __forceinline__ void tmem_alloc(uint32_t* smem_dst, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(smem_dst)),
               "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tmem_relinquish() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
__device__ __forceinline__ void tc_fence_before() {
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
}
__device__ __forceinline__ void tc_fence_after() {
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
}
// D[tmem] (+)= A[smem desc] * B[smem desc]; issued by ONE thread
__device__ __forceinline__ void umma_f16(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc,
                                         uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// fp8 e4m3/e5m2 (kind::f8f6f4), fp32 accumulate
__device__ __forceinline__ void umma_f8(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc,
                                        uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f8f6f4 [%0], %1, %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// kind::i8: signed/unsigned 8-bit operands, s32 accumulate
__device__ __forceinline__ void umma_i8(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc,
                                        uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::i8 [%0], %1, %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// all previously issued MMAs of this thread arrive on the mbarrier when complete
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(
                   smem_u32(bar))
               : "memory");
}
// 32 lanes x 32 consecutive columns: thread i of the warp gets lane (base+i)
__device__ __forceinline__ void tmem_ld_32x32(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
        "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]),
        "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]),
        "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]),
        "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }

// Shared-memory matrix descriptor for a K-major tile whose rows are 128 bytes
// (64 bf16 / 128 fp8) written by TMA with SWIZZLE_128B: 8-row groups are 1024 B apart.
__device__ __forceinline__ uint64_t umma_desc_k_sw128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);        // start address
  d |= (uint64_t)1 << 16;                               // leading byte offset (unused for swizzled K-major)
  d |= (uint64_t)(1024 >> 4) << 32;                     // stride byte offset: 8 rows * 128 B
  d |= (uint64_t)1 << 46;                               // descriptor version (sm_100)
  d |= (uint64_t)2 << 61;                               // SWIZZLE_128B
  return d;
}
// kind::f16 instruction descriptor: bf16 x bf16 -> fp32, both operands K-major, M x N tile
__host__ __device__ constexpr uint32_t umma_idesc_bf16(int M, int N) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(M >> 4) << 24);
}
// kind::f8f6f4 with e4m3 operands (format 0), fp32 accumulate
__host__ __device__ constexpr uint32_t umma_idesc_e4m3(int M, int N) {
  return (1u << 4) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(M >> 4) << 24);
}
// kind::i8 with signed 8-bit operands (format 1), s32 accumulate (format 2)
__host__ __device__ constexpr uint32_t umma_idesc_s8(int M, int N) {
  return (2u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(M >> 4) << 24);
}

// ------------------------------------------------- programmatic dependent launch
// wait: returns once every grid this launch depends on has completed and its writes are visible.
// launch_dependents: lets the next kernel of the stream (if launched with the programmatic
// attribute) start before this grid has finished.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}

// ------------------------------------------------- thread-block cluster / DSMEM
__device__ __forceinline__ uint32_t cluster_ctarank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
__device__ __forceinline__ void cluster_arrive_release() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
}
__device__ __forceinline__ void cluster_wait_acquire() {
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// shared::cta address -> shared::cluster address of the same offset in CTA `rank`
__device__ __forceinline__ uint32_t mapa_shared(uint32_t smem_addr, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(smem_addr), "r"(rank));
  return r;
}
__device__ __forceinline__ float4 ld_dsmem_v4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];"
               : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w)
               : "r"(addr)
               : "memory");
  return v;
}

// ------------------------------------------------- peer / flag helpers (NVLink)
__device__ __forceinline__ void st_release_sys(int* p, int v) {
  asm volatile("st.release.sys.global.s32 [%0], %1;" ::"l"(p), "r"(v) : "memory");
}
__device__ __forceinline__ int ld_acquire_sys(const int* p) {
  int v;
  asm volatile("ld.acquire.sys.global.s32 %0, [%1];" : "=r"(v) : "l"(p) : "memory");
  return v;
}
__device__ __forceinline__ void st_release_gpu(int* p, int v) {
  asm volatile("st.release.gpu.global.s32 [%0], %1;" ::"l"(p), "r"(v) : "memory");
}
__device__ __forceinline__ int ld_acquire_gpu(const int* p) {
  int v;
  asm volatile("ld.acquire.gpu.global.s32 %0, [%1];" : "=r"(v) : "l"(p) : "memory");
  return v;
}
// ---- bulk copy shared -> global (the destination may be a peer GPU's memory: a plain store stream,
// no multicast involved).  Groups complete in order; wait_group_read<N> returns once all but the N
// most recent groups have finished READING shared memory, wait_group<N> once they are fully done.
__device__ __forceinline__ void bulk_store_s2g(void* gdst, const void* ssrc, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;"
               :: "l"(gdst), "r"(smem_u32(ssrc)), "r"(bytes) : "memory");
}
__device__ __forceinline__ void bulk_commit_group() { asm volatile("cp.async.bulk.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void bulk_wait_group_read() {
  asm volatile("cp.async.bulk.wait_group.read %0;" :: "n"(N) : "memory");
}
template <int N>
__device__ __forceinline__ void bulk_wait_group() {
  asm volatile("cp.async.bulk.wait_group %0;" :: "n"(N) : "memory");
}
// generic-proxy writes to shared memory become visible to the async proxy (bulk copies, TMA)
__device__ __forceinline__ void fence_proxy_async_smem() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}

// Wait until *p >= want (flags only grow).  Bounded; false on timeout.
__device__ __forceinline__ bool wait_flag_ge(const int* p, int want, int* status, uint32_t limit) {
  for (uint32_t it = 0; it < limit; ++it) {
    if (ld_acquire_sys(p) - want >= 0) return true;
    if (it > 64) __nanosleep(40);
  }
  if (status) atomicCAS(status, ST_OK, ST_TIMEOUT_FLAG);
  return false;
}

__device__ __forceinline__ float bf16_to_f(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T warp_sum(T v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
template <typename T>
__device__ __forceinline__ T warp_max(T v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = max(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

__device__ __forceinline__ float gelu_erf(float v) { return 0.5f * v * (1.f + erff(v * 0.70710678118654752f)); }

// gelu in its tanh form, tanh from one exponential: 0.5 (1 + tanh z) = 1 - 1 / (1 + e^2z)
__device__ __forceinline__ float gelu_tanh(float v) {
  const float z = 0.7978845608028654f * (v + 0.044715f * v * v * v);
  return v * (1.f - __fdividef(1.f, 1.f + __expf(2.f * z)));
}
// gate and up projection of a feed-forward -> its activation.  ACT as the GEMMs number them: 0 silu(g) u,
// 3 gelu(g) u in the tanh form, 5 g' sigmoid(alpha g') (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit)
template <int ACT>
__device__ __forceinline__ float gated_pair(float g, float u, float alpha, float limit) {
  if constexpr (ACT == 3) return gelu_tanh(g) * u;
  if constexpr (ACT == 5) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.f + __expf(-alpha * g)) * (u + 1.f);
  }
  return g / (1.f + __expf(-g)) * u;
}

// First key that the query at position pos sees: of the last `window` ones (> 0), of its own chunk of -window positions (< 0,
// chunks are counted from position 0), of all (0).
__device__ __forceinline__ int first_key(int window, int pos) {
  return window > 0 ? max(0, pos - window + 1) : (window < 0 ? pos - pos % -window : 0);
}

__device__ __forceinline__ float relu_squared(float v) { return v > 0.f ? v * v : 0.f; }
__device__ __forceinline__ float soft_cap(float v, float cap) { return cap > 0.f ? cap * tanhf(v / cap) : v; }

// What follows the softmax of a head before the output projection, in the epilogue of the attention kernels:
//   lam:  query heads 2h and 2h + 1 are two maps of head h over the same values; o = o1 - lam * o2, then
//         o / rms(o over vdim) * keep.  The output has half as many heads.
//   gate: o times sigmoid(gate[t, h * vdim + d])
struct HeadFinish {
  const float* lam;
  const __nv_bfloat16* gate;
  int ldg, vdim;
  float keep, eps;
};
// v[i] *= sigmoid of the gate of columns col + i (those below vdim)
template <int N>
__device__ __forceinline__ void gate_columns(const HeadFinish& f, long long t, int head, int col, float* v) {
  const __nv_bfloat16* g = f.gate + (size_t)t * f.ldg + (size_t)head * f.vdim + col;
  if ((reinterpret_cast<uintptr_t>(g) & 15) == 0 && col + N <= f.vdim) {
    uint4 raw[N / 8];
#pragma unroll
    for (int i = 0; i < N / 8; ++i) raw[i] = reinterpret_cast<const uint4*>(g)[i];
#pragma unroll
    for (int i = 0; i < N; ++i)
      v[i] = __fdividef(v[i], 1.f + __expf(-__bfloat162float(reinterpret_cast<const __nv_bfloat16*>(raw)[i])));
    return;
  }
#pragma unroll
  for (int i = 0; i < N; ++i)
    if (col + i < f.vdim) v[i] = __fdividef(v[i], 1.f + __expf(-__bfloat162float(g[i])));
}

struct alignas(16) bf16x8 {
  __nv_bfloat162 v[4];
};

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = (lane < nw) ? red[lane] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

// 16-byte load that bypasses L1 (data written by a peer GPU or another SM during this kernel)
__device__ __forceinline__ uint4 ld_relaxed_sys_v4(const void* p) {
  uint4 v;
  asm volatile("ld.relaxed.sys.global.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "l"(p)
               : "memory");
  return v;
}

}  // namespace b200

// ---------------------------------------------------------------- host side
#define B200_CUDA_CHECK(expr)                                                        \
  do {                                                                               \
    cudaError_t _e = (expr);                                                         \
    if (_e != cudaSuccess) {                                                         \
      b200_set_last_error(cudaGetErrorString(_e), __FILE__, __LINE__);               \
      return (int)_e;                                                                \
    }                                                                                \
  } while (0)

extern "C" void b200_set_last_error(const char* msg, const char* file, int line);
extern "C" int b200_pdl_enabled();

// The dynamic shared-memory limit of a kernel is an attribute of (kernel, device): a process that
// uses a second device must set it there too.  `seen` is a per-call-site bit mask over device ordinals.
template <typename Kernel>
static inline cudaError_t ensure_dynamic_smem(Kernel kernel, int bytes, unsigned long long* seen) {
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  const unsigned long long bit = 1ull << (dev & 63);
  if (*seen & bit) return cudaSuccess;
  e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e == cudaSuccess) *seen |= bit;
  return e;
}

// Launch with the programmatic-stream-serialization attribute: the grid may be scheduled while the
// previous kernel of the stream is still draining.  The kernel must execute griddepcontrol.wait
// (pdl_wait()) before it reads anything an earlier kernel wrote.
template <typename... KArgs, typename... Args>
static inline cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                     cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = b200_pdl_enabled() ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
