// Ragged paged attention on the CUDA cores: 32-bit caches (full fp32 products and sums) and head sizes the tensor-core
// kernels are not built for.  Same cache layout, batch description and semantics as attention.cu (causal, optional
// sliding window, soft cap and sinks); decode and prefill alike.
//
// One warp per (query token, query head).  32 keys at a time: every lane scores one key, the running maximum and sum
// are kept by the warp, and the lanes then split the value columns.
#include "common.cuh"

namespace b200 {
namespace as {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

struct Params {
  const void *q, *kv;
  void* out;
  const int *block_tables, *seq_lens, *qsl;
  const float* sinks;
  int T, R, Hq, Hkv, D, max_blocks, block_size, window, ldo;
  long long num_blocks;
  float scale, softcap;
};

constexpr int WARPS = 4;

// NC: value columns per lane (D <= 32 * NC)
template <typename E, int NC>
__global__ void __launch_bounds__(32 * WARPS) attn_simt_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, t = blockIdx.y * WARPS + warp;
  if (t >= p.T) return;
  int r = -1;
  for (int i = 0; i < p.R; ++i)
    if (t >= p.qsl[i] && t < p.qsl[i + 1]) { r = i; break; }
  E* out = reinterpret_cast<E*>(p.out) + (size_t)t * p.ldo + h * p.D;
  if (r < 0) {                                    // a row of padding
    for (int d = lane; d < p.D; d += 32) put(out + d, 0.f);
    return;
  }
  float* q = smem + warp * p.D;
  const E* qp = reinterpret_cast<const E*>(p.q) + ((size_t)t * p.Hq + h) * p.D;
  for (int d = lane; d < p.D; d += 32) q[d] = to_f(qp[d]);
  __syncwarp();
  const int pos = p.seq_lens[r] - (p.qsl[r + 1] - t);
  const int first = first_key(p.window, pos);
  const int hk = h / (p.Hq / p.Hkv);
  const int* bt = p.block_tables + (size_t)r * p.max_blocks;
  const size_t page = (size_t)p.block_size * p.D;
  const E* kv = reinterpret_cast<const E*>(p.kv);
  float m = -INFINITY, l = 0.f, acc[NC];
#pragma unroll
  for (int i = 0; i < NC; ++i) acc[i] = 0.f;
  for (int k0 = first; k0 <= pos; k0 += 32) {
    const int key = k0 + lane;
    const bool ok = key <= pos;
    long long blk = 0;
    int off = 0;
    if (ok) {
      const int pg = key / p.block_size;
      off = key - pg * p.block_size;
      blk = pg < p.max_blocks ? bt[pg] : 0;
      if (blk < 0 || blk >= p.num_blocks) blk = 0;
    }
    const E* kp = kv + ((size_t)blk * 2 * p.Hkv + hk) * page + (size_t)off * p.D;
    float s = -INFINITY;
    if (ok) {
      float a = 0.f;
      for (int d = 0; d < p.D; d += 4) {
        const float4 kk = load4(kp + d);
        a = fmaf(q[d], kk.x, a);
        a = fmaf(q[d + 1], kk.y, a);
        a = fmaf(q[d + 2], kk.z, a);
        a = fmaf(q[d + 3], kk.w, a);
      }
      s = soft_cap(a * p.scale, p.softcap);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float alpha = expf(m - mn), w = ok ? expf(s - mn) : 0.f;
    m = mn;
    l = l * alpha + warp_sum(w);
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] *= alpha;
    const E* vp = kp + (size_t)p.Hkv * page;
    const unsigned long long va = reinterpret_cast<unsigned long long>(vp);
    const int n = min(32, pos - k0 + 1);
    for (int j = 0; j < n; ++j) {
      const float wj = __shfl_sync(0xffffffffu, w, j);
      const E* vj = reinterpret_cast<const E*>(__shfl_sync(0xffffffffu, va, j));
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (lane + 32 * i < p.D) acc[i] = fmaf(wj, to_f(vj[lane + 32 * i]), acc[i]);
    }
  }
  float sc = 1.f;
  if (p.sinks != nullptr) {
    const float sk = p.sinks[h], mn = fmaxf(m, sk);
    sc = expf(m - mn);
    l = l * sc + expf(sk - mn);
  }
  const float inv = sc / l;
#pragma unroll
  for (int i = 0; i < NC; ++i)
    if (lane + 32 * i < p.D) put(out + lane + 32 * i, acc[i] * inv);
}

template <typename E>
static int launch(const Params& p, cudaStream_t stream) {
  const dim3 grid(p.Hq, (p.T + WARPS - 1) / WARPS), block(32 * WARPS);
  const size_t smem = (size_t)WARPS * p.D * sizeof(float);
  const int nc = (p.D + 31) / 32;
  if (nc <= 2) B200_CUDA_CHECK(launch_pdl(attn_simt_kernel<E, 2>, grid, block, smem, stream, p));
  else if (nc <= 4) B200_CUDA_CHECK(launch_pdl(attn_simt_kernel<E, 4>, grid, block, smem, stream, p));
  else if (nc <= 8) B200_CUDA_CHECK(launch_pdl(attn_simt_kernel<E, 8>, grid, block, smem, stream, p));
  else B200_CUDA_CHECK(launch_pdl(attn_simt_kernel<E, 16>, grid, block, smem, stream, p));
  return 0;
}

}  // namespace as
}  // namespace b200

// q, out [T, Hq, D] (out: rows ldo elements apart, 0: Hq * D), kv [blocks, 2, Hkv, block_size, D]; D % 4 == 0, D <= 512; elem: 2 = bf16, 4 = fp32.
extern "C" int b200_attn_simt(const void* q, const void* kv, void* out, const int* block_tables, const int* seq_lens,
                              const int* qsl, int T, int R, int Hq, int Hkv, int D, int max_blocks, int block_size,
                              long long num_blocks, float scale, int window, float softcap, const float* sinks, int ldo,
                              int elem, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0 || R <= 0) return 0;
  if (D % 4 || D > 512 || Hkv <= 0 || Hq % Hkv || (T + as::WARPS - 1) / as::WARPS > 65535) {
    b200_set_last_error("attn_simt: head sizes of at most 512, a multiple of 4, and fewer than 262140 rows", __FILE__,
                        __LINE__);
    return -1;
  }
  as::Params p{q, kv, out, block_tables, seq_lens, qsl, sinks, T, R, Hq, Hkv, D, max_blocks, block_size, window,
               ldo > 0 ? ldo : Hq * D, num_blocks, scale, softcap};
  return elem == 4 ? as::launch<float>(p, stream) : as::launch<__nv_bfloat16>(p, stream);
}
