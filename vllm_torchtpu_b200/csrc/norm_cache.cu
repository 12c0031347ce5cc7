// q / k / v of grouped-query attention without rotation, in one launch in front of the paged attention:
//
//   q <- q / rms(all of q) * w_q * (1 + coef * ln(floor((p + 1) / every) + 1))      -> q_out [T, Hq, D]
//   k <- k / rms(all of k) * w_k                                                     -> page of the token's slot
//   v                                                                                -> page of the token's slot
//
// The norms run over the whole projection, before it is split into heads.  Heads of dim (vdim) elements are stored in
// D columns, zeros behind them.  Everything in fp32, rounded once.
#include "common.cuh"

namespace b200 {
namespace nc {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct Params {
  const void *row, *q_w, *k_w;
  void *q_out, *cache;
  const int *positions, *slots;
  const float *q_sumsq, *k_sumsq;      // squared sums of sharded rows, or null
  int ldr, k_off, v_off, Hq, Hkv, dim, vdim, D, block_size, temp_every;
  long long num_slots;
  float eps, q_size, k_size, temp_coef;
};

// One CTA per token.
template <typename E>
__global__ void __launch_bounds__(256) norm_cache_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x;
  const E* row = reinterpret_cast<const E*>(p.row) + (size_t)t * p.ldr;
  const int nq = p.Hq * p.dim, nk = p.Hkv * p.dim;
  float qs = 1.f, ks = 1.f;
  if (p.q_w != nullptr) {
    float sq = 0.f, sk = 0.f;
    if (p.q_sumsq != nullptr) {
      sq = p.q_sumsq[t];
      sk = p.k_sumsq[t];
    } else {
      for (int i = threadIdx.x; i < nq; i += blockDim.x) {
        const float v = to_f(row[i]);
        sq += v * v;
      }
      for (int i = threadIdx.x; i < nk; i += blockDim.x) {
        const float v = to_f(row[p.k_off + i]);
        sk += v * v;
      }
      sq = block_sum(sq, red);
      sk = block_sum(sk, red);
    }
    qs = 1.f / sqrtf(sq / p.q_size + p.eps);
    ks = 1.f / sqrtf(sk / p.k_size + p.eps);
  }
  float temp = 1.f;
  if (p.temp_every > 0) temp += p.temp_coef * logf((float)((p.positions[t] + 1) / p.temp_every) + 1.f);
  E* qo = reinterpret_cast<E*>(p.q_out) + (size_t)t * p.Hq * p.D;
  const E* qw = reinterpret_cast<const E*>(p.q_w);
  for (int i = threadIdx.x; i < p.Hq * p.D; i += blockDim.x) {
    const int h = i / p.D, d = i - h * p.D, src = h * p.dim + d;
    float v = 0.f;
    if (d < p.dim) {
      v = to_f(row[src]) * qs;
      if (qw != nullptr) v *= to_f(qw[src]);
      v *= temp;
    }
    put(qo + i, v);
  }
  const long long slot = p.slots[t];
  if (slot < 0 || slot >= p.num_slots) return;
  const long long blk = slot / p.block_size;
  const int off = (int)(slot - blk * p.block_size);
  const E* kw = reinterpret_cast<const E*>(p.k_w);
  const size_t page = (size_t)p.block_size * p.D;
  E* base = reinterpret_cast<E*>(p.cache) + (size_t)blk * 2 * p.Hkv * page + (size_t)off * p.D;
  for (int i = threadIdx.x; i < p.Hkv * p.D; i += blockDim.x) {
    const int h = i / p.D, d = i - h * p.D;
    float k = 0.f, v = 0.f;
    if (d < p.dim) {
      k = to_f(row[p.k_off + h * p.dim + d]) * ks;
      if (kw != nullptr) k *= to_f(kw[h * p.dim + d]);
    }
    if (d < p.vdim) v = to_f(row[p.v_off + h * p.vdim + d]);
    put(base + (size_t)h * page + d, k);
    put(base + (size_t)(p.Hkv + h) * page + d, v);
  }
}

}  // namespace nc
}  // namespace b200

// cache [blocks, 2, Hkv, block_size, D]; elem: 2 = bf16, 4 = fp32 (all tensors alike); temp_every 0: no temperature.
extern "C" int b200_norm_cache(const void* row, int ldr, int k_off, int v_off, const void* q_w, const void* k_w,
                               const int* positions, const int* slots, const float* q_sumsq, const float* k_sumsq,
                               void* q_out, void* cache, int T, int Hq, int Hkv, int dim, int vdim, int D,
                               int block_size, long long num_blocks, float eps, float q_size, float k_size,
                               float temp_coef, int temp_every, int elem, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0) return 0;
  if (dim > D || vdim > D || (q_w == nullptr) != (k_w == nullptr)) {
    b200_set_last_error("norm_cache: head sizes exceed the cache's, or only one norm weight", __FILE__, __LINE__);
    return -1;
  }
  nc::Params p{row, q_w, k_w, q_out, cache, positions, slots, q_sumsq, k_sumsq, ldr, k_off, v_off, Hq, Hkv, dim, vdim,
               D, block_size, temp_every, num_blocks * block_size, eps, q_size, k_size, temp_coef};
  int threads = ((Hq * dim + 3) / 4 + 31) / 32 * 32;
  threads = threads < 64 ? 64 : (threads > 256 ? 256 : threads);
  if (elem == 4)
    B200_CUDA_CHECK(launch_pdl(nc::norm_cache_kernel<float>, dim3(T), dim3(threads), (size_t)0, stream, p));
  else
    B200_CUDA_CHECK(launch_pdl(nc::norm_cache_kernel<__nv_bfloat16>, dim3(T), dim3(threads), (size_t)0, stream, p));
  return 0;
}
