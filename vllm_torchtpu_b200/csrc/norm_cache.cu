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

// V elements at a time: 16 bytes, or one element where sizes and strides are no multiple of that
template <int V, typename E>
__device__ __forceinline__ void load(const E* p, float (&v)[V]) {
  if constexpr (V == 1) {
    v[0] = to_f(p[0]);
  } else {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const E* e = reinterpret_cast<const E*>(&u);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = to_f(e[j]);
  }
}
template <int V, typename E>
__device__ __forceinline__ void store(E* p, const float (&v)[V]) {
  if constexpr (V == 1) {
    put(p, v[0]);
  } else {
    uint4 u;
    E* e = reinterpret_cast<E*>(&u);
#pragma unroll
    for (int j = 0; j < V; ++j) put(e + j, v[j]);
    *reinterpret_cast<uint4*>(p) = u;
  }
}

// One CTA per token.
template <typename E, int V>
__global__ void __launch_bounds__(256) norm_cache_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[2][8];
  const int t = blockIdx.x, tid = threadIdx.x;
  const E* row = reinterpret_cast<const E*>(p.row) + (size_t)t * p.ldr;
  const int nq = p.Hq * p.dim, nk = p.Hkv * p.dim;
  const long long slot = p.slots[t];
  float temp = 1.f;
  if (p.temp_every > 0) temp += p.temp_coef * logf((float)((p.positions[t] + 1) / p.temp_every) + 1.f);
  float qs = 1.f, ks = 1.f;
  if (p.q_w != nullptr) {
    float sq = 0.f, sk = 0.f;
    if (p.q_sumsq != nullptr) {
      sq = p.q_sumsq[t];
      sk = p.k_sumsq[t];
    } else {
      for (int i = tid * V; i < nq + nk; i += blockDim.x * V) {
        float v[V], s = 0.f;
        load<V>(row + (i < nq ? i : p.k_off + i - nq), v);
#pragma unroll
        for (int j = 0; j < V; ++j) s += v[j] * v[j];
        if (i < nq) sq += s;
        else sk += s;
      }
      sq = warp_sum(sq);
      sk = warp_sum(sk);
      if ((tid & 31) == 0) {
        red[0][tid >> 5] = sq;
        red[1][tid >> 5] = sk;
      }
      __syncthreads();
      sq = sk = 0.f;
      for (int i = 0; i < (int)blockDim.x / 32; ++i) {
        sq += red[0][i];
        sk += red[1][i];
      }
    }
    qs = 1.f / sqrtf(sq / p.q_size + p.eps);
    ks = 1.f / sqrtf(sk / p.k_size + p.eps);
  }
  qs *= temp;
  E* qo = reinterpret_cast<E*>(p.q_out) + (size_t)t * p.Hq * p.D;
  const E* qw = reinterpret_cast<const E*>(p.q_w);
  const E* kw = reinterpret_cast<const E*>(p.k_w);
  const bool cached = slot >= 0 && slot < p.num_slots;
  const long long blk = cached ? slot / p.block_size : 0;
  const int off = (int)(slot - blk * p.block_size);
  const size_t page = (size_t)p.block_size * p.D;
  E* base = reinterpret_cast<E*>(p.cache) + (size_t)blk * 2 * p.Hkv * page + (size_t)off * p.D;
  // heads: q, then k, then v
  const int total = (p.Hq + (cached ? 2 * p.Hkv : 0)) * p.D;
  for (int i = tid * V; i < total; i += blockDim.x * V) {
    const int h = i / p.D, d = i - h * p.D;
    float v[V], w[V];
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = 0.f;
    if (h < p.Hq) {
      if (d < p.dim) {
        load<V>(row + h * p.dim + d, v);
        if (qw != nullptr) load<V>(qw + h * p.dim + d, w);
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] *= qw != nullptr ? qs * w[j] : qs;
      }
      store<V>(qo + i, v);
    } else {
      const int hk = h - p.Hq;
      if (hk < p.Hkv) {
        if (d < p.dim) {
          load<V>(row + p.k_off + hk * p.dim + d, v);
          if (kw != nullptr) load<V>(kw + hk * p.dim + d, w);
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] *= kw != nullptr ? ks * w[j] : ks;
        }
      } else if (d < p.vdim) {
        load<V>(row + p.v_off + (hk - p.Hkv) * p.vdim + d, v);
      }
      store<V>(base + (size_t)hk * page + d, v);
    }
  }
}

template <typename E>
static int launch(const Params& p, int T, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(E);
  const uintptr_t a = (uintptr_t)p.row | (uintptr_t)p.q_w | (uintptr_t)p.k_w | (uintptr_t)p.q_out | (uintptr_t)p.cache;
  const bool vec = a % 16 == 0 && (p.ldr | p.k_off | p.v_off | p.dim | p.vdim | p.D) % V == 0;
  int threads = ((p.Hq + 2 * p.Hkv) * p.D / (vec ? V : 4) + 31) / 32 * 32;
  threads = threads < 64 ? 64 : (threads > 256 ? 256 : threads);
  if (vec) B200_CUDA_CHECK(launch_pdl(norm_cache_kernel<E, V>, dim3(T), dim3(threads), (size_t)0, stream, p));
  else B200_CUDA_CHECK(launch_pdl(norm_cache_kernel<E, 1>, dim3(T), dim3(threads), (size_t)0, stream, p));
  return 0;
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
  return elem == 4 ? nc::launch<float>(p, T, stream) : nc::launch<__nv_bfloat16>(p, T, stream);
}
