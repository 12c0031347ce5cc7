// CUDA-core GEMM for what the tensor-core kernels do not take: 32-bit activations and weights (full fp32
// products and sums, no reduced-precision mode), and bf16 operands whose sizes or strides are no multiple of
// the TMA granule.  Batched over heads, with the epilogues the tcgen05 kernels have:
//
//   Y[t, b * ys + n] = act( sum_k X[t, b * xs + k] * W[b * N + n, k] + bias[n] ) [ * sigmoid(G[t, b * N + n]) ]
//   with gate_rows:  Y[t, n] = gelu( . ) * G[gate_rows[t], n], gelu in its tanh form
//
// act: 0 none, 1 gelu (erf), 2 out_scale and soft cap (cap * tanh(. / cap), cap 0: none) with fp32 output.  64 x 64 output tile per CTA, 4 x 4 per thread, 16-wide K slices in shared memory.
#include "common.cuh"

namespace b200 {
namespace simt {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

struct Params {
  const void *x, *w, *bias, *gate;
  const int* gate_rows;
  int gate_count;
  void* y;
  int T, N, K, batch, act, y_f32;
  float cap, out_scale;
  long long ldx, ldw, ldy, ldg, xs, ys;
};

constexpr int TM = 64, TN = 64, TK = 16;

template <typename E>
__global__ void __launch_bounds__(256) gemm_kernel(const Params p) {
  __shared__ float sx[TK][TM + 4];
  __shared__ float sw[TK][TN + 4];
  pdl_launch_dependents();
  pdl_wait();
  const int n_tiles = (p.N + TN - 1) / TN;
  const int b = blockIdx.x / n_tiles, n0 = (blockIdx.x - b * n_tiles) * TN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const E* w = reinterpret_cast<const E*>(p.w) + (size_t)b * p.N * p.ldw;
  for (int t0 = blockIdx.y * TM; t0 < p.T; t0 += gridDim.y * TM) {
    const E* x = reinterpret_cast<const E*>(p.x) + (size_t)b * p.xs;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += TK) {
#pragma unroll
      for (int i = 0; i < TM * TK / 256; ++i) {
        const int idx = threadIdx.x + i * 256, k = idx & (TK - 1), r = idx / TK;
        const bool kin = k0 + k < p.K;
        sx[k][r] = (kin && t0 + r < p.T) ? to_f(x[(size_t)(t0 + r) * p.ldx + k0 + k]) : 0.f;
        sw[k][r] = (kin && n0 + r < p.N) ? to_f(w[(size_t)(n0 + r) * p.ldw + k0 + k]) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < TK; ++k) {
        const float4 a = *reinterpret_cast<const float4*>(&sx[k][ty * 4]);
        const float4 c = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
        const float av[4] = {a.x, a.y, a.z, a.w}, cv[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], cv[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = t0 + ty * 4 + i;
      if (t >= p.T) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + tx * 4 + j;
        if (n >= p.N) continue;
        float v = acc[i][j];
        if (p.bias) v += to_f(reinterpret_cast<const E*>(p.bias)[n]);
        if (p.act == 1) v = gelu_erf(v);
        if (p.act == 2) v = soft_cap(v * p.out_scale, p.cap);
        if (p.gate_rows) {
          const int row = min(max(p.gate_rows[t], 0), p.gate_count - 1);
          const float z = 0.7978845608028654f * (v + 0.044715f * v * v * v);
          v = 0.5f * v * (1.f + tanhf(z)) * to_f(reinterpret_cast<const E*>(p.gate)[(size_t)row * p.ldg + n]);
        } else if (p.gate) {
          const float g = to_f(reinterpret_cast<const E*>(p.gate)[(size_t)t * p.ldg + (size_t)b * p.N + n]);
          v *= 1.f / (1.f + expf(-g));
        }
        if (p.y_f32)
          reinterpret_cast<float*>(p.y)[(size_t)t * p.ldy + (size_t)b * p.ys + n] = v;
        else
          reinterpret_cast<E*>(p.y)[(size_t)t * p.ldy + (size_t)b * p.ys + n] = from_f<E>(v);
      }
    }
  }
}

// Rows [off[e], off[e + 1]) of x times w[e] [N, K]: experts on the CUDA cores.  grid (column tiles, experts); a CTA walks
// over the row tiles of its expert.
template <typename E>
__global__ void __launch_bounds__(256) grouped_kernel(const E* __restrict__ x, const E* __restrict__ w, E* __restrict__ y,
                                                      const int* __restrict__ off, int N, int K, int act) {
  __shared__ float sx[TK][TM + 4];
  __shared__ float sw[TK][TN + 4];
  pdl_launch_dependents();
  pdl_wait();
  const int e = blockIdx.y, n0 = blockIdx.x * TN, r0 = off[e], r1 = off[e + 1];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const E* we = w + (size_t)e * N * K;
  for (int t0 = r0; t0 < r1; t0 += TM) {
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += TK) {
#pragma unroll
      for (int i = 0; i < TM * TK / 256; ++i) {
        const int idx = threadIdx.x + i * 256, k = idx & (TK - 1), r = idx / TK;
        const bool kin = k0 + k < K;
        sx[k][r] = (kin && t0 + r < r1) ? to_f(x[(size_t)(t0 + r) * K + k0 + k]) : 0.f;
        sw[k][r] = (kin && n0 + r < N) ? to_f(we[(size_t)(n0 + r) * K + k0 + k]) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < TK; ++k) {
        const float4 a = *reinterpret_cast<const float4*>(&sx[k][ty * 4]);
        const float4 c = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
        const float av[4] = {a.x, a.y, a.z, a.w}, cv[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], cv[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
        if (t < r1 && n < N) y[(size_t)t * N + n] = from_f<E>(act == 4 ? relu_squared(acc[i][j]) : acc[i][j]);
      }
  }
}

}  // namespace simt
}  // namespace b200

// x [R, K], y [R, N], w [groups, N, K], off int[groups + 1] on the device; act 0 none, 4 the square of relu; elem: 2 = bf16,
// 4 = fp32 (all operands alike).
extern "C" int b200_grouped_gemm_simt(const void* x, const void* w, void* y, const int* off, int groups, int N, int K,
                                      int act, int elem, cudaStream_t stream) {
  using namespace b200;
  if (groups <= 0 || N <= 0) return 0;
  const dim3 grid((N + simt::TN - 1) / simt::TN, groups);
  if (elem == 4)
    B200_CUDA_CHECK(launch_pdl(simt::grouped_kernel<float>, grid, dim3(256), (size_t)0, stream, (const float*)x,
                               (const float*)w, (float*)y, off, N, K, act));
  else
    B200_CUDA_CHECK(launch_pdl(simt::grouped_kernel<__nv_bfloat16>, grid, dim3(256), (size_t)0, stream,
                               (const __nv_bfloat16*)x, (const __nv_bfloat16*)w, (__nv_bfloat16*)y, off, N, K, act));
  return 0;
}

// elem: 2 = bf16, 4 = fp32 (all operands alike); strides in elements.  gate_rows (or null): token t's gate is row
// gate_rows[t] of a table of gate_count rows.
extern "C" int b200_gemm_simt(const void* x, const void* w, void* y, const void* bias, const void* gate,
                              const int* gate_rows, int gate_count, int T, int N, int K, int batch, long long ldx, long long ldw, long long ldy, long long ldg,
                              long long xs, long long ys, int act, float cap, float out_scale, int elem, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0 || N <= 0 || batch <= 0) return 0;
  simt::Params p{x, w, bias, gate, gate_rows, gate_count, y, T, N, K, batch, act, act == 2 ? 1 : 0, cap, out_scale, ldx, ldw, ldy, ldg, xs, ys};
  const long long gx = (long long)batch * ((N + simt::TN - 1) / simt::TN);
  int gy = (T + simt::TM - 1) / simt::TM;
  if (gy > 65535) gy = 65535;
  const dim3 grid((unsigned)gx, gy);
  if (elem == 4)
    B200_CUDA_CHECK(launch_pdl(simt::gemm_kernel<float>, grid, dim3(256), (size_t)0, stream, p));
  else
    B200_CUDA_CHECK(launch_pdl(simt::gemm_kernel<__nv_bfloat16>, grid, dim3(256), (size_t)0, stream, p));
  return 0;
}
