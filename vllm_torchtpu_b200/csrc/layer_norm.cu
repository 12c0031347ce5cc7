// Layer normalisation with a weight and no bias, and the steps around it of blocks that normalise the OUTPUT of
// a sublayer and add it to a 32-bit residual stream:
//
//   ADD:    r' = r + LN(y) * w     (r' fp32, also stored rounded as the next projection's input)
//   plain:  o  = LN(x) * w
//
// and of blocks that normalise the INPUT of a sublayer (RMS norm, weight stored with an offset):
//
//   add_rms: r' = r (+ mult * y),  o = r' / rms(r') * (offset + w)     (r' fp32)
//
// and of blocks that do both: the output y is normalised and scaled first, r' = r + mult * y / rms(y) * post.
//
// mean and variance (mean of the squared deviations) in fp32 over the row, which stays in shared memory between
// the passes.  Also the tanh soft cap of the logits.
#include "common.cuh"

namespace b200 {
namespace ln {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }

template <int V, typename T>
__device__ __forceinline__ void load(const T* p, float (&v)[V]) {
  if constexpr (V == 8 && sizeof(T) == 2) {
    const bf16x8 a = *reinterpret_cast<const bf16x8*>(p);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = __bfloat1622float2(a.v[j]);
      v[2 * j] = f.x;
      v[2 * j + 1] = f.y;
    }
  } else if constexpr (V == 8) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  } else {
    v[0] = to_f(p[0]);
  }
}
template <int V, typename T>
__device__ __forceinline__ void store(T* p, const float (&v)[V]) {
  if constexpr (V == 8 && sizeof(T) == 2) {
    bf16x8 a;
#pragma unroll
    for (int j = 0; j < 4; ++j) a.v[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
    *reinterpret_cast<bf16x8*>(p) = a;
  } else if constexpr (V == 8) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
  } else if constexpr (sizeof(T) == 2) {
    p[0] = __float2bfloat16(v[0]);
  } else {
    p[0] = v[0];
  }
}

// One CTA per row.  TX: type of the row to normalise, TR: of the residual that comes in, TO: of w and of the
// rounded output.  ADD writes res_out (fp32) and, when out is given, its rounded copy; plain writes out.
template <int V, typename TX, typename TR, typename TO, bool ADD>
__global__ void layer_norm_kernel(const TX* __restrict__ x, const TR* __restrict__ res, const TO* __restrict__ w,
                                  float* __restrict__ res_out, TO* __restrict__ out, int H, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  const size_t base = (size_t)blockIdx.x * H;
  float s = 0.f;
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float v[V];
    load<V>(x + base + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) s += v[j];
    store<V>(row + i, v);
  }
  const float mean = block_sum(s, red) / (float)H;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float v[V];
    load<V>(row + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += (v[j] - mean) * (v[j] - mean);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)H + eps);
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float v[V], g[V];
    load<V>(row + i, v);
    load<V>(w + i, g);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = (v[j] - mean) * inv * g[j];
    if constexpr (ADD) {
      float r[V];
      load<V>(res + base + i, r);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] += r[j];
      store<V>(res_out + base + i, v);
    }
    if (out != nullptr) store<V>(out + base + i, v);
  }
}

template <int V, typename TX, typename TR, typename TO, bool ADD>
static int launch(const void* x, const void* res, const void* w, void* res_out, void* out, int T, int H, float eps,
                  cudaStream_t stream) {
  int threads = (H / V + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 512 ? 512 : threads);
  const int smem = H * (int)sizeof(float);
  static unsigned long long seen = 0;
  if (smem > 48 * 1024)
    B200_CUDA_CHECK(ensure_dynamic_smem(layer_norm_kernel<V, TX, TR, TO, ADD>, 200 * 1024, &seen));
  B200_CUDA_CHECK(launch_pdl(layer_norm_kernel<V, TX, TR, TO, ADD>, dim3(T), dim3(threads), (size_t)smem, stream,
                             (const TX*)x, (const TR*)res, (const TO*)w, (float*)res_out, (TO*)out, H, eps));
  return 0;
}

template <typename TX, typename TR, typename TO, bool ADD>
static int launch_v(const void* x, const void* res, const void* w, void* res_out, void* out, int T, int H, float eps,
                    cudaStream_t stream) {
  const uintptr_t a = (uintptr_t)x | (uintptr_t)res | (uintptr_t)w | (uintptr_t)res_out | (uintptr_t)out;
  if (H % 8 == 0 && a % 16 == 0) return launch<8, TX, TR, TO, ADD>(x, res, w, res_out, out, T, H, eps, stream);
  return launch<1, TX, TR, TO, ADD>(x, res, w, res_out, out, T, H, eps, stream);
}

// One CTA per row.  TY: type of the sublayer output y (null: nothing is added), TR: of the stream that comes in, TO: of
// w and of the normalised output; res_out (fp32, may be res itself) is written when given.  POST: y passes a norm with the
// weight post and the factor mult first.
template <int V, typename TY, typename TR, typename TO, bool POST>
__global__ void add_rms_norm_kernel(const TY* __restrict__ y, const TR* res, const TO* __restrict__ w,
                                    const TO* __restrict__ post, float* res_out, TO* __restrict__ out, int H, float eps,
                                    float offset, float mult) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  const size_t base = (size_t)blockIdx.x * H;
  float ss = 0.f, scale = 1.f;
  if constexpr (POST) {
    float sy = 0.f;
    for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
      float a[V];
      load<V>(y + base + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) sy += a[j] * a[j];
      store<V>(row + i, a);
    }
    scale = mult / sqrtf(block_sum(sy, red) / (float)H + eps);
  }
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float v[V];
    load<V>(res + base + i, v);
    if constexpr (POST) {
      float a[V], g[V];
      load<V>(row + i, a);
      load<V>(post + i, g);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] += a[j] * scale * g[j];
    } else if (y != nullptr) {
      float a[V];
      load<V>(y + base + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = fmaf(mult, a[j], v[j]);
    }
    if (res_out != nullptr) store<V>(res_out + base + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += v[j] * v[j];
    store<V>(row + i, v);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)H + eps);
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float v[V], g[V];
    load<V>(row + i, v);
    load<V>(w + i, g);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = v[j] * inv * (offset + g[j]);
    store<V>(out + base + i, v);
  }
}

template <typename TY, typename TR, typename TO, bool POST>
static int launch_add_rms(const void* y, const void* res, const void* w, const void* post, void* res_out, void* out, int T,
                          int H, float eps, float offset, float mult, cudaStream_t stream) {
  const uintptr_t a = (uintptr_t)y | (uintptr_t)res | (uintptr_t)w | (uintptr_t)post | (uintptr_t)res_out | (uintptr_t)out;
  const bool vec = H % 8 == 0 && a % 16 == 0;
  int threads = (H / (vec ? 8 : 1) + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 512 ? 512 : threads);
  const int smem = H * (int)sizeof(float);
  static unsigned long long seen8 = 0, seen1 = 0;
  if (vec) {
    if (smem > 48 * 1024)
      B200_CUDA_CHECK(ensure_dynamic_smem(add_rms_norm_kernel<8, TY, TR, TO, POST>, 200 * 1024, &seen8));
    B200_CUDA_CHECK(launch_pdl(add_rms_norm_kernel<8, TY, TR, TO, POST>, dim3(T), dim3(threads), (size_t)smem, stream,
                               (const TY*)y, (const TR*)res, (const TO*)w, (const TO*)post, (float*)res_out, (TO*)out, H,
                               eps, offset, mult));
  } else {
    if (smem > 48 * 1024)
      B200_CUDA_CHECK(ensure_dynamic_smem(add_rms_norm_kernel<1, TY, TR, TO, POST>, 200 * 1024, &seen1));
    B200_CUDA_CHECK(launch_pdl(add_rms_norm_kernel<1, TY, TR, TO, POST>, dim3(T), dim3(threads), (size_t)smem, stream,
                               (const TY*)y, (const TR*)res, (const TO*)w, (const TO*)post, (float*)res_out, (TO*)out, H,
                               eps, offset, mult));
  }
  return 0;
}

template <typename T>
__global__ void softcap_kernel(const T* __restrict__ x, float* __restrict__ y, size_t n, float cap, float inv_cap) {
  pdl_launch_dependents();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    y[i] = cap * tanhf(to_f(x[i]) * inv_cap);
}

}  // namespace ln
}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16;

// y, res, w: element bytes y_elem / res_elem / w_elem (2 = bf16, 4 = fp32); res_out fp32 (may be res itself);
// out: rounded copy in the type of w, or null.
extern "C" int b200_layer_norm_add(const void* y, int y_elem, const void* res, int res_elem, const void* w, int w_elem,
                                   void* res_out, void* out, int T, int H, float eps, cudaStream_t stream) {
  if (T <= 0 || H <= 0) return 0;
  if (H > 50000) {
    b200_set_last_error("layer_norm: rows of at most 50000 elements", __FILE__, __LINE__);
    return -1;
  }
  if (y_elem == 2 && res_elem == 2 && w_elem == 2)
    return ln::launch_v<bf16, bf16, bf16, true>(y, res, w, res_out, out, T, H, eps, stream);
  if (y_elem == 2 && res_elem == 4 && w_elem == 2)
    return ln::launch_v<bf16, float, bf16, true>(y, res, w, res_out, out, T, H, eps, stream);
  if (y_elem == 4 && res_elem == 4 && w_elem == 4)
    return ln::launch_v<float, float, float, true>(y, res, w, res_out, out, T, H, eps, stream);
  b200_set_last_error("layer_norm_add: unsupported combination of types", __FILE__, __LINE__);
  return -1;
}

extern "C" int b200_layer_norm(const void* x, int x_elem, const void* w, int w_elem, void* out, int T, int H, float eps,
                               cudaStream_t stream) {
  if (T <= 0 || H <= 0) return 0;
  if (H > 50000) {
    b200_set_last_error("layer_norm: rows of at most 50000 elements", __FILE__, __LINE__);
    return -1;
  }
  if (x_elem == 4 && w_elem == 2)
    return ln::launch_v<float, float, bf16, false>(x, nullptr, w, nullptr, out, T, H, eps, stream);
  if (x_elem == 2 && w_elem == 2)
    return ln::launch_v<bf16, float, bf16, false>(x, nullptr, w, nullptr, out, T, H, eps, stream);
  if (x_elem == 4 && w_elem == 4)
    return ln::launch_v<float, float, float, false>(x, nullptr, w, nullptr, out, T, H, eps, stream);
  b200_set_last_error("layer_norm: unsupported combination of types", __FILE__, __LINE__);
  return -1;
}

// y (or null): type of w; res: element bytes res_elem; w, post and out: w_elem (2 = bf16, 4 = fp32); res_out fp32 or null;
// post (or null): weight of the norm y passes first; mult: factor on what is added.
extern "C" int b200_add_rms_norm(const void* y, const void* res, int res_elem, const void* w, const void* post, int w_elem,
                                 void* res_out, void* out, int T, int H, float eps, float offset, float mult,
                                 cudaStream_t stream) {
  if (T <= 0 || H <= 0) return 0;
  if (H > 50000) {
    b200_set_last_error("add_rms_norm: rows of at most 50000 elements", __FILE__, __LINE__);
    return -1;
  }
  const bool pn = post != nullptr && y != nullptr;
#define ADD_RMS(TY, TR, TO)                                                                                             \
  return pn ? ln::launch_add_rms<TY, TR, TO, true>(y, res, w, post, res_out, out, T, H, eps, offset, mult, stream)      \
            : ln::launch_add_rms<TY, TR, TO, false>(y, res, w, nullptr, res_out, out, T, H, eps, offset, mult, stream)
  if (res_elem == 2 && w_elem == 2) ADD_RMS(bf16, bf16, bf16);
  if (res_elem == 4 && w_elem == 2) ADD_RMS(bf16, float, bf16);
  if (res_elem == 4 && w_elem == 4) ADD_RMS(float, float, float);
#undef ADD_RMS
  b200_set_last_error("add_rms_norm: unsupported combination of types", __FILE__, __LINE__);
  return -1;
}

// y = cap * tanh(x / cap), fp32 out (in place when x is fp32)
extern "C" int b200_softcap(const void* x, int x_elem, float* y, long long n, float cap, cudaStream_t stream) {
  if (n <= 0) return 0;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (x_elem == 2)
    B200_CUDA_CHECK(launch_pdl(ln::softcap_kernel<bf16>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream,
                               (const bf16*)x, y, (size_t)n, cap, 1.f / cap));
  else
    B200_CUDA_CHECK(launch_pdl(ln::softcap_kernel<float>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream,
                               (const float*)x, y, (size_t)n, cap, 1.f / cap));
  return 0;
}
