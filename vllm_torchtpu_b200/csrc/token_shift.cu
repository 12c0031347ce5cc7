// Token shift behind the norm of a sublayer's input, and the small steps around a 32-bit residual stream that no GEMM or
// norm takes along.
//
//   r' = r (+ mult * y, or + mult * y / rms(y) * post),   h = r' / rms(r') * (offset + w)
//   out_t = h_t + (h_(t-1) - h_t) * shift                     zeros in front of a sequence
//
// h stays fp32 until it is shifted.  h of every request's last token is kept in state [slots, H] (fp32, by batch slot); a
// portion that starts at position 0 does not read it.
//
// A CTA takes ROWS rows and computes the row in front of them as well, so that no row waits for another CTA; r' goes to a
// buffer of its own because that row's r is read twice.  The state is read and written by the CTA that holds the portion's
// first row: where the portion ends in another CTA, this one computes the last row once more.
#include "common.cuh"

namespace b200 {
namespace ts {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

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
  } else {
    put(p, v[0]);
  }
}

struct Params {
  const void *y, *res, *w, *post, *shift;
  float *res_out, *state, *rows;       // rows (or null): h itself, not shifted
  void* out;
  const int *qsl, *seq_lens, *slots;
  int T, H, R;
  float eps, offset, mult;
};

// sums of N values over the CTA
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float (*red)[32]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    v[i] = warp_sum(v[i]);
    if (lane == 0) red[i][warp] = v[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(lane < nw ? red[i][lane] : 0.f);
  __syncthreads();
}

// h of N rows, row t0 + i into hold[i] (a row outside [0, T) is zero); r' of the rows from `own` on is stored
template <int N, int V, typename TY, typename TR, typename TO>
__device__ __forceinline__ void normed_rows(const Params& p, int t0, int own, float* hold, float (*red)[32]) {
  const TY* y = reinterpret_cast<const TY*>(p.y);
  const TR* res = reinterpret_cast<const TR*>(p.res);
  const TO *w = reinterpret_cast<const TO*>(p.w), *post = reinterpret_cast<const TO*>(p.post);
  const int H = p.H;
  float s[N];
  if (p.post != nullptr) {
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = 0.f;
    for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int t = t0 + i;
        if (t < 0 || t >= p.T) continue;
        float a[V];
        load<V>(y + (size_t)t * H + c, a);
#pragma unroll
        for (int j = 0; j < V; ++j) s[i] = fmaf(a[j], a[j], s[i]);
        store<V>(hold + (size_t)i * H + c, a);
      }
    }
    block_sums<N>(s, red);
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = p.mult / sqrtf(s[i] / (float)H + p.eps);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = p.mult;
  }
  float ss[N];
#pragma unroll
  for (int i = 0; i < N; ++i) ss[i] = 0.f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float g[V];
    if (p.post != nullptr) load<V>(post + c, g);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int t = t0 + i;
      float v[V];
      if (t < 0 || t >= p.T) {
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = 0.f;
      } else {
        load<V>(res + (size_t)t * H + c, v);
        if (p.post != nullptr) {
          float a[V];
          load<V>(hold + (size_t)i * H + c, a);
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] += a[j] * s[i] * g[j];
        } else if (y != nullptr) {
          float a[V];
          load<V>(y + (size_t)t * H + c, a);
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = fmaf(s[i], a[j], v[j]);
        }
        if (i >= own) store<V>(p.res_out + (size_t)t * H + c, v);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) ss[i] = fmaf(v[j], v[j], ss[i]);
      store<V>(hold + (size_t)i * H + c, v);
    }
  }
  block_sums<N>(ss, red);
#pragma unroll
  for (int i = 0; i < N; ++i) ss[i] = 1.f / sqrtf(ss[i] / (float)H + p.eps);
  // (a thread reads back its own columns only)
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float g[V];
    load<V>(w + c, g);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      float v[V];
      load<V>(hold + (size_t)i * H + c, v);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = v[j] * ss[i] * (p.offset + g[j]);
      store<V>(hold + (size_t)i * H + c, v);
    }
  }
}

struct Row {
  int from;                            // 0: zeros, 1: the row in front of it, 2: the state
  int slot, last;                      // first rows of a portion: state slot (-1: none) and the portion's last row
};

// grid (ceil(T / ROWS)).  shared memory: [ROWS + 1][H]
template <int ROWS, int V, typename TY, typename TR, typename TO>
__global__ void __launch_bounds__(512) norm_shift_kernel(const Params p) {
  extern __shared__ __align__(16) float hold[];
  __shared__ float red[ROWS + 1][32];
  __shared__ Row info[ROWS];
  const int t0 = blockIdx.x * ROWS, H = p.H, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  for (int i = warp; i < ROWS; i += nw) {
    // request of the row: as many as end at it or before (qsl is monotone and repeats its last value behind the last one)
    const int t = t0 + i;
    int r = 0;
    for (int k = lane; k < p.R + lane; k += 32)
      r += __popc(__ballot_sync(0xffffffffu, k < p.R && p.qsl[min(k, p.R - 1) + 1] <= t));
    Row x{0, -1, -1};
    if (t < p.T && r < p.R) {
      const int qs = p.qsl[r], len = p.qsl[r + 1] - qs, start = p.seq_lens[r] - len;
      if (t > qs) {
        x.from = 1;
      } else {
        x.slot = p.slots[r];
        x.last = qs + len - 1;
        x.from = start > 0 && x.slot >= 0 ? 2 : 0;
      }
    }
    if (lane == 0) info[i] = x;
  }
  __syncthreads();
  bool before = false;                 // some row needs the one in front of the CTA's
  before = info[0].from == 1;
  if (before) normed_rows<ROWS + 1, V, TY, TR, TO>(p, t0 - 1, 1, hold, red);
  else normed_rows<ROWS, V, TY, TR, TO>(p, t0, 0, hold + H, red);
  const TO* shift = reinterpret_cast<const TO*>(p.shift);
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float m[V];
    load<V>(shift + c, m);
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int t = t0 + i;
      if (t >= p.T) break;
      const Row x = info[i];
      float v[V], b[V];
      load<V>(hold + (size_t)(i + 1) * H + c, v);
      if (x.from == 1) {
        load<V>(hold + (size_t)i * H + c, b);
      } else if (x.from == 2) {
        load<V>(p.state + (size_t)x.slot * H + c, b);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) b[j] = 0.f;
      }
      if (p.rows != nullptr) store<V>(p.rows + (size_t)t * H + c, v);
      if (x.slot >= 0 && x.last >= t && x.last < t0 + ROWS) {
        float l[V];
        load<V>(hold + (size_t)(x.last - t0 + 1) * H + c, l);
        store<V>(p.state + (size_t)x.slot * H + c, l);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] += (b[j] - v[j]) * m[j];
      store<V>(reinterpret_cast<TO*>(p.out) + (size_t)t * H + c, v);
    }
  }
  // a portion that goes on behind the CTA's rows (at most one does, the last to begin here)
  int slot = -1, last = -1;
  for (int i = 0; i < ROWS; ++i)
    if (info[i].slot >= 0 && info[i].last >= t0 + ROWS) {
      slot = info[i].slot;
      last = info[i].last;
    }
  if (slot < 0) return;
  // every thread is done with the old state (its own columns) and with its part of `hold`
  normed_rows<1, V, TY, TR, TO>(p, last, 1, hold, red);
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float l[V];
    load<V>(hold + c, l);
    store<V>(p.state + (size_t)slot * H + c, l);
  }
}

template <int ROWS, int V, typename TY, typename TR, typename TO>
static int launch_rows(const Params& p, cudaStream_t stream) {
  int threads = (p.H / V + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 512 ? 512 : threads);
  const int smem = (ROWS + 1) * p.H * (int)sizeof(float);
  static unsigned long long seen = 0;
  if (smem > 44 * 1024)
    B200_CUDA_CHECK(ensure_dynamic_smem(norm_shift_kernel<ROWS, V, TY, TR, TO>, 220 * 1024, &seen));
  norm_shift_kernel<ROWS, V, TY, TR, TO><<<(p.T + ROWS - 1) / ROWS, threads, smem, stream>>>(p);
  B200_CUDA_CHECK(cudaGetLastError());
  return 0;
}
template <int V, typename TY, typename TR, typename TO>
static int launch(const Params& p, int single, cudaStream_t stream) {
  // rows of a CTA share their loads' latency and one recomputed row; two CTAs have to fit on an SM
  if (single || p.H > 9000) return launch_rows<1, V, TY, TR, TO>(p, stream);
  if (p.H <= 4096) return launch_rows<4, V, TY, TR, TO>(p, stream);
  return launch_rows<2, V, TY, TR, TO>(p, stream);
}
template <typename TY, typename TR, typename TO>
static int launch_v(const Params& p, int single, cudaStream_t stream) {
  const uintptr_t a = (uintptr_t)p.y | (uintptr_t)p.res | (uintptr_t)p.w | (uintptr_t)p.post | (uintptr_t)p.shift |
                      (uintptr_t)p.res_out | (uintptr_t)p.state | (uintptr_t)p.rows | (uintptr_t)p.out;
  return p.H % 8 == 0 && a % 16 == 0 ? launch<8, TY, TR, TO>(p, single, stream) : launch<1, TY, TR, TO>(p, single, stream);
}

// r = res + mult * y, stored fp32 and rounded
template <typename E, int V>
__global__ void residual_add_kernel(const E* __restrict__ y, const float* res, float* r, E* __restrict__ out, size_t n,
                                    float mult) {
  for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; i < n; i += (size_t)gridDim.x * blockDim.x * V) {
    float a[V], v[V];
    load<V>(y + i, a);
    load<V>(res + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = fmaf(mult, a[j], v[j]);
    store<V>(r + i, v);
    store<V>(out + i, v);
  }
}

// y[t] + sigmoid(gate[t]) * z[t], a row per CTA
template <typename E>
__global__ void add_gated_kernel(const E* __restrict__ y, const E* __restrict__ z, const float* __restrict__ gate, int ldg,
                                 E* __restrict__ out, int H) {
  const size_t t = blockIdx.x;
  const float g = 1.f / (1.f + expf(-gate[t * ldg]));
  for (int i = threadIdx.x; i < H; i += blockDim.x) put(out + t * H + i, fmaf(g, to_f(z[t * H + i]), to_f(y[t * H + i])));
}

// columns of strided rows, in place
template <typename E>
__global__ void tanh_kernel(E* x, int ld, int T, int n) {
  const size_t total = (size_t)T * n;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    E* e = x + (i / n) * ld + i % n;
    put(e, tanhf(to_f(*e)));
  }
}

__global__ void resolve_kernel(const int* __restrict__ ids, const int* __restrict__ src, const int* __restrict__ last,
                               int* __restrict__ out, int T) {
  const int t = blockIdx.x * blockDim.x + threadIdx.x;
  if (t < T) out[t] = src[t] >= 0 ? last[src[t]] : ids[t];
}

static int grid_of(size_t work) {
  const size_t b = (work + 255) / 256;
  return b < 1 ? 1 : (b > 148 * 16 ? 148 * 16 : (int)b);
}

}  // namespace ts
}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16;

// y (or null), w, post (or null), shift, out: w_elem bytes an element (2 = bf16, 4 = fp32); res: res_elem; res_out [T, H]
// fp32, no part of it in res; single: portions have one token each.
extern "C" int b200_norm_shift(const void* y, const void* res, int res_elem, const void* w, const void* post,
                               const void* shift, int w_elem, float* res_out, float* state, float* rows, void* out,
                               const int* qsl, const int* seq_lens, const int* slots, int T, int H, int R, float eps,
                               float offset, float mult, int single, cudaStream_t stream) {
  if (T <= 0 || H <= 0) return 0;
  if (H > 27000 || R <= 0 || (const void*)res_out == res) {
    b200_set_last_error("norm_shift: rows of at most 27000 elements, a request, and an output apart from the input", __FILE__,
                        __LINE__);
    return -1;
  }
  ts::Params p{y, res, w, y == nullptr ? nullptr : post, shift, res_out, state, rows, out, qsl, seq_lens, slots, T, H, R, eps,
               offset, mult};
  if (res_elem == 2 && w_elem == 2) return ts::launch_v<bf16, bf16, bf16>(p, single, stream);
  if (res_elem == 4 && w_elem == 2) return ts::launch_v<bf16, float, bf16>(p, single, stream);
  if (res_elem == 4 && w_elem == 4) return ts::launch_v<float, float, float>(p, single, stream);
  b200_set_last_error("norm_shift: unsupported combination of types", __FILE__, __LINE__);
  return -1;
}

// r fp32 (may be res itself); elem of y and out: 2 = bf16, 4 = fp32
extern "C" int b200_residual_add(const void* y, const float* res, float* r, void* out, long long n, float mult, int elem,
                                 cudaStream_t stream) {
  if (n <= 0) return 0;
  const uintptr_t a = (uintptr_t)y | (uintptr_t)res | (uintptr_t)r | (uintptr_t)out;
  const bool vec = n % 8 == 0 && a % 16 == 0;
  const int grid = ts::grid_of((size_t)n / (vec ? 8 : 1));
  if (elem == 4 && vec)
    ts::residual_add_kernel<float, 8><<<grid, 256, 0, stream>>>((const float*)y, res, r, (float*)out, (size_t)n, mult);
  else if (elem == 4)
    ts::residual_add_kernel<float, 1><<<grid, 256, 0, stream>>>((const float*)y, res, r, (float*)out, (size_t)n, mult);
  else if (vec)
    ts::residual_add_kernel<bf16, 8><<<grid, 256, 0, stream>>>((const bf16*)y, res, r, (bf16*)out, (size_t)n, mult);
  else
    ts::residual_add_kernel<bf16, 1><<<grid, 256, 0, stream>>>((const bf16*)y, res, r, (bf16*)out, (size_t)n, mult);
  B200_CUDA_CHECK(cudaGetLastError());
  return 0;
}

extern "C" int b200_add_gated(const void* y, const void* z, const float* gate, int ldg, void* out, int T, int H, int elem,
                              cudaStream_t stream) {
  if (T <= 0 || H <= 0) return 0;
  if (elem == 4)
    ts::add_gated_kernel<float><<<T, 256, 0, stream>>>((const float*)y, (const float*)z, gate, ldg, (float*)out, H);
  else
    ts::add_gated_kernel<bf16><<<T, 256, 0, stream>>>((const bf16*)y, (const bf16*)z, gate, ldg, (bf16*)out, H);
  B200_CUDA_CHECK(cudaGetLastError());
  return 0;
}

extern "C" int b200_tanh_columns(void* x, int ld, int T, int n, int elem, cudaStream_t stream) {
  if (T <= 0 || n <= 0) return 0;
  if (elem == 4) ts::tanh_kernel<float><<<ts::grid_of((size_t)T * n), 256, 0, stream>>>((float*)x, ld, T, n);
  else ts::tanh_kernel<bf16><<<ts::grid_of((size_t)T * n), 256, 0, stream>>>((bf16*)x, ld, T, n);
  B200_CUDA_CHECK(cudaGetLastError());
  return 0;
}

// out[t] = src[t] >= 0 ? last[src[t]] : ids[t]
extern "C" int b200_resolve_tokens(const int* ids, const int* src, const int* last, int* out, int T, cudaStream_t stream) {
  if (T <= 0) return 0;
  ts::resolve_kernel<<<(T + 255) / 256, 256, 0, stream>>>(ids, src, last, out, T);
  B200_CUDA_CHECK(cudaGetLastError());
  return 0;
}
