// Attention layers with short convolutions: everything between the packed projection and the paged attention in one
// launch, and what follows the softmax of such layers.
//
//   y_t = sum_j w[j] u_(t - taps + 1 + j)     per channel of q, k and v (zeros in front of the sequence)
//   q, k: dimensions 2i, 2i + 1 of a head (of one map) turn by position * inv_freq[i], cos and sin times rot_mult
//   q -> q_out [T, heads * maps, D];   k, v -> page of the token's slot
//
// Heads are stored in D columns with zeros behind them.  With two maps per head a key row holds both maps side by side and
// query row 2h + m has its map's columns only, so that plain attention over D columns gives the scores of one map.
//
// The inputs of earlier steps are in a ring of `taps` rows per request (input of position p in row p % taps): the row that
// a single token writes is none of those it reads.  The last inputs of longer portions are written by a second launch,
// once all of their readers are done.  fp32 arithmetic, rounded once.
//
// A thread owns 16 bytes of channels over a run of tokens, so that every input is read once and the pairs of the rotation
// are its own; angles are evaluated once per token and CTA.
#include "common.cuh"

namespace b200 {
namespace cc {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct Params {
  const void *row, *w;                 // w [taps, channels]
  void *q_out, *cache, *ring;
  const float* inv_freq;
  const int *slots, *qsl, *seq_lens, *state_slots;
  int ldr, q_off, k_off, v_off, H, G, dim, vdim, maps, D, taps, pairs, block_size, T, R;
  long long num_slots;
  float rot_mult;
};

struct Token {
  int qs, len, pos, state;             // first row and length of its portion, position, state slot (-1: none)
  long long slot;
};

// request of row t: qsl is monotone and repeats its last value behind the last request
__device__ __forceinline__ Token token_of(const Params& p, int t) {
  Token k{t, 0, 0, -1, -1};
  if (t >= p.T || t >= p.qsl[p.R]) return k;
  int lo = 0, hi = p.R;                // qsl[lo] <= t < qsl[hi]
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (p.qsl[mid] <= t) lo = mid;
    else hi = mid;
  }
  k.qs = p.qsl[lo];
  k.len = p.qsl[lo + 1] - k.qs;
  k.pos = p.seq_lens[lo] - k.len + t - k.qs;
  k.state = p.state_slots[lo];
  k.slot = p.slots[t];
  return k;
}

template <typename E, int V, bool VEC>
__device__ __forceinline__ void load(const E* p, int e0, int e1, float (&v)[V]) {
  if constexpr (VEC) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const E* e = reinterpret_cast<const E*>(&u);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = to_f(e[j]);
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = j >= e0 && j < e1 ? to_f(p[j]) : 0.f;
  }
}
template <typename E, int V, bool VEC>
__device__ __forceinline__ void store(E* p, const float (&v)[V], int e0 = 0, int e1 = V) {
  if constexpr (VEC) {
    uint4 u;
    E* e = reinterpret_cast<E*>(&u);
#pragma unroll
    for (int j = 0; j < V; ++j) put(e + j, v[j]);
    *reinterpret_cast<uint4*>(p) = u;
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j)
      if (j >= e0 && j < e1) put(p + j, v[j]);
  }
}

// The channels that vector `vec` of the stored heads takes: row column and ring channel of its element 0 (elements e0 ..
// e1 - 1 exist, the others are zeros), head index (q rows, then k, then v heads) and first column in the head.
struct Where {
  int hh, d0, ch, col, e0, e1;
  bool rotated;
};
template <int V>
__device__ __forceinline__ Where where_is(const Params& p, int vec) {
  const int nv = p.D / V, nq = p.H * p.maps, cq = nq * p.dim, ck = p.G * p.maps * p.dim;
  Where w;
  w.hh = vec / nv;
  w.d0 = (vec - w.hh * nv) * V;
  int lo = 0, hi;
  w.rotated = p.pairs > 0;
  if (w.hh < nq) {
    const int h = w.hh / p.maps, m = w.hh - h * p.maps;
    w.ch = h * p.maps * p.dim + w.d0;
    w.col = p.q_off + w.ch;
    lo = m * p.dim;
    hi = lo + p.dim;
  } else if (w.hh < nq + p.G) {
    w.ch = (w.hh - nq) * p.maps * p.dim + w.d0;
    w.col = p.k_off + w.ch;
    w.ch += cq;
    hi = p.maps * p.dim;
  } else {
    w.ch = (w.hh - nq - p.G) * p.vdim + w.d0;
    w.col = p.v_off + w.ch;
    w.ch += cq + ck;
    hi = p.vdim;
    w.rotated = false;
  }
  w.e0 = max(lo - w.d0, 0);
  w.e1 = min(hi - w.d0, V);
  return w;
}

// grid (token runs of TT, parts of the vectors).  KM: taps the window is held in registers for (0: any number, re-read).
// A run is walked in groups of up to four tokens whose inputs are requested together; the inputs in front of the run are
// requested before the tokens' requests are known, and what turns out to belong to another portion is replaced.
template <typename E, int V, bool VEC, int KM, int TT>
__global__ void __launch_bounds__(256, 2) conv_cache_kernel(const Params p) {
  extern __shared__ __align__(16) float2 turn[];          // [TT][pairs]
  __shared__ Token tok[TT];
  const int tid = threadIdx.x, t0 = blockIdx.x * TT;
  const int nq = p.H * p.maps, C = (nq + p.G * p.maps) * p.dim + p.G * p.vdim, vecs = (nq + 2 * p.G) * (p.D / V);
  const E* row = reinterpret_cast<const E*>(p.row);
  E* ring = reinterpret_cast<E*>(p.ring);
  constexpr int HB = KM > 1 ? KM - 1 : 1;
  bool ready = false;
  for (int v0 = blockIdx.y * blockDim.x; v0 < vecs; v0 += gridDim.y * blockDim.x) {
    const int vec = v0 + tid;
    const Where x = where_is<V>(p, min(vec, vecs - 1));
    const bool any = x.e0 < x.e1 && vec < vecs;
    const E* w = reinterpret_cast<const E*>(p.w) + x.ch;
    constexpr int GR = TT < 4 ? TT : 4;
    uint4 raw[GR], before[HB];                             // inputs of a group and of the rows in front of the run
    uint4 wt[VEC && KM > 0 ? KM : 1];                      // wt[j]: weights of the inputs j positions before
    auto request = [&](int t) {
      return any && t >= 0 && t < p.T ? *reinterpret_cast<const uint4*>(row + (size_t)t * p.ldr + x.col)
                                      : make_uint4(0u, 0u, 0u, 0u);
    };
    if constexpr (VEC) {
#pragma unroll
      for (int i = 0; i < GR; ++i) raw[i] = request(t0 + i);
      if constexpr (KM > 0) {
#pragma unroll
        for (int i = 0; i < HB; ++i) before[i] = request(t0 - 1 - i);
      }
    }
    if constexpr (VEC && KM > 0) {
#pragma unroll
      for (int j = 0; j < KM; ++j) {
        wt[j] = make_uint4(0u, 0u, 0u, 0u);
        if (any && j < p.taps) wt[j] = *reinterpret_cast<const uint4*>(w + (size_t)(p.taps - 1 - j) * C);
      }
    }
    if (!ready) {                                          // uniform over the CTA
      if (tid < TT) tok[tid] = token_of(p, t0 + tid);
      __syncthreads();
      for (int i = tid; i < TT * p.pairs; i += blockDim.x) {
        const int k = i / p.pairs;
        float sn, cs;
        sincosf((float)tok[k].pos * p.inv_freq[i - k * p.pairs], &sn, &cs);
        turn[i] = make_float2(cs * p.rot_mult, sn * p.rot_mult);
      }
      __syncthreads();
      ready = true;
    }
    if (vec >= vecs) continue;
    // input of position pos - back for the token with info k in row t
    auto input = [&](const Token& k, int t, int back, float (&u)[V]) {
      const int pos = k.pos - back;
      if (pos >= 0 && t - back >= k.qs) {
        load<E, V, VEC>(row + (size_t)(t - back) * p.ldr + x.col, x.e0, x.e1, u);
      } else if (pos >= 0 && k.state >= 0) {
        load<E, V, VEC>(ring + ((size_t)k.state * p.taps + pos % p.taps) * C + x.ch, x.e0, x.e1, u);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = 0.f;
      }
    };
    auto unpack = [&](const uint4& r, float (&u)[V]) {
      const E* e = reinterpret_cast<const E*>(&r);
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] = to_f(e[j]);
    };
    float hist[HB][V];                                     // hist[j]: input of j + 1 positions before
    if constexpr (VEC && KM > 0) {
#pragma unroll
      for (int j = 0; j < HB; ++j) unpack(before[j], hist[j]);
    }
#pragma unroll 1
    for (int g0 = 0; g0 < TT && t0 + g0 < p.T; g0 += GR) {
      if constexpr (VEC) {
        if (g0 > 0) {
#pragma unroll
          for (int i = 0; i < GR; ++i) raw[i] = request(t0 + g0 + i);
        }
      }
#pragma unroll
    for (int gi = 0; gi < GR; ++gi) {
      const int i = g0 + gi, t = t0 + i;
      if (t >= p.T) break;
      const Token k = tok[i];
      float y[V], u[V];
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = u[e] = 0.f;
      if (any && k.len > 0) {
        if constexpr (VEC) unpack(raw[gi], u);
        else load<E, V, VEC>(row + (size_t)t * p.ldr + x.col, x.e0, x.e1, u);
        if constexpr (VEC && KM > 0) {
          if (t - k.qs < KM - 1 && (i == 0 || t == k.qs)) {       // the window reaches back in front of the portion
#pragma unroll
            for (int j = 0; j < KM - 1; ++j)
              if (j + 1 < p.taps && t - j - 1 < k.qs) input(k, t, j + 1, hist[j]);
          }
#pragma unroll
          for (int j = KM - 2; j >= 0; --j) {
            float g[V];
            unpack(wt[j + 1], g);
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = fmaf(g[e], hist[j][e], y[e]);
          }
          float g[V];
          unpack(wt[0], g);
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = fmaf(g[e], u[e], y[e]);
#pragma unroll
          for (int j = KM - 2; j > 0; --j)
#pragma unroll
            for (int e = 0; e < V; ++e) hist[j][e] = hist[j - 1][e];
#pragma unroll
          for (int e = 0; e < V; ++e) hist[0][e] = u[e];
        } else {
          for (int j = p.taps - 1; j >= 0; --j) {
            float z[V], g[V];
            input(k, t, j, z);
            load<E, V, VEC>(w + (size_t)(p.taps - 1 - j) * C, x.e0, x.e1, g);
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = fmaf(g[e], z[e], y[e]);
          }
        }
        if (k.len == 1 && k.state >= 0)
          store<E, V, VEC>(ring + ((size_t)k.state * p.taps + k.pos % p.taps) * C + x.ch, u, x.e0, x.e1);
        if (x.rotated) {
          const int first = x.d0 % p.dim;                  // (of one map: heads with two are rotated in even maps only)
#pragma unroll
          for (int e = 0; e < V; e += 2) {
            // a pair never straddles two maps or the end of the rotated part, both are even
            int f = first + e;
            if (f >= p.dim) f = (x.d0 + e) % p.dim;
            if (e + 1 < x.e1 && e >= x.e0 && f < 2 * p.pairs && f + 1 < p.dim) {
              const float2 cs = turn[i * p.pairs + (f >> 1)];
              const float a = y[e], b = y[e + 1];
              y[e] = a * cs.x - b * cs.y;
              y[e + 1] = b * cs.x + a * cs.y;
            }
          }
        }
      }
      if (x.hh < nq) {
        store<E, V, VEC>(reinterpret_cast<E*>(p.q_out) + ((size_t)t * nq + x.hh) * p.D + x.d0, y);
      } else if (k.slot >= 0 && k.slot < p.num_slots) {
        const long long blk = k.slot / p.block_size;
        const int off = (int)(k.slot - blk * p.block_size);
        store<E, V, VEC>(reinterpret_cast<E*>(p.cache) +
                             ((size_t)(blk * 2 * p.G + x.hh - nq) * p.block_size + off) * p.D + x.d0, y);
      }
    }
    }
  }
}

// The last inputs of every portion from request `first` on.  grid (channels / 256, requests)
template <typename E>
__global__ void ring_kernel(const Params p, int first) {
  const int r = first + blockIdx.y, qs = p.qsl[r], len = p.qsl[r + 1] - qs, slot = p.state_slots[r];
  const int cq = p.H * p.maps * p.dim, ck = p.G * p.maps * p.dim, C = cq + ck + p.G * p.vdim;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (len <= 0 || slot < 0 || c >= C) return;
  const int col = c < cq ? p.q_off + c : (c < cq + ck ? p.k_off + c - cq : p.v_off + c - cq - ck);
  const int end = p.seq_lens[r], start = end - len;
  for (int pos = max(start, end - p.taps); pos < end; ++pos)
    reinterpret_cast<E*>(p.ring)[((size_t)slot * p.taps + pos % p.taps) * C + c] =
        reinterpret_cast<const E*>(p.row)[(size_t)(qs + pos - start) * p.ldr + col];
}

// Launched in stream order, without programmatic overlap with the kernels around them.
template <typename E, int V, bool VEC, int KM, int TT>
static int launch_conv(const Params& p, cudaStream_t stream) {
  const int vecs = (p.H * p.maps + 2 * p.G) * (p.D / V), threads = vecs < 256 ? (vecs + 31) / 32 * 32 : 256;
  const int runs = (p.T + TT - 1) / TT, most = (vecs + threads - 1) / threads;
  int parts = (4 * 148 + runs - 1) / runs;                 // enough CTAs for every SM, else one over all vectors
  parts = parts > most ? most : parts;
  conv_cache_kernel<E, V, VEC, KM, TT><<<dim3(runs, parts), threads, (size_t)TT * p.pairs * sizeof(float2), stream>>>(p);
  B200_CUDA_CHECK(cudaGetLastError());
  return 0;
}

template <typename E>
static int launch(const Params& p, int ring_from, int only_ring, int single, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(E);
  if (!only_ring) {
    const uintptr_t a = (uintptr_t)p.row | (uintptr_t)p.w | (uintptr_t)p.q_out | (uintptr_t)p.cache | (uintptr_t)p.ring;
    const int v = p.G ? (p.k_off | p.v_off | p.vdim) : 0;
    const bool vec = a % 16 == 0 && (p.ldr | p.q_off | p.dim | p.D | v) % V == 0;
    int rc;
    if (!vec) rc = launch_conv<E, 2, false, 0, 4>(p, stream);
    else if (p.taps > 4) rc = launch_conv<E, V, true, 0, 4>(p, stream);
    else if (single) rc = launch_conv<E, V, true, 4, 1>(p, stream);
    else rc = launch_conv<E, V, true, 4, 16>(p, stream);
    if (rc) return rc;
  }
  if (ring_from < p.R && p.taps > 1) {
    const int C = p.H * p.maps * p.dim + p.G * (p.maps * p.dim + p.vdim);
    ring_kernel<E><<<dim3((C + 255) / 256, p.R - ring_from), 256, 0, stream>>>(p, ring_from);
    B200_CUDA_CHECK(cudaGetLastError());
  }
  return 0;
}

// ------------------------------------------------------------------------------------------- behind the softmax
struct CombineParams {
  const void *a, *gate;
  const float* lam;
  void* out;
  int heads, D, vdim, ldg;             // heads of the output
  float diff, eps;
  long long rows;                      // tokens * heads
};

// One warp per token and head, at most NV vectors per lane.
template <typename E, int V, bool VEC, int NV>
__global__ void __launch_bounds__(256) combine_kernel(const CombineParams p) {
  const long long n = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (n >= p.rows) return;
  const long long t = n / p.heads;
  const int h = (int)(n - t * p.heads);
  const E* a = reinterpret_cast<const E*>(p.a) + (size_t)n * (p.lam != nullptr ? 2 : 1) * p.D;
  float o[NV][V], ss = 0.f;
  const float lam = p.lam != nullptr ? *p.lam : 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (lane + 32 * i) * V;
    if (d >= p.D) break;
    load<E, V, VEC>(a + d, 0, p.D - d, o[i]);
    if (p.lam != nullptr) {
      float b[V];
      load<E, V, VEC>(a + p.D + d, 0, p.D - d, b);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        o[i][e] -= lam * b[e];
        if (d + e < p.vdim) ss += o[i][e] * o[i][e];
      }
    }
  }
  float sc = 1.f;
  if (p.lam != nullptr) sc = (1.f - p.diff) / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (lane + 32 * i) * V;
    if (d >= p.D) break;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      float v = o[i][e] * sc;
      if (p.gate != nullptr && d + e < p.vdim) {
        const float g = to_f(reinterpret_cast<const E*>(p.gate)[(size_t)t * p.ldg + h * p.vdim + d + e]);
        v *= 1.f / (1.f + expf(-g));
      }
      o[i][e] = v;
    }
    store<E, V, VEC>(reinterpret_cast<E*>(p.out) + (size_t)n * p.D + d, o[i], 0, p.D - d);
  }
}

template <typename E>
static int launch_combine(const CombineParams& p, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(E);
  const dim3 grid((unsigned)((p.rows + 7) / 8)), block(256);
  const bool vec = ((uintptr_t)p.a | (uintptr_t)p.out) % 16 == 0 && p.D % V == 0;
  if (vec && p.D <= 32 * V) combine_kernel<E, V, true, 1><<<grid, block, 0, stream>>>(p);
  else if (vec && p.D <= 128 * V) combine_kernel<E, V, true, 4><<<grid, block, 0, stream>>>(p);
  else combine_kernel<E, 2, false, 8><<<grid, block, 0, stream>>>(p);
  B200_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace cc
}  // namespace b200

// row: columns q_off, k_off, v_off of the packed projection; w [taps, channels]; ring [slots, taps, channels]; cache
// [blocks, 2, G, block_size, D] (G 0: none); elem: 2 = bf16, 4 = fp32 (all alike).  Requests from ring_from on may have
// portions of several tokens; single: every request has one token; only_ring: nothing but the rings advances.
extern "C" int b200_conv_cache(const void* row, int ldr, int q_off, int k_off, int v_off, const void* w, int taps,
                               void* ring, const float* inv_freq, int pairs, float rot_mult, void* q_out, void* cache,
                               const int* slots, const int* qsl, const int* seq_lens, const int* state_slots, int T, int R,
                               int H, int G, int dim, int vdim, int maps, int D, int block_size, long long num_blocks,
                               int ring_from, int single, int only_ring, int elem, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0 || R <= 0) return 0;
  if (taps < 1 || maps < 1 || maps * dim > D || (G > 0 && vdim > D) || D % 2 || 2 * pairs > dim || pairs > 512 ||
      (maps > 1 && pairs > 0 && dim % 2)) {
    b200_set_last_error("conv_cache: at least one tap, heads no wider than the cache's, rotated part no wider than a head",
                        __FILE__, __LINE__);
    return -1;
  }
  cc::Params p{row, w, q_out, cache, ring, inv_freq, slots, qsl, seq_lens, state_slots, ldr, q_off, k_off, v_off, H, G, dim,
               vdim, maps, D, taps, pairs, block_size, T, R, num_blocks * block_size, rot_mult};
  return elem == 4 ? cc::launch<float>(p, ring_from, only_ring, single, stream)
                   : cc::launch<__nv_bfloat16>(p, ring_from, only_ring, single, stream);
}

// a [T, heads * (lam ? 2 : 1), D] -> out [T, heads, D] (may be a without lam); gate [T, >= heads * vdim] or null.
extern "C" int b200_combine_heads(const void* a, const void* gate, int ldg, const float* lam, void* out, int T, int heads,
                                  int D, int vdim, float diff, float eps, int elem, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0 || heads <= 0) return 0;
  if (D > 512 || vdim > D || D % 2) {
    b200_set_last_error("combine_heads: heads of at most 512 columns", __FILE__, __LINE__);
    return -1;
  }
  cc::CombineParams p{a, gate, lam, out, heads, D, vdim, ldg, diff, eps, (long long)T * heads};
  return elem == 4 ? cc::launch_combine<float>(p, stream) : cc::launch_combine<__nv_bfloat16>(p, stream);
}
