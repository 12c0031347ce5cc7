// Attention layers with short convolutions: everything between the packed projection and the paged attention in one
// launch, and what follows the softmax of such layers.
//
//   y_t = sum_j w[j] u_(t - taps + 1 + j)     per channel of q, k and v (zeros in front of the sequence)
//   q, k: dimensions 2i, 2i + 1 of a head (of one map) turn by position * inv_freq[i], cos and sin times rot_mult
//   q times one number per head (q_scale, optional) -> q_out [T, heads * maps, D];   k, v -> page of the token's slot
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
  const float *inv_freq, *q_scale;
  const int *slots, *qsl, *seq_lens, *state_slots;
  int ldr, q_off, k_off, v_off, H, G, dim, vdim, maps, D, taps, pairs, block_size, T, R;
  long long num_slots;
  float rot_mult;
};

struct Token {
  int qs, len, pos, state;             // first row and length of its portion, position, state slot (-1: none)
  long long cell;                      // element of the cache where its first key head begins (-1: not cached)
};

// request of row t, by a whole warp: as many requests as end at t or before (qsl is monotone and repeats its last value
// behind the last request)
__device__ __forceinline__ Token token_of(const Params& p, int t, int lane) {
  int r = 0;
  for (int i = lane; i < p.R + lane; i += 32)
    r += __popc(__ballot_sync(0xffffffffu, i < p.R && p.qsl[min(i, p.R - 1) + 1] <= t));
  Token k{t, 0, 0, -1, -1};
  if (t >= p.T || r >= p.R) return k;
  k.qs = p.qsl[r];
  k.len = p.qsl[r + 1] - k.qs;
  k.pos = p.seq_lens[r] - k.len + t - k.qs;
  k.state = p.state_slots[r];
  const long long slot = p.slots[t];
  if (p.G > 0 && slot >= 0 && slot < p.num_slots) {
    const long long blk = slot / p.block_size;
    k.cell = (blk * 2 * p.G * p.block_size + slot - blk * p.block_size) * p.D;
  }
  return k;
}

// V elements as they lie in memory
template <int BYTES> struct Pack;
template <> struct Pack<16> { typedef uint4 type; };
template <> struct Pack<8> { typedef uint2 type; };
template <> struct Pack<4> { typedef uint32_t type; };
template <typename E, int V> using PackOf = typename Pack<V * sizeof(E)>::type;

template <typename E, int V, bool VEC>
__device__ __forceinline__ void load(const E* p, int e0, int e1, float (&v)[V]) {
  if constexpr (VEC) {
    const PackOf<E, V> u = *reinterpret_cast<const PackOf<E, V>*>(p);
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
    PackOf<E, V> u;
    E* e = reinterpret_cast<E*>(&u);
#pragma unroll
    for (int j = 0; j < V; ++j) put(e + j, v[j]);
    *reinterpret_cast<PackOf<E, V>*>(p) = u;
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j)
      if (j >= e0 && j < e1) put(p + j, v[j]);
  }
}

constexpr int THREADS = 128;

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

// grid (token runs of TT, parts of the vectors).  A run within one portion, as most are, takes the way with the window in
// registers (at most KM taps, 0: none do): the inputs of the next four tokens are on their way at any time, and the first
// ones are requested before the tokens' portion is known.  Other runs read every input where it lies.
template <typename E, int V, bool VEC, int KM, int TT>
__global__ void __launch_bounds__(THREADS, 4) conv_cache_kernel(const Params p) {
  extern __shared__ __align__(16) float2 turn[];          // [TT][pairs]
  __shared__ Token tok[TT];
  const int tid = threadIdx.x, t0 = blockIdx.x * TT;
  const int nq = p.H * p.maps, C = (nq + p.G * p.maps) * p.dim + p.G * p.vdim, vecs = (nq + 2 * p.G) * (p.D / V);
  const E* row = reinterpret_cast<const E*>(p.row);
  E* ring = reinterpret_cast<E*>(p.ring);
  constexpr int HB = KM > 1 ? KM - 1 : 1, GR = TT < 4 ? TT : 4;
  typedef PackOf<E, V> Raw;
  bool ready = false, whole = false;
  for (int v0 = blockIdx.y * THREADS; v0 < vecs; v0 += gridDim.y * THREADS) {
    const int vec = v0 + tid;
    const Where x = where_is<V>(p, min(vec, vecs - 1));
    const bool any = x.e0 < x.e1 && vec < vecs;
    const E* w = reinterpret_cast<const E*>(p.w) + x.ch;
    const E* col = row + x.col;
    Raw raw[GR];                                           // inputs of the next tokens
    float wt[KM > 0 ? KM : 1][V], hist[HB][V];             // weight of, and the input itself, j (+ 1) positions before
    auto request = [&](int t) { return any && t < p.T ? *reinterpret_cast<const Raw*>(col + (size_t)t * p.ldr) : Raw(); };
    auto unpack = [&](const Raw& r, float (&u)[V]) {
      const E* e = reinterpret_cast<const E*>(&r);
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] = to_f(e[j]);
    };
    if constexpr (VEC && KM > 0) {
#pragma unroll
      for (int i = 0; i < GR; ++i) raw[i] = request(t0 + i);
#pragma unroll
      for (int j = 0; j < KM; ++j)
        unpack(any && j < p.taps ? *reinterpret_cast<const Raw*>(w + (size_t)(p.taps - 1 - j) * C) : Raw(), wt[j]);
    }
    if (!ready) {                                          // uniform over the CTA
      for (int i = tid >> 5; i < TT; i += THREADS / 32) {
        const Token k = token_of(p, t0 + i, tid & 31);
        if ((tid & 31) == 0) tok[i] = k;
      }
      __syncthreads();
      for (int i = tid; i < TT * p.pairs; i += THREADS) {
        const int k = i / p.pairs;
        float sn, cs;
        sincosf((float)tok[k].pos * p.inv_freq[i - k * p.pairs], &sn, &cs);
        turn[i] = make_float2(cs * p.rot_mult, sn * p.rot_mult);
      }
      __syncthreads();
      ready = true;
      whole = tok[0].len > 0 && tok[TT - 1].len > 0 && tok[TT - 1].qs == tok[0].qs;
    }
    if (vec >= vecs) continue;
    const int first = x.d0 % p.dim;                        // index of element 0 within its map
    // input of position pos - back for the token with info k in row t
    auto input = [&](const Token& k, int t, int back, float (&u)[V]) {
      const int pos = k.pos - back;
      if (pos >= 0 && t - back >= k.qs) {
        load<E, V, VEC>(col + (size_t)(t - back) * p.ldr, x.e0, x.e1, u);
      } else if (pos >= 0 && k.state >= 0) {
        load<E, V, VEC>(ring + ((size_t)k.state * p.taps + pos % p.taps) * C + x.ch, x.e0, x.e1, u);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = 0.f;
      }
    };
    E* q_out = reinterpret_cast<E*>(p.q_out) + ((size_t)t0 * nq + x.hh) * p.D + x.d0;
    E* cache = reinterpret_cast<E*>(p.cache) + (size_t)(x.hh - nq) * p.block_size * p.D + x.d0;
    const size_t q_step = (size_t)nq * p.D;
    const bool is_q = x.hh < nq;
    const float scale = is_q && p.q_scale != nullptr ? p.q_scale[x.hh / p.maps] : 1.f;
    auto save = [&](int i, float (&y)[V]) {                // (a thread's rows of q are written in order)
      if (is_q) {
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] *= scale;
        store<E, V, VEC>(q_out, y);
        q_out += q_step;
      } else if (tok[i].cell >= 0) {
        store<E, V, VEC>(cache + tok[i].cell, y);
      }
    };
    if constexpr (VEC && KM > 0) {
      if (whole) {
        const int turns = x.rotated && any ? min(max(p.pairs - (first >> 1), 0), V / 2) : 0;   // pairs that rotate
        const Token k = tok[0];
#pragma unroll
        for (int j = 0; j < HB; ++j) {
          if (any && KM > 1 && j + 1 < p.taps) {
            input(k, t0, j + 1, hist[j]);
          } else {
#pragma unroll
            for (int e = 0; e < V; ++e) hist[j][e] = 0.f;
          }
        }
#pragma unroll 1
        for (int g0 = 0; g0 < TT; g0 += GR) {
          const E* ahead = col + (size_t)(t0 + g0 + GR) * p.ldr;
#pragma unroll
          for (int gi = 0; gi < GR; ++gi) {
            float u[V], y[V];
            unpack(raw[gi], u);
            if (TT > GR && any && g0 + GR < TT) raw[gi] = *reinterpret_cast<const Raw*>(ahead + (size_t)gi * p.ldr);
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = wt[0][e] * u[e];
#pragma unroll
            for (int j = 0; j < KM - 1; ++j)
#pragma unroll
              for (int e = 0; e < V; ++e) y[e] = fmaf(wt[j + 1][e], hist[j][e], y[e]);
#pragma unroll
            for (int j = KM - 2; j > 0; --j)
#pragma unroll
              for (int e = 0; e < V; ++e) hist[j][e] = hist[j - 1][e];
#pragma unroll
            for (int e = 0; e < V; ++e) hist[0][e] = u[e];
            if (TT == 1 && any && k.len == 1 && k.state >= 0)
              store<E, V, VEC>(ring + ((size_t)k.state * p.taps + k.pos % p.taps) * C + x.ch, u);
            if (turns > 0) {
              const float2* cs = turn + (g0 + gi) * p.pairs + (first >> 1);
#pragma unroll
              for (int e = 0; e < V; e += 2)
                if ((e >> 1) < turns) {
                  const float2 c = cs[e >> 1];
                  const float a = y[e], b = y[e + 1];
                  y[e] = a * c.x - b * c.y;
                  y[e + 1] = b * c.x + a * c.y;
                }
            }
            save(g0 + gi, y);
          }
        }
        continue;
      }
    }
#pragma unroll 1
    for (int i = 0; i < TT && t0 + i < p.T; ++i) {
      const Token k = tok[i];
      float y[V];
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = 0.f;
      if (any && k.len > 0) {
#pragma unroll 1
        for (int j = p.taps - 1; j >= 0; --j) {
          float z[V], g[V];
          input(k, t0 + i, j, z);
          load<E, V, VEC>(w + (size_t)(p.taps - 1 - j) * C, x.e0, x.e1, g);
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = fmaf(g[e], z[e], y[e]);
          if (j == 0 && k.len == 1 && k.state >= 0)
            store<E, V, VEC>(ring + ((size_t)k.state * p.taps + k.pos % p.taps) * C + x.ch, z, x.e0, x.e1);
        }
        if (x.rotated) {
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
      save(i, y);
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
  const int vecs = (p.H * p.maps + 2 * p.G) * (p.D / V), most = (vecs + THREADS - 1) / THREADS;
  const int runs = (p.T + TT - 1) / TT;
  int parts = 1;                                           // even shares of the vectors, enough CTAs for every SM
  while (parts < most && (most % parts || (long long)parts * runs < 12 * 148)) ++parts;
  conv_cache_kernel<E, V, VEC, KM, TT><<<dim3(runs, parts), THREADS, (size_t)TT * p.pairs * sizeof(float2), stream>>>(p);
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
                               void* ring, const float* inv_freq, int pairs, float rot_mult, const float* q_scale,
                               void* q_out, void* cache,
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
  cc::Params p{row, w, q_out, cache, ring, inv_freq, q_scale, slots, qsl, seq_lens, state_slots, ldr, q_off, k_off, v_off, H, G, dim,
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
