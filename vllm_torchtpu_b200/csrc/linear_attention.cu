// Linear attention with a carried state per request and head (S is [dk, dv], fp32), four rules:
//
//   FIXED, decay per head:       S <- decay_h S + k v^T
//   CHANNEL, decay per channel:  S <- g S (rows) + k v^T
//   DELTA, decay per channel:    S <- g S (rows);  u = beta (v - S^T k);  S <- S + k u^T
//   REMOVAL, decay and rate per channel, both on the old state:  S <- g S + b (S^T n)^T + k v^T,  n = k / |k|, b = -a * n
//
//   o = S^T q;   y = o / rms(o) [* norm] * act(gate)
//
// q, k, v are columns of a packed projection, optionally behind a causal short convolution with silu, a rotation of
// half-split pairs and unit length.  Decays, step sizes, norms, angles and the state are fp32 throughout.
//
// State pools are indexed by the request's slot.  The convolution's inputs live in a ring of `taps` rows (the input of
// position p in row p % taps): the row that a single token writes is none of those it reads.  A request whose first
// token of the step has position 0 starts from zeros.
//
// Kernels:
//  * lin_step_kernel: one CTA per (head, request), token by token, everything fused (convolution to gate).  The state
//    is held on chip, so a decoded token reads and writes it once.  Decoding, and prompts in 32-bit.
//  * prompts in bf16, chunks of 16 tokens:
//      lin_chunk_kernel (parallel over chunks): with G_i the decays accumulated up to token i of the chunk (log2),
//        A_ij = beta_i sum_c k_ic k_jc 2^(G_ic - G_jc) (i > j),  Q_ij the same with q_i and i >= j;
//        (I + A) U = beta v,  (I + A) W = beta k 2^G  by forward substitution;  q' = q 2^G,  k' = k 2^(G_last - G).
//        Decay factors only ever appear as 2^(difference <= 0).
//        REMOVAL, where M_i = S_(i-1)^T n_i:  with e_i = n_i / (decay of token i), a factor of at most 2 (exp(exp(-1/2))),
//        A_ij = sum_c e_ic a_jc n_jc 2^(G_ic - G_jc),  (I + A) M0 = (the same with k_j in place of a_j n_j) V,
//        (I + A) W = e 2^G;  Q_ij as above with b_j, K_ij with k_j;  b' = b 2^(G_last - G).
//      lin_scan_kernel (sequential over chunks, one warp per 16 value columns, no exchange between warps):
//        U' = U - W S,  O = q' S + Q U',  S <- 2^G_last S + k'^T U'
//        (REMOVAL: M = M0 + W S,  O = q' S + Q M + K V,  S <- 2^G_last S + b'^T M + k'^T V).
//        The warp keeps S^T as mma accumulators: they are at the same time the A operand of the two products with S
//        (the contraction index is permuted alike in the B operand), and U'^T comes out in the layout that the update
//        and Q U' take.  Every operand is a pair of tf32 numbers (three products), fp32 accumulation and state.
//      lin_finish_kernel: norm and gate.
//    The scratch of a slab of chunks is read back from the L2; the products of the next slab overlap the scan of this one.
#include <cstring>

#include "common.cuh"

namespace b200 {
namespace lin {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float silu(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float sigmoid(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
// the same from one exponential and one logarithm; ln(1 + e) by its series where 1 + e would drop digits
__device__ __forceinline__ float softplus_fast(float v) {
  const float e = __expf(-fabsf(v));
  const float s = e < 0.0156f ? e * fmaf(e, fmaf(e, 0.33333333f, -0.5f), 1.f) : __logf(1.f + e);
  return fmaxf(v, 0.f) + s;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// x = hi + lo, hi a tf32 number and lo what it leaves out: products of such pairs on the tf32 tensor path, lo * lo
// dropped, keep 21 bits of the operands
struct Split {
  uint32_t hi, lo;
};
__device__ __forceinline__ Split split(float v) {
  Split s;
  s.hi = __float_as_uint(v) & 0xffffe000u;
  s.lo = __float_as_uint(v - __uint_as_float(s.hi));
  return s;
}
__device__ __forceinline__ void mma_tf32(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct SplitA {
  uint32_t hi[4], lo[4];
};
// an accumulator tile (C layout) as the A operand of a product over its columns; see lin_scan_kernel
__device__ __forceinline__ SplitA split_tile(const float* c) {
  SplitA a;
  const Split x0 = split(c[0]), x1 = split(c[2]), x2 = split(c[1]), x3 = split(c[3]);
  a.hi[0] = x0.hi; a.hi[1] = x1.hi; a.hi[2] = x2.hi; a.hi[3] = x3.hi;
  a.lo[0] = x0.lo; a.lo[1] = x1.lo; a.lo[2] = x2.lo; a.lo[3] = x3.lo;
  return a;
}
// c += a b, the small terms into c2 (may be c)
__device__ __forceinline__ void mma_split(float* c, float* c2, const SplitA& a, float b0, float b1) {
  const Split x = split(b0), y = split(b1);
  mma_tf32(c, a.hi, x.hi, y.hi);
  mma_tf32(c2, a.lo, x.hi, y.hi);
  mma_tf32(c2, a.hi, x.lo, y.lo);
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}

constexpr int C = 16;                 // tokens per chunk
constexpr float UNIT_EPS = 1e-6f;
constexpr float LOG2E = 1.4426950408889634f;
constexpr int AQ_LD = 24;             // row stride of Q in the scratch
constexpr float REMOVAL_DECAY = 0.6065306597126334f;      // exp(-1/2): decays are exp(-exp(-1/2) sigmoid(z))

enum Rule { FIXED = 0, DELTA = 1, CHANNEL = 2, REMOVAL = 3 };

struct Params {
  const void *row, *a, *gate, *conv_w;
  void *ring, *y;
  float* state;
  const float *inv_freq, *decay, *A_log, *dt_bias, *rate_bias, *norm_w;
  const int *qsl, *seq_lens, *slots;
  int ldr, q_off, k_off, v_off, beta_off, lda, ldg, taps, pairs, unit, gate_silu;
  int T, H, Hk, dk, dv, req_begin, zero_rows, rate_off, ldy, norm_stride;
  float eps, q_mult, k_mult, inv_tau;
  // ---- chunked prompts
  float *qd, *w, *kd, *bd, *u, *v, *aq, *ak, *gl, *o;
  int dkp, dvp, slab, chunk_begin;
};

struct Req {
  int qs, len, start, slot;           // first row, rows, position of the first, state slot
};
__device__ __forceinline__ Req request(const Params& p, int r) {
  Req q;
  q.qs = p.qsl[r];
  q.len = p.qsl[r + 1] - q.qs;
  q.start = p.seq_lens[r] - q.len;
  q.slot = p.slots[r];
  return q;
}
// column of channel c (q | k | v) in the packed row
__device__ __forceinline__ int column(const Params& p, int c) {
  const int n = p.Hk * p.dk;
  return c < n ? p.q_off + c : (c < 2 * n ? p.k_off + c - n : p.v_off + c - 2 * n);
}
// input of channel c at position pos > start - taps (zero in front of the sequence): from this step's rows or from the
// ring, without a branch, so that several of these loads are in flight together
template <typename E>
__device__ __forceinline__ float input_at(const Params& p, const Req& q, int pos, int c, int col) {
  const int ch = 2 * p.Hk * p.dk + p.H * p.dv, m = pos % p.taps;
  const E* x = reinterpret_cast<const E*>(p.row) + (size_t)(q.qs + max(pos - q.start, 0)) * p.ldr + col;
  const E* y = reinterpret_cast<const E*>(p.ring) + ((size_t)q.slot * p.taps + (m < 0 ? m + p.taps : m)) * ch + c;
  const float v = to_f(*(pos >= q.start ? x : y));
  return pos < 0 ? 0.f : v;
}
// convolution and silu of channel c at position pos; KM: taps it is unrolled for (0: any number)
template <typename E, int KM>
__device__ __forceinline__ float conv_at(const Params& p, const Req& q, int pos, int c, int col) {
  const E* w = reinterpret_cast<const E*>(p.conv_w) + (size_t)c * p.taps;
  float v = 0.f;
  if constexpr (KM == 0) {
    for (int j = 0; j < p.taps; ++j) v = fmaf(to_f(w[j]), input_at<E>(p, q, pos - p.taps + 1 + j, c, col), v);
  } else {
    float x[KM], k[KM];
#pragma unroll
    for (int j = 0; j < KM; ++j) {
      const int back = min(KM - 1 - j, p.taps - 1);
      k[j] = to_f(w[p.taps - 1 - back]);
      x[j] = input_at<E>(p, q, pos - back, c, col);
    }
#pragma unroll
    for (int j = 0; j < KM; ++j)
      if (KM - 1 - j < p.taps) v = fmaf(k[j], x[j], v);
  }
  return silu(v);
}

// ------------------------------------------------------------------------------------------- token by token
// Thread (row group rg, column group cg) owns columns VEC * cg .. of rows rg, rg + RG, ... of the state.
// Between the reads of a token they are in shared memory, where a CTA's whole state arrives by asynchronous copies while
// q, k, v are prepared (SMEM), in registers, at most RPT rows (REGS), or nowhere: the pool is read twice (POOL).
enum Hold { POOL, REGS, SMEM };
template <typename E, int RULE, int VEC, int RPT, Hold HOLD>
__global__ void __launch_bounds__(HOLD == POOL ? 1024 : (HOLD == REGS ? 512 : 256), HOLD == SMEM ? 3 : 1)
lin_step_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  __shared__ float sc[4];
  constexpr bool MEM = RULE == DELTA || RULE == REMOVAL;     // the state is read along the key before it is written
  const int h = blockIdx.x, r = p.req_begin + blockIdx.y, tid = threadIdx.x, NT = blockDim.x;
  const Req q = request(p, r);
  if (q.len <= 0 || q.slot < 0) {
    if (p.zero_rows && r < p.T)
      for (int j = tid; j < p.dv; j += NT) put(reinterpret_cast<E*>(p.y) + (size_t)r * p.ldy + h * p.dv + j, 0.f);
    return;
  }
  const int dk = p.dk, dv = p.dv, n = p.Hk * dk, group = p.H / p.Hk, hk = h / group;
  const int ncg = dv / VEC, RG = NT / ncg, cg = tid % ncg, rg = tid / ncg;
  const bool act = rg < RG;
  float* sq = sm;                       // [dk]
  float* sk = sq + dk;                  // [dk]
  float* sg = sk + dk;                  // [dk]
  float* sa = sg + dk;                  // [dk] (REMOVAL: rates)
  float* sv = RULE == REMOVAL ? sa + dk : sa;               // [dv]
  float* su = sv + dv;                  // [dv]: what is added along k; REMOVAL: S^T n
  float* pm = su + dv;                  // [RG][dv]
  float* po = pm + RG * dv;             // [RG][dv]
  float* st = p.state + ((size_t)q.slot * p.H + h) * dk * dv + VEC * cg;
  const bool fresh = q.start == 0;
  const int rows = act ? (dk - rg + RG - 1) / RG : 0;
  auto load_row = [&](int i, float (&s)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 f = *reinterpret_cast<const float4*>(st + (size_t)i * dv);
      s[0] = f.x; s[1] = f.y; s[2] = f.z; s[3] = f.w;
    } else {
      s[0] = st[(size_t)i * dv];
    }
  };
  auto store_row = [&](int i, const float (&s)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(st + (size_t)i * dv) = make_float4(s[0], s[1], s[2], s[3]);
    else st[(size_t)i * dv] = s[0];
  };
  float* held = po + RG * dv + VEC * cg;      // SMEM: [dk][dv]
  if constexpr (HOLD == SMEM) {
    for (int x = 0; x < rows; ++x) {
      float* d = held + (size_t)(rg + x * RG) * dv;
      if (fresh) *reinterpret_cast<float4*>(d) = make_float4(0.f, 0.f, 0.f, 0.f);
      else cp_async16(smem_u32(d), st + (size_t)(rg + x * RG) * dv);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  float S[HOLD == REGS ? RPT : 1][VEC];
  if constexpr (HOLD == REGS) {
#pragma unroll
    for (int x = 0; x < RPT; ++x) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[x][e] = 0.f;
      if (!fresh && x < rows) load_row(rg + x * RG, S[x]);
    }
  }
  const float a_log = RULE == DELTA ? expf(p.A_log[h]) : 0.f;
  const float decay = RULE == FIXED ? p.decay[h] : 0.f;
  const float* norm_w = p.norm_w != nullptr ? p.norm_w + (size_t)h * p.norm_stride : nullptr;
  for (int t = q.qs; t < q.qs + q.len; ++t) {
    const int pos = q.start + t - q.qs;
    // needed late, loaded early: step size, output gate and norm weight of this thread's first value column
    const float b_raw = RULE == DELTA ? to_f(reinterpret_cast<const E*>(p.row)[(size_t)t * p.ldr + p.beta_off + h]) : 0.f;
    float g_raw = 0.f, nw = 1.f;
    if (tid < dv) {
      g_raw = to_f(reinterpret_cast<const E*>(p.gate)[(size_t)t * p.ldg + h * dv + tid]);
      if (norm_w != nullptr) nw = norm_w[tid];
    }
    for (int x = tid; x < 2 * dk + dv; x += NT) {
      const int c = x < dk ? hk * dk + x : (x < 2 * dk ? n + hk * dk + x - dk : 2 * n + h * dv + x - 2 * dk);
      const int col = column(p, c);
      float v;
      if (p.taps > 0) {
        v = p.taps <= 4 ? conv_at<E, 4>(p, q, pos, c, col) : conv_at<E, 0>(p, q, pos, c, col);
        // a single token enters the ring here; longer portions once all of their readers are done
        if (q.len == 1 && (x >= 2 * dk || h % group == 0))
          reinterpret_cast<E*>(p.ring)[((size_t)q.slot * p.taps + pos % p.taps) * (2 * n + p.H * dv) + c] =
              reinterpret_cast<const E*>(p.row)[(size_t)t * p.ldr + col];
      } else {
        v = to_f(reinterpret_cast<const E*>(p.row)[(size_t)t * p.ldr + col]);
      }
      if (x < dk) sq[x] = v;
      else if (x < 2 * dk) sk[x - dk] = v;
      else sv[x - 2 * dk] = v;
    }
    if constexpr (RULE != FIXED) {
      for (int i = tid; i < dk; i += NT) {
        const float z = to_f(reinterpret_cast<const E*>(p.a)[(size_t)t * p.lda + h * dk + i]) + p.dt_bias[h * dk + i];
        if constexpr (RULE == DELTA) sg[i] = expf(-a_log * softplus(z));
        if constexpr (RULE == CHANNEL) sg[i] = expf(-softplus(-z) * p.inv_tau);
        if constexpr (RULE == REMOVAL) {
          sg[i] = expf(-REMOVAL_DECAY * sigmoid(z));
          sa[i] = sigmoid(to_f(reinterpret_cast<const E*>(p.row)[(size_t)t * p.ldr + p.rate_off + h * dk + i]) +
                          p.rate_bias[h * dk + i]);
        }
      }
    }
    __syncthreads();
    if (p.pairs > 0) {
      for (int i = tid; i < 2 * p.pairs; i += NT) {
        const int f = i < p.pairs ? i : i - p.pairs;
        float* x = i < p.pairs ? sq : sk;
        float sn, cs;
        sincosf((float)pos * p.inv_freq[f], &sn, &cs);
        const float a = x[f], b = x[f + p.pairs];
        x[f] = a * cs - b * sn;
        x[f + p.pairs] = b * cs + a * sn;
      }
      __syncthreads();
    }
    if (tid < (RULE == REMOVAL ? 128 : 96)) {
      const int wq = tid >> 5, lane = tid & 31;
      const float* x = wq == 1 ? sk : sq;
      const float* y = wq == 0 ? sq : sk;
      float s = 0.f;
      for (int i = lane; i < dk; i += 32) s += x[i] * y[i] * (wq == 3 ? sa[i] : 1.f);
      s = warp_sum(s);
      if (lane == 0) sc[wq] = s;
    }
    __syncthreads();
    const float iq = p.q_mult * (p.unit ? 1.f / sqrtf(sc[0] + UNIT_EPS) : 1.f);
    const float ik = p.k_mult * (p.unit ? 1.f / sqrtf(sc[1] + UNIT_EPS) : 1.f);
    const float qk = sc[2] * iq * ik;
    const float in = RULE == REMOVAL ? 1.f / sqrtf(sc[1] + UNIT_EPS) : 0.f;       // n = k * in (before k_mult)
    const float qb = RULE == REMOVAL ? -sc[3] * iq * in : 0.f;
    float mem[VEC], os[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) mem[e] = os[e] = 0.f;
    const bool zero = HOLD == POOL && fresh && t == q.qs;
    auto pass = [&](int i, float (&s)[VEC]) {
      const float g = RULE == FIXED ? decay : sg[i], kk = sk[i] * (RULE == REMOVAL ? in : ik), qq = sq[i] * iq;
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (RULE == REMOVAL) mem[e] = fmaf(kk, s[e], mem[e]);
        s[e] *= g;
        if (RULE == DELTA) mem[e] = fmaf(kk, s[e], mem[e]);
        os[e] = fmaf(qq, s[e], os[e]);
      }
    };
    if constexpr (HOLD == REGS) {
#pragma unroll
      for (int x = 0; x < RPT; ++x)
        if (x < rows) pass(rg + x * RG, S[x]);
    } else if constexpr (HOLD == SMEM) {
      asm volatile("cp.async.wait_all;" ::: "memory");      // a thread copies and reads its own elements only
#pragma unroll 4
      for (int x = 0; x < rows; ++x) {
        const float4 f = *reinterpret_cast<const float4*>(held + (size_t)(rg + x * RG) * dv);
        float s[4] = {f.x, f.y, f.z, f.w};
        pass(rg + x * RG, reinterpret_cast<float(&)[VEC]>(s));
      }
    } else if (!zero) {
      for (int x = 0; x < rows; ++x) {
        float s[VEC];
        load_row(rg + x * RG, s);
        pass(rg + x * RG, s);
      }
    }
    if (act) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (MEM) pm[rg * dv + VEC * cg + e] = mem[e];
        po[rg * dv + VEC * cg + e] = os[e];
      }
    }
    __syncthreads();
    const float beta = RULE == DELTA ? sigmoid(b_raw) : 1.f;
    float ss = 0.f;
    for (int j = tid; j < dv; j += NT) {
      float m = 0.f, o = 0.f;
      for (int x = 0; x < RG; ++x) {
        if (MEM) m += pm[x * dv + j];
        o += po[x * dv + j];
      }
      const float u = RULE == DELTA ? beta * (sv[j] - m) : sv[j];
      o = fmaf(qk, u, o);
      if (RULE == REMOVAL) o = fmaf(qb, m, o);
      su[j] = RULE == REMOVAL ? m : u;
      po[j] = o;                        // (row group 0; only this thread reads column j)
      ss += o * o;
    }
    ss = block_sum(ss, red);            // also orders su for the update
    const float inv = 1.f / sqrtf(ss / (float)dv + p.eps);
    for (int j = tid; j < dv; j += NT) {
      float v = po[j] * inv, g = g_raw;
      if (j == tid) {
        v *= nw;
      } else {
        if (norm_w != nullptr) v *= norm_w[j];
        g = to_f(reinterpret_cast<const E*>(p.gate)[(size_t)t * p.ldg + h * dv + j]);
      }
      v *= p.gate_silu ? silu(g) : sigmoid(g);
      put(reinterpret_cast<E*>(p.y) + (size_t)t * p.ldy + h * dv + j, v);
    }
    float u[VEC], m[VEC];                // REMOVAL: value and -S^T n, otherwise what is added along k
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      u[e] = act ? (RULE == REMOVAL ? sv : su)[VEC * cg + e] : 0.f;
      m[e] = RULE == REMOVAL && act ? -su[VEC * cg + e] : 0.f;
    }
    // row i of the new state from the decayed old one
    auto write = [&](int i, float (&s)[VEC]) {
      const float kk = sk[i] * ik, an = RULE == REMOVAL ? sa[i] * sk[i] * in : 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        s[e] = fmaf(kk, u[e], s[e]);
        if (RULE == REMOVAL) s[e] = fmaf(an, m[e], s[e]);
      }
    };
    if constexpr (HOLD == SMEM) {
      const bool last = t + 1 == q.qs + q.len;
#pragma unroll 4
      for (int x = 0; x < rows; ++x) {
        const int i = rg + x * RG;
        const float g = RULE == FIXED ? decay : sg[i];
        float4* d = reinterpret_cast<float4*>(held + (size_t)i * dv);
        const float4 f = *d;
        float s[4] = {f.x * g, f.y * g, f.z * g, f.w * g};
        write(i, reinterpret_cast<float(&)[VEC]>(s));
        const float4 n4 = make_float4(s[0], s[1], s[2], s[3]);
        if (last) *reinterpret_cast<float4*>(st + (size_t)i * dv) = n4;
        else *d = n4;
      }
    } else if constexpr (HOLD == REGS) {
#pragma unroll
      for (int x = 0; x < RPT; ++x)
        if (x < rows) write(rg + x * RG, S[x]);
    } else {
      for (int x = 0; x < rows; ++x) {
        const int i = rg + x * RG;
        const float g = RULE == FIXED ? decay : sg[i];
        float s[VEC];
        if (zero) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) s[e] = 0.f;
        } else {
          load_row(i, s);
#pragma unroll
          for (int e = 0; e < VEC; ++e) s[e] *= g;
        }
        write(i, s);
        store_row(i, s);
      }
    }
    __syncthreads();                    // before the next token's q, k, v
  }
  if constexpr (HOLD == REGS) {
#pragma unroll
    for (int x = 0; x < RPT; ++x)
      if (x < rows) store_row(rg + x * RG, S[x]);
  }
}

// The last inputs of a prompt's portion, once the convolutions have run.  grid (channels / 256, requests)
template <typename E>
__global__ void lin_ring_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  const Req q = request(p, p.req_begin + blockIdx.y);
  const int ch = 2 * p.Hk * p.dk + p.H * p.dv, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (q.len <= 0 || q.slot < 0 || c >= ch) return;
  const int col = column(p, c), end = q.start + q.len;
  for (int pos = max(q.start, end - p.taps); pos < end; ++pos)
    reinterpret_cast<E*>(p.ring)[((size_t)q.slot * p.taps + pos % p.taps) * ch + c] =
        reinterpret_cast<const E*>(p.row)[(size_t)(q.qs + pos - q.start) * p.ldr + col];
}

// ------------------------------------------------------------------------------------------- chunks of 16 tokens
typedef __nv_bfloat16 bf16;

// The 16 values of channel c in a chunk that begins at position pos0 (n of them exist; zeros behind).  KM: taps the
// window is unrolled for (0: no convolution).
template <int KM>
__device__ __forceinline__ void chunk_column(const Params& p, const Req& q, int pos0, int n, int c, float (&v)[C]) {
  const int col = column(p, c), t0 = pos0 - q.start;
  // rows of this step, in one batch of loads; rows outside the chunk's window are clamped and dropped below
  const bf16* row = reinterpret_cast<const bf16*>(p.row) + (size_t)q.qs * p.ldr + col;
  if constexpr (KM == 0) {
    if (n == C) {
      const bf16* x = row + (size_t)t0 * p.ldr;
#pragma unroll
      for (int i = 0; i < C; ++i, x += p.ldr) v[i] = to_f(*x);
    } else {
#pragma unroll
      for (int i = 0; i < C; ++i) v[i] = to_f(row[(size_t)(t0 + min(i, n - 1)) * p.ldr]);
#pragma unroll
      for (int i = 0; i < C; ++i) v[i] = i < n ? v[i] : 0.f;
    }
  } else {
    float x[C + KM - 1], w[KM];
    const bf16* wp = reinterpret_cast<const bf16*>(p.conv_w) + (size_t)c * p.taps;
#pragma unroll
    for (int j = 0; j < KM; ++j) w[j] = to_f(wp[max(0, j - (KM - p.taps))]);
    if (n == C && t0 > 0) {
      const bf16* y = row + (size_t)(t0 - (KM - 1)) * p.ldr;
#pragma unroll
      for (int m = 0; m < C + KM - 1; ++m, y += p.ldr) x[m] = to_f(*y);
    } else {
#pragma unroll
      for (int m = 0; m < C + KM - 1; ++m)
        x[m] = to_f(row[(size_t)max(0, t0 + min(m - (KM - 1), n - 1)) * p.ldr]);
    }
#pragma unroll
    for (int j = 0; j < KM; ++j)
      if (j < KM - p.taps) w[j] = 0.f;
    if (t0 == 0) {                       // the portion's first chunk looks back into the ring
#pragma unroll
      for (int m = 0; m < KM - 1; ++m)
        x[m] = m - (KM - 1) > -p.taps ? input_at<bf16>(p, q, pos0 + m - (KM - 1), c, col) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < C; ++i) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < KM; ++j) s = fmaf(w[j], x[i + j], s);
      v[i] = i < n ? __fdividef(s, 1.f + __expf(-s)) : 0.f;
    }
  }
}

// grid (requests * slab, H), 256 threads
template <int RULE, int KM, int DKP>
__global__ void __launch_bounds__(256, RULE == REMOVAL ? 2 : 3) lin_chunk_kernel(const Params p) {
  constexpr int dkp = DKP, ds = DKP + 4;
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  __shared__ float beta[C], power[C + 1];
  __shared__ __align__(16) float sa[C][C + 4];
  __shared__ __align__(16) float sx[RULE == REMOVAL ? C : 1][C + 4];       // REMOVAL: A with k_j, and |k| of every token
  __shared__ float len[C];
  const int slot = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const Req q = request(p, p.req_begin + slot / p.slab);
  const int t0 = (p.chunk_begin + slot % p.slab) * C, n = min(C, q.len - t0);
  if (n <= 0 || q.slot < 0) return;
  const int pos0 = q.start + t0, row0 = q.qs + t0;
  const int dk = p.dk, dv = p.dv, nk = p.Hk * dk, hk = h / (p.H / p.Hk);
  float* sq = sm;                       // [C][ds]
  float* sk = sq + C * ds;
  float* sg = sk + C * ds;              // decays accumulated from the chunk's first token on, log2 (per channel)
  float* se = sg + C * ds;              // REMOVAL: n over the decay of its own token
  float* sr = se + C * ds;              // REMOVAL: rates
  // ---- q, k and the accumulated decays
#pragma unroll 1
  for (int x = tid; x < 2 * dkp; x += 256) {
    const int i0 = x < dkp ? x : x - dkp;
    float v[C];
    if (i0 < dk) {
      chunk_column<KM>(p, q, pos0, n, (x < dkp ? 0 : nk) + hk * dk + i0, v);
    } else {
#pragma unroll
      for (int i = 0; i < C; ++i) v[i] = 0.f;
    }
    float* d = x < dkp ? sq : sk;
#pragma unroll
    for (int i = 0; i < C; ++i) d[i * ds + i0] = v[i];
  }
  if constexpr (RULE != FIXED) {
    const float a_log = RULE == DELTA ? expf(p.A_log[h]) * LOG2E : (RULE == CHANNEL ? p.inv_tau : REMOVAL_DECAY) * LOG2E;
#pragma unroll 1
    for (int c = tid; c < dkp; c += 256) {
      float g = 0.f;
      const int cc = min(c, dk - 1);
      const float b = p.dt_bias[h * dk + cc];
      const bf16* a = reinterpret_cast<const bf16*>(p.a) + (size_t)row0 * p.lda + h * dk + cc;
      float z[C];
#pragma unroll
      for (int i = 0; i < C; ++i) z[i] = to_f(a[(size_t)min(i, n - 1) * p.lda]);
#pragma unroll
      for (int i = 0; i < C; ++i) {
        // a factor below 2^-64 leaves nothing of the state in fp32: the sum keeps its digits
        if (c < dk && i < n) {
          const float x = z[i] + b;
          const float step = RULE == REMOVAL ? __fdividef(1.f, 1.f + __expf(-x)) : softplus_fast(RULE == DELTA ? x : -x);
          g -= fminf(a_log * step, 64.f);
          if constexpr (RULE == REMOVAL) se[i * ds + c] = ex2(a_log * step);
        } else if constexpr (RULE == REMOVAL) {
          se[i * ds + c] = 0.f;
        }
        sg[i * ds + c] = g;
      }
      if constexpr (RULE == REMOVAL) {
        const float rb = p.rate_bias[h * dk + cc];
        const bf16* rr = reinterpret_cast<const bf16*>(p.row) + (size_t)row0 * p.ldr + p.rate_off + h * dk + cc;
#pragma unroll
        for (int i = 0; i < C; ++i) z[i] = to_f(rr[(size_t)min(i, n - 1) * p.ldr]);
#pragma unroll
        for (int i = 0; i < C; ++i) sr[i * ds + c] = c < dk && i < n ? __fdividef(1.f, 1.f + __expf(-(z[i] + rb))) : 0.f;
      }
    }
    if (RULE == DELTA && tid < C)
      beta[tid] = tid < n ? sigmoid(to_f(reinterpret_cast<const bf16*>(p.row)[(size_t)(row0 + tid) * p.ldr + p.beta_off + h]))
                          : 0.f;
  }
  __syncthreads();
  if (p.pairs > 0) {
#pragma unroll 1
    for (int x = tid; x < C * p.pairs; x += 256) {
      const int i = x / p.pairs, f = x - i * p.pairs;
      float sn, cs;
      sincosf((float)(pos0 + i) * p.inv_freq[f], &sn, &cs);
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        float* d = (s ? sk : sq) + i * ds + f;
        const float a = d[0], b = d[p.pairs];
        d[0] = a * cs - b * sn;
        d[p.pairs] = b * cs + a * sn;
      }
    }
    __syncthreads();
  }
  {
    const int warp = tid >> 5, lane = tid & 31;
    for (int x = warp; x < 2 * C; x += 8) {
      float* d = (x < C ? sq : sk) + (x & (C - 1)) * ds;
      float m = x < C ? p.q_mult : p.k_mult;
      if (p.unit) {
        float s = 0.f;
        for (int i = lane; i < dk; i += 32) s += d[i] * d[i];
        m /= sqrtf(warp_sum(s) + UNIT_EPS);
      }
      if (RULE == REMOVAL && x >= C) {   // k becomes n, its length is kept; e = n over the token's decay
        float s = 0.f;
        for (int i = lane; i < dk; i += 32) s += d[i] * d[i];
        const float l = sqrtf(warp_sum(s) + UNIT_EPS);
        if (lane == 0) len[x - C] = l * m;
        m = 1.f / l;
        for (int i = lane; i < dk; i += 32) se[(x - C) * ds + i] *= d[i] * m;
      }
      for (int i = lane; i < dk; i += 32) d[i] *= m;
    }
    if (RULE == FIXED && tid <= C) power[tid] = exp2f(fmaxf(log2f(p.decay[h]), -64.f) * (float)tid);
  }
  __syncthreads();
  const size_t unit = (size_t)slot * p.H + h;
  // ---- products of the tokens of the chunk
  {
    // thread -> pair (i, j <= i): rows r and 15 - r of the triangle are 17 pairs together
    int i = 0, j = C;
    if (tid < 8 * 17) {
      const int r = tid / 17, x = tid - 17 * r;
      i = x <= r ? r : 15 - r;
      j = x <= r ? x : x - r - 1;
    } else if (tid - 8 * 17 < 120) {     // pairs above the diagonal: zeros
      const int y = tid - 8 * 17, r = y / 15, x = y - 15 * r;
      i = x < 15 - r ? r : 15 - r;
      j = x < 15 - r ? r + 1 + x : x + 1;
    }
    if (tid < 8 * 17) {
      float qk = 0.f, kk = 0.f, qb = 0.f, kb = 0.f;
      const float *qi = sq + i * ds, *ki = sk + i * ds, *kj = sk + j * ds, *gi = sg + i * ds, *gj = sg + j * ds;
      for (int c = 0; c < dkp; c += 4) {
        const float4 a = *reinterpret_cast<const float4*>(qi + c), b = *reinterpret_cast<const float4*>(kj + c);
        if constexpr (RULE == REMOVAL) {
          const float4 e = *reinterpret_cast<const float4*>(se + i * ds + c), r = *reinterpret_cast<const float4*>(sr + j * ds + c),
                       x = *reinterpret_cast<const float4*>(gi + c), y = *reinterpret_cast<const float4*>(gj + c);
          const float d0 = b.x * ex2(x.x - y.x), d1 = b.y * ex2(x.y - y.y), d2 = b.z * ex2(x.z - y.z),
                      d3 = b.w * ex2(x.w - y.w);
          const float f0 = d0 * r.x, f1 = d1 * r.y, f2 = d2 * r.z, f3 = d3 * r.w;
          qk = fmaf(a.x, d0, qk); qk = fmaf(a.y, d1, qk); qk = fmaf(a.z, d2, qk); qk = fmaf(a.w, d3, qk);
          kk = fmaf(e.x, d0, kk); kk = fmaf(e.y, d1, kk); kk = fmaf(e.z, d2, kk); kk = fmaf(e.w, d3, kk);
          qb = fmaf(a.x, f0, qb); qb = fmaf(a.y, f1, qb); qb = fmaf(a.z, f2, qb); qb = fmaf(a.w, f3, qb);
          kb = fmaf(e.x, f0, kb); kb = fmaf(e.y, f1, kb); kb = fmaf(e.z, f2, kb); kb = fmaf(e.w, f3, kb);
        } else if constexpr (RULE == CHANNEL) {
          const float4 x = *reinterpret_cast<const float4*>(gi + c), y = *reinterpret_cast<const float4*>(gj + c);
          qk = fmaf(a.x, b.x * ex2(x.x - y.x), qk); qk = fmaf(a.y, b.y * ex2(x.y - y.y), qk);
          qk = fmaf(a.z, b.z * ex2(x.z - y.z), qk); qk = fmaf(a.w, b.w * ex2(x.w - y.w), qk);
        } else if constexpr (RULE == DELTA) {
          const float4 e = *reinterpret_cast<const float4*>(ki + c), x = *reinterpret_cast<const float4*>(gi + c),
                       y = *reinterpret_cast<const float4*>(gj + c);
          const float d0 = b.x * ex2(x.x - y.x), d1 = b.y * ex2(x.y - y.y), d2 = b.z * ex2(x.z - y.z),
                      d3 = b.w * ex2(x.w - y.w);
          qk = fmaf(a.x, d0, qk); qk = fmaf(a.y, d1, qk); qk = fmaf(a.z, d2, qk); qk = fmaf(a.w, d3, qk);
          kk = fmaf(e.x, d0, kk); kk = fmaf(e.y, d1, kk); kk = fmaf(e.z, d2, kk); kk = fmaf(e.w, d3, kk);
        } else {
          qk = fmaf(a.x, b.x, qk); qk = fmaf(a.y, b.y, qk); qk = fmaf(a.z, b.z, qk); qk = fmaf(a.w, b.w, qk);
        }
      }
      if constexpr (RULE == FIXED) qk *= power[i - j];
      if constexpr (RULE == REMOVAL) {
        p.aq[(unit * C + i) * AQ_LD + j] = -qb;
        p.ak[(unit * C + i) * AQ_LD + j] = qk * len[j];
        sa[i][j] = j < i ? kb : 0.f;
        sx[i][j] = j < i ? kk * len[j] : 0.f;
      } else {
        p.aq[(unit * C + i) * AQ_LD + j] = qk;
      }
      if constexpr (RULE == DELTA) sa[i][j] = j < i ? beta[i] * kk : 0.f;
    } else if (j < C) {
      p.aq[(unit * C + i) * AQ_LD + j] = 0.f;
      if constexpr (RULE == REMOVAL) p.ak[(unit * C + i) * AQ_LD + j] = 0.f;
    }
  }
  if constexpr (RULE == DELTA || RULE == REMOVAL) __syncthreads();
  // ---- columns of W and U (forward substitution), q', k', last decay
#pragma unroll 1
  for (int x = tid; x < dkp + p.dvp; x += 256) {
    float v[C];
    asm volatile("" ::: "memory");       // values that do not depend on the column stay in shared memory
    if (x < dkp) {
      float *qd = p.qd + unit * C * (dkp + 8) + x, *kd = p.kd + unit * C * (dkp + 4) + x;
      if constexpr (RULE != FIXED) {
        const float last = sg[(C - 1) * ds + x];
#pragma unroll
        for (int i = 0; i < C; ++i) {
          const float g = sg[i * ds + x], e = ex2(g), k = sk[i * ds + x], left = ex2(last - g);
          qd[i * (dkp + 8)] = sq[i * ds + x] * e;
          if constexpr (RULE == REMOVAL) {
            kd[i * (dkp + 4)] = k * len[i] * left;
            p.bd[unit * C * (dkp + 4) + x + i * (dkp + 4)] = -(k * sr[i * ds + x]) * left;
            v[i] = se[i * ds + x] * e;
          } else {
            kd[i * (dkp + 4)] = k * left;
          }
          if constexpr (RULE == DELTA) v[i] = beta[i] * k * e;
        }
        p.gl[unit * dkp + x] = ex2(last);
      } else {
#pragma unroll
        for (int i = 0; i < C; ++i) {
          qd[i * (dkp + 8)] = sq[i * ds + x] * power[i + 1];
          kd[i * (dkp + 4)] = sk[i * ds + x] * power[max(n - 1 - i, 0)];      // k is zero from token n on
        }
        p.gl[unit * dkp + x] = power[n];
      }
    } else {
      const int j = x - dkp;
      if (j < dv) {
        chunk_column<KM>(p, q, pos0, n, 2 * nk + h * dv + j, v);
      } else {
#pragma unroll
        for (int i = 0; i < C; ++i) v[i] = 0.f;
      }
      if constexpr (RULE == DELTA) {
#pragma unroll
        for (int i = 0; i < C; ++i) v[i] *= beta[i];
      }
      if constexpr (RULE == REMOVAL) {   // the values go to the scan as they are; M0 starts from their products with A
        float* d = p.v + (unit * (p.dvp / 64) + j / 64) * C * 64 + j % 64;
#pragma unroll
        for (int i = 0; i < C; ++i) d[i * 64] = v[i];
#pragma unroll
        for (int i = C - 1; i >= 0; --i) {
          asm volatile("" ::: "memory");
          float s = 0.f;
#pragma unroll
          for (int l = 0; l < i; l += 4) {
            const float4 a = *reinterpret_cast<const float4*>(&sx[RULE == REMOVAL ? i : 0][l]);      // zeros from column i on
            s = fmaf(a.x, v[l], s);
            if (l + 1 < i) s = fmaf(a.y, v[l + 1], s);
            if (l + 2 < i) s = fmaf(a.z, v[l + 2], s);
            if (l + 3 < i) s = fmaf(a.w, v[l + 3], s);
          }
          v[i] = s;
        }
      }
    }
    if constexpr (RULE == DELTA || RULE == REMOVAL) {
#pragma unroll
      for (int i = 1; i < C; ++i) {
        asm volatile("" ::: "memory");   // one row of A in registers at a time
#pragma unroll
        for (int j = 0; j < i; j += 4) {
          const float4 a = *reinterpret_cast<const float4*>(&sa[i][j]);      // zeros from column i on
          v[i] = fmaf(-a.x, v[j], v[i]);
          if (j + 1 < i) v[i] = fmaf(-a.y, v[j + 1], v[i]);
          if (j + 2 < i) v[i] = fmaf(-a.z, v[j + 2], v[i]);
          if (j + 3 < i) v[i] = fmaf(-a.w, v[j + 3], v[i]);
        }
      }
      if (x < dkp) {
        float* w = p.w + unit * C * (dkp + 8) + x;
#pragma unroll
        for (int i = 0; i < C; ++i) w[i * (dkp + 8)] = RULE == REMOVAL ? v[i] : -v[i];
      }
    }
    if (x >= dkp) {
      const int j = x - dkp;             // [dvp / 64][C][64]: a CTA of the scan reads one block
      float* u = p.u + (unit * (p.dvp / 64) + j / 64) * C * 64 + j % 64;
#pragma unroll
      for (int i = 0; i < C; ++i) u[i * 64] = v[i];
    }
  }
}

// grid (H * dvp / 64, requests), 128 threads: warp w owns value columns 16 w .. 16 w + 15 of the CTA's 64
template <int RULE, int NT>
struct Scan {
  static constexpr bool MEM = RULE == DELTA || RULE == REMOVAL, TWO = RULE == REMOVAL;
  static constexpr int DKP = 8 * NT, U_LD = 68;
  static constexpr int QD = 0, W = C * (DKP + 8), KD = W + (MEM ? C * (DKP + 8) : 0), BD = KD + C * (DKP + 4);
  static constexpr int U = BD + (TWO ? C * (DKP + 4) : 0), V = U + C * U_LD, AQ = V + (TWO ? C * U_LD : 0);
  static constexpr int AK = AQ + C * AQ_LD, GL = AK + (TWO ? C * AQ_LD : 0), WORDS = GL + DKP;
  static constexpr int STAGES = 3 * WORDS * 4 > 220 * 1024 ? 2 : 3;
  static constexpr int BYTES = STAGES * WORDS * 4;
};

template <int RULE, int NT>
__global__ void __launch_bounds__(128) lin_scan_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  using L = Scan<RULE, NT>;
  constexpr bool MEM = L::MEM, TWO = L::TWO;
  constexpr int DKP = L::DKP;
  extern __shared__ __align__(16) float sm[];
  const int splits = p.dvp / 64, h = blockIdx.x / splits, col0 = (blockIdx.x % splits) * 64;
  const Req q = request(p, p.req_begin + blockIdx.y);
  const int chunks = min(p.slab, (q.len + C - 1) / C - p.chunk_begin);
  if (chunks <= 0 || q.slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int dk = p.dk, dv = p.dv;
  const uint32_t base = smem_u32(sm);
  auto issue = [&](int c, int stage) {
    const size_t unit = ((size_t)blockIdx.y * p.slab + c) * p.H + h;
    const uint32_t d = base + stage * L::WORDS * 4;
    auto copy = [&](int word, const float* src, int words) {
      for (int i = tid * 4; i < words; i += 128 * 4) cp_async16(d + (word + i) * 4, src + i);
    };
    copy(L::QD, p.qd + unit * C * (DKP + 8), C * (DKP + 8));
    if constexpr (MEM) copy(L::W, p.w + unit * C * (DKP + 8), C * (DKP + 8));
    copy(L::KD, p.kd + unit * C * (DKP + 4), C * (DKP + 4));
    copy(L::AQ, p.aq + unit * C * AQ_LD, C * AQ_LD);
    if constexpr (TWO) {
      copy(L::BD, p.bd + unit * C * (DKP + 4), C * (DKP + 4));
      copy(L::AK, p.ak + unit * C * AQ_LD, C * AQ_LD);
    }
    copy(L::GL, p.gl + unit * DKP, DKP);
#pragma unroll
    for (int i = tid; i < C * 16; i += 128) {
      const int r = i >> 4, s = (i & 15) * 4;
      cp_async16(d + (L::U + r * L::U_LD + s) * 4, p.u + ((unit * splits + col0 / 64) * C + r) * 64 + s);
      if constexpr (TWO) cp_async16(d + (L::V + r * L::U_LD + s) * 4, p.v + ((unit * splits + col0 / 64) * C + r) * 64 + s);
    }
  };
  float* st = p.state + ((size_t)q.slot * p.H + h) * dk * dv;
  const int j0 = col0 + warp * 16 + g, j1 = j0 + 8;          // value columns of this thread
  const bool fresh = q.start == 0 && p.chunk_begin == 0;
  float S[NT][4];
#pragma unroll
  for (int x = 0; x < NT; ++x) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = 8 * x + 2 * t + (e & 1), j = e < 2 ? j0 : j1;
      S[x][e] = (!fresh && i < dk && j < dv) ? st[(size_t)i * dv + j] : 0.f;
    }
  }
#pragma unroll
  for (int s = 0; s < L::STAGES - 1; ++s) {
    if (s < chunks) issue(s, s);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  for (int c = 0; c < chunks; ++c) {
    asm volatile("cp.async.wait_group %0;" ::"n"(L::STAGES - 2) : "memory");
    __syncthreads();
    if (c + L::STAGES - 1 < chunks) issue(c + L::STAGES - 1, (c + L::STAGES - 1) % L::STAGES);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float* b = sm + (c % L::STAGES) * L::WORDS;
    float U[2][4], O[2][4];              // transposed: rows value columns, columns tokens 8 x + 2 t, + 1
    float U2[2][4], O2[2][4];            // small terms
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const float* u = b + L::U + (8 * x + 2 * t) * L::U_LD + warp * 16 + g;
      U[x][0] = u[0]; U[x][1] = u[L::U_LD]; U[x][2] = u[8]; U[x][3] = u[L::U_LD + 8];
#pragma unroll
      for (int e = 0; e < 4; ++e) O[x][e] = O2[x][e] = U2[x][e] = 0.f;
    }
    const float* qd = b + L::QD + g * (DKP + 8) + 2 * t;
    const float* w = b + L::W + g * (DKP + 8) + 2 * t;
#pragma unroll
    for (int x = 0; x < NT; ++x) {
      const SplitA a = split_tile(S[x]);
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        if constexpr (MEM) {
          const float2 bw = *reinterpret_cast<const float2*>(w + 8 * y * (DKP + 8) + 8 * x);
          mma_split(U[y], U2[y], a, bw.x, bw.y);
        }
        const float2 bq = *reinterpret_cast<const float2*>(qd + 8 * y * (DKP + 8) + 8 * x);
        mma_split(O[y], O2[y], a, bq.x, bq.y);
      }
    }
    SplitA ua[2], va[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
#pragma unroll
      for (int e = 0; e < 4; ++e) U[x][e] += U2[x][e];
      ua[x] = split_tile(U[x]);
      if constexpr (TWO) {
        const float* v = b + L::V + (8 * x + 2 * t) * L::U_LD + warp * 16 + g;
        const float f[4] = {v[0], v[L::U_LD], v[8], v[L::U_LD + 8]};
        va[x] = split_tile(f);
      }
    }
#pragma unroll
    for (int y = 0; y < 2; ++y) {
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        if (x > y) continue;             // Q is lower triangular
        const float2 bq = *reinterpret_cast<const float2*>(b + L::AQ + (8 * y + g) * AQ_LD + 8 * x + 2 * t);
        mma_split(O[y], O2[y], ua[x], bq.x, bq.y);
        if constexpr (TWO) {
          const float2 bk = *reinterpret_cast<const float2*>(b + L::AK + (8 * y + g) * AQ_LD + 8 * x + 2 * t);
          mma_split(O[y], O2[y], va[x], bk.x, bk.y);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) O[y][e] += O2[y][e];
    }
    const float* kd = b + L::KD + 2 * t * (DKP + 4) + g;
    const float* gl = b + L::GL + 2 * t;
#pragma unroll
    for (int x = 0; x < NT; ++x) {
      const float2 e = *reinterpret_cast<const float2*>(gl + 8 * x);
      S[x][0] *= e.x; S[x][1] *= e.y; S[x][2] *= e.x; S[x][3] *= e.y;
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const float* k = kd + 8 * y * (DKP + 4) + 8 * x;
        if constexpr (TWO) {
          const float* m = k + (L::BD - L::KD);
          mma_split(S[x], S[x], va[y], k[0], k[DKP + 4]);
          mma_split(S[x], S[x], ua[y], m[0], m[DKP + 4]);
        } else {
          mma_split(S[x], S[x], ua[y], k[0], k[DKP + 4]);
        }
      }
    }
    const int rows = min(C, q.len - (p.chunk_begin + c) * C);
    float* o = p.o + ((((size_t)blockIdx.y * p.slab + c) * C) * p.H + h) * dv;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = 8 * x + 2 * t + (e & 1), j = e < 2 ? j0 : j1;
        if (i < rows && j < dv) o[(size_t)i * p.H * dv + j] = O[x][e];
      }
    }
  }
#pragma unroll
  for (int x = 0; x < NT; ++x) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = 8 * x + 2 * t + (e & 1), j = e < 2 ? j0 : j1;
      if (i < dk && j < dv) st[(size_t)i * dv + j] = S[x][e];
    }
  }
}

// One warp per (token of the slab, head).
__global__ void __launch_bounds__(256) lin_finish_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  const int idx = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const Req q = request(p, p.req_begin + idx / (p.slab * C));
  const int i = p.chunk_begin * C + idx % (p.slab * C);
  if (i >= q.len || q.slot < 0) return;
  const int dv = p.dv;
  const float* o = p.o + ((size_t)idx * p.H + h) * dv;
  float ss = 0.f;
  for (int j = lane; j < dv; j += 32) ss += o[j] * o[j];
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
  const size_t t = q.qs + i;
  const bf16* gate = reinterpret_cast<const bf16*>(p.gate) + t * p.ldg + h * dv;
  bf16* y = reinterpret_cast<bf16*>(p.y) + t * p.ldy + h * dv;
  for (int j = lane; j < dv; j += 32) {
    float v = o[j] * inv;
    if (p.norm_w != nullptr) v *= p.norm_w[(size_t)h * p.norm_stride + j];
    const float g = to_f(gate[j]);
    put(y + j, v * (p.gate_silu ? silu(g) : sigmoid(g)));
  }
}

// ------------------------------------------------------------------------------------------- host
template <typename E, int RULE, int VEC, int RPT, Hold HOLD>
static int launch_step_as(const Params& p, int R, int threads, cudaStream_t stream) {
  const int RG = threads / (p.dv / VEC);
  const int smem = ((RULE == REMOVAL ? 4 : 3) * p.dk + 2 * p.dv + 2 * RG * p.dv + (HOLD == SMEM ? p.dk * p.dv : 0)) * (int)sizeof(float);
  static unsigned long long seen = 0;
  if (smem > 46 * 1024)
    B200_CUDA_CHECK(ensure_dynamic_smem(lin_step_kernel<E, RULE, VEC, RPT, HOLD>, 220 * 1024, &seen));
  B200_CUDA_CHECK(launch_pdl(lin_step_kernel<E, RULE, VEC, RPT, HOLD>, dim3(p.H, R), dim3(threads), (size_t)smem,
                             stream, p));
  return 0;
}

template <typename E, int RULE, int VEC>
static int launch_step_v(const Params& p, int R, cudaStream_t stream) {
  const int ncg = p.dv / VEC;
  if constexpr (VEC == 4) {
    // q, k and the decays are read as floats: the state behind them starts on 16 bytes when 3 dk is a multiple of 4
    if (p.dk % 4 == 0 && ncg <= 256 && p.dk * p.dv <= 48 * 1024)
      return launch_step_as<E, RULE, VEC, 1, SMEM>(p, R, p.dk * p.dv <= 2048 && ncg <= 128 ? 128 : 256, stream);
  } else {
    for (int threads = 128; threads <= 512; threads *= 2) {
      if (threads < ncg) continue;
      const int RG = threads / ncg, rows = (p.dk + RG - 1) / RG;
      if (rows <= 4) return launch_step_as<E, RULE, VEC, 4, REGS>(p, R, threads, stream);
      if (rows <= 16) return launch_step_as<E, RULE, VEC, 16, REGS>(p, R, threads, stream);
    }
  }
  int threads = 512;
  while (threads < ncg) threads *= 2;
  if (threads > 1024) {
    b200_set_last_error("linear attention: at most 1024 value columns per thread group", __FILE__, __LINE__);
    return -1;
  }
  return launch_step_as<E, RULE, VEC, 1, POOL>(p, R, threads, stream);
}

template <typename E>
static int launch_step(const Params& p, int rule, int R, cudaStream_t stream) {
  const bool v4 = p.dv % 4 == 0;
  switch (rule) {
    case FIXED: return v4 ? launch_step_v<E, FIXED, 4>(p, R, stream) : launch_step_v<E, FIXED, 1>(p, R, stream);
    case DELTA: return v4 ? launch_step_v<E, DELTA, 4>(p, R, stream) : launch_step_v<E, DELTA, 1>(p, R, stream);
    case CHANNEL: return v4 ? launch_step_v<E, CHANNEL, 4>(p, R, stream) : launch_step_v<E, CHANNEL, 1>(p, R, stream);
    default: return v4 ? launch_step_v<E, REMOVAL, 4>(p, R, stream) : launch_step_v<E, REMOVAL, 1>(p, R, stream);
  }
}

template <int RULE, int NT>
static int launch_scan(const Params& p, int R, cudaStream_t stream) {
  static unsigned long long seen = 0;
  using L = Scan<RULE, NT>;
  B200_CUDA_CHECK(ensure_dynamic_smem(lin_scan_kernel<RULE, NT>, L::BYTES, &seen));
  B200_CUDA_CHECK(launch_pdl(lin_scan_kernel<RULE, NT>, dim3(p.H * (p.dvp / 64), R), dim3(128), (size_t)L::BYTES,
                             stream, p));
  return 0;
}

template <int RULE, int KM, int DKP>
static int launch_chunk_as(const Params& p, int R, cudaStream_t stream) {
  constexpr int smem = (RULE == REMOVAL ? 5 : (RULE == FIXED ? 2 : 3)) * C * (DKP + 4) * (int)sizeof(float);
  static unsigned long long seen = 0;
  if (smem > 44 * 1024) B200_CUDA_CHECK(ensure_dynamic_smem(lin_chunk_kernel<RULE, KM, DKP>, smem, &seen));
  B200_CUDA_CHECK(launch_pdl(lin_chunk_kernel<RULE, KM, DKP>, dim3(R * p.slab, p.H), dim3(256), (size_t)smem, stream, p));
  return 0;
}
template <int RULE, int KM>
static int launch_chunk(const Params& p, int R, cudaStream_t stream) {
  switch (p.dkp) {
    case 32: return launch_chunk_as<RULE, KM, 32>(p, R, stream);
    case 64: return launch_chunk_as<RULE, KM, 64>(p, R, stream);
    case 128: return launch_chunk_as<RULE, KM, 128>(p, R, stream);
    default: return launch_chunk_as<RULE, KM, 256>(p, R, stream);
  }
}

static int padded_dk(int dk) { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : 256)); }

// floats of scratch per chunk and head
static size_t chunk_words(int dk, int dv, int rule) {
  const int dkp = padded_dk(dk), dvp = (dv + 63) / 64 * 64, two = rule == REMOVAL ? 2 : 1;
  return (size_t)C * ((rule == DELTA || rule == REMOVAL ? 2 : 1) * (dkp + 8) + two * (dkp + 4 + dvp + AQ_LD) + dv) + dkp;
}

// one of the three kernels of a slab of chunks
template <int RULE>
static int launch_chunks(Params& p, int R, float* scratch, int mode, cudaStream_t stream) {
  const size_t units = (size_t)R * p.slab * p.H;
  p.qd = scratch;
  p.w = p.qd + units * C * (p.dkp + 8);
  constexpr bool mem = RULE == DELTA || RULE == REMOVAL, two = RULE == REMOVAL;
  p.kd = p.w + (mem ? units * C * (p.dkp + 8) : 0);
  p.bd = p.kd + units * C * (p.dkp + 4);
  p.u = p.bd + (two ? units * C * (p.dkp + 4) : 0);
  p.v = p.u + units * C * p.dvp;
  p.aq = p.v + (two ? units * C * p.dvp : 0);
  p.ak = p.aq + units * C * AQ_LD;
  p.gl = p.ak + (two ? units * C * AQ_LD : 0);
  p.o = p.gl + units * p.dkp;
  if (mode == 1)
    return p.taps == 0 ? launch_chunk<RULE, 0>(p, R, stream)
                       : (p.taps <= 4 && (RULE == FIXED || RULE == DELTA) ? launch_chunk<RULE, RULE < CHANNEL ? 4 : 8>(p, R, stream)
                                                                          : launch_chunk<RULE, 8>(p, R, stream));
  if (mode == 3) {
    switch (p.dkp) {
      case 32: return launch_scan<RULE, 4>(p, R, stream);
      case 64: return launch_scan<RULE, 8>(p, R, stream);
      case 128: return launch_scan<RULE, 16>(p, R, stream);
      default: return launch_scan<RULE, 32>(p, R, stream);
    }
  }
  B200_CUDA_CHECK(launch_pdl(lin_finish_kernel, dim3(R * p.slab * C, (p.H + 7) / 8), dim3(256), (size_t)0, stream, p));
  return 0;
}

}  // namespace lin
}  // namespace b200

// Bytes of scratch per (chunk of 16 tokens, head) of b200_linear_attention in mode 1.
extern "C" size_t b200_linear_attention_chunk_bytes(int dk, int dv, int rule) {
  return b200::lin::chunk_words(dk, dv, rule) * sizeof(float);
}

// Requests [req_begin, req_end) of the batch.  mode 0: token by token (any sizes; the ring takes portions of more than
// one token through mode 2); mode 1: products of chunks [chunk_begin, chunk_begin + slab) of every request (bf16, dk <=
// 256, taps <= 8; into scratch for (req_end - req_begin) * slab * H chunks), mode 3: their recurrence, mode 4: their
// norm and gate; mode 2: the ring of a prompt.  rule: 0 fixed decay per head (decay), 1 delta rule (a, A_log, dt_bias and
// the step sizes in column beta_off of the row), 2 decay per channel (a, dt_bias, tau), 3 removal (a, dt_bias, the rates in
// column rate_off with rate_bias).  norm_w: heads are norm_stride elements apart; y: rows are ldy apart.
// elem: 2 = bf16, 4 = fp32.
extern "C" int b200_linear_attention(int mode, int rule, const void* row, int ldr, int q_off, int k_off, int v_off,
                                     int beta_off, int rate_off, const void* a, int lda, const void* gate, int ldg,
                                     const void* conv_w, void* ring, int taps, const float* inv_freq, int pairs,
                                     const float* decay, const float* A_log, const float* dt_bias, const float* rate_bias,
                                     float tau, const float* norm_w, int norm_stride, float* state, void* y, int ldy,
                                     const int* qsl, const int* seq_lens, const int* slots, int req_begin, int req_end,
                                     int T, int H, int Hk, int dk, int dv, int unit, int gate_silu, float eps,
                                     float q_mult, float k_mult, int zero_rows, void* scratch, int chunk_begin, int slab,
                                     int elem, cudaStream_t stream) {
  using namespace b200;
  const int R = req_end - req_begin;
  if (R <= 0 || T <= 0) return 0;
  if (Hk <= 0 || H % Hk || 2 * pairs > dk || R > 65535 || dk <= 0 || dv <= 0) {
    b200_set_last_error("linear attention: heads must be a multiple of the q / k heads, pairs at most dk / 2", __FILE__,
                        __LINE__);
    return -1;
  }
  if (rule < 0 || rule > 3 || (rule == 0 && decay == nullptr) || (rule != 0 && (a == nullptr || dt_bias == nullptr)) ||
      (rule == 1 && A_log == nullptr) || (rule == 2 && !(tau > 0.f)) || (rule == 3 && (rate_bias == nullptr || unit))) {
    b200_set_last_error("linear attention: parameters of the rule are missing", __FILE__, __LINE__);
    return -1;
  }
  lin::Params p;
  memset(&p, 0, sizeof(p));
  p.row = row; p.a = a; p.gate = gate; p.conv_w = conv_w; p.ring = ring; p.y = y; p.state = state;
  p.inv_freq = inv_freq; p.decay = decay; p.A_log = A_log; p.dt_bias = dt_bias; p.norm_w = norm_w;
  p.qsl = qsl; p.seq_lens = seq_lens; p.slots = slots;
  p.ldr = ldr; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.beta_off = beta_off; p.lda = lda; p.ldg = ldg;
  p.taps = taps; p.pairs = pairs; p.unit = unit; p.gate_silu = gate_silu;
  p.T = T; p.H = H; p.Hk = Hk; p.dk = dk; p.dv = dv; p.req_begin = req_begin; p.zero_rows = zero_rows;
  p.eps = eps; p.q_mult = q_mult; p.k_mult = k_mult; p.inv_tau = rule == 2 ? 1.f / tau : 0.f;
  p.rate_off = rate_off; p.rate_bias = rate_bias; p.norm_stride = norm_stride; p.ldy = ldy;
  p.dkp = lin::padded_dk(dk); p.dvp = (dv + 63) / 64 * 64;
  p.slab = slab; p.chunk_begin = chunk_begin;
  if (mode == 0) return elem == 4 ? lin::launch_step<float>(p, rule, R, stream)
                                  : lin::launch_step<__nv_bfloat16>(p, rule, R, stream);
  if (mode == 1 || mode == 3 || mode == 4) {
    if (elem != 2 || dk > 256 || taps > 8 || slab <= 0 || scratch == nullptr) {
      b200_set_last_error("linear attention in chunks: bf16, dk of at most 256, at most 8 taps", __FILE__, __LINE__);
      return -1;
    }
    switch (rule) {
      case lin::FIXED: return lin::launch_chunks<lin::FIXED>(p, R, (float*)scratch, mode, stream);
      case lin::DELTA: return lin::launch_chunks<lin::DELTA>(p, R, (float*)scratch, mode, stream);
      case lin::CHANNEL: return lin::launch_chunks<lin::CHANNEL>(p, R, (float*)scratch, mode, stream);
      default: return lin::launch_chunks<lin::REMOVAL>(p, R, (float*)scratch, mode, stream);
    }
  }
  const dim3 grid((2 * Hk * dk + H * dv + 255) / 256, R);
  if (elem == 4) B200_CUDA_CHECK(launch_pdl(lin::lin_ring_kernel<float>, grid, dim3(256), (size_t)0, stream, p));
  else B200_CUDA_CHECK(launch_pdl(lin::lin_ring_kernel<__nv_bfloat16>, grid, dim3(256), (size_t)0, stream, p));
  return 0;
}
