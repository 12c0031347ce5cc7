// Multi-head latent attention over the paged latent cache (absorbed-query form, MQA over one latent
// "head"), dense or sparse (top-k indexed), for decode, spec-verify, chunked prefill and mixed batches.
//
//   q_latent [T, H, Dq]  Dq = kv_lora + rope (576 for DeepSeek-V3), already multiplied by W_UK; a row may end
//                        in zero padding up to a multiple of 16 (in the cache as well)
//   cache    [blocks, block_size, Dq] bf16; the value of a row is its first L = kv_lora dims
//   out      [T, H, L]   rows behind the step's tokens are written as zeros
//
// One CTA per (token, group of 16 heads): all 16 rows of the MMA tile share the query position, so
// the causal limit and (sparse) the token's top-k list are uniform over the tile.  Prefill of models whose
// head count is no multiple of 16 tiles the (token, head) rows of a request as one list instead (`flat`):
// every row of a tile keeps its own causal limit and no MMA row is left empty.  KV rows stream
// in 16-row chunks through a 2-stage cp.async ring (rows are gathered by pointer, so the dense and
// the top-k case share the loop).  The four warps split the Dq contraction of Q K^T (partials summed
// through shared memory) and each owns a quarter of the L value columns for P V, which keeps the
// 16 x 512 fp32 output in registers.  bf16 mma.sync m16n8k16, fp32 online softmax in the log2 domain.
//
// Semantics of the reference's dense / sparse MLA kernels and latent cache write
// (reference: src/vllm_torchtpu/kernels/mla/v2/, kernels/mla/sparse/, layers/adapter/attention.py:2659-2879).
#include "common.cuh"

namespace b200 {
namespace mla {

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm volatile("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, const uint32_t* b) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
      "{%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp16(uint32_t smem, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem), "l"(g) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}

__device__ __forceinline__ void store2(__nv_bfloat16* d, float a, float b, bool c0, bool c1) {
  if (c0 && c1 && (reinterpret_cast<uintptr_t>(d) & 3) == 0) {
    *reinterpret_cast<uint32_t*>(d) = pack2(a, b);
  } else {
    if (c0) d[0] = __float2bfloat16(a);
    if (c1) d[1] = __float2bfloat16(b);
  }
}

constexpr int KS_MAX = 9;             // k-steps of 16 per warp: Dq <= 4 * 9 * 16 = 576

struct Params {
  const __nv_bfloat16* q;
  const __nv_bfloat16* cache;
  __nv_bfloat16* out;
  float* lse;
  const int* block_tables;
  const int* seq_lens;
  const int* qsl;
  const int* topk;                    // optional [T, topk_k] context positions, -1 = unused
  int topk_k, T, H, Dq, L, num_reqs, max_blocks, block_size;
  int flat;                           // 1: 16-row tiles over the (token, head) rows of a request
  long long num_blocks;
  float scale_log2;
  // split-KV: CTA (token, head group, split) covers an equal share of the token's 16-row chunks and writes a
  // normalised partial [splits, T, H, L] with its log-sum-exp [splits, T, H]; mla_merge_kernel combines them
  int splits;
  __nv_bfloat16* part_o;
  float* part_lse;
};

constexpr int NST = 3;                // cp.async stages of 16 cache rows

// LW = value columns per warp (L / 4).
template <int LW>
__global__ void __launch_bounds__(128) mla_attn_kernel(const Params p) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ const __nv_bfloat16* s_ptr[NST][16];
  __shared__ int s_pos[NST][16];      // position of the key, INT_MAX: not visible to any row
  __shared__ float s_part[4][16][17];
  pdl_launch_dependents();
  pdl_wait();
  const int groups = (p.H + 15) >> 4;
  const int sp = blockIdx.x % p.splits, tg = blockIdx.x / p.splits;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // the tile: rows_valid consecutive rows of the [T * H] query rows of request r, starting at row f0; qpos0 /
  // qpos1: positions of this thread's two rows, qpos: of the last row (which bounds the keys of the tile)
  int r, rows_valid, qpos, qpos0, qpos1, t = 0;
  size_t f0;
  if (p.flat) {
    int tile = tg;
    for (r = 0; r < p.num_reqs; ++r) {
      const int n = ((p.qsl[r + 1] - p.qsl[r]) * p.H + 15) >> 4;
      if (tile < n) break;
      tile -= n;
    }
    if (r == p.num_reqs) return;                                         // more CTAs than tiles
    const int qs = p.qsl[r], q_len = p.qsl[r + 1] - qs, kv_len = p.seq_lens[r];
    const int i0 = tile << 4;
    rows_valid = min(16, q_len * p.H - i0);
    f0 = (size_t)qs * p.H + i0;
    const int first = kv_len - q_len;
    qpos = first + (i0 + rows_valid - 1) / p.H;
    qpos0 = first + (i0 + (lane >> 2)) / p.H;
    qpos1 = first + (i0 + (lane >> 2) + 8) / p.H;
  } else {
    const int g = tg % groups;
    t = tg / groups;
    rows_valid = min(16, p.H - g * 16);
    f0 = (size_t)t * p.H + g * 16;
    // request of this token: largest r with qsl[r] <= t
    int lo = 0, hi = p.num_reqs;
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.qsl[mid] <= t) lo = mid; else hi = mid;
    }
    r = lo;
    const int qs = p.qsl[r], q_len = p.qsl[r + 1] - qs, kv_len = p.seq_lens[r];
    if (t >= p.qsl[p.num_reqs] || q_len <= 0 || kv_len <= 0) {           // padded token
      if (sp == 0) {
        for (int i = threadIdx.x; i < rows_valid * p.L; i += blockDim.x) p.out[f0 * p.L + i] = __float2bfloat16(0.f);
        if (p.lse && (int)threadIdx.x < rows_valid) p.lse[f0 + threadIdx.x] = -INFINITY;
      }
      if (p.splits > 1 && (int)threadIdx.x < rows_valid)
        p.part_lse[(size_t)sp * p.T * p.H + f0 + threadIdx.x] = -INFINITY;
      return;
    }
    qpos = qpos0 = qpos1 = kv_len - q_len + (t - qs);
  }
  const int n_kv = p.topk ? p.topk_k : qpos + 1;
  const int chunks_all = (n_kv + 15) >> 4;
  const int per_split = (chunks_all + p.splits - 1) / p.splits;
  const int chunk_lo = sp * per_split;
  const int chunks = max(0, min(chunks_all, chunk_lo + per_split) - chunk_lo);     // of this split
  const int ksteps = p.Dq >> 4;                    // Dq % 16 == 0
  const int nch = p.Dq >> 3;                       // 16-byte chunks per row
  const int RS = ((nch + 7) & ~7) << 4;            // row stride in shared memory (swizzle groups of 8)
  const int STAGE = 16 * RS;
  const uint32_t sbase = smem_u32(smem);

  // Q fragments of this warp's k-steps (ks = warp, warp + 4, ...)
  uint32_t qf[KS_MAX][4];
  {
    const int r0 = lane >> 2, r1 = r0 + 8, cb = 2 * (lane & 3);
    const __nv_bfloat16* q0 = r0 < rows_valid ? p.q + (f0 + r0) * p.Dq : nullptr;
    const __nv_bfloat16* q1 = r1 < rows_valid ? p.q + (f0 + r1) * p.Dq : nullptr;
#pragma unroll
    for (int i = 0; i < KS_MAX; ++i) {
      const int ks = warp + 4 * i;
      const bool in = ks < ksteps;
      qf[i][0] = (in && q0) ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + cb) : 0u;
      qf[i][1] = (in && q1) ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + cb) : 0u;
      qf[i][2] = (in && q0) ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 8 + cb) : 0u;
      qf[i][3] = (in && q1) ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 8 + cb) : 0u;
    }
  }
  const int* bt = p.block_tables + (size_t)r * p.max_blocks;

  auto prefetch = [&](int c, int stage) {
    if (threadIdx.x < 16) {
      const int i = ((chunk_lo + c) << 4) + threadIdx.x;
      int pos = -1;
      if (i < n_kv) pos = p.topk ? p.topk[(size_t)t * p.topk_k + i] : i;
      const bool ok = pos >= 0 && pos <= qpos;         // qpos < kv_len
      long long blk = 0;
      int off = 0;
      if (ok) {
        const int page = pos / p.block_size;
        blk = page < p.max_blocks ? bt[page] : -1;
        off = pos % p.block_size;
        if (blk < 0 || blk >= p.num_blocks) {
          B200_NOTE_BAD_INDEX();
          blk = 0;
        }
      }
      s_ptr[stage][threadIdx.x] = p.cache + ((size_t)blk * p.block_size + off) * p.Dq;
      s_pos[stage][threadIdx.x] = ok ? pos : 0x7fffffff;
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < 16 * nch; idx += 128) {
      const int row = idx / nch, ch = idx - row * nch;
      cp16(sbase + stage * STAGE + row * RS + ((ch ^ (row & 7)) << 4), s_ptr[stage][row] + ch * 8);
    }
  };

  float o[LW / 8][4];
#pragma unroll
  for (int i = 0; i < LW / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int mi = lane >> 3, rr = lane & 7;

#pragma unroll
  for (int c = 0; c < NST - 1; ++c) {
    if (c < chunks) prefetch(c, c);
    cp_commit();
  }
  for (int c = 0; c < chunks; ++c) {
    const int stage = c % NST;
    // the stage refilled here was consumed in the previous iteration (which ended with a barrier)
    if (c + NST - 1 < chunks) prefetch(c + NST - 1, (c + NST - 1) % NST);
    cp_commit();
    cp_wait<NST - 1>();
    __syncthreads();
    const uint32_t sb = sbase + stage * STAGE;
    // ---- partial scores over this warp's part of Dq
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    {
      const int tok = (mi >> 1) * 8 + rr;
#pragma unroll
      for (int i = 0; i < KS_MAX; ++i) {
        const int ks = warp + 4 * i;
        if (ks < ksteps) {
          const int ch = 2 * ks + (mi & 1);
          uint32_t b[4];
          ldsm4(b, sb + (uint32_t)(tok * RS + ((ch ^ (tok & 7)) << 4)));
          mma16816(s[0], qf[i], &b[0]);
          mma16816(s[1], qf[i], &b[2]);
        }
      }
    }
    const int row0 = lane >> 2, row1 = row0 + 8, col = 2 * (lane & 3);
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      s_part[warp][row0][nb * 8 + col] = s[nb][0];
      s_part[warp][row0][nb * 8 + col + 1] = s[nb][1];
      s_part[warp][row1][nb * 8 + col] = s[nb][2];
      s_part[warp][row1][nb * 8 + col + 1] = s[nb][3];
    }
    __syncthreads();
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int rrow = (e < 2) ? row0 : row1, cc = nb * 8 + col + (e & 1);
        float v = s_part[0][rrow][cc] + s_part[1][rrow][cc] + s_part[2][rrow][cc] + s_part[3][rrow][cc];
        v = s_pos[stage][cc] <= (e < 2 ? qpos0 : qpos1) ? v * p.scale_log2 : -INFINITY;
        s[nb][e] = v;
        if (e < 2) mx0 = fmaxf(mx0, v); else mx1 = fmaxf(mx1, v);
      }
    }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float mn0 = fmaxf(m[0], mx0), mn1 = fmaxf(m[1], mx1);
    const float base0 = mn0 == -INFINITY ? 0.f : mn0, base1 = mn1 == -INFINITY ? 0.f : mn1;
    const float a0 = ex2(m[0] - base0), a1 = ex2(m[1] - base1);
    m[0] = mn0; m[1] = mn1;
    float ps0 = 0.f, ps1 = 0.f;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      s[nb][0] = ex2(s[nb][0] - base0); s[nb][1] = ex2(s[nb][1] - base0);
      s[nb][2] = ex2(s[nb][2] - base1); s[nb][3] = ex2(s[nb][3] - base1);
      ps0 += s[nb][0] + s[nb][1];
      ps1 += s[nb][2] + s[nb][3];
    }
    l[0] = l[0] * a0 + ps0;
    l[1] = l[1] * a1 + ps1;
#pragma unroll
    for (int i = 0; i < LW / 8; ++i) {
      o[i][0] *= a0; o[i][1] *= a0; o[i][2] *= a1; o[i][3] *= a1;
    }
    const uint32_t pa[4] = {pack2(s[0][0], s[0][1]), pack2(s[0][2], s[0][3]), pack2(s[1][0], s[1][1]),
                            pack2(s[1][2], s[1][3])};
    // ---- P V on this warp's value columns [warp * LW, (warp + 1) * LW)
    {
      const int tok = (mi & 1) * 8 + rr;
#pragma unroll
      for (int np = 0; np < LW / 16; ++np) {
        if (warp * LW + np * 16 >= p.L) break;         // L < 4 * LW
        const int ch = (warp * LW >> 3) + 2 * np + (mi >> 1);
        uint32_t b[4];
        ldsm4t(b, sb + (uint32_t)(tok * RS + ((ch ^ (tok & 7)) << 4)));
        mma16816(o[2 * np], pa, &b[0]);
        mma16816(o[2 * np + 1], pa, &b[2]);
      }
    }
    __syncthreads();                 // the stage and s_part are rewritten by the next iteration
  }
  cp_wait<0>();
  l[0] += __shfl_xor_sync(0xffffffffu, l[0], 1); l[0] += __shfl_xor_sync(0xffffffffu, l[0], 2);
  l[1] += __shfl_xor_sync(0xffffffffu, l[1], 1); l[1] += __shfl_xor_sync(0xffffffffu, l[1], 2);
  const int row0 = lane >> 2, row1 = row0 + 8;
  const float inv0 = l[0] > 0.f ? 1.f / l[0] : 0.f, inv1 = l[1] > 0.f ? 1.f / l[1] : 0.f;
  __nv_bfloat16* out = p.splits > 1 ? p.part_o + (size_t)sp * p.T * p.H * p.L : p.out;
  float* lse = p.splits > 1 ? p.part_lse + (size_t)sp * p.T * p.H : p.lse;
#pragma unroll
  for (int i = 0; i < LW / 8; ++i) {
    const int colv = warp * LW + i * 8 + 2 * (lane & 3);
    const bool c0 = colv < p.L, c1 = colv + 1 < p.L;
    if (row0 < rows_valid) store2(out + (f0 + row0) * p.L + colv, o[i][0] * inv0, o[i][1] * inv0, c0, c1);
    if (row1 < rows_valid) store2(out + (f0 + row1) * p.L + colv, o[i][2] * inv1, o[i][3] * inv1, c0, c1);
  }
  if (lse != nullptr && warp == 0 && (lane & 3) == 0) {
    if (row0 < rows_valid) lse[f0 + row0] = l[0] > 0.f ? (m[0] + log2f(l[0])) * 0.6931471805599453f : -INFINITY;
    if (row1 < rows_valid) lse[f0 + row1] = l[1] > 0.f ? (m[1] + log2f(l[1])) * 0.6931471805599453f : -INFINITY;
  }
}

// out[t, h, :] = sum_s softmax_s(lse[s, t, h]) * part_o[s, t, h, :]; one CTA per (t, h), 8 columns per thread.
// A (token, head) whose splits all saw no key (padded rows) keeps zeros and lse = -inf.
__global__ void mla_merge_kernel(const __nv_bfloat16* __restrict__ part_o, const float* __restrict__ part_lse,
                                 __nv_bfloat16* __restrict__ out, float* __restrict__ lse, int splits, int TH, int L) {
  pdl_launch_dependents();
  pdl_wait();
  const int th = blockIdx.x;
  float mx = -INFINITY;
  for (int s = 0; s < splits; ++s) mx = fmaxf(mx, part_lse[(size_t)s * TH + th]);
  float den = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float v = part_lse[(size_t)s * TH + th];
    den += v == -INFINITY ? 0.f : __expf(v - mx);
  }
  if (lse != nullptr && threadIdx.x == 0) lse[th] = den > 0.f ? mx + __logf(den) : -INFINITY;
  if (L & 7) {                        // rows that are not made of 16-byte pieces
    for (int c = threadIdx.x; c < L; c += blockDim.x) {
      float a = 0.f;
      for (int s = 0; s < splits && den > 0.f; ++s) {
        const float v = part_lse[(size_t)s * TH + th];
        if (v != -INFINITY) a += __expf(v - mx) / den * __bfloat162float(part_o[((size_t)s * TH + th) * L + c]);
      }
      out[(size_t)th * L + c] = __float2bfloat16(a);
    }
    return;
  }
  for (int c = threadIdx.x * 8; c < L; c += blockDim.x * 8) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (den > 0.f) {
      for (int s = 0; s < splits; ++s) {
        const float v = part_lse[(size_t)s * TH + th];
        if (v == -INFINITY) continue;
        const float w = __expf(v - mx) / den;
        const uint4 raw = *reinterpret_cast<const uint4*>(part_o + ((size_t)s * TH + th) * L + c);
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = __bfloat1622float2(h2[j]);
          acc[2 * j] += w * f.x;
          acc[2 * j + 1] += w * f.y;
        }
      }
    }
    uint4 o;
    o.x = pack2(acc[0], acc[1]); o.y = pack2(acc[2], acc[3]); o.z = pack2(acc[4], acc[5]); o.w = pack2(acc[6], acc[7]);
    *reinterpret_cast<uint4*>(out + (size_t)th * L + c) = o;
  }
}

// cache row of slot s = kv_c[t] (L values) followed by k_pe[t] (R values); slot < 0: skipped
__global__ void mla_write_cache_kernel(__nv_bfloat16* __restrict__ cache, const __nv_bfloat16* __restrict__ kv_c,
                                       const __nv_bfloat16* __restrict__ k_pe, const int* __restrict__ slots,
                                       int L, int R, int ld_c, int ld_pe, long long num_slots) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const long long slot = slots[t];
  if (slot < 0 || slot >= num_slots) return;
  __nv_bfloat16* dst = cache + (size_t)slot * (L + R);
  for (int i = threadIdx.x; i < L + R; i += blockDim.x)
    dst[i] = i < L ? kv_c[(size_t)t * ld_c + i] : k_pe[(size_t)t * ld_pe + (i - L)];
}

}  // namespace mla
}  // namespace b200

namespace b200 {
namespace mla {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename E> __device__ __forceinline__ E from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// dst[b * dst_sb + a * dst_sa + d] = src[a * src_sa + b * src_sb + d] for a < A, b < B, d < D (elements;
// D and all strides multiples of 8 so that the copy runs in 16-byte pieces).  Turns [T, H, D] slices into
// the head-major [H, T, D] rows the grouped GEMM wants (heads as groups) and back.
__global__ void permute_rows_kernel(const __nv_bfloat16* __restrict__ src, __nv_bfloat16* __restrict__ dst, int A,
                                    int B, int D8, long long src_sa, long long src_sb, long long dst_sa,
                                    long long dst_sb) {
  pdl_launch_dependents();
  pdl_wait();
  const long long total = (long long)A * B * D8;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total;
       i += (long long)gridDim.x * blockDim.x) {
    const int d = (int)(i % D8);
    const long long ab = i / D8;
    const int b = (int)(ab % B);
    const int a = (int)(ab / B);
    const uint4 v = *reinterpret_cast<const uint4*>(src + a * src_sa + b * src_sb + d * 8);
    *reinterpret_cast<uint4*>(dst + a * dst_sa + b * dst_sb + d * 8) = v;
  }
}

// Rotary embedding of `pairs` dimension pairs of src[t, h, :] (strides in elements) written to dst[t, h, :]:
// interleaved pairs (2i, 2i+1) or split halves (i, i + pairs), angles position * inv_freq[i] in fp32, cos and
// sin times `mult`.  The dims behind the rotated ones up to D are copied, those from D to D + pad zeroed.
template <typename E>
__global__ void rope_rows_kernel(const E* __restrict__ src, E* __restrict__ dst, const int* __restrict__ positions,
                                 const float* __restrict__ inv_freq, float mult, int T, int H, int pairs, int D,
                                 int pad, int interleaved, long long src_st, long long src_sh, long long dst_st,
                                 long long dst_sh) {
  pdl_launch_dependents();
  pdl_wait();
  const int per_row = pairs + (D - 2 * pairs) + pad;
  const long long total = (long long)T * H * per_row;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total;
       i += (long long)gridDim.x * blockDim.x) {
    const int j = (int)(i % per_row);
    const long long th = i / per_row;
    const int h = (int)(th % H);
    const int t = (int)(th / H);
    const E* s = src + t * src_st + h * src_sh;
    E* d = dst + t * dst_st + h * dst_sh;
    if (j >= pairs) {
      const int c = j + pairs;
      d[c] = c < D ? s[c] : from_f<E>(0.f);
      continue;
    }
    float sn, cs;
    sincosf((float)positions[t] * inv_freq[j], &sn, &cs);
    sn *= mult;
    cs *= mult;
    const int i0 = interleaved ? 2 * j : j, i1 = interleaved ? 2 * j + 1 : j + pairs;
    const float x0 = to_f(s[i0]), x1 = to_f(s[i1]);
    d[i0] = from_f<E>(x0 * cs - x1 * sn);
    d[i1] = from_f<E>(x1 * cs + x0 * sn);
  }
}

// The small per-token work behind the packed input projection of a latent-attention layer, one CTA per token:
//   cq[t]        = rms(row[0 : Q]) * wq                      input of the query expansion (Q = 0: absent)
//   cache[slot]  = rms(row[Q : Q + L]) * wc ‖ rope(row[Q + L : Q + L + R])     (L = 0: the layer shares another
//                                                            layer's cache; slot < 0: not stored)
// Norms and angles in fp32; the cache row is Dc wide, its padding is left alone.
struct PrepParams {
  const void *row, *wq, *wc;
  void *cq, *cache;
  const int *slots, *positions;
  const float* inv_freq;
  float eps, mult;
  int Q, L, R, pairs, interleaved, ld, ld_cq, Dc;
  long long num_slots;
};

template <typename E, int V>
__global__ void latent_prep_kernel(const PrepParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x;
  const E* row = reinterpret_cast<const E*>(p.row) + (size_t)t * p.ld;
  auto norm = [&](const E* src, const E* w, E* dst, int n, bool keep) {
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
      if constexpr (V == 8) {
        const bf16x8 a = *reinterpret_cast<const bf16x8*>(src + i);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = __bfloat1622float2(a.v[j]);
          ss += f.x * f.x + f.y * f.y;
        }
      } else {
        const float f = to_f(src[i]);
        ss += f * f;
      }
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)n + p.eps);
    if (!keep) return;
    for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
      if constexpr (V == 8) {
        const bf16x8 a = *reinterpret_cast<const bf16x8*>(src + i), g = *reinterpret_cast<const bf16x8*>(w + i);
        bf16x8 o;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = __bfloat1622float2(a.v[j]), gg = __bfloat1622float2(g.v[j]);
          o.v[j] = __floats2bfloat162_rn(f.x * inv * gg.x, f.y * inv * gg.y);
        }
        *reinterpret_cast<bf16x8*>(dst + i) = o;
      } else {
        dst[i] = from_f<E>(to_f(src[i]) * inv * to_f(w[i]));
      }
    }
  };
  if (p.Q > 0)
    norm(row, reinterpret_cast<const E*>(p.wq), reinterpret_cast<E*>(p.cq) + (size_t)t * p.ld_cq, p.Q, true);
  if (p.L > 0) {
    const long long slot = p.slots[t];
    const bool keep = slot >= 0 && slot < p.num_slots;
    E* dst = reinterpret_cast<E*>(p.cache) + (size_t)(keep ? slot : 0) * p.Dc;
    norm(row + p.Q, reinterpret_cast<const E*>(p.wc), dst, p.L, keep);
    if (!keep) return;
    const E* s = row + p.Q + p.L;
    const float pos = (float)p.positions[t];
    for (int j = threadIdx.x; j < p.R - p.pairs; j += blockDim.x) {
      if (j >= p.pairs) {
        dst[p.L + j + p.pairs] = s[j + p.pairs];
        continue;
      }
      float sn, cs;
      sincosf(pos * p.inv_freq[j], &sn, &cs);
      sn *= p.mult;
      cs *= p.mult;
      const int i0 = p.interleaved ? 2 * j : j, i1 = p.interleaved ? 2 * j + 1 : j + p.pairs;
      const float x0 = to_f(s[i0]), x1 = to_f(s[i1]);
      dst[p.L + i0] = from_f<E>(x0 * cs - x1 * sn);
      dst[p.L + i1] = from_f<E>(x1 * cs + x0 * sn);
    }
  }
}

// Latent attention on the CUDA cores: 32-bit caches, and row widths beyond the tensor-core kernel.  One warp per
// (token, head): 32 keys at a time, their scores by a dot product over the lanes, then an online softmax and the
// weighted sum of the value columns, all in fp32.
template <typename E>
__global__ void __launch_bounds__(256) mla_simt_kernel(const E* __restrict__ q, const E* __restrict__ cache,
                                                       E* __restrict__ out, const int* __restrict__ block_tables,
                                                       const int* __restrict__ seq_lens, const int* __restrict__ qsl,
                                                       int T, int H, int Dq, int L, int num_reqs, int max_blocks,
                                                       int block_size, long long num_blocks, float scale) {
  extern __shared__ float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const long long f = (long long)blockIdx.x * nw + warp;
  if (f >= (long long)T * H) return;
  float* sq = sm + (size_t)warp * (Dq + L);
  float* acc = sq + Dq;
  const int t = (int)(f / H);
  int lo = 0, hi = num_reqs;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (qsl[mid] <= t) lo = mid; else hi = mid;
  }
  const int qs = qsl[lo], q_len = qsl[lo + 1] - qs, kv_len = seq_lens[lo];
  const bool live = t < qsl[num_reqs] && q_len > 0 && kv_len > 0;
  for (int d = lane; d < Dq; d += 32) sq[d] = live ? to_f(q[f * Dq + d]) : 0.f;
  for (int d = lane; d < L; d += 32) acc[d] = 0.f;
  __syncwarp();
  const int n_kv = live ? kv_len - q_len + (t - qs) + 1 : 0;
  const int* bt = block_tables + (size_t)lo * max_blocks;
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < n_kv; k0 += 32) {
    const int nk = min(32, n_kv - k0);
    long long my_row = 0;
    if (lane < nk) {
      const int page = (k0 + lane) / block_size;
      long long blk = page < max_blocks ? bt[page] : -1;
      if (blk < 0 || blk >= num_blocks) {
        B200_NOTE_BAD_INDEX();
        blk = 0;
      }
      my_row = (blk * block_size + (k0 + lane) % block_size) * Dq;
    }
    float s = -INFINITY;
    for (int j = 0; j < nk; ++j) {
      const E* row = cache + __shfl_sync(0xffffffffu, my_row, j);
      float d = 0.f;
      for (int c = lane; c < Dq; c += 32) d = fmaf(sq[c], to_f(row[c]), d);
      d = warp_sum(d);
      if (lane == j) s = d * scale;
    }
    const float mn = fmaxf(m, warp_max(s));
    const float a = expf(m - mn), pr = lane < nk ? expf(s - mn) : 0.f;
    l = l * a + warp_sum(pr);
    m = mn;
    for (int d = lane; d < L; d += 32) acc[d] *= a;
    for (int j = 0; j < nk; ++j) {
      const E* row = cache + __shfl_sync(0xffffffffu, my_row, j);
      const float w = __shfl_sync(0xffffffffu, pr, j);
      for (int d = lane; d < L; d += 32) acc[d] = fmaf(w, to_f(row[d]), acc[d]);
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int d = lane; d < L; d += 32) out[f * L + d] = from_f<E>(acc[d] * inv);
}

}  // namespace mla
}  // namespace b200

using namespace b200;

extern "C" int b200_permute_rows(const void* src, void* dst, int A, int B, int D, long long src_sa, long long src_sb,
                                 long long dst_sa, long long dst_sb, cudaStream_t stream) {
  if (A <= 0 || B <= 0 || D <= 0) return 0;
  if (D % 8 || src_sa % 8 || src_sb % 8 || dst_sa % 8 || dst_sb % 8 || (reinterpret_cast<uintptr_t>(src) & 15) ||
      (reinterpret_cast<uintptr_t>(dst) & 15)) {
    b200_set_last_error("permute_rows: D, the strides and both addresses must be multiples of 8 elements",
                        __FILE__, __LINE__);
    return -1;
  }
  const long long total = (long long)A * B * (D / 8);
  long long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  B200_CUDA_CHECK(launch_pdl(mla::permute_rows_kernel, dim3((unsigned)blocks), dim3(256), (size_t)0, stream,
                             (const __nv_bfloat16*)src, (__nv_bfloat16*)dst, A, B, D / 8, src_sa, src_sb, dst_sa,
                             dst_sb));
  return 0;
}

// elem: 2 = bf16, 4 = fp32; D: dims of a row (>= 2 * pairs), pad: zeroed dims behind them
extern "C" int b200_rope_rows(const void* src, void* dst, const int* positions, const float* inv_freq, float mult,
                              int T, int H, int pairs, int D, int pad, int interleaved, long long src_st,
                              long long src_sh, long long dst_st, long long dst_sh, int elem, cudaStream_t stream) {
  if (T <= 0 || H <= 0 || D + pad <= 0) return 0;
  if (D < 2 * pairs) {
    b200_set_last_error("rope_rows: more rotated dims than the row has", __FILE__, __LINE__);
    return -1;
  }
  const long long total = (long long)T * H * (D - pairs + pad);
  long long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
#define ROPE_LAUNCH(E)                                                                                         \
  B200_CUDA_CHECK(launch_pdl(mla::rope_rows_kernel<E>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream,   \
                             (const E*)src, (E*)dst, positions, inv_freq, mult, T, H, pairs, D, pad,           \
                             interleaved, src_st, src_sh, dst_st, dst_sh))
  if (elem == 4) ROPE_LAUNCH(float);
  else ROPE_LAUNCH(__nv_bfloat16);
#undef ROPE_LAUNCH
  return 0;
}

// row [T, ld] = [Q query latent | L latent | R shared rotated key | ...]; see latent_prep_kernel
extern "C" int b200_latent_prep(const void* row, const void* wq, const void* wc, void* cq, void* cache,
                                const int* slots, const int* positions, const float* inv_freq, float eps, float mult,
                                int T, int Q, int L, int R, int pairs, int interleaved, int ld, int ld_cq, int Dc,
                                long long num_slots, int elem, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (L > 0 && (L + R > Dc || R < 2 * pairs)) {
    b200_set_last_error("latent_prep: the cache row is narrower than latent + rotated key", __FILE__, __LINE__);
    return -1;
  }
  mla::PrepParams p{row, wq, wc, cq, cache, slots, positions, inv_freq, eps, mult,
                    Q, L, R, pairs, interleaved, ld, ld_cq, Dc, num_slots};
  const uintptr_t a = (uintptr_t)row | (uintptr_t)wq | (uintptr_t)wc | (uintptr_t)cq | (uintptr_t)cache;
  const bool vec = elem == 2 && Q % 8 == 0 && L % 8 == 0 && ld % 8 == 0 && ld_cq % 8 == 0 && Dc % 8 == 0 && a % 16 == 0;
  const int n = Q > L ? Q : L;
  int threads = ((vec ? n / 8 : n) + 31) / 32 * 32;
  threads = threads < 64 ? 64 : (threads > 256 ? 256 : threads);
  if (elem == 4)
    B200_CUDA_CHECK(launch_pdl(mla::latent_prep_kernel<float, 1>, dim3(T), dim3(threads), (size_t)0, stream, p));
  else if (vec)
    B200_CUDA_CHECK(launch_pdl(mla::latent_prep_kernel<__nv_bfloat16, 8>, dim3(T), dim3(threads), (size_t)0, stream, p));
  else
    B200_CUDA_CHECK(launch_pdl(mla::latent_prep_kernel<__nv_bfloat16, 1>, dim3(T), dim3(threads), (size_t)0, stream, p));
  return 0;
}

// q [T, H, Dq], cache [num_blocks, block_size, Dq], out [T, H, L], all of `elem` bytes (2 = bf16, 4 = fp32)
extern "C" int b200_mla_attention_simt(const void* q, const void* cache, void* out, const int* block_tables,
                                       const int* seq_lens, const int* qsl, int T, int num_reqs, int H, int Dq, int L,
                                       int max_blocks, int block_size, long long num_blocks, float scale, int elem,
                                       cudaStream_t stream) {
  if (T <= 0 || num_reqs <= 0) return 0;
  int warps = 8;
  while (warps > 1 && warps * (Dq + L) * 4 > 48 * 1024) warps >>= 1;
  const int smem = warps * (Dq + L) * 4;
  if (L > Dq || smem > 200 * 1024) {
    b200_set_last_error("mla_attention_simt: latent wider than the row, or rows too wide", __FILE__, __LINE__);
    return -1;
  }
  const long long blocks = ((long long)T * H + warps - 1) / warps;
#define SIMT_LAUNCH(E)                                                                                           \
  do {                                                                                                           \
    static unsigned long long seen = 0;                                                                          \
    if (smem > 48 * 1024) B200_CUDA_CHECK(ensure_dynamic_smem(mla::mla_simt_kernel<E>, 200 * 1024, &seen));      \
    B200_CUDA_CHECK(launch_pdl(mla::mla_simt_kernel<E>, dim3((unsigned)blocks), dim3(warps * 32), (size_t)smem,  \
                               stream, (const E*)q, (const E*)cache, (E*)out, block_tables, seq_lens, qsl, T, H, \
                               Dq, L, num_reqs, max_blocks, block_size, num_blocks, scale));                     \
  } while (0)
  if (elem == 4) SIMT_LAUNCH(float);
  else SIMT_LAUNCH(__nv_bfloat16);
#undef SIMT_LAUNCH
  return 0;
}

extern "C" int b200_mla_write_cache(void* cache, const void* kv_c, const void* k_pe, const int* slots, int T, int L,
                                    int R, int ld_c, int ld_pe, long long num_slots, cudaStream_t stream) {
  if (T == 0) return 0;
  B200_CUDA_CHECK(launch_pdl(mla::mla_write_cache_kernel, dim3(T), dim3(128), 0, stream, (__nv_bfloat16*)cache,
                             (const __nv_bfloat16*)kv_c, (const __nv_bfloat16*)k_pe, slots, L, R, ld_c, ld_pe,
                             num_slots));
  return 0;
}

// q [T, H, Dq], cache [num_blocks, block_size, Dq], out [T, H, L], lse [T, H] or null,
// topk [T, topk_k] or null.  Dq % 16 == 0, Dq <= 576, L <= 512.
// flat_tiles > 0: 16-row tiles over the (token, head) rows of each request, that many in all (dense only).
// splits > 1: part_o [splits, T, H, L] bf16 and part_lse [splits, T, H] fp32 are scratch of the caller.
extern "C" int b200_mla_attention(const void* q, const void* cache, void* out, float* lse, const int* block_tables,
                                  const int* seq_lens, const int* qsl, const int* topk, int topk_k, int T,
                                  int num_reqs, int H, int Dq, int L, int max_blocks, int block_size,
                                  long long num_blocks, float scale, int flat_tiles, int splits, void* part_o,
                                  float* part_lse, cudaStream_t stream) {
  if (T <= 0 || num_reqs <= 0) return 0;
  if (Dq % 16 || Dq > 4 * mla::KS_MAX * 16 || L > Dq || L < 1 || L > 512 || (flat_tiles > 0 && topk)) {
    b200_set_last_error("mla_attention: Dq % 16 == 0, Dq <= 576, kv_lora <= 512 and no flat tiles with top-k required",
                        __FILE__, __LINE__);
    return -1;
  }
  mla::Params p;
  p.q = (const __nv_bfloat16*)q; p.cache = (const __nv_bfloat16*)cache; p.out = (__nv_bfloat16*)out;
  p.lse = lse; p.block_tables = block_tables; p.seq_lens = seq_lens; p.qsl = qsl;
  p.topk = topk; p.topk_k = topk_k;
  p.T = T; p.H = H; p.Dq = Dq; p.L = L; p.num_reqs = num_reqs; p.max_blocks = max_blocks;
  p.block_size = block_size; p.num_blocks = num_blocks;
  p.scale_log2 = scale * 1.4426950408889634f;
  if (splits < 1 || (splits > 1 && (part_o == nullptr || part_lse == nullptr))) {
    b200_set_last_error("mla_attention: split-KV needs its scratch", __FILE__, __LINE__);
    return -1;
  }
  p.splits = splits; p.part_o = (__nv_bfloat16*)part_o; p.part_lse = part_lse;
  const int nch = Dq / 8;
  const int smem = mla::NST * 16 * (((nch + 7) & ~7) << 4);
  p.flat = flat_tiles > 0 ? 1 : 0;
  const dim3 grid((p.flat ? flat_tiles : T * ((H + 15) / 16)) * splits);
#define MLA_LAUNCH(LWV)                                                                                      \
  do {                                                                                                       \
    B200_CUDA_CHECK(cudaFuncSetAttribute(mla::mla_attn_kernel<LWV>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                         smem));                                                             \
    B200_CUDA_CHECK(launch_pdl(mla::mla_attn_kernel<LWV>, grid, dim3(128), (size_t)smem, stream, p));         \
  } while (0)
  if (L <= 64) MLA_LAUNCH(16);
  else if (L <= 128) MLA_LAUNCH(32);
  else if (L <= 192) MLA_LAUNCH(48);
  else if (L <= 256) MLA_LAUNCH(64);
  else if (L <= 384) MLA_LAUNCH(96);
  else MLA_LAUNCH(128);
#undef MLA_LAUNCH
  if (splits > 1)
    B200_CUDA_CHECK(launch_pdl(mla::mla_merge_kernel, dim3(T * H), dim3(64), (size_t)0, stream,
                               (const __nv_bfloat16*)part_o, (const float*)part_lse, (__nv_bfloat16*)out, lse,
                               splits, T * H, L));
  return 0;
}

// see b200_bad_index_count_attention
extern "C" int b200_bad_index_count_attention_mla(unsigned int* out) {
  B200_TAKE_BAD_INDEX_COUNT(out);
  return 0;
}
