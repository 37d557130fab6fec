// Gated linear attention of prompts in 64-token chunks on the tensor cores (bf16 activations, key
// sizes that are multiples of 16 up to 128). With b_t the running sum of log alpha inside a chunk
// (b_end its last entry) and S the state before the chunk,
//
//   o_t = S^T (q_t e^{b_t}) + sum_{s <= t} A_ts v_s,     A_ts = sum_d q_td k_sd e^{b_td - b_sd}
//   S' = diag(e^{b_end}) S + sum_s (k_s e^{b_end - b_s}) v_s^T
//
// Everything that enters the recurrence keeps 32-bit accuracy: the decays, their sums and
// exponentials are fp32, the state is fp32 (in tensor memory), and every factor that is not a plain
// bf16 projection (decayed q and k, A, the state as an operand) goes into the products as a sum of
// two bf16 parts, high and low, whose cross terms are accumulated in fp32. All exponents are <= 0
// but inside a 16-token diagonal block, which takes an exact path where its decay is steep.
//
//   gla_chunk_prep  one CTA per (chunk, head): decays, decayed q / k, A
//   gla_chunk_scan  one CTA per (sequence, head, 128 value columns): walks the chunks in order. The
//                   state is held transposed in tensor memory (lane = value column, column = key
//                   channel), so that the decay is a per-column factor and the state becomes the
//                   tensor-memory operand of S^T q without passing through shared memory:
//                       S^T += V^T K        (128 x dim,  k = 64 tokens, 2 parts)
//                       O^T  = V^T A^T + S^T Q^T   (128 x 64 tokens, 2 + 3 part products)
//                   Roles: TMA producer, tcgen05 issuer, eight state warps, four output warps.
//
// All mbarrier waits are bounded; a time-out sets the status word, the CTA stops issuing copies,
// waits (bounded) for those in flight, reaches its barriers and frees its tensor memory.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <string.h>
#include <mutex>

#include "flash_common.cuh"
#include "gla.cuh"
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar_types.cuh"

namespace e2h {

constexpr int kC = 64;                 // tokens per chunk
constexpr float kSteep = 40.f;         // decay (in e) up to which its inverse is harmless

__device__ __forceinline__ int chunk_place(const E2hGlaParams& p, int sg, int c) {
  return p.seg[sg] / kC + sg + c;
}
__device__ __forceinline__ float exp_ftz(float x) { return ex2_approx(x * 1.4426950408889634f); }
__device__ __forceinline__ float lg2_ftz(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_ftz(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// log sigmoid(z) to about 1e-7 absolute: it is only ever added up and exponentiated
__device__ __forceinline__ float log_sigmoid_c(float z) {
  const float e = exp_ftz(-fabsf(z));
  // log(1 + e): Taylor series where 1 + e would round e away
  const float l = e < 0.03f ? e * (1.f - e * (0.5f - e * (1.f / 3.f - e * 0.25f)))
                            : lg2_ftz(1.f + e) * 0.6931471805599453f;
  return fminf(z, 0.f) - l;
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// two values as packed bf16 high parts and packed bf16 low parts
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack2(a, b);
  lo = pack2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ void mma_16816(float* c, const uint32_t* a, const uint32_t* b) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
      "{%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

constexpr int kPrepThreads = 512;
constexpr int kAT = kC + 4;            // row pitch of the transposed decay input

__host__ __device__ inline int prep_smem_bytes(int dim, int r) {
  // b [64][dim + 4] fp32, four bf16 [64][dim + 8] (q and k in two parts), a^T [r][68] fp32,
  // partial sums [512], decay of the whole chunk [dim]
  return kC * (dim + 4) * 4 + 4 * kC * (dim + 8) * 2 + r * kAT * 4 + kPrepThreads * 4 + dim * 4;
}

// Decay logits of J x 4 consecutive tokens (from tb on) of one key channel: w . a_t + bias.
template <int J>
__device__ __forceinline__ void decay_logits(float* z, const __nv_bfloat16* w, bool wvec, int r,
                                             const float* at, float bias) {
#pragma unroll
  for (int j = 0; j < 4 * J; ++j) z[j] = bias;
  for (int i0 = 0; i0 < r; i0 += 8) {
    float wv[8];
    if (wvec) {
      load8(w + i0, wv);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) wv[e] = i0 + e < r ? to_f(w[i0 + e]) : 0.f;
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      if (i0 + e >= r) break;
#pragma unroll
      for (int j = 0; j < J; ++j) {
        const float4 av = *reinterpret_cast<const float4*>(at + (i0 + e) * kAT + 4 * j);
        z[4 * j] = fmaf(wv[e], av.x, z[4 * j]);
        z[4 * j + 1] = fmaf(wv[e], av.y, z[4 * j + 1]);
        z[4 * j + 2] = fmaf(wv[e], av.z, z[4 * j + 2]);
        z[4 * j + 3] = fmaf(wv[e], av.w, z[4 * j + 3]);
      }
    }
  }
}

// MMA fragments of rows r0.. and columns k0.. of a [64][pitch] bf16 tile
__device__ __forceinline__ uint32_t frag(const __nv_bfloat16* x, int row, int col, int pitch) {
  return *reinterpret_cast<const uint32_t*>(x + row * pitch + col);
}

__global__ void __launch_bounds__(kPrepThreads, 2) gla_chunk_prep_kernel(const E2hGlaParams p) {
  extern __shared__ __align__(16) uint8_t prep_raw[];
  const int D = p.dim, LB = D + 4, LQ = D + 8;
  float* b_s = reinterpret_cast<float*>(prep_raw);                        // [64][LB]
  __nv_bfloat16* qh_s = reinterpret_cast<__nv_bfloat16*>(b_s + kC * LB);  // [64][LQ] each
  __nv_bfloat16* ql_s = qh_s + kC * LQ;
  __nv_bfloat16* kh_s = ql_s + kC * LQ;
  __nv_bfloat16* kl_s = kh_s + kC * LQ;
  float* at_s = reinterpret_cast<float*>(kl_s + kC * LQ);                 // [r][kAT]
  float* sum_s = at_s + p.r * kAT;                                        // [512]
  float* g_s = sum_s + kPrepThreads;                                      // [dim]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int c = blockIdx.x, head = blockIdx.y, sg = blockIdx.z;
  const int s0 = p.seg[sg], s1 = p.seg[sg + 1];
  const int t0 = s0 + c * kC;
  if (s0 < 0 || s1 > p.n || t0 >= s1) return;
  const int nt = min(kC, s1 - t0);
  const int place = chunk_place(p, sg, c);
  if (place >= p.chunks) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  const int tid = threadIdx.x;
  const __nv_bfloat16* act = static_cast<const __nv_bfloat16*>(p.act) + (long long)t0 * p.ld +
                             (long long)head * D;
  // the thread's q and k (at most 2 pieces of 8 columns): in flight under the decays
  uint4 q4[2], k4[2];
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int i = tid + n * kPrepThreads, t = i / (D / 8), d = (i - t * (D / 8)) * 8;
    q4[n] = k4[n] = make_uint4(0, 0, 0, 0);
    if (t < nt) {
      q4[n] = *reinterpret_cast<const uint4*>(act + (long long)t * p.ld + p.off_q + d);
      k4[n] = *reinterpret_cast<const uint4*>(act + (long long)t * p.ld + p.off_k + d);
    }
  }
  for (int i = tid; i < kC * p.r; i += kPrepThreads) {
    const int t = i / p.r, k = i - t * p.r;
    at_s[k * kAT + t] = t < nt ? p.a[(long long)(t0 + t) * p.lda + k] : 0.f;
  }
  __syncthreads();
  // running sums of log alpha: `ng` groups of threads take consecutive runs of tokens of a column
  {
    const int ng = min(kPrepThreads / D, 16), run = ((kC + ng - 1) / ng + 3) / 4 * 4;   // <= 16
    const int g = tid / D, d = tid - g * D, tb = g * run;
    const bool work = g < ng && tb < kC;
    float z[16];
    float add = 0.f;
    if (work) {
      const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(p.w2) +
                               ((long long)head * D + d) * p.ldw;
      const bool wvec = (p.ldw & 7) == 0 && (p.r & 7) == 0 &&
                        (reinterpret_cast<uintptr_t>(p.w2) & 15) == 0;
      const float bias = p.b2[head * D + d];
      // a run of 12 computes 16: the columns read past the row are in shared memory, not used
      if (run == 4) decay_logits<1>(z, w, wvec, p.r, at_s + tb, bias);
      else if (run == 8) decay_logits<2>(z, w, wvec, p.r, at_s + tb, bias);
      else decay_logits<4>(z, w, wvec, p.r, at_s + tb, bias);
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        if (j < run && tb + j < nt) acc += log_sigmoid_c(z[j]) * p.inv_tau;
        z[j] = acc;
      }
      sum_s[tid] = acc;
    }
    __syncthreads();
    if (work) {
      for (int k = 0; k < g; ++k) add += sum_s[k * D + d];
#pragma unroll
      for (int j = 0; j < 16; ++j)
        if (j < run && tb + j < kC) b_s[(tb + j) * LB + d] = z[j] + add;
    }
  }
  __syncthreads();
  const float* b_end = b_s + (kC - 1) * LB;
  bool mine = false;
  for (int d = tid; d < D; d += kPrepThreads) {
    mine = mine || !(-b_end[d] <= kSteep);
    g_s[d] = exp_ftz(b_end[d]);
    p.cg[((long long)place * p.H + head) * D + d] = g_s[d];
  }
  // steep: the inverse decay of the chunk leaves the fp32 range; A then takes its exact form and
  // the shared tiles hold the plain q and k
  const bool steep = __syncthreads_or(mine) != 0;
  const long long row0 = ((long long)place * p.H + head) * kC;
  const long long part = (long long)p.chunks * p.H * kC * D;
  __nv_bfloat16* cq = static_cast<__nv_bfloat16*>(p.cq) + row0 * D;
  __nv_bfloat16* ck = static_cast<__nv_bfloat16*>(p.ck) + row0 * D;
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int i = tid + n * kPrepThreads, t = i / (D / 8), d = (i - t * (D / 8)) * 8;
    if (t >= kC) break;
    float q[8], k[8], b[8];
    load8(reinterpret_cast<const __nv_bfloat16*>(&q4[n]), q);
    load8(reinterpret_cast<const __nv_bfloat16*>(&k4[n]), k);
    load8(b_s + t * LB + d, b);
    uint32_t qh[4], ql[4], kh[4], kl[4], eh[4], el[4];
    float gd[8];
    load8(g_s + d, gd);
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const float e0 = exp_ftz(b[e]), e1 = exp_ftz(b[e + 1]);
      split2(q[e] * p.qscale * e0, q[e + 1] * p.qscale * e1, qh[e / 2], ql[e / 2]);
      if (!steep) {
        const float k0 = k[e] * rcp_ftz(e0), k1 = k[e + 1] * rcp_ftz(e1);
        split2(k0, k1, kh[e / 2], kl[e / 2]);
        split2(k0 * gd[e], k1 * gd[e + 1], eh[e / 2], el[e / 2]);
      } else {
        split2(k[e] * exp_ftz(b_end[d + e] - b[e]), k[e + 1] * exp_ftz(b_end[d + e + 1] - b[e + 1]),
               eh[e / 2], el[e / 2]);
      }
    }
    const long long o = (long long)t * D + d;
    const uint4 qh4 = make_uint4(qh[0], qh[1], qh[2], qh[3]);
    const uint4 ql4 = make_uint4(ql[0], ql[1], ql[2], ql[3]);
    *reinterpret_cast<uint4*>(cq + o) = qh4;
    *reinterpret_cast<uint4*>(cq + part + o) = ql4;
    *reinterpret_cast<uint4*>(ck + o) = make_uint4(eh[0], eh[1], eh[2], eh[3]);
    *reinterpret_cast<uint4*>(ck + part + o) = make_uint4(el[0], el[1], el[2], el[3]);
    if (!steep) {
      *reinterpret_cast<uint4*>(qh_s + t * LQ + d) = qh4;
      *reinterpret_cast<uint4*>(ql_s + t * LQ + d) = ql4;
      *reinterpret_cast<uint4*>(kh_s + t * LQ + d) = make_uint4(kh[0], kh[1], kh[2], kh[3]);
      *reinterpret_cast<uint4*>(kl_s + t * LQ + d) = make_uint4(kl[0], kl[1], kl[2], kl[3]);
    } else {
      store4(qh_s + t * LQ + d, q);
      store4(qh_s + t * LQ + d + 4, q + 4);
      store4(kh_s + t * LQ + d, k);
      store4(kh_s + t * LQ + d + 4, k + 4);
    }
  }
  __syncthreads();
  // A in 16 x 16 blocks
  const int warp = tid >> 5, lane = tid & 31;
  const int gr = lane >> 2, c2 = (lane & 3) * 2;
  __nv_bfloat16* ca = static_cast<__nv_bfloat16*>(p.ca) + row0 * kC;
  const long long apart = (long long)p.chunks * p.H * kC * kC;
  {
    const int bi = warp >> 2, bj = warp & 3;      // one block per warp, those above the diagonal 0
    float acc[2][4];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int y = 0; y < 4; ++y) acc[x][y] = 0.f;
    if (bj <= bi && !steep) {
      const int ra = 16 * bi + gr, rb = 16 * bj + gr;
      for (int k0 = 0; k0 < D; k0 += 16) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {              // (row, k): (g, c) (g + 8, c) (g, c + 8) ..
          ah[x] = frag(qh_s, ra + (x & 1) * 8, k0 + c2 + (x >> 1) * 8, LQ);
          al[x] = frag(ql_s, ra + (x & 1) * 8, k0 + c2 + (x >> 1) * 8, LQ);
        }
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            bh[x] = frag(kh_s, rb + nb * 8, k0 + c2 + x * 8, LQ);
            bl[x] = frag(kl_s, rb + nb * 8, k0 + c2 + x * 8, LQ);
          }
          mma_16816(acc[nb], ah, bh);
          mma_16816(acc[nb], ah, bl);
          mma_16816(acc[nb], al, bh);
        }
      }
    } else if (bj <= bi) {
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int y = 0; y < 4; ++y) {
          const int t = 16 * bi + gr + (y >> 1) * 8, s = 16 * bj + nb * 8 + c2 + (y & 1);
          if (s > t) continue;
          float v = 0.f;
          for (int d = 0; d < D; ++d)
            v = fmaf(to_f(qh_s[t * LQ + d]) * p.qscale,
                     to_f(kh_s[s * LQ + d]) * exp_ftz(b_s[t * LB + d] - b_s[s * LB + d]), v);
          acc[nb][y] = v;
        }
    }
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int t = 16 * bi + gr + hf * 8, s = 16 * bj + nb * 8 + c2;
        uint32_t hi, lo;
        split2(s <= t ? acc[nb][2 * hf] : 0.f, s + 1 <= t ? acc[nb][2 * hf + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(ca + t * kC + s) = hi;
        *reinterpret_cast<uint32_t*>(ca + apart + t * kC + s) = lo;
      }
  }
}

// ---------------------------------------------------------------------------------------------
constexpr int kGsThreads = 448;      // producer, issuer, eight state warps, four output warps
constexpr int kGsStages = 2;

struct GlaCtrl {
  uint64_t full[kGsStages], empty[kGsStages];
  uint64_t s_ready;          // state warps: decayed state and its operand parts are in place
  uint64_t s_full;           // issuer: the state of the chunk is complete
  uint64_t o_full[2], o_empty[2];
  uint32_t tmem_base;
  int abort_flag;
};

// Dropping the low part x low part product, S^T q takes three of the four part products.
template <int NH>            // 64-wide blocks of the key size
__global__ void __launch_bounds__(kGsThreads, 1)
gla_chunk_scan_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                      const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmV,
                      const E2hGlaParams p) {
  constexpr int kBlk = 64 * 128;                       // [64 rows x 64] bf16
  constexpr int kQ = NH * kBlk, kStage = 4 * kQ + 2 * kBlk + 2 * kBlk;   // Qh Ql Kh Kl Ah Al V
  constexpr int DP = NH * 64;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~uintptr_t(1023));
  GlaCtrl* ctrl = reinterpret_cast<GlaCtrl*>(smem);
  float* g_s = reinterpret_cast<float*>(smem + 1024);  // [2][DP] chunk decays
  uint8_t* tiles = smem + 2048 + 1024;

  pdl_launch_dependents();
  pdl_wait_prior();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int v0 = blockIdx.x * 128, head = blockIdx.y, sg = blockIdx.z;
  const int t_begin = p.seg[sg], len = p.seg[sg + 1] - t_begin;
  if (t_begin < 0 || t_begin + len > p.n || len <= 0) return;
  const int slot = p.slot[t_begin];
  const int n_ch = (len + kC - 1) / kC;
  const int place0 = chunk_place(p, sg, 0);
  if (slot < 0 || slot >= p.slots || place0 + n_ch > p.chunks) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  volatile int* abort_flag = &ctrl->abort_flag;
  if (threadIdx.x == 0) {
    for (int s = 0; s < kGsStages; ++s) {
      mbar_init(smem_u32(&ctrl->full[s]), 1);
      mbar_init(smem_u32(&ctrl->empty[s]), 1);
    }
    mbar_init(smem_u32(&ctrl->s_ready), 8);
    mbar_init(smem_u32(&ctrl->s_full), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&ctrl->o_full[s]), 1);
      mbar_init(smem_u32(&ctrl->o_empty[s]), 4);
    }
    ctrl->abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&ctrl->tmem_base), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // tensor memory: S^T fp32 [0, 128), O^T [128, 256) in two buffers, S^T as operand (high, low)
  // [256, 512) in two buffers
  const uint32_t tm = ctrl->tmem_base;
  const uint32_t tm_s = tm, tm_o = tm + 128, tm_c = tm + 256;

  if (warp == 0 && lane == 0) {
    // ---------------- TMA producer ----------------
    const int low = p.chunks * p.H * kC;               // rows between the high and low parts
    int issued = 0;
    for (int c = 0; c < n_ch; ++c) {
      const int s = c % kGsStages;
      if (!mbar_wait(smem_u32(&ctrl->empty[s]), ((c / kGsStages) & 1) ^ 1, abort_flag, p.status,
                     kStatusTimeoutEmpty))
        break;
      const uint32_t bar = smem_u32(&ctrl->full[s]);
      const uint32_t st = smem_u32(tiles + s * kStage);
      const int row = ((place0 + c) * p.H + head) * kC;
      mbar_expect_tx(bar, kStage);
#pragma unroll
      for (int part = 0; part < 2; ++part) {
#pragma unroll
        for (int hf = 0; hf < NH; ++hf) {
          tma_load_2d(st + part * kQ + hf * kBlk, &tmQ, hf * 64, part * low + row, bar);
          tma_load_2d(st + (2 + part) * kQ + hf * kBlk, &tmK, hf * 64, part * low + row, bar);
        }
        tma_load_2d(st + 4 * kQ + part * kBlk, &tmA, 0, part * low + row, bar);
        tma_load_4d(st + 4 * kQ + (2 + part) * kBlk, &tmV, v0 + 64 * part, t_begin + c * kC, head,
                    0, bar);
      }
      issued = c + 1;
    }
    if (*abort_flag) {
      for (int c = issued > kGsStages ? issued - kGsStages : 0; c < issued; ++c) {
        const long long tq = clock64();
        while (!mbar_try_wait(smem_u32(&ctrl->full[c % kGsStages]), (c / kGsStages) & 1))
          if (clock64() - tq > kWaitLimitCycles / 8) break;
      }
    }
  } else if (warp == 1 && lane == 0) {
    // ---------------- UMMA issuer ----------------
    const uint32_t i_upd = make_idesc_bf16(128, DP, 1, 1);   // S^T += V^T K
    const uint32_t i_va = make_idesc_bf16(128, kC, 1, 0);    // O^T = V^T A^T
    const uint32_t i_sq = make_idesc_bf16(128, kC, 0, 0);    // O^T += S^T Q^T (S^T in TMEM)
    const uint32_t d_hi = sw128_desc_hi(1024);
    for (int c = 0; c < n_ch; ++c) {
      const int s = c % kGsStages, b = c & 1;
      if (!mbar_wait(smem_u32(&ctrl->full[s]), (c / kGsStages) & 1, abort_flag, p.status,
                     kStatusTimeoutFull))
        break;
      if (!mbar_wait(smem_u32(&ctrl->s_ready), c & 1, abort_flag, p.status,
                     kStatusTimeoutTmemEmpty))
        break;
      tc_fence_after();
      const uint32_t st = smem_u32(tiles + s * kStage);
      const uint32_t v_mn = sw128_desc_lo(st + 4 * kQ + 2 * kBlk, kBlk);
      // the state first: the next chunk's decay waits for it
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const uint32_t k_mn = sw128_desc_lo(st + (2 + part) * kQ, kBlk);
#pragma unroll
        for (int kk = 0; kk < kC / 16; ++kk)
          umma_f16_lohi(tm_s, v_mn + ((kk * 2048) >> 4), d_hi, k_mn + ((kk * 2048) >> 4), d_hi,
                        i_upd, 1u);
      }
      umma_commit(smem_u32(&ctrl->s_full));
      if (!mbar_wait(smem_u32(&ctrl->o_empty[b]), ((c >> 1) & 1) ^ 1, abort_flag, p.status,
                     kStatusTimeoutTmemEmpty))
        break;
      tc_fence_after();
      const uint32_t o = tm_o + b * 64;
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const uint32_t a_k = sw128_desc_lo(st + 4 * kQ + part * kBlk, 16);
#pragma unroll
        for (int kk = 0; kk < kC / 16; ++kk)
          umma_f16_lohi(o, v_mn + ((kk * 2048) >> 4), d_hi, a_k + ((kk * 32) >> 4), d_hi, i_va,
                        (part | kk) ? 1u : 0u);
      }
#pragma unroll
      for (int pr = 0; pr < 3; ++pr) {                 // (high, high), (high, low), (low, high)
        const uint32_t s_op = tm_c + b * 128 + (pr == 2 ? 64 : 0);
        const uint32_t q_k = sw128_desc_lo(st + (pr == 1 ? kQ : 0), 16);
#pragma unroll
        for (int kk = 0; kk < NH * 4; ++kk)
          umma_f16_ts(o, s_op + kk * 8, q_k + (((kk / 4) * kBlk + (kk % 4) * 32) >> 4), d_hi, i_sq,
                      1u);
      }
      umma_commit(smem_u32(&ctrl->empty[s]));
      umma_commit(smem_u32(&ctrl->o_full[b]));
    }
  } else if (warp >= 2 && warp < 10) {
    // ---------------- state warps: lane = value column, two warps share the key channels --------
    const int q = warp & 3;
    const int d_lo = (warp - 2) >> 2 ? DP / 2 : 0, d_hi = d_lo + DP / 2;
    const int row = q * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    const int col = v0 + row;
    const bool live = col < p.vp;
    const int st_tid = threadIdx.x - 64;               // 0..255
    float* S = p.state + ((long long)slot * p.H + head) * p.dim * p.vp + col;
    const bool fresh = p.pos[t_begin] == 0;
    auto g_fetch = [&](int c) {
      if (st_tid < DP)
        g_s[(c & 1) * DP + st_tid] =
            st_tid < p.dim ? p.cg[((long long)(place0 + c) * p.H + head) * p.dim + st_tid] : 0.f;
    };
    g_fetch(0);
    bool ok = true;
    for (int c = 0; c <= n_ch; ++c) {
      if (c > 0) {
        if (ok) ok = mbar_wait(smem_u32(&ctrl->s_full), (c - 1) & 1, abort_flag, p.status,
                               kStatusTimeoutTmemFull);
        ok = __all_sync(0xffffffffu, ok);
        tc_fence_after();
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");   // g_s of this chunk is written
      if (c + 1 < n_ch) g_fetch(c + 1);
      const float* g = g_s + (c & 1) * DP;
#pragma unroll 1
      for (int d0 = d_lo; d0 < d_hi; d0 += 32) {
        float v[32];
        if (c == 0) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            v[i] = (!fresh && live && d0 + i < p.dim) ? S[(long long)(d0 + i) * p.vp] : 0.f;
        } else {
          if (ok) tmem_ld_x32(tm_s + lane_off + d0, v);
          tmem_ld_wait();
        }
        if (c == n_ch) {
          if (ok && live) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (d0 + i < p.dim) S[(long long)(d0 + i) * p.vp] = v[i];
          }
          continue;
        }
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          split2(v[2 * i], v[2 * i + 1], hi[i], lo[i]);
          v[2 * i] *= g[d0 + 2 * i];
          v[2 * i + 1] *= g[d0 + 2 * i + 1];
        }
        if (ok) {
          const uint32_t cb = tm_c + lane_off + (c & 1) * 128 + d0 / 2;
          tmem_st_x32(tm_s + lane_off + d0, v);
          tmem_st_x16(cb, hi);
          tmem_st_x16(cb + 64, lo);
        }
      }
      if (c == n_ch) break;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&ctrl->s_ready));
    }
  } else if (warp >= 10) {
    // ---------------- output warps: lane = value column, register = token ----------------
    const int q = warp & 3;
    const int col = v0 + q * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    bool ok = true;
    for (int c = 0; c < n_ch; ++c) {
      const int b = c & 1;
      if (ok) ok = mbar_wait(smem_u32(&ctrl->o_full[b]), (c >> 1) & 1, abort_flag, p.status,
                             kStatusTimeoutTmemFull);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      const int nt = min(kC, len - c * kC);
      float* dst = p.o + ((long long)(t_begin + c * kC) * p.H + head) * p.vdim + col;
      const long long ts = (long long)p.H * p.vdim;
      float v[64];
      if (ok) {
        tmem_ld_x32(tm_o + lane_off + b * 64, v);
        tmem_ld_x32(tm_o + lane_off + b * 64 + 32, v + 32);
      }
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&ctrl->o_empty[b]));
      if (ok && col < p.vdim) {
#pragma unroll
        for (int t = 0; t < 64; ++t)
          if (t < nt) dst[t * ts] = v[t];
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tm, 512);
}

// 2-D map of [rows, cols] bf16 rows, box 64 x 64, zeros past the last column.
static int chunk_map(CUtensorMap* m, const void* base, int cols, long long rows) {
  EncodeTiledFn fn = flash_encode_fn();
  if (!fn) return -10;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
  cuuint32_t box[2] = {64u, 64u}, estr[2] = {1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides,
                  box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                  CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -11;
}

template <int NH>
static int scan_launch(const E2hGlaParams& p, cudaStream_t stream) {
  CUtensorMap tq, tk, ta, tv;
  const long long rows = 2LL * p.chunks * p.H * kC;
  int r = chunk_map(&tq, p.cq, p.dim, rows);
  if (!r) r = chunk_map(&tk, p.ck, p.dim, rows);
  if (!r) r = chunk_map(&ta, p.ca, kC, rows);
  if (!r)
    r = make_map4d(&tv, static_cast<const __nv_bfloat16*>(p.act) + p.off_v, p.vdim, p.n, p.H, 1,
                   (long long)p.n * p.ld, p.ld, p.vdim, kC);
  if (r) return r;
  const size_t smem = 1024 + 3072 + (size_t)kGsStages * (4 * NH + 4) * 64 * 128;
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [&] {
    err = cudaFuncSetAttribute(gla_chunk_scan_kernel<NH>,
                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  });
  if (err != cudaSuccess) return (int)err;
  const dim3 grid((p.vdim + 127) / 128, p.H, p.n_seg);
  return (int)launch(gla_chunk_scan_kernel<NH>, grid, dim3(kGsThreads), smem, stream, tq, tk, ta,
                     tv, p);
}

}  // namespace e2h

// Both kernels of the chunked form; the caller provides cq, ck, ca, cg for `chunks` places.
extern "C" int e2h_gla_chunk(const E2hGlaParams* pp, void* stream_v) {
  using namespace e2h;
  const E2hGlaParams& p = *pp;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_v);
  if (p.n <= 0 || p.H <= 0 || p.H > 65535 || p.n_seg <= 0 || p.n_seg > 65535 || p.seg_max <= 0)
    return -1;
  if (p.dim <= 0 || p.dim > 128 || p.dim % 16 || p.vdim <= 0 || p.vdim % 8 || p.r <= 0) return -2;
  if (p.ld % 8 || p.off_q % 8 || p.off_k % 8 || p.off_v % 8 || p.vp < p.vdim) return -2;
  if ((reinterpret_cast<uintptr_t>(p.act) | reinterpret_cast<uintptr_t>(p.cq) |
       reinterpret_cast<uintptr_t>(p.ck) | reinterpret_cast<uintptr_t>(p.ca)) & 15)
    return -3;
  if (!p.o || !p.cg || !p.state || !p.status || p.chunks < p.n / kC + p.n_seg) return -3;
  if (2LL * p.chunks * p.H * kC > 0x7fffffffLL) return -4;
  const int smem = prep_smem_bytes(p.dim, p.r);
  if (smem > 200 * 1024 || p.r > 128) return -5;
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [] {
    err = cudaFuncSetAttribute(gla_chunk_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                               200 * 1024);
  });
  if (err != cudaSuccess) return (int)err;
  int r = (int)launch(gla_chunk_prep_kernel, dim3((p.seg_max + kC - 1) / kC, p.H, p.n_seg),
                      dim3(kPrepThreads), (size_t)smem, stream, p);
  if (r) return r;
  return p.dim <= 64 ? scan_launch<1>(p, stream) : scan_launch<2>(p, stream);
}
