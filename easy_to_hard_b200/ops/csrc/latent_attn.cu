// Latent attention of the hybrid decoders over the slot cache. A position keeps one normed latent c
// (`rank` columns) and one rotated key part (`rot` columns) that all heads share; the keys and values
// of the heads are linear in c:
//
//   score(i, j) = (q_h . W_uk,h c_j + qr_h . r_j) * scale = ((W_uk,h^T q_h) . c_j + qr_h . r_j) * scale
//   out_h(i)    = W_uv,h (sum_j p_ij c_j)
//
// so that with absorbed queries ql_h = W_uk,h^T q_h the cache row [c | r] is the key of every head and
// c is its value: H query heads over one kv head of `rank + rot` columns. The window is
// 0 <= i - j < window (0: unlimited).
//
// The projections of a token lie in one row of a packed activation [tokens, ld]: q at off_q, head by
// head [dim | rot], and [c (not normed) | r (not rotated)] at off_c. The cache is
// [slots, smax, rank + rot]. All sizes are multiples of 8 (filled with zeros); `rank_n` is the number
// of columns the latent's norm averages over. Rotations pair neighbouring columns (2i, 2i + 1).
//
//   latent_prep   prompts: norms c, rotates r, writes both to the cache and, for the segments whose
//                 keys are expanded per head, to the rows of a context buffer; copies the context's
//                 earlier positions there from the cache; rotates q in place. One CTA per row.
//   latent_attn   absorbed attention, one token per cluster of CTAs: its keys are split over the CTAs
//                 and merged through distributed shared memory.
//     bf16        warp-level matrix products on a ring of cache rows that TMA fills. A token brings
//                 at most 16 or 32 query rows, far below a tcgen05 tile, and the kernel is a stream of
//                 the cache; in its fused form (decode) it also does the work of latent_prep.
//                 Prompts expand the keys and use flash_window.cu instead.
//     any         fp32, and sizes the other form does not take: one warp per head on CUDA cores.
#include <cooperative_groups.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <float.h>
#include <stdint.h>
#include <string.h>
#include <mutex>

#include "flash_common.cuh"
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar_types.cuh"

namespace cg = cooperative_groups;

namespace e2h {

struct LatentParams {
  void* act;                 // T [n, ld]
  long long ld;
  int off_q, off_c;
  const void* ql;            // T [n, H * rank] absorbed queries
  void* ol;                  // T [n, H * rank] sum_j p_ij c_j
  void* cache;               // T [slots, smax, rank + rot]
  const int* pos;            // [n]
  const int* slot;           // [n]
  int n, slots, smax;
  int H, dim, rank, rot;
  int rank_n;                // columns of the latent that are not filling
  const float* rot_table;    // fp32 [smax, rot / 2, 2]: (cos, sin)
  const float* norm;         // fp32 [rank]
  float eps, scale;
  int window;                // 0: unlimited
  int splits;                // CTAs per cluster
  // latent_prep: rows 0 .. n_ctx - 1 are the context rows of the segments that expand their keys
  // (ctx_src: token, or -1 for an earlier position given by ctx_pos / ctx_slot), the others the
  // tokens n_long .. n - 1
  void* ctx;                 // T [n_ctx, rank + rot]
  const int* ctx_src;
  const int* ctx_pos;
  const int* ctx_slot;
  int n_ctx, n_long;
  int* status;
};

// (cos, sin) pairs cs[0..8) applied to 8 columns
__device__ __forceinline__ void rotate8(float* x, const float* cs) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float u = x[2 * i], v = x[2 * i + 1], c = cs[2 * i], s = cs[2 * i + 1];
    x[2 * i] = u * c - v * s;
    x[2 * i + 1] = v * c + u * s;
  }
}

template <typename T>
__device__ __forceinline__ float latent_rstd(const LatentParams& p, const T* c, float* red) {
  float ss = 0.f;
  for (int i = threadIdx.x * 8; i < p.rank; i += blockDim.x * 8) {
    float x[8];
    load8(c + i, x);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
  }
  return 1.f / sqrtf(block_sum(ss, red) / p.rank_n + p.eps);
}

// 8 columns of a token's cache row: c at its columns `col` normed, or r rotated (col >= rank)
template <typename T>
__device__ __forceinline__ void latent_row8(const LatentParams& p, const T* c, int col, float rstd,
                                            const float* cs, float* x) {
  load8(c + col, x);
  if (col < p.rank) {
    float w[8];
    load8(p.norm + col, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] *= rstd * w[e];
  } else {
    float f[8];
    load8(cs + col - p.rank, f);
    rotate8(x, f);
  }
}

template <typename T>
__device__ __forceinline__ void store8(T* p, const float* v) {
  store4(p, v);
  store4(p + 4, v + 4);
}

template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentParams p) {
  __shared__ float red[33];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int b = blockIdx.x, kd = p.rank + p.rot;
  const bool in_ctx = b < p.n_ctx;
  const int t = in_ctx ? p.ctx_src[b] : p.n_long + b - p.n_ctx;
  if (t >= p.n || (!in_ctx && t < 0)) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  const int pos = t < 0 ? p.ctx_pos[b] : p.pos[t], slot = t < 0 ? p.ctx_slot[b] : p.slot[t];
  if (pos < 0 || pos >= p.smax || slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  T* row = static_cast<T*>(p.cache) + ((long long)slot * p.smax + pos) * kd;
  T* ctx = in_ctx ? static_cast<T*>(p.ctx) + (long long)b * kd : nullptr;
  if (t < 0) {
    const int n = kd * (int)sizeof(T) / 16;
    for (int i = threadIdx.x; i < n; i += 128)
      reinterpret_cast<uint4*>(ctx)[i] = reinterpret_cast<const uint4*>(row)[i];
    return;
  }
  T* act = static_cast<T*>(p.act) + t * p.ld;
  const T* c = act + p.off_c;
  const float* cs = p.rot_table + (long long)pos * p.rot;
  const float rstd = latent_rstd(p, c, red);
  for (int i = threadIdx.x * 8; i < kd; i += 128 * 8) {
    float x[8];
    latent_row8(p, c, i, rstd, cs, x);
    store8(row + i, x);
    if (ctx) store8(ctx + i, x);
  }
  const int per = p.rot / 8;
  for (int i = threadIdx.x; i < p.H * per; i += 128) {
    const int h = i / per, d = (i - h * per) * 8;
    T* q = act + p.off_q + h * (p.dim + p.rot) + p.dim + d;
    float x[8], f[8];
    load8(q, x);
    load8(cs + d, f);
    rotate8(x, f);
    store8(q, x);
  }
}

// ------------------------------------------------------------------ CUDA-core form
constexpr int kLatHeads = 8;       // one warp each
constexpr int kLatKeys = 16;

// NC: 32-wide column groups of the latent
template <typename T, int NC>
__global__ void __launch_bounds__(kLatHeads * 32) latent_attn_kernel(const LatentParams p) {
  extern __shared__ __align__(16) float lat_s[];
  const int kd = p.rank + p.rot, pitch = kd + 4;
  float* q_s = lat_s;                            // [heads][kd]
  float* k_s = q_s + kLatHeads * kd;             // [keys][pitch]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int t = blockIdx.y, h0 = blockIdx.x * kLatHeads;
  const int pos = p.pos[t], slot = p.slot[t];
  if (pos < 0 || pos >= p.smax || slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  const T* act = static_cast<const T*>(p.act) + t * p.ld;
  const float sl2 = p.scale * 1.4426950408889634f;
  for (int i = threadIdx.x * 8; i < kLatHeads * kd; i += kLatHeads * 32 * 8) {
    const int r = i / kd, d = i - r * kd, h = h0 + r;
    float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (h < p.H) {
      if (d < p.rank) load8(static_cast<const T*>(p.ql) + ((long long)t * p.H + h) * p.rank + d, x);
      else load8(act + p.off_q + h * (p.dim + p.rot) + p.dim + (d - p.rank), x);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) q_s[i + e] = x[e] * sl2;
  }
  const T* cache = static_cast<const T*>(p.cache) + (long long)slot * p.smax * kd;
  const int lo = p.window > 0 ? max(pos - p.window + 1, 0) : 0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int key = lane & (kLatKeys - 1), part = lane >> 4;
  float acc[NC], m = -FLT_MAX, l = 0.f;
#pragma unroll
  for (int j = 0; j < NC; ++j) acc[j] = 0.f;
  for (int k0 = lo; k0 <= pos; k0 += kLatKeys) {
    const int cnt = min(kLatKeys, pos + 1 - k0);
    __syncthreads();
    for (int i = threadIdx.x * 8; i < kLatKeys * kd; i += kLatHeads * 32 * 8) {
      const int r = i / kd, d = i - r * kd;
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (r < cnt) load8(cache + (long long)(k0 + r) * kd + d, x);
      store8(k_s + r * pitch + d, x);
    }
    __syncthreads();
    // the two half-warps take alternate groups of four columns
    float s = 0.f;
    const float* q = q_s + warp * kd;
    const float* k = k_s + key * pitch;
    for (int d = part * 4; d < kd; d += 8) {
      float a[4], b[4];
      load4(q + d, a);
      load4(k + d, b);
#pragma unroll
      for (int e = 0; e < 4; ++e) s = fmaf(a[e], b[e], s);
    }
    s += __shfl_xor_sync(0xffffffffu, s, 16);
    if (key >= cnt) s = -FLT_MAX;
    const float mx = fmaxf(m, warp_max(s));
    const float al = exp2f(m - mx);
    const float w = key < cnt ? exp2f(s - mx) : 0.f;
    m = mx;
    l = l * al + warp_sum(part == 0 ? w : 0.f);
#pragma unroll
    for (int j = 0; j < NC; ++j) acc[j] *= al;
    for (int i = 0; i < cnt; ++i) {
      const float wi = __shfl_sync(0xffffffffu, w, i);
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        const int d = lane + 32 * j;
        if (d < p.rank) acc[j] = fmaf(wi, k_s[i * pitch + d], acc[j]);
      }
    }
  }
  const int h = h0 + warp;
  if (h >= p.H) return;
  T* out = static_cast<T*>(p.ol) + ((long long)t * p.H + h) * p.rank;
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    const int d = lane + 32 * j;
    if (d < p.rank) out[d] = from_f<T>(acc[j] / l);
  }
}

// ------------------------------------------------------------------ bf16 form
constexpr int kMmaThreads = 256;
constexpr int kMmaKeys = 64, kMmaRows = 32, kMmaStages = 5;    // keys of a tile; rows of a stage, stages
constexpr int kMmaSmem = 224 * 1024;             // dynamic shared memory; some 2 KB are static
constexpr int kPartPitch = 72, kProbPitch = 72;
constexpr int kMmaBlock = kMmaRows * 128;        // 64 columns of a stage's rows, 128-byte swizzle

__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
      "{%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() {
  asm volatile("cp.async.wait_all;" ::: "memory");
}

// Shared memory of a CTA with R = 16 MT query rows: the ring of key rows, the parts of the scores, the
// probabilities, the token's own row. The query rows start where the parts and probabilities are
// later; the output tile takes the place of the ring.
struct LatentPlan {
  int kd16, pitch;           // row length rounded up to a k-step; distance of query rows (elements), 16
                             // bytes past a multiple of 32 so that ldmatrix rows fall on all banks
  int stage, part, prob, own, total;   // bytes of a stage; byte offsets
  __host__ __device__ LatentPlan(int kd, int rank, int mt) {
    const int R = 16 * mt;
    kd16 = (kd + 15) / 16 * 16;
    pitch = kd16 + 8;
    stage = (kd + 63) / 64 * kMmaBlock;
    part = kMmaStages * stage;
    const int out = R * (rank + 4) * 4;
    if (part < out) part = (out + 1023) / 1024 * 1024;
    prob = part + 4 * R * kPartPitch * 4;
    own = prob + R * kProbPitch * 2;
    const int q = part + R * pitch * 2;
    if (own < q) own = q;
    total = own + kd16 * 2;
  }
};

// Column c of row r of a stage.
__device__ __forceinline__ uint32_t tile_at(uint32_t tile, int r, int c) {
  return tile + (c >> 6) * kMmaBlock + r * 128 + ((((c >> 3) ^ r) & 7) << 4) + (c & 7) * 2;
}

// MT: blocks of 16 query heads; KQ: 16-column steps of a row per warp (a quarter of the row); NP: pairs
// of 8-column tiles of the latent per warp.
//
// TMA fills the ring 32 rows at a time (rows past the last key are read and masked), a stage as soon
// as every warp is past the tile that read it last. Work of the eight warps on a tile of 64 keys:
// scores - warp (quarter of the columns, half of the keys), its query fragments stay in registers; the
// four partial scores of a (head, key) meet in shared memory, where 256 / R threads run the softmax of
// a head; output - warp (1/8 of the latent columns, all keys). Every byte of a cache row is read twice
// from shared memory, once per product. Two barriers per tile.
template <int MT, int KQ, int NP, bool FUSED>
__global__ void __launch_bounds__(kMmaThreads, 1)
latent_attn_mma_kernel(const __grid_constant__ CUtensorMap tm, const int boxes,
                       const LatentParams p) {
  using T = __nv_bfloat16;
  constexpr int R = 16 * MT, TPR = kMmaThreads / R, KPT = kMmaKeys / TPR;
  static_assert(KPT % 4 == 0, "keys of a softmax thread come in fours");
  extern __shared__ __align__(1024) uint8_t lat_raw[];
  uint8_t* lat_b = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lat_raw) + 1023) &
                                              ~uintptr_t(1023));
  __shared__ __align__(8) uint64_t full[kMmaStages];
  __shared__ float red[33];
  __shared__ float alpha_s[R], fin[R][2];
  __shared__ int abort_s;
  const int kd = p.rank + p.rot;
  const LatentPlan plan(kd, p.rank, MT);
  const int pitch = plan.pitch;
  float* part_s = reinterpret_cast<float*>(lat_b + plan.part);
  T* q_s = reinterpret_cast<T*>(lat_b + plan.part);
  T* prob_s = reinterpret_cast<T*>(lat_b + plan.prob);
  T* own_s = reinterpret_cast<T*>(lat_b + plan.own);

  cg::cluster_group cluster = cg::this_cluster();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int s = 0; s < kMmaStages; ++s) mbar_init(smem_u32(&full[s]), 1);
    abort_s = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tm);
  }
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait_prior();

  const int rank = blockIdx.x, h0 = blockIdx.y * R, t = blockIdx.z;
  const int nr = min(R, p.H - h0);
  const bool has_own = FUSED && rank == p.splits - 1;   // holds the token's own key
  const T* act = static_cast<const T*>(p.act) + t * p.ld;
  // every load that does not depend on the position first: indices, query rows, own latent, norm
  int pos = p.pos[t], slot = p.slot[t];
  const int qv = p.rank / 8;
  for (int i = tid; i < nr * qv; i += kMmaThreads) {
    const int r = i / qv, d = (i - r * qv) * 8;
    cp_async16(smem_u32(q_s + r * pitch + d),
               static_cast<const T*>(p.ql) + ((long long)t * p.H + h0 + r) * p.rank + d);
  }
  const int per = (plan.kd16 - p.rank) / 8;      // pieces of a query row behind the latent columns
  auto piece = [&](int i, int& r, int& d) -> const T* {
    r = i / max(per, 1);
    d = (i - r * per) * 8;
    return i < R * per && r < nr && d < p.rot
               ? act + p.off_q + (h0 + r) * (p.dim + p.rot) + p.dim + d : nullptr;
  };
  int r0, d0;
  const T* src0 = piece(tid, r0, d0);
  const uint4 zero4 = make_uint4(0, 0, 0, 0);
  const uint4 x0 = src0 ? *reinterpret_cast<const uint4*>(src0) : zero4;
  const int oc = tid * 8;                        // columns of the own row (at most 576)
  float own[8], wn[8];
  if (has_own && oc < kd) {
    load8(act + p.off_c + oc, own);
    if (oc < p.rank) load8(p.norm + oc, wn);
  }

  const bool ok = pos >= 0 && pos < p.smax && slot >= 0 && slot < p.slots;
  if (!ok) {                                     // indices come from device memory
    if (tid == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    pos = min(max(pos, 0), p.smax - 1);
    slot = min(max(slot, 0), p.slots - 1);
  }
  // keys lo .. pos, split over the cluster
  const int lo = p.window > 0 ? max(pos - p.window + 1, 0) : 0;
  const int n_keys = pos + 1 - lo;
  const int k_begin = lo + (int)((long long)n_keys * rank / p.splits);
  const int k_end = lo + (int)((long long)n_keys * (rank + 1) / p.splits);
  const int n_loads = (k_end - k_begin + kMmaRows - 1) / kMmaRows;
  const int n_tiles = (k_end - k_begin + kMmaKeys - 1) / kMmaKeys;
  auto load = [&](int i) {                       // thread 0
    const int s = i % kMmaStages;
    const uint32_t bar = smem_u32(&full[s]);
    mbar_expect_tx(bar, plan.stage);
    for (int b = 0; b < boxes; ++b)              // one box for all columns if they are whole blocks
      tma_load_3d(smem_u32(lat_b + s * plan.stage + b * kMmaBlock), &tm, b * 64,
                  slot * p.smax + k_begin + i * kMmaRows, 0, bar);
  };
  if (tid == 0)
    for (int i = 0; i < min(n_loads, kMmaStages); ++i) load(i);

  const float* cs = p.rot_table + (long long)pos * p.rot;
  float f0[8], fo[8];
  if (FUSED && src0) load8(cs + d0, f0);
  if (has_own && oc >= p.rank && oc < kd) load8(cs + oc - p.rank, fo);
  auto put = [&](int r, int d, bool live, uint4 x, const float* f) {
    if (FUSED && live) {
      float v[8];
      load8(reinterpret_cast<const T*>(&x), v);
      rotate8(v, f);
      store8(reinterpret_cast<T*>(&x), v);
    }
    *reinterpret_cast<uint4*>(q_s + r * pitch + p.rank + d) = x;
  };
  if (tid < R * per) put(r0, d0, src0 != nullptr, x0, f0);
  for (int i = tid + kMmaThreads; i < R * per; i += kMmaThreads) {
    int r, d;
    const T* src = piece(i, r, d);
    float f[8];
    if (FUSED && src) load8(cs + d, f);
    put(r, d, src != nullptr, src ? *reinterpret_cast<const uint4*>(src) : zero4, f);
  }
  for (int i = nr * qv + tid; i < R * qv; i += kMmaThreads) {
    const int r = i / qv, d = (i - r * qv) * 8;
    *reinterpret_cast<uint4*>(q_s + r * pitch + d) = zero4;
  }
  if (has_own) {
    float ss = 0.f;
    if (oc < p.rank) {
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += own[e] * own[e];
    }
    const float rstd = 1.f / sqrtf(block_sum(ss, red) / p.rank_n + p.eps);
    if (oc < kd) {
      if (oc < p.rank) {
#pragma unroll
        for (int e = 0; e < 8; ++e) own[e] *= rstd * wn[e];
      } else {
        rotate8(own, fo);
      }
      store8(own_s + oc, own);
      if (ok && blockIdx.y == 0)
        store8(static_cast<T*>(p.cache) + ((long long)slot * p.smax + pos) * kd + oc, own);
    }
  }
  cp_async_wait_all();
  __syncthreads();

  const int op = p.rank + 4;                     // row distance of the output tile
  float* out_s = reinterpret_cast<float*>(lat_b);
  const int ks = plan.kd16 / 16, kq = warp >> 1, kh = warp & 1;   // column quarter, key half
  const int per_q = (ks + 3) / 4;
  const int s_begin = kq * per_q, s_count = max(0, min(per_q, ks - s_begin));
  const int c8_last = ks * 2 - 2;                // steps past the row repeat its end, times zero
  uint32_t qf[KQ][MT][4];
  const int lr = lane & 7, lt = lane >> 3;       // row and tile of this lane's ldmatrix address
#pragma unroll
  for (int s = 0; s < KQ; ++s)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      if (s < s_count) {
        ldsm4(qf[s][mt], smem_u32(q_s + (mt * 16 + (lt & 1) * 8 + lr) * pitch +
                                  (s_begin + s) * 16 + (lt >> 1) * 8));
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) qf[s][mt][e] = 0;
      }
    }
  float acc[MT][NP][2][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int b = 0; b < NP; ++b)
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[a][b][c][e] = 0.f;
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  const int row = tid / TPR, sub = tid % TPR;  // softmax: head, keys 4 sub .., 4 (sub + TPR) ..
  const int n_pairs = (p.rank + 15) / 16;
  const float sl2 = p.scale * 1.4426950408889634f;
  float m = -FLT_MAX, l = 0.f;
  __syncthreads();                        // the query rows give way to the score parts

  int st[2] = {0, 1};                          // stages of the tile's halves
  uint32_t ph[2] = {0, 0};
  for (int it = 0; it < n_tiles; ++it) {
    const int cnt = min(kMmaKeys, k_end - k_begin - it * kMmaKeys);
    const bool two = cnt > kMmaRows;           // the second half was loaded
    const uint32_t half[2] = {smem_u32(lat_b + st[0] * plan.stage),
                              smem_u32(lat_b + st[1] * plan.stage)};
    mbar_wait(smem_u32(&full[st[0]]), ph[0], &abort_s, p.status, kStatusTimeoutFull);
    if (two) mbar_wait(smem_u32(&full[st[1]]), ph[1], &abort_s, p.status, kStatusTimeoutFull);
    if (has_own && it == n_tiles - 1) {        // the token's own row
      const uint32_t base = two ? half[1] : half[0];
      for (int i = tid; i < kd / 8; i += kMmaThreads)
        *reinterpret_cast<uint4*>(lat_b + (tile_at(base, (cnt - 1) % kMmaRows, i * 8) -
                                           smem_u32(lat_b))) =
            *reinterpret_cast<const uint4*>(own_s + i * 8);
      __syncthreads();
    }
    float sc[MT][4][4];
#pragma unroll
    for (int a = 0; a < MT; ++a)
#pragma unroll
      for (int b = 0; b < 4; ++b)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[a][b][e] = 0.f;
    if (kh == 0 || two) {
      const uint32_t krow = (kh ? half[1] : half[0]) + ((lt >> 1) * 8 + lr) * 128;
#pragma unroll
      for (int s = 0; s < KQ; ++s) {
        const int c8 = min((s_begin + s) * 2, c8_last) + (lt & 1);   // 8-column group
        const uint32_t a = krow + (c8 >> 3) * kMmaBlock + (((c8 ^ lr) & 7) << 4);
        uint32_t b[2][4];
        ldsm4(b[0], a);
        ldsm4(b[1], a + 16 * 128);
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma16816(sc[mt][2 * x], qf[s][mt], b[x][0], b[x][1]);
            mma16816(sc[mt][2 * x + 1], qf[s][mt], b[x][2], b[x][3]);
          }
      }
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        float* d = part_s + (kq * R + mt * 16 + g) * kPartPitch + kh * 32 + b * 8 + c2;
        *reinterpret_cast<float2*>(d) = make_float2(sc[mt][b][0], sc[mt][b][1]);
        *reinterpret_cast<float2*>(d + 8 * kPartPitch) = make_float2(sc[mt][b][2], sc[mt][b][3]);
      }
    __syncthreads();
    if (tid == 0 && it > 0)                      // everyone is done with the tile before
      for (int i = 2 * it + kMmaStages - 2; i < min(2 * it + kMmaStages, n_loads); ++i) load(i);
    {
      float s[KPT], mx = m;
#pragma unroll
      for (int i = 0; i < KPT / 4; ++i) {
        const int k = 4 * (sub + TPR * i);
        float a[4][4];
#pragma unroll
        for (int x = 0; x < 4; ++x) load4(part_s + (x * R + row) * kPartPitch + k, a[x]);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float v = (a[0][e] + a[1][e]) + (a[2][e] + a[3][e]);
          s[4 * i + e] = k + e < cnt ? v * sl2 : -FLT_MAX;
          mx = fmaxf(mx, s[4 * i + e]);
        }
      }
#pragma unroll
      for (int o = TPR / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float al = ex2_approx(m - mx);     // a tile has at least one key: mx is a score
      m = mx;
      l *= al;
      if (sub == 0) alpha_s[row] = al;
#pragma unroll
      for (int i = 0; i < KPT / 4; ++i) {
        float w[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          w[e] = ex2_approx(s[4 * i + e] - mx);
          l += w[e];
        }
        store4(prob_s + row * kProbPitch + 4 * (sub + TPR * i), w);
      }
    }
    __syncthreads();
    float al[MT][2];
    bool scale = false;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        al[mt][e] = alpha_s[mt * 16 + e * 8 + g];
        scale |= al[mt][e] != 1.f;
      }
    if (__any_sync(0xffffffffu, scale)) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int j = 0; j < NP; ++j)
#pragma unroll
          for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[mt][j][c][e] *= al[mt][e >> 1];
    }
#pragma unroll
    for (int kk = 0; kk < kMmaKeys / 16; ++kk) {
      if (kk * 16 >= cnt) continue;            // (rows that were not loaded are not numbers)
      const uint32_t vrow = half[kk >> 1] + ((kk & 1) * 16 + (lt & 1) * 8 + lr) * 128;
      uint32_t pf[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        ldsm4(pf[mt], smem_u32(prob_s + (mt * 16 + (lt & 1) * 8 + lr) * kProbPitch + kk * 16 +
                               (lt >> 1) * 8));
      uint32_t b[NP][4];
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int c8 = min(warp + 8 * j, n_pairs - 1) * 2 + (lt >> 1);
        ldsm4_t(b[j], vrow + (c8 >> 3) * kMmaBlock + (((c8 ^ lr) & 7) << 4));
      }
#pragma unroll
      for (int j = 0; j < NP; ++j)
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma16816(acc[mt][j][0], pf[mt], b[j][0], b[j][1]);
          mma16816(acc[mt][j][1], pf[mt], b[j][2], b[j][3]);
        }
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      st[x] += 2;
      if (st[x] >= kMmaStages) {
        st[x] -= kMmaStages;
        ph[x] ^= 1;
      }
    }
  }
#pragma unroll
  for (int o = TPR / 2; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  if (sub == 0) {
    fin[row][0] = m;
    fin[row][1] = l;
  }
  __syncthreads();                               // every stage has been read
  if (abort_s) {                                 // bounded wait for copies still in flight
    for (int i = max(n_loads - kMmaStages, 0); i < n_loads; ++i) {
      const long long tq = clock64();
      while (!mbar_try_wait(smem_u32(&full[i % kMmaStages]), (i / kMmaStages) & 1))
        if (clock64() - tq > kWaitLimitCycles / 8) break;
    }
    __syncthreads();
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int j = 0; j < NP; ++j)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int col = (warp + 8 * j) * 16 + c * 8 + c2;
        if (col < p.rank) {
          float* d = out_s + (mt * 16 + g) * op + col;
          *reinterpret_cast<float2*>(d) = make_float2(acc[mt][j][c][0], acc[mt][j][c][1]);
          *reinterpret_cast<float2*>(d + 8 * op) = make_float2(acc[mt][j][c][2], acc[mt][j][c][3]);
        }
      }

  // the CTA's sums, then the cluster's: every CTA finishes its share of the columns
  if (p.splits > 1) cluster.sync();
  else __syncthreads();
  // a warp per head: lane k fetches (m, l) of CTA k, then the lanes walk the columns
  T* out = static_cast<T*>(p.ol) + ((long long)t * p.H + h0) * p.rank;
  for (int r = rank + p.splits * warp; r < nr; r += p.splits * (kMmaThreads / 32)) {
    float mk = -FLT_MAX, lk = 0.f;
    if (lane < p.splits) {
      const float* f = cluster.map_shared_rank(&fin[r][0], lane);
      mk = f[0];
      lk = f[1];
    }
    const float w = exp2f(mk - warp_max(mk));
    const float wn_ = w / warp_sum(w * lk);
    constexpr int U = (NP * 128 + 127) / 128;    // 128 columns per pass of the warp
    float4 o[U];
#pragma unroll
    for (int u = 0; u < U; ++u) o[u] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 2
    for (int k = 0; k < p.splits; ++k) {
      const float* src = (p.splits > 1 ? cluster.map_shared_rank(out_s, k) : out_s) + r * op;
      const float x = __shfl_sync(0xffffffffu, wn_, k);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = u * 128 + lane * 4;
        if (c < p.rank) {
          const float4 a = *reinterpret_cast<const float4*>(src + c);
          o[u].x = fmaf(x, a.x, o[u].x);
          o[u].y = fmaf(x, a.y, o[u].y);
          o[u].z = fmaf(x, a.z, o[u].z);
          o[u].w = fmaf(x, a.w, o[u].w);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = u * 128 + lane * 4;
      if (c < p.rank) store4(out + (long long)r * p.rank + c, reinterpret_cast<const float*>(&o[u]));
    }
  }
  if (p.splits > 1) cluster.sync();              // peers may still read this CTA's shared memory
}

// Rows of kd columns; a box brings kMmaRows of them, 64 columns wide, or (whole) all blocks of 64 columns
// one after the other.
static int latent_map(CUtensorMap* m, const void* base, int kd, long long rows, bool whole) {
  EncodeTiledFn fn = flash_encode_fn();
  if (!fn) return -10;
  cuuint64_t dims[3] = {whole ? 64u : (cuuint64_t)kd, (cuuint64_t)rows,
                        whole ? (cuuint64_t)(kd / 64) : 1u};
  cuuint64_t strides[2] = {(cuuint64_t)kd * 2, whole ? 128u : (cuuint64_t)(rows * kd * 2)};
  cuuint32_t box[3] = {64u, (cuuint32_t)kMmaRows, (cuuint32_t)dims[2]};
  cuuint32_t estr[3] = {1u, 1u, 1u};
  const CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims,
                        strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                        CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -11;
}

template <int MT, int KQ, int NP, bool FUSED>
static int latent_mma_launch(const LatentParams& p, cudaStream_t stream) {
  const int kd = p.rank + p.rot;
  const LatentPlan plan(kd, p.rank, MT);
  if (plan.total + 1024 > kMmaSmem) return -2;
  // the cache as rows of kd columns
  CUtensorMap tm;
  const long long rows = (long long)p.slots * p.smax;
  if (rows > 0x7fffffff) return -2;
  const int boxes = kd % 64 ? (kd + 63) / 64 : 1;
  const int r = latent_map(&tm, p.cache, kd, rows, kd % 64 == 0);
  if (r) return r;
  auto kern = latent_attn_mma_kernel<MT, KQ, NP, FUSED>;
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [&] {
    err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMmaSmem);
  });
  if (err != cudaSuccess) return (int)err;
  cudaLaunchConfig_t cfg;
  memset(&cfg, 0, sizeof(cfg));
  cfg.gridDim = dim3(p.splits, (p.H + 16 * MT - 1) / (16 * MT), p.n);
  cfg.blockDim = dim3(kMmaThreads);
  cfg.dynamicSmemBytes = plan.total + 1024;      // alignment slack
  cfg.stream = stream;
  cudaLaunchAttribute attrs[2];
  int na = 0;
  attrs[na].id = cudaLaunchAttributeClusterDimension;
  attrs[na].val.clusterDim.x = p.splits;
  attrs[na].val.clusterDim.y = 1;
  attrs[na].val.clusterDim.z = 1;
  ++na;
  if (g_pdl) {
    attrs[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attrs[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  cfg.attrs = attrs;
  cfg.numAttrs = na;
  return (int)cudaLaunchKernelEx(&cfg, kern, tm, boxes, p);
}

template <int MT>
static int latent_mma_pick(const LatentParams& p, bool fused, cudaStream_t s) {
  const int kd = p.rank + p.rot;
  if (kd <= 192 && p.rank <= 128)
    return fused ? latent_mma_launch<MT, 3, 1, true>(p, s) : latent_mma_launch<MT, 3, 1, false>(p, s);
  if (kd <= 384 && p.rank <= 384)
    return fused ? latent_mma_launch<MT, 6, 3, true>(p, s) : latent_mma_launch<MT, 6, 3, false>(p, s);
  return fused ? latent_mma_launch<MT, 9, 4, true>(p, s) : latent_mma_launch<MT, 9, 4, false>(p, s);
}

template <typename T, int NC>
static int latent_any_launch(const LatentParams& p, cudaStream_t stream) {
  const int kd = p.rank + p.rot;
  const size_t smem = sizeof(float) * (kLatHeads * kd + kLatKeys * (kd + 4));
  if (smem > 200 * 1024) return -2;
  auto kern = latent_attn_kernel<T, NC>;
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [&] {
    err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  });
  if (err != cudaSuccess) return (int)err;
  return (int)launch(kern, dim3((p.H + kLatHeads - 1) / kLatHeads, p.n), dim3(kLatHeads * 32), smem,
                     stream, p);
}

template <typename T>
static int latent_any(const LatentParams& p, cudaStream_t s) {
  if (p.rank <= 128) return latent_any_launch<T, 4>(p, s);
  if (p.rank <= 512) return latent_any_launch<T, 16>(p, s);
  return latent_any_launch<T, 32>(p, s);
}

static int latent_check(const LatentParams& p) {
  if (p.n <= 0 || p.H <= 0 || p.dim <= 0 || p.rank <= 0 || p.rot < 0 || p.rank > 1024 ||
      p.rank_n <= 0 || p.window < 0 || !p.status)
    return -1;
  if ((p.dim | p.rank | p.rot | p.off_q | p.off_c) % 8 || p.ld % 8) return -1;
  if ((reinterpret_cast<uintptr_t>(p.act) | reinterpret_cast<uintptr_t>(p.cache) |
       reinterpret_cast<uintptr_t>(p.norm) | reinterpret_cast<uintptr_t>(p.rot_table)) & 15)
    return -3;
  return 0;
}

}  // namespace e2h

extern "C" int e2h_latent_prep(const e2h::LatentParams* p, int is_bf16, void* stream) {
  using namespace e2h;
  const int r = latent_check(*p);
  if (r) return r;
  if (p->n_ctx < 0 || p->n_long < 0 || p->n_long > p->n ||
      (p->n_ctx > 0 && (!p->ctx || !p->ctx_src || !p->ctx_pos || !p->ctx_slot)))
    return -1;
  const int rows = p->n_ctx + p->n - p->n_long;
  if (rows <= 0) return 0;
  return is_bf16 ? (int)launch(latent_prep_kernel<__nv_bfloat16>, dim3(rows), dim3(128), 0,
                               (cudaStream_t)stream, *p)
                 : (int)launch(latent_prep_kernel<float>, dim3(rows), dim3(128), 0,
                               (cudaStream_t)stream, *p);
}

// Tokens n_long .. n - 1 (ql, ol: rows of these tokens only). fused: one token per sequence,
// projections as the GEMM left them (bf16, rank <= 512, rank + rot <= 576); otherwise latent_prep ran.
extern "C" int e2h_latent_attn(const e2h::LatentParams* p, int fused, int is_bf16, void* stream_v) {
  using namespace e2h;
  int r = latent_check(*p);
  if (r) return r;
  if (!p->ql || !p->ol || p->splits < 1 || p->splits > 8 || p->n_long < 0) return -1;
  if ((reinterpret_cast<uintptr_t>(p->ql) | reinterpret_cast<uintptr_t>(p->ol)) & 15) return -3;
  cudaStream_t stream = (cudaStream_t)stream_v;
  const long long es = is_bf16 ? 2 : 4;
  const bool mma = is_bf16 && p->rank <= 512 && p->rank + p->rot <= 576;
  if (fused && !mma) return -2;
  for (int t0 = p->n_long; t0 < p->n; t0 += 65535) {   // grid.z / grid.y hold 65535 tokens
    LatentParams q = *p;
    q.n = p->n - t0 < 65535 ? p->n - t0 : 65535;
    q.pos = p->pos + t0;
    q.slot = p->slot + t0;
    q.act = static_cast<char*>(p->act) + t0 * p->ld * es;
    const long long o = (long long)(t0 - p->n_long) * p->H * p->rank * es;
    q.ql = static_cast<const char*>(p->ql) + o;
    q.ol = static_cast<char*>(p->ol) + o;
    if (mma)
      r = p->H <= 16 ? latent_mma_pick<1>(q, fused != 0, stream)
                     : latent_mma_pick<2>(q, fused != 0, stream);
    else
      r = is_bf16 ? latent_any<__nv_bfloat16>(q, stream) : latent_any<float>(q, stream);
    if (r) return r;
  }
  return 0;
}
