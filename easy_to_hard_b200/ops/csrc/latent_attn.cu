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
//     bf16        warp-level matrix products on a ring of cache rows that bulk copies fill. A token
//                 brings at most 16 or 32 query rows, far below a tcgen05 tile, and the kernel is a
//                 stream of the cache; in its fused form (decode) it also does the work of
//                 latent_prep. Prompts expand the keys and use flash_window.cu instead.
//     any         fp32, and sizes the other form does not take: one warp per head on CUDA cores.
#include <cooperative_groups.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <float.h>
#include <stdint.h>
#include <string.h>
#include <mutex>

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
constexpr int kMmaThreads = 256, kMmaKeys = 64, kPartPitch = 72, kProbPitch = 72;

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
// stream: the row is read once per step (L2 evict-first)
__device__ __forceinline__ void bulk_row(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar,
                                         bool stream, uint64_t policy) {
  if (stream)
    asm volatile(
        "cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint "
        "[%0], [%1], %2, [%3], %4;"
        ::"r"(dst), "l"(src), "r"(bytes), "r"(bar), "l"(policy)
        : "memory");
  else
    asm volatile(
        "cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
        ::"r"(dst), "l"(src), "r"(bytes), "r"(bar)
        : "memory");
}

// Shared memory of a CTA with R = 16 MT query rows.
struct LatentPlan {
  int kd16, pitch;           // row length rounded up to a k-step; row distance (elements), 16 bytes
                             // past a multiple of 32 so that ldmatrix rows fall on all banks
  int stage, part, prob, nk, total;   // byte offsets
  __host__ __device__ LatentPlan(int kd, int rank, int mt) {
    const int R = 16 * mt;
    kd16 = (kd + 15) / 16 * 16;
    pitch = kd16 + 8;
    stage = 0;
    int end = 2 * kMmaKeys * pitch * 2;
    const int out = R * (rank + 4) * 4;           // the output tile takes the place of the ring
    if (end < out) end = out;
    part = (end + 15) / 16 * 16;                  // score parts; the query rows before them
    prob = part + 4 * R * kPartPitch * 4;
    nk = prob + R * kProbPitch * 2;
    const int q = part + R * pitch * 2;
    if (nk < q) nk = q;
    total = nk + pitch * 2;
  }
};

// MT: blocks of 16 query heads; KQ: 16-column steps of a row per warp (a quarter of the row); NP: pairs
// of 8-column tiles of the latent per warp.
//
// Work of the eight warps on a tile of 64 keys: scores - warp (quarter of the columns, half of the
// keys), its query fragments stay in registers; the four partial scores of a (head, key) meet in
// shared memory, where 256 / R threads run the softmax of a head; output - warp (1/8 of the latent
// columns, all keys). Every byte of a cache row is read twice from shared memory, once per product.
template <int MT, int KQ, int NP, bool FUSED>
__global__ void __launch_bounds__(kMmaThreads, 1) latent_attn_mma_kernel(const LatentParams p) {
  using T = __nv_bfloat16;
  constexpr int R = 16 * MT, TPR = kMmaThreads / R, KPT = kMmaKeys / TPR;
  extern __shared__ __align__(128) uint8_t lat_b[];
  __shared__ __align__(8) uint64_t full[2];
  __shared__ float red[33];
  __shared__ float alpha_s[R], fin[R][2];
  __shared__ int abort_s;
  const int kd = p.rank + p.rot;
  const LatentPlan plan(kd, p.rank, MT);
  const int pitch = plan.pitch;
  T* ring = reinterpret_cast<T*>(lat_b + plan.stage);
  float* part_s = reinterpret_cast<float*>(lat_b + plan.part);
  T* q_s = reinterpret_cast<T*>(lat_b + plan.part);
  T* prob_s = reinterpret_cast<T*>(lat_b + plan.prob);
  T* new_s = reinterpret_cast<T*>(lat_b + plan.nk);

  cg::cluster_group cluster = cg::this_cluster();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    mbar_init(smem_u32(&full[0]), 1);
    mbar_init(smem_u32(&full[1]), 1);
    abort_s = 0;
    fence_mbar_init();
  }
  // columns past a row's end are multiplied by zero: they have to be numbers
  for (int i = tid; i < 2 * kMmaKeys; i += kMmaThreads)
    for (int d = kd; d < pitch; d += 8)
      *reinterpret_cast<uint4*>(ring + i * pitch + d) = make_uint4(0, 0, 0, 0);
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait_prior();

  const int rank = blockIdx.x, h0 = blockIdx.y * R, t = blockIdx.z;
  const int nr = min(R, p.H - h0);
  int pos = p.pos[t], slot = p.slot[t];
  const bool ok = pos >= 0 && pos < p.smax && slot >= 0 && slot < p.slots;
  if (!ok) {                                     // indices come from device memory
    if (tid == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    pos = min(max(pos, 0), p.smax - 1);
    slot = min(max(slot, 0), p.slots - 1);
  }
  T* cache = static_cast<T*>(p.cache) + (long long)slot * p.smax * kd;
  const T* act = static_cast<const T*>(p.act) + t * p.ld;
  const float* cs = p.rot_table + (long long)pos * p.rot;
  const float sl2 = p.scale * 1.4426950408889634f;

  // keys lo .. pos, split over the cluster; the fused form holds the last one itself
  const int lo = p.window > 0 ? max(pos - p.window + 1, 0) : 0;
  const int n_keys = pos + 1 - lo;
  const int k_begin = lo + (int)((long long)n_keys * rank / p.splits);
  const int k_end = lo + (int)((long long)n_keys * (rank + 1) / p.splits);
  const int n_tiles = (k_end - k_begin + kMmaKeys - 1) / kMmaKeys;
  const bool has_new = FUSED && rank == p.splits - 1;
  const bool stream = FUSED && gridDim.y == 1;
  const uint64_t policy = policy_evict_first();
  auto load_tile = [&](int it) {                 // warp 0
    const int k0 = k_begin + it * kMmaKeys;
    const int rows = min(kMmaKeys, k_end - (has_new ? 1 : 0) - k0);
    const uint32_t bar = smem_u32(&full[it & 1]);
    if (lane == 0) mbar_expect_tx(bar, max(rows, 0) * kd * 2);
    __syncwarp();
    const uint32_t dst = smem_u32(ring + (it & 1) * kMmaKeys * pitch);
    for (int r = lane; r < rows; r += 32)
      bulk_row(dst + r * pitch * 2, cache + (long long)(k0 + r) * kd, kd * 2, bar, stream,
               policy);
  };
  if (warp == 0) {
    if (n_tiles > 0) load_tile(0);
    if (n_tiles > 1) load_tile(1);
  }

  // query rows, rotated part included
  for (int i = tid; i < R * (plan.kd16 / 8); i += kMmaThreads) {
    const int r = i / (plan.kd16 / 8), d = (i - r * (plan.kd16 / 8)) * 8, h = h0 + r;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (r < nr && d < kd) {
      if (d < p.rank) {
        x = *reinterpret_cast<const uint4*>(static_cast<const T*>(p.ql) +
                                            ((long long)t * p.H + h) * p.rank + d);
      } else {
        const T* src = act + p.off_q + h * (p.dim + p.rot) + p.dim + (d - p.rank);
        if constexpr (FUSED) {
          float v[8], f[8];
          load8(src, v);
          load8(cs + d - p.rank, f);
          rotate8(v, f);
          store8(reinterpret_cast<T*>(&x), v);
        } else {
          x = *reinterpret_cast<const uint4*>(src);
        }
      }
    }
    *reinterpret_cast<uint4*>(q_s + r * pitch + d) = x;
  }
  if (has_new) {
    const T* c = act + p.off_c;
    const float rstd = latent_rstd(p, c, red);
    for (int i = tid * 8; i < plan.kd16; i += kMmaThreads * 8) {
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (i < kd) latent_row8(p, c, i, rstd, cs, x);
      store8(new_s + i, x);
      if (ok && blockIdx.y == 0 && i < kd) store8(cache + (long long)pos * kd + i, x);
    }
  }
  __syncthreads();

  const int ks = plan.kd16 / 16, kq = warp >> 1, kh = warp & 1;   // column quarter, key half
  const int per_q = (ks + 3) / 4;
  const int s_begin = kq * per_q, s_count = max(0, min(per_q, ks - s_begin));
  uint32_t qf[KQ][MT][4];
  const int lr = lane & 7, lt = lane >> 3;       // row and tile of this lane's ldmatrix address
#pragma unroll
  for (int s = 0; s < KQ; ++s)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      if (s < s_count) {
        ldsm4(qf[s][mt], smem_u32(q_s + (mt * 16 + (lt & 1) * 8 + lr) * pitch + (s_begin + s) * 16 +
                                  (lt >> 1) * 8));
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
  const int row = tid / TPR, sub = tid % TPR;    // softmax: head, keys sub, sub + TPR, ...
  const int n_pairs = (p.rank + 15) / 16;
  float m = -FLT_MAX, l = 0.f;
  __syncthreads();                               // the query rows give way to the score parts

  for (int it = 0; it < n_tiles; ++it) {
    T* tile = ring + (it & 1) * kMmaKeys * pitch;
    const int k0 = k_begin + it * kMmaKeys;
    const int cnt = min(kMmaKeys, k_end - k0);
    mbar_wait(smem_u32(&full[it & 1]), (it >> 1) & 1, &abort_s, p.status, kStatusTimeoutFull);
    if (it == n_tiles - 1 && (cnt < kMmaKeys || has_new)) {
      const int per = plan.kd16 / 8;             // the token's own row, zeros behind the last key
      for (int i = tid; i < (kMmaKeys - cnt + 1) * per; i += kMmaThreads) {
        const int r = i / per, d = (i - r * per) * 8;
        if (r > 0)
          *reinterpret_cast<uint4*>(tile + (cnt - 1 + r) * pitch + d) = make_uint4(0, 0, 0, 0);
        else if (has_new)
          *reinterpret_cast<uint4*>(tile + (cnt - 1) * pitch + d) =
              *reinterpret_cast<const uint4*>(new_s + d);
      }
      __syncthreads();
    }
    float sc[MT][4][4];
#pragma unroll
    for (int a = 0; a < MT; ++a)
#pragma unroll
      for (int b = 0; b < 4; ++b)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[a][b][e] = 0.f;
#pragma unroll
    for (int s = 0; s < KQ; ++s) {
      if (s < s_count) {
        const T* col = tile + (kh * 32 + (lt >> 1) * 8 + lr) * pitch + (s_begin + s) * 16 +
                       (lt & 1) * 8;
#pragma unroll
        for (int h = 0; h < 2; ++h) {            // 16 keys each
          uint32_t b[4];
          ldsm4(b, smem_u32(col + h * 16 * pitch));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma16816(sc[mt][2 * h], qf[s][mt], b[0], b[1]);
            mma16816(sc[mt][2 * h + 1], qf[s][mt], b[2], b[3]);
          }
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
    {
      float s[KPT], mx = m;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const int k = sub + TPR * i;
        const float* d = part_s + row * kPartPitch + k;
        s[i] = (d[0] + d[R * kPartPitch]) + (d[2 * R * kPartPitch] + d[3 * R * kPartPitch]);
        s[i] = k < cnt ? s[i] * sl2 : -FLT_MAX;
        mx = fmaxf(mx, s[i]);
      }
#pragma unroll
      for (int o = TPR / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float al = exp2f(m - mx);
      m = mx;
      l *= al;
      if (sub == 0) alpha_s[row] = al;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const int k = sub + TPR * i;
        const float w = k < cnt ? exp2f(s[i] - mx) : 0.f;
        l += w;
        prob_s[row * kProbPitch + k] = __float2bfloat16_rn(w);
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
      uint32_t pf[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        ldsm4(pf[mt], smem_u32(prob_s + (mt * 16 + (lt & 1) * 8 + lr) * kProbPitch + kk * 16 +
                               (lt >> 1) * 8));
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int pair = warp + 8 * j;
        if (pair < n_pairs) {
          uint32_t b[4];
          ldsm4_t(b, smem_u32(tile + (kk * 16 + (lt & 1) * 8 + lr) * pitch + pair * 16 +
                              (lt >> 1) * 8));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma16816(acc[mt][j][0], pf[mt], b[0], b[1]);
            mma16816(acc[mt][j][1], pf[mt], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();                             // everyone is done with this tile and the parts
    if (warp == 0 && it + 2 < n_tiles) {
      fence_proxy_async_smem();
      load_tile(it + 2);
    }
  }

  if (abort_s) {                                 // bounded wait for copies still in flight
    for (int it = max(n_tiles - 2, 0); it < n_tiles; ++it) {
      const long long tq = clock64();
      while (!mbar_try_wait(smem_u32(&full[it & 1]), (it >> 1) & 1))
        if (clock64() - tq > kWaitLimitCycles / 8) break;
    }
    __syncthreads();
  }

  // the CTA's (m, l) and sums, then the cluster's: every CTA finishes its share of the columns
#pragma unroll
  for (int o = TPR / 2; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  if (sub == 0) {
    fin[row][0] = m;
    fin[row][1] = l;
  }
  const int op = p.rank + 4;
  float* out_s = reinterpret_cast<float*>(lat_b);
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
  if (p.splits > 1) cluster.sync();
  else __syncthreads();
  const int vec = p.rank / 4, total = nr * vec;
  const int per = (total + p.splits - 1) / p.splits;
  for (int i = rank * per + tid; i < min(total, (rank + 1) * per); i += kMmaThreads) {
    const int r = i / vec, d = (i - r * vec) * 4;
    float o[4] = {0.f, 0.f, 0.f, 0.f}, ls = 0.f, mx = -FLT_MAX;
    if (p.splits > 1) {
      for (int k = 0; k < p.splits; ++k)
        mx = fmaxf(mx, cluster.map_shared_rank(&fin[r][0], k)[0]);
      for (int k = 0; k < p.splits; ++k) {
        const float* f = cluster.map_shared_rank(&fin[r][0], k);
        const float w = exp2f(f[0] - mx);
        const float4 a = *reinterpret_cast<const float4*>(cluster.map_shared_rank(out_s, k) +
                                                          r * op + d);
        ls += w * f[1];
        o[0] += w * a.x;
        o[1] += w * a.y;
        o[2] += w * a.z;
        o[3] += w * a.w;
      }
    } else {
      load4(out_s + r * op + d, o);
      ls = fin[r][1];
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] /= ls;
    store4(static_cast<T*>(p.ol) + ((long long)t * p.H + h0 + r) * p.rank + d, o);
  }
  if (p.splits > 1) cluster.sync();              // peers may still read this CTA's shared memory
}

template <int MT, int KQ, int NP, bool FUSED>
static int latent_mma_launch(const LatentParams& p, cudaStream_t stream) {
  const LatentPlan plan(p.rank + p.rot, p.rank, MT);
  if (plan.total > 220 * 1024) return -2;
  auto kern = latent_attn_mma_kernel<MT, KQ, NP, FUSED>;
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [&] {
    err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  });
  if (err != cudaSuccess) return (int)err;
  cudaLaunchConfig_t cfg;
  memset(&cfg, 0, sizeof(cfg));
  cfg.gridDim = dim3(p.splits, (p.H + 16 * MT - 1) / (16 * MT), p.n);
  cfg.blockDim = dim3(kMmaThreads);
  cfg.dynamicSmemBytes = plan.total;
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
  return (int)cudaLaunchKernelEx(&cfg, kern, p);
}

template <int MT>
static int latent_mma_pick(const LatentParams& p, bool fused, cudaStream_t s) {
  const int kd = p.rank + p.rot;
  if (kd <= 192 && p.rank <= 128)
    return fused ? latent_mma_launch<MT, 3, 1, true>(p, s) : latent_mma_launch<MT, 3, 1, false>(p, s);
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
