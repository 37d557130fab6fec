// Prompt attention of the hybrid decoders on the tensor cores (bf16, head sizes up to 128): packed
// sequences of unequal length, continued from the slot cache, a sliding window beside which the
// first `keep` tokens stay visible, grouped queries, separate query/key and value sizes, sigmoid
// output gate. attn_prep (attn_window.cu) or latent_prep (latent_attn.cu) has normed and rotated q in
// place and filled the cache.
//
// Keys and values are rows of the slot cache, or of a buffer that holds, segment after segment, the
// positions this forward looks at (keys and values expanded from latents): row = position + shift of
// the segment. A key may have a second part of up to 64 columns that all heads share (the rotated
// part of latent attention); it meets the columns of q behind the first part.
//
// One CTA = one (sequence, query head, 128-query block). Same roles as the causal kernel in
// flash_attn.cu: a TMA producer, a tcgen05 issuer, eight softmax warps (two threads per query row),
// O accumulated in tensor memory with lazy rescaling. What differs:
//   * the probabilities go from registers into tensor memory and are the tensor-memory A operand of
//     P V, so they take no shared memory and 192-wide keys fit with two stages;
//   * the key tiles of a block are the tiles of the kept tokens followed by those from the window's
//     lower edge to the diagonal; tiles in between are never loaded, and only tiles that an edge
//     crosses test their keys;
//   * head sizes below 64 / 128 are filled up with zeros by the TMA unit (the boxes reach past the
//     innermost dimension), so any multiple of 8 runs;
//   * the rows of a block belong to one sequence of the packed batch; keys past its end are stale
//     cache rows and are masked;
//   * the epilogue multiplies with sigmoid(gate) and overwrites the gate columns.
//
// All mbarrier waits are bounded; a time-out sets the status word and the CTA still reaches every
// barrier and frees its tensor memory.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <float.h>
#include <limits.h>
#include <string.h>
#include <mutex>

#include "flash_common.cuh"
#include "launch.cuh"
#include "ptx.cuh"

namespace e2h {

constexpr int kWQ = 128, kWK = 128;
constexpr int kWThreads = 320;
constexpr float kWRescale = 8.f;

struct FlashWindowParams {
  int H, G, n, slots, smax;
  int vdim;
  const int* shift;            // [n_seg] key row - position, or null: rows of the slot cache
  float scale;
  int window, keep;            // window INT_MAX: unlimited
  const int* seg;              // [n_seg + 1]
  const int* pos;              // [n]
  const int* slot;             // [n]
  __nv_bfloat16* gate;         // act + off_g: gate columns in, gated heads out
  long long ld;
  int* status;
};

struct FlashWindowCtrl {
  uint64_t q_full;
  uint64_t k_full[2], k_empty[2], v_full[2], v_empty[2];
  uint64_t s_full, s_empty, p_full, o_full;
  uint64_t p_empty[2];
  uint32_t tmem_base;
  int abort_flag;
};

// KN / KR / VH: 64-wide column blocks of the query/key heads (own part, shared part) and of the values.
template <int KN, int KR, int VH>
__global__ void __launch_bounds__(kWThreads, 1)
flash_window_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmQ2,
                    const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmK2,
                    const __grid_constant__ CUtensorMap tmV, const FlashWindowParams p) {
  constexpr int KH = KN + KR;
  constexpr int kHalf = 128 * 128;               // [128 rows x 64] bf16
  constexpr int kKT = KH * kHalf, kVT = VH * kHalf;
  constexpr int DV = VH * 64, DH = DV / 2;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~uintptr_t(1023));
  FlashWindowCtrl* ctrl = reinterpret_cast<FlashWindowCtrl*>(smem);
  float* xch = reinterpret_cast<float*>(smem + 1024);   // [2 halves][128 rows]
  uint8_t* q_s = smem + 2048;
  uint8_t* k_s = q_s + kKT;                      // 2 stages
  uint8_t* v_s = k_s + 2 * kKT;                  // 2 stages

  pdl_wait_prior();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qb = gridDim.x - 1 - blockIdx.x, h = blockIdx.y, sg = blockIdx.z;
  const int t_begin = p.seg[sg], len = p.seg[sg + 1] - t_begin;
  const int q0 = qb * kWQ;
  if (t_begin < 0 || t_begin + len > p.n || q0 >= len) return;
  const int slot = p.slot[t_begin], pos0 = p.pos[t_begin];
  if (slot < 0 || slot >= p.slots || pos0 < 0 || pos0 + len > p.smax) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  const int hk = h / (p.H / p.G);
  const int n_keys = pos0 + len;                 // keys this sequence holds
  const int p0 = pos0 + q0;                      // position of the block's first query
  const int p1 = min(p0 + kWQ, n_keys) - 1;      // and of its last
  const int lo = p.window < p0 ? p0 - p.window + 1 : 0;   // first windowed key of the block
  const int j_win = lo / kWK;
  const int n_kt = min((p.keep + kWK - 1) / kWK, j_win);  // tiles of kept tokens before it
  const int n_j = n_kt + p1 / kWK + 1 - j_win;
  const int shift = p.shift ? p.shift[sg] : 0;   // key row = position + shift
  const int kslot = p.shift ? 0 : slot;
  auto tile_key = [&](int it) { return (it < n_kt ? it : j_win + it - n_kt) * kWK; };
  volatile int* abort_flag = &ctrl->abort_flag;

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&ctrl->q_full), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&ctrl->k_full[s]), 1);
      mbar_init(smem_u32(&ctrl->k_empty[s]), 1);
      mbar_init(smem_u32(&ctrl->v_full[s]), 1);
      mbar_init(smem_u32(&ctrl->v_empty[s]), 1);
      mbar_init(smem_u32(&ctrl->p_empty[s]), 1);
    }
    mbar_init(smem_u32(&ctrl->s_full), 1);
    mbar_init(smem_u32(&ctrl->s_empty), 8);
    mbar_init(smem_u32(&ctrl->p_full), 8);
    mbar_init(smem_u32(&ctrl->o_full), 1);
    ctrl->abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
    if (KR) {
      tma_prefetch_desc(&tmQ2);
      tma_prefetch_desc(&tmK2);
    }
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&ctrl->tmem_base), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();      // with the tensor memory in hand: a dependent cannot take it first
  const uint32_t tmem_s = ctrl->tmem_base;
  const uint32_t tmem_o = tmem_s + 128;
  const uint32_t tmem_p = tmem_s + 256;          // 2 buffers of 64 columns (128 bf16 per row)

  if (warp == 0 && lane == 0) {
    // ---------------- TMA producer ----------------
    int issued_k = 0, issued_v = 0;
    mbar_expect_tx(smem_u32(&ctrl->q_full), kKT);
#pragma unroll
    for (int hf = 0; hf < KH; ++hf)
      tma_load_4d(smem_u32(q_s + hf * kHalf), hf < KN ? &tmQ : &tmQ2, (hf < KN ? hf : hf - KN) * 64,
                  t_begin + q0, h, 0, smem_u32(&ctrl->q_full));
    for (int it = 0; it < n_j; ++it) {
      const int s = it & 1;
      const uint32_t ph = (it >> 1) & 1;
      const int key0 = tile_key(it) + shift;
      if (!mbar_wait(smem_u32(&ctrl->k_empty[s]), ph ^ 1, abort_flag, p.status,
                     kStatusTimeoutEmpty))
        break;
      mbar_expect_tx(smem_u32(&ctrl->k_full[s]), kKT);
#pragma unroll
      for (int hf = 0; hf < KH; ++hf)
        if (hf < KN)
          tma_load_4d(smem_u32(k_s + s * kKT + hf * kHalf), &tmK, hf * 64, key0, hk, kslot,
                      smem_u32(&ctrl->k_full[s]));
        else
          tma_load_4d(smem_u32(k_s + s * kKT + hf * kHalf), &tmK2, (hf - KN) * 64, key0, 0, kslot,
                      smem_u32(&ctrl->k_full[s]));
      issued_k = it + 1;
      if (!mbar_wait(smem_u32(&ctrl->v_empty[s]), ph ^ 1, abort_flag, p.status,
                     kStatusTimeoutEmpty))
        break;
      mbar_expect_tx(smem_u32(&ctrl->v_full[s]), kVT);
#pragma unroll
      for (int hf = 0; hf < VH; ++hf)
        tma_load_4d(smem_u32(v_s + s * kVT + hf * kHalf), &tmV, hf * 64, key0, hk, kslot,
                    smem_u32(&ctrl->v_full[s]));
      issued_v = it + 1;
    }
    if (*abort_flag) {   // bounded wait for the copies still in flight into this CTA's smem
      auto drain = [&](uint64_t* bars, int n) {
        for (int j = n > 2 ? n - 2 : 0; j < n; ++j) {
          const long long tq = clock64();
          while (!mbar_try_wait(smem_u32(&bars[j & 1]), (j >> 1) & 1))
            if (clock64() - tq > kWaitLimitCycles / 8) break;
        }
      };
      drain(ctrl->k_full, issued_k);
      drain(ctrl->v_full, issued_v);
    }
  } else if (warp == 1 && lane == 0) {
    // ---------------- UMMA issuer ----------------
    const uint32_t idesc_s = make_idesc_bf16(128, kWK, 0, 0);
    const uint32_t idesc_o = make_idesc_bf16(128, DV, 0, 1);
    const uint32_t d_hi = sw128_desc_hi(1024);
    bool ok = mbar_wait(smem_u32(&ctrl->q_full), 0, abort_flag, p.status, kStatusTimeoutFull);
    auto issue_s = [&](int it) {
      const int s = it & 1;
      ok = ok && mbar_wait(smem_u32(&ctrl->k_full[s]), (it >> 1) & 1, abort_flag, p.status,
                           kStatusTimeoutFull);
      if (!ok) return;
      tc_fence_after();
      const uint32_t qa = sw128_desc_lo(smem_u32(q_s), 16);
      const uint32_t ka = sw128_desc_lo(smem_u32(k_s + s * kKT), 16);
#pragma unroll
      for (int kk = 0; kk < KH * 4; ++kk) {
        const uint32_t o = ((kk / 4) * kHalf + (kk % 4) * 32) >> 4;
        umma_f16_lohi(tmem_s, qa + o, d_hi, ka + o, d_hi, idesc_s, kk > 0 ? 1u : 0u);
      }
      umma_commit(smem_u32(&ctrl->k_empty[s]));
      umma_commit(smem_u32(&ctrl->s_full));
    };
    issue_s(0);
    for (int it = 0; it < n_j && ok; ++it) {
      const int s = it & 1;
      if (it + 1 < n_j) {
        ok = mbar_wait(smem_u32(&ctrl->s_empty), it & 1, abort_flag, p.status,
                       kStatusTimeoutTmemEmpty);
        if (!ok) break;
        issue_s(it + 1);
        if (!ok) break;
      }
      ok = mbar_wait(smem_u32(&ctrl->p_full), it & 1, abort_flag, p.status, kStatusTimeoutFull) &&
           mbar_wait(smem_u32(&ctrl->v_full[s]), (it >> 1) & 1, abort_flag, p.status,
                     kStatusTimeoutFull);
      if (!ok) break;
      tc_fence_after();
      const uint32_t pa = tmem_p + (it & 1) * 64;
      const uint32_t va = sw128_desc_lo(smem_u32(v_s + s * kVT), kHalf);
#pragma unroll
      for (int kk = 0; kk < kWK / 16; ++kk)
        umma_f16_ts(tmem_o, pa + kk * 8, va + ((kk * 2048) >> 4), d_hi, idesc_o,
                    (it > 0 || kk > 0) ? 1u : 0u);
      umma_commit(smem_u32(&ctrl->v_empty[s]));
      umma_commit(smem_u32(&ctrl->p_empty[it & 1]));
      umma_commit(smem_u32(&ctrl->o_full));
    }
  }

  if (warp >= 2) {
    // ---------------- softmax / output warps ----------------
    const int qrt = warp & 3;
    const int ch = (warp - 2) >> 2;
    const int row = qrt * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>(qrt * 32) << 16;
    const int qpos = p0 + row;
    const int q_lo = p.window <= qpos ? qpos - p.window + 1 : 0;   // first windowed key of the row
    const float sl2 = p.scale * 1.4426950408889634f;
    float m = -FLT_MAX, l = 0.f;
    bool ok = true;
    for (int it = 0; it < n_j; ++it) {
      const int key0 = tile_key(it);
      if (ok) ok = mbar_wait(smem_u32(&ctrl->s_full), it & 1, abort_flag, p.status,
                             kStatusTimeoutTmemFull);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      float sv[64];
      if (ok) {
        tmem_ld_x32(tmem_s + lane_off + ch * 64, sv);
        tmem_ld_x32(tmem_s + lane_off + ch * 64 + 32, sv + 32);
      }
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&ctrl->s_empty));
      // every row of the block sees every key of the tile?
      const bool full_tile = key0 + kWK - 1 <= p0 &&
                             (key0 + kWK <= p.keep || p0 + kWQ - 1 - key0 < p.window);
      float mx = -FLT_MAX;
      if (full_tile) {
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          sv[i] *= sl2;
          mx = fmaxf(mx, sv[i]);
        }
      } else {
        const int cbase = key0 + ch * 64;
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          const int j = cbase + i;
          const bool vis = j <= qpos && (j >= q_lo || j < p.keep) && j < n_keys;
          sv[i] = vis ? sv[i] * sl2 : -INFINITY;
          mx = fmaxf(mx, sv[i]);
        }
      }
      xch[ch * 128 + row] = mx;
      pair_bar_sync(1 + qrt);
      const float m_new = fmaxf(m, fmaxf(mx, xch[(ch ^ 1) * 128 + row]));
      pair_bar_sync(1 + qrt);
      const bool need = (it > 0) && (m != -FLT_MAX) && (m_new - m > kWRescale);
      if (__any_sync(0xffffffffu, need)) {
        const float alpha = (m == -FLT_MAX) ? 1.f : ex2_approx(m - m_new);
        if (ok) ok = mbar_wait(smem_u32(&ctrl->o_full), (it - 1) & 1, abort_flag, p.status,
                               kStatusTimeoutTmemFull);
        ok = __all_sync(0xffffffffu, ok);
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < DH; c += 32) {
          float ov[32];
          if (ok) tmem_ld_x32(tmem_o + lane_off + ch * DH + c, ov);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) ov[i] *= alpha;
          if (ok) tmem_st_x32(tmem_o + lane_off + ch * DH + c, ov);
        }
        tmem_st_wait();
        l *= alpha;
        m = m_new;
      } else if (m == -FLT_MAX) {
        m = m_new;
      }
      const float msafe = (m == -FLT_MAX) ? 0.f : m;
      if (ok) ok = mbar_wait(smem_u32(&ctrl->p_empty[it & 1]), ((it >> 1) & 1) ^ 1, abort_flag,
                             p.status, kStatusTimeoutEmpty);
      ok = __all_sync(0xffffffffu, ok);
      float rs = 0.f;
      tc_fence_after();
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        uint32_t packed[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const float p0_ = ex2_approx(sv[32 * q + 2 * e] - msafe);
          const float p1_ = ex2_approx(sv[32 * q + 2 * e + 1] - msafe);
          rs += p0_ + p1_;
          const __nv_bfloat162 pk = __floats2bfloat162_rn(p0_, p1_);
          packed[e] = *reinterpret_cast<const uint32_t*>(&pk);
        }
        if (ok) tmem_st_x16(tmem_p + (it & 1) * 64 + lane_off + ch * 32 + q * 16, packed);
      }
      l += rs;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&ctrl->p_full));
    }
    // ---- epilogue: O / l * sigmoid(gate) ----
    // the gate row first, all pieces in flight at once, while the last product finishes
    const bool in_seq = q0 + row < len;
    __nv_bfloat16* grow = p.gate + (long long)(t_begin + q0 + row) * p.ld + (long long)h * p.vdim +
                          ch * DH;
    const int n_col = min(DH, p.vdim - ch * DH);      // live columns of this thread (may be <= 0)
    uint4 gr[DH / 8];
#pragma unroll
    for (int i = 0; i < DH / 8; ++i)
      gr[i] = in_seq && i * 8 < n_col ? *reinterpret_cast<const uint4*>(grow + i * 8)
                                      : make_uint4(0, 0, 0, 0);
    if (ok) ok = mbar_wait(smem_u32(&ctrl->o_full), (n_j - 1) & 1, abort_flag, p.status,
                           kStatusTimeoutTmemFull);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    xch[ch * 128 + row] = l;
    pair_bar_sync(1 + qrt);
    const float l_tot = l + xch[(ch ^ 1) * 128 + row];
    const float inv = l_tot > 0.f ? 1.f / l_tot : 0.f;
    const bool store = ok && in_seq;
#pragma unroll
    for (int c = 0; c < DH; c += 32) {
      float ov[32];
      if (ok) tmem_ld_x32(tmem_o + lane_off + ch * DH + c, ov);   // warp-uniform
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        uint4 g = gr[c / 8 + i];
        __nv_bfloat162* g2 = reinterpret_cast<__nv_bfloat162*>(&g);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float a = ov[8 * i + 2 * e] * inv *
                          __fdividef(1.f, 1.f + __expf(-__bfloat162float(g2[e].x)));
          const float b = ov[8 * i + 2 * e + 1] * inv *
                          __fdividef(1.f, 1.f + __expf(-__bfloat162float(g2[e].y)));
          g2[e] = __floats2bfloat162_rn(a, b);
        }
        if (store && c + i * 8 < n_col) *reinterpret_cast<uint4*>(grow + c + i * 8) = g;
      }
    }
    tc_fence_before();
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(ctrl->tmem_base, 512);
}

struct FlashWindowMaps {
  CUtensorMap q, q2, k, k2, v;
};

template <int KN, int KR, int VH>
static int flash_window_launch(const FlashWindowMaps& m, const FlashWindowParams& p, dim3 grid,
                               cudaStream_t stream) {
  const size_t smem = 1024 + 2048 + (size_t)(3 * (KN + KR) + 2 * VH) * 128 * 128;
  static_assert(1024 + 2048 + (3 * (KN + KR) + 2 * VH) * 128 * 128 <= 227 * 1024, "shared memory");
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [&] {
    err = cudaFuncSetAttribute(flash_window_kernel<KN, KR, VH>,
                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  });
  if (err != cudaSuccess) return (int)err;
  return (int)launch(flash_window_kernel<KN, KR, VH>, grid, dim3(kWThreads), smem, stream, m.q,
                     m.q2, m.k, m.k2, m.v, p);
}

struct FlashWindowArgs {
  void* act;                   // bf16 [n, ld]
  long long ld;
  int off_q, q_head;           // column of head 0 of q (rotated), columns from head to head
  int off_g;                   // gate columns (H x vdim)
  const void* k;               // key rows: strides of rows, heads and slots, in elements
  long long ld_k, k_head, k_slot;
  const void* v;
  long long ld_v, v_head, v_slot;
  const void* k2;              // shared key part [rows, ld_k2] or null
  long long ld_k2;
  int rows, slots, smax;       // rows of a slot (or of the buffer), slots, positions of a sequence
  const int* shift;            // [n_seg] key row - position: keys lie in a buffer; null: in the slots
  const int* seg;              // [n_seg + 1]
  int n_seg, seg_max;
  const int* pos;
  const int* slot;
  int n, H, G;
  int dim, dim2, vdim;         // own and shared part of a key, value
  float scale;
  int window, keep;
  int* status;
};

}  // namespace e2h

extern "C" int e2h_flash_window(const e2h::FlashWindowArgs* ap, void* stream_v) {
  using namespace e2h;
  const FlashWindowArgs& a = *ap;
  if (a.n <= 0 || a.n_seg <= 0 || a.n_seg > 65535 || a.seg_max <= 0 || a.G <= 0 || a.H % a.G ||
      a.H > 65535 || a.rows <= 0 || a.slots <= 0)
    return -1;
  if (a.dim <= 0 || a.vdim <= 0 || a.dim > 128 || a.vdim > 128 || a.dim2 < 0 || a.dim2 > 64 ||
      (a.dim | a.dim2 | a.vdim | a.off_q | a.q_head | a.off_g) % 8 ||
      (a.ld | a.ld_k | a.k_head | a.k_slot | a.ld_v | a.v_head | a.v_slot | a.ld_k2) % 8)
    return -2;
  if ((a.dim2 > 0) != (a.k2 != nullptr) || (a.k2 && !a.shift)) return -2;
  __nv_bfloat16* act = static_cast<__nv_bfloat16*>(a.act);
  if ((reinterpret_cast<uintptr_t>(act) | reinterpret_cast<uintptr_t>(a.k) |
       reinterpret_cast<uintptr_t>(a.k2) | reinterpret_cast<uintptr_t>(a.v)) & 15)
    return -3;
  FlashWindowMaps m;
  const long long all_q = (long long)a.n * a.ld;
  int r = make_map4d(&m.q, act + a.off_q, a.dim, a.n, a.H, 1, all_q, a.ld, a.q_head, kWQ);
  if (r) return r;
  r = make_map4d(&m.k, a.k, a.dim, a.rows, a.G, a.slots, a.k_slot, a.ld_k, a.k_head, kWK);
  if (r) return r;
  r = make_map4d(&m.v, a.v, a.vdim, a.rows, a.G, a.slots, a.v_slot, a.ld_v, a.v_head, kWK);
  if (r) return r;
  m.q2 = m.q;
  m.k2 = m.k;
  if (a.dim2) {
    r = make_map4d(&m.q2, act + a.off_q + a.dim, a.dim2, a.n, a.H, 1, all_q, a.ld, a.q_head, kWQ);
    if (r) return r;
    const long long all_k = (long long)a.rows * a.ld_k2;
    r = make_map4d(&m.k2, a.k2, a.dim2, a.rows, 1, 1, all_k, a.ld_k2, all_k, kWK);
    if (r) return r;
  }
  FlashWindowParams p;
  p.H = a.H; p.G = a.G; p.n = a.n; p.slots = a.shift ? INT_MAX : a.slots; p.smax = a.smax;
  p.vdim = a.vdim;
  p.shift = a.shift;
  p.scale = a.scale;
  p.window = a.window > 0 ? a.window : INT_MAX;
  p.keep = a.keep;
  p.seg = a.seg; p.pos = a.pos; p.slot = a.slot;
  p.gate = act + a.off_g;
  p.ld = a.ld;
  p.status = a.status;
  const dim3 grid((a.seg_max + kWQ - 1) / kWQ, a.H, a.n_seg);
  cudaStream_t s = static_cast<cudaStream_t>(stream_v);
#define E2H_FW(KN_, KR_)                                              \
  return a.vdim <= 64 ? flash_window_launch<KN_, KR_, 1>(m, p, grid, s) \
                      : flash_window_launch<KN_, KR_, 2>(m, p, grid, s)
  if (a.dim2) {
    if (a.dim <= 64) E2H_FW(1, 1);
    E2H_FW(2, 1);
  }
  if (a.dim <= 64) E2H_FW(1, 0);
  E2H_FW(2, 0);
#undef E2H_FW
}
