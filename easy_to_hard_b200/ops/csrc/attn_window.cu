// Attention of the hybrid decoders over the slot cache: any head sizes up to 256 (query/key and
// value sizes may differ), grouped queries, a sliding window that never drops the leading tokens, partial rotary
// positions from a table, query/key norms over the whole projection, and a sigmoid output gate.
//
//   visible(i, j) = j <= i and (i - j < window or j < keep)
//
// The projections of a token lie in one row of a packed activation [tokens, ld]: q (H x dim),
// k (G x dim), v (G x vdim) and the gate (H x vdim) at given column offsets; the gated heads
// replace the gate columns, where the output projection reads them. Caches are
// [slots, G, smax, dimp] / [slots, G, smax, vdimp] with the sizes rounded up to 8 (the rounding
// columns hold zeros).
//
//   attn_prep    prompts: norms and rotates q and k of every token in place, writes k and v to the
//                cache. One CTA per token (a vectorised form for sizes in multiples of 8).
//   attn_window  one (token, kv head) per cluster of CTAs: the visible keys are split over the CTAs
//                of the cluster and merged through distributed shared memory. In its fused form
//                (decode) it does the work of attn_prep itself, so that a decode step has one
//                attention kernel; otherwise every token, also of a prompt, reads its keys from
//                the cache (portions and head sizes that the tensor-core prompt kernel does not
//                take). Two forms: fp32 on the CUDA cores, bf16 on warp-level matrix products.
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

struct AttnWindowParams {
  void* act;                 // T [n, ld]
  long long ld;
  int off_q, off_k, off_v, off_g;
  void* kc;                  // T [slots, G, smax, dimp]
  void* vc;                  // T [slots, G, smax, vdimp]
  const int* pos;            // [n]
  const int* slot;           // [n]
  int n, slots, smax;
  int H, G, dim, vdim, dimp, vdimp;
  int rot;                   // rotated dimensions
  const float* rot_table;    // fp32 [smax, rot / 2, 2]: (cos, sin), amplitude included
  float scale;
  int window;                // 0: unlimited
  int keep;
  const float* qn;           // fp32 [H * dim] or null (no norm)
  const float* kn;           // fp32 [G * dim] or null
  float eps;
  int splits;                // CTAs per cluster
  int* status;
};

// Element d of a head after norm and rotation: x points at the head's columns, w at its norm
// weights (or null), r is the reciprocal root mean square of the projection.
template <typename T>
__device__ __forceinline__ float norm_rot(const T* x, const float* w, float r, int d, int rot,
                                          const float* cs) {
  auto val = [&](int i) { return to_f(x[i]) * (w ? r * w[i] : 1.f); };
  const int half = rot >> 1;
  if (d >= 2 * half) return val(d);
  const int i = d < half ? d : d - half;
  const float c = cs[2 * i], s = cs[2 * i + 1];
  const float u = val(i), v = val(i + half);
  return d < half ? u * c - v * s : v * c + u * s;
}

template <typename T>
__device__ __forceinline__ float rms_of(const T* x, int n, float eps, float* red) {
  float ss = 0.f;
  if ((n & 3) == 0 && (reinterpret_cast<uintptr_t>(x) & (4 * sizeof(T) - 1)) == 0) {
    for (int c = threadIdx.x * 4; c < n; c += blockDim.x * 4) {
      float v[4];
      load4(x + c, v);
      ss += v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
    }
  } else {
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float v = to_f(x[c]);
      ss += v * v;
    }
  }
  ss = block_sum(ss, red);
  return 1.f / sqrtf(ss / n + eps);
}

// 16-byte-vectorised form: head sizes and half the rotated width are multiples of 8, rows aligned.
// A thread takes 8 columns of a pair's first halves together with the 8 of the second halves (or 16
// unrotated columns), twice: once for the sums of squares, once (from L1) to write.
template <typename T>
__global__ void __launch_bounds__(128) attn_prep_vec_kernel(const AttnWindowParams p) {
  __shared__ float red[2][4];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int t = blockIdx.x;
  const int pos = p.pos[t], slot = p.slot[t];
  if (pos < 0 || pos >= p.smax || slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  T* row = static_cast<T*>(p.act) + t * p.ld;
  T* q = row + p.off_q;
  const T* k = row + p.off_k;
  const T* v = row + p.off_v;
  const int vq = p.H * p.dim / 8, vk = p.G * p.dim / 8;
  float rq = 1.f, rk = 1.f;
  if (p.qn || p.kn) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < vq + vk; i += 128) {
      float x[8], ss = 0.f;
      load8(i < vq ? q + 8 * i : k + 8 * (i - vq), x);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
      if (i < vq) sq += ss;
      else sk += ss;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
      red[0][threadIdx.x >> 5] = sq;
      red[1][threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    sq = red[0][0] + red[0][1] + red[0][2] + red[0][3];
    sk = red[1][0] + red[1][1] + red[1][2] + red[1][3];
    if (p.qn) rq = 1.f / sqrtf(sq / (p.H * p.dim) + p.eps);
    if (p.kn) rk = 1.f / sqrtf(sk / (p.G * p.dim) + p.eps);
  }
  const int half = p.rot >> 1;
  const int up = half / 8, ur = (p.dim - p.rot) / 8, per = up + ur;   // work units of a head
  const float* cs = p.rot_table + (long long)pos * p.rot;
  T* kc = static_cast<T*>(p.kc) + ((long long)slot * p.G * p.smax + pos) * p.dimp;
  for (int i = threadIdx.x; i < (p.H + p.G) * per; i += 128) {
    const int head = i / per, u = i - head * per;
    const bool is_q = head < p.H;
    const int hk = head - p.H;
    const T* src = is_q ? q + head * p.dim : k + hk * p.dim;
    const float* w = is_q ? (p.qn ? p.qn + head * p.dim : nullptr)
                          : (p.kn ? p.kn + hk * p.dim : nullptr);
    const float r = is_q ? rq : rk;
    T* dst = is_q ? q + head * p.dim : kc + (long long)hk * p.smax * p.dimp;
    auto fetch = [&](int d, float* x) {
      load8(src + d, x);
      if (w) {
        float wv[8];
        load8(w + d, wv);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] *= r * wv[e];
      }
    };
    if (u < up) {
      const int d = 8 * u;
      float a[8], b[8], c[16];
      fetch(d, a);
      fetch(half + d, b);
      load8(cs + 2 * d, c);
      load8(cs + 2 * d + 8, c + 8);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float co = c[2 * e], si = c[2 * e + 1], x = a[e], y = b[e];
        a[e] = x * co - y * si;
        b[e] = y * co + x * si;
      }
      store4(dst + d, a);
      store4(dst + d + 4, a + 4);
      store4(dst + half + d, b);
      store4(dst + half + d + 4, b + 4);
    } else {
      const int d = p.rot + 8 * (u - up);
      float a[8];
      fetch(d, a);
      store4(dst + d, a);
      store4(dst + d + 4, a + 4);
    }
  }
  T* vc = static_cast<T*>(p.vc) + ((long long)slot * p.G * p.smax + pos) * p.vdimp;
  const int vv = p.vdim * (int)sizeof(T) / 16;               // 16-byte pieces of a value head
  for (int i = threadIdx.x; i < p.G * vv; i += 128) {
    const int head = i / vv, c = i - head * vv;
    reinterpret_cast<uint4*>(vc + (long long)head * p.smax * p.vdimp)[c] =
        reinterpret_cast<const uint4*>(v + head * p.vdim)[c];
  }
}

template <typename T>
__global__ void __launch_bounds__(256) attn_prep_kernel(const AttnWindowParams p) {
  extern __shared__ float row_s[];   // q and k of the token: (H + G) * dim
  __shared__ float red[33];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int t = blockIdx.x;
  const int pos = p.pos[t], slot = p.slot[t];
  if (pos < 0 || pos >= p.smax || slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  T* q = static_cast<T*>(p.act) + t * p.ld + p.off_q;
  T* k = static_cast<T*>(p.act) + t * p.ld + p.off_k;
  const T* v = static_cast<const T*>(p.act) + t * p.ld + p.off_v;
  const int nq = p.H * p.dim, nk = p.G * p.dim;
  const float rq = p.qn ? rms_of(q, nq, p.eps, red) : 1.f;
  const float rk = p.kn ? rms_of(k, nk, p.eps, red) : 1.f;
  for (int c = threadIdx.x; c < nq + nk; c += blockDim.x) {
    float x;
    if (c < nq) {
      x = to_f(q[c]);
      if (p.qn) x *= rq * p.qn[c];
    } else {
      x = to_f(k[c - nq]);
      if (p.kn) x *= rk * p.kn[c - nq];
    }
    row_s[c] = x;
  }
  __syncthreads();
  const int half = p.rot >> 1;
  const float* cs = p.rot_table + (long long)pos * 2 * half;
  const long long kbase = ((long long)slot * p.G * p.smax + pos) * p.dimp;
  T* kc = static_cast<T*>(p.kc) + kbase;
  for (int c = threadIdx.x; c < nq + nk; c += blockDim.x) {
    const int head = c / p.dim, d = c - head * p.dim;
    const float* x = row_s + head * p.dim;
    float y;
    if (d >= 2 * half) {
      y = x[d];
    } else {
      const int i = d < half ? d : d - half;
      const float co = cs[2 * i], si = cs[2 * i + 1];
      y = d < half ? x[i] * co - x[i + half] * si : x[i + half] * co + x[i] * si;
    }
    if (head < p.H) q[c] = from_f<T>(y);
    else kc[(long long)(head - p.H) * p.smax * p.dimp + d] = from_f<T>(y);
  }
  T* vc = static_cast<T*>(p.vc) + ((long long)slot * p.G * p.smax + pos) * p.vdimp;
  for (int c = threadIdx.x; c < p.G * p.vdim; c += blockDim.x) {
    const int head = c / p.vdim, d = c - head * p.vdim;
    vc[(long long)head * p.smax * p.vdimp + d] = v[c];
  }
}

constexpr int kWinThreads = 128;
constexpr int kWinUnroll = 4;      // keys a lane group has in flight

// Merges the (m, l, acc) of a CTA's key groups (in shared memory), then those of the cluster's CTAs,
// and writes the gated heads: every CTA of the cluster finishes its share of the columns.
template <typename T, int GROUPS, int R, int DP>
__device__ __forceinline__ void window_finish(const AttnWindowParams& p,
                                              cg::cluster_group& cluster, const float* mrg,
                                              float* acc_s, float (*fin)[2], T* row, int h0,
                                              int nr, int rank) {
  __syncthreads();
  for (int i = threadIdx.x; i < R * DP; i += kWinThreads) {
    const int r = i / DP, d = i - r * DP;
    float mx = -FLT_MAX;
    for (int k = 0; k < GROUPS; ++k) mx = fmaxf(mx, mrg[(k * R + r) * 2]);
    float a = 0.f, ls = 0.f;
    for (int k = 0; k < GROUPS; ++k) {
      const float w = exp2f(mrg[(k * R + r) * 2] - mx);
      a += w * acc_s[(k * R + r) * DP + d];
      ls += w * mrg[(k * R + r) * 2 + 1];
    }
    acc_s[i] = a;                       // entry (0, r, d) is read by this thread only
    if (d == 0) {
      fin[r][0] = mx;
      fin[r][1] = ls;
    }
  }
  if (p.splits > 1) cluster.sync();
  else __syncthreads();
  // merge the cluster: every CTA finishes its share of the columns
  const int total = nr * p.vdim;
  const int per = (total + p.splits - 1) / p.splits;
  for (int i = rank * per + threadIdx.x; i < min(total, (rank + 1) * per); i += kWinThreads) {
    const int r = i / p.vdim, d = i - r * p.vdim;
    float o;
    if (p.splits > 1) {
      float mx = -FLT_MAX;
      for (int k = 0; k < p.splits; ++k) mx = fmaxf(mx, cluster.map_shared_rank(&fin[r][0], k)[0]);
      float a = 0.f, ls = 0.f;
      for (int k = 0; k < p.splits; ++k) {
        const float* f = cluster.map_shared_rank(&fin[r][0], k);
        const float w = exp2f(f[0] - mx);
        ls += w * f[1];
        a += w * cluster.map_shared_rank(acc_s, k)[r * DP + d];
      }
      o = a / ls;
    } else {
      o = acc_s[r * DP + d] / fin[r][1];
    }
    T* gate = row + p.off_g + (h0 + r) * p.vdim + d;
    *gate = from_f<T>(o * sigmoid_f(to_f(*gate)));
  }
  if (p.splits > 1) cluster.sync();     // peers may still read this CTA's shared memory
}

// LPK lanes share a key (8 elements each), R query heads of the kv head's group per CTA.
template <typename T, int LPK, int R, bool FUSED>
__global__ void __launch_bounds__(kWinThreads) attn_window_kernel(const AttnWindowParams p) {
  constexpr int GROUPS = kWinThreads / LPK;      // keys in work at a time
  extern __shared__ __align__(16) float win_s[];
  float* q_s = win_s;                            // [R][LPK * 8] scaled queries
  float* k_new = q_s + R * LPK * 8;              // fused: the token's own key and value
  float* v_new = k_new + LPK * 8;
  float* mrg = v_new + LPK * 8;                  // [GROUPS][R] m, l
  float* acc_s = mrg + GROUPS * R * 2;           // [GROUPS][R][LPK * 8]; group 0 = the CTA's sum
  __shared__ float red[33];
  __shared__ float fin[R][2];                    // the CTA's (m, l), read by its cluster peers

  cg::cluster_group cluster = cg::this_cluster();
  pdl_launch_dependents();
  pdl_wait_prior();
  const int rank = blockIdx.x, t = blockIdx.z;
  const int per_g = p.H / p.G;
  const int n_rb = (per_g + R - 1) / R;
  const int g = blockIdx.y / n_rb, rb = blockIdx.y - g * n_rb;
  const int h0 = g * per_g + rb * R;             // first query head
  const int nr = min(R, per_g - rb * R);         // live query heads
  int pos = p.pos[t], slot = p.slot[t];
  bool ok = pos >= 0 && pos < p.smax && slot >= 0 && slot < p.slots;
  if (!ok) {                                     // indices come from device memory
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    pos = min(max(pos, 0), p.smax - 1);
    slot = min(max(slot, 0), p.slots - 1);
  }
  T* row = static_cast<T*>(p.act) + t * p.ld;
  const T* q = row + p.off_q;
  const long long hb = (long long)slot * p.G + g;
  T* kc = static_cast<T*>(p.kc) + hb * p.smax * p.dimp;
  T* vc = static_cast<T*>(p.vc) + hb * p.smax * p.vdimp;
  const int half = p.rot >> 1;
  const float* cs = p.rot_table + (long long)pos * 2 * half;
  const float sl2 = p.scale * 1.4426950408889634f;

  float rq = 1.f, rk = 1.f;
  if constexpr (FUSED) {
    if (p.qn) rq = rms_of(q, p.H * p.dim, p.eps, red);
    if (p.kn && rank == 0) rk = rms_of(row + p.off_k, p.G * p.dim, p.eps, red);
  }
  for (int i = threadIdx.x; i < R * LPK * 8; i += kWinThreads) {
    const int r = i / (LPK * 8), d = i - r * (LPK * 8);
    float x = 0.f;
    if (r < nr && d < p.dim) {
      const int h = h0 + r;
      if constexpr (FUSED)
        x = norm_rot(q + h * p.dim, p.qn ? p.qn + h * p.dim : nullptr, rq, d, p.rot, cs);
      else
        x = to_f(q[h * p.dim + d]);
    }
    q_s[i] = x * sl2;
  }
  if constexpr (FUSED) {
    if (rank == 0) {
      for (int d = threadIdx.x; d < LPK * 8; d += kWinThreads) {
        float x = 0.f, y = 0.f;
        if (d < p.dim)
          x = norm_rot(row + p.off_k + g * p.dim, p.kn ? p.kn + g * p.dim : nullptr, rk, d, p.rot,
                       cs);
        if (d < p.vdim) y = to_f(row[p.off_v + g * p.vdim + d]);
        // what the cache keeps is what this step uses, too
        const T xs = from_f<T>(x), ys = from_f<T>(y);
        if (rb == 0 && ok) {
          if (d < p.dim) kc[(long long)pos * p.dimp + d] = xs;
          if (d < p.vdim) vc[(long long)pos * p.vdimp + d] = ys;
        }
        k_new[d] = to_f(xs);
        v_new[d] = to_f(ys);
      }
    }
  }
  __syncthreads();

  // keys of the cache this token sees: [0, n_keep) and [lo, last)
  const int last = FUSED ? pos : pos + 1;
  int lo = p.window > 0 ? pos - p.window + 1 : 0;
  lo = max(lo, 0);
  const int n_keep = min(p.keep, lo);
  const int n_keys = n_keep + max(last - lo, 0);
  const int k_begin = (int)((long long)n_keys * rank / p.splits);
  const int k_end = (int)((long long)n_keys * (rank + 1) / p.splits);

  const int grp = threadIdx.x / LPK, gl = threadIdx.x % LPK;
  const bool k_lane = gl * 8 < p.dimp, v_lane = gl * 8 < p.vdimp;
  float qf[R][8], acc[R][8], m[R], l[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    m[r] = -FLT_MAX;
    l[r] = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      acc[r][e] = 0.f;
      qf[r][e] = q_s[r * LPK * 8 + gl * 8 + e];
    }
  }
  // one step: U keys (kf / vf in registers, live[u] false = no key)
  auto absorb = [&](auto U_, const float (*kf)[8], const float (*vf)[8], const bool* live) {
    constexpr int U = decltype(U_)::value;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      float s[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        float d = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) d = fmaf(qf[r][e], kf[u][e], d);
#pragma unroll
        for (int o = LPK / 2; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
        s[u] = live[u] ? d : -FLT_MAX;
      }
      float mx = m[r];
#pragma unroll
      for (int u = 0; u < U; ++u) mx = fmaxf(mx, s[u]);
      const float al = exp2f(m[r] - mx);
      m[r] = mx;
      l[r] *= al;
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[r][e] *= al;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const float w = live[u] ? exp2f(s[u] - mx) : 0.f;
        l[r] += w;
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r][e] = fmaf(w, vf[u][e], acc[r][e]);
      }
    }
  };
  // the loop count is the same for every lane of the CTA: the shuffles need whole warps
  for (int i0 = k_begin; i0 < k_end; i0 += GROUPS * kWinUnroll) {
    float kf[kWinUnroll][8], vf[kWinUnroll][8];
    bool live[kWinUnroll];
#pragma unroll
    for (int u = 0; u < kWinUnroll; ++u) {
      const int i = i0 + u * GROUPS + grp;
      live[u] = i < k_end;
      const int j = i < n_keep ? i : lo + (i - n_keep);
#pragma unroll
      for (int e = 0; e < 8; ++e) kf[u][e] = vf[u][e] = 0.f;
      if (live[u] && k_lane) load8(kc + (long long)j * p.dimp + gl * 8, kf[u]);
      if (live[u] && v_lane) load8(vc + (long long)j * p.vdimp + gl * 8, vf[u]);
    }
    absorb(std::integral_constant<int, kWinUnroll>{}, kf, vf, live);
  }
  if constexpr (FUSED) {
    if (rank == 0) {
      float kf[1][8], vf[1][8];
      const bool live[1] = {grp == 0};
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        kf[0][e] = k_new[gl * 8 + e];
        vf[0][e] = v_new[gl * 8 + e];
      }
      absorb(std::integral_constant<int, 1>{}, kf, vf, live);
    }
  }

  // merge the CTA's key groups
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (gl == 0) {
      mrg[(grp * R + r) * 2] = m[r];
      mrg[(grp * R + r) * 2 + 1] = l[r];
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) acc_s[(grp * R + r) * LPK * 8 + gl * 8 + e] = acc[r][e];
  }
  window_finish<T, GROUPS, R, LPK * 8>(p, cluster, mrg, acc_s, fin, row, h0, nr, rank);
}

__device__ __forceinline__ void window_mma(float* c, uint32_t a0, uint32_t a2, uint32_t b0,
                                           uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
      "{%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(0u), "r"(a2), "r"(0u), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}

// bf16 form: the query heads of a group (up to 8) are the rows of warp-level matrix products, so a
// key costs a few instructions however many heads share it and the kernel is a stream of the cache.
// A warp takes 16 keys at a time. Lane (g, c) = (lane / 4, lane % 4). The contraction of q k^T runs
// over the head columns in any order as long as both operands agree: the lane's 16-byte piece of key
// g holds the fragment words of two k-steps. The scores leave in the layout of the A operand of
// p v; the value fragments pair two keys, packed from the 16-byte pieces of both (the columns of the
// result are permuted accordingly).
template <int LPK, bool FUSED>
__global__ void __launch_bounds__(kWinThreads) attn_window_mma_kernel(const AttnWindowParams p) {
  using T = __nv_bfloat16;
  constexpr int R = 8, DP = LPK * 8, GROUPS = kWinThreads / 32;
  constexpr int KI = (LPK + 3) / 4;              // 16-byte pieces of a key per lane
  constexpr int VI = (LPK + 7) / 8;              // value pieces of one key per lane
  extern __shared__ __align__(16) float win_s[];
  float* mrg = win_s;                            // [GROUPS][R] m, l
  float* acc_s = mrg + GROUPS * R * 2;           // [GROUPS][R][DP]; group 0 = the CTA's sum
  T* q_s = reinterpret_cast<T*>(acc_s + GROUPS * R * DP);   // [R][DP]
  T* k_new = q_s + R * DP;                       // fused: the token's own key and value
  T* v_new = k_new + DP;
  __shared__ float red[33];
  __shared__ float fin[R][2];

  cg::cluster_group cluster = cg::this_cluster();
  pdl_launch_dependents();
  pdl_wait_prior();
  const int rank = blockIdx.x, t = blockIdx.z;
  const int per_g = p.H / p.G;
  const int n_rb = (per_g + R - 1) / R;
  const int g = blockIdx.y / n_rb, rb = blockIdx.y - g * n_rb;
  const int h0 = g * per_g + rb * R;
  const int nr = min(R, per_g - rb * R);
  int pos = p.pos[t], slot = p.slot[t];
  const bool ok = pos >= 0 && pos < p.smax && slot >= 0 && slot < p.slots;
  if (!ok) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    pos = min(max(pos, 0), p.smax - 1);
    slot = min(max(slot, 0), p.slots - 1);
  }
  T* row = static_cast<T*>(p.act) + t * p.ld;
  const T* q = row + p.off_q;
  const long long hb = (long long)slot * p.G + g;
  T* kc = static_cast<T*>(p.kc) + hb * p.smax * p.dimp;
  T* vc = static_cast<T*>(p.vc) + hb * p.smax * p.vdimp;
  const float* cs = p.rot_table + (long long)pos * (p.rot & ~1);
  const float sl2 = p.scale * 1.4426950408889634f;

  float rq = 1.f, rk = 1.f;
  if constexpr (FUSED) {
    if (p.qn) rq = rms_of(q, p.H * p.dim, p.eps, red);
    if (p.kn && rank == 0) rk = rms_of(row + p.off_k, p.G * p.dim, p.eps, red);
  }
  for (int i = threadIdx.x; i < R * DP; i += kWinThreads) {
    const int r = i / DP, d = i - r * DP;
    T x = from_f<T>(0.f);
    if (r < nr && d < p.dim) {
      const int h = h0 + r;
      if constexpr (FUSED)
        x = from_f<T>(norm_rot(q + h * p.dim, p.qn ? p.qn + h * p.dim : nullptr, rq, d, p.rot,
                               cs));
      else
        x = q[h * p.dim + d];
    }
    q_s[i] = x;
  }
  if constexpr (FUSED) {
    if (rank == 0) {
      for (int d = threadIdx.x; d < DP; d += kWinThreads) {
        T x = from_f<T>(0.f), y = x;
        if (d < p.dim)
          x = from_f<T>(norm_rot(row + p.off_k + g * p.dim, p.kn ? p.kn + g * p.dim : nullptr, rk,
                                 d, p.rot, cs));
        if (d < p.vdim) y = row[p.off_v + g * p.vdim + d];
        if (rb == 0 && ok) {
          if (d < p.dim) kc[(long long)pos * p.dimp + d] = x;
          if (d < p.vdim) vc[(long long)pos * p.vdimp + d] = y;
        }
        k_new[d] = x;
        v_new[d] = y;
      }
    }
  }
  __syncthreads();

  const int last = FUSED ? pos : pos + 1;
  int lo = p.window > 0 ? pos - p.window + 1 : 0;
  lo = max(lo, 0);
  const int n_keep = min(p.keep, lo);
  const int n_keys = n_keep + max(last - lo, 0);
  const int k_begin = (int)((long long)n_keys * rank / p.splits);
  const int k_end = (int)((long long)n_keys * (rank + 1) / p.splits);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gr = lane >> 2, c = lane & 3;
  const int k_pieces = p.dimp / 8, v_pieces = p.vdimp / 8;
  uint32_t qa[KI][4];                            // fragment words of head gr, pieces c + 4 i
#pragma unroll
  for (int i = 0; i < KI; ++i) {
    const uint4 x = *reinterpret_cast<const uint4*>(q_s + gr * DP + min(c + 4 * i, LPK - 1) * 8);
    const bool in = c + 4 * i < LPK;
    qa[i][0] = in ? x.x : 0;
    qa[i][1] = in ? x.y : 0;
    qa[i][2] = in ? x.z : 0;
    qa[i][3] = in ? x.w : 0;
  }
  float acc[VI][8][4];
#pragma unroll
  for (int i = 0; i < VI; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  float m = -FLT_MAX, l = 0.f;
  const uint4 zero4 = make_uint4(0, 0, 0, 0);

  // 16 keys: key(x), val(x) point at key x of them or are null
  auto absorb = [&](auto key, auto val) {
    uint4 kf[2][KI], vf[4][VI];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const T* kp = key(gr + 8 * x);
#pragma unroll
      for (int i = 0; i < KI; ++i)
        kf[x][i] = kp && c + 4 * i < k_pieces
                       ? *reinterpret_cast<const uint4*>(kp + (c + 4 * i) * 8) : zero4;
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const T* vp = val(2 * c + (x & 1) + 8 * (x >> 1));
#pragma unroll
      for (int i = 0; i < VI; ++i)
        vf[x][i] = vp && gr + 8 * i < v_pieces
                       ? *reinterpret_cast<const uint4*>(vp + (gr + 8 * i) * 8) : zero4;
    }
    float s[2][4];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
#pragma unroll
      for (int e = 0; e < 4; ++e) s[x][e] = 0.f;
#pragma unroll
      for (int i = 0; i < KI; ++i) {
        window_mma(s[x], qa[i][0], qa[i][1], kf[x][i].x, kf[x][i].y);
        window_mma(s[x], qa[i][2], qa[i][3], kf[x][i].z, kf[x][i].w);
      }
    }
    // this lane: head gr, keys 2c, 2c + 1, 2c + 8, 2c + 9
    float mx = m;
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        s[x][e] = key(2 * c + e + 8 * x) ? s[x][e] * sl2 : -FLT_MAX;
        mx = fmaxf(mx, s[x][e]);
      }
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    const float al = exp2f(m - mx);
    m = mx;
    float w[2][2];
    l *= al;
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        w[x][e] = s[x][e] == -FLT_MAX ? 0.f : exp2f(s[x][e] - mx);
        l += w[x][e];
      }
    const uint32_t pa0 = pack_bf16(w[0][0], w[0][1]), pa2 = pack_bf16(w[1][0], w[1][1]);
#pragma unroll
    for (int i = 0; i < VI; ++i) {
      const uint32_t* v0 = reinterpret_cast<const uint32_t*>(&vf[0][i]);
      const uint32_t* v1 = reinterpret_cast<const uint32_t*>(&vf[1][i]);
      const uint32_t* v2 = reinterpret_cast<const uint32_t*>(&vf[2][i]);
      const uint32_t* v3 = reinterpret_cast<const uint32_t*>(&vf[3][i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        acc[i][j][0] *= al;
        acc[i][j][1] *= al;
        const uint32_t sel = (j & 1) ? 0x7632 : 0x5410;   // column j of two keys
        window_mma(acc[i][j], pa0, pa2, __byte_perm(v0[j >> 1], v1[j >> 1], sel),
                   __byte_perm(v2[j >> 1], v3[j >> 1], sel));
      }
    }
  };
  for (int i0 = k_begin + warp * 16; i0 < k_end; i0 += GROUPS * 16) {
    auto at = [&](int x) -> long long {
      const int i = i0 + x;
      return i >= k_end ? -1 : i < n_keep ? i : lo + (i - n_keep);
    };
    auto in = [&](const T* base, int pitch, int x) -> const T* {
      const long long j = at(x);
      return j < 0 ? nullptr : base + j * pitch;
    };
    absorb([&](int x) { return in(kc, p.dimp, x); }, [&](int x) { return in(vc, p.vdimp, x); });
  }
  if constexpr (FUSED) {
    if (rank == 0 && warp == 0)
      absorb([&](int x) -> const T* { return x ? nullptr : k_new; },
             [&](int x) -> const T* { return x ? nullptr : v_new; });
  }
  l += __shfl_xor_sync(0xffffffffu, l, 1);
  l += __shfl_xor_sync(0xffffffffu, l, 2);
  if (c == 0) {
    mrg[(warp * R + gr) * 2] = m;
    mrg[(warp * R + gr) * 2 + 1] = l;
  }
#pragma unroll
  for (int i = 0; i < VI; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = (2 * c + e + 8 * i) * 8 + j;
        if (col < DP) acc_s[(warp * R + gr) * DP + col] = acc[i][j][e];
      }
  window_finish<T, GROUPS, R, DP>(p, cluster, mrg, acc_s, fin, row, h0, nr, rank);
}

static int win_start(void (*kern)(const AttnWindowParams), const AttnWindowParams& p, int heads,
                     size_t smem, cudaStream_t stream) {
  const int per_g = p.H / p.G, n_rb = (per_g + heads - 1) / heads;
  cudaLaunchConfig_t cfg;
  memset(&cfg, 0, sizeof(cfg));
  cfg.gridDim = dim3(p.splits, p.G * n_rb, p.n);
  cfg.blockDim = dim3(kWinThreads);
  cfg.dynamicSmemBytes = smem;
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

template <int LPK, int R, bool FUSED>
static int win_launch(const AttnWindowParams& p, cudaStream_t stream) {
  constexpr int GROUPS = kWinThreads / LPK;
  constexpr size_t smem = sizeof(float) * (R * LPK * 8 + 2 * LPK * 8 + GROUPS * R * 2 +
                                           GROUPS * R * LPK * 8);
  static_assert(smem < 48 * 1024, "fits the default limit");
  return win_start(attn_window_kernel<float, LPK, R, FUSED>, p, R, smem, stream);
}

template <int LPK, bool FUSED>
static int win_launch_mma(const AttnWindowParams& p, cudaStream_t stream) {
  constexpr int R = 8, DP = LPK * 8, GROUPS = kWinThreads / 32;
  constexpr size_t smem = sizeof(float) * (GROUPS * R * 2 + GROUPS * R * DP) + 2 * (R + 2) * DP;
  static_assert(smem < 48 * 1024, "fits the default limit");
  return win_start(attn_window_mma_kernel<LPK, FUSED>, p, R, smem, stream);
}

template <int LPK>
static int win_pick(const AttnWindowParams& p, bool fused, bool bf16, cudaStream_t stream) {
  const int per_g = p.H / p.G;
  if (bf16)
    return fused ? win_launch_mma<LPK, true>(p, stream) : win_launch_mma<LPK, false>(p, stream);
#define E2H_WIN(R_) return fused ? win_launch<LPK, R_, true>(p, stream) \
                                 : win_launch<LPK, R_, false>(p, stream)
  if (per_g == 1) E2H_WIN(1);
  if (per_g == 2) E2H_WIN(2);
  E2H_WIN(4);
#undef E2H_WIN
}

static int win_check(const AttnWindowParams& p) {
  if (p.n <= 0 || p.G <= 0 || p.H % p.G || p.dim <= 0 || p.vdim <= 0 || p.dim > 256 ||
      p.vdim > 256)
    return -1;
  if (p.dimp % 8 || p.vdimp % 8 || p.dimp < p.dim || p.vdimp < p.vdim || p.rot % 2 ||
      p.rot > p.dim || p.rot < 0 || p.keep < 0 || p.window < 0)
    return -1;
  if (p.splits < 1 || p.splits > 8 || !p.status) return -1;
  return 0;
}

}  // namespace e2h

extern "C" int e2h_attn_prep(const e2h::AttnWindowParams* p, int is_bf16, void* stream) {
  using namespace e2h;
  int r = win_check(*p);
  if (r) return r;
  const bool vec = p->dim % 8 == 0 && p->vdim % 8 == 0 && p->rot % 16 == 0 && p->ld % 8 == 0 &&
                   p->off_q % 8 == 0 && p->off_k % 8 == 0 && p->off_v % 8 == 0 &&
                   !((reinterpret_cast<uintptr_t>(p->act) | reinterpret_cast<uintptr_t>(p->qn) |
                      reinterpret_cast<uintptr_t>(p->kn)) & 15);
  if (vec)
    return is_bf16 ? (int)launch(attn_prep_vec_kernel<__nv_bfloat16>, dim3(p->n), dim3(128), 0,
                                 (cudaStream_t)stream, *p)
                   : (int)launch(attn_prep_vec_kernel<float>, dim3(p->n), dim3(128), 0,
                                 (cudaStream_t)stream, *p);
  const size_t smem = (size_t)(p->H + p->G) * p->dim * 4;
  if (smem > 200 * 1024) return -2;
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [] {
    err = cudaFuncSetAttribute(attn_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                               200 * 1024);
    if (err == cudaSuccess)
      err = cudaFuncSetAttribute(attn_prep_kernel<__nv_bfloat16>,
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  });
  if (err != cudaSuccess) return (int)err;
  return is_bf16 ? (int)launch(attn_prep_kernel<__nv_bfloat16>, dim3(p->n), dim3(256), smem,
                               (cudaStream_t)stream, *p)
                 : (int)launch(attn_prep_kernel<float>, dim3(p->n), dim3(256), smem,
                               (cudaStream_t)stream, *p);
}

// fused: one token per sequence, projections as the GEMM left them. Otherwise attn_prep ran.
extern "C" int e2h_attn_window(const e2h::AttnWindowParams* p, int fused, int is_bf16,
                               void* stream_v) {
  using namespace e2h;
  int r = win_check(*p);
  if (r) return r;
  cudaStream_t stream = (cudaStream_t)stream_v;
  const int big = p->dimp > p->vdimp ? p->dimp : p->vdimp;
  AttnWindowParams q = *p;
  // grid.z holds at most 65535 tokens
  for (int t0 = 0; t0 < p->n; t0 += 65535) {
    q.n = p->n - t0 < 65535 ? p->n - t0 : 65535;
    q.pos = p->pos + t0;
    q.slot = p->slot + t0;
    q.act = static_cast<char*>(p->act) + (long long)t0 * p->ld * (is_bf16 ? 2 : 4);
    const bool bf = is_bf16 != 0;
    r = big <= 32    ? win_pick<4>(q, fused != 0, bf, stream)
        : big <= 64  ? win_pick<8>(q, fused != 0, bf, stream)
        : big <= 128 ? win_pick<16>(q, fused != 0, bf, stream)
                     : win_pick<32>(q, fused != 0, bf, stream);
    if (r) return r;
  }
  return 0;
}
