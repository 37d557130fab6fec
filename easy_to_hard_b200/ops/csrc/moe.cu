// Mixture-of-experts routing: top-k of the fp32 router logits, their weights (softmax over the chosen
// ones, or the sigmoid of each), and the regrouping of the tokens by expert for the grouped GEMMs
// (rows of expert e are off[e] .. off[e + 1] of the regrouped activation, in token order, so nothing
// depends on timing). The regrouped rows may carry their weight (designs that weight the expert's
// input instead of its output).
//
//   moe_route_small   one launch for a decode-sized batch: every CTA (one token) routes the whole
//                     batch redundantly from its few logits and copies its own token's rows
//   moe_topk + moe_group + moe_gather    the same for many tokens
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <float.h>
#include <stdint.h>

#include "launch.cuh"
#include "ptx.cuh"
#include "scalar_types.cuh"

namespace e2h {

constexpr int kMoeMaxTop = 16;
constexpr int kMoeMaxExperts = 1024;
constexpr int kMoeSmall = 1024;      // token * top bound of the one-launch form

enum : int { kScoreSoftmax = 0, kScoreSigmoid = 1 };

// One warp: the `top` largest of z[0..E) (ties: lower index), and their weights: softmax over them or
// the sigmoid of each. Every lane returns with the whole result in idx / val (val holds the weights).
__device__ __forceinline__ void warp_topk(const float* z, int E, int top, int score, int* idx,
                                          float* val) {
  const int lane = threadIdx.x & 31;
  float last = INFINITY;
  int last_i = -1;
  float mx = 0.f, sum = 0.f;
  for (int j = 0; j < top; ++j) {
    // best entry after (last, last_i) in the order (value descending, index ascending)
    float bv = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float v = z[e];
      if (!(v < last || (v == last && e > last_i))) continue;
      if (v > bv || (v == bv && e < bi)) {
        bv = v;
        bi = e;
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) {
        bv = ov;
        bi = oi;
      }
    }
    if (bi >= E) bi = 0;               // only with NaN logits
    last = bv;
    last_i = bi;
    if (j == 0) mx = bv;
    idx[j] = bi;
    val[j] = score == kScoreSigmoid ? sigmoid_f(bv) : expf(bv - mx);
    sum += val[j];
  }
  if (score != kScoreSigmoid)
    for (int j = 0; j < top; ++j) val[j] /= sum;
}

// dst = src * f (f == 1: a plain copy)
template <typename T>
__device__ __forceinline__ void copy_row(T* dst, const T* src, int W, float f = 1.f) {
  if (f != 1.f) {
    if (W % 4 == 0 && ((reinterpret_cast<uintptr_t>(dst) | reinterpret_cast<uintptr_t>(src)) &
                       (4 * sizeof(T) - 1)) == 0) {
      for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {
        float v[4];
        load4(src + i, v);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] *= f;
        store4(dst + i, v);
      }
    } else {
      for (int i = threadIdx.x; i < W; i += blockDim.x) dst[i] = from_f<T>(to_f(src[i]) * f);
    }
    return;
  }
  if ((W * sizeof(T)) % 16 == 0 && ((reinterpret_cast<uintptr_t>(dst) |
                                     reinterpret_cast<uintptr_t>(src)) & 15) == 0) {
    const int n = W * sizeof(T) / 16;
    for (int i = threadIdx.x; i < n; i += blockDim.x)
      reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) dst[i] = src[i];
  }
}

constexpr int kRouteThreads = 512;
constexpr int kRouteLogits = 8192;   // logits staged in shared memory

template <typename T>
__global__ void __launch_bounds__(kRouteThreads)
moe_route_small_kernel(const float* z, long long ldz, int n, int E, int top, int score, int scale_in,
                       const T* h, long long ldh, int W, T* hg, long long ldg, int* off, int* place,
                       float* w) {
  __shared__ int sel[kMoeSmall];
  __shared__ int count[kMoeMaxExperts];
  __shared__ int my_off[kMoeMaxTop], my_before[kMoeMaxTop];
  __shared__ float my_w[kMoeMaxTop];
  extern __shared__ float z_s[];
  pdl_launch_dependents();
  pdl_wait_prior();
  const bool staged = n * E <= kRouteLogits;
  if (staged)
    for (int i = threadIdx.x; i < n * E; i += blockDim.x) z_s[i] = z[i / E * ldz + i % E];
  const int t_me = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  if (threadIdx.x < top) my_off[threadIdx.x] = my_before[threadIdx.x] = 0;
  __syncthreads();
  for (int t = warp; t < n; t += blockDim.x >> 5) {
    int idx[kMoeMaxTop];
    float val[kMoeMaxTop];
    warp_topk(staged ? z_s + t * E : z + t * ldz, E, top, score, idx, val);
    if (lane == 0) {
      for (int j = 0; j < top; ++j) {
        sel[t * top + j] = idx[j];
        if (t == t_me) w[t * top + j] = my_w[j] = val[j];
      }
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n * top; i += blockDim.x) {
    const int e = sel[i];
    for (int j = 0; j < top; ++j) {
      const int me = sel[t_me * top + j];
      if (e < me) atomicAdd(&my_off[j], 1);
      if (e == me && i < t_me * top + j) atomicAdd(&my_before[j], 1);
    }
    if (t_me == 0) atomicAdd(&count[e], 1);
  }
  __syncthreads();
  for (int j = 0; j < top; ++j) {
    const int at = my_off[j] + my_before[j];
    if (threadIdx.x == 0) place[t_me * top + j] = at;
    copy_row(hg + at * ldg, h + t_me * ldh, W, scale_in ? my_w[j] : 1.f);
  }
  if (t_me == 0 && warp == 0) {
    int run = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int c = e0 + lane < E ? count[e0 + lane] : 0;
      int x = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, o);
        if (lane >= o) x += y;
      }
      if (e0 + lane < E) off[e0 + lane] = run + x - c;
      run += __shfl_sync(0xffffffffu, x, 31);
    }
    if (lane == 0) off[E] = run;
  }
}

__global__ void moe_topk_kernel(const float* z, long long ldz, int n, int E, int top, int score,
                                int* sel, float* w) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (t >= n) return;
  int idx[kMoeMaxTop];
  float val[kMoeMaxTop];
  warp_topk(z + t * ldz, E, top, score, idx, val);
  if ((threadIdx.x & 31) == 0)
    for (int j = 0; j < top; ++j) {
      sel[t * top + j] = idx[j];
      w[t * top + j] = val[j];
    }
}

// CTA e numbers the tokens that chose expert e: place[i] for every choice i with sel[i] == e.
__global__ void __launch_bounds__(1024)
moe_group_kernel(const int* sel, int m, int E, int* off, int* place) {
  __shared__ int wsum[32];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int e = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int less = 0, eq = 0;
  for (int i = threadIdx.x; i < m; i += 1024) {
    const int s = sel[i];
    less += s < e;
    eq += s == e;
  }
  auto sum = [&](int v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();
    if (lane == 0) wsum[warp] = v;
    __syncthreads();
    int s = 0;
    for (int k = 0; k < 32; ++k) s += wsum[k];
    return s;
  };
  less = sum(less);
  eq = sum(eq);
  if (threadIdx.x == 0) {
    off[e] = less;
    if (e == E - 1) off[E] = less + eq;
  }
  int run = less;
  for (int i0 = 0; i0 < m; i0 += 1024) {
    const int i = i0 + threadIdx.x;
    const bool hit = i < m && sel[i] == e;
    const unsigned b = __ballot_sync(0xffffffffu, hit);
    __syncthreads();
    if (lane == 0) wsum[warp] = __popc(b);
    __syncthreads();
    int before = run, tot = 0;
    for (int k = 0; k < 32; ++k) {
      if (k < warp) before += wsum[k];
      tot += wsum[k];
    }
    if (hit) place[i] = before + __popc(b & ((1u << lane) - 1));
    run += tot;
  }
}

template <typename T>
__global__ void moe_gather_kernel(const T* h, long long ldh, int W, int top, const int* place,
                                  const float* w, int rows, T* hg, long long ldg) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const int t = blockIdx.x;
  for (int j = 0; j < top; ++j) {
    const int at = place[t * top + j];
    if (at >= 0 && at < rows)
      copy_row(hg + at * ldg, h + t * ldh, W, w ? w[(long long)t * top + j] : 1.f);
  }
}

template <typename T>
static int route(const float* z, long long ldz, int n, int E, int top, int score, int scale_in,
                 const void* h, long long ldh, int W, void* hg, long long ldg, int* off, int* place,
                 float* w, int* sel, cudaStream_t s) {
  if (n * top <= kMoeSmall && n <= 256)
    return (int)launch(moe_route_small_kernel<T>, dim3(n), dim3(kRouteThreads),
                       n * E <= kRouteLogits ? (size_t)n * E * 4 : 0, s, z, ldz, n, E, top, score,
                       scale_in, static_cast<const T*>(h), ldh, W, static_cast<T*>(hg), ldg, off, place, w);
  int r = (int)launch(moe_topk_kernel, dim3((n + 7) / 8), dim3(256), 0, s, z, ldz, n, E, top,
                      score, sel, w);
  if (r) return r;
  r = (int)launch(moe_group_kernel, dim3(E), dim3(1024), 0, s, sel, n * top, E, off, place);
  if (r) return r;
  return (int)launch(moe_gather_kernel<T>, dim3(n), dim3(256), 0, s, static_cast<const T*>(h), ldh,
                     W, top, place, scale_in ? w : nullptr, n * top, static_cast<T*>(hg), ldg);
}

}  // namespace e2h

// z fp32 [n, ldz] router logits (bias included); h [n, ldh]; hg [n * top, ldg]; off int [E + 1];
// place, w, sel [n, top]. score: 0 softmax over the chosen, 1 sigmoid; scale_in: the rows of hg carry
// their weight.
extern "C" int e2h_moe_route(const float* z, long long ldz, int n, int E, int top, int score,
                             int scale_in, const void* h, long long ldh, int W, void* hg,
                             long long ldg, int* off, int* place, float* w, int* sel, int is_bf16,
                             void* stream) {
  using namespace e2h;
  if (n <= 0 || E <= 0 || E > kMoeMaxExperts || top <= 0 || top > kMoeMaxTop || top > E) return -1;
  if ((long long)n * top > 0x3fffffff) return -1;
  return is_bf16 ? route<__nv_bfloat16>(z, ldz, n, E, top, score, scale_in, h, ldh, W, hg, ldg, off,
                                        place, w, sel, (cudaStream_t)stream)
                 : route<float>(z, ldz, n, E, top, score, scale_in, h, ldh, W, hg, ldg, off, place, w,
                                sel, (cudaStream_t)stream);
}
