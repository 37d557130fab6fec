// Gated linear attention (equations in gla.cuh).
//
//   gla_step   decode: one token per sequence, a cluster of CTAs per (sequence, head). Decay,
//              state update, output, per-head norm and output gate in one kernel; the state is
//              read and written once (a pure HBM stream), the sum of squares of the norm crosses
//              the cluster through distributed shared memory.
//   gla_decay  prompts: log alpha of every token and channel.
//   gla_scan   prompts, exact fp32 recurrence: a CTA owns 16 value columns of a head of one
//              sequence, the state stays in registers, tokens are staged in batches. Serves fp32
//              models, short portions and head sizes that the chunked kernel does not take.
//   gla_out    prompts: norm and gate of the scratch output.
#include <cooperative_groups.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <string.h>

#include "gla.cuh"
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar_types.cuh"

namespace cg = cooperative_groups;

namespace e2h {

__device__ __forceinline__ float log_sigmoid(float z) {
  return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

template <typename T>
__device__ __forceinline__ float decay_logit(const T* w, const float* a, int r, float b) {
  float z = 0.f;
  int i = 0;
  if ((r & 7) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0) {
    for (; i < r; i += 8) {
      float v[8];
      load8(w + i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) z = fmaf(v[e], a[i + e], z);
    }
  }
  for (; i < r; ++i) z = fmaf(to_f(w[i]), a[i], z);
  return z + b;
}

constexpr int kStepThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kStepThreads) gla_step_kernel(const E2hGlaParams p) {
  extern __shared__ __align__(16) float gs[];
  cg::cluster_group cluster = cg::this_cluster();
  __shared__ float red[33];
  __shared__ float ss_s;
  const int rank = blockIdx.x, head = blockIdx.y, t = blockIdx.z;
  const int vb = (p.vp / 4 + p.splits - 1) / p.splits * 4;   // value columns of this CTA
  const int v0 = rank * vb, nv = max(min(vb, p.vp - v0), 0);
  const int nq4 = vb / 4;                                     // column quads
  const int groups = kStepThreads / nq4 > 0 ? kStepThreads / nq4 : 1;
  const int dp = (p.dim + 3) / 4 * 4;   // every array starts on a 16-byte boundary
  float* al = gs;                       // [dim] decay
  float* ks = al + dp;                  // [dim]
  float* qs = ks + dp;                  // [dim]
  float* as = qs + dp;                  // [r]
  float* vs = as + (p.r + 3) / 4 * 4;   // [vb]
  float* os = vs + vb;                  // [groups][vb]
  pdl_launch_dependents();
  pdl_wait_prior();
  int slot = p.slot[t];
  const int pos = p.pos[t];
  if (slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    slot = min(max(slot, 0), p.slots - 1);
  }
  T* row = static_cast<T*>(p.act) + t * p.ld;
  for (int i = threadIdx.x; i < p.r; i += kStepThreads) as[i] = p.a[t * p.lda + i];
  for (int i = threadIdx.x; i < p.dim; i += kStepThreads) {
    ks[i] = to_f(row[p.off_k + head * p.dim + i]);
    qs[i] = to_f(row[p.off_q + head * p.dim + i]) * p.qscale;
  }
  for (int i = threadIdx.x; i < nv; i += kStepThreads)
    vs[i] = v0 + i < p.vdim ? to_f(row[p.off_v + head * p.vdim + v0 + i]) : 0.f;
  __syncthreads();
  for (int i = threadIdx.x; i < p.dim; i += kStepThreads) {
    const long long c = (long long)head * p.dim + i;
    const float z = decay_logit(static_cast<const T*>(p.w2) + c * p.ldw, as, p.r, p.b2[c]);
    al[i] = expf(log_sigmoid(z) * p.inv_tau);
  }
  __syncthreads();
  float* S = p.state + ((long long)slot * p.H + head) * p.dim * p.vp + v0;
  const bool fresh = pos == 0;
  for (int qd0 = 0; qd0 < nq4; qd0 += kStepThreads) {       // one round unless vb > 1024
    const int qd = qd0 + threadIdx.x % (nq4 < kStepThreads ? nq4 : kStepThreads);
    const int grp = threadIdx.x / (nq4 < kStepThreads ? nq4 : kStepThreads);
    if (grp < groups && qd < nq4 && qd * 4 < nv) {
      float o[4] = {0.f, 0.f, 0.f, 0.f};
      const float v[4] = {vs[qd * 4], vs[qd * 4 + 1], vs[qd * 4 + 2], vs[qd * 4 + 3]};
      constexpr int U = 8;
      for (int d0 = grp; d0 < p.dim; d0 += groups * U) {
        float s[U][4];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + u * groups;
          if (d < p.dim && !fresh) load4(S + (long long)d * p.vp + qd * 4, s[u]);
          else s[u][0] = s[u][1] = s[u][2] = s[u][3] = 0.f;
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + u * groups;
          if (d < p.dim) {
            const float a = al[d], k = ks[d], q = qs[d];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              s[u][e] = fmaf(a, s[u][e], k * v[e]);
              o[e] = fmaf(q, s[u][e], o[e]);
            }
            store4(S + (long long)d * p.vp + qd * 4, s[u]);
          }
        }
      }
      store4(os + grp * vb + qd * 4, o);
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < nv; i += kStepThreads) {
    float o = 0.f;
    for (int k = 0; k < groups; ++k) o += os[k * vb + i];
    vs[i] = o;                      // the value itself is no longer needed
    ss += o * o;
  }
  ss = block_sum(ss, red);
  if (p.splits > 1) {
    if (threadIdx.x == 0) ss_s = ss;
    cluster.sync();
    ss = 0.f;
    for (int k = 0; k < p.splits; ++k) ss += *cluster.map_shared_rank(&ss_s, k);
    cluster.sync();                 // peers may still read ss_s
  }
  const float rstd = 1.f / sqrtf(ss / p.vdim + p.eps);
  for (int i = threadIdx.x; i < nv; i += kStepThreads) {
    if (v0 + i >= p.vdim) continue;
    T* g = row + p.off_g + head * p.vdim + v0 + i;
    const float z = to_f(*g);
    *g = from_f<T>(vs[i] * rstd * p.norm[v0 + i] * (z * sigmoid_f(z)));
  }
}

constexpr int kDecTok = 16;

template <typename T>
__global__ void __launch_bounds__(128) gla_decay_kernel(const E2hGlaParams p) {
  extern __shared__ __align__(16) float a_s[];   // [kDecTok][rp]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int rp = (p.r + 3) / 4 * 4;
  const int t0 = blockIdx.y * kDecTok, nt = min(kDecTok, p.n - t0);
  for (int i = threadIdx.x; i < nt * p.r; i += 128)
    a_s[i / p.r * rp + i % p.r] = p.a[(long long)(t0 + i / p.r) * p.lda + i % p.r];
  __syncthreads();
  const int c = blockIdx.x * 128 + threadIdx.x, C = p.H * p.dim;
  if (c >= C) return;
  const T* w = static_cast<const T*>(p.w2) + (long long)c * p.ldw;
  const float b = p.b2[c];
  for (int t = 0; t < nt; ++t)
    p.logdec[(long long)(t0 + t) * C + c] =
        log_sigmoid(decay_logit(w, a_s + t * rp, p.r, b)) * p.inv_tau;
}

constexpr int kScanThreads = 128, kScanCols = 16;

// 8 lanes share a value column, each with NV x 4 of its state rows (rows (i * 8 + kg) * 4 + e).
template <typename T, int NV>
__global__ void __launch_bounds__(kScanThreads) gla_scan_kernel(const E2hGlaParams p) {
  constexpr int DP = NV * 32;                      // dim rounded up
  constexpr int kScanTok = NV > 4 ? 8 : 16;        // tokens staged at a time
  __shared__ __align__(16) float a_s[kScanTok][DP], k_s[kScanTok][DP], q_s[kScanTok][DP];
  __shared__ float v_s[kScanTok][kScanCols];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int head = blockIdx.y, sg = blockIdx.z;
  const int t_begin = p.seg[sg], t_end = p.seg[sg + 1];
  if (t_begin < 0 || t_end > p.n || t_begin >= t_end) return;
  const int slot = p.slot[t_begin];
  if (slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
    return;
  }
  const bool fresh = p.pos[t_begin] == 0;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int kg = lane & 7, vc = warp * 4 + (lane >> 3);
  const int col = blockIdx.x * kScanCols + vc;
  const bool col_ok = col < p.vp;
  float* S = p.state + ((long long)slot * p.H + head) * p.dim * p.vp + col;
  float s[NV * 4];
#pragma unroll
  for (int i = 0; i < NV * 4; ++i) {
    const int d = ((i >> 2) * 8 + kg) * 4 + (i & 3);
    s[i] = (!fresh && col_ok && d < p.dim) ? S[(long long)d * p.vp] : 0.f;
  }
  const int C = p.H * p.dim;
  for (int t0 = t_begin; t0 < t_end; t0 += kScanTok) {
    const int nt = min(kScanTok, t_end - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * DP; i += kScanThreads) {
      const int t = i / DP, d = i - t * DP;
      float a = 1.f, k = 0.f, q = 0.f;
      if (d < p.dim) {
        const T* row = static_cast<const T*>(p.act) + (long long)(t0 + t) * p.ld + head * p.dim + d;
        a = expf(p.logdec[(long long)(t0 + t) * C + head * p.dim + d]);
        k = to_f(row[p.off_k]);
        q = to_f(row[p.off_q]) * p.qscale;
      }
      a_s[t][d] = a;
      k_s[t][d] = k;
      q_s[t][d] = q;
    }
    for (int i = threadIdx.x; i < nt * kScanCols; i += kScanThreads) {
      const int t = i / kScanCols, c = blockIdx.x * kScanCols + i % kScanCols;
      v_s[t][i % kScanCols] =
          c < p.vdim ? to_f(static_cast<const T*>(
                           p.act)[(long long)(t0 + t) * p.ld + p.off_v + head * p.vdim + c])
                     : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float v = v_s[t][vc];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        float a[4], k[4], q[4];
        load4(&a_s[t][(i * 8 + kg) * 4], a);
        load4(&k_s[t][(i * 8 + kg) * 4], k);
        load4(&q_s[t][(i * 8 + kg) * 4], q);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[4 * i + e] = fmaf(a[e], s[4 * i + e], k[e] * v);
          o = fmaf(q[e], s[4 * i + e], o);
        }
      }
#pragma unroll
      for (int m = 1; m < 8; m <<= 1) o += __shfl_xor_sync(0xffffffffu, o, m);
      if (kg == 0 && col < p.vdim)
        p.o[((long long)(t0 + t) * p.H + head) * p.vdim + col] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < NV * 4; ++i) {
    const int d = ((i >> 2) * 8 + kg) * 4 + (i & 3);
    if (col_ok && d < p.dim) S[(long long)d * p.vp] = s[i];
  }
}

// One warp per (token, head). NV > 0: value columns in multiples of 4, at most NV x 128, whose
// output and gate are fetched at once; 0: any size.
template <typename T, int NV>
__global__ void __launch_bounds__(256) gla_out_kernel(const E2hGlaParams p) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const long long w = blockIdx.x * 8LL + (threadIdx.x >> 5);
  if (w >= (long long)p.n * p.H) return;
  const int lane = threadIdx.x & 31;
  const long long t = w / p.H;
  const int head = (int)(w - t * p.H);
  const float* o = p.o + w * p.vdim;
  T* g = static_cast<T*>(p.act) + t * p.ld + p.off_g + (long long)head * p.vdim;
  float ss = 0.f;
  if constexpr (NV > 0) {
    float x[NV][4], z[NV][4];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = lane * 4 + k * 128;
      if (i < p.vdim) {
        load4(o + i, x[k]);
        load4(g + i, z[k]);
#pragma unroll
        for (int e = 0; e < 4; ++e) ss += x[k][e] * x[k][e];
      }
    }
    ss = warp_sum(ss);
    const float rstd = 1.f / sqrtf(ss / p.vdim + p.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = lane * 4 + k * 128;
      if (i < p.vdim) {
        float wt[4];
        load4(p.norm + i, wt);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[k][e] *= rstd * wt[e] * (z[k][e] * sigmoid_f(z[k][e]));
        store4(g + i, x[k]);
      }
    }
  } else {
    for (int i = lane; i < p.vdim; i += 32) ss += o[i] * o[i];
    ss = warp_sum(ss);
    const float rstd = 1.f / sqrtf(ss / p.vdim + p.eps);
    for (int i = lane; i < p.vdim; i += 32) {
      const float z = to_f(g[i]);
      g[i] = from_f<T>(o[i] * rstd * p.norm[i] * (z * sigmoid_f(z)));
    }
  }
}

template <typename T>
static int gla_out(const E2hGlaParams& p, cudaStream_t s) {
  const long long warps = (long long)p.n * p.H;
  const dim3 grid((unsigned)((warps + 7) / 8));
  const bool vec = (p.vdim & 3) == 0 && (p.ld & 3) == 0 && (p.off_g & 3) == 0;
  if (vec && p.vdim <= 128) return (int)launch(gla_out_kernel<T, 1>, grid, dim3(256), 0, s, p);
  if (vec && p.vdim <= 256) return (int)launch(gla_out_kernel<T, 2>, grid, dim3(256), 0, s, p);
  if (vec && p.vdim <= 512) return (int)launch(gla_out_kernel<T, 4>, grid, dim3(256), 0, s, p);
  return (int)launch(gla_out_kernel<T, 0>, grid, dim3(256), 0, s, p);
}

static int gla_check(const E2hGlaParams& p) {
  if (p.n <= 0 || p.H <= 0 || p.dim <= 0 || p.dim > 256 || p.vdim <= 0 || p.r <= 0 || p.r > 1024)
    return -1;
  if (p.vp < p.vdim || p.vp % 4 || !p.state || !p.status) return -1;
  return 0;
}

template <typename T>
static int step(const E2hGlaParams& p, cudaStream_t stream) {
  const int vb = (p.vp / 4 + p.splits - 1) / p.splits * 4;
  const int groups = kStepThreads / (vb / 4) > 0 ? kStepThreads / (vb / 4) : 1;
  const size_t smem = 4 * ((size_t)3 * ((p.dim + 3) / 4 * 4) + (p.r + 3) / 4 * 4 + vb + (size_t)groups * vb);
  if (smem > 48 * 1024 || vb > 1024) return -2;
  cudaLaunchConfig_t cfg;
  memset(&cfg, 0, sizeof(cfg));
  cfg.gridDim = dim3(p.splits, p.H, p.n);
  cfg.blockDim = dim3(kStepThreads);
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
  return (int)cudaLaunchKernelEx(&cfg, gla_step_kernel<T>, p);
}

template <typename T>
static int scan(const E2hGlaParams& p, cudaStream_t s) {
  const dim3 grid((p.vp + kScanCols - 1) / kScanCols, p.H, p.n_seg);
  if (p.dim <= 32) return (int)launch(gla_scan_kernel<T, 1>, grid, dim3(kScanThreads), 0, s, p);
  if (p.dim <= 64) return (int)launch(gla_scan_kernel<T, 2>, grid, dim3(kScanThreads), 0, s, p);
  if (p.dim <= 128) return (int)launch(gla_scan_kernel<T, 4>, grid, dim3(kScanThreads), 0, s, p);
  return (int)launch(gla_scan_kernel<T, 8>, grid, dim3(kScanThreads), 0, s, p);
}

}  // namespace e2h

extern "C" {

int e2h_gla_step(const E2hGlaParams* p, int is_bf16, void* stream) {
  using namespace e2h;
  int r = gla_check(*p);
  if (r) return r;
  if (p->splits < 1 || p->splits > 8 || p->n > 65535) return -1;
  return is_bf16 ? step<__nv_bfloat16>(*p, (cudaStream_t)stream)
                 : step<float>(*p, (cudaStream_t)stream);
}

int e2h_gla_decay(const E2hGlaParams* p, int is_bf16, void* stream) {
  using namespace e2h;
  int r = gla_check(*p);
  if (r) return r;
  if (!p->logdec) return -1;
  const dim3 grid((p->H * p->dim + 127) / 128, (p->n + kDecTok - 1) / kDecTok);
  const size_t smem = (size_t)kDecTok * ((p->r + 3) / 4 * 4) * 4;
  if (grid.y > 65535 || smem > 48 * 1024) return -2;
  return is_bf16 ? (int)launch(gla_decay_kernel<__nv_bfloat16>, grid, dim3(128), smem,
                               (cudaStream_t)stream, *p)
                 : (int)launch(gla_decay_kernel<float>, grid, dim3(128), smem,
                               (cudaStream_t)stream, *p);
}

int e2h_gla_scan(const E2hGlaParams* p, int is_bf16, void* stream) {
  using namespace e2h;
  int r = gla_check(*p);
  if (r) return r;
  if (!p->logdec || !p->o || !p->seg || p->n_seg <= 0 || p->n_seg > 65535) return -1;
  return is_bf16 ? scan<__nv_bfloat16>(*p, (cudaStream_t)stream)
                 : scan<float>(*p, (cudaStream_t)stream);
}

int e2h_gla_out(const E2hGlaParams* p, int is_bf16, void* stream) {
  using namespace e2h;
  int r = gla_check(*p);
  if (r) return r;
  if (!p->o) return -1;
  return is_bf16 ? gla_out<__nv_bfloat16>(*p, (cudaStream_t)stream)
                 : gla_out<float>(*p, (cudaStream_t)stream);
}

}  // extern "C"
