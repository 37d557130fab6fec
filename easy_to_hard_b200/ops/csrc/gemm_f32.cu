// Linear layers in true 32-bit (FFMA, no reduced-precision tensor mode): the same parameter block
// and conventions as e2h_gemm_umma with fp32 operands, for models that run in fp32. 64 x 64 tiles,
// 256 threads with 4 x 4 outputs each. Epilogues: plain store, fp32 residual, SwiGLU on a dual
// operand, sigmoid gate; bias, activations, the tail columns, grouped and batched products, scale and
// soft cap as in gemm_umma.cu.
#include <cuda_runtime.h>
#include <stdint.h>

#include "gemm_umma.cuh"
#include "launch.cuh"
#include "ptx.cuh"

namespace e2h {

constexpr int kF32Tile = 64, kF32K = 16;

template <bool DUAL>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const E2hGemmParams p) {
  __shared__ float as[DUAL ? 2 : 1][kF32K][kF32Tile + 4], bs[kF32K][kF32Tile + 4];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int f0 = blockIdx.x * kF32Tile;
  int t0 = blockIdx.y * kF32Tile, t_end = p.T;
  const float* a = static_cast<const float*>(p.a);
  const float* a2 = static_cast<const float*>(p.a2);
  const float* b = static_cast<const float*>(p.b);
  if (p.n_groups > 0) {
    const int per = (p.group_tmax + kF32Tile - 1) / kF32Tile;
    const int g = blockIdx.y / per;
    t0 = p.group_off[g] + (blockIdx.y - g * per) * kF32Tile;
    t_end = min(p.group_off[g + 1], p.T);
    if (t0 >= t_end || t0 < 0) return;
    a += (long long)g * p.F * p.lda;
    if (DUAL) a2 += (long long)g * p.F * p.lda2;
  }
  int o_col = 0;
  if (p.n_batch > 0) {
    const int per = (p.T + kF32Tile - 1) / kF32Tile;
    const int g = blockIdx.y / per;
    t0 = (blockIdx.y - g * per) * kF32Tile;
    a += (long long)g * p.F * p.lda;
    b += g * p.batch_k;
    o_col = g * p.batch_out;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;   // features 4 tx.., tokens 4 ty..
  float acc[4][4], acc2[DUAL ? 4 : 1][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      acc[i][j] = 0.f;
      if constexpr (DUAL) acc2[i][j] = 0.f;
    }
  const int lk = threadIdx.x & 15, lr = threadIdx.x >> 4;   // loader: k column, row (of 16)
  for (int k0 = 0; k0 < p.K; k0 += kF32K) {
    const int k = k0 + lk;
#pragma unroll
    for (int r = 0; r < kF32Tile; r += 16) {
      const int f = f0 + lr + r, t = t0 + lr + r;
      as[0][lk][lr + r] = (f < p.F && k < p.K) ? a[(long long)f * p.lda + k] : 0.f;
      if constexpr (DUAL)
        as[1][lk][lr + r] = (f < p.F && k < p.K) ? a2[(long long)f * p.lda2 + k] : 0.f;
      bs[lk][lr + r] = (t < t_end && k < p.K) ? b[(long long)t * p.ldb + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kF32K; ++kk) {
      const float4 av = *reinterpret_cast<const float4*>(&as[0][kk][4 * tx]);
      const float4 bv = *reinterpret_cast<const float4*>(&bs[kk][4 * ty]);
      const float ar[4] = {av.x, av.y, av.z, av.w}, br[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(br[i], ar[j], acc[i][j]);
      if constexpr (DUAL) {
        const float4 cv = *reinterpret_cast<const float4*>(&as[1][kk][4 * tx]);
        const float cr[4] = {cv.x, cv.y, cv.z, cv.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc2[i][j] = fmaf(br[i], cr[j], acc2[i][j]);
      }
    }
    __syncthreads();
  }
  float* out = static_cast<float*>(p.out);
  const float* res = static_cast<const float*>(p.aux);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + 4 * ty + i;
    if (t >= t_end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int f = f0 + 4 * tx + j;
      if (f >= p.F) continue;
      float v = acc[i][j];
      if constexpr (DUAL) {
        v = v / (1.f + expf(-v)) * acc2[i][j];
      } else {
        if (p.bias) v += p.bias[f];
        if (p.act && f >= p.act_from && (p.tail_from <= 0 || f < p.tail_from)) {
          if (p.act == 1) {
            v = fmaxf(v, 0.f);
            v *= v;
          } else {
            v = gelu_erf(v);
          }
        }
        if (p.out_scale != 0.f) v *= p.out_scale;
        if (p.softcap != 0.f) v = p.softcap * tanhf(v / p.softcap);
        if (p.epi == E2H_EPI_GATE) v *= 1.f / (1.f + expf(-out[(long long)t * p.ldo + o_col + f]));
        if (p.epi == E2H_EPI_RESIDUAL_F32) v += res[(long long)t * p.ldo + f];
        if (p.tail_from > 0 && f >= p.tail_from) {
          p.tail[(long long)t * p.ldt + (f - p.tail_from)] = v;
          continue;
        }
      }
      out[(long long)t * p.ldo + o_col + f] = v;
    }
  }
}

}  // namespace e2h

extern "C" int e2h_gemm_f32(const E2hGemmParams* p, void* stream) {
  using namespace e2h;
  if (p->F <= 0 || p->T <= 0 || p->K <= 0 || p->a_mn_major || p->b_mn_major || p->scale) return -1;
  if (p->epi != E2H_EPI_STORE_F32 && p->epi != E2H_EPI_RESIDUAL_F32 && p->epi != E2H_EPI_SWIGLU &&
      p->epi != E2H_EPI_GATE)
    return -2;
  if (p->n_batch > 0 && (p->n_groups > 0 || p->dual || p->tail_from || p->bias || p->act)) return -2;
  if ((p->epi == E2H_EPI_SWIGLU) != (p->dual != 0)) return -2;
  if (p->tail_from && (!p->tail || p->epi != E2H_EPI_STORE_F32)) return -2;
  if (p->n_groups > 0 && (!p->group_off || p->group_tmax <= 0)) return -2;
  const int tt = p->n_groups > 0 ? p->n_groups * ((p->group_tmax + kF32Tile - 1) / kF32Tile)
                                 : (p->n_batch > 0 ? p->n_batch : 1) *
                                       ((p->T + kF32Tile - 1) / kF32Tile);
  if (tt > 65535) return -3;
  const dim3 grid((p->F + kF32Tile - 1) / kF32Tile, tt);
  if (p->dual)
    return (int)launch(gemm_f32_kernel<true>, grid, dim3(256), 0, (cudaStream_t)stream, *p);
  return (int)launch(gemm_f32_kernel<false>, grid, dim3(256), 0, (cudaStream_t)stream, *p);
}
