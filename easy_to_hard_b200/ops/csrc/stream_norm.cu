// The fp32 residual stream of the hybrid decoders: one kernel per layer boundary that builds (or
// completes) a token's residual row and writes its RMS norm for the next projections.
//
//   row  = emb[token] * emb_scale                         (tokens given: start of the network)
//        | x[row] + sum_j w[row, j] * y[place[row, j]]    (expert outputs of the layer before)
//        | x[row]
//   x[row] = row                                          (tokens or expert outputs, unless `rows`)
//   out[i] = row / sqrt(mean(row^2) + eps) * (offset + weight)
//
// `rows` picks the rows to normalise (the positions whose logits are wanted); output i then
// belongs to row rows[i] and x is left alone. `offset` is 1 for norms whose weight is stored
// around zero and 0 for plain ones. One CTA per output row; the row stays in shared memory
// between the two passes. In a decode step the kernel also turns the shared column counter and
// the left padding of every sequence into per-token positions.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <mutex>

#include "launch.cuh"
#include "ptx.cuh"
#include "scalar_types.cuh"

namespace e2h {

struct StreamNormParams {
  float* x;                 // [rows, W] fp32 residual
  const int* tokens;        // [n] or null
  const void* emb;          // T [vocab, lde]
  long long lde;
  int vocab;
  float emb_scale;
  const void* y;            // T [n * top, ldy] expert outputs or null
  long long ldy;
  const int* place;         // [n, top] row of y
  const float* ew;          // [n, top] weights or null (the outputs are weighted already)
  int top, y_rows;
  const int* rows;          // [n] or null
  int x_rows;
  const float* weight;      // fp32 [W]
  float offset, eps;
  void* out;                // T [n, ldo] or null
  long long ldo;
  int W;
  const int* col;           // decode: column of the newest token (device scalar) or null
  const int* left_pad;      // [n] or null
  int* pos_out;             // [n] = *col - left_pad
  int* status;
};

template <typename T>
__global__ void stream_norm_kernel(const StreamNormParams p) {
  extern __shared__ float row_s[];
  __shared__ float red[33];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int i = blockIdx.x;
  int r = i;
  if (p.rows) {
    r = p.rows[i];
    if (r < 0 || r >= p.x_rows) {
      if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
      r = 0;
    }
  }
  if (p.col && threadIdx.x == 0) {
    const int q = *p.col - (p.left_pad ? p.left_pad[i] : 0);
    p.pos_out[i] = q < 0 ? 0 : q;
  }
  float* x = p.x + (long long)r * p.W;
  const T* e = nullptr;
  if (p.tokens) {
    int tok = p.tokens[i];
    if (tok < 0 || tok >= p.vocab) {
      if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgs);
      tok = 0;
    }
    e = static_cast<const T*>(p.emb) + (long long)tok * p.lde;
  }
  const bool vec = (p.W & 3) == 0 && (p.lde & 3) == 0 && (p.ldy & 3) == 0 && (p.ldo & 3) == 0;
  float ss = 0.f;
  if (vec) {
    for (int c = threadIdx.x * 4; c < p.W; c += blockDim.x * 4) {
      float v[4];
      if (e) {
        load4(e + c, v);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] *= p.emb_scale;
      } else {
        load4(x + c, v);
      }
      if (p.y) {
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        for (int j = 0; j < p.top; ++j) {
          int at = p.place[(long long)r * p.top + j];
          at = min(max(at, 0), p.y_rows - 1);
          const float w = p.ew ? p.ew[(long long)r * p.top + j] : 1.f;
          float u[4];
          load4(static_cast<const T*>(p.y) + at * p.ldy + c, u);
#pragma unroll
          for (int k = 0; k < 4; ++k) s[k] += w * u[k];
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] += s[k];
      }
      if (!p.rows && (e || p.y)) store4(x + c, v);
      store4(row_s + c, v);
#pragma unroll
      for (int k = 0; k < 4; ++k) ss += v[k] * v[k];
    }
  } else {
    for (int c = threadIdx.x; c < p.W; c += blockDim.x) {
      float v = e ? to_f(e[c]) * p.emb_scale : x[c];
      if (p.y) {
        float s = 0.f;
        for (int j = 0; j < p.top; ++j) {
          int at = p.place[(long long)r * p.top + j];
          at = min(max(at, 0), p.y_rows - 1);
          s += (p.ew ? p.ew[(long long)r * p.top + j] : 1.f) *
               to_f(static_cast<const T*>(p.y)[at * p.ldy + c]);
        }
        v += s;
      }
      if (!p.rows && (e || p.y)) x[c] = v;
      row_s[c] = v;
      ss += v * v;
    }
  }
  if (!p.out) return;
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / p.W + p.eps);
  T* o = static_cast<T*>(p.out) + (long long)i * p.ldo;
  if (vec) {
    for (int c = threadIdx.x * 4; c < p.W; c += blockDim.x * 4) {
      float v[4], w[4];
      load4(row_s + c, v);
      load4(p.weight + c, w);
#pragma unroll
      for (int k = 0; k < 4; ++k) v[k] = v[k] * rstd * (p.offset + w[k]);
      store4(o + c, v);
    }
  } else {
    for (int c = threadIdx.x; c < p.W; c += blockDim.x)
      o[c] = from_f<T>(row_s[c] * rstd * (p.offset + p.weight[c]));
  }
}

template <typename T>
static int stream_norm_launch(const StreamNormParams& p, int n, cudaStream_t stream) {
  const size_t smem = (size_t)p.W * 4;
  if (smem > 200 * 1024) return -2;
  auto kern = stream_norm_kernel<T>;
  static std::once_flag once;
  static cudaError_t err = cudaSuccess;
  std::call_once(once, [&] {
    err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  });
  if (err != cudaSuccess) return (int)err;
  const int per = (p.W + 3) / 4;
  const int threads = per >= 512 ? 512 : per >= 256 ? 256 : 128;
  return (int)launch(kern, dim3(n), dim3(threads), smem, stream, p);
}

}  // namespace e2h

extern "C" int e2h_stream_norm(const e2h::StreamNormParams* p, int n, int is_bf16, void* stream) {
  if (n <= 0 || p->W <= 0 || !p->x || !p->status) return -1;
  if (p->y && (!p->place || p->top <= 0 || p->y_rows <= 0)) return -1;
  return is_bf16 ? e2h::stream_norm_launch<__nv_bfloat16>(*p, n, (cudaStream_t)stream)
                 : e2h::stream_norm_launch<float>(*p, n, (cudaStream_t)stream);
}
