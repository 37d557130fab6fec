// Parameter block of the gated-linear-attention kernels (gla.cu, gla_chunk.cu).
//
//   alpha_t = sigmoid(W_a2 a_t + b)^(1 / tau)            (per key channel, fp32)
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T              (per head, fp32 [dim, vdim])
//   o_t = S_t^T (qscale q_t)
//   y_t = o_t / rms(o_t) * w * silu(g_t)                 (replaces the gate columns)
//
// q, k (H x dim), v, g (H x vdim) are columns of a packed activation row; a_t (the low-rank input
// of the decay) is fp32. The state of a slot is fp32 [H, dim, vp], vp = vdim rounded up to 4 (the
// rounding columns stay zero). A token at position 0 starts from a zero state whatever the slot
// holds, so that slots need no clearing.
#pragma once
#include <stdint.h>

struct E2hGlaParams {
  void* act;               // T [n, ld]
  long long ld;
  int off_q, off_k, off_v, off_g;
  const float* a;          // fp32 [n, lda], r columns
  long long lda;
  int r;
  const void* w2;          // T [H * dim, ldw]
  long long ldw;
  const float* b2;         // fp32 [H * dim]
  float inv_tau, qscale, eps;
  const float* norm;       // fp32 [vdim]
  float* state;            // fp32 [slots, H, dim, vp]
  int slots, H, dim, vdim, vp;
  const int* pos;          // [n]
  const int* slot;         // [n]
  int n;
  int splits;              // decode: CTAs of a cluster that share a head's value columns
  // prompts: segment s holds tokens seg[s] .. seg[s + 1] of one sequence
  const int* seg;          // [n_seg + 1]
  int n_seg, seg_max;      // host bound of a segment's length
  float* logdec;           // fp32 [n, H * dim] scratch: log alpha (scan)
  float* o;                // fp32 [n, H * vdim] scratch
  // chunked form: 64-token chunks, chunk c of segment s in place seg[s] / 64 + s + c
  int chunks;              // places: n / 64 + n_seg + 1
  void* cq;                // bf16 [2 (high, low part)][chunks, H, 64, dim]: q e^{b_t}
  void* ck;                // bf16 [2][chunks, H, 64, dim]: k e^{b_end - b_t}
  void* ca;                // bf16 [2][chunks, H, 64, 64]: lower-triangular scores in the chunk
  float* cg;               // fp32 [chunks, H, dim]: e^{b_end}
  int* status;
};
