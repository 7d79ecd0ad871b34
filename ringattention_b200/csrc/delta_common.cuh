// Arguments and shared device code of the gated-delta kernels (delta_sm100.cu, delta_chunk_sm100.cu).
#pragma once
#include "common/bounds.cuh"
#include "common/host_util.h"
#include "common/numeric.cuh"

namespace ra {
namespace delta {

struct Params {
  int B, T, H, G, dk, dv, taps;  // T tokens per sequence in this step; row b * T + t
  const void* proj;              // (rows, ldp): columns off_q / off_k / off_v / off_g
  long long ldp;
  int off_q, off_k, off_v, off_g;
  const float* ba;               // (rows, ldba): beta's projection at 0, the decay's at off_a
  long long ldba;
  int off_a;
  const void *conv_q, *conv_k, *conv_v;  // (channels, taps)
  const void *a_log, *dt_bias, *norm_w;  // (H), (H), (dv)
  float* ring;                   // (B, taps, C) with C = 2 G dk + H dv, channels in the order q, k, v
  float* state;                  // (B, H, dv, dk)
  float *q, *k, *v, *gb, *o;     // (rows, G, dk) x 2, (rows, H, dv), (rows, H, 2), (rows, H, dv)
  void* out;                     // (rows, ldo)
  long long ldo;
  float eps, q_scale;
  const long long* pos;          // position of the step's first token
  // workspace of the chunked form, n_chunks = ceil(T / 64) (delta_chunk_sm100.cu)
  int n_chunks;
  void* ws_qk;                   // (B, G, n_chunks) images of q and k
  void* ws_w;                    // (B, H, n_chunks) images of -W
  float* ws_u;                   // (B, H, n_chunks, dv, 64)
  void* ws_m;                    // (B, H, n_chunks) images of M, and the decays from the chunk's start
  float* ws_d;                   // (B, H, n_chunks, 68): decays to the chunk's end, the chunk's whole decay
  int* status;
};

__device__ __forceinline__ int ring_slot(long long p, int taps) { return static_cast<int>(p % taps); }

// silu(convolution) of one channel at token t of the step. `c`: channel in the ring's order, `col`: its projection column.
template <typename T>
__device__ __forceinline__ float conv_silu(const Params& p, const T* proj_b, const float* ring_b, const T* w, int t,
                                           long long pos0, int C, int c, int col) {
  float s = 0.f;
  for (int j = 0; j < p.taps; ++j) {
    const int tt = t - (p.taps - 1 - j);
    float x = 0.f;
    if (tt >= 0)
      x = to_f(proj_b[tt * p.ldp + col]);
    else if (pos0 + tt >= 0)
      x = ring_b[static_cast<long long>(ring_slot(pos0 + tt, p.taps)) * C + c];
    s = fmaf(to_f(w[j]), x, s);
  }
  return silu_f(s);
}

// logarithm of the decay g
__device__ __forceinline__ float log_decay(float a, float a_log, float dt) { return -expf(a_log) * softplus_f(a + dt); }

// The rows of the step's last tokens go into the convolution ring; `me` of `total` threads of sequence b.
template <typename T>
__device__ __forceinline__ void save_ring(const Params& p, int b, long long pos0, int me, int total) {
  const int C = 2 * p.G * p.dk + p.H * p.dv;
  const int keep = min(p.T, p.taps);
  const T* proj_b = static_cast<const T*>(p.proj) + static_cast<long long>(b) * p.T * p.ldp;
  float* ring_b = p.ring + static_cast<long long>(b) * p.taps * C;
  for (int i = me; i < keep * C; i += total) {
    const int t = p.T - keep + i / C, c = i % C, nq = p.G * p.dk;
    const int src = c < nq ? p.off_q + c : (c < 2 * nq ? p.off_k + c - nq : p.off_v + c - 2 * nq);
    ring_b[static_cast<long long>(ring_slot(pos0 + t, p.taps)) * C + c] = to_f(proj_b[t * p.ldp + src]);
  }
}

int check(const Params* p);  // delta_sm100.cu

}  // namespace delta
}  // namespace ra
