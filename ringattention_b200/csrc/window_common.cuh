// Arguments of the windowed-attention kernels (window_sm100.cu, window_decode_sm100.cu).
#pragma once
#include "common/bounds.cuh"
#include "common/host_util.h"
#include "common/numeric.cuh"

namespace ra {
namespace window {

struct Params {
  int B, T, H, G, dk, dv;      // T tokens per sequence in this step; row b * T + t; H query heads share G key/value heads
  int rot_half;                // pairs (i, i + rot_half), i < rot_half, of a head turn
  void* proj;                  // (rows, ldp): query, key and value heads at off_q, off_k, off_v
  long long ldp;
  int off_q, off_k, off_v;
  const void *q_norm, *k_norm; // gains over all query (key) dimensions of a row
  const float* inv_freq;       // (rot_half)
  // ring of R rows per head: position p lives in row p % R; rows are kw (vw) elements wide, padding is zero
  void *k_cache, *v_cache;     // (B, G, R, kw), (B, G, R, vw)
  int R, kw, vw;
  int window;                  // a query sees keys at distances 0 .. window - 1
  const float* sink;           // (H)
  void* out;                   // (rows, ldo)
  long long ldo;
  float eps, scale;
  const long long* pos;        // position of the step's first token
  int splits;                  // decode: CTAs of a cluster
  long long n_max;             // decode: upper bound of the visible keys
};

// eight consecutive bf16 numbers (16-byte aligned)
struct Piece {
  uint4 u;
};
__device__ __forceinline__ Piece load_piece(const __nv_bfloat16* p) { return {*reinterpret_cast<const uint4*>(p)}; }
__device__ __forceinline__ void unpack(const Piece& s, float (&f)[8]) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&s.u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 v = __bfloat1622float2(h[i]);
    f[2 * i] = v.x;
    f[2 * i + 1] = v.y;
  }
}
__device__ __forceinline__ Piece pack(const float (&f)[8]) {
  Piece s;
  uint32_t* w = reinterpret_cast<uint32_t*>(&s.u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&v);
  }
  return s;
}
__device__ __forceinline__ float square_sum(const Piece& s) {
  float f[8], a = 0.f;
  unpack(s, f);
#pragma unroll
  for (int e = 0; e < 8; ++e) a += f[e] * f[e];
  return a;
}
// A head's pieces in units: unit u < half / 8 is the pair of pieces u and u + half / 8, which turn; the units after it are
// pieces u + half / 8 that pass. `lo` (turning units) and `hi` are normed by rs and the gains gl and gh, and turned.
__device__ __forceinline__ void norm_turn(Piece& lo, Piece& hi, const float (&gl)[8], const float (&gh)[8], float rs, int u,
                                          int h8, const float* sn, const float* cs) {
  float x[8], y[8];
  unpack(hi, x);
#pragma unroll
  for (int e = 0; e < 8; ++e) x[e] *= rs * gh[e];
  if (u < h8) {
    unpack(lo, y);
    float s[8], c[8];
    *reinterpret_cast<float4*>(s) = load4(sn + u * 8);
    *reinterpret_cast<float4*>(s + 4) = load4(sn + u * 8 + 4);
    *reinterpret_cast<float4*>(c) = load4(cs + u * 8);
    *reinterpret_cast<float4*>(c + 4) = load4(cs + u * 8 + 4);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float a = y[e] * rs * gl[e];
      y[e] = a * c[e] - x[e] * s[e];
      x[e] = x[e] * c[e] + a * s[e];
    }
    lo = pack(y);
  }
  hi = pack(x);
}
// Two sums over the CTA at once; `red` holds 64 floats. Every thread gets the results.
__device__ __forceinline__ float2 sum_block2(float a, float b, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  a = sum_warp(a);
  b = sum_warp(b);
  __syncthreads();
  if (lane == 0) {
    red[warp] = a;
    red[32 + warp] = b;
  }
  __syncthreads();
  return make_float2(sum_warp(lane < nw ? red[lane] : 0.f), sum_warp(lane < nw ? red[32 + lane] : 0.f));
}

int check(const Params* p);  // window_sm100.cu

}  // namespace window
}  // namespace ra
