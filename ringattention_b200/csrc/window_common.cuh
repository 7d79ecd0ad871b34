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

int check(const Params* p);  // window_sm100.cu

}  // namespace window
}  // namespace ra
