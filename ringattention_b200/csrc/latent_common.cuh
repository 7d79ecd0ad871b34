// Arguments and shared device code of the latent-attention kernels (latent_sm100.cu, latent_decode_sm100.cu).
#pragma once
#include "common/bounds.cuh"
#include "common/host_util.h"
#include "common/numeric.cuh"

namespace ra {
namespace latent {

struct Params {
  int B, T, H, dn, dr, dv, r;  // T tokens per sequence in this step; row b * T + t
  int r_pad, row_w;            // columns before the rotated key in a cached row, columns of a cached row
  int rot_dims;                // leading dimensions of the rotated part that turn
  void* proj;                  // (rows, ldp): q heads at off_q (dn + dr each), [c | k_rot] at off_c, gates at off_g
  long long ldp;
  int off_q, off_c, off_g;
  const void* c_norm;          // (r)
  const float* inv_freq;       // (rot_dims / 2)
  void* cache;                 // (B, S_max, row_w)
  long long S_max;
  const void *w_uk, *w_uv;     // (H * dn, ldw), (H * dv, ldw)
  long long ldw;
  const float* sink;           // (H), or null
  void* q_lat;                 // (rows, H, row_w): fp32, in the tensor-core form bf16
  float *o_part, *lse_part;    // (rows, H, splits, r), (rows, H, splits)
  int splits;
  void* out;                   // (rows, ldo)
  long long ldo;
  float eps, scale;
  const long long* pos;        // position of the step's first token
  int* status;
};

// Turn pair j of the `dr` rotated dimensions at src by position `pos` and store it at dst (which may be src).
template <typename T>
__device__ __forceinline__ void rotate_pair(const Params& p, const T* src, T* dst, int j, long long pos) {
  float u = to_f(src[2 * j]), v = 2 * j + 1 < p.dr ? to_f(src[2 * j + 1]) : 0.f;
  if (2 * j + 1 < p.rot_dims) {
    float sn, cs;
    sincosf(static_cast<float>(pos) * p.inv_freq[j], &sn, &cs);
    const float u2 = u * cs - v * sn;
    v = v * cs + u * sn;
    u = u2;
  }
  from_f(dst[2 * j], u);
  if (2 * j + 1 < p.dr) from_f(dst[2 * j + 1], v);
}

// The row's normed latent and rotated key part go to its place in the cache (whole CTA; `red`: 32 floats of shared memory).
template <typename T>
__device__ __forceinline__ void append_row(const Params& p, long long row, int b, long long pos, float* red) {
  const T* c = static_cast<const T*>(p.proj) + row * p.ldp + p.off_c;
  const int n = blockDim.x;
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.r; i += n) {
    const float x = to_f(c[i]);
    ss += x * x;
  }
  const float rs = 1.f / sqrtf(sum_block(ss, red) / p.r + p.eps);
  if (pos >= p.S_max || !RA_IN_BOUNDS(pos, 1, p.S_max, kTagDecodeCacheRow)) return;
  T* dst = static_cast<T*>(p.cache) + (b * p.S_max + pos) * p.row_w;
  for (int i = threadIdx.x; i < p.r_pad; i += n)
    from_f(dst[i], i < p.r ? to_f(c[i]) * rs * to_f(static_cast<const T*>(p.c_norm)[i]) : 0.f);
  for (int i = p.r_pad + p.dr + threadIdx.x; i < p.row_w; i += n) from_f(dst[i], 0.f);
  for (int j = threadIdx.x; j < (p.dr + 1) / 2; j += n) rotate_pair(p, c + p.r, dst + p.r_pad, j, pos);
}

int check(const Params* p);  // latent_sm100.cu

}  // namespace latent
}  // namespace ra
