// Arguments and shared device code of the routed-expert kernels (moe.cu, moe_gemm_sm100.cu).
#pragma once
#include "common/bounds.cuh"
#include "common/host_util.h"
#include "common/numeric.cuh"

namespace ra {
namespace moe {

constexpr int MAX_EXPERTS = 1024, MAX_TOP = 32;

struct Params {
  int rows, d, dp;             // tokens; model width and its padded form (the K of gate and up, leading dimension of h)
  int E, top, F, Fs;           // experts, experts per token, padded widths of the routed and of the shared expert (Fs 0: none)
  const void* h;               // (rows, dp) normed input
  const float* logits;         // (rows, ld_logits) router logits
  long long ld_logits;
  const void *gu, *down;       // (E, 2 F, dp) gate rows, then up rows; (E, dp, F)
  const void *sh_gu, *sh_down; // (2 Fs, dp); (dp, Fs)
  int* ids;                    // (rows, top) chosen experts
  float* weight;               // (rows, top) their scores
  void* act;                   // few rows: (rows, top * F + Fs); many rows: (128 row tiles, F), see moe_gemm_sm100.cu
  float* x;                    // (rows, ldx) residual stream
  long long ldx;
  // many rows: entries t * top + k by expert, list[e * rows + i], i < count[e]
  int *count, *list;
  void* y;                     // (rows * top, dp): expert outputs by entry
  int* status;
};

// The warp picks the `top` experts with the largest logits (ties: the lower index) and their sigmoid scores; lane k returns
// the k-th. `key` holds E words of shared memory that belong to this warp. Call with all lanes.
__device__ __forceinline__ void choose(const float* z, int E, int top, uint32_t* key, int& id, float& score) {
  const int lane = threadIdx.x & 31;
  for (int e = lane; e < E; e += 32) {
    const uint32_t u = __float_as_uint(z[e]);
    key[e] = max(1u, (u >> 31) ? ~u : u | 0x80000000u);  // the order of the numbers; 0 is left for "taken"
  }
  __syncwarp();
  id = 0;
  for (int k = 0; k < top; ++k) {
    uint32_t best = 0;
    int at = E;
    for (int e = lane; e < E; e += 32)
      if (key[e] > best) {
        best = key[e];
        at = e;
      }
    const uint32_t mx = __reduce_max_sync(0xffffffffu, best);
    const int e = min(static_cast<int>(__reduce_min_sync(0xffffffffu, best == mx ? static_cast<unsigned>(at) : 0x7fffffffu)),
                      E - 1);
    if (lane == k) id = e;
    if (lane == 0) key[e] = 0;
    __syncwarp();
  }
  score = lane < top ? sigmoid_f(z[id]) : 0.f;
}

int check(const Params* p);  // moe.cu

}  // namespace moe
}  // namespace ra
