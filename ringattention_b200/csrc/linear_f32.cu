// Linear layers in true fp32 on the CUDA cores: C[M,N] = A[M,K] * B[N,K]^T with the same epilogues as the bf16 GEMM
// (scale and bias by column, addend, squared relu, last columns to a second output). This is the matrix product of the engine's 32-bit mode; it
// never rounds an operand. 64 x 64 output tile per CTA, 4 x 4 outputs per thread, K in steps of 16 through shared memory.
#include "common/bounds.cuh"
#include "common/host_util.h"
#include "common/numeric.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace lin32 {

constexpr int TM = 64, TN = 64, TK = 16, THREADS = 256;

struct Params {
  const float* A; const float* B; float* C; const float* R; float* C2;
  long long lda, ldb, ldc, ldr, ldc2;
  int M, N, K;
  int n_split;  // columns from here on go to C2 (N: none)
  int relu2;    // C = max(v, 0)^2
  const float* bias;  // by column, or null
  float alpha;        // v = alpha * v + bias
};

__global__ void __launch_bounds__(THREADS) linear_f32_kernel(const Params p) {
  __shared__ float sA[TK][TM + 4], sB[TK][TN + 4];
  const int m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += TK) {
    for (int i = threadIdx.x; i < TM * TK; i += THREADS) {
      const int r = i / TK, k = i % TK;
      sA[k][r] = (m0 + r < p.M && k0 + k < p.K) ? p.A[(m0 + r) * p.lda + k0 + k] : 0.f;
      sB[k][r] = (n0 + r < p.N && k0 + k < p.K) ? p.B[(n0 + r) * p.ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = sA[k][ty * 4 + i];
        b[i] = sB[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const long long m = m0 + ty * 4 + i;
    if (m >= p.M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      float v = acc[i][j] * p.alpha;
      if (p.bias) v += p.bias[n];
      if (n >= p.n_split) {
        p.C2[m * p.ldc2 + n - p.n_split] = v;
        continue;
      }
      if (p.R) v += p.R[m * p.ldr + n];
      if (p.relu2) {
        v = fmaxf(v, 0.f);
        v *= v;
      }
      if (RA_IN_BOUNDS(m * p.ldc + n, 1, (p.M - 1) * p.ldc + p.N, kTagGemmStore)) p.C[m * p.ldc + n] = v;
    }
  }
}

}  // namespace lin32
}  // namespace ra

// R may be C (in-place accumulation). Leading dimensions in elements, no alignment rules.
extern "C" int ra_linear_f32(const float* A, const float* B, float* C, const float* R, float* C2, int M, int N, int K,
                             long long lda, long long ldb, long long ldc, long long ldr, long long ldc2, int n_split,
                             int relu2, const float* bias, float alpha, void* stream) {
  using namespace ra;
  if (M < 1 || N < 1 || K < 1 || (n_split < N && !C2)) {
    set_error("ra_linear_f32: bad shape");
    return kHostBadArg;
  }
  lin32::Params p{A, B, C, R, C2, lda, ldb, ldc, ldr, ldc2, M, N, K, n_split, relu2, bias, alpha};
  dim3 grid((N + lin32::TN - 1) / lin32::TN, (M + lin32::TM - 1) / lin32::TM);
  if (grid.y > 65535) {
    set_error("ra_linear_f32: too many rows");
    return kHostTooLarge;
  }
  lin32::linear_f32_kernel<<<grid, lin32::THREADS, 0, static_cast<cudaStream_t>(stream)>>>(p);
  return check_launch("linear_f32_kernel");
}
