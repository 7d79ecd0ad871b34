// The 32-bit residual stream: embedding lookup into it, and RMS norms out of it. A norm call writes one or two
// normalised copies of the same rows (a layer whose mixer and feed-forward read the same input through norms of their
// own needs two) and reads the rows once; gains are stored either as they are or around zero (`gain_offset` 1). Also the rows
// that enter a pass over looped layers ([stream | embedding] side by side, one product's input), and the gated activation of
// fp32 engines.
#include "common/bounds.cuh"
#include "common/host_util.h"
#include "common/numeric.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace resid {

template <typename T>
__global__ void embed_kernel(const int* __restrict__ tokens, const T* __restrict__ table, long long ld_table,
                             float* __restrict__ x, long long ldx, int d, int vocab, bool vec) {
  const long long r = blockIdx.x;
  int tok = tokens[r];
  if (!RA_IN_BOUNDS(tok, 1, vocab, kTagEmbeddingToken)) tok = 0;
  tok = min(max(tok, 0), vocab - 1);
  const T* src = table + tok * ld_table;
  float* dst = x + r * ldx;
  if (vec) {  // ldx, ld_table multiples of four; the last group may hold padding
#pragma unroll 4
    for (int i = threadIdx.x * 4; i + 3 < d; i += blockDim.x * 4) store4(dst + i, load4(src + i));
    for (int i = (d & ~3) + threadIdx.x; i < ldx; i += blockDim.x) dst[i] = i < d ? to_f(src[i]) : 0.f;
  } else {
    for (int i = threadIdx.x; i < ldx; i += blockDim.x) dst[i] = i < d ? to_f(src[i]) : 0.f;
  }
}

// out (rows, 2 dp) = [x | table[token]], each half padded with zeros from d on
template <typename T>
__global__ void pair_kernel(const int* __restrict__ tokens, const T* __restrict__ table, long long ld_table,
                            const float* __restrict__ x, long long ldx, T* __restrict__ out, int d, int dp, int vocab) {
  const long long r = blockIdx.x;
  const int tok = min(max(tokens[r], 0), vocab - 1);
  const T* src = table + tok * ld_table;
  T* dst = out + r * 2 * dp;
  if (!RA_IN_BOUNDS(tokens[r], 1, vocab, kTagEmbeddingToken)) return;
  if (ld_table % 4 == 0 && d % 4 == 0) {
    for (int i = threadIdx.x * 4; i < dp; i += blockDim.x * 4) {
      const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
      store4(dst + i, i < d ? load4(x + r * ldx + i) : z);
      store4(dst + dp + i, i < d ? load4(src + i) : z);
    }
    return;
  }
  for (int i = threadIdx.x; i < dp; i += blockDim.x) {
    from_f(dst[i], i < d ? x[r * ldx + i] : 0.f);
    dst[dp + i] = i < d ? src[i] : T(0.f);
  }
}

// y (rows, F) = silu(gu[:, :F]) * gu[:, F:], fp32
__global__ void gated_act_kernel(const float* __restrict__ gu, float* __restrict__ y, long long ldy, int F) {
  const long long r = blockIdx.x;
  for (int i = threadIdx.x; i < F; i += blockDim.x)
    if (RA_IN_BOUNDS(i, 1, ldy, kTagSwiglu)) y[r * ldy + i] = silu_f(gu[r * 2 * F + i]) * gu[r * 2 * F + F + i];
}

struct NormParams {
  const float* x;
  const int* rows_idx;  // row r of the output comes from row rows_idx[r] of x, or null
  const void *w1, *w2;
  void *y1, *y2;        // y2 null: one output
  long long ldx, ldy;
  int d, dp;            // columns that count, and padded columns (multiple of 4, zero in x) that are written
  float eps, gain_offset;
};

template <typename T, int MAXV>
__global__ void __launch_bounds__(256) norm_kernel(const NormParams p) {
  __shared__ float red[32];
  const long long r = blockIdx.x;
  const float* xr = p.x + (p.rows_idx ? p.rows_idx[r] : r) * p.ldx;
  const int nv = p.dp >> 2;
  float4 v[MAXV];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < MAXV; ++j) {
    const int i = threadIdx.x + j * 256;
    v[j] = i < nv ? load4(xr + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
  }
  const float rs = 1.f / sqrtf(sum_block(ss, red) / p.d + p.eps);
#pragma unroll
  for (int j = 0; j < MAXV; ++j) {
    const int i = threadIdx.x + j * 256;
    if (i >= nv || !RA_IN_BOUNDS(4 * i, 4, p.ldy, kTagRmsnorm)) continue;
    const float4 a = make_float4(v[j].x * rs, v[j].y * rs, v[j].z * rs, v[j].w * rs);
    float4 g = load4(static_cast<const T*>(p.w1) + 4 * i);
    store4(static_cast<T*>(p.y1) + r * p.ldy + 4 * i,
           make_float4(a.x * (p.gain_offset + g.x), a.y * (p.gain_offset + g.y), a.z * (p.gain_offset + g.z),
                       a.w * (p.gain_offset + g.w)));
    if (p.y2) {
      g = load4(static_cast<const T*>(p.w2) + 4 * i);
      store4(static_cast<T*>(p.y2) + r * p.ldy + 4 * i,
             make_float4(a.x * (p.gain_offset + g.x), a.y * (p.gain_offset + g.y), a.z * (p.gain_offset + g.z),
                         a.w * (p.gain_offset + g.w)));
    }
  }
}

template <typename T>
int launch_norm(const NormParams& p, int rows, cudaStream_t s) {
  const int nv = p.dp / 4;
  if (nv <= 256) norm_kernel<T, 1><<<rows, 256, 0, s>>>(p);
  else if (nv <= 512) norm_kernel<T, 2><<<rows, 256, 0, s>>>(p);
  else if (nv <= 1024) norm_kernel<T, 4><<<rows, 256, 0, s>>>(p);
  else if (nv <= 2048) norm_kernel<T, 8><<<rows, 256, 0, s>>>(p);
  else if (nv <= 4096) norm_kernel<T, 16><<<rows, 256, 0, s>>>(p);
  else {
    set_error("ra_norm_f32: more than 16384 columns");
    return kHostTooLarge;
  }
  return check_launch("norm_kernel");
}

}  // namespace resid
}  // namespace ra

// x (rows, ldx) fp32 <- table[token]; columns d..ldx are zeroed. `f32`: the table is fp32, else bf16.
extern "C" int ra_embed_f32(const int* tokens, const void* table, long long ld_table, float* x, long long ldx, int rows,
                            int d, int vocab, int f32, void* stream) {
  using namespace ra;
  if (rows < 1 || d < 1 || vocab < 1 || ldx < d || ld_table < d) {
    set_error("ra_embed_f32: bad shape");
    return kHostBadArg;
  }
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool vec = ldx % 4 == 0 && ld_table % 4 == 0 &&
                   !((reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(x)) & 15);
  if (f32)
    resid::embed_kernel<float><<<rows, 256, 0, s>>>(tokens, static_cast<const float*>(table), ld_table, x, ldx, d, vocab, vec);
  else
    resid::embed_kernel<__nv_bfloat16>
        <<<rows, 256, 0, s>>>(tokens, static_cast<const __nv_bfloat16*>(table), ld_table, x, ldx, d, vocab, vec);
  return check_launch("embed_kernel");
}

// y1 (and y2) = x / rms(x) * (gain_offset + w). Leading dimensions and dp are multiples of 4; pointers 16-byte aligned.
extern "C" int ra_norm_f32(const float* x, const int* rows_idx, const void* w1, const void* w2, void* y1, void* y2, int rows,
                           int d, int dp, long long ldx, long long ldy, float eps, float gain_offset, int f32,
                           void* stream) {
  using namespace ra;
  if (rows < 1 || d < 1 || dp < d || dp % 4 || ldx % 4 || ldy % 4 || ldx < dp || ldy < dp || (y2 && !w2)) {
    set_error("ra_norm_f32: bad shape");
    return kHostBadArg;
  }
  resid::NormParams p{x, rows_idx, w1, w2, y1, y2, ldx, ldy, d, dp, eps, gain_offset};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return f32 ? resid::launch_norm<float>(p, rows, s) : resid::launch_norm<__nv_bfloat16>(p, rows, s);
}

// out (rows, 2 dp) = [x | table[token]]: what enters a pass over looped layers. dp a multiple of 8; `f32`: table and out are
// fp32, else bf16.
extern "C" int ra_stream_pair(const int* tokens, const void* table, long long ld_table, const float* x, long long ldx,
                              void* out, int rows, int d, int dp, int vocab, int f32, void* stream) {
  using namespace ra;
  if (rows < 1 || d < 1 || vocab < 1 || dp < d || dp % 8 || ldx % 4 || ldx < d || ld_table < d) {
    set_error("ra_stream_pair: bad shape");
    return kHostBadArg;
  }
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32)
    resid::pair_kernel<float><<<rows, 256, 0, s>>>(tokens, static_cast<const float*>(table), ld_table, x, ldx,
                                                   static_cast<float*>(out), d, dp, vocab);
  else
    resid::pair_kernel<__nv_bfloat16><<<rows, 256, 0, s>>>(tokens, static_cast<const __nv_bfloat16*>(table), ld_table, x, ldx,
                                                           static_cast<__nv_bfloat16*>(out), d, dp, vocab);
  return check_launch("pair_kernel");
}

// y (rows, ldy >= F) = silu(gu[:, :F]) * gu[:, F:2F], fp32; gu dense.
extern "C" int ra_gated_act_f32(const float* gu, float* y, long long ldy, int rows, int F, void* stream) {
  using namespace ra;
  if (rows < 1 || F < 1 || ldy < F) {
    set_error("ra_gated_act_f32: bad shape");
    return kHostBadArg;
  }
  resid::gated_act_kernel<<<rows, 256, 0, static_cast<cudaStream_t>(stream)>>>(gu, y, ldy, F);
  return check_launch("gated_act_kernel");
}
