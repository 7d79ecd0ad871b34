// Routed experts: sigmoid scores, the largest `top` of them, gated feed-forwards whose input is multiplied by the score
// (the gate and up products are linear, so the score multiplies their 32-bit results), and a shared expert.
//   moe_route_kernel   : many rows. One warp per token chooses; entries are appended to their expert's list (ranks inside a
//                        CTA through shared memory, one atomic per CTA and expert). The products are in moe_gemm_sm100.cu.
//   moe_combine_kernel : many rows. Adds a token's expert outputs to the 32-bit residual stream, in a fixed order.
//   moe_gateup_kernel, moe_down_kernel : few rows (and fp32, any number). One warp per output streams the weight rows of the
//                        experts that the token uses; every CTA of the first chooses for itself, so that routing is no launch.
#include "moe_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace moe {

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = load4(p), b = load4(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 v = __bfloat1622float2(h[i]);
    f[2 * i] = v.x;
    f[2 * i + 1] = v.y;
  }
}
// eight elements as they lie in memory: weights are loaded a batch ahead of the arithmetic
template <typename T> struct Raw8;
template <> struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = load4(p); b = load4(p + 4); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
};
template <> struct Raw8<__nv_bfloat16> {
  uint4 u;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { u = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 v = __bfloat1622float2(h[i]);
      f[2 * i] = v.x;
      f[2 * i + 1] = v.y;
    }
  }
};
template <typename T>
__device__ __forceinline__ void dot2(const Raw8<T>& w0, const Raw8<T>& w1, const float* x, float& a0, float& a1) {
  float f0[8], f1[8], v[8];
  w0.get(f0);
  w1.get(f1);
  load8(x, v);
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    a0 = fmaf(f0[e], v[e], a0);
    a1 = fmaf(f1[e], v[e], a1);
  }
}

constexpr int FEW_THREADS = 256, FEW_WARPS = 8, BATCH = 4;

// grid (chunks of the outputs, rows)
template <typename T>
__global__ void __launch_bounds__(FEW_THREADS) moe_gateup_kernel(const Params p) {
  extern __shared__ __align__(16) float sm_few[];  // [dp] the row, then E words for the choice
  __shared__ int s_id[MAX_TOP];
  __shared__ float s_w[MAX_TOP];
  const int row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* h = static_cast<const T*>(p.h) + static_cast<long long>(row) * p.dp;
  float* sx = sm_few;
  if (warp == 0) {
    int id;
    float w;
    choose(p.logits + row * p.ld_logits, p.E, p.top, reinterpret_cast<uint32_t*>(sx + p.dp), id, w);
    if (lane < p.top) {
      s_id[lane] = id;
      s_w[lane] = w;
      if (blockIdx.x == 0) {
        p.ids[row * p.top + lane] = id;
        p.weight[row * p.top + lane] = w;
      }
    }
  } else {
    for (int i = (tid - 32) * 8; i < p.dp; i += (FEW_THREADS - 32) * 8) {
      float f[8];
      load8(h + i, f);
      store4(sx + i, make_float4(f[0], f[1], f[2], f[3]));
      store4(sx + i + 4, make_float4(f[4], f[5], f[6], f[7]));
    }
  }
  __syncthreads();
  const int n_out = p.top * p.F + p.Fs;
  T* act = static_cast<T*>(p.act) + static_cast<long long>(row) * n_out;
  for (int o = blockIdx.x * FEW_WARPS + warp; o < n_out; o += gridDim.x * FEW_WARPS) {
    const int s = o / p.F;
    const bool routed = s < p.top;
    const int f = routed ? o - s * p.F : o - p.top * p.F, F = routed ? p.F : p.Fs;
    const T* g = routed ? static_cast<const T*>(p.gu) + (static_cast<long long>(s_id[s]) * 2 * F + f) * p.dp
                        : static_cast<const T*>(p.sh_gu) + static_cast<long long>(f) * p.dp;
    const T* u = g + static_cast<long long>(F) * p.dp;
    float a = 0.f, c = 0.f;
    for (int i0 = lane * 8; i0 < p.dp; i0 += 256 * BATCH) {
      Raw8<T> wg[BATCH], wu[BATCH];
#pragma unroll
      for (int j = 0; j < BATCH; ++j)
        if (i0 + 256 * j < p.dp) {
          wg[j].load(g + i0 + 256 * j);
          wu[j].load(u + i0 + 256 * j);
        }
#pragma unroll
      for (int j = 0; j < BATCH; ++j)
        if (i0 + 256 * j < p.dp) dot2(wg[j], wu[j], sx + i0 + 256 * j, a, c);
    }
    const float w = routed ? s_w[s] : 1.f;
    a = sum_warp(a) * w;
    c = sum_warp(c) * w;
    if (lane == 0 && RA_IN_BOUNDS(o, 1, n_out, kTagMoe)) from_f(act[o], silu_f(a) * c);
  }
}

constexpr int DOWN_COLS = 2;  // columns per warp, side by side

// grid (chunks of the columns, rows): x[row] += sum over the experts of W_down act. A lane's pieces run through the experts'
// rows one after the other, so that several experts' weights are on their way at once.
template <typename T>
__global__ void __launch_bounds__(FEW_THREADS) moe_down_kernel(const Params p) {
  extern __shared__ __align__(16) float sm_few[];  // [top * F + Fs]
  __shared__ const T* s_base[MAX_TOP];
  const int row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n_in = p.top * p.F + p.Fs;
  const T* act = static_cast<const T*>(p.act) + static_cast<long long>(row) * n_in;
  if (tid < p.top) s_base[tid] = static_cast<const T*>(p.down) + static_cast<long long>(p.ids[row * p.top + tid]) * p.dp * p.F;
  for (int i = tid * 8; i < n_in; i += FEW_THREADS * 8) {
    float f[8];
    load8(act + i, f);
    store4(sm_few + i, make_float4(f[0], f[1], f[2], f[3]));
    store4(sm_few + i + 4, make_float4(f[4], f[5], f[6], f[7]));
  }
  __syncthreads();
  const int c0 = (blockIdx.x * FEW_WARPS + warp) * DOWN_COLS;
  if (c0 >= p.d) return;
  const int c1 = min(c0 + 1, p.d - 1), F8 = p.F >> 3, routed = p.top * F8, pieces = n_in >> 3;
  float a0 = 0.f, a1 = 0.f;
  for (int q0 = lane; q0 < pieces; q0 += 32 * BATCH) {
    Raw8<T> w0[BATCH], w1[BATCH];
#pragma unroll
    for (int j = 0; j < BATCH; ++j) {
      const int q = q0 + 32 * j;
      if (q >= pieces) continue;
      const int s = q / F8;
      const bool in = q < routed;
      const T* base = in ? s_base[s] : static_cast<const T*>(p.sh_down);
      const long long ld = in ? p.F : p.Fs;
      const int i = (in ? q - s * F8 : q - routed) * 8;
      w0[j].load(base + c0 * ld + i);
      w1[j].load(base + c1 * ld + i);
    }
#pragma unroll
    for (int j = 0; j < BATCH; ++j)
      if (q0 + 32 * j < pieces) dot2(w0[j], w1[j], sm_few + (q0 + 32 * j) * 8, a0, a1);
  }
  a0 = sum_warp(a0);
  a1 = sum_warp(a1);
  if (lane < DOWN_COLS && c0 + lane < p.d && RA_IN_BOUNDS(c0 + lane, 1, p.ldx, kTagMoe))
    p.x[row * p.ldx + c0 + lane] += lane ? a1 : a0;
}

constexpr int ROUTE_TOKENS = 32, ROUTE_WARPS = 8;  // tokens per CTA

__global__ void __launch_bounds__(32 * ROUTE_WARPS) moe_route_kernel(const Params p) {
  extern __shared__ uint32_t sm_route[];  // [ROUTE_WARPS][E] keys, [E] counts, [E] bases
  __shared__ int s_id[ROUTE_TOKENS * MAX_TOP], s_rank[ROUTE_TOKENS * MAX_TOP];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int* hist = reinterpret_cast<int*>(sm_route + ROUTE_WARPS * p.E);
  int* base = hist + p.E;
  for (int e = tid; e < p.E; e += blockDim.x) hist[e] = 0;
  __syncthreads();
  const int t0 = blockIdx.x * ROUTE_TOKENS;
  for (int i = warp; i < ROUTE_TOKENS && t0 + i < p.rows; i += ROUTE_WARPS) {
    int id;
    float w;
    choose(p.logits + static_cast<long long>(t0 + i) * p.ld_logits, p.E, p.top, sm_route + warp * p.E, id, w);
    if (lane < p.top) {
      p.weight[static_cast<long long>(t0 + i) * p.top + lane] = w;
      s_id[i * p.top + lane] = id;
      s_rank[i * p.top + lane] = atomicAdd(&hist[id], 1);
    }
    __syncwarp();
  }
  __syncthreads();
  for (int e = tid; e < p.E; e += blockDim.x) base[e] = hist[e] ? atomicAdd(&p.count[e], hist[e]) : 0;
  __syncthreads();
  const int n = min(ROUTE_TOKENS, p.rows - t0) * p.top;
  for (int i = tid; i < n; i += blockDim.x) {
    const int e = s_id[i], at = base[e] + s_rank[i];
    if (RA_IN_BOUNDS(at, 1, p.rows, kTagMoe)) p.list[static_cast<long long>(e) * p.rows + at] = t0 * p.top + i;
  }
}

__global__ void __launch_bounds__(256) moe_combine_kernel(const Params p) {
  const long long row = blockIdx.x;
  const __nv_bfloat16* y = static_cast<const __nv_bfloat16*>(p.y) + row * p.top * p.dp;
  float* x = p.x + row * p.ldx;
  for (int i = threadIdx.x * 8; i < p.dp; i += 256 * 8) {
    float a[8], v[8];
    load8(x + i, a);
#pragma unroll 4
    for (int k = 0; k < p.top; ++k) {
      load8(y + static_cast<long long>(k) * p.dp + i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) a[e] += v[e];
    }
    if (!RA_IN_BOUNDS(i, 8, p.ldx, kTagMoe)) continue;
    store4(x + i, make_float4(a[0], a[1], a[2], a[3]));
    store4(x + i + 4, make_float4(a[4], a[5], a[6], a[7]));
  }
}

int check(const Params* p) {
  const char* why = nullptr;
  if (p->rows < 1 || p->d < 1 || p->dp < p->d || p->dp % 8 || p->F < 8 || p->F % 8 || p->Fs < 0 || p->Fs % 8 || p->ldx % 8 ||
      p->ldx < p->dp)
    why = "moe: bad shape";
  else if (p->E < 1 || p->E > MAX_EXPERTS || p->top < 1 || p->top > p->E || p->top > MAX_TOP || p->ld_logits < p->E)
    why = "moe: bad number of experts";
  if (!why) return kHostOk;
  set_error(why);
  return kHostBadArg;
}

template <typename K>
int shared_memory(K kern, size_t bytes) {
  if (bytes <= 48 * 1024) return kHostOk;
  if (bytes <= 200 * 1024 &&
      cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)) == cudaSuccess)
    return kHostOk;
  cudaGetLastError();
  set_error("moe: a row does not fit in shared memory");
  return kHostTooLarge;
}

template <typename T>
int launch_few(const Params& p, cudaStream_t s) {
  const int n = p.top * p.F + p.Fs;
  if (p.rows > 65535) {
    set_error("moe: too many rows for the kernels of few rows");
    return kHostTooLarge;
  }
  const size_t smem1 = 4 * (static_cast<size_t>(p.dp) + p.E), smem2 = 4 * static_cast<size_t>(n);
  if (int rc = shared_memory(moe_gateup_kernel<T>, smem1)) return rc;
  if (int rc = shared_memory(moe_down_kernel<T>, smem2)) return rc;
  // a CTA loads the row and chooses before it streams weights: not more CTAs than fit at once, equally many outputs each
  const int want = (n + FEW_WARPS - 1) / FEW_WARPS, fit = (5 * sm_count() + p.rows - 1) / p.rows;
  const int rounds = (want + fit - 1) / fit;
  moe_gateup_kernel<T><<<dim3((want + rounds - 1) / rounds, p.rows), FEW_THREADS, smem1, s>>>(p);
  if (int rc = check_launch("moe_gateup_kernel")) return rc;
  const int per = DOWN_COLS * FEW_WARPS;
  moe_down_kernel<T><<<dim3((p.d + per - 1) / per, p.rows), FEW_THREADS, smem2, s>>>(p);
  return check_launch("moe_down_kernel");
}

}  // namespace moe
}  // namespace ra

// x += routed experts and shared expert of h, one weight pass per row: decode steps (bf16) and fp32 engines. Two launches.
extern "C" int ra_moe_few(const ra::moe::Params* p, int f32, void* stream) {
  using namespace ra;
  if (const int rc = moe::check(p)) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return f32 ? moe::launch_few<float>(*p, s) : moe::launch_few<__nv_bfloat16>(*p, s);
}

// Chooses for every row: weight, count (zeroed by the caller) and list.
extern "C" int ra_moe_route(const ra::moe::Params* p, void* stream) {
  using namespace ra;
  if (const int rc = moe::check(p)) return rc;
  const size_t smem = 4 * static_cast<size_t>(moe::ROUTE_WARPS + 2) * p->E;
  moe::moe_route_kernel<<<(p->rows + moe::ROUTE_TOKENS - 1) / moe::ROUTE_TOKENS, 32 * moe::ROUTE_WARPS, smem,
                          static_cast<cudaStream_t>(stream)>>>(*p);
  return check_launch("moe_route_kernel");
}

// x += the rows of y that belong to a token.
extern "C" int ra_moe_combine(const ra::moe::Params* p, void* stream) {
  using namespace ra;
  if (const int rc = moe::check(p)) return rc;
  moe::moe_combine_kernel<<<p->rows, 256, 0, static_cast<cudaStream_t>(stream)>>>(*p);
  return check_launch("moe_combine_kernel");
}
