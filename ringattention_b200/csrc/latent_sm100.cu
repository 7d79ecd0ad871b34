// Latent attention: per token one latent vector c (rank r) and one rotated key part shared by all heads are cached;
// keys and values of the heads are linear images of c. Kernels that work on the cached rows directly, with the key
// projection moved to the query and the value projection to the output ("absorbed" form), at any sizes:
//   latent_prep_kernel   : RMS norm of c, rotary positions (interleaved pairs) on the shared key part and on the rotated part
//                          of every query head, append of [c | rotated key] to the cache
//   latent_absorb_kernel : q_lat[h] = [W_uk[h]^T q_unrotated | q_rotated], fp32
//   latent_attend_kernel : split-KV attention of the q_lat rows over the cached rows, fp32 online softmax
//   latent_merge_kernel  : merge of the splits, attention sink, value projection, per-head output gate
// A cached row is [c, padded to a multiple of 8 | rotated key, padded to a multiple of 8] in the engine's storage type.
// Everything between the stored operands and the stored output is fp32.
#include "latent_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace latent {

// a pair of neighbouring elements (aligned to both), loaded and stored together
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void store2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float2 v) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
}

// grid (rows): the row's latent and keys go to the cache, its queries are rotated in place. The sines and cosines of the
// row's position are made once for all heads; a warp walks heads, its lanes the pairs. PAIRED: every pair starts at an
// even element.
constexpr int PREP_THREADS = 128;
template <typename T, bool PAIRED>
__global__ void __launch_bounds__(PREP_THREADS, 12) latent_prep_kernel(const Params p) {
  extern __shared__ float2 turn[];  // (rot_dims / 2) cosine, sine
  __shared__ float red[32];
  const long long row = blockIdx.x;
  const int b = blockIdx.x / p.T, t = blockIdx.x - b * p.T;
  const long long pos = *p.pos + t;
  const int pairs = p.rot_dims / 2, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, hd = p.dn + p.dr;
  for (int j = threadIdx.x; j < pairs; j += PREP_THREADS) {
    float sn, cs;
    sincosf(static_cast<float>(pos) * p.inv_freq[j], &sn, &cs);
    turn[j] = make_float2(cs, sn);
  }
  append_row<T>(p, row, b, pos, red);  // its sums synchronise the CTA
  T* q0 = static_cast<T*>(p.proj) + row * p.ldp + p.off_q + p.dn;
  for (int j = lane; j < pairs; j += 32) {
    const float2 f = turn[j];
    T* q = q0 + warp * hd + 2 * j;
#pragma unroll 4
    for (int h = warp; h < p.H; h += PREP_THREADS / 32, q += (PREP_THREADS / 32) * hd) {
      const float2 x = PAIRED ? load2(q) : make_float2(to_f(q[0]), to_f(q[1]));
      const float2 y = make_float2(x.x * f.x - x.y * f.y, x.y * f.x + x.x * f.y);
      if (PAIRED) {
        store2(q, y);
      } else {
        from_f(q[0], y.x);
        from_f(q[1], y.y);
      }
    }
  }
}

template <typename T>
int launch_prep(const Params& p, cudaStream_t s) {
  const int smem = (p.rot_dims / 2) * static_cast<int>(sizeof(float2));
  const bool paired = !((p.dn | p.dr | p.off_q | p.ldp) & 1) && !(reinterpret_cast<uintptr_t>(p.proj) & 7);
  if (paired) latent_prep_kernel<T, true><<<p.B * p.T, PREP_THREADS, smem, s>>>(p);
  else latent_prep_kernel<T, false><<<p.B * p.T, PREP_THREADS, smem, s>>>(p);
  return check_launch("latent_prep_kernel");
}

// grid (rows, H, ceil(row_w / 128)): one thread per latent column
template <typename T>
__global__ void __launch_bounds__(128) latent_absorb_kernel(const Params p) {
  extern __shared__ float sq[];  // (dn)
  const long long row = blockIdx.x;
  const int h = blockIdx.y;
  const T* q = static_cast<const T*>(p.proj) + row * p.ldp + p.off_q + h * (p.dn + p.dr);
  for (int i = threadIdx.x; i < p.dn; i += 128) sq[i] = to_f(q[i]);
  __syncthreads();
  const int c = blockIdx.z * 128 + threadIdx.x;
  if (c >= p.row_w) return;
  float a = 0.f;
  if (c < p.r) {
    const T* w = static_cast<const T*>(p.w_uk) + static_cast<long long>(h) * p.dn * p.ldw + c;
    for (int i = 0; i < p.dn; ++i) a = fmaf(sq[i], to_f(w[i * p.ldw]), a);
  } else if (c >= p.r_pad && c < p.r_pad + p.dr) {
    a = to_f(q[p.dn + c - p.r_pad]);
  }
  static_cast<float*>(p.q_lat)[(row * p.H + h) * p.row_w + c] = a;
}

constexpr int ATT_WARPS = 8;

// grid (splits, H, rows): a warp per cached row at a time, lanes over its columns. NV: columns per lane (row_w <= 32 NV).
template <typename T, int NV>
__global__ void __launch_bounds__(ATT_WARPS * 32) latent_attend_kernel(const Params p) {
  __shared__ float sm_m[ATT_WARPS], sm_l[ATT_WARPS];
  extern __shared__ float sm_o[];  // [ATT_WARPS][r]
  const int split = blockIdx.x, h = blockIdx.y;
  const long long row = blockIdx.z;
  const int b = blockIdx.z / p.T, t = blockIdx.z - b * p.T;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  long long n = *p.pos + t + 1;  // visible rows
  if (n > p.S_max) n = p.S_max;
  const long long per = (n + p.splits - 1) / p.splits;
  const long long r0 = split * per, r1 = min(n, r0 + per);
  const float* ql = static_cast<const float*>(p.q_lat) + (row * p.H + h) * p.row_w;
  float q[NV], acc[NV];
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int c = lane + 32 * j;
    q[j] = c < p.row_w ? ql[c] * p.scale : 0.f;
    acc[j] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const T* base = static_cast<const T*>(p.cache) + b * p.S_max * p.row_w;
  for (long long i = r0 + warp; i < r1; i += ATT_WARPS) {  // uniform over the warp
    const T* kr = base + i * p.row_w;
    float x[NV], s = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = lane + 32 * j;
      x[j] = c < p.row_w ? to_f(kr[c]) : 0.f;
      s = fmaf(q[j], x[j], s);
    }
    s = sum_warp(s);
    const float mn = fmaxf(m, s), alpha = expf(m - mn), w = expf(s - mn);
    l = l * alpha + w;
    m = mn;
#pragma unroll
    for (int j = 0; j < NV; ++j) acc[j] = fmaf(w, x[j], acc[j] * alpha);
  }
  if (lane == 0) {
    sm_m[warp] = m;
    sm_l[warp] = l;
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int c = lane + 32 * j;
    if (c < p.r) sm_o[warp * p.r + c] = acc[j];
  }
  __syncthreads();
  float mx = -INFINITY, lt = 0.f, f[ATT_WARPS];
#pragma unroll
  for (int w = 0; w < ATT_WARPS; ++w) mx = fmaxf(mx, sm_m[w]);
#pragma unroll
  for (int w = 0; w < ATT_WARPS; ++w) {
    f[w] = sm_m[w] == -INFINITY ? 0.f : expf(sm_m[w] - mx);
    lt += sm_l[w] * f[w];
  }
  const long long pi = (row * p.H + h) * p.splits + split;
  for (int c = threadIdx.x; c < p.r; c += ATT_WARPS * 32) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < ATT_WARPS; ++w) o += sm_o[w * p.r + c] * f[w];
    if (RA_IN_BOUNDS(pi * p.r + c, 1, static_cast<long long>(p.B) * p.T * p.H * p.splits * p.r, kTagLatentWork))
      p.o_part[pi * p.r + c] = lt > 0.f ? o / lt : 0.f;
  }
  if (threadIdx.x == 0) p.lse_part[pi] = lt > 0.f ? mx + logf(lt) : -INFINITY;
}

// grid (H, rows): latent output of the head from its splits, then the head's value projection
template <typename T>
__global__ void __launch_bounds__(256) latent_merge_kernel(const Params p) {
  extern __shared__ float so[];  // (r)
  const int h = blockIdx.x;
  const long long row = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float* lp = p.lse_part + (row * p.H + h) * p.splits;
  const float* op = p.o_part + (row * p.H + h) * p.splits * p.r;
  float mx = p.sink ? p.sink[h] : -INFINITY;
  for (int s = 0; s < p.splits; ++s) mx = fmaxf(mx, lp[s]);
  float den = p.sink ? expf(p.sink[h] - mx) : 0.f;
  for (int s = 0; s < p.splits; ++s) den += expf(lp[s] - mx);
  const T* proj = static_cast<const T*>(p.proj) + row * p.ldp;
  const float mul = sigmoid_f(to_f(proj[p.off_g + h])) / den;
  for (int c = threadIdx.x; c < p.r; c += 256) {
    float o = 0.f;
    for (int s = 0; s < p.splits; ++s) o = fmaf(expf(lp[s] - mx), op[s * p.r + c], o);
    so[c] = o * mul;
  }
  __syncthreads();
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * p.dv;
  for (int v = warp; v < p.dv; v += 8) {
    const T* w = static_cast<const T*>(p.w_uv) + (static_cast<long long>(h) * p.dv + v) * p.ldw;
    float a = 0.f;
    for (int c = lane; c < p.r; c += 32) a = fmaf(so[c], to_f(w[c]), a);
    a = sum_warp(a);
    if (lane == 0 && RA_IN_BOUNDS(h * p.dv + v, 1, p.H * p.dv, kTagLatent)) from_f(out[v], a);
  }
}

template <typename T, int NV>
int launch_attend(const Params& p, cudaStream_t s) {
  const int smem = ATT_WARPS * p.r * static_cast<int>(sizeof(float));
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(latent_attend_kernel<T, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) {
    set_error("ra_latent_attend: shared memory");
    return kHostLaunchFail;
  }
  latent_attend_kernel<T, NV><<<dim3(p.splits, p.H, p.B * p.T), ATT_WARPS * 32, smem, s>>>(p);
  return check_launch("latent_attend_kernel");
}

template <typename T>
int run_absorbed(const Params& p, cudaStream_t s) {
  const int rows = p.B * p.T;
  latent_absorb_kernel<T><<<dim3(rows, p.H, (p.row_w + 127) / 128), 128, p.dn * sizeof(float), s>>>(p);
  int rc = check_launch("latent_absorb_kernel");
  if (rc) return rc;
  if (p.row_w <= 128) rc = launch_attend<T, 4>(p, s);
  else if (p.row_w <= 256) rc = launch_attend<T, 8>(p, s);
  else if (p.row_w <= 640) rc = launch_attend<T, 20>(p, s);
  else rc = launch_attend<T, 40>(p, s);
  if (rc) return rc;
  latent_merge_kernel<T><<<dim3(p.H, rows), 256, p.r * sizeof(float), s>>>(p);
  return check_launch("latent_merge_kernel");
}

int check(const Params* p) {
  if (p->B < 1 || p->T < 1 || p->H < 1 || p->H > 65535 || p->dn < 0 || p->dr < 0 || p->dv < 1 || p->r < 1 || p->row_w > 1280 ||
      p->r_pad < p->r || p->row_w < p->r_pad + p->dr || p->rot_dims > p->dr || p->rot_dims > 4096 || p->rot_dims % 2 || p->splits < 1 ||
      static_cast<long long>(p->B) * p->T > 65535) {
    set_error("ra_latent: bad shape (a cached row has at most 1280 columns, a call at most 65535 rows)");
    return kHostBadArg;
  }
  return kHostOk;
}

}  // namespace latent
}  // namespace ra

extern "C" int ra_latent_prep(const ra::latent::Params* p, int f32, void* stream) {
  using namespace ra;
  int rc = latent::check(p);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return f32 ? latent::launch_prep<float>(*p, s) : latent::launch_prep<__nv_bfloat16>(*p, s);
}

// after ra_latent_prep: attention of the step's rows over the cache in the absorbed form
extern "C" int ra_latent_absorbed(const ra::latent::Params* p, int f32, void* stream) {
  using namespace ra;
  int rc = latent::check(p);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return f32 ? latent::run_absorbed<float>(*p, s) : latent::run_absorbed<__nv_bfloat16>(*p, s);
}
