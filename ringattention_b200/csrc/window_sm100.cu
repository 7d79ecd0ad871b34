// Attention over a sliding window with grouped key/value heads, a sink per head, RMS norms over the whole query and key
// projections and rotary positions on the first dimensions of a head:
//   window_prep_kernel, window_prep_pieces_kernel : norms, rotation (queries in place) and the new rows of the key/value
//                          ring. One CTA per token; bf16 in 16-byte pieces where the sizes allow it, a row read once.
//   window_attend_kernel : one warp per (token, head) on the CUDA cores; any sizes, bf16 or fp32 throughout. bf16 prompts of
//                          the common sizes run on the tensor cores (attn_fwd_sm100.cu), single tokens in
//                          window_decode_sm100.cu.
#include "window_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace window {

constexpr int PREP_THREADS = 256;
constexpr int MAX_HALF = 256;  // (dk <= 512)

// bf16, head sizes and rot_half multiples of eight. A CTA takes NROW consecutive tokens of a sequence, a thread the same NI
// units of query and key heads of each: the kernel is bound by its instructions, and index arithmetic and gains serve all
// rows. grid (tokens / NROW, sequences).
template <int NI, int NROW>
__global__ void __launch_bounds__(PREP_THREADS, NI <= 2 ? 4 : 1) window_prep_pieces_kernel(const Params p) {
  __shared__ __align__(16) float red[2 * NROW][8], sn[NROW][MAX_HALF], cs[NROW][MAX_HALF];
  const int b = blockIdx.y, t0 = blockIdx.x * NROW, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rows = min(NROW, p.T - t0);
  __nv_bfloat16* x = static_cast<__nv_bfloat16*>(p.proj) + (static_cast<long long>(b) * p.T + t0) * p.ldp;
  const int h8 = p.rot_half >> 3, units = (p.dk >> 3) - h8, n = (p.H + p.G) * units, v8 = p.dv >> 3;
  Piece lo[NI][NROW], hi[NI][NROW];
  int heads[NI], unit[NI];  // the thread's heads, query heads first, and units (-1: none)
  float s[2 * NROW];
#pragma unroll
  for (int e = 0; e < 2 * NROW; ++e) s[e] = 0.f;
#pragma unroll
  for (int j = 0; j < NI; ++j) {
    const int i = tid + j * PREP_THREADS, head = i / units;
    unit[j] = i < n ? i - head * units : -1;
    heads[j] = head;
    const __nv_bfloat16* src = x + (head < p.H ? p.off_q : p.off_k - p.H * p.dk) + head * p.dk;
#pragma unroll
    for (int r = 0; r < NROW; ++r)
      if (unit[j] >= 0 && r < rows) {
        hi[j][r] = load_piece(src + r * p.ldp + (unit[j] + h8) * 8);
        if (unit[j] < h8) lo[j][r] = load_piece(src + r * p.ldp + unit[j] * 8);
      }
  }
  const long long pos = *p.pos + t0;
  for (int i = tid; i < rows * p.rot_half; i += PREP_THREADS) {
    const int r = i / p.rot_half, e = i - r * p.rot_half;
    sincosf(static_cast<float>(pos + r) * p.inv_freq[e], &sn[r][e], &cs[r][e]);
  }
#pragma unroll
  for (int j = 0; j < NI; ++j)
#pragma unroll
    for (int r = 0; r < NROW; ++r)
      if (unit[j] >= 0 && r < rows) {
        const float v = square_sum(hi[j][r]) + (unit[j] < h8 ? square_sum(lo[j][r]) : 0.f);
        s[2 * r] += heads[j] < p.H ? v : 0.f;
        s[2 * r + 1] += heads[j] < p.H ? 0.f : v;
      }
#pragma unroll
  for (int e = 0; e < 2 * NROW; ++e) {
    s[e] = sum_warp(s[e]);
    if (lane == 0) red[e][warp] = s[e];
  }
  __syncthreads();
  {  // lane e of every warp makes the e-th factor
    const int e = lane < 2 * NROW ? lane : 0;
    const float4 u = load4(red[e]), w = load4(red[e] + 4);
    const float sum = ((u.x + u.y) + (u.z + u.w)) + ((w.x + w.y) + (w.z + w.w));
    const float rs = 1.f / sqrtf(sum / (e & 1 ? p.G * p.dk : p.H * p.dk) + p.eps);
#pragma unroll
    for (int i = 0; i < 2 * NROW; ++i) s[i] = __shfl_sync(0xffffffffu, rs, i);
  }
  if (!RA_IN_BOUNDS(t0, rows, p.T, kTagWindow)) return;
  const int ring0 = static_cast<int>(static_cast<unsigned>(pos) % static_cast<unsigned>(p.R));
  auto ring_row = [&](int r) { return ring0 + r >= p.R ? ring0 + r - p.R : ring0 + r; };
  __nv_bfloat16* kc = static_cast<__nv_bfloat16*>(p.k_cache) + static_cast<long long>(b) * p.G * p.R * p.kw;
  __nv_bfloat16* vc = static_cast<__nv_bfloat16*>(p.v_cache) + static_cast<long long>(b) * p.G * p.R * p.vw;
#pragma unroll
  for (int j = 0; j < NI; ++j) {
    if (unit[j] < 0) continue;
    const int u = unit[j], head = heads[j], at = head * p.dk;
    const bool is_q = head < p.H;
    const __nv_bfloat16* gain = is_q ? static_cast<const __nv_bfloat16*>(p.q_norm) + at
                                     : static_cast<const __nv_bfloat16*>(p.k_norm) + at - p.H * p.dk;
    float gh[8], gl[8];
    unpack(load_piece(gain + (u + h8) * 8), gh);
    if (u < h8) unpack(load_piece(gain + u * 8), gl);
#pragma unroll
    for (int r = 0; r < NROW; ++r) {
      if (r >= rows) break;
      norm_turn(lo[j][r], hi[j][r], gl, gh, is_q ? s[2 * r] : s[2 * r + 1], u, h8, sn[r], cs[r]);
      __nv_bfloat16* dst = is_q ? x + r * p.ldp + p.off_q + at
                                : kc + (static_cast<long long>(head - p.H) * p.R + ring_row(r)) * p.kw;
      *reinterpret_cast<uint4*>(dst + (u + h8) * 8) = hi[j][r].u;
      if (u < h8) *reinterpret_cast<uint4*>(dst + u * 8) = lo[j][r].u;
    }
  }
  for (int i = tid; i < p.G * v8; i += PREP_THREADS) {
    const int g = i / v8, u = i - g * v8;
#pragma unroll
    for (int r = 0; r < NROW; ++r)
      if (r < rows)
        *reinterpret_cast<uint4*>(vc + (static_cast<long long>(g) * p.R + ring_row(r)) * p.vw + u * 8) =
            load_piece(x + r * p.ldp + p.off_v + i * 8).u;
  }
}

template <int NI>
void launch_pieces(const Params& p, cudaStream_t s) {
  constexpr int NROW = 2;
  if (p.T >= 64)
    window_prep_pieces_kernel<NI, NROW><<<dim3((p.T + NROW - 1) / NROW, p.B), PREP_THREADS, 0, s>>>(p);
  else window_prep_pieces_kernel<NI, 1><<<dim3(p.T, p.B), PREP_THREADS, 0, s>>>(p);
}

template <typename T>
__global__ void __launch_bounds__(PREP_THREADS) window_prep_kernel(const Params p) {
  __shared__ float red[64], sn[MAX_HALF], cs[MAX_HALF];
  const long long row = blockIdx.x;
  const int b = static_cast<int>(row / p.T), t = static_cast<int>(row - static_cast<long long>(b) * p.T);
  const long long pos = *p.pos + t;
  const int r = static_cast<int>(pos % p.R), tid = threadIdx.x;
  T* q = static_cast<T*>(p.proj) + row * p.ldp + p.off_q;
  const T* k = static_cast<const T*>(p.proj) + row * p.ldp + p.off_k;
  const T* v = static_cast<const T*>(p.proj) + row * p.ldp + p.off_v;
  T* kc = static_cast<T*>(p.k_cache) + (static_cast<long long>(b) * p.G * p.R + r) * p.kw;  // head g: + g * R * kw
  T* vc = static_cast<T*>(p.v_cache) + (static_cast<long long>(b) * p.G * p.R + r) * p.vw;
  const T *qw = static_cast<const T*>(p.q_norm), *kw = static_cast<const T*>(p.k_norm);
  const int nq = p.H * p.dk, nk = p.G * p.dk, half = p.rot_half;
  for (int i = tid; i < half; i += PREP_THREADS) sincosf(static_cast<float>(pos) * p.inv_freq[i], &sn[i], &cs[i]);
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < nq; i += PREP_THREADS) sq += to_f(q[i]) * to_f(q[i]);
  for (int i = tid; i < nk; i += PREP_THREADS) sk += to_f(k[i]) * to_f(k[i]);
  const float2 ss = sum_block2(sq, sk, red);  // its barriers also cover the sines
  const float rq = 1.f / sqrtf(ss.x / nq + p.eps), rk = 1.f / sqrtf(ss.y / nk + p.eps);
  if (!RA_IN_BOUNDS(row, 1, static_cast<long long>(p.B) * p.T, kTagWindow)) return;
  const int rest = p.dk - 2 * half, per = half + rest;  // pairs, then dimensions that pass
  for (int i = tid; i < (p.H + p.G) * per; i += PREP_THREADS) {
    const int head = i / per, u = i - head * per;
    const bool is_q = head < p.H;
    const int hh = is_q ? head : head - p.H;
    const T* src = is_q ? q + hh * p.dk : k + hh * p.dk;
    const T* gain = is_q ? qw + hh * p.dk : kw + hh * p.dk;
    T* dst = is_q ? q + hh * p.dk : kc + static_cast<long long>(hh) * p.R * p.kw;
    const float rs = is_q ? rq : rk;
    if (u < half) {
      const float a = to_f(src[u]) * rs * to_f(gain[u]), c = to_f(src[u + half]) * rs * to_f(gain[u + half]);
      from_f(dst[u], a * cs[u] - c * sn[u]);
      from_f(dst[u + half], c * cs[u] + a * sn[u]);
    } else {
      from_f(dst[u + half], to_f(src[u + half]) * rs * to_f(gain[u + half]));
    }
  }
  for (int i = tid; i < p.G * p.dv; i += PREP_THREADS) {
    const int g = i / p.dv, u = i - g * p.dv;
    vc[static_cast<long long>(g) * p.R * p.vw + u] = v[i];
  }
}

constexpr int ATT_WARPS = 4;

// NR: dimensions per lane (dk and dv at most 32 NR).
template <typename T, int NR>
__global__ void __launch_bounds__(32 * ATT_WARPS) window_attend_kernel(const Params p) {
  const long long row = blockIdx.x;
  const int h = blockIdx.y * ATT_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int b = static_cast<int>(row / p.T), t = static_cast<int>(row - static_cast<long long>(b) * p.T);
  const long long pos = *p.pos + t;
  const int g = h / (p.H / p.G);
  const T* q = static_cast<const T*>(p.proj) + row * p.ldp + p.off_q + h * p.dk;
  const T* kb = static_cast<const T*>(p.k_cache) + (static_cast<long long>(b) * p.G + g) * p.R * p.kw;
  const T* vb = static_cast<const T*>(p.v_cache) + (static_cast<long long>(b) * p.G + g) * p.R * p.vw;
  float qr[NR], o[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = lane + 32 * i;
    qr[i] = d < p.dk ? to_f(q[d]) * p.scale : 0.f;
    o[i] = 0.f;
  }
  float m = p.sink[h], l = 1.f;  // the sink comes first: weight 1 at the running maximum, no value
  const int n = static_cast<int>(pos + 1 < p.window ? pos + 1 : p.window);
  int r = static_cast<int>((pos - n + 1) % p.R);
  for (int j = 0; j < n; ++j, r = r + 1 == p.R ? 0 : r + 1) {
    const T* kr = kb + static_cast<long long>(r) * p.kw;
    const T* vr = vb + static_cast<long long>(r) * p.vw;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = lane + 32 * i;
      if (d < p.dk) s = fmaf(qr[i], to_f(kr[d]), s);
    }
    s = sum_warp(s);
    if (s > m) {
      const float a = expf(m - s);
      l *= a;
#pragma unroll
      for (int i = 0; i < NR; ++i) o[i] *= a;
      m = s;
    }
    const float w = expf(s - m);
    l += w;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = lane + 32 * i;
      if (d < p.dv) o[i] = fmaf(w, to_f(vr[d]), o[i]);
    }
  }
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * p.dv;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = lane + 32 * i;
    if (d < p.dv && RA_IN_BOUNDS(h * p.dv + d, 1, p.ldo, kTagWindow)) from_f(out[d], o[i] / l);
  }
}

int check(const Params* p) {
  const char* why = nullptr;
  if (p->B < 1 || p->T < 1 || p->H < 1 || p->G < 1 || p->H % p->G || p->dk < 1 || p->dv < 1) why = "window: bad shape";
  else if (p->dk > 512 || p->dv > 512) why = "window: head sizes above 512";
  else if (p->rot_half < 0 || 2 * p->rot_half > p->dk || p->rot_half > MAX_HALF) why = "window: bad rotary size";
  else if (p->kw < p->dk || p->vw < p->dv || p->kw % 8 || p->vw % 8 || p->ldp % 8 || p->off_q % 8 || p->off_k % 8 || p->off_v % 8)
    why = "window: bad row width";
  else if (p->window < 1 || p->R < 1) why = "window: bad window";
  if (!why) return kHostOk;
  set_error(why);
  return kHostBadArg;
}

template <typename T>
int launch_attend(const Params& p, cudaStream_t s) {
  const dim3 grid(p.B * p.T, (p.H + ATT_WARPS - 1) / ATT_WARPS);
  const int d = p.dk > p.dv ? p.dk : p.dv;
  if (d <= 64) window_attend_kernel<T, 2><<<grid, 32 * ATT_WARPS, 0, s>>>(p);
  else if (d <= 128) window_attend_kernel<T, 4><<<grid, 32 * ATT_WARPS, 0, s>>>(p);
  else window_attend_kernel<T, 16><<<grid, 32 * ATT_WARPS, 0, s>>>(p);
  return check_launch("window_attend_kernel");
}

}  // namespace window
}  // namespace ra

extern "C" int ra_window_prep(const ra::window::Params* p, int f32, void* stream) {
  using namespace ra;
  if (const int rc = window::check(p)) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int rows = p->B * p->T;
  const int units = (p->H + p->G) * ((p->dk - p->rot_half) / 8);
  if (f32) window::window_prep_kernel<float><<<rows, window::PREP_THREADS, 0, s>>>(*p);
  else if (p->dk % 8 || p->dv % 8 || p->rot_half % 8 || units > 4 * window::PREP_THREADS || p->B > 65535)
    window::window_prep_kernel<__nv_bfloat16><<<rows, window::PREP_THREADS, 0, s>>>(*p);
  else if (units <= window::PREP_THREADS) window::launch_pieces<1>(*p, s);
  else if (units <= 2 * window::PREP_THREADS) window::launch_pieces<2>(*p, s);
  else window::launch_pieces<4>(*p, s);
  return check_launch("window_prep_kernel");
}

// After ra_window_prep of the same step.
extern "C" int ra_window_attend(const ra::window::Params* p, int f32, void* stream) {
  using namespace ra;
  if (const int rc = window::check(p)) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return f32 ? window::launch_attend<float>(*p, s) : window::launch_attend<__nv_bfloat16>(*p, s);
}
