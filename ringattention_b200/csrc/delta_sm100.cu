// Gated delta rule with short convolutions: the kernels around and of the recurrence
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// with one state S (dk x dv, fp32) per value head and per sequence.
//   delta_prep_kernel : causal convolution over time + silu of the q, k and v channels, unit norms of q and k per head,
//                       decay g and step size beta from their projections. One warp per (token, head).
//   delta_scan_kernel : the recurrence over the tokens of a step. Columns of S (one per value channel) are independent:
//                       eight lanes own one column, dk / 8 state elements each, in registers for the whole step; both
//                       read-outs of a token (with k and with q) are taken from the decayed state before the write,
//                       o = S'^T q + (q.k) u, so a token costs one reduction over eight lanes.
//   delta_out_kernel  : per-head RMS norm of o, gain, silu gate.
//   delta_step_kernel : all of it for one token per sequence (decode), a cluster of four CTAs per value head.
// The convolution's history is a ring of `taps` rows per sequence, the row of position p at p % taps, kept in fp32: a
// step reads the rows of the taps - 1 tokens before it and writes the rows of its own last tokens. The state is stored
// transposed, (dv, dk), so that the eight lanes of a column read 128 contiguous bytes.
// Everything here is fp32 except the projections that come in.
#include <cooperative_groups.h>

#include "delta_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace delta {

// grid (rows, ceil((2 G + H) / 4)), four warps; unit u: q head u, k head u - G, v head u - 2 G
template <typename T>
__global__ void __launch_bounds__(128) delta_prep_kernel(const Params p) {
  const int row = blockIdx.x, u = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (u >= 2 * p.G + p.H) return;
  const int b = row / p.T, t = row - b * p.T;
  const long long pos0 = *p.pos;
  const int C = 2 * p.G * p.dk + p.H * p.dv;
  const T* proj_b = static_cast<const T*>(p.proj) + static_cast<long long>(b) * p.T * p.ldp;
  const float* ring_b = p.ring + static_cast<long long>(b) * p.taps * C;
  if (u < 2 * p.G) {
    const bool is_q = u < p.G;
    const int hd = is_q ? u : u - p.G;
    const T* w = static_cast<const T*>(is_q ? p.conv_q : p.conv_k) + static_cast<long long>(hd) * p.dk * p.taps;
    const int col = (is_q ? p.off_q : p.off_k) + hd * p.dk, c0 = u * p.dk;
    float* dst = (is_q ? p.q : p.k) + (static_cast<long long>(row) * p.G + hd) * p.dk;
    float ss = 0.f;
    for (int i = lane; i < p.dk; i += 32) {
      const float x = conv_silu(p, proj_b, ring_b, w + i * p.taps, t, pos0, C, c0 + i, col + i);
      dst[i] = x;
      ss += x * x;
    }
    const float mul = (is_q ? p.q_scale : 1.f) / sqrtf(sum_warp(ss) + 1e-6f);
    for (int i = lane; i < p.dk; i += 32) dst[i] *= mul;
  } else {
    const int hd = u - 2 * p.G;
    const T* w = static_cast<const T*>(p.conv_v) + static_cast<long long>(hd) * p.dv * p.taps;
    const int c0 = 2 * p.G * p.dk + hd * p.dv;
    float* dst = p.v + (static_cast<long long>(row) * p.H + hd) * p.dv;
    for (int i = lane; i < p.dv; i += 32)
      dst[i] = conv_silu(p, proj_b, ring_b, w + i * p.taps, t, pos0, C, c0 + i, p.off_v + hd * p.dv + i);
    if (lane == 0) {
      const float* ba = p.ba + row * p.ldba;
      float* gb = p.gb + (static_cast<long long>(row) * p.H + hd) * 2;
      gb[0] = expf(log_decay(ba[p.off_a + hd], to_f(static_cast<const T*>(p.a_log)[hd]), to_f(static_cast<const T*>(p.dt_bias)[hd])));
      gb[1] = sigmoid_f(ba[hd]);
    }
  }
}

constexpr int SCAN_TB = 16;      // tokens staged in shared memory at a time
constexpr int SCAN_COLS = 16;    // columns per CTA (four warps, eight lanes per column)

// NJ: groups of four state elements per lane (dk <= 32 NJ). Lane l of a column owns elements 32 j + 4 l .. + 3.
template <typename T, int NJ>
__global__ void __launch_bounds__(128) delta_scan_kernel(const Params p) {
  constexpr int DKP = 32 * NJ;
  __shared__ __align__(16) float sq[SCAN_TB][DKP], sk[SCAN_TB][DKP];
  __shared__ float sv[SCAN_TB][SCAN_COLS], sgb[SCAN_TB][2];
  const int h = blockIdx.y, b = blockIdx.z, kvh = h / (p.H / p.G);
  const int tid = threadIdx.x, l = tid & 7, cl = tid >> 3;
  const int col = blockIdx.x * SCAN_COLS + cl;
  const bool in = col < p.dv;
  const long long pos0 = *p.pos;

  // nobody reads the ring in this launch
  save_ring<T>(p, b, pos0, (blockIdx.y * gridDim.x + blockIdx.x) * 128 + tid, gridDim.x * gridDim.y * 128);

  float S[NJ][4];
  float* st = p.state + ((static_cast<long long>(b) * p.H + h) * p.dv + (in ? col : 0)) * p.dk;
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = 32 * j + 4 * l + e;
      S[j][e] = (in && i < p.dk) ? st[i] : 0.f;
    }
  for (int t0 = 0; t0 < p.T; t0 += SCAN_TB) {
    const int nt = min(SCAN_TB, p.T - t0);
    __syncthreads();
    for (int i = tid; i < SCAN_TB * DKP; i += 128) {
      const int t = i / DKP, e = i % DKP;
      const bool ok = t < nt && e < p.dk;
      const long long src = ((static_cast<long long>(b) * p.T + t0 + t) * p.G + kvh) * p.dk + e;
      sq[t][e] = ok ? p.q[src] : 0.f;
      sk[t][e] = ok ? p.k[src] : 0.f;
    }
    for (int i = tid; i < SCAN_TB * SCAN_COLS; i += 128) {
      const int t = i / SCAN_COLS, c = blockIdx.x * SCAN_COLS + i % SCAN_COLS;
      sv[t][i % SCAN_COLS] =
          (t < nt && c < p.dv) ? p.v[((static_cast<long long>(b) * p.T + t0 + t) * p.H + h) * p.dv + c] : 0.f;
    }
    if (tid < SCAN_TB * 2) {
      const int t = tid >> 1;
      sgb[t][tid & 1] = t < nt ? p.gb[((static_cast<long long>(b) * p.T + t0 + t) * p.H + h) * 2 + (tid & 1)] : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float g = sgb[t][0], beta = sgb[t][1];
      float4 kk[NJ];
      float dk_[4] = {0.f, 0.f, 0.f, 0.f}, dq_[4] = {0.f, 0.f, 0.f, 0.f}, qk = 0.f;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        kk[j] = load4(&sk[t][32 * j + 4 * l]);
        const float4 qq = load4(&sq[t][32 * j + 4 * l]);
        dk_[0] = fmaf(S[j][0], kk[j].x, dk_[0]);
        dk_[1] = fmaf(S[j][1], kk[j].y, dk_[1]);
        dk_[2] = fmaf(S[j][2], kk[j].z, dk_[2]);
        dk_[3] = fmaf(S[j][3], kk[j].w, dk_[3]);
        dq_[0] = fmaf(S[j][0], qq.x, dq_[0]);
        dq_[1] = fmaf(S[j][1], qq.y, dq_[1]);
        dq_[2] = fmaf(S[j][2], qq.z, dq_[2]);
        dq_[3] = fmaf(S[j][3], qq.w, dq_[3]);
        qk = fmaf(kk[j].x, qq.x, fmaf(kk[j].y, qq.y, fmaf(kk[j].z, qq.z, fmaf(kk[j].w, qq.w, qk))));
      }
      float a = (dk_[0] + dk_[1]) + (dk_[2] + dk_[3]), c = (dq_[0] + dq_[1]) + (dq_[2] + dq_[3]);
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) {
        a += __shfl_xor_sync(0xffffffffu, a, o);
        c += __shfl_xor_sync(0xffffffffu, c, o);
        qk += __shfl_xor_sync(0xffffffffu, qk, o);
      }
      const float u = beta * (sv[t][cl] - g * a);
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        S[j][0] = fmaf(kk[j].x, u, g * S[j][0]);
        S[j][1] = fmaf(kk[j].y, u, g * S[j][1]);
        S[j][2] = fmaf(kk[j].z, u, g * S[j][2]);
        S[j][3] = fmaf(kk[j].w, u, g * S[j][3]);
      }
      if (l == 0 && in && RA_IN_BOUNDS(col, 1, p.dv, kTagDelta)) p.o[((static_cast<long long>(b) * p.T + t0 + t) * p.H + h) * p.dv + col] = fmaf(qk, u, g * c);
    }
  }
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = 32 * j + 4 * l + e;
      if (in && i < p.dk) st[i] = S[j][e];
    }
}

// out = o / rms(o) * norm_w * silu(gate) per (row, head)
template <typename T>
__device__ __forceinline__ float gate_f(float g) {
  return sizeof(T) == 2 ? silu_fast(g) : silu_f(g);
}
// one warp per (row, head), any sizes
template <typename T>
__global__ void __launch_bounds__(128) delta_out_kernel(const Params p) {
  const long long unit = static_cast<long long>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<long long>(p.B) * p.T * p.H) return;
  const long long row = unit / p.H;
  const int h = static_cast<int>(unit - row * p.H);
  const float* o = p.o + unit * p.dv;
  float ss = 0.f;
  for (int i = lane; i < p.dv; i += 32) ss += o[i] * o[i];
  const float rs = 1.f / sqrtf(sum_warp(ss) / p.dv + p.eps);
  const T* gate = static_cast<const T*>(p.proj) + row * p.ldp + p.off_g + h * p.dv;
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * p.dv;
  for (int i = lane; i < p.dv; i += 32)
    if (RA_IN_BOUNDS(h * p.dv + i, 1, p.H * p.dv, kTagDelta))
      from_f(out[i], o[i] * rs * to_f(static_cast<const T*>(p.norm_w)[i]) * gate_f<T>(to_f(gate[i])));
}
// dv = 4 * LANES: LANES lanes per (row, head), four values each, and four rows' heads per lane with all loads in flight;
// everything starts at multiples of four elements
template <typename T, int LANES>
__global__ void __launch_bounds__(256) delta_out_vec_kernel(const Params p) {
  constexpr int UPB = 256 / LANES, UNITS = 4;  // units per CTA and round, rounds
  const unsigned n = static_cast<unsigned>(p.B) * p.T * p.H, H = p.H;  // below 2^31 (checked by the launcher)
  const unsigned u0 = blockIdx.x * (UPB * UNITS) + threadIdx.x / LANES;
  const int i = (threadIdx.x % LANES) * 4;
  const float4 w = load4(static_cast<const T*>(p.norm_w) + i);
  float4 x[UNITS], g[UNITS];
#pragma unroll
  for (int k = 0; k < UNITS; ++k) {
    const unsigned u = min(u0 + k * UPB, n - 1), row = u / H, h = u - row * H;
    x[k] = load4(p.o + static_cast<long long>(u) * p.dv + i);
    g[k] = load4(static_cast<const T*>(p.proj) + row * p.ldp + p.off_g + h * p.dv + i);
  }
#pragma unroll
  for (int k = 0; k < UNITS; ++k) {
    float ss = x[k].x * x[k].x + x[k].y * x[k].y + x[k].z * x[k].z + x[k].w * x[k].w;
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rs = 1.f / sqrtf(ss / p.dv + p.eps);
    const unsigned u = u0 + k * UPB, row = u / H, h = u - row * H;
    if (u < n && RA_IN_BOUNDS(h * p.dv + i, 4, p.H * p.dv, kTagDelta))
      store4(static_cast<T*>(p.out) + row * p.ldo + h * p.dv + i,
             make_float4(x[k].x * rs * w.x * gate_f<T>(g[k].x), x[k].y * rs * w.y * gate_f<T>(g[k].y),
                         x[k].z * rs * w.z * gate_f<T>(g[k].z), x[k].w * rs * w.w * gate_f<T>(g[k].w)));
  }
}

// One token per sequence: grid (4 H, B), clusters of four CTAs per value head. Every CTA takes a quarter of the head's value
// channels (columns of S; eight lanes per column), starts by loading them, and makes q and k for itself; the sum of squares
// of o meets through distributed shared memory. The convolution ring is only read at the rows of earlier tokens and only
// written at the row of this one (taps rows apart), so the CTAs that share a q/k head need no order among themselves.
constexpr int STEP_THREADS = 256, STEP_CTAS = 4;
constexpr int STEP_COLS = STEP_THREADS / 8;  // columns per round
template <typename T, int NJ>
__global__ void __cluster_dims__(STEP_CTAS, 1, 1) __launch_bounds__(STEP_THREADS) delta_step_kernel(const Params p) {
  constexpr int DKP = 32 * NJ;
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  extern __shared__ float step_smem[];  // q[DKP], k[DKP], v[nv], o[nv]
  __shared__ float red[32];
  __shared__ float scal[4];             // 1 / |q| * scale, 1 / |k|, g, beta
  __shared__ float sums[STEP_CTAS];
  const int part = static_cast<int>(cluster.block_rank()), h = blockIdx.x / STEP_CTAS, b = blockIdx.y, kvh = h / (p.H / p.G);
  const int nv = (p.dv + STEP_CTAS - 1) / STEP_CTAS, v0 = min(p.dv, part * nv), v1 = min(p.dv, v0 + nv);
  float *sq = step_smem, *sk = sq + DKP, *sv = sk + DKP, *so = sv + nv;
  const int tid = threadIdx.x, l = tid & 7, lane = tid & 31, warp = tid >> 5;
  float* st = p.state + (static_cast<long long>(b) * p.H + h) * p.dv * p.dk;
  const bool vec = (p.dk & 3) == 0;
  float4 S[NJ];
  auto load_cols = [&](int c0) {
    const int col = c0 + (tid >> 3);
    const float* sc = st + static_cast<long long>(col < v1 ? col : 0) * p.dk;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int i = 32 * j + 4 * l, n = col < v1 ? p.dk : 0;
      if (vec) {
        S[j] = i < n ? load4(sc + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      } else {
        S[j].x = i < n ? sc[i] : 0.f;
        S[j].y = i + 1 < n ? sc[i + 1] : 0.f;
        S[j].z = i + 2 < n ? sc[i + 2] : 0.f;
        S[j].w = i + 3 < n ? sc[i + 3] : 0.f;
      }
    }
  };
  load_cols(v0);

  const long long pos = *p.pos;
  const int C = 2 * p.G * p.dk + p.H * p.dv;
  const T* proj_b = static_cast<const T*>(p.proj) + static_cast<long long>(b) * p.ldp;
  float* ring_b = p.ring + static_cast<long long>(b) * p.taps * C;
  float* ring_now = ring_b + static_cast<long long>(ring_slot(pos, p.taps)) * C;
  const bool first_of_group = part == 0 && h % (p.H / p.G) == 0;
  for (int i = tid; i < 2 * DKP + (v1 - v0); i += STEP_THREADS) {
    const int kind = i < DKP ? 0 : (i < 2 * DKP ? 1 : 2);
    const int e = kind == 0 ? i : (kind == 1 ? i - DKP : i - 2 * DKP);
    float x = 0.f;
    if (kind == 2 || e < p.dk) {
      const int nq = p.G * p.dk, hv = h * p.dv + v0 + e;
      const int c = kind == 2 ? 2 * nq + hv : kind * nq + kvh * p.dk + e;
      const int col = kind == 2 ? p.off_v + hv : (kind == 0 ? p.off_q : p.off_k) + kvh * p.dk + e;
      const T* w = static_cast<const T*>(kind == 0 ? p.conv_q : (kind == 1 ? p.conv_k : p.conv_v)) +
                   static_cast<long long>(kind == 2 ? hv : kvh * p.dk + e) * p.taps;
      x = conv_silu(p, proj_b, ring_b, w, 0, pos, C, c, col);
      if (kind == 2 || first_of_group) ring_now[c] = to_f(proj_b[col]);
    }
    step_smem[i] = x;
  }
  if (tid == STEP_THREADS - 1) {
    const float* ba = p.ba + b * p.ldba;
    scal[2] = expf(log_decay(ba[p.off_a + h], to_f(static_cast<const T*>(p.a_log)[h]), to_f(static_cast<const T*>(p.dt_bias)[h])));
    scal[3] = sigmoid_f(ba[h]);
  }
  __syncthreads();
  if (warp < 2) {
    const float* s = warp == 0 ? sq : sk;
    float ss = 0.f;
    for (int i = lane; i < DKP; i += 32) ss += s[i] * s[i];
    ss = sum_warp(ss);
    if (lane == 0) scal[warp] = (warp == 0 ? p.q_scale : 1.f) / sqrtf(ss + 1e-6f);
  }
  __syncthreads();
  const float qm = scal[0], km = scal[1], g = scal[2], beta = scal[3];
  float4 kk[NJ], qq[NJ];
  float qk = 0.f;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    kk[j] = load4(sk + 32 * j + 4 * l);
    qq[j] = load4(sq + 32 * j + 4 * l);
    kk[j] = make_float4(kk[j].x * km, kk[j].y * km, kk[j].z * km, kk[j].w * km);
    qq[j] = make_float4(qq[j].x * qm, qq[j].y * qm, qq[j].z * qm, qq[j].w * qm);
    qk += kk[j].x * qq[j].x + kk[j].y * qq[j].y + kk[j].z * qq[j].z + kk[j].w * qq[j].w;
  }
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) qk += __shfl_xor_sync(0xffffffffu, qk, o);
  float ss = 0.f;
  // the trip count is the same for every thread: the shuffles below see whole warps
  for (int c0 = v0; c0 < v1; c0 += STEP_COLS) {
    if (c0 > v0) load_cols(c0);
    const int col = c0 + (tid >> 3);
    const bool in = col < v1;
    float* sc = st + static_cast<long long>(in ? col : 0) * p.dk;
    float a = 0.f, c = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      a += S[j].x * kk[j].x + S[j].y * kk[j].y + S[j].z * kk[j].z + S[j].w * kk[j].w;
      c += S[j].x * qq[j].x + S[j].y * qq[j].y + S[j].z * qq[j].z + S[j].w * qq[j].w;
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
      a += __shfl_xor_sync(0xffffffffu, a, o);
      c += __shfl_xor_sync(0xffffffffu, c, o);
    }
    const float u = beta * ((in ? sv[col - v0] : 0.f) - g * a);
    const float ov = fmaf(qk, u, g * c);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int i = 32 * j + 4 * l;
      const float4 n = make_float4(fmaf(kk[j].x, u, g * S[j].x), fmaf(kk[j].y, u, g * S[j].y),
                                   fmaf(kk[j].z, u, g * S[j].z), fmaf(kk[j].w, u, g * S[j].w));
      if (!in) continue;
      if (vec) {
        if (i < p.dk) store4(sc + i, n);
      } else {
        if (i < p.dk) sc[i] = n.x;
        if (i + 1 < p.dk) sc[i + 1] = n.y;
        if (i + 2 < p.dk) sc[i + 2] = n.z;
        if (i + 3 < p.dk) sc[i + 3] = n.w;
      }
    }
    if (in && l == 0) {
      so[col - v0] = ov;
      ss += ov * ov;
    }
  }
  ss = sum_block(ss, red);
  cluster.sync();  // every CTA of the cluster has started: its shared memory can be written
  if (tid < STEP_CTAS) cluster.map_shared_rank(sums, tid)[part] = ss;
  cluster.sync();
  const float rs = 1.f / sqrtf((sums[0] + sums[1] + sums[2] + sums[3]) / p.dv + p.eps);
  const T* gate = proj_b + p.off_g + h * p.dv;
  T* out = static_cast<T*>(p.out) + b * p.ldo + h * p.dv;
  for (int i = v0 + tid; i < v1; i += STEP_THREADS)
    if (RA_IN_BOUNDS(h * p.dv + i, 1, p.H * p.dv, kTagDelta)) from_f(out[i], so[i - v0] * rs * to_f(static_cast<const T*>(p.norm_w)[i]) * silu_f(to_f(gate[i])));
}

template <typename T>
int launch_prep(const Params& p, cudaStream_t s) {
  delta_prep_kernel<T><<<dim3(p.B * p.T, (2 * p.G + p.H + 3) / 4), 128, 0, s>>>(p);
  return check_launch("delta_prep_kernel");
}

template <typename T>
int launch_scan(const Params& p, cudaStream_t s) {
  const dim3 grid((p.dv + SCAN_COLS - 1) / SCAN_COLS, p.H, p.B);
  if (p.dk <= 32) delta_scan_kernel<T, 1><<<grid, 128, 0, s>>>(p);
  else if (p.dk <= 64) delta_scan_kernel<T, 2><<<grid, 128, 0, s>>>(p);
  else if (p.dk <= 96) delta_scan_kernel<T, 3><<<grid, 128, 0, s>>>(p);
  else if (p.dk <= 128) delta_scan_kernel<T, 4><<<grid, 128, 0, s>>>(p);
  else delta_scan_kernel<T, 8><<<grid, 128, 0, s>>>(p);
  return check_launch("delta_scan_kernel");
}

template <typename T>
int launch_out(const Params& p, cudaStream_t s) {
  const long long n = static_cast<long long>(p.B) * p.T * p.H;
  const bool vec = (p.dv == 128 || p.dv == 64) && p.ldo % 4 == 0 && p.ldp % 4 == 0 && p.off_g % 4 == 0 &&
                   !((reinterpret_cast<uintptr_t>(p.out) | reinterpret_cast<uintptr_t>(p.proj) |
                      reinterpret_cast<uintptr_t>(p.norm_w) | reinterpret_cast<uintptr_t>(p.o)) & 15);
  if (vec && p.dv == 128)
    delta_out_vec_kernel<T, 32><<<static_cast<unsigned>((n + 31) / 32), 256, 0, s>>>(p);
  else if (vec)
    delta_out_vec_kernel<T, 16><<<static_cast<unsigned>((n + 63) / 64), 256, 0, s>>>(p);
  else
    delta_out_kernel<T><<<static_cast<unsigned>((n + 3) / 4), 128, 0, s>>>(p);
  return check_launch("delta_out_kernel");
}

template <typename T>
int launch_step(const Params& p, cudaStream_t s) {
  const dim3 grid(STEP_CTAS * p.H, p.B);
  const int nv = (p.dv + STEP_CTAS - 1) / STEP_CTAS;
#define RA_STEP(NJ) delta_step_kernel<T, NJ><<<grid, STEP_THREADS, (64 * NJ + 2 * nv) * sizeof(float), s>>>(p)
  if (p.dk <= 32) RA_STEP(1);
  else if (p.dk <= 64) RA_STEP(2);
  else if (p.dk <= 96) RA_STEP(3);
  else if (p.dk <= 128) RA_STEP(4);
  else RA_STEP(8);
#undef RA_STEP
  return check_launch("delta_step_kernel");
}

int check(const Params* p) {
  if (p->B < 1 || p->T < 1 || p->H < 1 || p->G < 1 || p->H % p->G || p->dk < 1 || p->dk > 256 || p->dv < 1 ||
      p->dv > 4096 || p->taps < 1 || p->B > 65535 || p->H > 65535 ||
      static_cast<long long>(p->B) * p->T * p->H > (1ll << 31) - 4) {
    set_error("ra_delta: bad shape (key dim at most 256, value dim at most 4096)");
    return kHostBadArg;
  }
  return kHostOk;
}

}  // namespace delta
}  // namespace ra

// One launcher per kernel. `f32`: proj, out and the mixer's vectors are fp32, else bf16. ra_delta_step takes T = 1 and
// leaves q, k, v, gb and o unused; the other three together are a step of any length.
#define RA_DELTA_ENTRY(NAME, LAUNCH)                                                                       \
  extern "C" int NAME(const ra::delta::Params* p, int f32, void* stream) {                                 \
    const int rc = ra::delta::check(p);                                                                    \
    if (rc) return rc;                                                                                     \
    cudaStream_t s = static_cast<cudaStream_t>(stream);                                                    \
    return f32 ? ra::delta::LAUNCH<float>(*p, s) : ra::delta::LAUNCH<__nv_bfloat16>(*p, s);                \
  }
RA_DELTA_ENTRY(ra_delta_prep, launch_prep)
RA_DELTA_ENTRY(ra_delta_scan, launch_scan)
RA_DELTA_ENTRY(ra_delta_out, launch_out)
RA_DELTA_ENTRY(ra_delta_step, launch_step)
#undef RA_DELTA_ENTRY
