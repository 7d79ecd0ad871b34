// One token per sequence of windowed attention in one launch: query and key norms, rotation, the new row of the key/value
// ring, scores, softmax with the sink, and the output.
//
// A cluster of up to eight CTAs serves one key/value head (up to sixteen of the query heads that share it) of one sequence;
// every CTA takes a share of the window's earlier keys. The query heads are the M side of mma.sync m16n8k16 (eight or sixteen
// rows), sixteen keys a warp's chunk; chunks come through a per-warp cp.async ring that starts before the norms are known.
// The new token's own key and value never go through the ring: the first CTA makes them, writes their row and adds them as
// one more partial result. Partial results stay in shared memory; after a cluster barrier every CTA merges a share of the
// output through distributed shared memory. A window is small beside the memory bandwidth, so the kernel is bound by this
// chain of steps and not by the bytes; a 128-row tcgen05 tile would bring nothing.
#include <cooperative_groups.h>

#include "common/mma_sync.cuh"
#include "window_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace window {

namespace cg = cooperative_groups;

constexpr int WARPS = 8, THREADS = 256, ST = 3, ROWS = 16, MAX_CLUSTER = 8;

// D: padded head size of keys and values in shared memory; FULL: more than eight query rows.
template <int D, bool FULL>
struct DecodeSmem {
  static constexpr int NQ = FULL ? 16 : 8;
  static constexpr int TILE = ROWS * D * 2;
  static constexpr int RING = WARPS * ST * 2 * TILE;         // reused for the warps' partial outputs
  static constexpr int OUT_OFF = RING;                       // float [NQ][D]: this CTA's partial output
  static constexpr int Q_OFF = OUT_OFF + NQ * D * 4;         // bf16 [16][D], 16-byte pieces swizzled by the row
  static constexpr int NEW_OFF = Q_OFF + 16 * D * 2;         // float [2][D]: the new key and value
  static constexpr int TOTAL = NEW_OFF + 2 * D * 4;
  static_assert(RING >= WARPS * NQ * D * 4, "the ring holds the warps' partial outputs");
};

template <int D, bool FULL>
__global__ void __launch_bounds__(THREADS) window_decode_kernel(const Params p) {
  using SM = DecodeSmem<D, FULL>;
  constexpr int NQ = SM::NQ, TILE = SM::TILE, RB = D * 2, PPR = D / 8, NT = D / 8;
  constexpr float kLog2e = 1.4426950408889634f;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ __align__(16) float sn[D / 2], cs[D / 2];
  __shared__ float red[64], part_m[NQ + 1], part_l[NQ], warp_m[WARPS][NQ], warp_l[WARPS][NQ];
  __shared__ float new_s[NQ];
  float* part_o = reinterpret_cast<float*>(smem + SM::OUT_OFF);
  float* new_kv = reinterpret_cast<float*>(smem + SM::NEW_OFF);
  cg::cluster_group cluster = cg::this_cluster();
  const int C = p.splits, rank = static_cast<int>(cluster.block_rank());
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, fg = lane >> 2, ft = lane & 3;
  const int share = p.H / p.G, blocks = (share + NQ - 1) / NQ;
  const int g = blockIdx.y / blocks, h0 = g * share + (blockIdx.y % blocks) * NQ;
  const int nh = min(NQ, (g + 1) * share - h0), b = blockIdx.z;
  const long long pos = *p.pos;
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(p.proj) + b * p.ldp;
  const long long head_row = (static_cast<long long>(b) * p.G + g) * p.R;
  __nv_bfloat16* kb = static_cast<__nv_bfloat16*>(p.k_cache) + head_row * p.kw;
  __nv_bfloat16* vb = static_cast<__nv_bfloat16*>(p.v_cache) + head_row * p.vw;

  // ---- earlier keys of the window: this CTA's share [i0, i1) of the n at positions pos - n .. pos - 1
  const int n = static_cast<int>(pos < p.window - 1 ? pos : p.window - 1);
  const int per = (n + C - 1) / C, i0 = min(n, rank * per), i1 = min(n, i0 + per);
  const int row0 = static_cast<int>((pos - n + p.R) % p.R);
  uint8_t* ring = smem + warp * (ST * 2 * TILE);
  auto issue = [&](int c, int slot) {
    const int base = i0 + (warp + WARPS * c) * ROWS;
    uint8_t* kt = ring + slot * 2 * TILE;
#pragma unroll
    for (int j = 0; j < ROWS * PPR / 32; ++j) {
      const int piece = lane + 32 * j, row = piece / PPR, ch = piece % PPR, i = base + row;
      const bool in = i < i1;
      int r = row0 + (in ? i : 0);
      if (r >= p.R) r -= p.R;
      const bool ik = in && ch * 8 < p.kw && RA_IN_BOUNDS(r, 1, p.R, kTagWindow), iv = in && ch * 8 < p.vw;
      const int off = row * RB + ((ch ^ (row & 7)) << 4);
      cp_async16(kt + off, kb + static_cast<long long>(r) * p.kw + (ik ? ch * 8 : 0), ik ? 16 : 0);
      cp_async16(kt + TILE + off, vb + static_cast<long long>(r) * p.vw + (iv ? ch * 8 : 0), iv ? 16 : 0);
    }
  };
  const int my_rows = i1 - (i0 + warp * ROWS);
  const int n_chunks = my_rows <= 0 ? 0 : (my_rows + WARPS * ROWS - 1) / (WARPS * ROWS);
#pragma unroll
  for (int i = 0; i < ST - 1; ++i) {
    if (i < n_chunks) issue(i, i);
    cp_async_commit();
  }

  // ---- norms over the whole projections, sines, this cluster's query rows and (first CTA) the new key and value
  const int nq = p.H * p.dk, nk = p.G * p.dk, half = p.rot_half, h8 = half >> 3;
  const bool turn8 = !(half & 7);
  uint8_t* sq_rows = smem + SM::Q_OFF;
  float sq = 0.f, sk = 0.f;
  for (int i = tid * 8; i < nq; i += THREADS * 8) sq += square_sum(load_piece(x + p.off_q + i));
  if (rank == 0)
    for (int i = tid * 8; i < nk; i += THREADS * 8) sk += square_sum(load_piece(x + p.off_k + i));
  for (int i = tid; i < half; i += THREADS) sincosf(static_cast<float>(pos) * p.inv_freq[i], &sn[i], &cs[i]);
  for (int i = tid; i < 16 * PPR; i += THREADS) reinterpret_cast<uint4*>(sq_rows)[i] = make_uint4(0u, 0u, 0u, 0u);
  for (int i = tid; i < 2 * D; i += THREADS) new_kv[i] = 0.f;
  const float2 ss = sum_block2(sq, sk, red);
  const float rq = 1.f / sqrtf(ss.x / nq + p.eps), rk = 1.f / sqrtf(ss.y / nk + p.eps);
  const bool writer = rank == 0 && blockIdx.y % blocks == 0;
  const int new_row = static_cast<int>(pos % p.R);
  // dimensions d .. d + 7 of query head h0 + r, or (r = nh) of the new key
  auto put = [&](int r, int d, const Piece& v) {
    if (r < nh) {
      *reinterpret_cast<uint4*>(sq_rows + r * RB + (((d >> 3) ^ (r & 7)) << 4)) = v.u;
      return;
    }
    float f[8];
    unpack(v, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) new_kv[d + e] = f[e];
    if (writer) *reinterpret_cast<uint4*>(kb + static_cast<long long>(new_row) * p.kw + d) = v.u;
  };
  const int heads = rank == 0 ? nh + 1 : nh;
  if (turn8) {
    const int units = (p.dk >> 3) - h8;
    for (int i = tid; i < heads * units; i += THREADS) {
      const int r = i / units, u = i - r * units;
      const __nv_bfloat16* src = r < nh ? x + p.off_q + (h0 + r) * p.dk : x + p.off_k + g * p.dk;
      const __nv_bfloat16* gain = r < nh ? static_cast<const __nv_bfloat16*>(p.q_norm) + (h0 + r) * p.dk
                                         : static_cast<const __nv_bfloat16*>(p.k_norm) + g * p.dk;
      Piece hi = load_piece(src + (u + h8) * 8), lo = hi;
      if (u < h8) lo = load_piece(src + u * 8);
      float gl[8], gh[8];
      unpack(load_piece(gain + (u + h8) * 8), gh);
      if (u < h8) unpack(load_piece(gain + u * 8), gl);
      norm_turn(lo, hi, gl, gh, r < nh ? rq : rk, u, h8, sn, cs);
      put(r, (u + h8) * 8, hi);
      if (u < h8) put(r, u * 8, lo);
    }
  } else {  // pairs that do not fall into pieces
    for (int i = tid; i < heads * (p.dk >> 3); i += THREADS) {
      const int r = i / (p.dk >> 3), d0 = (i - r * (p.dk >> 3)) * 8;
      const __nv_bfloat16* src = r < nh ? x + p.off_q + (h0 + r) * p.dk : x + p.off_k + g * p.dk;
      const __nv_bfloat16* gain = r < nh ? static_cast<const __nv_bfloat16*>(p.q_norm) + (h0 + r) * p.dk
                                         : static_cast<const __nv_bfloat16*>(p.k_norm) + g * p.dk;
      const float rs = r < nh ? rq : rk;
      auto normed = [&](int d) { return __bfloat162float(src[d]) * rs * __bfloat162float(gain[d]); };
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int d = d0 + e;
        f[e] = normed(d);
        if (d < half) f[e] = f[e] * cs[d] - normed(d + half) * sn[d];
        else if (d < 2 * half) f[e] = f[e] * cs[d - half] + normed(d - half) * sn[d - half];
      }
      put(r, d0, pack(f));
    }
  }
  if (rank == 0)
    for (int d = tid * 8; d < p.dv; d += THREADS * 8) {
      const Piece v = load_piece(x + p.off_v + g * p.dv + d);
      float f[8];
      unpack(v, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) new_kv[D + d + e] = f[e];
      if (writer) *reinterpret_cast<uint4*>(vb + static_cast<long long>(new_row) * p.vw + d) = v.u;
    }
  __syncthreads();
  if (rank == 0) {  // the new token's own score, one head a warp at a time
    for (int r = warp; r < nh; r += WARPS) {
      float s = 0.f;
      for (int d = lane; d < p.dk; d += 32)
        s += __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sq_rows + r * RB + (((d >> 3) ^ (r & 7)) << 4) +
                                                                     (d & 7) * 2)) * new_kv[d];
      s = sum_warp(s);
      if (lane == 0) new_s[r] = s * p.scale * kLog2e;
    }
  }
  // query fragments: matrices (rows 0-7 | 8-15) x (piece 2 ks | 2 ks + 1)
  const int mat = lane >> 3, rr = lane & 7;
  uint32_t qa[D / 16][4];
#pragma unroll
  for (int ks = 0; ks < D / 16; ++ks) {
    const int row = rr + 8 * (mat & 1), ch = 2 * ks + (mat >> 1);
    ldmatrix_x4(qa[ks], sq_rows + row * RB + ((ch ^ (row & 7)) << 4));
  }
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  constexpr int NR = FULL ? 2 : 1;  // query rows of a lane: fg and fg + 8
  float m[NR], l[NR];
#pragma unroll
  for (int e = 0; e < NR; ++e) {
    m[e] = -INFINITY;
    l[e] = 0.f;
  }
  const float sc = p.scale * kLog2e;
  int slot = 0;
  for (int c = 0; c < n_chunks; ++c) {
    __syncwarp();
    if (c + ST - 1 < n_chunks) issue(c + ST - 1, (slot + ST - 1) % ST);
    cp_async_commit();
    cp_async_wait<ST - 1>();
    __syncwarp();
    const uint8_t* kt = ring + slot * 2 * TILE;
    const uint8_t* vt = kt + TILE;
    const int base = i0 + (warp + WARPS * c) * ROWS;
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
    {
      const int row = rr + 8 * (mat >> 1);
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        const int ch = 2 * ks + (mat & 1);
        uint32_t bf[4];
        ldmatrix_x4(bf, kt + row * RB + ((ch ^ (row & 7)) << 4));
        if (FULL) {
          mma_16816(s[0], qa[ks], bf[0], bf[1]);
          mma_16816(s[1], qa[ks], bf[2], bf[3]);
        } else {
          mma_16816_top(s[0], qa[ks][0], qa[ks][2], bf[0], bf[1]);
          mma_16816_top(s[1], qa[ks][0], qa[ks][2], bf[2], bf[3]);
        }
      }
    }
    uint32_t pa[4] = {0u, 0u, 0u, 0u};
#pragma unroll
    for (int q = 0; q < NR; ++q) {
      float xv[2][2], mx = -INFINITY;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          xv[nt][e] = base + 8 * nt + 2 * ft + e < i1 ? s[nt][2 * q + e] * sc : -INFINITY;
          mx = fmaxf(mx, xv[nt][e]);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m[q], mx);  // finite: a chunk has at least one key
      const float alpha = exp2f(m[q] - m_new);
      float sum = 0.f;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          xv[nt][e] = exp2f(xv[nt][e] - m_new);
          sum += xv[nt][e];
        }
      l[q] = l[q] * alpha + sum;
      m[q] = m_new;
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        o[j][2 * q] *= alpha;
        o[j][2 * q + 1] *= alpha;
      }
      const __nv_bfloat162 p0 = __floats2bfloat162_rn(xv[0][0], xv[0][1]), p1 = __floats2bfloat162_rn(xv[1][0], xv[1][1]);
      pa[q] = *reinterpret_cast<const uint32_t*>(&p0);
      pa[2 + q] = *reinterpret_cast<const uint32_t*>(&p1);
    }
    {
      const int row = rr + 8 * (mat & 1);
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        const int ch = 2 * j + (mat >> 1);
        uint32_t bf[4];
        ldmatrix_x4_trans(bf, vt + row * RB + ((ch ^ (row & 7)) << 4));
        if (FULL) {
          mma_16816(o[2 * j], pa, bf[0], bf[1]);
          mma_16816(o[2 * j + 1], pa, bf[2], bf[3]);
        } else {
          mma_16816_top(o[2 * j], pa[0], pa[2], bf[0], bf[1]);
          mma_16816_top(o[2 * j + 1], pa[0], pa[2], bf[2], bf[3]);
        }
      }
    }
    slot = slot + 1 == ST ? 0 : slot + 1;
  }
  cp_async_wait<0>();
  __syncthreads();  // every warp is done with the ring

  // ---- the CTA's partial result: maxima, sums and outputs of its warps (the first CTA adds the new token)
  float* warp_o = reinterpret_cast<float*>(smem);  // [WARPS][NQ][D]
#pragma unroll
  for (int q = 0; q < NR; ++q) {
    l[q] += __shfl_xor_sync(0xffffffffu, l[q], 1);
    l[q] += __shfl_xor_sync(0xffffffffu, l[q], 2);
    const int r = fg + 8 * q;
    if (ft == 0) {
      warp_m[warp][r] = m[q];
      warp_l[warp][r] = l[q];
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
      *reinterpret_cast<float2*>(warp_o + (warp * NQ + r) * D + 8 * j + 2 * ft) = make_float2(o[j][2 * q], o[j][2 * q + 1]);
  }
  __syncthreads();
  for (int i = tid; i < nh * D; i += THREADS) {
    const int r = i / D, d = i % D;
    float mx = rank == 0 ? new_s[r] : -INFINITY;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) mx = fmaxf(mx, warp_m[w][r]);
    const float mu = mx == -INFINITY ? 0.f : mx;
    float lt = 0.f, ot = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float a = exp2f(warp_m[w][r] - mu);
      lt += warp_l[w][r] * a;
      ot += warp_o[(w * NQ + r) * D + d] * a;
    }
    if (rank == 0) {
      const float a = exp2f(new_s[r] - mu);
      lt += a;
      ot += new_kv[D + d] * a;
    }
    part_o[r * D + d] = ot;
    if (d == 0) {
      part_m[r] = mx;
      part_l[r] = lt;
    }
  }
  cluster.sync();
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + b * p.ldo + h0 * p.dv;
  for (int i = rank * THREADS + tid; i < nh * p.dv; i += C * THREADS) {
    const int r = i / p.dv, d = i - r * p.dv;
    const float s = p.sink[h0 + r] * kLog2e;
    float pm[MAX_CLUSTER], pl[MAX_CLUSTER], po[MAX_CLUSTER], mx = s;
#pragma unroll
    for (int c = 0; c < MAX_CLUSTER; ++c) {  // all reads of other CTAs' shared memory on their way at once
      const int cc = c < C ? c : 0;
      pm[c] = cluster.map_shared_rank(part_m, cc)[r];
      pl[c] = cluster.map_shared_rank(part_l, cc)[r];
      po[c] = cluster.map_shared_rank(part_o, cc)[r * D + d];
    }
#pragma unroll
    for (int c = 0; c < MAX_CLUSTER; ++c)
      if (c < C) mx = fmaxf(mx, pm[c]);
    float lt = exp2f(s - mx), ot = 0.f;
#pragma unroll
    for (int c = 0; c < MAX_CLUSTER; ++c)
      if (c < C) {
        const float a = exp2f(pm[c] - mx);
        lt += pl[c] * a;
        ot += po[c] * a;
      }
    if (RA_IN_BOUNDS(h0 * p.dv + i, 1, p.ldo, kTagWindow)) out[i] = __float2bfloat16(ot / lt);
  }
  cluster.sync();  // nobody's shared memory goes away while it is read
}

template <int D, bool FULL>
int launch_decode(const Params& p, cudaStream_t s) {
  using SM = DecodeSmem<D, FULL>;
  auto kern = window_decode_kernel<D, FULL>;
  if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM::TOTAL) != cudaSuccess) {
    cudaGetLastError();
    set_error("window_decode: smem attribute");
    return kHostLaunchFail;
  }
  const int share = p.H / p.G;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.splits, p.G * ((share + SM::NQ - 1) / SM::NQ), p.B);
  cfg.blockDim = dim3(THREADS);
  cfg.dynamicSmemBytes = SM::TOTAL;
  cfg.stream = s;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = p.splits;
  at[0].val.clusterDim.y = 1;
  at[0].val.clusterDim.z = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  if (cudaLaunchKernelEx(&cfg, kern, p) != cudaSuccess) {
    cudaGetLastError();
    set_error("window_decode: launch failed");
    return kHostLaunchFail;
  }
  return check_launch("window_decode_kernel");
}

}  // namespace window
}  // namespace ra

// One token per sequence (T = 1), bf16, head sizes that are multiples of eight up to 128; norms, rotation and the append
// included (no ra_window_prep before it).
extern "C" int ra_window_decode(const ra::window::Params* pp, void* stream) {
  using namespace ra;
  using namespace ra::window;
  if (const int rc = check(pp)) return rc;
  Params p = *pp;
  if (p.T != 1 || p.dk % 8 || p.dv % 8 || p.dk > 128 || p.dv > 128 || p.n_max < 1) {
    set_error("ra_window_decode: bad shape");
    return kHostBadArg;
  }
  const int share = p.H / p.G, nq = share > 8 ? 16 : 8;
  const bool small = p.dk <= 64 && p.dv <= 64;
  const long long work = static_cast<long long>(p.G) * ((share + nq - 1) / nq) * p.B;
  const long long keys = p.n_max < p.window ? p.n_max : p.window;
  const long long fit = static_cast<long long>(sm_count()) * (small ? 2 : 1);  // CTAs that run at once
  int c = MAX_CLUSTER;  // CTAs of a cluster: as many as run at once, at least 32 keys each
  while (c > 1 && (work * c > fit || keys < 32ll * c)) c >>= 1;
  p.splits = c;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (nq == 8) return small ? launch_decode<64, false>(p, s) : launch_decode<128, false>(p, s);
  return small ? launch_decode<64, true>(p, s) : launch_decode<128, true>(p, s);
}
