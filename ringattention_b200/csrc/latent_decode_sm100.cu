// Latent attention for a few new tokens over a long cache (decode steps and short portions), bf16: the absorbed form of
// latent_sm100.cu on the tensor cores. The rows of one step, T tokens x H heads of a sequence, all read the same cached
// latents, so a CTA takes 16 or 32 of them against a range of the cache, which it reads once, as keys and as values:
//   latent_query_kernel  : per (head, row) the absorbed query, one extra CTA per row appends the row to the cache
//   latent_splitkv_kernel: tiles of 64 cached rows arrive by TMA (128-byte swizzle) in a three-stage ring; S = Q_lat K^T with the
//                          query fragments in registers, the tile's rows divided over the warps; row maxima meet in shared memory;
//                          P goes through shared memory; O += P C with the latent columns divided over the warps
//   latent_output_kernel : merge of the splits, sink, value projection, output gate
#include <cooperative_groups.h>

#include "common/mma_sync.cuh"
#include "common/sm100.cuh"
#include "latent_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace latent {

using bf16 = __nv_bfloat16;

// grid (H + 1, rows, ceil(r / 128)). Head CTAs take 128 latent columns: eight per thread, the head's unrotated dimensions
// divided over 32 groups of threads; the first weights are on their way before the query is read. Block H appends the row.
constexpr int QRY_THREADS = 512;
constexpr int QRY_COLS = 128;
constexpr int QRY_GROUPS = QRY_THREADS / (QRY_COLS / 8);
constexpr int QRY_AHEAD = 4;  // weight rows per thread that are loaded up front
__global__ void __launch_bounds__(QRY_THREADS) latent_query_kernel(const Params p) {
  extern __shared__ float sq[];  // q[dn]
  __shared__ __align__(16) float part[QRY_GROUPS][QRY_COLS];
  __shared__ float red[32];
  const int h = blockIdx.x, c0 = blockIdx.z * QRY_COLS;
  const long long row = blockIdx.y;
  const int b = blockIdx.y / p.T, t = blockIdx.y - b * p.T;
  if (h == p.H) {
    if (blockIdx.z == 0) append_row<bf16>(p, row, b, *p.pos + t, red);
    return;
  }
  const int cg = threadIdx.x % (QRY_COLS / 8), grp = threadIdx.x / (QRY_COLS / 8);
  const bool in = c0 + cg * 8 < p.r;
  const bf16* w = static_cast<const bf16*>(p.w_uk) + static_cast<long long>(h) * p.dn * p.ldw + (in ? c0 + cg * 8 : 0);
  uint4 u[QRY_AHEAD];
#pragma unroll
  for (int k = 0; k < QRY_AHEAD; ++k) {
    const int i = grp + k * QRY_GROUPS;
    u[k] = i < p.dn ? __ldg(reinterpret_cast<const uint4*>(w + i * p.ldw)) : make_uint4(0u, 0u, 0u, 0u);
  }
  const bf16* q = static_cast<const bf16*>(p.proj) + row * p.ldp + p.off_q + h * (p.dn + p.dr);
  bf16* dst = static_cast<bf16*>(p.q_lat) + (row * p.H + h) * p.row_w;
  for (int i = threadIdx.x; i < p.dn; i += QRY_THREADS) sq[i] = to_f(q[i]);
  if (blockIdx.z == 0) {
    const long long pos = *p.pos + t;
    for (int j = threadIdx.x; j < p.dr / 2; j += QRY_THREADS) rotate_pair(p, q + p.dn, dst + p.r_pad, j, pos);
    for (int i = p.r_pad + p.dr + threadIdx.x; i < p.row_w; i += QRY_THREADS) dst[i] = __float2bfloat16(0.f);
  }
  __syncthreads();
  float a[8] = {};
  auto add = [&](int i, const uint4& v) {
    const __nv_bfloat162* b2 = reinterpret_cast<const __nv_bfloat162*>(&v);
    const float x = sq[i];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(b2[e]);
      a[2 * e] = fmaf(x, f.x, a[2 * e]);
      a[2 * e + 1] = fmaf(x, f.y, a[2 * e + 1]);
    }
  };
#pragma unroll
  for (int k = 0; k < QRY_AHEAD; ++k)
    if (grp + k * QRY_GROUPS < p.dn) add(grp + k * QRY_GROUPS, u[k]);
  for (int i = grp + QRY_AHEAD * QRY_GROUPS; i < p.dn; i += QRY_GROUPS)
    add(i, __ldg(reinterpret_cast<const uint4*>(w + i * p.ldw)));
  store4(&part[grp][cg * 8], make_float4(a[0], a[1], a[2], a[3]));
  store4(&part[grp][cg * 8 + 4], make_float4(a[4], a[5], a[6], a[7]));
  __syncthreads();
  const int c = threadIdx.x;
  if (c < QRY_COLS && c0 + c < p.r) {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < QRY_GROUPS; ++k) s += part[k][c];
    if (RA_IN_BOUNDS(c0 + c, 1, p.row_w, kTagLatentWork)) dst[c0 + c] = __float2bfloat16(s);
  }
}

constexpr int ROWS = 64;          // cached rows per tile
constexpr int STAGES = 3;
constexpr int KV_THREADS = 256;
constexpr int SLAB = ROWS * 128;  // 64 columns of a tile

// element address: 16-byte piece pc of row `row` in a tile of 64-column slabs with the TMA's 128-byte swizzle
__device__ __forceinline__ const uint8_t* slab_piece(const uint8_t* tile, int row, int pc) {
  return tile + (pc >> 3) * SLAB + row * 128 + (((pc & 7) ^ (row & 7)) << 4);
}

template <int KS>
struct KvSmem {
  static constexpr int SLABS = (KS + 3) / 4;
  static constexpr int STAGE = SLABS * SLAB;
  static constexpr int P = STAGES * STAGE;     // (32, 64) bf16, swizzled
  static constexpr int MAX = P + 32 * 128;     // (32, 8) floats
  static constexpr int BAR = MAX + 32 * 8 * 4;
  static constexpr int TOTAL = BAR + 64 + 1024 /*align*/;
};

// KS: k-steps of 16 columns that cover a cached row; MT: query tiles of 16 rows per CTA (1 or 2). r <= 16 * KS. FULL: the
// latent columns are exactly those of the warps' pairs (no tests in the product loop).
template <int KS, int MT, bool FULL>
__global__ void __launch_bounds__(KV_THREADS, 1)
latent_splitkv_kernel(const __grid_constant__ CUtensorMap tma, const Params p) {
  using SM = KvSmem<KS>;
  constexpr int NG = 8 / MT;                        // groups of tile rows, one per warp (pair)
  constexpr int PAIRS = (KS > 32 ? 32 : KS) / 8 + (((KS > 32 ? 32 : KS) % 8) ? 1 : 0);  // 16-column pairs of O per warp
  extern __shared__ uint8_t kv_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(kv_smem) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t* sP = smem + SM::P;
  float* sMax = reinterpret_cast<float*>(smem + SM::MAX);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + SM::BAR);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(full + STAGES);
  const WaitCtx wc{abort_flag, p.status};
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3, mat = lane >> 3, rr = lane & 7;
  const int split = blockIdx.x, b = blockIdx.z, row0 = blockIdx.y * 16 * MT, n_q = p.T * p.H;
  const int mt = MT == 2 ? warp & 1 : 0, ng = MT == 2 ? warp >> 1 : warp;
  const long long pos0 = *p.pos;
  long long n_ll = pos0 + p.T;
  if (n_ll > p.S_max) n_ll = p.S_max;
  const int n = static_cast<int>(n_ll);             // rows of the cache that hold tokens
  const int tiles = (n + ROWS - 1) / ROWS, per = (tiles + p.splits - 1) / p.splits;
  const int j0 = split * per, j1 = min(tiles, j0 + per);
  constexpr int slabs = SM::SLABS;  // all of them, also where a row is narrower: columns past it arrive as zeros

  if (tid == 0) {
    for (int s = 0; s < STAGES; ++s) mbar_init(&full[s], 1);
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tma);
  }
  __syncthreads();
  auto fill = [&](int j) {  // tile j0 + i goes to stage i % STAGES
    const int s = (j - j0) % STAGES;
    mbar_arrive_expect_tx(&full[s], slabs * SLAB);
    for (int k = 0; k < slabs; ++k) tma_load_3d(smem + s * SM::STAGE + k * SLAB, &tma, &full[s], k * 64, j * ROWS, b);
  };
  if (tid == 0) {
    if (j0 < j1) fill(j0);
    if (j0 + 1 < j1) fill(j0 + 1);
  }

  // ---- query fragments of this warp's 16 rows, through the third stage's buffer (first filled in the first round)
  uint32_t qa[KS][4];
  {
    uint8_t* sq = smem + 2 * SM::STAGE;  // (16 MT, 64 SLABS) in slabs like a tile
    constexpr int PIECES = SM::SLABS * 8;
    const bf16* q = static_cast<const bf16*>(p.q_lat) + static_cast<long long>(b) * n_q * p.row_w;
    for (int i = tid; i < 16 * MT * PIECES; i += KV_THREADS) {
      const int r = i / PIECES, pc = i % PIECES;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (row0 + r < n_q && pc * 8 < p.row_w)
        v = __ldg(reinterpret_cast<const uint4*>(q + static_cast<long long>(row0 + r) * p.row_w + pc * 8));
      *reinterpret_cast<uint4*>(const_cast<uint8_t*>(slab_piece(sq, r, pc))) = v;
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) ldmatrix_x4(qa[ks], slab_piece(sq, mt * 16 + (mat & 1) * 8 + rr, 2 * ks + (mat >> 1)));
    fence_proxy_async_smem();  // these generic accesses before the bulk copy that refills the buffer
  }
  // last visible row (exclusive) of the two score rows of this thread
  int lim[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = row0 + mt * 16 + g + 8 * i;
    lim[i] = r < n_q ? min(n, static_cast<int>(pos0) + r / p.H + 1) : 0;
  }
  float o[MT][2 * PAIRS][4];
  float m[MT][2], l[2] = {0.f, 0.f};  // l: this thread's share of its score rows' sums
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    m[i][0] = m[i][1] = -INFINITY;
#pragma unroll
    for (int j = 0; j < 2 * PAIRS; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][j][e] = 0.f;
  }
  const float scale2 = p.scale * 1.4426950408889634f;

  for (int j = j0; j < j1; ++j) {
    const int it = j - j0, st = it % STAGES;
    uint8_t* tile = smem + st * SM::STAGE;
    mbar_wait(&full[st], (it / STAGES) & 1, wc, kTimeoutSmemFull);
    const int base = j * ROWS;
    if (base + ROWS > n) {  // the last tile: rows that hold no token yet must not reach a product (0 * NaN)
      for (int i = tid; i < slabs * ROWS * 8; i += KV_THREADS) {
        const int row = (i >> 3) % ROWS, k = (i >> 3) / ROWS;
        if (base + row >= n) *reinterpret_cast<uint4*>(tile + k * SLAB + row * 128 + (i & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
      }
      __syncthreads();
    }
    // ---- S: rows of the query tile x this warp's 8 MT cached rows
    float s[2][MT][4];  // even and odd k-steps apart: two independent chains
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[h][i][e] = 0.f;
    if (MT == 2) {
      const int row = ng * 16 + (mat >> 1) * 8 + rr;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t bf[4];
        ldmatrix_x4(bf, slab_piece(tile, row, 2 * ks + (mat & 1)));
        mma_16816(s[ks & 1][0], qa[ks], bf[0], bf[1]);
        mma_16816(s[ks & 1][MT - 1], qa[ks], bf[2], bf[3]);
      }
    } else {
      const int row = ng * 8 + rr;
#pragma unroll
      for (int ks = 0; ks < KS; ks += 2) {
        uint32_t bf[4];
        ldmatrix_x4(bf, slab_piece(tile, row, 2 * ks + mat));
        mma_16816(s[0][0], qa[ks], bf[0], bf[1]);
        if (ks + 1 < KS) mma_16816(s[1][0], qa[ks + 1 < KS ? ks + 1 : ks], bf[2], bf[3]);
      }
    }
    float x[MT][4], mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int kv = base + (ng * MT + i) * 8 + 2 * t + (e & 1);
        x[i][e] = kv < lim[e >> 1] ? (s[0][i][e] + s[1][i][e]) * scale2 : -INFINITY;
        mx[e >> 1] = fmaxf(mx[e >> 1], x[i][e]);
      }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      if (t == 0) sMax[(mt * 16 + g + 8 * i) * 8 + ng] = mx[i];
    }
    __syncthreads();
    if (tid == 0 && j + STAGES - 1 < j1) fill(j + STAGES - 1);  // every warp is done with the tile before this one
    // ---- running maxima of all rows (the same in every warp), probabilities of this thread's
    float alpha[MT][2];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const float* sm = sMax + (i * 16 + g + 8 * k) * 8;
        float v = m[i][k];
#pragma unroll
        for (int q = 0; q < NG; q += 4) {
          const float4 f = *reinterpret_cast<const float4*>(sm + q);
          v = fmaxf(v, fmaxf(fmaxf(f.x, f.y), fmaxf(f.z, f.w)));
        }
        const float mu = v == -INFINITY ? 0.f : v;
        alpha[i][k] = exp2_approx(m[i][k] - mu);
        m[i][k] = v;
      }
    float mrow[2], arow[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const float v = MT == 2 && mt ? m[MT - 1][k] : m[0][k];
      mrow[k] = v == -INFINITY ? 0.f : v;
      arow[k] = MT == 2 && mt ? alpha[MT - 1][k] : alpha[0][k];
      l[k] *= arow[k];
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const float p0 = exp2_approx(x[i][2 * k] - mrow[k]), p1 = exp2_approx(x[i][2 * k + 1] - mrow[k]);
        l[k] += p0 + p1;
        const int row = mt * 16 + g + 8 * k, pc = ng * MT + i;
        *reinterpret_cast<uint32_t*>(sP + row * 128 + ((pc ^ (row & 7)) << 4) + 4 * t) = pack_bf16x2(p0, p1);
      }
    __syncthreads();
    // ---- O: all rows x this warp's latent columns
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int q = 0; q < 2 * PAIRS; ++q) {
        o[i][q][0] *= alpha[i][0];
        o[i][q][1] *= alpha[i][0];
        o[i][q][2] *= alpha[i][1];
        o[i][q][3] *= alpha[i][1];
      }
#pragma unroll
    for (int ks = 0; ks < ROWS / 16; ++ks) {
      uint32_t pa[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const int row = i * 16 + (mat & 1) * 8 + rr, pc = 2 * ks + (mat >> 1);
        ldmatrix_x4(pa[i], sP + row * 128 + ((pc ^ (row & 7)) << 4));
      }
#pragma unroll
      for (int q = 0; q < PAIRS; ++q) {
        const int pair = warp + 8 * q;
        if (!FULL && pair * 16 >= p.r) continue;
        uint32_t bf[4];
        ldmatrix_x4_trans(bf, slab_piece(tile, ks * 16 + (mat & 1) * 8 + rr, 2 * pair + (mat >> 1)));
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_16816(o[i][2 * q], pa[i], bf[0], bf[1]);
          mma_16816(o[i][2 * q + 1], pa[i], bf[2], bf[3]);
        }
      }
    }
  }
  // ---- row sums over the warps, normalised partial outputs
  __syncthreads();
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    l[k] += __shfl_xor_sync(0xffffffffu, l[k], 1);
    l[k] += __shfl_xor_sync(0xffffffffu, l[k], 2);
    if (t == 0) sMax[(mt * 16 + g + 8 * k) * 8 + ng] = l[k];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int r = row0 + i * 16 + g + 8 * k;
      float lt = 0.f;
#pragma unroll
      for (int q = 0; q < NG; ++q) lt += sMax[(i * 16 + g + 8 * k) * 8 + q];
      const float inv = lt > 0.f ? 1.f / lt : 0.f;
      if (r >= n_q) continue;
      const long long pi = (static_cast<long long>(b) * n_q + r) * p.splits + split;
#pragma unroll
      for (int q = 0; q < PAIRS; ++q) {
        const int c = (warp + 8 * q) * 16 + 2 * t;
        if (c >= p.r || !RA_IN_BOUNDS(pi * p.r + c, 10, static_cast<long long>(p.B) * n_q * p.splits * p.r, kTagLatentWork)) continue;
        float* dst = p.o_part + pi * p.r + c;
        *reinterpret_cast<float2*>(dst) = make_float2(o[i][2 * q][2 * k] * inv, o[i][2 * q][2 * k + 1] * inv);
        *reinterpret_cast<float2*>(dst + 8) = make_float2(o[i][2 * q + 1][2 * k] * inv, o[i][2 * q + 1][2 * k + 1] * inv);
      }
      if (warp == 0 && t == 0) p.lse_part[pi] = lt > 0.f ? (m[i][k] + log2f(lt)) * 0.6931471805599453f : -INFINITY;
    }
  if (*abort_flag) bounded_drain_pause();
}

// grid (4 H, rows), clusters of four CTAs per head and row. CTA k of a cluster merges the splits of a quarter of the latent
// columns, hands its quarter to the other three through distributed shared memory, and multiplies a quarter of the head's
// value projection with the whole; the first weights are on their way meanwhile. r a multiple of 16.
constexpr int OUT_THREADS = 256, OUT_CTAS = 4, OUT_WARPS = OUT_THREADS / 32;
constexpr int OUT_MAX_R = 512;
__global__ void __cluster_dims__(OUT_CTAS, 1, 1) __launch_bounds__(OUT_THREADS) latent_output_kernel(const Params p) {
  extern __shared__ float sw[];  // weights of the splits
  __shared__ __align__(16) float o_lat[OUT_MAX_R], part[OUT_THREADS][4];
  __shared__ float red[32];
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int k = static_cast<int>(cluster.block_rank()), h = blockIdx.x / OUT_CTAS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long row = blockIdx.y;
  // ---- this CTA's rows of the value projection: v0 + warp, + OUT_WARPS, ...; the first two rows of a warp up front
  const int nv = (p.dv + OUT_CTAS - 1) / OUT_CTAS, v0 = k * nv, v1 = min(p.dv, v0 + nv);
  const bf16* wv = static_cast<const bf16*>(p.w_uv) + static_cast<long long>(h) * p.dv * p.ldw;
  constexpr int AHEAD = 4;
  uint4 u[AHEAD][OUT_MAX_R / 256];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
#pragma unroll
    for (int j = 0; j < OUT_MAX_R / 256; ++j) {
      const int v = v0 + warp + i * OUT_WARPS, c = j * 256 + lane * 8;
      u[i][j] = v < v1 && c < p.r ? __ldg(reinterpret_cast<const uint4*>(wv + v * p.ldw + c)) : make_uint4(0u, 0u, 0u, 0u);
    }
  const float* lp = p.lse_part + (row * p.H + h) * p.splits;
  const float* op = p.o_part + (row * p.H + h) * p.splits * p.r;
  float mx = p.sink ? p.sink[h] : -INFINITY;
  for (int s = lane; s < p.splits; s += 32) mx = fmaxf(mx, lp[s]);  // every warp takes them all
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
  float den = 0.f;
  for (int s = threadIdx.x; s < p.splits; s += OUT_THREADS) {
    sw[s] = expf(lp[s] - mx);
    den += sw[s];
  }
  den = sum_block(den, red) + (p.sink ? expf(p.sink[h] - mx) : 0.f);
  const float mul = sigmoid_f(to_f(static_cast<const bf16*>(p.proj)[row * p.ldp + p.off_g + h])) / den;
  // ---- a quarter of the columns: nc groups of four, the splits divided over the thread groups
  const int nc = p.r / 16, groups = OUT_THREADS / nc, c4 = threadIdx.x % nc, grp = threadIdx.x / nc;
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  if (grp < groups) {
#pragma unroll 8
    for (int s = grp; s < p.splits; s += groups) {
      const float w = sw[s];
      const float4 v = load4(op + static_cast<long long>(s) * p.r + k * (p.r / 4) + 4 * c4);
      a.x = fmaf(w, v.x, a.x);
      a.y = fmaf(w, v.y, a.y);
      a.z = fmaf(w, v.z, a.z);
      a.w = fmaf(w, v.w, a.w);
    }
  }
  store4(part[threadIdx.x], a);
  cluster.sync();  // also: every CTA of the cluster has started, its shared memory can be written
  for (int c = threadIdx.x; c < p.r / 4; c += OUT_THREADS) {
    float s = 0.f;
    for (int q = 0; q < groups; ++q) s += part[q * nc + (c >> 2)][c & 3];
    s *= mul;
#pragma unroll
    for (int q = 0; q < OUT_CTAS; ++q) cluster.map_shared_rank(o_lat, q)[k * (p.r / 4) + c] = s;
  }
  cluster.sync();
  bf16* out = static_cast<bf16*>(p.out) + row * p.ldo + h * p.dv;
  auto dot = [&](const uint4& v, int c) {
    const __nv_bfloat162* b2 = reinterpret_cast<const __nv_bfloat162*>(&v);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(b2[e]);
      s = fmaf(o_lat[c + 2 * e], f.x, fmaf(o_lat[c + 2 * e + 1], f.y, s));
    }
    return s;
  };
#pragma unroll
  for (int i = 0; i < AHEAD; ++i) {
    const int v = v0 + warp + i * OUT_WARPS;
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < OUT_MAX_R / 256; ++j) {
      const int c = j * 256 + lane * 8;
      if (c < p.r) s += dot(u[i][j], c);
    }
    s = sum_warp(s);
    if (lane == 0 && v < v1 && RA_IN_BOUNDS(h * p.dv + v, 1, p.H * p.dv, kTagLatent)) out[v] = __float2bfloat16(s);
  }
  for (int v = v0 + warp + AHEAD * OUT_WARPS; v < v1; v += OUT_WARPS) {
    float s = 0.f;
    for (int c = lane * 8; c < p.r; c += 256) s += dot(__ldg(reinterpret_cast<const uint4*>(wv + v * p.ldw + c)), c);
    s = sum_warp(s);
    if (lane == 0 && RA_IN_BOUNDS(h * p.dv + v, 1, p.H * p.dv, kTagLatent)) out[v] = __float2bfloat16(s);
  }
}

template <int KS, int MT>
int launch_splitkv(const CUtensorMap& tma, const Params& p, cudaStream_t s) {
  auto kern = p.r == 512 ? latent_splitkv_kernel<KS, MT, (KS > 32)> : latent_splitkv_kernel<KS, MT, false>;
  constexpr int smem = KvSmem<KS>::TOTAL;
  static_assert(smem <= 227 * 1024, "the tile ring does not fit in shared memory");
  if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) {
    set_error("latent_splitkv: shared memory");
    return kHostLaunchFail;
  }
  const dim3 grid(p.splits, (p.T * p.H + 16 * MT - 1) / (16 * MT), p.B);
  kern<<<grid, KV_THREADS, smem, s>>>(tma, p);
  return check_launch("latent_splitkv_kernel");
}

int check_few(const Params* p) {
  const int rc = check(p);
  if (rc) return rc;
  if (p->r % 16 || p->r > 512 || p->row_w % 16 || p->row_w > 576 || p->dr % 2 || p->dn < 1 || p->dn > 1024 || p->ldw % 8 ||
      p->r_pad != p->r || p->S_max > (1ll << 31) - 64 || p->splits > 4096 ||
      ((reinterpret_cast<uintptr_t>(p->w_uk) | reinterpret_cast<uintptr_t>(p->w_uv) | reinterpret_cast<uintptr_t>(p->cache) |
        reinterpret_cast<uintptr_t>(p->q_lat) | reinterpret_cast<uintptr_t>(p->o_part)) & 15)) {
    set_error("ra_latent_few: latent rank and row width in multiples of 16, at most 512 and 576");
    return kHostBadArg;
  }
  return kHostOk;
}

}  // namespace latent
}  // namespace ra

// bf16. The three launches are the whole mixer of a step of few tokens (no ra_latent_prep before them); q_lat is bf16.
extern "C" int ra_latent_few_query(const ra::latent::Params* p, void* stream) {
  using namespace ra::latent;
  const int rc = check_few(p);
  if (rc) return rc;
  const dim3 grid(p->H + 1, p->B * p->T, (p->r + QRY_COLS - 1) / QRY_COLS);
  latent_query_kernel<<<grid, QRY_THREADS, p->dn * sizeof(float), static_cast<cudaStream_t>(stream)>>>(*p);
  return ra::check_launch("latent_query_kernel");
}

extern "C" int ra_latent_few_attend(const ra::latent::Params* p, void* stream) {
  using namespace ra;
  using namespace ra::latent;
  int rc = check_few(p);
  if (rc) return rc;
  CUtensorMap tma;
  uint64_t dims[3] = {static_cast<uint64_t>(p->row_w), static_cast<uint64_t>(p->S_max), static_cast<uint64_t>(p->B)};
  uint64_t str[2] = {static_cast<uint64_t>(p->row_w) * 2, static_cast<uint64_t>(p->row_w) * 2 * static_cast<uint64_t>(p->S_max)};
  uint32_t box[3] = {64, ROWS, 1};
  if ((rc = make_tmap_bf16_sw128(&tma, p->cache, 3, dims, str, box))) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool one = p->T * p->H <= 16;
  if (p->row_w <= 192) return one ? launch_splitkv<12, 1>(tma, *p, s) : launch_splitkv<12, 2>(tma, *p, s);
  if (p->row_w <= 320) return one ? launch_splitkv<20, 1>(tma, *p, s) : launch_splitkv<20, 2>(tma, *p, s);
  return one ? launch_splitkv<36, 1>(tma, *p, s) : launch_splitkv<36, 2>(tma, *p, s);
}

extern "C" int ra_latent_few_output(const ra::latent::Params* p, void* stream) {
  using namespace ra::latent;
  const int rc = check_few(p);
  if (rc) return rc;
  latent_output_kernel<<<dim3(OUT_CTAS * p->H, p->B * p->T), OUT_THREADS, p->splits * sizeof(float),
                         static_cast<cudaStream_t>(stream)>>>(*p);
  return ra::check_launch("latent_output_kernel");
}
