// Gated delta rule over many tokens, in chunks of 64, on the tensor cores.
//
// Within a chunk that starts from state S, with the running decay c_i = g_1 ... g_i, the recurrence
//     S_i = g_i S_{i-1} + k_i u_i^T,   u_i = beta_i (v_i - g_i S_{i-1}^T k_i),   o_i = S_i^T q_i
// unrolls to  S_i = c_i S + sum_{j <= i} (c_i / c_j) k_j u_j^T, so that with
//     A_ij = beta_i (c_i / c_j) (k_i . k_j)  (j < i),     M_ij = (c_i / c_j) (q_i . k_j)  (j <= i)
// the chunk is
//     (I + A) [W | U0] = [diag(beta c) K | diag(beta) V]      (unit lower triangular solves)
//     U = U0 - W S,    O = diag(c) Q S + M U,    S <- c_64 S + K^T diag(c_64 / c) U
// (the WY form of the product of the tokens' rank-one updates). Two kernels:
//   delta_chunk_prep_kernel : one CTA per (chunk, value head); chunks do not depend on one another. Convolutions + silu, unit
//       norms, decays, K K^T and Q K^T on the tensor cores, the triangular solve with one column of [W | U0] per thread in
//       registers. Leaves -W, M, Q, K as images of the shared-memory tiles the second kernel wants.
//   delta_chunk_scan_kernel : walks the chunks. A warp owns 16 value channels; S^T (16 x dk) stays in its accumulators. In the
//       transposed form the accumulator fragments of S^T and U^T are the A operands of the products that follow, so
//       nothing passes between warps. Tiles arrive by bulk copies, each refilled as soon as all warps are done with it.
// Every operand of the recurrence is carried as a sum of two bf16 numbers (three MMAs per product, fp32 accumulation);
// the solve, the decays, the norms and the state are plain fp32.
#include "common/mma_sync.cuh"
#include "common/sm100.cuh"
#include "delta_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace delta {

using bf16 = __nv_bfloat16;
constexpr int CH = 64;         // tokens per chunk
constexpr int CONV_MAX = 4;    // taps the register window holds
constexpr int PREP_THREADS = 256;
constexpr int M_TILE = CH * CH * 2;
constexpr int M_IMAGE = 2 * M_TILE + CH * 4;  // hi, lo, decays from the chunk's start
constexpr int D_FLOATS = CH + 4;

// byte offset of element (row, col) in a tile of `width` bf16 columns: 16-byte pieces, XOR-swizzled for ldmatrix
__device__ __forceinline__ uint32_t tile_off(int row, int col, int width) {
  return row * width * 2 + (((col >> 3) ^ (row & 7)) << 4) + (col & 7) * 2;
}
__device__ __forceinline__ const uint8_t* piece(const uint8_t* tile, int row, int pc, int width) {
  return tile + row * width * 2 + ((pc ^ (row & 7)) << 4);
}

template <int DK, int DV>
struct PrepSmem {
  static constexpr int QK = CH * DK * 2;                // one tile of q or k
  static constexpr int Q_HI = 0, Q_LO = QK, K_HI = 2 * QK, K_LO = 3 * QK;
  static constexpr int V = 4 * QK;                      // fp32 (CH, DV)
  static constexpr int A = V + CH * DV * 4;             // fp32 (CH, CH)
  static constexpr int S = A + CH * CH * 4;             // beta, log-decay sums, -beta c
  static constexpr int TOTAL = S + 3 * CH * 4;
};

// The rows t0 - 3 .. t0 + 7 of N neighbouring channels, as they lie in the projections (rows outside the step: zero).
constexpr int CONV_ROWS = 8 + CONV_MAX - 1;
template <int N>
__device__ __forceinline__ void conv_load(const Params& p, const bf16* src, int t0, uint32_t (&raw)[CONV_ROWS][N / 2]) {
#pragma unroll
  for (int i = 0; i < CONV_ROWS; ++i) {
    const int t = t0 - (CONV_MAX - 1) + i;
    const bool in = t >= 0 && t < p.T;
    const bf16* s = src + (in ? t : 0) * p.ldp;
    if (N == 4) {
      const uint2 v = __ldg(reinterpret_cast<const uint2*>(s));
      raw[i][0] = in ? v.x : 0u;
      raw[i][N / 2 - 1] = in ? v.y : 0u;
    } else {
      const uint32_t v = __ldg(reinterpret_cast<const uint32_t*>(s));
      raw[i][0] = in ? v : 0u;
    }
  }
}

// silu(convolution) of those channels at the eight tokens t0 .. t0 + 7; fn(row, values). `c`: first channel in the ring's order.
template <int N, typename F>
__device__ __forceinline__ void conv_rows(const Params& p, const uint32_t (&raw)[CONV_ROWS][N / 2], const float* ring_b, int C,
                                          const bf16* w, int c, int t0, long long pos0, F fn) {
  float wt[CONV_MAX][N], win[CONV_MAX][N];
#pragma unroll
  for (int j = 0; j < CONV_MAX; ++j)
#pragma unroll
    for (int e = 0; e < N; ++e) {
      const int jj = j - (CONV_MAX - p.taps);
      wt[j][e] = jj >= 0 ? to_f(w[e * p.taps + jj]) : 0.f;
    }
  auto row = [&](int i, float (&x)[N]) {
#pragma unroll
    for (int e = 0; e < N; e += 2) {
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[i][e / 2]));
      x[e] = v.x;
      x[e + 1] = v.y;
    }
    const int t = t0 - (CONV_MAX - 1) + i;
    if (t < 0 && pos0 + t >= 0 && -t < p.taps) {  // the step's first tokens look at earlier steps
      const float* src = ring_b + static_cast<long long>(ring_slot(pos0 + t, p.taps)) * C + c;
#pragma unroll
      for (int e = 0; e < N; ++e) x[e] = src[e];
    }
  };
#pragma unroll
  for (int j = 1; j < CONV_MAX; ++j) row(j - 1, win[j]);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
#pragma unroll
    for (int j = 0; j + 1 < CONV_MAX; ++j)
#pragma unroll
      for (int e = 0; e < N; ++e) win[j][e] = win[j + 1][e];
    row(i + CONV_MAX - 1, win[CONV_MAX - 1]);
    float y[N];
#pragma unroll
    for (int e = 0; e < N; ++e) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < CONV_MAX; ++j) s = fmaf(wt[j][e], win[j][e], s);
      y[e] = t0 + i < p.T ? silu_fast(s) : 0.f;
    }
    fn(i, y);
  }
}

template <int DK, int DV>
__global__ void __launch_bounds__(PREP_THREADS, 2) delta_chunk_prep_kernel(const Params p) {
  using SM = PrepSmem<DK, DV>;
  extern __shared__ __align__(128) uint8_t smem[];
  float* sV = reinterpret_cast<float*>(smem + SM::V);
  float* sA = reinterpret_cast<float*>(smem + SM::A);
  float* sBeta = reinterpret_cast<float*>(smem + SM::S);
  float *sCs = sBeta + CH, *sBc = sCs + CH;
  const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z, rep = p.H / p.G, kvh = h / rep;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = chunk * CH;
  const long long pos0 = *p.pos;
  const int C = 2 * p.G * p.dk + p.H * p.dv;
  const bf16* proj_b = static_cast<const bf16*>(p.proj) + static_cast<long long>(b) * p.T * p.ldp;
  const float* ring_b = p.ring + static_cast<long long>(b) * p.taps * C;
  const long long bhc = (static_cast<long long>(b) * p.H + h) * p.n_chunks + chunk;
  uint8_t* g_qk = static_cast<uint8_t*>(p.ws_qk) + ((static_cast<long long>(b) * p.G + kvh) * p.n_chunks + chunk) * (4 * SM::QK);
  uint8_t* g_w = static_cast<uint8_t*>(p.ws_w) + bhc * (2 * SM::QK);
  float* g_u = p.ws_u + bhc * (DV * CH);
  uint8_t* g_m = static_cast<uint8_t*>(p.ws_m) + bhc * M_IMAGE;
  float* g_d = p.ws_d + bhc * D_FLOATS;

  // ---- step sizes and running sums of the log decays (padding tokens: no decay, no step)
  if (warp == 0) {
    float lg[2], be[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 2 * lane + i;
      lg[i] = 0.f;
      float& beta = be[i];
      beta = 0.f;
      if (t0 + t < p.T) {
        const float* ba = p.ba + (static_cast<long long>(b) * p.T + t0 + t) * p.ldba;
        lg[i] = log_decay(ba[p.off_a + h], to_f(static_cast<const bf16*>(p.a_log)[h]),
                          to_f(static_cast<const bf16*>(p.dt_bias)[h]));
        beta = sigmoid_f(ba[h]);
      }
      sBeta[t] = beta;
    }
    float s = lg[0] + lg[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += up;
    }
    const float last = __shfl_sync(0xffffffffu, s, 31);
    const float c0 = s - lg[1], c1 = s;
    sCs[2 * lane] = c0;
    sCs[2 * lane + 1] = c1;
    float* g_c = reinterpret_cast<float*>(g_m + 2 * M_TILE);
    const float e0 = expf(c0), e1 = expf(c1);
    g_c[2 * lane] = e0;
    g_c[2 * lane + 1] = e1;
    sBc[2 * lane] = -be[0] * e0;
    sBc[2 * lane + 1] = -be[1] * e1;
    g_d[2 * lane] = expf(last - c0);
    g_d[2 * lane + 1] = expf(last - c1);
    if (lane == 0) g_d[CH] = expf(last);
  }

  // ---- convolutions, silu, unit norms: a warp takes eight tokens, a lane DK / 32 channels
  {
    constexpr int N = DK / 32, NV = DV / 32;
    const bool write = h % rep == 0;
    const int tw = t0 + warp * 8, cq = kvh * DK + lane * N, cv = h * DV + lane * NV;
    uint32_t rq[CONV_ROWS][N / 2], rk[CONV_ROWS][N / 2], rv[CONV_ROWS][NV / 2];
    conv_load<N>(p, proj_b + p.off_q + cq, tw, rq);
    conv_load<N>(p, proj_b + p.off_k + cq, tw, rk);
    conv_load<NV>(p, proj_b + p.off_v + cv, tw, rv);
    auto unit_row = [&](int i, float (&y)[N], float mul, uint8_t* hi_tile, uint8_t* lo_tile) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < N; ++e) ss += y[e] * y[e];
      const float f = mul / sqrtf(sum_warp(ss) + 1e-6f);
      const uint32_t off = tile_off(warp * 8 + i, lane * N, DK);
      uint32_t hi[N / 2], lo[N / 2];
#pragma unroll
      for (int e = 0; e < N; e += 2) split_pack(y[e] * f, y[e + 1] * f, hi[e / 2], lo[e / 2]);
      if (N == 4) {
        *reinterpret_cast<uint2*>(hi_tile + off) = make_uint2(hi[0], hi[N / 2 - 1]);
        *reinterpret_cast<uint2*>(lo_tile + off) = make_uint2(lo[0], lo[N / 2 - 1]);
      } else {
        *reinterpret_cast<uint32_t*>(hi_tile + off) = hi[0];
        *reinterpret_cast<uint32_t*>(lo_tile + off) = lo[0];
      }
    };
    conv_rows<N>(p, rq, ring_b, C, static_cast<const bf16*>(p.conv_q) + static_cast<long long>(cq) * p.taps, cq, tw, pos0,
                 [&](int i, float (&y)[N]) { unit_row(i, y, p.q_scale, smem + SM::Q_HI, smem + SM::Q_LO); });
    conv_rows<N>(p, rk, ring_b, C, static_cast<const bf16*>(p.conv_k) + static_cast<long long>(cq) * p.taps, p.G * DK + cq, tw,
                 pos0, [&](int i, float (&y)[N]) { unit_row(i, y, 1.f, smem + SM::K_HI, smem + SM::K_LO); });
    conv_rows<NV>(p, rv, ring_b, C, static_cast<const bf16*>(p.conv_v) + static_cast<long long>(cv) * p.taps,
                  2 * p.G * DK + cv, tw, pos0, [&](int i, float (&y)[NV]) {
                    float* dst = sV + (warp * 8 + i) * DV + lane * NV;
                    if (NV == 4) store4(dst, make_float4(y[0], y[1], y[2 % NV], y[3 % NV]));
                    else *reinterpret_cast<float2*>(dst) = make_float2(y[0], y[1]);
                  });
    __syncthreads();
    if (write) {  // the four tiles are contiguous and already have the image's layout
      const uint4* src = reinterpret_cast<const uint4*>(smem);
      uint4* dst = reinterpret_cast<uint4*>(g_qk);
      for (int i = tid; i < 4 * SM::QK / 16; i += PREP_THREADS)
        if (RA_IN_BOUNDS(chunk, 1, p.n_chunks, kTagDeltaWork)) dst[i] = src[i];
    }
  }

  // ---- K K^T (warps 0-3) and Q K^T (warps 4-7), 16 rows per warp, columns up to the diagonal block
  {
    const int mt = warp & 3;
    const bool is_m = warp >= 4;
    const uint8_t *a_hi = smem + (is_m ? SM::Q_HI : SM::K_HI), *a_lo = smem + (is_m ? SM::Q_LO : SM::K_LO);
    const uint8_t *b_hi = smem + SM::K_HI, *b_lo = smem + SM::K_LO;
    const int mat = lane >> 3, rr = lane & 7, g = lane >> 2, t = lane & 3;
    float acc[4][2][4];
#pragma unroll
    for (int np = 0; np < 4; ++np)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[np][n][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t ah[4], al[4];
      const int ar = mt * 16 + (mat & 1) * 8 + rr, ap = 2 * ks + (mat >> 1);
      ldmatrix_x4(ah, piece(a_hi, ar, ap, DK));
      ldmatrix_x4(al, piece(a_lo, ar, ap, DK));
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (np > mt) continue;
        uint32_t bh[1][4], bl[1][4];
        const int br = np * 16 + (mat >> 1) * 8 + rr, bp = 2 * ks + (mat & 1);
        ldmatrix_x4(bh[0], piece(b_hi, br, bp, DK));
        ldmatrix_x4(bl[0], piece(b_lo, br, bp, DK));
        float(*const d[2])[4] = {&acc[np][0], &acc[np][1]};
        mma_split<1>(d, ah, al, bh, bl);
      }
    }
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (np > mt) continue;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int i = mt * 16 + g + 8 * r, j = np * 16 + n * 8 + 2 * t;
          const float ci = sCs[i];
          // j > i: the exponent would be positive without bound; the entry is zero there
          const float f0 = j <= i ? expf(ci - sCs[j]) : 0.f, f1 = j + 1 <= i ? expf(ci - sCs[j + 1]) : 0.f;
          const float x0 = acc[np][n][2 * r] * f0, x1 = acc[np][n][2 * r + 1] * f1;
          if (is_m) {
            uint32_t hi, lo;
            split_pack(x0, x1, hi, lo);
            *reinterpret_cast<uint32_t*>(g_m + tile_off(i, j, CH)) = hi;
            *reinterpret_cast<uint32_t*>(g_m + M_TILE + tile_off(i, j, CH)) = lo;
          } else {
            const float be = sBeta[i];
            sA[i * CH + j] = j < i ? be * x0 : 0.f;
            sA[i * CH + j + 1] = j + 1 < i ? be * x1 : 0.f;
          }
        }
    }
  }
  __syncthreads();

  // ---- (I + A) X = right-hand sides, one column per thread: columns of -diag(beta c) K, then of diag(beta) V
  if (tid < DK + DV) {
    const bool is_w = tid < DK;
    const int col = is_w ? tid : tid - DK;
    float x[CH];
    if (is_w) {
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const uint32_t off = tile_off(i, col, DK);
        x[i] = sBc[i] * (to_f(*reinterpret_cast<const bf16*>(smem + SM::K_HI + off)) +
                         to_f(*reinterpret_cast<const bf16*>(smem + SM::K_LO + off)));
      }
    } else {
#pragma unroll
      for (int i = 0; i < CH; ++i) x[i] = sBeta[i] * sV[i * DV + col];
    }
#pragma unroll
    for (int i = 1; i < CH; ++i) {
      float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        const float4 a = *reinterpret_cast<const float4*>(sA + i * CH + j);  // entries from the diagonal on are zero
        s0 = fmaf(a.x, x[j], s0);
        if (j + 1 < i) s1 = fmaf(a.y, x[j + 1], s1);
        if (j + 2 < i) s2 = fmaf(a.z, x[j + 2], s2);
        if (j + 3 < i) s3 = fmaf(a.w, x[j + 3], s3);
      }
      x[i] -= (s0 + s1) + (s2 + s3);
    }
    if (is_w) {
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        bf16 hi, lo;
        split_bf16(x[i], hi, lo);
        *reinterpret_cast<bf16*>(g_w + tile_off(i, col, DK)) = hi;
        *reinterpret_cast<bf16*>(g_w + SM::QK + tile_off(i, col, DK)) = lo;
      }
    } else {
#pragma unroll
      for (int i = 0; i < CH; i += 4)
        store4(g_u + col * CH + i, make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]));
    }
  }
}

template <int DK>
struct ScanSmem {
  static constexpr int T = CH * DK * 2;
  static constexpr int W = 0, Q = 2 * T, K = 4 * T, M = 6 * T;
  static constexpr int D = M + M_IMAGE;
  static constexpr int BAR = D + D_FLOATS * 4;
  static constexpr int TOTAL = BAR + 64;
};

template <int DK, int NW>
__global__ void __launch_bounds__(NW * 32) delta_chunk_scan_kernel(const Params p) {
  using SM = ScanSmem<DK>;
  constexpr int NS = DK / 8;      // column tiles of S^T
  extern __shared__ __align__(128) uint8_t smem[];
  uint64_t* bar_wq = reinterpret_cast<uint64_t*>(smem + SM::BAR);
  uint64_t *bar_m = bar_wq + 1, *bar_k = bar_wq + 2;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bar_wq + 3);
  const WaitCtx wc{abort_flag, p.status};
  const int h = blockIdx.y, b = blockIdx.z, kvh = h / (p.H / p.G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int mat = lane >> 3, rr = lane & 7;
  const int v0 = (blockIdx.x * NW + warp) * 16;  // the grid covers dv exactly
  const int n = p.n_chunks;
  const long long bh = static_cast<long long>(b) * p.H + h;
  const uint8_t* g_qk = static_cast<const uint8_t*>(p.ws_qk) + (static_cast<long long>(b) * p.G + kvh) * n * (4 * SM::T);
  const uint8_t* g_w = static_cast<const uint8_t*>(p.ws_w) + bh * n * (2 * SM::T);
  const uint8_t* g_m = static_cast<const uint8_t*>(p.ws_m) + bh * n * M_IMAGE;
  const float* g_d = p.ws_d + bh * n * D_FLOATS;
  const float* g_u = p.ws_u + bh * n * static_cast<long long>(p.dv) * CH;

  if (tid == 0) {
    mbar_init(bar_wq, 1);
    mbar_init(bar_m, 1);
    mbar_init(bar_k, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  __syncthreads();
  auto fill_wq = [&](int c) {
    mbar_arrive_expect_tx(bar_wq, 4 * SM::T);
    bulk_load(smem + SM::W, g_w + static_cast<long long>(c) * (2 * SM::T), 2 * SM::T, bar_wq);
    bulk_load(smem + SM::Q, g_qk + static_cast<long long>(c) * (4 * SM::T), 2 * SM::T, bar_wq);
  };
  auto fill_m = [&](int c) {
    mbar_arrive_expect_tx(bar_m, M_IMAGE);
    bulk_load(smem + SM::M, g_m + static_cast<long long>(c) * M_IMAGE, M_IMAGE, bar_m);
  };
  auto fill_k = [&](int c) {
    mbar_arrive_expect_tx(bar_k, 2 * SM::T + D_FLOATS * 4);
    bulk_load(smem + SM::K, g_qk + static_cast<long long>(c) * (4 * SM::T) + 2 * SM::T, 2 * SM::T, bar_k);
    bulk_load(smem + SM::D, g_d + static_cast<long long>(c) * D_FLOATS, D_FLOATS * 4, bar_k);
  };
  if (tid == 0) {
    fill_wq(0);
    fill_m(0);
    fill_k(0);
  }
  save_ring<bf16>(p, b, *p.pos, (blockIdx.y * gridDim.x + blockIdx.x) * (NW * 32) + tid, gridDim.x * gridDim.y * NW * 32);

  float S[NS][4];
  float* st = p.state + (bh * p.dv + v0) * DK;
#pragma unroll
  for (int j = 0; j < NS; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const float2 x = *reinterpret_cast<const float2*>(st + (g + 8 * r) * DK + 8 * j + 2 * t);
      S[j][2 * r] = x.x;
      S[j][2 * r + 1] = x.y;
    }
  bool ok = true;
  for (int c = 0; c < n; ++c) {
    float U[8][4], O[8][4];
    const float* uc = g_u + (static_cast<long long>(c) * p.dv + v0) * CH;
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float2 x = *reinterpret_cast<const float2*>(uc + (g + 8 * r) * CH + 8 * j + 2 * t);
        U[j][2 * r] = x.x;
        U[j][2 * r + 1] = x.y;
        O[j][2 * r] = O[j][2 * r + 1] = 0.f;
      }
    ok = mbar_wait(bar_wq, c & 1, wc, kTimeoutSmemFull) && ok;
    // ---- U^T = U0^T + S^T (-W)^T and O^T = S^T Q^T
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t ah[4], al[4];
      split_a_frag(S[2 * ks], S[2 * ks + 1], ah, al);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        const int row = np * 16 + (mat >> 1) * 8 + rr, pc = 2 * ks + (mat & 1);
        uint32_t bhi[2][4], blo[2][4];
        ldmatrix_x4(bhi[0], piece(smem + SM::W, row, pc, DK));
        ldmatrix_x4(blo[0], piece(smem + SM::W + SM::T, row, pc, DK));
        ldmatrix_x4(bhi[1], piece(smem + SM::Q, row, pc, DK));
        ldmatrix_x4(blo[1], piece(smem + SM::Q + SM::T, row, pc, DK));
        float(*const d[4])[4] = {&U[2 * np], &U[2 * np + 1], &O[2 * np], &O[2 * np + 1]};
        mma_split<2>(d, ah, al, bhi, blo);
      }
    }
    ok = __syncthreads_and(ok);
    if (!ok) break;
    if (tid == 0 && c + 1 < n) fill_wq(c + 1);
    // ---- O^T = O^T diag(c) + U^T M^T
    ok = mbar_wait(bar_m, c & 1, wc, kTimeoutSmemFull);
    const float* sc = reinterpret_cast<const float*>(smem + SM::M + 2 * M_TILE);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float2 f = *reinterpret_cast<const float2*>(sc + 8 * j + 2 * t);
      O[j][0] *= f.x;
      O[j][1] *= f.y;
      O[j][2] *= f.x;
      O[j][3] *= f.y;
    }
#pragma unroll
    for (int ks = 0; ks < CH / 16; ++ks) {
      uint32_t ah[4], al[4];
      split_a_frag(U[2 * ks], U[2 * ks + 1], ah, al);
#pragma unroll
      for (int np = ks; np < 4; ++np) {  // tokens before this block of writes do not see it
        const int row = np * 16 + (mat >> 1) * 8 + rr, pc = 2 * ks + (mat & 1);
        uint32_t bhi[1][4], blo[1][4];
        ldmatrix_x4(bhi[0], piece(smem + SM::M, row, pc, CH));
        ldmatrix_x4(blo[0], piece(smem + SM::M + M_TILE, row, pc, CH));
        float(*const d[2])[4] = {&O[2 * np], &O[2 * np + 1]};
        mma_split<1>(d, ah, al, bhi, blo);
      }
    }
    ok = __syncthreads_and(ok);
    if (!ok) break;
    if (tid == 0 && c + 1 < n) fill_m(c + 1);
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int tok = c * CH + 8 * j + 2 * t + e;
        if (tok < p.T && RA_IN_BOUNDS(v0 + g + 8, 1, p.dv, kTagDelta)) {
          float* dst = p.o + ((static_cast<long long>(b) * p.T + tok) * p.H + h) * p.dv + v0 + g;
          dst[0] = O[j][e];
          dst[8] = O[j][2 + e];
        }
      }
    // ---- S^T = c_64 S^T + (U^T diag(c_64 / c)) K
    ok = mbar_wait(bar_k, c & 1, wc, kTimeoutSmemFull);
    const float* sd = reinterpret_cast<const float*>(smem + SM::D);
    const float cend = sd[CH];
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[j][e] *= cend;
#pragma unroll
    for (int ks = 0; ks < CH / 16; ++ks) {
#pragma unroll
      for (int j = 2 * ks; j < 2 * ks + 2; ++j) {
        const float2 f = *reinterpret_cast<const float2*>(sd + 8 * j + 2 * t);
        U[j][0] *= f.x;
        U[j][1] *= f.y;
        U[j][2] *= f.x;
        U[j][3] *= f.y;
      }
      uint32_t ah[4], al[4];
      split_a_frag(U[2 * ks], U[2 * ks + 1], ah, al);
#pragma unroll
      for (int np = 0; np < NS / 2; np += 2) {
        const int row = ks * 16 + (mat & 1) * 8 + rr, pc = 2 * np + (mat >> 1);
        uint32_t bhi[2][4], blo[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          ldmatrix_x4_trans(bhi[i], piece(smem + SM::K, row, pc + 2 * i, DK));
          ldmatrix_x4_trans(blo[i], piece(smem + SM::K + SM::T, row, pc + 2 * i, DK));
        }
        float(*const d[4])[4] = {&S[2 * np], &S[2 * np + 1], &S[2 * np + 2], &S[2 * np + 3]};
        mma_split<2>(d, ah, al, bhi, blo);
      }
    }
    ok = __syncthreads_and(ok);
    if (!ok) break;
    if (tid == 0 && c + 1 < n) fill_k(c + 1);
  }
  if (!ok) bounded_drain_pause();  // copies in flight land before the CTA ends
#pragma unroll
  for (int j = 0; j < NS; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float2*>(st + (g + 8 * r) * DK + 8 * j + 2 * t) = make_float2(S[j][2 * r], S[j][2 * r + 1]);
}

template <int DK, int DV>
int launch_chunk_prep(const Params& p, cudaStream_t s) {
  constexpr int smem = PrepSmem<DK, DV>::TOTAL;
  if (cudaFuncSetAttribute(delta_chunk_prep_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) {
    set_error("delta_chunk_prep: shared memory");
    return kHostLaunchFail;
  }
  delta_chunk_prep_kernel<DK, DV><<<dim3(p.n_chunks, p.H, p.B), PREP_THREADS, smem, s>>>(p);
  return check_launch("delta_chunk_prep_kernel");
}

template <int DK, int NW>
int launch_chunk_scan(const Params& p, cudaStream_t s) {
  constexpr int smem = ScanSmem<DK>::TOTAL;
  if (cudaFuncSetAttribute(delta_chunk_scan_kernel<DK, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) {
    set_error("delta_chunk_scan: shared memory");
    return kHostLaunchFail;
  }
  delta_chunk_scan_kernel<DK, NW><<<dim3(p.dv / (16 * NW), p.H, p.B), NW * 32, smem, s>>>(p);
  return check_launch("delta_chunk_scan_kernel");
}

int check_chunk(const Params* p) {
  const int rc = check(p);
  if (rc) return rc;
  if ((p->dk != 64 && p->dk != 128) || (p->dv != 64 && p->dv != 128) || p->taps > CONV_MAX || p->n_chunks != (p->T + CH - 1) / CH ||
      p->ldp % 4 || (p->off_q | p->off_k | p->off_v) % 4 || (reinterpret_cast<uintptr_t>(p->proj) & 15) || !p->ws_qk ||
      !p->ws_w || !p->ws_u || !p->ws_m || !p->ws_d) {
    set_error("ra_delta_chunk: key and value dims 64 or 128, at most 4 taps");
    return kHostBadArg;
  }
  return kHostOk;
}

}  // namespace delta
}  // namespace ra

// bf16 only. The two launches replace ra_delta_prep and ra_delta_scan; ra_delta_out follows as there.
extern "C" int ra_delta_chunk_prep(const ra::delta::Params* p, int, void* stream) {
  using namespace ra::delta;
  const int rc = check_chunk(p);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (p->dk == 128) return p->dv == 128 ? launch_chunk_prep<128, 128>(*p, s) : launch_chunk_prep<128, 64>(*p, s);
  return p->dv == 128 ? launch_chunk_prep<64, 128>(*p, s) : launch_chunk_prep<64, 64>(*p, s);
}

extern "C" int ra_delta_chunk_scan(const ra::delta::Params* p, int, void* stream) {
  using namespace ra::delta;
  const int rc = check_chunk(p);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int w = p->B * p->H * p->dv / 16;  // warps in all: few of them are spread over the SMs, many share tiles
  if (p->dk == 128)
    return w <= ra::sm_count() ? launch_chunk_scan<128, 1>(*p, s)
                               : (w <= 2 * ra::sm_count() ? launch_chunk_scan<128, 2>(*p, s) : launch_chunk_scan<128, 4>(*p, s));
  return w <= ra::sm_count() ? launch_chunk_scan<64, 1>(*p, s)
                             : (w <= 2 * ra::sm_count() ? launch_chunk_scan<64, 2>(*p, s) : launch_chunk_scan<64, 4>(*p, s));
}
