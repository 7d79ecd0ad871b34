// Matrix products of routed experts for many rows: a persistent tcgen05 GEMM over the row tiles of all experts.
//   UP   : act[128 tile + i] = silu(w g) * (w u) with g, u = the gate and up products of the token of the tile's i-th entry
//          and w = its score. Four warps gather the tokens' rows with cp.async straight into the swizzled tile (a TMA gather
//          of four rows a copy ran at a third of this speed), so no sorted copy of the input is made.
//   DOWN : y[entry] = W_down act[128 tile + i]; tiles of act are plain TMA boxes, the rows are scattered by the list.
// Row tiles are numbered expert after expert; column tiles of one row tile run first. Each CTA finds its tiles from the
// experts' counts, which it sums up itself. Pipeline and accumulators as in gemm_kernel.cuh: 128 x 256 x 64 tiles, four
// stages, two accumulators; a gate/up tile is 128 gate columns and the 128 matching up columns.
#include "common/mma_sync.cuh"
#include "common/sm100.cuh"
#include "moe_common.cuh"

RA_BOUNDS_TRANSLATION_UNIT()

namespace ra {
namespace moe {

constexpr int BM = 128, BN = 256, BK = 64, STAGES = 4, NUM_ACC = 2, GATHER = 128;
constexpr int GEMM_THREADS = 192;      // TMA, MMA and four epilogue warps; UP has GATHER threads more
constexpr int IN_FLIGHT = 2;           // stages of gathered rows on their way per thread
constexpr int A_BYTES = BM * BK * 2, B_BYTES = BN * BK * 2;
constexpr int GEMM_SMEM = STAGES * (A_BYTES + B_BYTES) + 1024 + 256 + MAX_EXPERTS * 4 + 16;

// Walks a CTA's tiles; every role keeps its own.
struct TileWalk {
  int e, first;  // current expert and its first row tile
  __device__ __forceinline__ bool find(const int* tile_end, int E, int mt) {
    while (e < E && mt >= tile_end[e]) {
      first = tile_end[e];
      ++e;
    }
    return e < E;
  }
};

// Rows of act: every expert may leave its last row tile partly empty.
__host__ __device__ __forceinline__ long long act_rows(const Params& p) {
  const long long n = static_cast<long long>(p.rows) * p.top;
  return BM * (n / BM + (n < p.E ? n : p.E));
}

template <bool UP>
__global__ void __launch_bounds__(GEMM_THREADS + (UP ? GATHER : 0), 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap tma_a, const __grid_constant__ CUtensorMap tma_b, const Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t* sA = smem;
  uint8_t* sB = smem + STAGES * A_BYTES;
  uint64_t* full = reinterpret_cast<uint64_t*>(sB + STAGES * B_BYTES);
  uint64_t* empty = full + STAGES;
  uint64_t* tfull = empty + STAGES;
  uint64_t* tempty = tfull + NUM_ACC;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tempty + NUM_ACC);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* tile_end = reinterpret_cast<int*>(reinterpret_cast<uint8_t*>(full) + 256);  // [E] row tiles up to and with expert e

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const WaitCtx wc{abort_flag, p.status};
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&full[s], UP ? 1 + GATHER : 1);
      mbar_init(&empty[s], 1);
    }
    for (int a = 0; a < NUM_ACC; ++a) {
      mbar_init(&tfull[a], 1);
      mbar_init(&tempty[a], 128);
    }
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tma_a);
    tma_prefetch_desc(&tma_b);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  if (warp == 2) {  // running sums of the experts' row tiles, 32 experts at a time
    int carry = 0;
    for (int e0 = 0; e0 < p.E; e0 += 32) {
      int v = e0 + lane < p.E ? (min(p.count[e0 + lane], p.rows) + BM - 1) / BM : 0;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += u;
      }
      if (e0 + lane < p.E) tile_end[e0 + lane] = carry + v;
      carry += __shfl_sync(0xffffffffu, v, 31);
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  const int K = UP ? p.dp : p.F, N = UP ? p.F : p.dp;      // N: output columns
  const int per_tile = UP ? BN / 2 : BN;
  const int tiles_n = (N + per_tile - 1) / per_tile, num_kb = (K + BK - 1) / BK;
  const int num_tiles = tile_end[p.E - 1] * tiles_n;
  TileWalk walk{0, 0};

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer (warp-uniform flow)
    const bool leader = elect_one();
    int stage = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
      const int mt = tile / tiles_n, tn = tile - mt * tiles_n;
      if (!walk.find(tile_end, p.E, mt)) break;
      const int row = UP ? walk.e * 2 * p.F + tn * (BN / 2) : walk.e * p.dp + tn * BN;
      for (int kb = 0; kb < num_kb; ++kb) {
        const int k0 = kb * BK;
        if (!mbar_wait(&empty[stage], phase ^ 1u, wc, kTimeoutSmemEmpty)) {
          ok = false;
          break;
        }
        uint8_t* b_dst = sB + stage * B_BYTES;
        if (leader) {
          mbar_arrive_expect_tx(&full[stage], B_BYTES + (UP ? 0 : A_BYTES));
          if (UP) {
            tma_load_2d(b_dst, &tma_b, &full[stage], k0, row);
            tma_load_2d(b_dst + B_BYTES / 2, &tma_b, &full[stage], k0, row + p.F);
          } else {
            tma_load_2d(sA + stage * A_BYTES, &tma_a, &full[stage], k0, mt * BM);
            tma_load_2d(b_dst, &tma_b, &full[stage], k0, row);
          }
        }
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1u;
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer (warp-uniform flow)
    const bool leader = elect_one();
    constexpr uint32_t idesc = make_idesc_bf16(BM, BN, 0, 0);
    int stage = 0, acc = 0;
    uint32_t phase = 0, acc_phase = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
      if (!mbar_wait(&tempty[acc], acc_phase ^ 1u, wc, kTimeoutTmemEmpty)) break;
      tc_fence_after();
      const uint32_t d_tmem = tmem_base + static_cast<uint32_t>(acc * BN);
      for (int kb = 0; kb < num_kb; ++kb) {
        if (!mbar_wait(&full[stage], phase, wc, kTimeoutSmemFull)) {
          ok = false;
          break;
        }
        tc_fence_after();
        const uint32_t a_addr = smem_u32(sA + stage * A_BYTES), b_addr = smem_u32(sB + stage * B_BYTES);
#pragma unroll
        for (int kk = 0; kk < BK / 16; ++kk) {
          const uint64_t adesc = make_smem_desc(a_addr + kk * 32, 16, 1024);
          const uint64_t bdesc = make_smem_desc(b_addr + kk * 32, 16, 1024);
          if (leader) umma_ss(d_tmem, adesc, bdesc, idesc, (kb | kk) != 0 ? 1u : 0u);
        }
        if (leader) umma_commit(&empty[stage]);
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1u;
        }
      }
      if (!ok) break;
      if (leader) umma_commit(&tfull[acc]);
      if (++acc == NUM_ACC) {
        acc = 0;
        acc_phase ^= 1u;
      }
    }
    __syncwarp();
  } else if (UP && warp >= 6) {
    // ------------------------------------------------------------------ gather (4 warps)
    // Thread t copies 16-byte piece t % 8 of rows t / 8 + 16 j. A stage is handed over when its copies have landed, which
    // is known IN_FLIGHT stages later; the fence makes them visible to the tensor core.
    const int t = threadIdx.x - GEMM_THREADS, piece = t & 7, r0 = t >> 3;
    int stage = 0, issued = 0;
    uint32_t phase = 0;
    bool ok = true;
    const __nv_bfloat16* h = static_cast<const __nv_bfloat16*>(p.h);
    for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
      const int mt = tile / tiles_n;
      if (!walk.find(tile_end, p.E, mt)) break;
      const int cnt = min(p.count[walk.e], p.rows), m0 = (mt - walk.first) * BM;
      const int* list = p.list + static_cast<long long>(walk.e) * p.rows;
      const __nv_bfloat16* src[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {  // rows past the end repeat the last one; their outputs are not stored
        const int token = list[min(m0 + r0 + 16 * j, cnt - 1)] / p.top;
        src[j] = h + static_cast<long long>(min(max(token, 0), p.rows - 1)) * p.dp + piece * 8;
      }
      for (int kb = 0; kb < num_kb; ++kb) {
        const int k0 = kb * BK;
        if (!mbar_wait(&empty[stage], phase ^ 1u, wc, kTimeoutSmemEmpty)) {
          ok = false;
          break;
        }
        const bool in = k0 + piece * 8 < K;
        uint8_t* dst = sA + stage * A_BYTES + r0 * 128 + ((piece ^ (r0 & 7)) << 4);
#pragma unroll
        for (int j = 0; j < 8; ++j) cp_async16(dst + j * 16 * 128, src[j] + (in ? k0 : -piece * 8), in ? 16 : 0);
        cp_async_commit();
        if (++issued > IN_FLIGHT) {
          cp_async_wait<IN_FLIGHT>();
          fence_proxy_async_smem();
          mbar_arrive(&full[(stage + STAGES - IN_FLIGHT) % STAGES]);
        }
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1u;
        }
      }
    }
    cp_async_wait<0>();
    fence_proxy_async_smem();
    if (ok)
      for (int i = min(issued, IN_FLIGHT); i > 0; --i) mbar_arrive(&full[(stage + STAGES - i) % STAGES]);
  } else {
    // ------------------------------------------------------------------ epilogue (4 warps)
    const int quad = warp & 3;
    int acc = 0;
    uint32_t acc_phase = 0;
    for (int tile = blockIdx.x; tile < num_tiles; tile += gridDim.x) {
      const int mt = tile / tiles_n, tn = tile - mt * tiles_n;
      if (!walk.find(tile_end, p.E, mt)) break;
      const int cnt = min(p.count[walk.e], p.rows), i = (mt - walk.first) * BM + quad * 32 + lane;
      const bool valid = i < cnt;
      const int entry = valid ? p.list[static_cast<long long>(walk.e) * p.rows + i] : 0;
      const float w = UP && valid ? p.weight[entry] : 0.f;
      const long long out_row = UP ? static_cast<long long>(mt) * BM + quad * 32 + lane : entry;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(UP ? p.act : p.y) + out_row * N;
      const bool store = valid && RA_IN_BOUNDS(out_row, 1, UP ? act_rows(p) : static_cast<long long>(p.rows) * p.top, kTagMoe);
      if (!mbar_wait(&tfull[acc], acc_phase, wc, kTimeoutTmemFull)) break;
      tc_fence_after();
      const uint32_t t_row = tmem_base + (static_cast<uint32_t>(quad * 32) << 16) + static_cast<uint32_t>(acc * BN);
#pragma unroll 1
      for (int c = 0; c < per_tile / 32; ++c) {
        uint32_t r[32], ru[32];
        tmem_ld_x32(t_row + c * 32, r);
        if (UP) tmem_ld_x32(t_row + BN / 2 + c * 32, ru);
        tmem_ld_wait();
        const int col0 = tn * per_tile + c * 32;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (!store || col0 + j * 8 >= N) continue;
          float f[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            f[e] = __uint_as_float(r[8 * j + e]);
            if (UP) {
              const float g = f[e] * w;
              f[e] = __fdividef(g, 1.f + __expf(-g)) * (__uint_as_float(ru[8 * j + e]) * w);
            }
          }
          uint4 v;
          v.x = pack_bf16x2(f[0], f[1]);
          v.y = pack_bf16x2(f[2], f[3]);
          v.z = pack_bf16x2(f[4], f[5]);
          v.w = pack_bf16x2(f[6], f[7]);
          *reinterpret_cast<uint4*>(dst + col0 + 8 * j) = v;
        }
      }
      tc_fence_before();
      mbar_arrive(&tempty[acc]);
      if (++acc == NUM_ACC) {
        acc = 0;
        acc_phase ^= 1u;
      }
    }
  }
  // ------------------------------------------------------------------ teardown
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) bounded_drain_pause();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <bool UP>
int launch_gemm(const Params& p, cudaStream_t s) {
  const long long K = UP ? p.dp : p.F, a_rows = UP ? p.rows : act_rows(p);
  const long long b_rows = static_cast<long long>(p.E) * (UP ? 2 * p.F : p.dp);
  const void *A = UP ? p.h : p.act, *B = UP ? p.gu : p.down;
  if (b_rows > (1ll << 31) - 1 || a_rows > (1ll << 31) - 1 ||
      ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(B) | reinterpret_cast<uintptr_t>(p.y) |
        reinterpret_cast<uintptr_t>(p.act)) & 15)) {
    set_error("moe_gemm: too many rows or bad alignment");
    return kHostBadArg;
  }
  CUtensorMap ta, tb;
  uint64_t dims[2] = {static_cast<uint64_t>(K), static_cast<uint64_t>(a_rows)}, str[1] = {static_cast<uint64_t>(K) * 2};
  uint32_t box[2] = {BK, BM};
  if (int rc = make_tmap_bf16_sw128(&ta, A, 2, dims, str, box)) return rc;
  dims[1] = static_cast<uint64_t>(b_rows);
  box[1] = UP ? BN / 2 : BN;
  if (int rc = make_tmap_bf16_sw128(&tb, B, 2, dims, str, box)) return rc;
  auto kern = moe_gemm_kernel<UP>;
  if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, GEMM_SMEM) != cudaSuccess) {
    cudaGetLastError();
    set_error("moe_gemm: smem attribute");
    return kHostLaunchFail;
  }
  kern<<<sm_count(), GEMM_THREADS + (UP ? GATHER : 0), GEMM_SMEM, s>>>(ta, tb, p);
  return check_launch("moe_gemm_kernel");
}

}  // namespace moe
}  // namespace ra

// After ra_moe_route: act (act_rows, F) by row tile and y (rows * top, dp) by entry, bf16. Two launches.
extern "C" int ra_moe_gemm(const ra::moe::Params* p, void* stream) {
  using namespace ra;
  if (const int rc = moe::check(p)) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (int rc = moe::launch_gemm<true>(*p, s)) return rc;
  return moe::launch_gemm<false>(*p, s);
}

