// Warp-level tensor-core products (mma.sync m16n8k16, bf16 operands, fp32 accumulation), their ldmatrix operand loads and
// per-thread asynchronous copies: for kernels that are bound by memory or by a serial chain, where a 128-row tcgen05 tile
// would not fill.
//   A (16 x 16): a0 row g, k 2t..; a1 row g + 8; a2 row g, k 8 + 2t..; a3 row g + 8, k 8 + 2t..   (g = lane / 4, t = lane % 4)
//   B (16 x 8) : b0 k 2t.., column g; b1 k 8 + 2t..
//   C (16 x 8) : c0, c1 row g, columns 2t, 2t + 1; c2, c3 row g + 8
// The C fragments of two neighbouring column tiles are the A fragment of the product that consumes them.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace ra {

// 16-byte asynchronous copy global -> shared; `bytes` = 0 writes zeros without reading the source.
__device__ __forceinline__ void cp_async16(void* smem_dst, const void* gsrc, int bytes) {
  const uint32_t d = static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst));
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(gsrc), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
  const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(a));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem_row) {
  const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(a));
}
// d += a * b for m16n8k16, bf16 inputs, fp32 accumulation; rows 8..15 of a are zero (a1 = a3 = 0)
__device__ __forceinline__ void mma_16816_top(float (&d)[4], uint32_t a0, uint32_t a2, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(0u), "r"(a2), "r"(0u), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// ---- fp32 operands as sums of two bf16 numbers: x = hi + lo up to 2^-17 |x|. A product of two such operands without the
// lo * lo term is three MMAs and is exact to about 2^-16 of its terms, with fp32 accumulation.
__device__ __forceinline__ void split_bf16(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(x);
  lo = __float2bfloat16(x - __bfloat162float(hi));
}
__device__ __forceinline__ void split_pack(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
// A fragment (hi and lo) of accumulator tiles c and d (columns 0-7 and 8-15 of the k range)
__device__ __forceinline__ void split_a_frag(const float (&c)[4], const float (&d)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  split_pack(c[0], c[1], hi[0], lo[0]);
  split_pack(c[2], c[3], hi[1], lo[1]);
  split_pack(d[0], d[1], hi[2], lo[2]);
  split_pack(d[2], d[3], hi[3], lo[3]);
}
// Two column tiles (b[0..1] and b[2..3], as ldmatrix.x4 delivers them) of each of N products that share the A fragment:
// d[2 i], d[2 i + 1] += A B_i. The three terms run over all tiles in turn, so that no MMA waits for the one before it.
template <int N>
__device__ __forceinline__ void mma_split(float (*const (&d)[2 * N])[4], const uint32_t (&ah)[4], const uint32_t (&al)[4],
                                          const uint32_t (&bh)[N][4], const uint32_t (&bl)[N][4]) {
#pragma unroll
  for (int i = 0; i < 2 * N; ++i) mma_16816(*d[i], ah, bh[i >> 1][2 * (i & 1)], bh[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
  for (int i = 0; i < 2 * N; ++i) mma_16816(*d[i], ah, bl[i >> 1][2 * (i & 1)], bl[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
  for (int i = 0; i < 2 * N; ++i) mma_16816(*d[i], al, bh[i >> 1][2 * (i & 1)], bh[i >> 1][2 * (i & 1) + 1]);
}

}  // namespace ra
