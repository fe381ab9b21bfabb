// Warp-level bf16 matrix products (m16n8k16) over swizzled shared-memory tiles, for kernels whose tiles are too
// small or too irregular for tensor memory: attention over a window, chunked linear attention.
//
// A tile is rows of W bf16 (W = 64 or 128) stored as 16-byte pieces; piece p of row r lies at position p ^ (r & 7),
// so that ldmatrix reads eight rows without bank conflicts.
#pragma once

#include "b2_common.cuh"

namespace b2 {

template <int W>
__device__ __forceinline__ uint32_t tile_addr(uint32_t base, int row, int piece) {
  return base + static_cast<uint32_t>(row) * (W * 2) + (static_cast<uint32_t>(piece ^ (row & 7)) << 4);
}
// 16 bytes global -> shared; zeros when !valid (the source is then not read)
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// A operand rows row0 .. row0+15, columns k0 .. k0+15 of a tile stored [row][k]
template <int W>
__device__ __forceinline__ void frag_a(uint32_t base, int row0, int k0, int lane, uint32_t (&r)[4]) {
  ldsm_x4(tile_addr<W>(base, row0 + (lane & 15), (k0 >> 3) + (lane >> 4)), r);
}
// A operand of a tile stored transposed, [k][row]
template <int W>
__device__ __forceinline__ void frag_a_t(uint32_t base, int row0, int k0, int lane, uint32_t (&r)[4]) {
  ldsm_x4_t(tile_addr<W>(base, k0 + (lane & 7) + ((lane >> 4) << 3), (row0 >> 3) + ((lane >> 3) & 1)), r);
}
// B operands of two 8-column tiles (columns n0 .. n0+15, k0 .. k0+15) of a tile stored [n][k]: r[0..1], r[2..3]
template <int W>
__device__ __forceinline__ void frag_b(uint32_t base, int n0, int k0, int lane, uint32_t (&r)[4]) {
  ldsm_x4(tile_addr<W>(base, n0 + (lane & 7) + ((lane >> 4) << 3), (k0 >> 3) + ((lane >> 3) & 1)), r);
}
// the same for a tile stored [k][n]
template <int W>
__device__ __forceinline__ void frag_b_t(uint32_t base, int n0, int k0, int lane, uint32_t (&r)[4]) {
  ldsm_x4_t(tile_addr<W>(base, k0 + (lane & 15), (n0 >> 3) + (lane >> 4)), r);
}
// d (16 x 8 fp32) += a (16 x 16) b (16 x 8)
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// an fp32 pair as a sum of two bf16 pairs (16 significant bits): hi + lo
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}

}  // namespace b2
