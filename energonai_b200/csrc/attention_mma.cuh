// Building blocks of the mma.sync attention kernels (attention.cu, attention_group.cu): swizzled
// 16-bit tiles, their loads, and the warp-level product.
#pragma once

#include "common.cuh"

namespace eb {
namespace {

__device__ __forceinline__ uint32_t smem_u32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src, bool valid) {
  const int bytes = valid ? 16 : 0;   // src-size 0 zero-fills the destination
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
template <typename T> __device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1);
template <> __device__ __forceinline__ void mma16816<__half>(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
template <> __device__ __forceinline__ void mma16816<__nv_bfloat16>(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Byte offset of 16-byte chunk `chunk` of row `row` in a [rows][D] 16-bit tile whose chunks are
// XOR-swizzled with the row index (conflict-free ldmatrix and cp.async).
template <int D> __device__ __forceinline__ uint32_t tile_off(int row, int chunk) {
  return (uint32_t)(row * D * 2 + ((chunk ^ (row & 7)) << 4));
}

// The 16 rows [warp*16, warp*16+16) of a tile, loaded by that warp alone: the generation-step
// kernel gives every warp its own slice of each tile, so the warps need no CTA-wide barrier
// inside the key loop.  Lane l moves chunk l % (D/8) of rows l / (D/8) + k * (32 / (D/8)).
template <typename T, int D>
__device__ __forceinline__ void load_warp_rows(uint32_t tile, const T *base, long long rs, int row0, int row_end,
                                               int warp, int lane) {
  constexpr int kChunks = D / 8, kRowStep = 32 / kChunks, kIters = 16 / kRowStep;
  const int c = lane % kChunks, rl = lane / kChunks;
  int row = row0 + warp * 16 + rl;
  const T *src = base + (long long)row * rs + c * 8;
  const long long src_step = (long long)kRowStep * rs;
  const uint32_t dst0 = tile + (uint32_t)((warp * 16 + rl) * D * 2);
#pragma unroll
  for (int k = 0; k < kIters; ++k) {
    const bool ok = row < row_end;
    // swizzle term of row warp*16 + rl + k*kRowStep (warp*16 is a multiple of 8)
    const uint32_t dst = dst0 + (uint32_t)(k * kRowStep * D * 2) + (uint32_t)((c ^ ((rl + k * kRowStep) & 7)) << 4);
    cp_async16(dst, ok ? src : base, ok);
    src += src_step;
    row += kRowStep;
  }
}

// The same for a ring of R rows: entry i of the tile is position rel0 + i of `count`, the first of them in
// row r0 (count <= R, so a position wraps at most once).
template <typename T, int D>
__device__ __forceinline__ void load_warp_ring(uint32_t tile, const T *base, long long rs, int rel0, int count, int r0, int R, int warp, int lane) {
  constexpr int kChunks = D / 8, kRowStep = 32 / kChunks, kIters = 16 / kRowStep;
  const int c = lane % kChunks, rl = lane / kChunks;
#pragma unroll
  for (int k = 0; k < kIters; ++k) {
    const int i = warp * 16 + rl + k * kRowStep, rel = rel0 + i;
    const bool ok = rel < count;
    int r = r0 + rel;
    if (r >= R) r -= R;
    cp_async16(tile + tile_off<D>(i, c), ok ? base + (long long)r * rs + c * 8 : base, ok);
  }
}

// The same with `kept` rows in front: entry rel < kept is row rel, the others follow in the ring, which begins at
// row ring0 (its first wanted row is r0).
template <typename T, int D>
__device__ __forceinline__ void load_warp_kept(uint32_t tile, const T *base, long long rs, int rel0, int count, int kept, int ring0, int r0, int R, int warp,
                                               int lane) {
  constexpr int kChunks = D / 8, kRowStep = 32 / kChunks, kIters = 16 / kRowStep;
  const int c = lane % kChunks, rl = lane / kChunks;
#pragma unroll
  for (int k = 0; k < kIters; ++k) {
    const int i = warp * 16 + rl + k * kRowStep, rel = rel0 + i;
    const bool ok = rel < count;
    int r = r0 + rel - kept;
    if (r >= R) r -= R;
    r = rel < kept ? rel : ring0 + r;
    cp_async16(tile + tile_off<D>(i, c), ok ? base + (long long)r * rs + c * 8 : base, ok);
  }
}

}  // namespace
}  // namespace eb
