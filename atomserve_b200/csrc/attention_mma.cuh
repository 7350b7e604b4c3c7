// What the mma.sync attention kernels share: asynchronous copies into shared memory, fragment loads,
// the bfloat16 tensor-core instruction, swizzled tiles, and the walk from a flat row to its request.
#pragma once

#include "common.cuh"

namespace asb {
namespace mma {

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return (uint32_t)__cvta_generic_to_shared(p);
}

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int bytes = valid ? 16 : 0;  // 0: the 16 bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;\n" ::"n"(N));
}

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// Shared-memory tile of `rows` x HD bfloat16, 16-byte chunks XOR-swizzled by the row.
template <int HD>
__device__ __forceinline__ uint32_t tile_offset(int row, int chunk) {
  return (uint32_t)(row * (HD * 2) + ((chunk ^ (row & 7)) << 4));
}

// One warp: acc[HD/8][4] += P (16 rows x 16 keys, as an A fragment) . V (16 keys x HD).
template <int HD>
__device__ __forceinline__ void pv_16keys(float (&acc)[HD / 8][4], const uint32_t (&pf)[4],
                                          uint32_t v_tile, int key0, int lane) {
  const int vrow = key0 + (lane & 7) + (((lane >> 3) & 1) << 3);
  const int vchunk = lane >> 4;
#pragma unroll
  for (int nc = 0; nc < HD / 16; ++nc) {
    uint32_t b[4];
    ldmatrix_x4_trans(b, v_tile + tile_offset<HD>(vrow, nc * 2 + vchunk));
    mma_bf16(acc[nc * 2], pf, b[0], b[1]);
    mma_bf16(acc[nc * 2 + 1], pf, b[2], b[3]);
  }
}

__device__ __forceinline__ int find_request(const int* req_q_start, int R, int row) {
  int lo = 0, hi = R - 1;  // the last r with req_q_start[r] <= row
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (req_q_start[mid] <= row) lo = mid; else hi = mid - 1;
  }
  return lo;
}

}  // namespace mma
}  // namespace asb
