// Warp-level tensor-core helpers of the hybrid family's kernels: asynchronous 16-byte copies to shared memory, 8x8 matrix
// loads, the m16n8k16 bf16 product with fp32 sums, and the split of a pair of fp32 numbers into bf16 plus bf16 remainder.
#pragma once
#include "hybrid_common.cuh"

namespace hyb {

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
// 16 bytes to shared memory; valid == false writes zeros and reads nothing
__device__ __forceinline__ void cp16(bf16* dst, const bf16* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0));
}
// How `threads` threads share the 16-byte groups of rows that are `per` groups wide: a thread keeps its group and walks rows
// r, r + step, ..; worked out once, so that a copy inside a loop costs an addition.  Needs per <= threads.
struct RowCopy {
  int r, c, step;
  bool on;
  __device__ __forceinline__ RowCopy(int per, int tid, int threads) {
    step = threads / per;
    r = tid / per;
    c = (tid - r * per) * 8;
    on = r < step;
  }
  // rows [0, rows) of src (row length `stride`) to dst (row length ld); rows from `live` on, and groups from column `cols` on, become zero
  __device__ __forceinline__ void run(bf16* dst, int ld, const bf16* src, long long stride, int rows, int live, int cols) const {
    if (!on) return;
    const bool in = c < cols;
    const bf16* p = src + (size_t)r * stride + c;
    bf16* d = dst + r * ld + c;
    const size_t ps = (size_t)step * stride;
    const int ds = step * ld;
#pragma unroll 4
    for (int j = r; j < rows; j += step, p += ps, d += ds) {
      const bool ok = in && j < live;
      cp16(d, ok ? p : src, ok);
    }
  }
};
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N)); }
__device__ __forceinline__ void ldm4(uint32_t* r, const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldm4t(uint32_t* r, const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldm2(uint32_t* r, const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldm2t(uint32_t* r, const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}
// c[16 x 8] += a[16 x 16] b[16 x 8]; lane (g = lane / 4, t = lane % 4) holds c = {(g, 2t), (g, 2t+1), (g+8, 2t), (g+8, 2t+1)}
__device__ __forceinline__ void mma(float* c, const uint32_t* a, const uint32_t* b) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  __nv_bfloat162 l = __floats2bfloat162_rn(x - __bfloat162float(h.x), y - __bfloat162float(h.y));
  hi = *reinterpret_cast<uint32_t*>(&h);
  lo = *reinterpret_cast<uint32_t*>(&l);
}

}  // namespace hyb
