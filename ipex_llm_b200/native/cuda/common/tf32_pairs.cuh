// 32-bit products on the tensor cores: every fp32 operand is split into two tf32 parts (22 bits together), a product takes
// three mma.sync with fp32 accumulation, or two when one operand is exact in a single part (16-bit values are).
#pragma once
#include <stdint.h>

#include "../tcgen05_common.cuh"

namespace {

__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xFFFFE000u;
  lo = __float_as_uint(x - __uint_as_float(hi));       // exact; the instruction reads its upper 19 bits
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
struct FragA { uint32_t hi[4], lo[4]; };
struct FragB { uint32_t hi[2], lo[2]; };
// lane (g, t): A rows g, g + 8 and columns t, t + 4; B row (k) t, t + 4 of column g; C rows g, g + 8, columns 2t, 2t + 1
template <typename F>
__device__ __forceinline__ FragA frag_a(F&& at, int g, int t) {
  FragA f;
  split_tf32(at(g, t), f.hi[0], f.lo[0]);
  split_tf32(at(g + 8, t), f.hi[1], f.lo[1]);
  split_tf32(at(g, t + 4), f.hi[2], f.lo[2]);
  split_tf32(at(g + 8, t + 4), f.hi[3], f.lo[3]);
  return f;
}
template <typename F>
__device__ __forceinline__ FragB frag_b(F&& at, int g, int t) {
  FragB f;
  split_tf32(at(t, g), f.hi[0], f.lo[0]);
  split_tf32(at(t + 4, g), f.hi[1], f.lo[1]);
  return f;
}
// independent accumulators for the main and the two correction products: three short chains instead of a long one
struct Acc {
  float m[4], x[4], y[4];
  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int i = 0; i < 4; ++i) m[i] = x[i] = y[i] = 0.f;
  }
  __device__ __forceinline__ void mac(const FragA& a, const FragB& b) {
    mma_tf32(m, a.hi, b.hi);
    mma_tf32(x, a.hi, b.lo);
    mma_tf32(y, a.lo, b.hi);
  }
  __device__ __forceinline__ float get(int i) const { return m[i] + (x[i] + y[i]); }
};

// c += a b with both operands in two parts, or with an a that a single part holds exactly
__device__ __forceinline__ void mac3(float (&c)[4], const FragA& a, const FragB& b) {
  mma_tf32(c, a.lo, b.hi);
  mma_tf32(c, a.hi, b.lo);
  mma_tf32(c, a.hi, b.hi);
}
__device__ __forceinline__ void mac2(float (&c)[4], const uint32_t (&a)[4], const FragB& b) {
  mma_tf32(c, a, b.lo);
  mma_tf32(c, a, b.hi);
}

// bytes of global memory into shared memory, reported to an mbarrier: 16-byte boundaries and sizes
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                   tc5::smem_u32(dst)), "l"(src), "r"(bytes), "r"(tc5::smem_u32(bar))
               : "memory");
}

}  // namespace
