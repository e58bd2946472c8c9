// f32 products on the tensor cores: every operand as a pair of tf32 terms (x = hi + lo to 2^-21; hi hi + hi lo +
// lo hi, the "3xTF32" scheme of CUTLASS's examples), mma.sync m16n8k8 fragments.
#pragma once

#include <stdint.h>

namespace dyn {

struct Tf32Pair {
  uint32_t hi, lo;
};
__device__ __forceinline__ Tf32Pair tf32_split(float x) {
  // integer arithmetic on the bits (hi to nearest, lo cut off): conversions run at a fraction of its rate
  Tf32Pair p;
  p.hi = (__float_as_uint(x) + 0x1000u) & 0xffffe000u;
  p.lo = __float_as_uint(x - __uint_as_float(p.hi)) & 0xffffe000u;
  return p;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct AFrag {
  uint32_t hi[4], lo[4];
};
__device__ __forceinline__ void split_into(AFrag& f, int i, float x) {
  const Tf32Pair p = tf32_split(x);
  f.hi[i] = p.hi, f.lo[i] = p.lo;
}
// c[nt] += a b[nt] for NT column tiles of one k-step whose operands are split already. Term by term, so that the
// products of consecutive instructions are independent.
template <int NT>
__device__ __forceinline__ void mma3_split(float (&c)[NT][4], const AFrag& a, const Tf32Pair (&p)[NT], const Tf32Pair (&q)[NT]) {
#pragma unroll
  for (int nt = 0; nt < NT; nt++) mma_tf32(c[nt], a.lo, p[nt].hi, q[nt].hi);
#pragma unroll
  for (int nt = 0; nt < NT; nt++) mma_tf32(c[nt], a.hi, p[nt].lo, q[nt].lo);
#pragma unroll
  for (int nt = 0; nt < NT; nt++) mma_tf32(c[nt], a.hi, p[nt].hi, q[nt].hi);
}
// The same with b(nt, 0 / 1), the tile's two operand values, split here.
template <int NT, class B>
__device__ __forceinline__ void mma3(float (&c)[NT][4], const AFrag& a, B b) {
  Tf32Pair p[NT], q[NT];
#pragma unroll
  for (int nt = 0; nt < NT; nt++) p[nt] = tf32_split(b(nt, 0)), q[nt] = tf32_split(b(nt, 1));
  mma3_split<NT>(c, a, p, q);
}

}  // namespace dyn
