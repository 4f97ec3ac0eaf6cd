// 32-bit products on the tensor cores from split tf32 operands.
#pragma once
#include "common.cuh"

namespace js {

// x = hi + lo as two tf32 operands (at least 20 significant bits together); three products of such halves make a 32-bit product
// on the tensor cores: a b ~ ahi bhi + ahi blo + alo bhi.  The tensor cores read the upper 19 bits of a tf32 operand, so hi
// is x itself and lo what those bits leave; the rounding conversion runs at a quarter of the rate of these two steps or less.
JS_DEVICE void tf32_split(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x);
  lo = __float_as_uint(x - __uint_as_float(hi & 0xffffe000u));
}
// d += a b, a 16 x 8 (row), b 8 x 8 (col), fp32 accumulators.  With gr = lane / 4, qd = lane % 4: a = rows gr, gr + 8 at column qd, then
// at column qd + 4; b = rows qd, qd + 4 at column gr; d = row gr at columns 2 qd, 2 qd + 1, then row gr + 8.
JS_DEVICE void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// d = a b
JS_DEVICE void mma_tf32_first(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%10, %10, %10, %10};"
      : "=f"(d[0]), "=f"(d[1]), "=f"(d[2]), "=f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1), "f"(0.f));
}

}  // namespace js
