// tf32 tensor-core tiles with 32-bit accumulation.
#pragma once
#include "common.cuh"

namespace pie {

__device__ __forceinline__ uint32_t tf32(float x) {
    uint32_t r;
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(x));
    return r;
}
__device__ __forceinline__ float tf32_f(float x) { return __uint_as_float(tf32(x)); }
// C (16 x 8) += A (16 x 8, row) B (8 x 8, col); lane (g = lane / 4, t = lane % 4) holds A (g | g + 8, t | t + 4),
// B (t | t + 4, g) and C (g | g + 8, 2 t | 2 t + 1). Operands are already rounded to tf32.
__device__ __forceinline__ void mma_tf32(float (&c)[4], const float (&a)[4], float b0, float b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])),
                   "r"(__float_as_uint(b0)), "r"(__float_as_uint(b1)));
}

}  // namespace pie
